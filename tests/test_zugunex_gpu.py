"""Zugunex on the GPU: each new kernel or option alone against the plain function of its mechanism
(tests/plain_zugunex.py), then whole models through replay, the engine and the command line."""
import json
import math
import os
import subprocess
import sys
from types import SimpleNamespace

import pytest
import torch

import plain_zugunex as plain
import zugunex_helpers as zh
from helpers import random_tokens, run_steps

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32, BF16, F64 = torch.float32, torch.bfloat16, torch.float64
DTYPES = [F32, BF16]


@pytest.fixture(scope="module")
def ops():
    from qwen_engine_b200 import ops as _ops
    _ops.lib()
    return _ops


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("zugunex_gpu")
    return {name: zh.make_folder(str(root / name), name) for name in zh.ZUGUNEX}


def _close(got, want, dtype, what="", tol=None):
    got, want = got.detach().to("cpu", F64), want.to(F64)
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} vs {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: not finite"
    tol = tol if tol is not None else {F32: 2e-5, BF16: 1.5e-2}[dtype]
    err = float((got - want).abs().max())
    scale = max(1e-6, float(want.abs().max()))
    assert err <= tol * scale, f"{what}: max |diff| {err:.3e} > {tol} * {scale:.3e}"


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


# ---- products with an activation of their sums ------------------------------------------------------------------------
PLAIN_ACT = {"gelu_tanh": plain.gelu_tanh, "relu_squared": plain.relu_squared, "silu": lambda z: z * torch.sigmoid(z)}


@pytest.mark.parametrize("dtype,M,N,K", [(F32, 5, 40, 24), (F32, 130, 77, 50), (BF16, 3, 96, 64), (BF16, 1, 1024, 2048), (BF16, 9, 520, 4096),
                                         (BF16, 40, 4096, 256), (BF16, 40, 512, 1024), (BF16, 130, 384, 256), (BF16, 100, 3072, 512),
                                         (BF16, 1500, 3072, 256), (BF16, 600, 512, 4096), (BF16, 2100, 130, 64), (BF16, 7, 33, 22)])
@pytest.mark.parametrize("act", sorted(PLAIN_ACT))
def test_a_product_with_an_activation_in_its_epilogue(ops, dtype, M, N, K, act):
    g = torch.Generator().manual_seed(M + N + K)
    x = torch.randn(M, K, generator=g).to(dtype)
    w = (torch.randn(N, K, generator=g) / math.sqrt(K) * 1.5).to(dtype)
    want = PLAIN_ACT[act](x.double() @ w.double().T)
    for out_dtype in (dtype, F32):
        out = torch.full((M, N), float("nan"), dtype=out_dtype, device=DEV)
        ops.linear(x.to(DEV), w.to(DEV), out, activation=act)
        _close(out, want, dtype, f"{act} into {out_dtype}", tol={F32: 1e-5, BF16: 6e-3 if out_dtype == BF16 else 1e-3}[dtype])
    assert ops.device_status() == {}
    with pytest.raises(ops.KernelRefused, match="unknown activation"):
        ops.linear(x.to(DEV), w.to(DEV), out, activation="relu")


def test_the_embedding_leaves_its_rows_in_the_compute_type_too(ops):
    g = torch.Generator().manual_seed(1)
    for dtype, H in ((BF16, 40), (BF16, 1030), (F32, 24)):
        table = torch.randn(30, H, generator=g).to(dtype).to(DEV)
        ids = _i32([0, 29, 7, 7, 12])
        stream = ops.ResidualStream(torch.empty(5, H, device=DEV), torch.empty(5, H, device=DEV, dtype=dtype), None,
                                    torch.empty(5, H, device=DEV, dtype=dtype))
        ops.embedding(ids, table, stream)
        assert stream.copy_current and torch.equal(stream.copy, table[ids.long()]) and torch.equal(stream.resid, table[ids.long()].float())
        # somebody else changed the stream: the copy is made anew when it is asked for
        stream.resid.mul_(1.1)
        stream.copy_current = False
        assert torch.equal(stream.rounded(), stream.resid.to(dtype)) and stream.copy_current


# ---- latent attention: per token and per head --------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dn,R,Dr", [(3, 8, 24, 8), (1, 16, 16, 16), (8, 64, 96, 32)])
def test_a_layer_that_reads_anothers_cache_only_turns_its_queries(ops, dtype, H, dn, R, Dr):
    g = torch.Generator().manual_seed(H + R)
    T, D, base = 13, R + Dr, 200.0
    q = torch.randn(T, H * (dn + Dr) + 5, generator=g).to(dtype)
    positions = torch.randint(0, 2000, (T,), generator=g, dtype=torch.int32)
    inv = (base ** (-2.0 * torch.arange(Dr // 2, dtype=F64) / Dr)).to(F32)
    cache = torch.full((3, 1, 1, 8, D), 7.0, dtype=dtype, device=DEV)
    qlat = torch.full((T, H * D), 3.0, dtype=dtype, device=DEV)
    ops.latent_prepare(None, q.to(DEV)[:, :H * (dn + Dr)], None, 0.0, positions.to(DEV), inv.to(DEV), Dr, cache, _i32([-1] * T), qlat,
                       H, dn, R, Dr, write_kv=False)
    assert bool((cache == 7.0).all()) and bool((qlat.reshape(T, H, D)[:, :, :R] == 3.0).all())
    # the kernels turn half-split pairs: the rows of the interleaved channels are reordered at load
    order = list(range(0, Dr, 2)) + list(range(1, Dr, 2))
    back = torch.empty(Dr, dtype=torch.long)
    back[order] = torch.arange(Dr)
    part = q.double()[:, :H * (dn + Dr)].reshape(T, H, dn + Dr)[:, :, dn:]
    want = plain.rotate_interleaved(part[..., back], positions, base, Dr)[..., order]
    _close(qlat.reshape(T, H, D)[:, :, R:], want, dtype, "rotated parts", tol={F32: 5e-4, BF16: 1.5e-2}[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,H,N,K", [(1, 3, 24, 8), (70, 2, 10, 6), (130, 8, 64, 32), (8, 16, 128, 192), (33, 5, 129, 65), (300, 3, 200, 72),
                                     (65, 16, 192, 128), (1000, 2, 256, 264), (129, 5, 40, 8), (2050, 16, 128, 192), (70, 4, 520, 64)])
def test_a_product_per_head_with_a_gate_per_head(ops, dtype, M, H, N, K):
    g = torch.Generator().manual_seed(M + N)
    xs = K + (8 if K % 8 == 0 else 3)
    x = torch.randn(M, H * xs, generator=g).to(dtype)
    w = (torch.randn(H, N, K, generator=g) / math.sqrt(K)).to(dtype)
    wide = (torch.randn(M, H + 6, generator=g) * 4).to(dtype)
    out = torch.empty(M, H * N, dtype=dtype, device=DEV)
    ops.head_linear(x.to(DEV), w.to(DEV), out, xs, N, gate=wide.to(DEV)[:, 2:2 + H])
    xh = torch.stack([x[:, h * xs:h * xs + K] for h in range(H)], dim=1).double()
    want = torch.einsum("mhk,hnk->mhn", xh, w.double()) * torch.sigmoid(wide.double()[:, 2:2 + H, None])
    _close(out.reshape(M, H, N), want, dtype, "gated heads")
    # heads further apart in the output than they are wide: what lies between them stays as it was
    apart = torch.full((M, H * (N + 8) + 8), 9.0, dtype=dtype, device=DEV)
    ops.head_linear(x.to(DEV), w.to(DEV), apart[:, :H * (N + 8)], xs, N + 8)
    got = apart[:, :H * (N + 8)].reshape(M, H, N + 8)
    _close(got[:, :, :N], torch.einsum("mhk,hnk->mhn", xh, w.double()), dtype, "heads")
    assert bool((got[:, :, N:] == 9.0).all()) and bool((apart[:, H * (N + 8):] == 9.0).all()) and ops.device_status() == {}


# ---- attention over a latent cache with a window and a sink ----------------------------------------------------------------
def _case(H, D, P, q_lens, ctx_lens, dtype, seed, window=0, spikes=()):
    """Queries, cache and block tables; pages whose tokens no query sees hold a large number.  ``spikes``: (request, query's
    index, key's position, head): that key's channels point where that query does, so that its score stands out."""
    g = torch.Generator().manual_seed(seed)
    blocks = [-(-(c + n) // P) for c, n in zip(ctx_lens, q_lens)]
    n_pages = sum(blocks) + 2
    perm = iter(torch.randperm(n_pages, generator=g).tolist())
    table = torch.zeros((len(q_lens), max(blocks)), dtype=torch.int32)
    cache = torch.full((n_pages, 1, 1, P, D), 1.0e4, dtype=dtype)
    for r in range(len(q_lens)):
        first = max(0, ctx_lens[r] - window + 1) if window else 0
        for b in range(blocks[r]):
            p = next(perm)
            table[r, b] = p
            if (b + 1) * P > first:
                cache[p, 0, 0] = torch.randn(P, D, generator=g).to(dtype)
    q = torch.randn(sum(q_lens), H * D, generator=g).to(dtype)
    for r, q_index, key_pos, head in spikes:
        d = torch.randn(D, generator=g)
        d = d / d.norm()
        cache[int(table[r, key_pos // P]), 0, 0, key_pos % P] = (d * 8.0).to(dtype)
        q[sum(q_lens[:r]) + q_index, head * D:(head + 1) * D] = (d * 8.0 * math.sqrt(D)).to(dtype)
    return q, cache, table


def _plain_rows(q, cache, table, H, D, R, P, q_lens, ctx_lens, scale, window, sinks):
    out = torch.zeros(q.shape[0], H, R, dtype=F64)
    row = 0
    for r, (n, c) in enumerate(zip(q_lens, ctx_lens)):
        pos = torch.arange(c + n)
        keys = cache[table[r, pos // P].long(), 0, 0, pos % P].double()
        allowed = plain.window_mask(c + n, window or None)[c:]
        for h in range(H):
            s = q[row:row + n, h * D:(h + 1) * D].double() @ keys.T * scale
            out[row:row + n, h] = plain.softmax_with_sink(s, allowed, sinks[h].double()) @ keys[:, :R]
        row += n
    return out


def _run(ops, q, cache, table, H, D, P, q_lens, ctx_lens, scale, window, sinks, dtype, fast, uniform=None):
    from qwen_engine_b200.engine.runner import ModelRunner
    from qwen_engine_b200.parts.base import Arena
    geos = ((H, 1, D, window, False, 1),) if fast else ()
    plan = ops.plan_attention(list(q_lens), list(ctx_lens), P, geos, dtype, **({} if uniform is None else {"uniform_splits": {geos[0]: uniform}}))
    devplan = ModelRunner._device_plan(plan, {"plan_" + k: _i32(v) for k, v in plan.items()}, geos)
    cu = [0]
    for n in q_lens:
        cu.append(cu[-1] + n)
    ctx = SimpleNamespace(cu_q=_i32(cu), ctx_lens=_i32(list(ctx_lens)), slot_ids=_i32([0] * len(q_lens)), num_reqs=len(q_lens),
                          max_q_len=max(q_lens), q_lens_host=list(q_lens), ctx_lens_host=list(ctx_lens), attn_plan=devplan, arena=Arena(DEV))
    out = torch.zeros(q.shape[0], H * D, dtype=dtype, device=DEV)
    ops.paged_attention(q.to(DEV), cache.to(DEV), table.to(DEV), ctx, out, scale, window, H, 1, D, sinks=sinks.to(DEV))
    torch.cuda.synchronize()
    assert ops.device_status() == {}
    return out, ops.last_attention_kernel


SHAPES = [(3, 32, 24, 4), (1, 48, 40, 16), (2, 15, 9, 8), (8, 128, 96, 16), (16, 256, 192, 16), (6, 160, 128, 16), (20, 64, 48, 8), (5, 352, 320, 16),
          (16, 128, 64, 16), (12, 192, 128, 32)]
BATCHES = [([30], [0]), ([1], [95]), ([1, 1, 1], [4, 77, 31]), ([7, 1, 2, 40], [9, 40, 0, 63]), ([2, 33], [64, 31]), ([150], [20]),
           ([1] * 8, [0, 1, 2, 300, 47, 48, 600, 15]), ([1, 90], [700, 5])]


@pytest.mark.parametrize("dtype,fast", [(F32, False), (BF16, False), (BF16, True)])
@pytest.mark.parametrize("H,D,R,P", SHAPES)
@pytest.mark.parametrize("window", [0, 1, 17, 48, 100])
def test_attention_over_latents_with_a_window_and_sinks(ops, dtype, fast, H, D, R, P, window):
    if dtype == BF16 and not fast and window not in (0, 48):
        pytest.skip("the generic kernel's windows are covered in float32")
    scale = 1.1 / math.sqrt(D)
    g = torch.Generator().manual_seed(D)
    sinks = torch.randn(H, generator=g) * 2.0 + 1.0
    for i, (q_lens, ctx_lens) in enumerate(BATCHES):
        q, cache, table = _case(H, D, P, q_lens, ctx_lens, dtype, 10 * D + i, window)
        got, kernel = _run(ops, q, cache, table, H, D, P, q_lens, ctx_lens, scale, window, sinks, dtype, fast)
        want = _plain_rows(q, cache, table, H, D, R, P, q_lens, ctx_lens, scale, window, sinks)
        _close(got.reshape(-1, H, D)[:, :, :R], want, dtype, f"window {window} on {kernel}, batch {i}", tol={F32: 2e-5, BF16: 2e-2}[dtype])
        if fast and D % 16 == 0 and D <= 256:
            assert kernel != "paged_attention_generic"


@pytest.mark.parametrize("H,D,R,P", [(16, 256, 192, 16), (8, 128, 96, 16), (6, 160, 128, 16), (3, 64, 40, 8), (16, 192, 128, 16), (1, 80, 64, 16)])
@pytest.mark.parametrize("parts", [1, 2, 3, 4, 8])
def test_decoded_tokens_with_their_contexts_in_parts(ops, H, D, R, P, parts):
    """Steps of single tokens whose contexts are cut into the same number of parts (as in steps replayed from a CUDA graph):
    parts without keys, windows that begin inside a part, the sink counted once."""
    g = torch.Generator().manual_seed(D + parts)
    sinks = torch.randn(H, generator=g) * 2.0 + 1.0
    scale = 1.1 / math.sqrt(D)
    for window in (0, 17, 300):
        for q_lens, ctx_lens in (([1] * 7, [0, 1, 15, 16, 2500, 700, 63]), ([1], [1000])):
            q, cache, table = _case(H, D, P, q_lens, ctx_lens, BF16, D + window, window)
            got, kernel = _run(ops, q, cache, table, H, D, P, q_lens, ctx_lens, scale, window, sinks, BF16, True, uniform=parts)
            want = _plain_rows(q, cache, table, H, D, R, P, q_lens, ctx_lens, scale, window, sinks)
            _close(got.reshape(-1, H, D)[:, :, :R], want, BF16, f"{parts} parts, window {window} on {kernel}", tol=2e-2)


@pytest.mark.parametrize("dtype,fast", [(F32, False), (BF16, True)])
@pytest.mark.parametrize("H,D,R,P", [(4, 128, 96, 16), (2, 48, 40, 8), (16, 256, 192, 16), (6, 160, 128, 16)])
@pytest.mark.parametrize("window", [64, 72, 200])
@pytest.mark.parametrize("decoded", [False, True])
def test_keys_just_inside_and_just_outside_the_window(ops, dtype, fast, H, D, R, P, window, decoded):
    """A key whose score stands out by far, as the window's last token (it takes the row), one token further back (it is
    not seen at all), at the query's own position, and at a page's first and last place inside the window."""
    own = 3 * window + 5
    inside, outside = own - window + 1, own - window
    page_first = -(-inside // P) * P
    for key_pos, seen in ((inside, True), (outside, False), (own, True), (page_first, True), (page_first + P - 1, True)):
        q_lens, ctx_lens = ([1, 1], [own, 7]) if decoded else ([40, 90], [own - 39, 0])
        q_index = 0 if decoded else 39
        q, cache, table = _case(H, D, P, q_lens, ctx_lens, dtype, 5 + key_pos, 0, [(0, q_index, key_pos, H - 1)])
        sinks = torch.full((H,), 0.5)
        got, kernel = _run(ops, q, cache, table, H, D, P, q_lens, ctx_lens, 1.0 / math.sqrt(D), window, sinks, dtype, fast)
        want = _plain_rows(q, cache, table, H, D, R, P, q_lens, ctx_lens, 1.0 / math.sqrt(D), window, sinks)
        got = got.reshape(-1, H, D)[:, :, :R]
        _close(got, want, dtype, f"key at {key_pos} on {kernel}", tol={F32: 2e-5, BF16: 2e-2}[dtype])
        key = cache[int(table[0, key_pos // P]), 0, 0, key_pos % P, :R].float()
        near = float((got[q_index, H - 1].float().cpu() - key).abs().max()) < 0.05
        assert near == seen, f"key at {key_pos}"


def test_a_sink_that_takes_nearly_everything(ops):
    """A large sink leaves the output a small share; a very negative one leaves the plain softmax."""
    H, D, R, P = 4, 128, 96, 16
    q_lens, ctx_lens = [1, 70, 3], [200, 10, 0]
    for dtype, fast in ((F32, False), (BF16, True)):
        q, cache, table = _case(H, D, P, q_lens, ctx_lens, dtype, 3)
        sinks = torch.tensor([12.0, -60.0, 0.0, 5.0])
        got, kernel = _run(ops, q, cache, table, H, D, P, q_lens, ctx_lens, 1.0 / math.sqrt(D), 50, sinks, dtype, fast)
        want = _plain_rows(q, cache, table, H, D, R, P, q_lens, ctx_lens, 1.0 / math.sqrt(D), 50, sinks)
        for h in range(H):                               # head by head: the outputs differ by orders of magnitude
            _close(got.reshape(-1, H, D)[:, h, :R], want[:, h], dtype, f"head {h} on {kernel}", tol={F32: 2e-5, BF16: 2e-2}[dtype])


# ---- experts ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,E,top,pieces,scale", [(1, 40, 2, 1, 1, 1.0), (9, 64, 5, 2, 0, 1.5), (70, 96, 8, 3, 2, 2.5), (33, 50, 200, 8, 3, 0.3), (5, 32, 4, 4, 1, 1.2)])
def test_router_whose_weights_sum_to_one(ops, dtype, T, W, E, top, pieces, scale):
    g = torch.Generator().manual_seed(T + E)
    x = torch.randn(T, W, generator=g).to(dtype)
    w = torch.randn(E + (pieces > 0), W, generator=g) * 0.3
    idx = torch.full((T, top + pieces), -7, dtype=torch.int32, device=DEV)
    wgt = torch.empty(T, top + pieces, dtype=F32, device=DEV)
    ops.moe_route(x.to(DEV), w.to(DEV), None, idx, wgt, scoring="sigmoid_sum", weight_scale=scale, n_always=pieces)
    want_idx, want_w = plain.route(x.double(), {"router": w[:E].double()}, "", dict(top=top, scale=scale))
    assert torch.equal(idx.cpu()[:, :top].long(), want_idx)
    _close(wgt[:, :top], want_w, F32, "weights", tol=1e-5)
    if pieces:
        assert torch.equal(idx.cpu()[:, top:], torch.arange(E, E + pieces, dtype=torch.int32).expand(T, pieces))
        _close(wgt[:, top:], torch.sigmoid(x.double() @ w[E:].double().T).expand(T, pieces), F32, "shared weight", tol=1e-5)


def _experts_part(ops, W, ff, experts, top, shared, scale, dtype, seed):
    from qwen_engine_b200.parts.moe import RoutedExperts
    g = torch.Generator().manual_seed(seed)
    w = {f"e{e}.{n}": torch.randn(*s, generator=g) / math.sqrt(s[1]) for e in range(experts) for n, s in (("up", (ff, W)), ("down", (W, ff)))}
    w.update({"shared.up": torch.randn(shared, W, generator=g) / math.sqrt(W), "shared.down": torch.randn(W, shared, generator=g) / math.sqrt(shared),
              "shared.sg": torch.randn(1, W, generator=g) / math.sqrt(W), "router": torch.randn(experts, W, generator=g) / math.sqrt(W)})
    w = {k: v.to(BF16).float() for k, v in w.items()}
    part = RoutedExperts(W, ff, experts, top, activation="relu_squared", names=("up", "down"), router_bias_name=None, scoring="sigmoid_sum",
                         weight_scale=scale, gated=False, shared_size=shared)
    part.load("", SimpleNamespace(get=lambda n: w[n]), dtype, DEV)
    return part, w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,ff,E,top,shared", [(40, 12, 2, 1, 20), (64, 24, 5, 2, 24), (128, 64, 16, 4, 100), (256, 512, 8, 2, 512), (96, 40, 3, 3, 16),
                                               (200, 8, 64, 6, 30), (512, 1536, 4, 1, 768)])
def test_experts_without_a_gate_beside_a_shared_one(ops, dtype, W, ff, E, top, shared):
    """Steps of a few rows and of many; experts without any token among them; a token's row does not depend on the others."""
    from qwen_engine_b200.parts.base import Arena
    part, w = _experts_part(ops, W, ff, E, top, shared, 1.6, dtype, W + ff)
    mlp = dict(kind="moe", router=dict(experts=E, top=top, scale=1.6), expert=dict(ff=ff), shared=dict(ff=shared))
    g = torch.Generator().manual_seed(ff)
    base = torch.randn(300, W, generator=g)
    base[:150] = base[:1] + 0.05 * base[:150]            # many tokens that choose alike: crowded and empty experts
    x = base.to(dtype)
    margins: list = []
    want = plain.mixture_of_experts(x.double(), {k: v.double() for k, v in w.items()}, "", mlp, margins)
    clear = margins[0] > 1e-3
    assert int(clear.sum()) > 200

    def run(rows):
        out = torch.full((rows.shape[0], W), float("nan"), dtype=dtype, device=DEV)
        part.forward(SimpleNamespace(num_tokens=rows.shape[0], dtype=dtype, arena=Arena(DEV, 1 << 24)), rows.to(DEV), out)
        return out.cpu()
    for n in (300, 33, 8, 1):
        for first in ((0, 140) if n < 100 else (0,)):
            keep = clear[first:first + n]
            got = run(x[first:first + n])
            _close(got[keep], want[first:first + n][keep], dtype, f"{n} rows", tol={F32: 2e-5, BF16: 2e-2}[dtype])
    assert torch.equal(run(x[:1])[0], run(x[:8])[0])
    assert ops.device_status() == {}


@pytest.mark.parametrize("W,ff,counts", [(64, 40, [0, 1, 127, 128, 129, 256, 0, 300]), (128, 264, [513]), (520, 72, [0, 0, 640, 3]),
                                         (8, 8, [600, 1]), (256, 512, [130] * 40)])
def test_grouped_products_of_many_rows_at_the_tiles_borders(ops, W, ff, counts):
    """Experts whose rows fill tiles exactly, miss them by one, or are none; one choice a token, so a row is one expert's."""
    from qwen_engine_b200.parts.base import Arena
    g = torch.Generator().manual_seed(W + ff)
    E, T = len(counts), sum(counts)
    idx = torch.tensor([e for e, n in enumerate(counts) for _ in range(n)])[torch.randperm(T, generator=g)]
    x = torch.randn(T, W, generator=g).to(BF16)
    up = (torch.randn(E, ff, W, generator=g) / math.sqrt(W)).to(BF16)
    down = (torch.randn(E, W, ff, generator=g) / math.sqrt(ff)).to(BF16)
    wgt = torch.rand(T, 1, generator=g) + 0.5
    assert ops.moe_tc_applies(T, ff, W, W, BF16)
    outs = []
    for tc in (True, False):
        out = torch.full((T, W), float("nan"), dtype=BF16, device=DEV)
        saved, ops.MOE_TC_MIN_PAIRS = ops.MOE_TC_MIN_PAIRS, (1 if tc else 1 << 30)
        try:
            ops.moe_experts(x.to(DEV), idx.to(torch.int32)[:, None].contiguous().to(DEV), wgt.to(DEV), up.to(DEV), down.to(DEV), out, "relu_squared",
                            Arena(DEV, 1 << 24).alloc, gated=False)
        finally:
            ops.MOE_TC_MIN_PAIRS = saved
        outs.append(out)
    want = torch.empty(T, W, dtype=F64)
    for e in range(E):
        at = idx == e
        want[at] = wgt.double()[at] * (plain.relu_squared(x[at].double() @ up[e].double().T) @ down[e].double().T)
    for out in outs:
        _close(out, want, BF16, "grouped", tol=2e-2)
    assert ops.device_status() == {}


# ---- the mixer through its cache ---------------------------------------------------------------------------------------------
class _Dict:
    def __init__(self, d):
        self.d = d

    def get(self, n):
        return self.d[n]


def _mixers(m_own, m_reader, W, dtype, seed):
    """A layer with a latent and one that reads it, with their weights, as the design's layout makes them."""
    from qwen_engine_b200.config.zugunex_config import ZugunexConfig
    from qwen_engine_b200.models.zugunex import _mixer
    cfg = ZugunexConfig(vocab=10, width=W, norm_eps=1e-6)
    sizes = [m["mask"]["size"] for m in (m_own, m_reader)]
    g = torch.Generator().manual_seed(seed)
    out = []
    for m in (m_own, m_reader):
        H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        w = {"q": torch.randn(H * (dn + dr), W, generator=g) / math.sqrt(W), "uk": torch.randn(H * dn, R, generator=g) / math.sqrt(R),
             "uv": torch.randn(H * dv, R, generator=g) / math.sqrt(R), "o": torch.randn(W, H * dv, generator=g) / math.sqrt(H * dv),
             "g": torch.randn(H, W, generator=g) / math.sqrt(W) * 2.0, "sink": torch.randn(H, generator=g) + 1.0}
        if m.get("kv_from") is None:
            w.update({"dkv": torch.randn(R + dr, W, generator=g) / math.sqrt(W), "dkv.norm": 1.0 + 0.2 * torch.randn(R, generator=g)})
        w = {k: v.to(BF16).float() for k, v in w.items()}
        mixer = _mixer(cfg, m, max(sizes)).build("mixer")
        mixer.load("", _Dict(w), dtype, DEV)
        out.append((mixer, w))
    return out


def _run_mixers(ops, mixers, xs, dtype, P, portions):
    """The mixers of one cache slot over one request cut into ``portions``: each one's output rows."""
    from qwen_engine_b200.cache.manager import CacheManager
    from qwen_engine_b200.engine.runner import ModelRunner
    from qwen_engine_b200.parts.base import Arena, GroupStepView, StepContext
    total = sum(portions)
    cache = CacheManager([mixers[0].cache_spec()], P, -(-total // P) + 2, 4, dtype, DEV, poison=1.0e4)
    rc = cache.open("r")
    geos = tuple(dict.fromkeys(m.attention_geometry() for m in mixers))
    rows, done = [[] for _ in mixers], 0
    for n in portions:
        cache.append(rc, [0] * n)
        plan = ops.plan_attention([n], [done], P, geos, dtype)
        devplan = ModelRunner._device_plan(plan, {"plan_" + k: _i32(v) for k, v in plan.items()}, geos)
        table = rc.tables[0]
        ctx = StepContext(num_tokens=n, num_reqs=1, dtype=dtype, device=torch.device(DEV), page_size=P, token_ids=_i32([0] * n),
                          positions=_i32(list(range(done, done + n))), cu_q=_i32([0, n]), ctx_lens=_i32([done]), slot_ids=_i32([0]),
                          logit_rows=_i32([0]), num_logit_rows=0,
                          groups={0: GroupStepView(_i32([max(t, 0) for t in table]).view(1, len(table)), _i32(cache.slot_mapping(rc, 0)), len(table))},
                          q_lens_host=[n], ctx_lens_host=[done], arena=Arena(DEV, 1 << 26), attn_plan=devplan)
        for i, (mixer, x) in enumerate(zip(mixers, xs)):
            out = torch.empty(n, x.shape[1], dtype=dtype, device=DEV)
            mixer.forward(ctx, x[done:done + n].to(DEV), cache.layer_view(0), 0, out, i == 0)
            rows[i].append(out.float().cpu())
        torch.cuda.synchronize()
        cache.commit(rc)
        done += n
    return [torch.cat(r) for r in rows]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dn,dr,dv,R,P,windows", [(8, 64, 32, 48, 96, 16, (130, 90)), (3, 20, 12, 28, 24, 8, (40, 75)), (16, 32, 64, 64, 192, 16, (100, 101))])
@pytest.mark.parametrize("decoded", [False, True])
def test_two_layers_on_one_latent_with_windows_of_their_own(ops, dtype, H, dn, dr, dv, R, P, windows, decoded):
    """Every row of 500 tokens of a layer and of one that reads its latent, against the plain mixers.  The inputs repeat one
    token's row so that its latent stands out for the last queries: once as the last token inside the shorter window, once
    just outside it and still inside the longer one."""
    W, total = 160, 500
    short = min(windows)
    base = dict(heads=H, dim=dn, rot_dim=dr, vdim=dv, kv_rank=R, scale=2.0 / math.sqrt(dn + dr), rot=dict(base=10000.0, dims=dr))
    own = dict(base, mask=dict(size=windows[0]))
    reader = dict(base, heads=max(1, H // 2), vdim=dv + 8, mask=dict(size=windows[1]), kv_from=0)
    (m0, w0), (m1, w1) = _mixers(own, reader, W, dtype, H + R)
    g = torch.Generator().manual_seed(H)
    x0, x1 = torch.randn(total, W, generator=g), torch.randn(total, W, generator=g)
    # tokens whose latent points where the last queries of head 0 point (in both layers), at the shorter window's two sides
    for at, (w, x) in ((total - short, (w0, x0)), (total - 1 - short, (w1, x1))):
        q = (w["q"].double() @ x[-1].double()).reshape(-1, dn + dr)[0, :dn]
        want_c = w["uk"].double().reshape(-1, dn, R)[0].T @ q
        x0[at] = (torch.linalg.lstsq(w0["dkv"].double()[:R], want_c[:, None]).solution[:, 0] * 3.0 / want_c.norm()).float() * math.sqrt(R)
    x0, x1 = x0.to(dtype), x1.to(dtype)
    kept: dict = {}
    d = lambda w: {k: v.double() for k, v in w.items()}
    want = [plain.latent_attention(x0.double(), d(w0), "", own, 1e-6, kept, 0), plain.latent_attention(x1.double(), d(w1), "", reader, 1e-6, kept, 1)]
    portions = [total - 25] + [1] * 25 if decoded else [40, 2, 230, total - 272]
    got = _run_mixers(ops, (m0, m1), (x0, x1), dtype, P, portions)
    for i in range(2):
        _close(got[i], want[i], dtype, f"layer {i} on {ops.last_attention_kernel}", tol={F32: 1e-4, BF16: 4e-2}[dtype])
    # the planted keys count: with windows one token shorter the plain rows differ by far more than the tolerance
    other = plain.latent_attention(x0.double(), d(w0), "", dict(own, mask=dict(size=windows[0] - 1)), 1e-6, {}, 0)
    if windows[0] == short:
        assert float((other[-1] - want[0][-1]).abs().max()) > 0.1 * float(want[0][-1].abs().max())


# ---- whole models ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,name", [(d, n) for n in zh.ZUGUNEX for d in DTYPES])
def test_replay_against_the_plain_model(folders, dtype, name):
    folder = folders[name]
    zh.replay_cases(lambda n: zh.make_replayer(folder, name, dtype, n, poison=1.0e4), folder, name, dtype, f"{name}")


@pytest.mark.parametrize("name", ["z-a", "z-d", "z-e"])
def test_bfloat16_rows_do_not_depend_on_the_schedule(folders, name):
    """In bfloat16 a row behind a router's close call is judged loosely against the plain model; against the engine's own
    rows of the whole prompt the rows of a mixed schedule are judged tightly."""
    from helpers import live_tokens_needed, mixed_steps
    folder = folders[name]
    V = zh.vocab_of(name)
    reqs = {f"m{i}": random_tokens(V, n, 60 + i) for i, n in enumerate([40, 64, 23, 90, 17, 55])}
    steps = mixed_steps(reqs, seed=11)
    got = run_steps(zh.make_replayer(folder, name, BF16, live_tokens_needed(steps, 64), poison=1.0e4), steps)
    for rid, toks in reqs.items():
        whole = run_steps(zh.make_replayer(folder, name, BF16, 128),
                          [{"entries": [{"id": "a", "tokens": toks, "want": list(range(len(toks)))}], "end": ["a"]}])["a"]
        settled = zh.settled_positions(folder, toks, BF16)
        idx = [i for i in sorted(got[rid]) if i in settled]
        if not idx:
            continue
        err = zh.row_errors(torch.stack([got[rid][i] for i in idx]), torch.stack([whole[i] for i in idx]))
        assert float(err.max()) < 0.1, f"{name} {rid}: position {idx[int(err.argmax())]} differs by {float(err.max()):.3f}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_every_position_of_a_long_prompt_whole_and_decoded(folders, dtype):
    """Prompts of several windows at all positions: whole, and from the first token on one by one (the steps of single
    tokens are replayed from a CUDA graph): first tokens, pages' borders and windows' edges lie among them."""
    for name, n in (("z-b", 120), ("z-d", 330), ("z-e", 200)):
        folder = folders[name]
        toks = random_tokens(zh.vocab_of(name), n, 31)
        whole = [{"entries": [{"id": "a", "tokens": toks, "want": list(range(n))}], "end": ["a"]}]
        zh.check_requests(run_steps(zh.make_replayer(folder, name, dtype, 384), whole), folder, {"a": toks}, dtype, f"{name} whole")
        single = [{"entries": [{"id": "a", "tokens": [t], "want": [0]}]} for t in toks]
        rep = zh.make_replayer(folder, name, dtype, 384)
        zh.check_requests(run_steps(rep, single), folder, {"a": toks}, dtype, f"{name} decoded")
        assert rep.runner.num_graph_replays > n // 2


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt_in_portions_then_decoded(folders, dtype):
    """600 tokens: whole; and in portions of changing sizes (two tokens among them, cuts inside pages and windows) with the
    last 40 tokens one by one, beside a second request that comes and goes (its pages are used again)."""
    name = "z-d"
    folder = folders[name]
    V = zh.vocab_of(name)
    toks, other = random_tokens(V, 600, 3), random_tokens(V, 50, 4)
    want = sorted(set(range(0, 600, 7)) | set(range(560, 600)))
    whole = [{"entries": [{"id": "a", "tokens": toks, "want": want}], "end": ["a"]}]
    zh.check_requests(run_steps(zh.make_replayer(folder, name, dtype, 640), whole), folder, {"a": toks}, dtype, "whole")
    steps, p = [], 0
    for i, n in enumerate([64, 64, 100, 2, 30, 129, 16, 3, 95, 57] + [1] * 40):
        entries = [{"id": "a", "tokens": toks[p:p + n], "want": [w - p for w in want if p <= w < p + n]}]
        if i in (1, 5, 12):
            entries.append({"id": f"b{i}", "tokens": other, "want": [49]})
        steps.append({"entries": entries, "end": [f"b{i}"] if i in (1, 5, 12) else []})
        p += n
    assert p == 600
    rep = zh.make_replayer(folder, name, dtype, 704)
    got = run_steps(rep, steps)
    zh.check_requests(got, folder, {"a": toks, "b1": other, "b5": other, "b12": other}, dtype, "portions")


def test_greedy_generation_through_the_engine(folders):
    from qwen_engine_b200.sampling.params import SamplingParams
    for name in ("z-a", "z-c"):
        folder = folders[name]
        cfg, w = zh.plain_model(folder)
        V = zh.vocab_of(name)
        prompts = [random_tokens(V, n, 40 + i) for i, n in enumerate([5, 19, 33, 2, 11, 26, 47])]
        eng = zh.make_engine(folder, name, F32, max_num_seqs=3, max_num_batched_tokens=24, prefill_chunk_size=7)
        ids = [eng.add_request(p, SamplingParams(max_new_tokens=8, temperature=0.0)) for p in prompts]
        outs = {o.request_id: o for o in eng.serving()}
        for rid, p in zip(ids, prompts):
            assert list(outs[rid].output_token_ids) == plain.greedy(cfg, w, p, 8), f"{name}: prompt of {len(p)} tokens"
        assert eng.cache.slots.num_free == eng.cache.slots.num_slots and eng.cache.pages_in_use() == 0


def test_the_command_line_replays_a_trace(folders, tmp_path):
    name = "z-c"
    folder = folders[name]
    toks = random_tokens(zh.vocab_of(name), 30, 8)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:21], "want": [0, 20]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[21:23], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[23:], "want": [6]}, {"id": "y", "tokens": toks[:4], "want": [3]}],
              "end": ["x", "y"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (out / "1.f32").exists()
    V = zh.vocab_of(name)
    want = zh.plain_logits(folder, toks)
    first = torch.frombuffer(bytearray((out / "0.f32").read_bytes()), dtype=F32).reshape(-1, V)
    last = torch.frombuffer(bytearray((out / "2.f32").read_bytes()), dtype=F32).reshape(-1, V)
    zh.assert_close_rows(first, want[[0, 20]], F32, "step 0")
    zh.assert_close_rows(last, torch.stack([want[29], want[3]]), F32, "step 2")
