"""Funudra on the GPU: each new kernel and kernel option alone against the plain function of its mechanism
(tests/plain_funudra.py), then whole models through replay, the engine and the command line."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import pytest
import torch

import funudra_helpers as fh
import plain_funudra as plain
import ref_ops
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
    root = tmp_path_factory.mktemp("funudra_gpu")
    return {name: fh.make_folder(str(root / name), name) for name in fh.FUNUDRA}


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


def _ctx(q_lens, ctx_lens, slots, plan=None):
    from qwen_engine_b200.parts.base import Arena
    cu = [0]
    for n in q_lens:
        cu.append(cu[-1] + n)
    return SimpleNamespace(cu_q=_i32(cu), ctx_lens=_i32(ctx_lens), slot_ids=_i32(slots), num_reqs=len(q_lens), max_q_len=max(q_lens),
                           q_lens_host=list(q_lens), ctx_lens_host=list(ctx_lens), attn_plan=plan, arena=Arena(DEV, 1 << 26),
                           positions=_i32([c + i for n, c in zip(q_lens, ctx_lens) for i in range(n)]))


# steps that cut four unequal requests differently: (tokens of each request in the step); the last but one is single tokens
CUTS = [[5, 1, 40, 2], [1, 33, 2, 0], [17, 2, 1, 9], [1, 1, 1, 1], [3, 70, 1, 2]]
SLOTS = [2, 0, 3, 1]
TOTALS = [sum(c[r] for c in CUTS) for r in range(4)]


def _in_portions(seqs, call, widths):
    """Feed the four requests' rows to ``call(ctx, *step tensors)`` cut as CUTS says; returns each request's output rows.
    ``seqs``: per input a list of four [tokens, columns] tensors."""
    done, rows = [0] * 4, [[] for _ in range(4)]
    for cut in CUTS:
        ctx = _ctx(cut, done, SLOTS)
        step = [torch.cat([s[r][done[r]:done[r] + cut[r]] for r in range(4)]).to(DEV) for s in seqs]
        outs = call(ctx, *step)
        at = 0
        for r in range(4):
            rows[r].append([o[at:at + cut[r]].float().cpu() for o in outs])
            at += cut[r]
            done[r] += cut[r]
    torch.cuda.synchronize()
    return [[torch.cat([part[i] for part in rows[r]]) for i in range(widths)] for r in range(4)]


# ---- short convolutions -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,taps,pad", [(5, 1, 0), (40, 2, 8), (132, 3, 4), (130, 4, 6), (520, 4, 16), (24, 5, 0), (72, 16, 8)])
def test_convolution_with_bias_and_silu_in_portions_through_used_slots(ops, dtype, C, taps, pad):
    g = torch.Generator().manual_seed(C + taps)
    w, ob, ib = torch.randn(C, taps, generator=g), torch.randn(C, generator=g), torch.randn(C, generator=g)
    xs = [torch.randn(n, C, generator=g).to(dtype) for n in TOTALS]
    for silu, in_bias in ((True, None), (False, ib)):
        state = torch.full((4, taps - 1, C), 1e4, device=DEV)
        wt = w.t().contiguous().to(DEV)

        def call(ctx, x):
            wide = torch.zeros(x.shape[0], C + 2 * pad, dtype=dtype, device=DEV)
            wide[:, pad:pad + C] = x
            out = torch.full((x.shape[0], C + pad), 7.0, dtype=dtype, device=DEV)
            ops.conv_act(wide[:, pad:pad + C], wt, state if taps > 1 else None, ctx, out[:, :C], in_bias=None if in_bias is None else in_bias.to(DEV),
                         out_bias=ob.to(DEV), silu=silu)
            assert bool((out[:, C:] == 7.0).all())
            return [out[:, :C]]
        got = _in_portions([xs], call, 1)
        for r in range(4):
            u = xs[r].double() + (0.0 if in_bias is None else in_bias.double())
            want = plain.causal_conv(u, w.double()) + ob.double()
            _close(got[r][0], plain.silu(want) if silu else want, dtype, f"request {r}")
            if taps > 1:
                tail = torch.cat([torch.zeros(taps - 1, C, dtype=F64), u])[-(taps - 1):]
                _close(state[SLOTS[r]], tail, F32, f"state of request {r}")


def test_a_convolution_reads_a_state_it_does_not_write(ops):
    g = torch.Generator().manual_seed(1)
    C, taps = 24, 4
    w, x = torch.randn(taps, C, generator=g).to(DEV), torch.randn(3, C, generator=g).to(DEV)
    state = torch.randn(2, taps - 1, C, generator=g).to(DEV)
    before = state.clone()
    out = torch.empty(3, C, device=DEV)
    ops.conv_act(x, w, state, _ctx([3], [9], [1]), out, silu=False, write_state=False)
    want = plain.causal_conv(torch.cat([before[1], x]).cpu().double(), w.t().cpu().double())[taps - 1:]
    _close(out, want, F32)
    assert torch.equal(state, before)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,n,D,taps,rot,P", [(4, 2, 1, 48, 3, 16, 4), (3, 1, 2, 128, 4, 128, 16), (2, 2, 3, 32, 1, 0, 8), (1, 1, 1, 16, 6, 10, 16),
                                                (4, 4, 2, 128, 2, 32, 16), (2, 1, 1, 48, 4, 22, 8)])
@pytest.mark.parametrize("table", [False, True])
def test_projected_rows_to_turned_queries_and_pages(ops, dtype, H, G, n, D, taps, rot, P, table):
    """Bias, convolution, rotation and cache write in portions through used slots and pages, against the plain functions."""
    g = torch.Generator().manual_seed(H + D + taps)
    C = (H + G * (1 + n)) * D
    w, bias = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    xs = [torch.randn(t, C, generator=g).to(dtype) for t in TOTALS]
    freqs = plain.rotation_frequencies(1000.0, rot, 3.0) if rot else []
    inv = torch.tensor(freqs, dtype=F32, device=DEV) if rot else None
    blocks = [-(-t // P) for t in TOTALS]
    order = torch.randperm(sum(blocks), generator=g).tolist()
    tables = [[order.pop() for _ in range(b)] for b in blocks]
    pages = torch.full((sum(blocks), 1 + n, G, P, D), 1e4, dtype=dtype, device=DEV)
    state = torch.full((4, taps - 1, C), 1e4, device=DEV)
    wt, bt = w.t().contiguous().to(DEV), bias.to(DEV)

    def call(ctx, x):
        slots = _i32([tables[r][(c + i) // P] * P + (c + i) % P for r, (c, m) in enumerate(zip(ctx.ctx_lens_host, ctx.q_lens_host)) for i in range(m)])
        q = torch.empty(x.shape[0], H * D, dtype=dtype, device=DEV)
        cs = None
        if table and rot:
            cs = torch.empty(x.shape[0], rot // 2, 2, device=DEV)
            ops.rope_table(ctx.positions, inv, cs)
        ops.conv_qkv(x, wt, state if taps > 1 else None, ctx, q, pages, slots, H, G, D, in_bias=bt, inv_freq=inv, rotary_dim=rot, cos_sin=cs)
        return [q]
    got = _in_portions([xs], call, 1)
    for r in range(4):
        y = plain.causal_conv(xs[r].double() + bias.double(), w.double())
        turn = lambda rows: plain.rotate_half_split(rows, rot, freqs) if rot else rows
        want_q = torch.cat([turn(y[:, h * D:(h + 1) * D]) for h in range(H)], dim=1)
        _close(got[r][0], want_q, dtype, f"queries of request {r}")
        where = [(tables[r][i // P], i % P) for i in range(TOTALS[r])]
        pg = pages.float().cpu()
        for kv in range(G):
            k = torch.stack([pg[p, 0, kv, o] for p, o in where])
            _close(k, turn(y[:, (H + kv) * D:(H + kv + 1) * D]), dtype, f"keys of request {r}")
            for b in range(n):
                v = torch.stack([pg[p, 1 + b, kv, o] for p, o in where])
                at = (H + G + kv * n + b) * D
                _close(v, y[:, at:at + D], dtype, f"values of request {r}, block {b}")


# ---- recurrences ------------------------------------------------------------------------------------------------------------
SSM_SIZES = [(6, 3, 20, 12), (1, 1, 7, 33), (2, 1, 300, 5), (8, 2, 128, 64), (4, 4, 64, 32), (3, 1, 256, 24), (2, 2, 1, 1), (5, 5, 48, 130)]


def _ssm_case(H, G, N, P, seed, totals, dtype):
    g = torch.Generator().manual_seed(seed)
    mk = lambda width, std=1.0: [(torch.randn(t, width, generator=g) * std).to(dtype) for t in totals]
    x, B, C, dt = mk(H * P), mk(G * N, N ** -0.5), mk(G * N), mk(H)
    const = dict(bias=torch.randn(H, generator=g) - 1.0, rate=torch.randn(H, generator=g) * 1.5 - 0.5, skip=torch.randn(H, generator=g))
    return x, B, C, dt, const


def _ssm_plain(x, B, C, dt, const, H, G, N, P):
    x, B, C, dt = (t.double() for t in (x, B, C, dt))
    d = plain.softplus(dt + const["bias"].double())
    return torch.cat([plain.state_space_recurrence(x[:, i * P:(i + 1) * P], B[:, (i // (H // G)) * N:(i // (H // G) + 1) * N],
                                                   C[:, (i // (H // G)) * N:(i // (H // G) + 1) * N], d[:, i],
                                                   torch.exp(const["rate"][i].double()), const["skip"][i].double()) for i in range(H)], dim=1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,N,P", SSM_SIZES)
def test_state_space_recurrence_in_portions_through_used_slots(ops, dtype, H, G, N, P):
    x, B, C, dt, const = _ssm_case(H, G, N, P, N + P, TOTALS, dtype)
    state = torch.full((4, H, P, N), 1e4, device=DEV)
    dev = {k: v.to(DEV) for k, v in const.items()}

    def call(ctx, x, B, C, dt):
        wide = torch.cat([torch.zeros(x.shape[0], 8, dtype=dtype, device=DEV), x, B, C, dt], dim=1)        # columns of one wider row
        n, m = H * P, G * N
        out = torch.empty(x.shape[0], n, device=DEV)
        ops.state_space_scan(wide[:, 8:8 + n], wide[:, 8 + n:8 + n + m], wide[:, 8 + n + m:8 + n + 2 * m], wide[:, 8 + n + 2 * m:], dev["bias"],
                             dev["rate"], dev["skip"], state, ctx, out, H, G, N, P)
        return [out]
    got = _in_portions([x, B, C, dt], call, 1)
    for r in range(4):
        _close(got[r][0], _ssm_plain(x[r], B[r], C[r], dt[r], const, H, G, N, P), F32, f"request {r}")


MEM_SIZES = [(3, 16, 24), (1, 7, 9), (2, 300, 5), (2, 128, 192), (4, 24, 72), (1, 256, 64), (2, 1, 1), (3, 33, 130)]


def _mem_case(H, dk, dv, seed, totals, dtype):
    g = torch.Generator().manual_seed(seed)
    mk = lambda width, std=1.0: [(torch.randn(t, width, generator=g) * std).to(dtype) for t in totals]
    q, k, v, gi, gf = mk(H * dk), mk(H * dk), mk(H * dv), mk(H, 4.0), mk(H, 4.0)
    return q, k, v, gi, gf, dict(bi=torch.randn(H, generator=g), bf=torch.randn(H, generator=g) + 2.0)


def _mem_plain(q, k, v, gi, gf, const, cap, H, dk, dv):
    q, k, v, gi, gf = (t.double() for t in (q, k, v, gi, gf))
    li = plain.soft_bound(gi + const["bi"].double(), cap)
    lf = plain.log_sigmoid(plain.soft_bound(gf + const["bf"].double(), cap))
    return torch.cat([plain.matrix_memory(q[:, i * dk:(i + 1) * dk] * dk ** -0.5, k[:, i * dk:(i + 1) * dk], v[:, i * dv:(i + 1) * dv],
                                          li[:, i], lf[:, i]) for i in range(H)], dim=1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dk,dv", MEM_SIZES)
@pytest.mark.parametrize("gates_f32", [False, True])
def test_matrix_memory_in_portions_through_used_slots(ops, dtype, H, dk, dv, gates_f32):
    cap = 7.0
    q, k, v, gi, gf, const = _mem_case(H, dk, dv, dk + dv, TOTALS, dtype)
    state, maxima = torch.full((4, H, dv + 1, dk), 1e4, device=DEV), torch.full((4, H, dv + 1), 1e4, device=DEV)
    bi, bf = const["bi"].to(DEV), const["bf"].to(DEV)

    def call(ctx, q, k, v, gi, gf):
        wide = torch.cat([q, k, v, gi, gf], dim=1)
        n, m = H * dk, H * dv
        gates = [wide[:, 2 * n + m:2 * n + m + H], wide[:, 2 * n + m + H:]]
        if gates_f32:
            gates = [t.float() for t in gates]
        out, div = torch.empty(q.shape[0], m, device=DEV), torch.empty(q.shape[0], H, device=DEV)
        ops.matrix_memory_scan(wide[:, :n], wide[:, n:2 * n], wide[:, 2 * n:2 * n + m], gates[0], gates[1], bi, bf, cap, state, maxima, ctx, out,
                               div, dk ** -0.5, 1e-6, H, dk, dv)
        return [(out.view(-1, H, dv) / div[:, :, None]).view(-1, m)]
    got = _in_portions([q, k, v, gi, gf], call, 1)
    for r in range(4):
        _close(got[r][0], _mem_plain(q[r], k[r], v[r], gi[r], gf[r], const, cap, H, dk, dv), F32, f"request {r}", tol=1e-4)


def test_recurrences_whole_and_token_by_token_to_the_bit(ops):
    """The bits of a row do not depend on the cut: a long prompt whole, in portions, and token by token."""
    T, dtype = 300, BF16
    H, G, N, P = 4, 2, 128, 64
    x, B, C, dt, const = (t[0] if isinstance(t, list) else t for t in _ssm_case(H, G, N, P, 5, [T], dtype))
    q, k, v, gi, gf, mc = (t[0] if isinstance(t, list) else t for t in _mem_case(2, 64, 72, 6, [T], dtype))
    d = lambda t: t.to(DEV)
    outs = []
    for portions in ([T], [77, 2, 150, 71], [1] * T):
        st, ms, mx = torch.zeros(1, H, P, N, device=DEV), torch.zeros(1, 2, 73, 64, device=DEV), torch.zeros(1, 2, 73, device=DEV)
        ys, os_, at = [], [], 0
        for n in portions:
            ctx, sl = _ctx([n], [at], [0]), slice(at, at + n)
            y, o, div = torch.empty(n, H * P, device=DEV), torch.empty(n, 144, device=DEV), torch.empty(n, 2, device=DEV)
            ops.state_space_scan(d(x[sl]), d(B[sl]), d(C[sl]), d(dt[sl]), d(const["bias"]), d(const["rate"]), d(const["skip"]), st, ctx, y, H, G, N, P)
            ops.matrix_memory_scan(d(q[sl]), d(k[sl]), d(v[sl]), d(gi[sl]), d(gf[sl]), d(mc["bi"]), d(mc["bf"]), 7.0, ms, mx, ctx, o, div, 0.125,
                                   1e-6, 2, 64, 72)
            ys.append(y.cpu()), os_.append(torch.cat([o, div], dim=1).cpu())
            at += n
        outs.append((torch.cat(ys), torch.cat(os_), st.cpu(), ms.cpu(), mx.cpu()))
    _close(outs[0][0], _ssm_plain(x, B, C, dt, const, H, G, N, P), F32, "whole")
    for other in outs[1:]:
        for a, b in zip(outs[0], other):
            assert torch.equal(a, b)


def test_a_recurrence_reads_a_state_it_does_not_write(ops):
    H, G, N, P = 2, 1, 16, 8
    for n in (1, 5):
        x, B, C, dt, const = (t[0] if isinstance(t, list) else t for t in _ssm_case(H, G, N, P, 3, [n], F32))
        state = torch.randn(2, H, P, N, device=DEV)
        before, out = state.clone(), torch.empty(n, H * P, device=DEV)
        ops.state_space_scan(x.to(DEV), B.to(DEV), C.to(DEV), dt.to(DEV), const["bias"].to(DEV), const["rate"].to(DEV), None, state,
                             _ctx([n], [4], [1]), out, H, G, N, P, write_state=False)
        assert torch.equal(state, before)
        ref = torch.empty(n, H * P)
        ref_ops.state_space_scan(x, B, C, dt, const["bias"], const["rate"], None, before.cpu(),
                                 SimpleNamespace(cu_q=torch.tensor([0, n]), ctx_lens=torch.tensor([4]), slot_ids=torch.tensor([1])), ref, H, G, N, P)
        _close(out, ref, F32)


# ---- norms ------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W", [(1, 40), (9, 256), (70, 1024), (5, 3000), (33, 97), (3, 8192), (2, 9000), (17, 2560)])
@pytest.mark.parametrize("deltas,bias,pair", [(0, False, True), (1, True, True), (2, True, True), (2, False, False)])
def test_two_norms_of_one_stream(ops, dtype, T, W, deltas, bias, pair):
    g = torch.Generator().manual_seed(T + W)
    resid = torch.randn(T, W, generator=g) * 3.0
    ds = [torch.randn(T, W, generator=g).to(dtype) for _ in range(deltas)]
    w1, w2, b = (torch.randn(W, generator=g) for _ in range(3))
    r = resid.to(DEV)
    o1, o2 = (torch.empty(T, W, dtype=dtype, device=DEV) for _ in range(2))
    dd = [t.to(DEV) for t in ds] + [None, None]
    ops.add_rmsnorm_pair(r, dd[0], dd[1], b.to(DEV) if bias else None, w1.to(DEV), o1, w2.to(DEV) if pair else None, o2 if pair else None, 1e-5)
    x = resid.double() + sum(t.double() for t in ds)
    _close(o1, plain.norm_plain(x, w1.double(), 1e-5), dtype, "first")
    if pair:
        _close(o2, plain.norm_plain(x, w2.double(), 1e-5), dtype, "second")
    _close(r, x + (b.double() if bias else 0.0), F32, "stream")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,G,D,pad", [(1, 1, 40, 0), (9, 3, 24, 8), (70, 8, 128, 16), (5, 2, 200, 4), (33, 1, 97, 3), (3, 2, 512, 8), (4, 1, 2048, 0),
                                       (2, 1, 8192, 0), (2, 1, 9000, 0), (6, 4, 300, 4), (3, 2, 1024, 4)])
def test_groups_normed_and_gated(ops, dtype, T, G, D, pad):
    g = torch.Generator().manual_seed(G + D)
    C = G * D
    x, w = torch.randn(T, C, generator=g) * 2.0, torch.randn(C, generator=g)
    gate = torch.randn(T, C, generator=g).to(dtype)
    div = torch.rand(T, G, generator=g) + 0.1
    wide = torch.zeros(T, C + pad, dtype=dtype)
    wide[:, pad:] = gate
    wide = wide.to(DEV)
    unit = lambda y: plain.rms_unit(y.reshape(T, G, D), 1e-5).reshape(T, C) * w.double()
    xd, gd = x.double(), gate.double()
    for kw, want in ((dict(gate_kind="silu", gate_first=True), unit(xd * plain.silu(gd))),
                     (dict(gate_kind="sigmoid", divisor=div.to(DEV), scale=0.7), unit((xd.reshape(T, G, D) / div.double()[:, :, None]).reshape(T, C)) * torch.sigmoid(gd) * 0.7),
                     (dict(gate_kind="silu"), unit(xd) * plain.silu(gd))):
        out = torch.full((T, C + pad), 7.0, dtype=dtype, device=DEV)
        ops.group_norm_gate(x.to(DEV), wide[:, pad:], w.to(DEV), 1e-5, G, out[:, :C], **kw)
        _close(out[:, :C], want, dtype, str(sorted(kw)))
        assert bool((out[:, C:] == 7.0).all())


# ---- attention over pages with several blocks of values ----------------------------------------------------------------------
def _attention(ops, dtype, H, G, D, n, P, q_lens, ctx_lens, softcap, seed, window=0, fast=True, plant=None, parts=None):
    """paged_attention on a cache of 1 + n planes: (output on the device, plain output, kernel names)."""
    from qwen_engine_b200.engine.runner import ModelRunner
    g = torch.Generator().manual_seed(seed)
    R, T = len(q_lens), sum(q_lens)
    blocks = [-(-(c + m) // P) for c, m in zip(ctx_lens, q_lens)]
    order = torch.randperm(sum(blocks) + 3, generator=g).tolist()
    table = torch.full((R, max(blocks)), -1, dtype=torch.int32)
    for r, b in enumerate(blocks):
        for i in range(b):
            table[r, i] = order.pop()
    pages = torch.randn(sum(blocks) + 3, 1 + n, G, P, D, generator=g).to(dtype)
    q = torch.randn(T, H * D, generator=g).to(dtype)
    cu = [0]
    for m in q_lens:
        cu.append(cu[-1] + m)
    if plant is not None:
        plant(q, pages, table, cu)
    geo = (H, G, D, window, False, 1 + n)
    uniform = {geo: parts} if parts else None
    plan = ops.plan_attention(list(q_lens), list(ctx_lens), P, (geo,) if fast else (), dtype, uniform_splits=uniform)
    dev = ModelRunner._device_plan(plan, {"plan_" + k: _i32(v) for k, v in plan.items()}, (geo,) if fast else ())
    ctx = _ctx(q_lens, ctx_lens, list(range(R)), dev)
    out = torch.full((T, H * n * D), 3.0, dtype=dtype, device=DEV)
    ops.paged_attention(q.to(DEV), pages.to(DEV), table.to(DEV), ctx, out, 1.5 * D ** -0.5, window, H, G, D, softcap=softcap)
    torch.cuda.synchronize()
    want = torch.zeros(T, H * n * D)
    ref_ops.paged_attention(q.float(), pages.float(), table, SimpleNamespace(cu_q=torch.tensor(cu), ctx_lens=torch.tensor(ctx_lens)), want,
                            1.5 * D ** -0.5, window, H, G, D, softcap=softcap)
    return out, want, ops.last_attention_kernel


ATT = [([70, 3, 1, 200], [0, 40, 300, 17]), ([1, 1, 1, 1], [0, 15, 16, 700]), ([300], [0]), ([40, 130], [500, 1000]), ([1, 5, 2], [600, 64, 127])]


@pytest.mark.parametrize("dtype,fast", [(F32, True), (BF16, False), (BF16, True)])
@pytest.mark.parametrize("H,G,D,n,P", [(4, 2, 128, 2, 16), (3, 3, 128, 3, 16), (8, 1, 128, 2, 8), (2, 2, 48, 2, 4), (2, 1, 256, 1, 16)])
@pytest.mark.parametrize("case", range(len(ATT)))
def test_attention_with_blocks_of_values_and_bent_scores(ops, dtype, fast, H, G, D, n, P, case):
    q_lens, ctx_lens = ATT[case]
    for softcap, window in ((4.0, 0), (0.0, 33)):
        out, want, kernel = _attention(ops, dtype, H, G, D, n, P, q_lens, ctx_lens, softcap, H + D + n + case, window=window, fast=fast)
        _close(out, want, dtype, f"{kernel}, cap {softcap}, window {window}", tol={F32: 3e-5, BF16: 2e-2}[dtype])


@pytest.mark.parametrize("H,G,D,n,P", [(4, 2, 128, 2, 16), (8, 8, 128, 2, 16), (2, 1, 64, 3, 16)])
@pytest.mark.parametrize("parts", [1, 2, 3, 4, 8])
def test_decoded_tokens_over_blocks_of_values_in_parts(ops, H, G, D, n, P, parts):
    out, want, kernel = _attention(ops, BF16, H, G, D, n, P, [1, 1, 1], [1000, 517, 2047], 5.0, parts + H, parts=parts)
    _close(out, want, BF16, f"{kernel}, {parts} parts", tol=2e-2)
    assert kernel == ("decode_attention_mma" if D == 128 else "flash_attention")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("far", [0, 15, 16, 300, 639])
def test_a_far_key_decides_the_row_in_every_block_of_values(ops, dtype, decoded, far):
    """One key points where the last query points and takes nearly all of its weight: the row is that key's values, in
    every block, whether the key lies at a page's border, at the beginning or right behind the query."""
    H, G, D, n, P, ctx = 4, 2, 128, 2, 16, 639
    q_lens, ctx_lens = ([1], [ctx]) if decoded else ([ctx + 1], [0])

    def plant(q, pages, table, cu):
        last = q[cu[1] - 1].view(H, D)
        last *= 4.0
        for kv in range(G):
            pages[table[0, far // P], 0, kv, far % P] = (last[kv * (H // G)].float() * 0.5).to(q.dtype)
    out, want, kernel = _attention(ops, dtype, H, G, D, n, P, q_lens, ctx_lens, 40.0, far, plant=plant)
    _close(out, want, dtype, kernel, tol={F32: 3e-5, BF16: 2e-2}[dtype])
    w = want[-1].view(H, n * D)
    for kv in range(G):
        assert float(w[kv * (H // G)].abs().max()) > 1.5          # (a mean over hundreds of keys would be far smaller)


# ---- whole models -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,name", [(d, n) for n in fh.FUNUDRA for d in DTYPES])
def test_replay_against_the_plain_model(folders, dtype, name):
    folder = folders[name]
    fh.replay_cases(lambda n: fh.make_replayer(folder, name, dtype, n, poison=1.0e4), folder, name, dtype, f"{name}")


@pytest.mark.parametrize("name", ["f-a", "f-d", "f-e"])
def test_rows_do_not_depend_on_the_schedule(folders, name):
    """The rows of a mixed schedule against the engine's own rows of each whole prompt alone, in both types."""
    from helpers import live_tokens_needed, mixed_steps
    folder = folders[name]
    V = fh.vocab_of(name)
    reqs = {f"m{i}": random_tokens(V, n, 60 + i) for i, n in enumerate([40, 64, 23, 90, 17, 55])}
    steps = mixed_steps(reqs, seed=11)
    for dtype, bound in ((F32, 2e-5), (BF16, 0.05)):
        got = run_steps(fh.make_replayer(folder, name, dtype, live_tokens_needed(steps, 64), poison=1.0e4), steps)
        for rid, toks in reqs.items():
            whole = run_steps(fh.make_replayer(folder, name, dtype, 128),
                              [{"entries": [{"id": "a", "tokens": toks, "want": list(range(len(toks)))}], "end": ["a"]}])["a"]
            idx = sorted(got[rid])
            err = fh.row_errors(torch.stack([got[rid][i] for i in idx]), torch.stack([whole[i] for i in idx]))
            assert float(err.max()) < bound, f"{name} {rid} {dtype}: position {idx[int(err.argmax())]} differs by {float(err.max()):.2e}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_every_position_of_a_long_prompt_whole_and_decoded(folders, dtype):
    """Every position whole, and from the first token on one by one (the steps of single tokens are replayed from a CUDA
    graph): first tokens, pages' borders and long decoding lie among them."""
    for name, n in (("f-b", 120), ("f-c", 150), ("f-e", 300)):
        folder = folders[name]
        toks = random_tokens(fh.vocab_of(name), n, 31)
        whole = [{"entries": [{"id": "a", "tokens": toks, "want": list(range(n))}], "end": ["a"]}]
        fh.check_requests(run_steps(fh.make_replayer(folder, name, dtype, 320), whole), folder, {"a": toks}, dtype, f"{name} whole")
        single = [{"entries": [{"id": "a", "tokens": [t], "want": [0]}]} for t in toks]
        rep = fh.make_replayer(folder, name, dtype, 320)
        fh.check_requests(run_steps(rep, single), folder, {"a": toks}, dtype, f"{name} decoded")
        assert rep.runner.num_graph_replays > n // 2


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt_in_portions_then_decoded(folders, dtype):
    """600 tokens: whole; and in portions of changing sizes (two tokens among them, cuts inside pages) with the last 40
    tokens one by one, beside a second request that comes and goes (its pages and its slot are used again)."""
    name = "f-e"
    folder = folders[name]
    V = fh.vocab_of(name)
    toks, other = random_tokens(V, 600, 3), random_tokens(V, 50, 4)
    want = sorted(set(range(0, 600, 7)) | set(range(560, 600)))
    whole = [{"entries": [{"id": "a", "tokens": toks, "want": want}], "end": ["a"]}]
    fh.check_requests(run_steps(fh.make_replayer(folder, name, dtype, 640), whole), folder, {"a": toks}, dtype, "whole")
    steps, p = [], 0
    for i, n in enumerate([64, 64, 100, 2, 30, 129, 16, 3, 95, 57] + [1] * 40):
        entries = [{"id": "a", "tokens": toks[p:p + n], "want": [w - p for w in want if p <= w < p + n]}]
        if i in (1, 5, 12):
            entries.append({"id": f"b{i}", "tokens": other, "want": [49]})
        steps.append({"entries": entries, "end": [f"b{i}"] if i in (1, 5, 12) else []})
        p += n
    assert p == 600
    got = run_steps(fh.make_replayer(folder, name, dtype, 704, poison=1.0e4), steps)
    fh.check_requests(got, folder, {"a": toks, "b1": other, "b5": other, "b12": other}, dtype, "portions")


def test_greedy_generation_through_the_engine(folders):
    from qwen_engine_b200.sampling.params import SamplingParams
    for name in ("f-a", "f-b", "f-c"):
        folder = folders[name]
        cfg, w = fh.plain_model(folder)
        V = fh.vocab_of(name)
        prompts = [random_tokens(V, n, 40 + i) for i, n in enumerate([5, 19, 33, 2, 11, 26, 47])]
        eng = fh.make_engine(folder, name, F32, max_num_seqs=3, max_num_batched_tokens=24, prefill_chunk_size=7)
        ids = [eng.add_request(p, SamplingParams(max_new_tokens=8, temperature=0.0)) for p in prompts]
        outs = {o.request_id: o for o in eng.serving()}
        for rid, p in zip(ids, prompts):
            assert list(outs[rid].output_token_ids) == plain.greedy(cfg, w, p, 8), f"{name}: prompt of {len(p)} tokens"
        assert eng.cache.slots.num_free == eng.cache.slots.num_slots and eng.cache.pages_in_use() == 0


def test_the_command_line_replays_a_trace(folders, tmp_path):
    name = "f-a"
    folder = folders[name]
    toks = random_tokens(fh.vocab_of(name), 30, 8)
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
    V = fh.vocab_of(name)
    want = fh.plain_logits(folder, toks)
    first = torch.frombuffer(bytearray((out / "0.f32").read_bytes()), dtype=F32).reshape(-1, V)
    last = torch.frombuffer(bytearray((out / "2.f32").read_bytes()), dtype=F32).reshape(-1, V)
    fh.assert_close_rows(first, want[[0, 20]], F32, "step 0")
    fh.assert_close_rows(last, torch.stack([want[29], want[3]]), F32, "step 2")
