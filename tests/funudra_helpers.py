"""Shared by the Funudra tests: small configurations that differ in every size and constant, model folders with seeded
random weights, and the plain implementation's logits."""
from __future__ import annotations

import torch

import plain_funudra
from ganidra_helpers import ROW_TOL, ROW_WORST, assert_close_rows  # noqa: F401  (one measure of a row's error for the recurrent designs)
from qwen_engine_b200.registry import config_from_dict
from qwen_engine_b200.weights import write_model_folder


def _ssm(heads, vdim, state, groups, conv, norm_groups):
    return dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)


def _soft(heads, kv, dim, vdim, conv, scale, softcap, dims, base=10000.0, factor=4.0):
    return dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv, scale=scale, softcap=softcap,
                rot=dict(base=base, dims=dims, scaling=None if factor is None else dict(factor=factor)))


def _mem(heads, dim, vdim, cap):
    return dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)


def _layer(kind, mixer, ff=None, of=None):
    out = dict(type=kind, mixer=mixer, mlp=None if ff is None else dict(kind="dense", ff=ff))
    return out if of is None else dict(out, weights_of=of)


def _par(left, right, a, b):
    return dict(left=left, right=right, left_scale=a, right_scale=b)


def _model(vocab, width, eps, layers):
    return dict(architecture="Funudra", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)


_A_SSM, _A_PAR = _ssm(6, 12, 20, 3, 2, 6), _par(_soft(4, 2, 24, 40, 4, 0.3, 6.0, 8), _mem(3, 16, 24, 5.0), 0.8, 0.6)
_E_PAR = _par(_soft(4, 2, 128, 200, 4, 0.1, 25.0, 64, 500000.0, 16.0), _mem(2, 128, 192, 15.0), 0.7, 0.9)
FUNUDRA = {
    # grouped heads, sizes that are no multiples of 16, a layer without feed-forward, a layer that is run three times and one
    # that stands before the layer it takes its weights from
    "f-a": dict(cfg=_model(211, 64, 1e-5, [
        _layer("mamba2", _A_SSM, 96), _layer("parallel", _A_PAR, of=3), _layer("mamba2", _A_SSM, 96, of=0), _layer("parallel", _A_PAR),
        _layer("mamba2", _A_SSM, 96, of=2)]), seed=3, std=0.12, norm_std=0.2, page=4),
    # parallel layers alone: convolutions of one tap (nothing kept) and of six, one kv head, values smaller than keys, odd
    # sizes in the memory, frequencies as they are, negative and large weights of the two sides
    "f-b": dict(cfg=_model(97, 40, 3e-6, [
        _layer("parallel", _par(_soft(3, 1, 16, 8, 1, 0.4, 2.0, 16, 100.0, None), _mem(3, 7, 9, 2.0), -0.5, 1.4)),
        _layer("parallel", _par(_soft(2, 2, 40, 16, 6, 0.2, 9.0, 22, 2000.0, 2.0), _mem(1, 33, 5, 20.0), 1.2, 0.3), 50)]),
        seed=5, std=0.15, norm_std=0.3, page=8),
    # state-space layers alone (no pages at all): a state of more than 256 channels, one head, odd sizes, six and one taps
    "f-c": dict(cfg=_model(150, 48, 1e-6, [
        _layer("mamba2", _ssm(2, 5, 300, 1, 6, 1), 64), _layer("mamba2", _ssm(1, 33, 7, 1, 1, 3)),
        _layer("mamba2", _ssm(8, 4, 12, 8, 3, 2), 40)]), seed=9, std=0.15, norm_std=0.2, page=16),
    # values of more than one block of 128 channels, the second block in part; a whole head turned; many groups
    "f-d": dict(cfg=_model(513, 192, 1e-6, [
        _layer("parallel", _par(_soft(4, 4, 64, 192, 2, 0.12, 12.0, 64, 10000.0, 8.0), _mem(4, 24, 72, 6.0), 0.5, 0.5), 256),
        _layer("mamba2", _ssm(8, 32, 64, 4, 4, 8), 256)]), seed=13, std=0.06, norm_std=0.1, page=16),
    # the head sizes the fastest kernels are made for, grouped heads, 128 state channels
    "f-e": dict(cfg=_model(389, 320, 1e-6, [
        _layer("mamba2", _ssm(8, 64, 128, 2, 4, 4), 384), _layer("parallel", _E_PAR, 512), _layer("parallel", _E_PAR, 512, of=1)]),
        seed=17, std=0.05, norm_std=0.1, page=16),
}


def make_folder(path: str, name: str) -> str:
    spec = FUNUDRA[name]
    write_model_folder(config_from_dict(spec["cfg"]), path, spec["seed"], spec["std"], spec["norm_std"], torch.bfloat16)
    return path


_plain: dict = {}


def plain_model(folder: str):
    if folder not in _plain:
        _plain[folder] = plain_funudra.read_model_folder(folder)
    return _plain[folder]


def plain_logits(folder: str, tokens) -> torch.Tensor:
    key = (folder, tuple(tokens))
    if key not in _plain:
        cfg, w = plain_model(folder)
        _plain[key] = plain_funudra.forward(cfg, w, list(tokens)).to(torch.float32)
    return _plain[key]


def vocab_of(name: str) -> int:
    return FUNUDRA[name]["cfg"]["vocab"]


def row_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """A row's error: the root mean square of the difference over that of the row, means taken off."""
    d, w = got.double() - want.double(), want.double()
    d, w = d - d.mean(dim=-1, keepdim=True), w - w.mean(dim=-1, keepdim=True)
    return d.pow(2).mean(dim=-1).sqrt() / w.pow(2).mean(dim=-1).sqrt()


def make_replayer(folder, name, dtype, max_tokens, device="cuda:0", slots=4, poison=False):
    from qwen_engine_b200.engine.loading import load_model
    from qwen_engine_b200.engine.trace import TraceReplayer
    page = FUNUDRA[name]["page"]
    num_pages = -(-max_tokens // 64) * (64 // page)
    loaded = load_model(folder, dtype, device, page, num_pages, slots, poison_cache=poison, check_device=(device != "cpu"))
    if poison:                         # what an earlier request would have left in the state slots
        for g in loaded.cache.groups:
            if not g.is_paged:
                g.tensor.fill_(float(poison) if poison is not True else float("nan"))
    return TraceReplayer(folder, dtype, max_tokens, page_size=page, loaded=loaded)


def check_requests(got, folder, requests, dtype, what):
    for rid, toks in requests.items():
        want = plain_logits(folder, toks)
        rows = got[rid]
        idx = sorted(rows)
        assert_close_rows(torch.stack([rows[i] for i in idx]), want[idx], dtype, f"{what} {rid} (positions {idx[0]}..)")


def make_engine(folder, name, dtype, device="cuda:0", **engine_kwargs):
    from qwen_engine_b200.config import EngineConfig
    from qwen_engine_b200.engine.llm import LLMEngine
    from qwen_engine_b200.engine.loading import load_model
    kw = dict(dtype=dtype, device=device, block_size=FUNUDRA[name]["page"], max_model_len=160, max_num_seqs=4,
              max_num_batched_tokens=48)
    kw.update(engine_kwargs)
    ec = EngineConfig(**kw)
    loaded = load_model(folder, ec.dtype, ec.device, ec.block_size, ec.resolved_num_blocks(), ec.max_num_seqs,
                        ec.enable_prefix_cache, check_device=(device != "cpu"))
    return LLMEngine(loaded, ec)


def replay_cases(rep_factory, folder, name, dtype, what):
    """The ways of cutting requests into steps, each against the plain implementation: whole prompts; a prompt and then
    single tokens; from the first token on one by one; portions of changing sizes down to two tokens; up to four live
    requests mixed, with pages and slots that come back and go out again."""
    from helpers import live_tokens_needed, mixed_steps, random_tokens, run_steps
    V = vocab_of(name)
    reqs = {"w0": random_tokens(V, 61, 1), "w1": random_tokens(V, 9, 2), "w2": random_tokens(V, 1, 3)}
    steps = [{"entries": [{"id": r, "tokens": t, "want": list(range(len(t)))}], "end": [r]} for r, t in reqs.items()]
    check_requests(run_steps(rep_factory(128), steps), folder, reqs, dtype, f"{what} whole")
    toks = random_tokens(V, 75, 3)
    steps = [{"entries": [{"id": "d", "tokens": toks[:35], "want": [0, 17, 34]}]}]
    steps += [{"entries": [{"id": "d", "tokens": [t], "want": [0]}]} for t in toks[35:]]
    check_requests(run_steps(rep_factory(128), steps), folder, {"d": toks}, dtype, f"{what} decode")
    steps = [{"entries": [{"id": "s", "tokens": [t], "want": [0]}]} for t in toks[:24]]
    check_requests(run_steps(rep_factory(64), steps), folder, {"s": toks[:24]}, dtype, f"{what} single tokens")
    toks = random_tokens(V, 90, 4)
    steps, p = [], 0
    for n in [2, 7, 3, 2, 16, 5, 2, 13, 9, 2, 11] + [1] * 18:
        steps.append({"entries": [{"id": "c", "tokens": toks[p:p + n], "want": list(range(n))}]})
        p += n
    assert p == len(toks)
    check_requests(run_steps(rep_factory(128), steps), folder, {"c": toks}, dtype, f"{what} portions")
    reqs = {f"m{i}": random_tokens(V, n, 20 + i) for i, n in enumerate([40, 64, 23, 90, 17, 55, 70, 33])}
    steps = mixed_steps(reqs, seed=7)
    rep = rep_factory(live_tokens_needed(steps, 64))
    check_requests(run_steps(rep, steps), folder, reqs, dtype, f"{what} mixed")
    assert rep.cache.pages_in_use() == 0 and rep.cache.slots.num_free == rep.cache.slots.num_slots
