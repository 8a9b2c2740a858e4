"""Shared by the Zugunex tests: small configurations that differ in every size and constant, model folders with
seeded random weights, and the plain implementation's logits."""
from __future__ import annotations

import torch

import plain_zugunex
from pufivik_helpers import CLOSE_CALL, LOOSE_WORST, assert_close_rows, row_errors
from qwen_engine_b200.registry import config_from_dict
from qwen_engine_b200.weights import write_model_folder


def _mixer(heads, dim, rot_dim, vdim, kv_rank, scale, window, base, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=dict(base=base, dims=rot_dim))
    if window is not None:
        m["mask"] = dict(size=window)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _layer(mixer, mlp):
    return dict(type="latent_attention", mixer=mixer, mlp=mlp)


def _dense(ff):
    return dict(kind="dense", ff=ff)


def _moe(experts, top, ff, shared, scale):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale), shared=dict(ff=shared))


def _model(vocab, width, eps, layers):
    return dict(architecture="Zugunex", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)


ZUGUNEX = {
    # one latent read by two later layers, one of them behind a layer with a latent of its own; the readers' windows are
    # longer and shorter than the owner's (one sees the token alone), their heads, key and value sizes others; a layer
    # without feed-forward; a shared expert that is no whole number of experts and one smaller than an expert; all experts
    # chosen in one layer
    "z-a": dict(cfg=_model(211, 64, 1e-6, [
        _layer(_mixer(4, 16, 8, 12, 24, 0.3, 9, 100.0), _moe(5, 2, 24, 40, 1.5)),
        _layer(_mixer(2, 8, 8, 24, 24, 0.25, 21, 100.0, kv_from=0), _dense(96)),
        _layer(_mixer(3, 16, 4, 20, 24, 0.2, 5, 3000.0), None),
        _layer(_mixer(5, 24, 8, 8, 24, 0.2, 1, 100.0, kv_from=0), _moe(3, 3, 16, 8, 0.7))]), seed=3, std=0.12, norm_std=0.2, page=4),
    # cache rows of 64 channels, three heads; two latents of different sizes with windows of a page and one token and of
    # several pages; one expert a token
    "z-b": dict(cfg=_model(300, 96, 1e-5, [
        _layer(_mixer(3, 24, 24, 32, 40, 0.15, 17, 50000.0), _dense(128)),
        _layer(_mixer(3, 24, 24, 32, 40, 0.15, 17, 50000.0, kv_from=0), _moe(4, 1, 32, 32, 1.0)),
        _layer(_mixer(6, 16, 16, 16, 80, 0.2, 40, 1000.0), _moe(6, 2, 8, 64, 2.0))]), seed=5, std=0.1, norm_std=0.1, page=16),
    # sizes that are no multiples of four or eight, one head, values wider than keys
    "z-c": dict(cfg=_model(97, 40, 3e-6, [
        _layer(_mixer(1, 10, 6, 14, 9, 0.25, 7, 20.0), _moe(2, 1, 12, 20, 1.3)),
        _layer(_mixer(2, 6, 6, 7, 9, 0.3, 3, 20.0, kv_from=0), _dense(28)),
        _layer(_mixer(3, 3, 2, 5, 13, 0.5, 11, 7.0), _moe(7, 4, 5, 3, 0.4))]), seed=9, std=0.15, norm_std=0.3, page=8),
    # sizes of real heads: cache rows of 128 and 192 channels, windows of many pages, eight experts of which three are used
    "z-d": dict(cfg=_model(513, 384, 1e-6, [
        _layer(_mixer(8, 64, 32, 64, 96, 0.1, 100, 500000.0), _dense(512)),
        _layer(_mixer(8, 64, 32, 64, 96, 0.1, 100, 500000.0, kv_from=0), _moe(8, 3, 128, 256, 2.5)),
        _layer(_mixer(16, 64, 64, 32, 128, 0.09, 64, 1000000.0), _moe(8, 3, 128, 256, 2.5)),
        _layer(_mixer(4, 32, 64, 128, 128, 0.1, 33, 1000000.0, kv_from=2), None)]), seed=13, std=0.05, norm_std=0.1, page=16),
    # no window at all in one layer and a window in the reader of its latent; more than sixteen heads on one latent; cache
    # rows wider than 256 channels
    "z-e": dict(cfg=_model(389, 256, 1e-6, [
        _layer(_mixer(20, 32, 64, 48, 192, 0.1, None, 10000.0), _moe(6, 2, 64, 96, 1.0)),
        _layer(_mixer(6, 48, 64, 32, 192, 0.12, 50, 10000.0, kv_from=0), _moe(4, 2, 64, 128, 1.7)),
        _layer(_mixer(2, 64, 32, 64, 256, 0.1, 70, 2000.0), _dense(384))]), seed=17, std=0.06, norm_std=0.1, page=16),
}


def make_folder(path: str, name: str) -> str:
    spec = ZUGUNEX[name]
    write_model_folder(config_from_dict(spec["cfg"]), path, spec["seed"], spec["std"], spec["norm_std"], torch.bfloat16)
    return path


_plain: dict = {}


def plain_model(folder: str):
    if folder not in _plain:
        _plain[folder] = plain_zugunex.read_model_folder(folder)
    return _plain[folder]


def plain_logits(folder: str, tokens) -> torch.Tensor:
    key = (folder, tuple(tokens))
    if key not in _plain:
        cfg, w = plain_model(folder)
        margins: list = []
        _plain[key] = plain_zugunex.forward(cfg, w, list(tokens), margins=margins).to(torch.float32)
        _plain[("margin",) + key] = torch.stack(margins).min(dim=0).values if margins else torch.full((len(tokens),), float("inf"))
    return _plain[key]


def settled_positions(folder: str, tokens, dtype) -> set:
    """The positions up to which no router of the plain model makes a close call: bfloat16 rounding may decide such a call
    the other way, and the row, and through its keys in part the rows behind it, is then another expert's.  In float32
    every position counts."""
    plain_logits(folder, tokens)
    m = _plain[("margin", folder, tuple(tokens))]
    if dtype == torch.float32:
        return set(range(len(tokens)))
    close = [i for i in range(len(tokens)) if float(m[i]) < CLOSE_CALL]
    return set(range(close[0] if close else len(tokens)))


def vocab_of(name: str) -> int:
    return ZUGUNEX[name]["cfg"]["vocab"]


def make_replayer(folder, name, dtype, max_tokens, device="cuda:0", slots=4, poison=False, prefix_cache=True):
    from qwen_engine_b200.engine.loading import load_model
    from qwen_engine_b200.engine.trace import TraceReplayer
    page = ZUGUNEX[name]["page"]
    unit = max(64, page)
    unit = -(-unit // page) * page
    num_pages = -(-max_tokens // unit) * (unit // page)
    loaded = load_model(folder, dtype, device, page, num_pages, slots, enable_prefix_cache=prefix_cache, poison_cache=poison,
                        check_device=(device != "cpu"))
    return TraceReplayer(folder, dtype, max_tokens, page_size=page, loaded=loaded)


def check_requests(got, folder, requests, dtype, what):
    """Rows up to a request's first close call are judged sharply; in bfloat16 the rows behind it are only kept from being
    as far off as a row that read another request's pages would be."""
    behind = []
    for rid, toks in requests.items():
        want = plain_logits(folder, toks)
        rows = got[rid]
        settled = settled_positions(folder, toks, dtype)
        idx = [i for i in sorted(rows) if i in settled]
        if idx:
            assert_close_rows(torch.stack([rows[i] for i in idx]), want[idx], dtype, f"{what} {rid} (positions {idx[0]}..)")
        m = _plain[("margin", folder, tuple(toks))]
        rest = [i for i in sorted(rows) if i not in settled and float(m[i]) >= CLOSE_CALL]
        if rest:
            behind.append(row_errors(torch.stack([rows[i] for i in rest]), want[rest]))
    if behind:
        err = torch.cat(behind)
        assert float(err.max()) <= LOOSE_WORST, f"{what}: a row behind a close call is off by {float(err.max()):.3f}"


def make_engine(folder, name, dtype, device="cuda:0", **engine_kwargs):
    from qwen_engine_b200.config import EngineConfig
    from qwen_engine_b200.engine.llm import LLMEngine
    from qwen_engine_b200.engine.loading import load_model
    kw = dict(dtype=dtype, device=device, block_size=ZUGUNEX[name]["page"], max_model_len=160, max_num_seqs=4,
              max_num_batched_tokens=48)
    kw.update(engine_kwargs)
    ec = EngineConfig(**kw)
    loaded = load_model(folder, ec.dtype, ec.device, ec.block_size, ec.resolved_num_blocks(), ec.max_num_seqs,
                        ec.enable_prefix_cache, check_device=(device != "cpu"))
    return LLMEngine(loaded, ec)


def replay_cases(rep_factory, folder, name, dtype, what):
    """The ways of cutting requests into steps, each against the plain implementation: whole prompts; a prompt and
    then single tokens; from the first token one by one; portions of changing sizes down to two tokens; up to four
    live requests mixed, with pages that come back and go out again.  Every position of every prompt is looked at, so the
    places just inside and outside every window are among them."""
    from helpers import live_tokens_needed, mixed_steps, random_tokens, run_steps
    V = vocab_of(name)
    reqs = {"w0": random_tokens(V, 61, 1), "w1": random_tokens(V, 9, 2), "w2": random_tokens(V, 1, 3)}
    steps = [{"entries": [{"id": r, "tokens": t, "want": list(range(len(t)))}], "end": [r]} for r, t in reqs.items()]
    check_requests(run_steps(rep_factory(128), steps), folder, reqs, dtype, f"{what} whole")
    toks = random_tokens(V, 75, 3)
    steps = [{"entries": [{"id": "d", "tokens": toks[:35], "want": [0, 17, 34]}]}]
    steps += [{"entries": [{"id": "d", "tokens": [t], "want": [0]}]} for t in toks[35:]]
    check_requests(run_steps(rep_factory(128), steps), folder, {"d": toks}, dtype, f"{what} decode")
    steps = [{"entries": [{"id": "s", "tokens": [t], "want": [0]}]} for t in toks[:30]]
    check_requests(run_steps(rep_factory(64), steps), folder, {"s": toks[:30]}, dtype, f"{what} single tokens")
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
