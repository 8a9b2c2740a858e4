"""Zugunex on the host side of the engine: configuration, registry, weights and caches, and replay and generation on
the CPU with the plain operations in the place of the kernels, against the plain restatement of the design
(tests/plain_zugunex.py).  The same traces run on the GPU in test_zugunex_gpu.py."""
import copy

import pytest
import torch

import plain_zugunex
import zugunex_helpers as zh
from helpers import random_tokens, run_steps
from qwen_engine_b200.config import ConfigError, ZugunexConfig
from qwen_engine_b200.registry import architecture_of, build_model, config_from_dict
from qwen_engine_b200.weights import SafetensorsSource, WeightError, check_against_manifest

F32 = torch.float32


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("zugunex")
    return {name: zh.make_folder(str(root / name), name) for name in ("z-a", "z-b", "z-c")}


def test_config_reads_its_own_keys_and_round_trips():
    raw = zh.ZUGUNEX["z-a"]["cfg"]
    assert architecture_of(raw).name == "Zugunex"
    cfg = config_from_dict(raw)
    assert isinstance(cfg, ZugunexConfig)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, len(cfg.layers)) == (211, 64, 1e-6, 4)
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="attention"), "not a mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "at most rot_dim"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"].update(kv_from=0), "earlier layer"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=2), "earlier layer"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "no latent of its own"),
    (lambda c: c["layers"][1]["mixer"].update(kv_rank=32), "differs from layer 0"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(base=7.0), "rot differs"),
    (lambda c: c["layers"][1].update(mlp=dict(kind="glu", ff=8)), "feed-forward"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "exceeds"),
    (lambda c: c["layers"][0]["mlp"]["router"].pop("scale"), "router.scale"),
    (lambda c: c["norm"].pop("eps"), "norm.eps is missing"),
    (lambda c: c.pop("width"), "'width' is missing"),
])
def test_config_refuses_what_it_cannot_run(change, text):
    raw = copy.deepcopy(zh.ZUGUNEX["z-a"]["cfg"])
    change(raw)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(raw)


def test_a_cache_slot_keeps_what_its_longest_reader_sees():
    """One slot per latent; a layer that reads another's is given that layer's slot and writes nothing; the slot keeps the
    longest window among its readers, or everything where one of them has no window."""
    model = build_model(config_from_dict(zh.ZUGUNEX["z-a"]["cfg"]))
    specs = model.cache_specs()
    assert [(s.num_kv_heads, s.head_dim, s.window, s.planes) for s in specs] == [(1, 32, 21, 1), (1, 28, 5, 1)]
    assert [(e.cache_slot, e.write_cache) for e in model.layout.plan] == [(0, True), (0, False), (1, True), (0, False)]
    assert model.attention_geometries == ((4, 1, 32, 9, False, 1), (2, 1, 32, 21, False, 1), (3, 1, 28, 5, False, 1), (5, 1, 32, 1, False, 1))
    model = build_model(config_from_dict(zh.ZUGUNEX["z-e"]["cfg"]))
    assert [s.window for s in model.cache_specs()] == [None, 70]


def test_tensor_names(folders):
    src = SafetensorsSource(folders["z-a"])
    names = set(src.names())
    assert {"embed", "final.norm", "head", "l0.norm1", "l0.norm2", "l0.mix.q", "l0.mix.dkv", "l0.mix.dkv.norm", "l0.mix.uk", "l0.mix.uv",
            "l0.mix.sink", "l0.mix.g", "l0.mix.o", "l0.mlp.router", "l0.mlp.e4.up", "l0.mlp.e4.down", "l0.mlp.shared.up",
            "l0.mlp.shared.down", "l0.mlp.shared.sg", "l1.mlp.up", "l1.mlp.down", "l1.mix.uk"} <= names
    assert not {"l1.mix.dkv", "l1.mix.dkv.norm", "l3.mix.dkv", "l2.norm2", "l0.mlp.e5.up", "l0.mlp.e0.gate", "l1.mlp.router"} & names
    assert src.shape("l0.mix.q") == (96, 64) and src.shape("l0.mix.dkv") == (32, 64) and src.shape("l0.mix.g") == (4, 64)
    assert src.shape("l0.mlp.shared.sg") == (1, 64) and src.shape("l0.mlp.shared.up") == (40, 64)
    raw = copy.deepcopy(zh.ZUGUNEX["z-a"]["cfg"])
    check_against_manifest(src, build_model(config_from_dict(raw)).weight_manifest(), "folder")
    raw["layers"][1]["mixer"].pop("kv_from")
    with pytest.raises(WeightError, match="l1.mix.dkv"):
        check_against_manifest(src, build_model(config_from_dict(raw)).weight_manifest(), "folder")


def test_the_rotated_rows_are_reordered_together():
    """Queries and key part are brought into half-split order by the same reordering, so every product of two rotated
    vectors is that of the interleaved pairs (also with channels that pass unturned behind them)."""
    from qwen_engine_b200.parts.latent_attention import LatentAttention
    m = LatentAttention(hidden_size=12, num_heads=2, plain_dim=3, rot_dim=8, value_dim=4, latent_dim=5, query_rank=None, scale=1.0,
                        norm_eps=1e-6, rope_base=100.0, rope_dims=6, pairing="interleaved", output_gate=None)
    w = torch.arange(22.0)[:, None].expand(22, 12).contiguous()
    got = m._rotated_rows(w, 2, 3)[:, 0].tolist()
    assert got == [0, 1, 2, 3, 5, 7, 4, 6, 8, 9, 10, 11, 12, 13, 14, 16, 18, 15, 17, 19, 20, 21]


def test_a_shared_expert_is_cut_into_pieces_of_the_experts_size(cpu_ops):
    """Pieces with zero channels behind them add up to the whole shared expert, times one number per token."""
    from types import SimpleNamespace

    from qwen_engine_b200.parts.base import Arena
    from qwen_engine_b200.parts.moe import RoutedExperts
    g = torch.Generator().manual_seed(4)
    W = 12
    for ff, shared in ((8, 20), (8, 16), (8, 3)):
        w = {f"e{e}.{n}": torch.randn(*s, generator=g) for e in range(3) for n, s in (("up", (ff, W)), ("down", (W, ff)))}
        w.update({"shared.up": torch.randn(shared, W, generator=g), "shared.down": torch.randn(W, shared, generator=g),
                  "shared.sg": torch.randn(1, W, generator=g), "router": torch.randn(3, W, generator=g)})
        part = RoutedExperts(W, ff, 3, 2, activation="relu_squared", names=("up", "down"), router_bias_name=None, scoring="sigmoid_sum",
                             weight_scale=1.7, gated=False, shared_size=shared)
        part.load("", SimpleNamespace(get=lambda n: w[n]), F32, "cpu")
        assert part.shared_pieces == -(-shared // ff)
        x = torch.randn(9, W, generator=g)
        out = torch.empty(9, W)
        part.forward(SimpleNamespace(num_tokens=9, dtype=F32, arena=Arena("cpu")), x, out)
        mlp = dict(kind="moe", router=dict(experts=3, top=2, scale=1.7), expert=dict(ff=ff), shared=dict(ff=shared))
        want = plain_zugunex.mixture_of_experts(x.double(), {k: v.double() for k, v in w.items()}, "", mlp)
        assert float((out.double() - want).abs().max()) < 1e-4 * float(want.abs().max())


@pytest.mark.parametrize("name", ["z-a", "z-b", "z-c"])
def test_replay_on_the_host(folders, cpu_ops, name):
    folder = folders[name]
    zh.replay_cases(lambda n: zh.make_replayer(folder, name, F32, n, device="cpu", poison=True), folder, name, F32,
                    f"host {name}")


def test_a_window_that_is_one_off_or_a_sink_left_out_shows(folders):
    """The plain model itself tells such mistakes apart: planted in its configuration or weights, each moves rows of the
    random models by far more than the tests allow."""
    folder = folders["z-a"]
    cfg, w = zh.plain_model(folder)
    toks = random_tokens(zh.vocab_of("z-a"), 40, 9)
    right = plain_zugunex.forward(cfg, w, toks)
    for change in (lambda c, t: c["layers"][0]["mixer"]["mask"].update(size=10), lambda c, t: c["layers"][1]["mixer"]["mask"].update(size=20),
                   lambda c, t: t.update({"l0.mix.sink": torch.full_like(t["l0.mix.sink"], -1e4)}),
                   lambda c, t: t.update({"l1.mix.g": torch.zeros_like(t["l1.mix.g"])}),
                   lambda c, t: c["layers"][0]["mlp"]["router"].update(scale=1.0)):
        c, t = copy.deepcopy(cfg), dict(w)
        change(c, t)
        err = zh.row_errors(plain_zugunex.forward(c, t, toks), right)
        assert float(err.max()) > 0.02, float(err.max())


def test_greedy_generation_through_the_engine_on_the_host(folders, cpu_ops):
    from qwen_engine_b200.sampling.params import SamplingParams
    name = "z-a"
    folder = folders[name]
    cfg, w = zh.plain_model(folder)
    V = zh.vocab_of(name)
    prompts = [random_tokens(V, n, 40 + i) for i, n in enumerate([5, 19, 33, 2, 11, 26])]
    eng = zh.make_engine(folder, name, F32, device="cpu", max_num_seqs=3, max_num_batched_tokens=24, prefill_chunk_size=7)
    ids = [eng.add_request(p, SamplingParams(max_new_tokens=6, temperature=0.0)) for p in prompts]
    outs = {o.request_id: o for o in eng.serving()}
    for rid, p in zip(ids, prompts):
        assert list(outs[rid].output_token_ids) == plain_zugunex.greedy(cfg, w, p, 6), f"prompt of {len(p)} tokens"
    assert eng.cache.slots.num_free == eng.cache.slots.num_slots and eng.cache.pages_in_use() == 0


def test_requests_with_equal_prefixes_share_the_pages_their_windows_reach(folders, cpu_ops):
    """Windowed slots hand over the pages that the next query still sees (the owner's slot those of its longest reader)."""
    name = "z-a"
    folder = folders[name]
    V = zh.vocab_of(name)
    first = random_tokens(V, 40, 5)
    second = first[:24] + random_tokens(V, 10, 6)
    rep = zh.make_replayer(folder, name, F32, 256, device="cpu")
    assert rep.cache.prefix_cache and len(rep.cache.paged_groups) == 2
    steps = [{"entries": [{"id": "a", "tokens": first[:26], "want": [25]}]},
             {"entries": [{"id": "a", "tokens": first[26:], "want": [13]}, {"id": "b", "tokens": second, "want": [30, 33]}], "end": ["a", "b"]}]
    got = run_steps(rep, steps)
    assert rep.cache.prefix_hit_tokens > 0
    zh.check_requests(got, folder, {"a": first, "b": second}, F32, "shared prefix")
