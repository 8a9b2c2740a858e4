"""Funudra on the host side of the engine: configuration, registry, weights, the plan of layer runs, and replay and
generation on the CPU with the plain operations in the place of the kernels, against the plain restatement of the design
(tests/plain_funudra.py).  The same traces run on the GPU in test_funudra_gpu.py."""
import copy

import pytest
import torch

import funudra_helpers as fh
import plain_funudra
import ref_ops
from helpers import random_tokens
from qwen_engine_b200.config import ConfigError, FunudraConfig
from qwen_engine_b200.registry import architecture_of, build_model, config_from_dict
from qwen_engine_b200.weights import SafetensorsSource, WeightError, check_against_manifest

F32 = torch.float32


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("funudra")
    return {name: fh.make_folder(str(root / name), name) for name in ("f-a", "f-b", "f-c")}


@pytest.fixture
def cpu_ops(monkeypatch):
    ref_ops.install(monkeypatch)


def test_config_reads_its_own_keys_and_round_trips():
    raw = fh.FUNUDRA["f-a"]["cfg"]
    assert architecture_of(raw).name == "Funudra"
    cfg = config_from_dict(raw)
    assert isinstance(cfg, FunudraConfig)
    assert (cfg.vocab, cfg.width, cfg.norm_eps) == (211, 64, 1e-5)
    assert [cfg.owner_of(i) for i in range(5)] == [0, 3, 0, 3, 0] == [plain_funudra.weights_index(raw, i) for i in range(5)]
    for name in fh.FUNUDRA:
        cfg = config_from_dict(fh.FUNUDRA[name]["cfg"])
        assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="conv"), "not a mixer"),
    (lambda c: [l["mixer"]["left"].update(kv_heads=3) for l in c["layers"] if "left" in l["mixer"]], "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(groups=4), "multiple of groups"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][3]["mixer"]["left"]["rot"].update(dims=26), "at most dim"),
    (lambda c: c["layers"][3]["mixer"]["left"]["rot"].update(dims=7), "must be even"),
    (lambda c: c["layers"][3]["mixer"]["right"].update(gate_cap=0), "positive"),
    (lambda c: [l.update(mlp=dict(kind="moe", ff=8)) for l in c["layers"]], "feed-forward"),
    (lambda c: c["layers"][2].update(weights_of=9), "names no layer"),
    (lambda c: c["layers"][2].update(weights_of=3), "is not like it"),
    (lambda c: c["layers"][0].update(weights_of=4), "leads back"),
    (lambda c: c.pop("norm"), "'norm' is missing"),
])
def test_config_refuses_what_it_cannot_run(change, text):
    raw = copy.deepcopy(fh.FUNUDRA["f-a"]["cfg"])
    change(raw)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(raw)


def test_every_run_of_a_layer_has_caches_of_its_own():
    model = build_model(config_from_dict(fh.FUNUDRA["f-a"]["cfg"]))
    plan = model.layout.plan
    assert [e.layer for e in plan] == [0, 1, 0, 1, 0] and len(model.blocks) == 2
    slots = [s for e in plan for s in e.slots]
    assert slots == list(range(len(slots))) and [len(e.slots) for e in plan] == [2, 4, 2, 4, 2]
    # one tap keeps nothing; values in blocks of the keys' size
    model = build_model(config_from_dict(fh.FUNUDRA["f-b"]["cfg"]))
    assert [len(e.slots) for e in model.layout.plan] == [3, 4]
    specs = build_model(config_from_dict(fh.FUNUDRA["f-e"]["cfg"])).cache_specs()
    assert (specs[2].head_dim, specs[2].planes) == (128, 3)
    assert build_model(config_from_dict(fh.FUNUDRA["f-e"]["cfg"])).attention_geometries == ((4, 2, 128, 0, False, 3),)
    assert build_model(config_from_dict(fh.FUNUDRA["f-c"]["cfg"])).attention_geometries == ()


def test_sizes_of_blocks_of_values():
    from qwen_engine_b200.ops import value_block_size
    assert value_block_size(24, 40) == (48, 1) and value_block_size(128, 128) == (128, 1) and value_block_size(40, 16) == (48, 1)
    assert value_block_size(64, 192) == (128, 2) and value_block_size(128, 257) == (128, 3) and value_block_size(200, 256) == (256, 1)


def test_tensor_names(folders):
    src = SafetensorsSource(folders["f-a"])
    names = set(src.names())
    assert {"embed", "embed.norm", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.in", "l0.mix.conv", "l0.mix.conv.b", "l0.mix.dt_bias",
            "l0.mix.A_log", "l0.mix.D", "l0.mix.norm", "l0.mix.o", "l0.mlp.up", "l0.mlp.down", "l3.norm1", "l3.mix.left.q", "l3.mix.left.q.b",
            "l3.mix.left.v.conv", "l3.mix.left.g", "l3.mix.left.o.b", "l3.mix.right.i", "l3.mix.right.f.b", "l3.mix.right.norm"} <= names
    assert not any(n.startswith(("l1.", "l2.", "l4.")) for n in names) and "l3.norm2" not in names and "head" not in names
    assert src.shape("l0.mix.in") == (2 * 72 + 2 * 60 + 6, 64) and src.shape("l3.mix.left.v.conv") == (80, 4)
    raw = copy.deepcopy(fh.FUNUDRA["f-a"]["cfg"])
    check_against_manifest(src, build_model(config_from_dict(raw)).weight_manifest(), "folder")
    raw["layers"][2].pop("weights_of")
    with pytest.raises(WeightError, match="l2.mix.in"):
        check_against_manifest(src, build_model(config_from_dict(raw)).weight_manifest(), "folder")


def test_a_mixer_whose_result_carries_a_bias_needs_a_block_that_adds_it(folders, cpu_ops):
    from qwen_engine_b200.models.decoder import DecoderModel, LayerSpec, ModelLayout
    from qwen_engine_b200.parts.base import PartSpec
    lo = build_model(config_from_dict(fh.FUNUDRA["f-a"]["cfg"])).layout
    spec = lo.layers[1].block
    block = PartSpec("pre_norm", dict(spec.params, mixer_prefix="mix.", ffn_prefix="mlp.", norm1_prefix="norm1", norm2_prefix="norm2"))
    import dataclasses
    model = DecoderModel(dataclasses.replace(lo, layers=(lo.layers[0], LayerSpec(block, "l3."))))
    assert isinstance(model.layout, ModelLayout)
    with pytest.raises(ValueError, match="does not add the bias"):
        model.load_weights(SafetensorsSource(folders["f-a"]), F32, "cpu")


@pytest.mark.parametrize("name", ["f-a", "f-b", "f-c"])
def test_replay_on_the_host(folders, cpu_ops, name):
    folder = folders[name]
    fh.replay_cases(lambda n: fh.make_replayer(folder, name, F32, n, device="cpu", poison=True), folder, name, F32, f"host {name}")


def test_mistakes_show(folders):
    """The plain model itself tells mistakes apart: planted in its configuration or weights, each moves rows of the random
    models by far more than the tests allow."""
    folder = folders["f-a"]
    cfg, w = fh.plain_model(folder)
    toks = random_tokens(fh.vocab_of("f-a"), 40, 9)
    right = plain_funudra.forward(cfg, w, toks)
    zero = lambda n: (lambda c, t: t.update({n: torch.zeros_like(t[n])}))
    left = lambda **kw: (lambda c, t: [c["layers"][i]["mixer"]["left"].update(**kw) for i in (1, 3)])
    for change in (zero("l0.mix.conv.b"), zero("l0.mix.dt_bias"), zero("l0.mix.D"), zero("l3.mix.left.q.b"), zero("l3.mix.left.o.b"),
                   zero("l3.mix.right.i.b"), zero("l3.mix.right.f.b"), left(softcap=60.0), left(scale=0.2),
                   lambda c, t: [c["layers"][i]["mixer"]["left"]["rot"].update(scaling=None) for i in (1, 3)],
                   lambda c, t: [c["layers"][i]["mixer"]["right"].update(gate_cap=20.0) for i in (1, 3)],
                   lambda c, t: [c["layers"][i]["mixer"].update(norm_groups=1) for i in (0, 2, 4)],
                   lambda c, t: t.update({"l3.mix.left.v.conv": t["l3.mix.left.v.conv"].flip(1)})):
        c, t = copy.deepcopy(cfg), dict(w)
        change(c, t)
        err = fh.row_errors(plain_funudra.forward(c, t, toks), right)
        assert float(err.max()) > 2e-3, float(err.max())          # (the tests' float32 bound is 1e-4)


def test_greedy_generation_through_the_engine_on_the_host(folders, cpu_ops):
    from qwen_engine_b200.sampling.params import SamplingParams
    for name in ("f-a", "f-c"):
        folder = folders[name]
        cfg, w = fh.plain_model(folder)
        V = fh.vocab_of(name)
        prompts = [random_tokens(V, n, 40 + i) for i, n in enumerate([5, 19, 33, 2, 11, 26])]
        eng = fh.make_engine(folder, name, F32, device="cpu", max_num_seqs=3, max_num_batched_tokens=24, prefill_chunk_size=7)
        ids = [eng.add_request(p, SamplingParams(max_new_tokens=6, temperature=0.0)) for p in prompts]
        outs = {o.request_id: o for o in eng.serving()}
        for rid, p in zip(ids, prompts):
            assert list(outs[rid].output_token_ids) == plain_funudra.greedy(cfg, w, p, 6), f"{name}: prompt of {len(p)} tokens"
        assert eng.cache.slots.num_free == eng.cache.slots.num_slots and eng.cache.pages_in_use() == 0
