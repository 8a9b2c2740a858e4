"""Funudra as a layout of parts.

Layers in the order config.json gives, each a ``side_by_side`` block: a mixer and an optional feed-forward (square of relu,
no gate) that read the same stream through norms of their own.  ``mamba2`` layers have a state-space mixer; ``parallel``
layers have softmax attention (biased projections, short convolutions of q, k and v, partial rotation with divided
frequencies, bent scores, a sigmoid gate, a biased output projection) and a matrix memory with exponential gates side by
side, their outputs weighted and summed.  A layer with ``weights_of`` is another run of the layer it names: the same parts
in the plan once more, with cache slots of its own.  The embedding output passes a norm of its own; the head is the
embedding table.

Tensor names: ``embed``, ``embed.norm``, ``final.norm``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` (``.left.*`` /
``.right.*`` in a parallel layer), ``l<i>.mlp.up``, ``l<i>.mlp.down``.
"""
from __future__ import annotations

from ..config.funudra_config import FunudraConfig
from ..parts.base import PartSpec
from .decoder import LayerSpec, ModelLayout, PlanEntry

_ATTENTION_NAMES = dict(q="q", k="k", v="v", out="o", gate="g", q_bias="q.b", k_bias="k.b", v_bias="v.b", out_bias="o.b",
                        q_conv="q.conv", k_conv="k.conv", v_conv="v.conv")


def _attention(cfg: FunudraConfig, m: dict) -> PartSpec:
    rot = m["rot"]
    scaling = rot.get("scaling")
    pos = PartSpec("rope_scaled", dict(head_dim=m["dim"], theta=rot["base"], rotary_dim=rot["dims"],
                                       scaling=None if scaling is None else ("linear", float(scaling["factor"]))))
    return PartSpec("gqa_attention", dict(
        hidden_size=cfg.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"],
        scale=m["scale"], position_encoding=pos, softcap=float(m["softcap"]), conv_taps=m["conv"], projection_bias=True,
        output_bias=True, output_gate="sigmoid", names=_ATTENTION_NAMES))


def _memory(cfg: FunudraConfig, m: dict) -> PartSpec:
    return PartSpec("matrix_memory", dict(hidden_size=cfg.width, num_heads=m["heads"], key_dim=m["dim"], value_dim=m["vdim"],
                                          gate_cap=float(m["gate_cap"]), norm_eps=cfg.norm_eps))


def _mixer(cfg: FunudraConfig, layer: dict) -> PartSpec:
    m = layer["mixer"]
    if layer["type"] == "mamba2":
        return PartSpec("state_space", dict(
            hidden_size=cfg.width, num_heads=m["heads"], value_dim=m["vdim"], state_dim=m["state"], num_groups=m["groups"],
            conv_taps=m["conv"], norm_groups=m["norm_groups"], norm_eps=cfg.norm_eps))
    return PartSpec("parallel_mixers", dict(
        branches=(_attention(cfg, m["left"]), _memory(cfg, m["right"])),
        scales=(m["left_scale"], m["right_scale"]), prefixes=("left.", "right.")))


def _caches(layer: dict) -> int:
    """Cache slots of a run: a convolution of one tap keeps no inputs."""
    m = layer["mixer"]
    if layer["type"] == "mamba2":
        return 1 + int(m["conv"] > 1)
    return 1 + int(m["left"]["conv"] > 1) + 2


def funudra_layout(cfg: FunudraConfig) -> ModelLayout:
    norm = PartSpec("rmsnorm", dict(width=cfg.width, eps=cfg.norm_eps, weight_name=""))
    layers, index_of, plan, slot = [], {}, [], 0
    for i, layer in enumerate(cfg.layers):
        if cfg.owner_of(i) != i:
            continue
        mlp = layer.get("mlp")
        ffn = None if mlp is None else PartSpec("mlp", dict(hidden_size=cfg.width, intermediate_size=mlp["ff"],
                                                            activation="relu_squared", names=("up", "down")))
        index_of[i] = len(layers)
        layers.append(LayerSpec(PartSpec("side_by_side", dict(hidden_size=cfg.width, mixer=_mixer(cfg, layer), feed_forward=ffn,
                                                              norm=norm)), f"l{i}."))
    for i, layer in enumerate(cfg.layers):
        n = _caches(layer)
        plan.append(PlanEntry(index_of[cfg.owner_of(i)], tuple(range(slot, slot + n)) if n > 1 else slot, True))
        slot += n
    return ModelLayout(
        vocab_size=cfg.vocab, hidden_size=cfg.width, layers=tuple(layers), plan=tuple(plan), final_norm=norm,
        embed_name="embed", final_norm_prefix="final.norm", head_name=None, tie_head=True, max_positions=None,
        embed_norm=norm, embed_norm_prefix="embed.norm")
