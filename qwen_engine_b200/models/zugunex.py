"""Zugunex as a layout of parts.

Layers in the order config.json gives, each a ``post_norm`` block (a sublayer reads the stream itself; its result is
normed and added) with latent attention: queries projected directly, interleaved rotation of their rotated part and of
the key part all heads share, a window, a sink per head, a sigmoid gate per head.  A layer with ``kv_from`` has no
latent of its own: its plan entry names the cache slot of the layer it reads and writes nothing.  The slot keeps as
many tokens as the longest window among its readers.  The feed-forward is absent, dense (tanh form of gelu, no gate)
or a mixture of experts (square of relu, no gate) scored by sigmoids that are made to sum to one, beside a shared
expert with a gate per token.  The head is a tensor of its own.

Tensor names: ``embed``, ``final.norm``, ``head``, and per layer ``l<i>.norm1/norm2``, ``l<i>.mix.q/uk/uv/sink/g/o``
(+ ``dkv``, ``dkv.norm`` where the layer has a latent), ``l<i>.mlp.up/down``, or ``l<i>.mlp.router``,
``l<i>.mlp.e<j>.up/down``, ``l<i>.mlp.shared.up/down/sg``.
"""
from __future__ import annotations

from ..config.zugunex_config import ZugunexConfig
from ..parts.base import PartSpec
from .decoder import LayerSpec, ModelLayout, PlanEntry


def _window(mixer: dict):
    mask = mixer.get("mask")
    return None if mask is None else mask["size"]


def _cache_windows(cfg: ZugunexConfig) -> dict:
    """Layer with a latent -> how many of the last tokens its cache slot keeps: the longest window of the layers that
    read it (None: all tokens)."""
    kept: dict = {}
    for i, layer in enumerate(cfg.layers):
        src = layer["mixer"].get("kv_from")
        src, w = (i if src is None else src), _window(layer["mixer"])
        kept[src] = w if src not in kept else None if (w is None or kept[src] is None) else max(w, kept[src])
    return kept


def _mixer(cfg: ZugunexConfig, m: dict, cache_window) -> PartSpec:
    return PartSpec("latent_attention", dict(
        hidden_size=cfg.width, num_heads=m["heads"], plain_dim=m["dim"], rot_dim=m["rot_dim"], value_dim=m["vdim"],
        latent_dim=m["kv_rank"], query_rank=None, scale=m["scale"], norm_eps=cfg.norm_eps, rope_base=m["rot"]["base"],
        rope_dims=m["rot"]["dims"], pairing="interleaved", window=_window(m), cache_window=cache_window, sink=True,
        output_gate="sigmoid_head", shared_kv=m.get("kv_from") is not None))


def _feed_forward(cfg: ZugunexConfig, mlp):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("mlp", dict(hidden_size=cfg.width, intermediate_size=mlp["ff"], activation="gelu_tanh", names=("up", "down")))
    r, shared = mlp["router"], mlp.get("shared")
    return PartSpec("routed_experts", dict(
        hidden_size=cfg.width, intermediate_size=mlp["expert"]["ff"], num_experts=r["experts"], top=r["top"], gated=False,
        activation="relu_squared", names=("up", "down"), router_bias_name=None, scoring="sigmoid_sum", weight_scale=float(r["scale"]),
        shared_size=None if shared is None else shared["ff"]))


def zugunex_layout(cfg: ZugunexConfig) -> ModelLayout:
    norm = PartSpec("rmsnorm", dict(width=cfg.width, eps=cfg.norm_eps, weight_name=""))
    kept = _cache_windows(cfg)
    layers, plan, slot_of = [], [], {}
    for i, layer in enumerate(cfg.layers):
        src = layer["mixer"].get("kv_from")
        own = src is None
        if own:
            src, slot_of[i] = i, len(slot_of)
        layers.append(LayerSpec(PartSpec("post_norm", dict(
            hidden_size=cfg.width, mixer=_mixer(cfg, layer["mixer"], kept[src]), feed_forward=_feed_forward(cfg, layer.get("mlp")),
            norm=norm)), f"l{i}."))
        plan.append(PlanEntry(i, slot_of[src], own))
    return ModelLayout(
        vocab_size=cfg.vocab, hidden_size=cfg.width, layers=tuple(layers), plan=tuple(plan), final_norm=norm,
        embed_name="embed", final_norm_prefix="final.norm", head_name="head", tie_head=False, max_positions=None)
