"""Zugunex, written down plainly: one function per mechanism, float64, whole
sequences at once, no cache, no batch, no code of the package.  The tests
compare the engine with this.

Notation: x is the residual stream [T, W], h what a sublayer reads (x itself),
weights are a dict name -> tensor stored [out, in] and applied as W h.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def rotate_interleaved(x, positions, base, dims):
    """x [T, ..., D]: the channels (2 i, 2 i + 1) of the first ``dims`` turn by position * base^(-2 i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(F64) * base ** (-2.0 * i / dims)
        a = a.reshape([-1] + [1] * (x.dim() - 2))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def window_mask(T, size):
    """allowed[i, j]: 0 <= i - j < size (size None: no window)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) if size is None else (d >= 0) & (d < size)


def softmax_with_sink(scores, allowed, sink):
    """Weights over the allowed keys; exp(sink) stands in the denominator and nowhere else."""
    s = scores.masked_fill(~allowed, -math.inf)
    top = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def latent_and_rotated_key(h, w, p, m, eps, positions):
    """What a layer with a W_dkv keeps of every token: the normed latent and the rotated key part of all heads."""
    R = m["kv_rank"]
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :R], w[p + "dkv.norm"], eps)
    return c, rotate_interleaved(down[:, R:], positions, m["rot"]["base"], m["rot"]["dims"])


def latent_attention(h, w, p, m, eps, kept, layer_index, positions=None):
    """``kept``: layer index -> (latent, rotated key part) of the layers so far."""
    T = h.shape[0]
    H, dn, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    positions = torch.arange(T) if positions is None else positions
    if m.get("kv_from") is None:
        kept[layer_index] = latent_and_rotated_key(h, w, p, m, eps, positions)
        c, k_rot = kept[layer_index]
    else:
        c, k_rot = kept[m["kv_from"]]
    q = (h @ w[p + "q"].T).reshape(T, H, dn + dr)
    q_rot = rotate_interleaved(q[..., dn:], positions, m["rot"]["base"], m["rot"]["dims"])
    k_plain = (c @ w[p + "uk"].T).reshape(T, H, dn)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    mask = m.get("mask")
    allowed = window_mask(T, None if mask is None else mask["size"])
    gate = torch.sigmoid(h @ w[p + "g"].T)
    out = torch.zeros(T, H, dv, dtype=F64)
    for hd in range(H):
        s = (q[:, hd, :dn] @ k_plain[:, hd].T + q_rot[:, hd] @ k_rot.T) * m["scale"]
        out[:, hd] = gate[:, hd:hd + 1] * (softmax_with_sink(s, allowed, w[p + "sink"][hd]) @ v[:, hd])
    return out.reshape(T, H * dv) @ w[p + "o"].T


def plain_feed_forward(h, w, p, act):
    return act(h @ w[p + "up"].T) @ w[p + "down"].T


def route(h, w, p, router, margins=None):
    """(chosen experts [T, top], their weights): sigmoid scores, the largest chosen, their scores made to sum to one,
    times the router's scale.  ``margins`` (a list) gets by how much the last chosen score leads the first one left out,
    in logits (inf when all are chosen)."""
    z = h @ w[p + "router"].T
    s = torch.sigmoid(z)
    chosen = torch.topk(s, router["top"], dim=-1).indices
    if margins is not None:
        ordered = torch.sort(z, dim=-1, descending=True).values
        margins.append(ordered[:, router["top"] - 1] - ordered[:, router["top"]] if router["top"] < z.shape[1]
                       else torch.full((h.shape[0],), math.inf, dtype=F64))
    weights = torch.gather(s, 1, chosen)
    return chosen, weights / (weights.sum(-1, keepdim=True) + 1e-20) * router["scale"]


def mixture_of_experts(h, w, p, mlp, margins=None):
    chosen, weights = route(h, w, p, mlp["router"], margins)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(chosen[t].tolist(), weights[t]):
            out[t] += a * plain_feed_forward(h[t], w, f"{p}e{e}.", relu_squared)
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * plain_feed_forward(h, w, p + "shared.", relu_squared)
    return out


def feed_forward(h, w, p, mlp, margins=None):
    if mlp["kind"] == "dense":
        return plain_feed_forward(h, w, p, gelu_tanh)
    return mixture_of_experts(h, w, p, mlp, margins)


def forward(cfg: dict, weights: dict, token_ids, return_layers: bool = False, margins=None):
    """Logits [T, vocab] of one sequence from its first token on."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(token_ids, dtype=torch.long)]
    kept: dict = {}
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + rms_norm(latent_attention(x, w, p + "mix.", layer["mixer"], eps, kept, i), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + rms_norm(feed_forward(x, w, p + "mlp.", layer["mlp"], margins), w[p + "norm2"], eps)
        after.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(after)) if return_layers else logits


def read_model_folder(folder: str):
    """(config.json as a dict, {tensor name: tensor}) of a model folder."""
    import json
    import os

    from safetensors import safe_open
    with open(os.path.join(folder, "config.json"), "r", encoding="utf-8") as f:
        cfg = json.load(f)
    w = {}
    with safe_open(os.path.join(folder, "model.safetensors"), framework="pt", device="cpu") as f:
        for name in f.keys():
            w[name] = f.get_tensor(name)
    return cfg, w


def greedy(cfg, w, prompt, n_new):
    """The prompt's greedy continuation, token by token over the whole sequence each time."""
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]
