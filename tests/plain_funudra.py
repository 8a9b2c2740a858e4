"""A plain, slow restatement of the Funudra design, one function per mechanism.

Everything runs on the CPU in one floating-point type (float64 by default), token
by token where the design is recurrent, with no cache, no batching and no code
of the package.  The tests compare the engine with it.

Notation: ``x`` [T, W] is the residual stream of ONE sequence, positions 0..T-1;
``w`` maps tensor names to tensors; ``cfg`` is the parsed config.json.
"""
from __future__ import annotations

import math

import torch

from plain_ganidra import read_model_folder  # noqa: F401  (config.json and the tensors of a model folder)


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_plain(x, weight, eps):
    return rms_unit(x, eps) * weight


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def log_sigmoid(z):
    return -softplus(-z)


def soft_bound(z, cap):
    """z bent smoothly into (-cap, cap)."""
    return cap * torch.tanh(z / cap)


def causal_conv(u, taps):
    """u [T, C], taps [C, n]: y_t[c] = sum_j taps[c, j] u_(t - n + 1 + j)[c], zeros before the first token."""
    T, n = u.shape[0], taps.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(n):
            s = t - n + 1 + j
            if s >= 0:
                y[t] = y[t] + taps[:, j] * u[s]
    return y


def rotation_frequencies(base, dims, factor):
    return [base ** (-2.0 * i / dims) / factor for i in range(dims // 2)]


def rotate_half_split(x, dims, freqs):
    """x [T, D]: the pairs (i, i + dims/2) of the first ``dims`` channels turn by position * freqs[i]."""
    half = dims // 2
    a = torch.arange(x.shape[0], dtype=x.dtype)[:, None] * torch.tensor(freqs, dtype=x.dtype)[None, :]
    out = x.clone()
    u, v = x[:, :half], x[:, half:dims]
    out[:, :half] = u * torch.cos(a) - v * torch.sin(a)
    out[:, half:dims] = v * torch.cos(a) + u * torch.sin(a)
    return out


def bent_causal_attention(q, k, v, scale, softcap):
    """One head.  q, k [T, dk], v [T, dv]: scores softcap * tanh(scale q.k / softcap), plain softmax over j <= i."""
    T = q.shape[0]
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    for i in range(T):
        s = soft_bound((k[:i + 1] @ q[i]) * scale, softcap)
        out[i] = torch.softmax(s, dim=0) @ v[:i + 1]
    return out


def attention_mixer(h, w, p, m):
    """Grouped-head attention: biased projections, a convolution over time on each of q, k and v, partial rotation,
    bent scores, a gate per channel, a biased output projection."""
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ w[p + n].T + w[p + n + ".b"], w[p + n + ".conv"]) for n in ("q", "k", "v"))
    rot = m["rot"]
    scaling = rot.get("scaling")
    freqs = rotation_frequencies(rot["base"], rot["dims"], scaling["factor"] if scaling else 1.0)
    keys = [rotate_half_split(k[:, g * dk:(g + 1) * dk], rot["dims"], freqs) for g in range(G)]
    heads = []
    for i in range(H):
        g = i // (H // G)
        qi = rotate_half_split(q[:, i * dk:(i + 1) * dk], rot["dims"], freqs)
        heads.append(bent_causal_attention(qi, keys[g], v[:, g * dv:(g + 1) * dv], m["scale"], m["softcap"]))
    o = torch.cat(heads, dim=1) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T + w[p + "o.b"]


def matrix_memory(q, k, v, log_in, log_keep):
    """One head of the matrix memory with exponential gates.  q (already scaled), k [T, dk]; v [T, dv]; log_in, log_keep
    [T].  The memory and its normaliser are kept divided by exp(m), m the running maximum, zero at the start."""
    T, dk = q.shape
    dv = v.shape[1]
    S = torch.zeros(dk, dv, dtype=q.dtype)
    n = torch.zeros(dk, dtype=q.dtype)
    m = torch.zeros((), dtype=q.dtype)
    out = torch.zeros(T, dv, dtype=q.dtype)
    for t in range(T):
        kept = log_keep[t] + m
        m = torch.maximum(kept, log_in[t])
        a, b = torch.exp(kept - m), torch.exp(log_in[t] - m)
        S = a * S + b * k[t][:, None] * v[t][None, :]
        n = a * n + b * k[t]
        out[t] = (S.T @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6)
    return out


def memory_mixer(h, w, p, m, eps):
    H, dk, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T) * dk ** -0.5
    k = h @ w[p + "k"].T
    v = h @ w[p + "v"].T
    log_in = soft_bound(h @ w[p + "i"].T + w[p + "i.b"], cap)
    log_keep = log_sigmoid(soft_bound(h @ w[p + "f"].T + w[p + "f.b"], cap))
    heads = [rms_unit(matrix_memory(q[:, i * dk:(i + 1) * dk], k[:, i * dk:(i + 1) * dk], v[:, i * dv:(i + 1) * dv],
                                    log_in[:, i], log_keep[:, i]), eps) for i in range(H)]
    o = torch.cat(heads, dim=1) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    left = attention_mixer(h, w, p + "left.", m["left"])
    right = memory_mixer(h, w, p + "right.", m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


def state_space_recurrence(x, B, C, dt, rate, D):
    """One head.  x [T, P], B and C [T, N], dt [T] (after its softplus): S <- exp(-rate dt) S + dt B x^T, y = S^T C + D x."""
    T, P = x.shape
    S = torch.zeros(B.shape[1], P, dtype=x.dtype)
    y = torch.zeros_like(x)
    for t in range(T):
        S = torch.exp(-rate * dt[t]) * S + dt[t] * B[t][:, None] * x[t][None, :]
        y[t] = S.T @ C[t] + D * x[t]
    return y


def state_space_mixer(h, w, p, m, eps):
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(causal_conv(xbc, w[p + "conv"]) + w[p + "conv.b"])
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    dt = softplus(dt + w[p + "dt_bias"])
    heads = []
    for i in range(H):
        g = i // (H // G)
        heads.append(state_space_recurrence(x[:, i * P:(i + 1) * P], B[:, g * N:(g + 1) * N], C[:, g * N:(g + 1) * N],
                                            dt[:, i], torch.exp(w[p + "A_log"][i]), w[p + "D"][i]))
    y = torch.cat(heads, dim=1) * silu(z)
    parts = m["norm_groups"]
    y = rms_unit(y.reshape(-1, parts, inner // parts), eps).reshape(-1, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def mixer(kind, h, w, p, m, eps):
    if kind == "parallel":
        return parallel_mixer(h, w, p, m, eps)
    if kind == "mamba2":
        return state_space_mixer(h, w, p, m, eps)
    raise ValueError(kind)


def feed_forward(h, w, p):
    return torch.clamp(h @ w[p + "up"].T, min=0.0) ** 2 @ w[p + "down"].T


def weights_index(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def layer(x, w, i, spec, eps):
    """Mixer and feed-forward side by side, each with a norm of its own of the same stream."""
    p = f"l{i}."
    y = mixer(spec["type"], norm_plain(x, w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps)
    if spec.get("mlp") is not None:
        y = y + feed_forward(norm_plain(x, w[p + "norm2"], eps), w, p + "mlp.")
    return x + y


def forward(cfg, w, tokens, dtype=torch.float64, keep_layers=False):
    """Logits [T, vocab] of one sequence (and the stream after every layer)."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = norm_plain(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], w["embed.norm"], eps)
    kept = []
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, weights_index(cfg, i), spec, eps)
        if keep_layers:
            kept.append(x.clone())
    logits = norm_plain(x, w["final.norm"], eps) @ w["embed"].T
    return (logits, kept) if keep_layers else logits


def greedy(cfg, w, prompt, n_new, dtype=torch.float64):
    """The prompt's greedy continuation, token by token over the whole sequence each time."""
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(cfg, w, toks, dtype)[-1])))
    return toks[len(prompt):]
