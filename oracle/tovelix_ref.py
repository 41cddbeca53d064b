"""Plain, slow restatement of the Tovelix decoder in numpy: one function per
mechanism, one token and one head at a time where that is the clearest form.
Test infrastructure; it shares no code with the package.

Weights are a dict name -> array (``embed``, ``embed.norm``, ``l<i>.mix.q`` ...),
the configuration the dict that config.json holds.  ``dt`` is the arithmetic type
(float64 by default).

Every function that could hide a fault behind random weights takes the fault as
an optional argument (``window_shift``, ``drop_state`` ...), so that a test can show
on the CPU that its inputs would expose it.
"""
from __future__ import annotations

import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + x.dtype.type(eps))


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z / (1 + np.exp(-z))


def sigmoid(z):
    return 1 / (1 + np.exp(-z))


def rotate_interleaved(x, pos, dims, base):
    """x [..., dim] at position pos: pairs (2i, 2i + 1) of the first ``dims`` turn by
    pos * base ** (-2i / dims)."""
    out = x.copy()
    i = np.arange(dims // 2)
    a = pos * np.power(float(base), -2.0 * i / dims)
    c, s = np.cos(a).astype(x.dtype), np.sin(a).astype(x.dtype)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def mix_values(v, v_first, lam):
    return (1 - lam) * v + lam * v_first


def window_attention(q, k, v, scale, window, window_shift=0):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] of one sequence from its start:
    query i sees keys j with 0 <= i - j < window."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    for h in range(H):
        kh, vh = k[:, h // rep], v[:, h // rep]
        for i in range(T):
            lo = max(0, i - (window + window_shift) + 1)
            s = (kh[lo:i + 1] @ q[i, h]) * q.dtype.type(scale)
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ vh[lo:i + 1]
    return out


def lightning_attention(q, k, v, decay, state=None, drop_state=False):
    """q, k [T, H, dim], v [T, H, vdim]: S <- d S + k v^T, o = S^T q, per head.
    Returns (o [T, H, vdim], final state [H, dim, vdim])."""
    T, H, dim = q.shape
    S = np.zeros((H, dim, v.shape[2]), q.dtype) if state is None or drop_state else state.copy()
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    d = np.asarray(decay, q.dtype)[:, None, None]
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out, S


def route(h, w_router, top):
    """Sigmoid scores of one token's ``top`` experts, largest first: [(expert, score)]."""
    s = sigmoid(w_router @ h)
    chosen = np.argsort(-s, kind="stable")[:top]
    return [(int(e), s[e]) for e in chosen]


def clamped_glu(gate, up, limit):
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(g * g.dtype.type(1.702)) * (u + 1)


def expert(h, w_gate, w_up, w_down, limit):
    return w_down @ clamped_glu(w_gate @ h, w_up @ h, limit)


def moe(h, w, prefix, spec):
    """Mixture of experts over tokens h [T, width]: the score multiplies an expert's input."""
    out = np.zeros_like(h)
    limit = h.dtype.type(spec["expert"]["limit"])
    for t in range(h.shape[0]):
        for e, s in route(h[t], w[prefix + "router"], spec["router"]["top"]):
            p = f"{prefix}e{e}."
            out[t] += expert(s * h[t], w[p + "gate"], w[p + "up"], w[p + "down"], limit)
    return out


def attention_mixer(h, w, prefix, spec, eps, v_first):
    """Returns (output, values to keep as v_first or None).  ``v_first`` is None in the first
    layer that mixes its values."""
    T = h.shape[0]
    H, G, dim, vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = (h @ w[prefix + "q"].T).reshape(T, H, dim)
    k = (h @ w[prefix + "k"].T).reshape(T, G, dim)
    v = (h @ w[prefix + "v"].T).reshape(T, G, vdim)
    keep = None
    if spec.get("v_mix"):
        if v_first is None:
            keep = v
        else:
            v = mix_values(v, v_first, w[prefix + "vmix"].reshape(()))
    for t in range(T):
        q[t] = rotate_interleaved(q[t], t, spec["rot"]["dims"], spec["rot"]["base"])
        k[t] = rotate_interleaved(k[t], t, spec["rot"]["dims"], spec["rot"]["base"])
    o = window_attention(rms(q, eps), rms(k, eps), v, spec["scale"], spec["mask"]["size"])
    return o.reshape(T, H * vdim) @ w[prefix + "o"].T, keep


def lightning_mixer(h, w, prefix, spec, eps):
    T = h.shape[0]
    H, dim, vdim = spec["heads"], spec["dim"], spec["vdim"]
    q = silu(h @ w[prefix + "q"].T).reshape(T, H, dim)
    k = silu(h @ w[prefix + "k"].T).reshape(T, H, dim)
    v = silu(h @ w[prefix + "v"].T).reshape(T, H, vdim)
    o, _ = lightning_attention(q, k, v, spec["decay"])
    o = rms_norm(o.reshape(T, H * vdim), w[prefix + "norm"], eps)
    return (o * sigmoid(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def forward(cfg, weights, tokens, dt=np.float64, layers_out=None):
    """Logits [T, vocab] of one sequence, computed from its start in one piece.
    ``layers_out`` (a list) collects the residual stream after every layer."""
    w = {n: np.asarray(a, dt) for n, a in weights.items()}
    eps = cfg["norm"]["eps"]
    x = rms_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        if layer["type"] == "attention":
            o, keep = attention_mixer(x, w, p + "mix.", layer["mixer"], eps, v_first)
            v_first = keep if keep is not None else v_first
        else:
            o = lightning_mixer(x, w, p + "mix.", layer["mixer"], eps)
        x = x + rms_norm(o, w[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + rms_norm(moe(x, w, p + "mlp.", layer["mlp"]), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T
