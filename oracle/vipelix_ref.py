"""Plain, slow restatement of the Vipelix decoder in numpy: one function per
mechanism.  Test infrastructure; it shares no code with the package.

Weights are a dict name -> array (``embed``, ``loop.step``, ``l<i>.mix.q`` ...), the
configuration the dict that config.json holds.  ``dt`` is the arithmetic type
(float64 by default).

Functions that could hide a fault behind random weights take the fault as an
optional argument (``lost``, ``shared_cache`` ...), so that a test can show on the
CPU that its inputs would expose it.
"""
from __future__ import annotations

import numpy as np


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + x.dtype.type(eps))


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def sigmoid(z):
    return 1 / (1 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def turn_pairs(x, positions, base):
    """x [T, ..., n]: the pair (2i, 2i + 1) of the row at position p turns by p * base ** (-2i / n)."""
    n = x.shape[-1]
    f = np.power(float(base), -2.0 * np.arange(n // 2) / n)
    a = np.asarray(positions, np.float64).reshape((-1,) + (1,) * (x.ndim - 1)) * f
    c, s = np.cos(a).astype(x.dtype), np.sin(a).astype(x.dtype)
    out = np.empty_like(x)
    u, v = x[..., 0::2], x[..., 1::2]
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


def latent_of(h, w_dkv, w_norm, rank, base, eps, positions):
    """What a token leaves in the cache: (normed latent [T, rank], turned key part [T, rot])."""
    z = h @ w_dkv.T
    return rms_norm(z[:, :rank], w_norm, eps), turn_pairs(z[:, rank:], positions, base)


def latent_attention(q, c, k_rot, w_uk, w_uv, scale, first=0, lost=()):
    """q [T, H, dim + rot] (its last part turned) of the positions first, first + 1, ...; c [P, rank] and
    k_rot [P, rot] of all positions up to the last query's.  Returns [T, H, vdim].  `lost` positions
    are left out where they are not the query's own."""
    T, H, _ = q.shape
    rot = k_rot.shape[1]
    dim, vdim = q.shape[2] - rot, w_uv.shape[0] // H
    k = (c @ w_uk.T).reshape(len(c), H, dim)
    v = (c @ w_uv.T).reshape(len(c), H, vdim)
    out = np.zeros((T, H, vdim), q.dtype)
    for i in range(T):
        n = first + i + 1
        s = (np.einsum("hd,jhd->hj", q[i, :, :dim], k[:n]) + q[i, :, dim:] @ k_rot[:n].T) * q.dtype.type(scale)
        for j in lost:
            if j < n - 1:
                s[:, j] = -np.inf
        p = np.exp(s - s.max(1, keepdims=True))
        out[i] = np.einsum("hj,jhv->hv", p / p.sum(1, keepdims=True), v[:n])
    return out


def latent_mixer(h, w, prefix, spec, eps, lost=()):
    """One sequence from its start: h [T, width] -> [T, width]."""
    T, H = h.shape[0], spec["heads"]
    pos = np.arange(T)
    q = (h @ w[prefix + "q"].T).reshape(T, H, spec["dim"] + spec["rot_dim"])
    q = np.concatenate([q[..., :spec["dim"]], turn_pairs(q[..., spec["dim"]:], pos, spec["rot"]["base"])], -1)
    c, k_rot = latent_of(h, w[prefix + "dkv"], w[prefix + "dkv.norm"], spec["kv_rank"], spec["rot"]["base"], eps, pos)
    o = latent_attention(q, c, k_rot, w[prefix + "uk"], w[prefix + "uv"], spec["scale"], lost=lost)
    o = o * sigmoid(h @ w[prefix + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[prefix + "o"].T


def poly_norm(z, coef, eps):
    """a N(z) + b N(z^2) + c N(z^3) + e with N the division by the root mean square."""
    a, b, c, e = coef
    return a * unit_rms(z, eps) + b * unit_rms(z * z, eps) + c * unit_rms(z * z * z, eps) + e


def dense_ffn(h, w, prefix, eps):
    return poly_norm(h @ w[prefix + "up"].T, w[prefix + "act"], eps) @ w[prefix + "down"].T


def gated_unit(h, w_gate, w_up, w_down):
    return (silu(h @ w_gate.T) * (h @ w_up.T)) @ w_down.T


def table_moe(h, tokens, w, prefix, spec):
    """Experts named by the token id, each with weight 1 / top, plus the shared expert."""
    out = np.zeros_like(h)
    table, top = w[prefix + "table"], spec["router"]["top"]
    for t, token in enumerate(tokens):
        for e in table[token]:
            p = f"{prefix}e{int(e)}."
            out[t] += gated_unit(h[t], w[p + "gate"], w[p + "up"], w[p + "down"]) / top
    if spec.get("shared"):
        p = prefix + "shared."
        out += gated_unit(h, w[p + "gate"], w[p + "up"], w[p + "down"])
    return out


def softcap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


def runs(cfg):
    """The layers in the order in which they run: [(layer, pass or None)], the pass only at its first layer."""
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 0}
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], len(cfg["layers"]))]


def forward(cfg, weights, tokens, dt=np.float64, layers_out=None, lost=(), stale_pass=False, no_inject=False):
    """Logits [T, vocab] of one sequence, computed from its start in one piece.  ``layers_out`` (a list)
    collects the residual stream after every layer run.  Faults: `lost` keys, passes that all get the
    step vector of the first (`stale_pass`), no embedding added before later passes (`no_inject`)."""
    w = {n: np.asarray(a) if np.asarray(a).dtype.kind == "i" else np.asarray(a, dt) for n, a in weights.items()}
    eps = cfg["norm"]["eps"]
    tokens = np.asarray(tokens)
    x = start = w["embed"][tokens]
    for i, t in runs(cfg):
        if t is not None:
            if t > 0 and not no_inject:
                x = x + start
            x = x + w["loop.step"][0 if stale_pass else t]
        layer, p = cfg["layers"][i], f"l{i}."
        o = latent_mixer(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps, lost)
        x = x + rms_norm(o, w[p + "norm1b"], eps)
        f = layer.get("mlp")
        if f:
            h = rms_norm(x, w[p + "norm2"], eps)
            o = dense_ffn(h, w, p + "mlp.", eps) if f["kind"] == "dense" else table_moe(h, tokens, w, p + "mlp.", f)
            x = x + rms_norm(o, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return softcap(rms_norm(x, w["final.norm"], eps) @ w["embed"].T, cfg.get("logit_softcap"))
