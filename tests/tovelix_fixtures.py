"""Small Tovelix checkpoints with random weights: configuration, numpy weights (bf16 values) and
the folder a user would load."""
import json
import os
import struct

import numpy as np
import torch

from helpers import pkg
from oracle import tovelix_ref as ref


def bf16_round(a):
    return torch.from_numpy(np.asarray(a, np.float32)).to(torch.bfloat16).float().numpy()


def attention(heads=4, kv_heads=2, dim=32, vdim=48, window=9, rot=16, base=500.0, scale=0.3, v_mix=True):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                                           "rot": {"dims": rot, "base": base}, "scale": scale, "v_mix": v_mix}}


def lightning(heads=3, dim=40, vdim=24, decay=(0.5, 0.93, 0.997)):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def moe(experts=5, top=2, ff=56, limit=0.7):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(layers, width=96, vocab=203, eps=1e-4):
    """layers: (mixer entry, feed-forward or None) pairs."""
    return {"architecture": "Tovelix", "layers": [dict(m, mlp=f) for m, f in layers], "norm": {"eps": eps}, "vocab": vocab, "width": width}


# every branch: layers of different sizes, a layer without feed-forward, values unmixed, one expert, all experts
VARIED = config([
    (lightning(), moe()),
    (attention(), moe(experts=4, top=1, ff=40)),
    (attention(heads=6, kv_heads=1, dim=64, vdim=48, window=33, rot=64, v_mix=False), None),
    (lightning(heads=2, dim=64, vdim=72, decay=(0.8, 1.0)), moe(experts=3, top=3)),
    (attention(heads=4, kv_heads=2, dim=48, vdim=48, window=20, rot=8, base=9000.0), moe(experts=1, top=1)),
])
# no choice among experts: rounding cannot flip one, so every position can be held to a tolerance in bf16
STEADY = config([
    (attention(heads=2, kv_heads=2, dim=64, vdim=64, window=70, rot=32), moe(experts=2, top=2, ff=64)),
    (lightning(heads=4, dim=64, vdim=64, decay=(0.7, 0.95, 0.99, 0.999)), moe(experts=1, top=1, ff=128)),
    (attention(heads=8, kv_heads=2, dim=64, vdim=64, window=70, rot=64, v_mix=False), None),
], width=128, vocab=320)


def weights(cfg, seed=0):
    rng = np.random.default_rng(seed)
    w = {}

    def lin(name, n, k, gain=1.0):
        w[name] = bf16_round(rng.standard_normal((n, k)) * gain / np.sqrt(k))

    def norm(name, n, gain=1.0):
        w[name] = bf16_round(gain * (1 + 0.3 * rng.standard_normal(n)))

    d, V = cfg["width"], cfg["vocab"]
    lin("embed", V, d, np.sqrt(d))
    norm("embed.norm", d)
    norm("final.norm", d, 0.3)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        if L["type"] == "lightning":
            for n, r in (("q", hd), ("k", hd), ("v", hv), ("g", hv)):
                lin(p + "mix." + n, r, d)
            norm(p + "mix.norm", hv)
        else:
            for n, r in (("q", hd), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                lin(p + "mix." + n, r, d)
            if m["v_mix"]:
                w[p + "mix.vmix"] = bf16_round(np.float32(rng.uniform(0.2, 0.8)))
        lin(p + "mix.o", d, hv)
        norm(p + "norm1", d, 0.7)
        f = L["mlp"]
        if f is None:
            continue
        norm(p + "norm2", d, 0.7)
        lin(p + "mlp.router", f["router"]["experts"], d, 2.0)
        for e in range(f["router"]["experts"]):
            lin(f"{p}mlp.e{e}.gate", f["expert"]["ff"], d)
            lin(f"{p}mlp.e{e}.up", f["expert"]["ff"], d)
            lin(f"{p}mlp.e{e}.down", d, f["expert"]["ff"])
    return w


def write_checkpoint(folder, cfg, w):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    table, blobs, off = {}, [], 0
    for name, a in w.items():
        b = torch.from_numpy(np.asarray(a, np.float32).reshape(-1)).to(torch.bfloat16).view(torch.int16).numpy().tobytes()
        table[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [off, off + len(b)]}
        off += len(b)
        blobs.append(b)
    head = json.dumps(table).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    return folder


def load(folder, cfg, w, dtype, max_tokens=256, max_seq_len=512):
    write_checkpoint(str(folder), cfg, w)
    return pkg().load_model(str(folder), dtype, max_tokens=max_tokens, max_seq_len=max_seq_len)


def expected(cfg, w, tokens):
    return ref.forward(cfg, w, tokens)


def errors(got, want):
    """Root mean square difference per position (the mean over the vocabulary taken off), in units of
    the expected logits' own root mean square."""
    got = got.detach().float().cpu().numpy().astype(np.float64) if isinstance(got, torch.Tensor) else got
    d = got - want
    d -= d.mean(-1, keepdims=True)
    c = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((c * c).mean())
