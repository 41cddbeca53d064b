"""Small Vipelix checkpoints with random weights: configuration, numpy weights (bf16 values) and the
folder a user would load."""
import json
import os
import struct

import numpy as np
import torch

from helpers import pkg
from oracle import vipelix_ref as ref
from tovelix_fixtures import bf16_round, errors  # noqa: F401


def latent(heads=3, dim=24, rot=8, vdim=40, rank=56, base=900.0, scale=0.21):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                                                  "rot": {"base": base, "dims": rot}, "scale": scale}}


def dense(ff=88):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=48, shared=72):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    return dict(m, shared={"ff": shared}) if shared else m


def config(layers, width=72, vocab=211, eps=3e-5, loop=(1, 3, 3), cap=9.0):
    c = {"architecture": "Vipelix", "layers": [dict(m, mlp=f) for m, f in layers], "norm": {"eps": eps}, "vocab": vocab, "width": width,
         "logit_softcap": cap}
    return dict(c, loop=dict(zip(("start", "stop", "times"), loop))) if loop else c


# every branch: layers of different sizes, one without feed-forward, one and all experts, no shared expert, a loop in
# the middle; sizes that no tensor-core path takes beside some that every one takes
VARIED = config([
    (latent(), moe()),
    (latent(heads=5, dim=20, rot=6, vdim=18, rank=44, base=70.0, scale=0.3), dense()),
    (latent(heads=1, dim=32, rot=16, vdim=64, rank=128), moe(experts=1, top=1, ff=40, shared=0)),
    (latent(heads=40, dim=8, rot=8, vdim=8, rank=16), None),
    (latent(heads=2, dim=64, rot=32, vdim=32, rank=72), moe(experts=3, top=3, ff=33, shared=50)),
])
# loop from the first layer to the last, one layer only, dense
ROUND = config([(latent(heads=4, dim=48, rot=16, vdim=56, rank=136, scale=0.15), dense(ff=160))], width=104, vocab=160, loop=(0, 1, 4), cap=20.0)
# no loop at all; everything in multiples of 16
PLAIN = config([
    (latent(heads=8, dim=32, rot=32, vdim=64, rank=192, base=5e4), moe(experts=6, top=3, ff=64, shared=128)),
    (latent(heads=16, dim=64, rot=32, vdim=32, rank=320), dense(ff=256)),
], width=128, vocab=320, loop=None, cap=30.0)


def weights(cfg, seed=0):
    rng = np.random.default_rng(seed)
    w = {}

    def lin(name, n, k, gain=1.0):
        w[name] = bf16_round(rng.standard_normal((n, k)) * gain / np.sqrt(k))

    def norm(name, n, gain=1.0):
        w[name] = bf16_round(gain * (1 + 0.3 * rng.standard_normal(n)))

    def unit(prefix, ff, d):
        lin(prefix + "gate", ff, d, 1.5)
        lin(prefix + "up", ff, d, 1.5)
        lin(prefix + "down", d, ff)

    d, V = cfg["width"], cfg["vocab"]
    lin("embed", V, d, np.sqrt(d))
    norm("final.norm", d, 0.4)
    if cfg.get("loop"):
        w["loop.step"] = bf16_round(rng.standard_normal((cfg["loop"]["times"], d)))
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        H = m["heads"]
        lin(p + "mix.q", H * (m["dim"] + m["rot_dim"]), d, 1.5)
        lin(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], d, 1.5)
        norm(p + "mix.dkv.norm", m["kv_rank"])
        lin(p + "mix.uk", H * m["dim"], m["kv_rank"], 1.5)
        lin(p + "mix.uv", H * m["vdim"], m["kv_rank"])
        lin(p + "mix.g", H, d, 2.0)
        lin(p + "mix.o", d, H * m["vdim"])
        norm(p + "norm1", d)
        norm(p + "norm1b", d, 0.7)
        f = L["mlp"]
        if f is None:
            continue
        norm(p + "norm2", d)
        norm(p + "norm2b", d, 0.7)
        if f["kind"] == "dense":
            lin(p + "mlp.up", f["ff"], d)
            lin(p + "mlp.down", d, f["ff"])
            w[p + "mlp.act"] = bf16_round([0.6, -0.4, 0.3, 0.1])
            continue
        E, top = f["router"]["experts"], f["router"]["top"]
        for e in range(E):
            unit(f"{p}mlp.e{e}.", f["expert"]["ff"], d)
        w[p + "mlp.table"] = np.stack([rng.permutation(E)[:top] for _ in range(V)]).astype(np.int32)
        if f.get("shared"):
            unit(p + "mlp.shared.", f["shared"]["ff"], d)
    return w


def tensors(w):
    """The weights as a checkpoint's tensors."""
    return {n: torch.from_numpy(a) if a.dtype == np.int32 else torch.from_numpy(np.asarray(a, np.float32)).to(torch.bfloat16) for n, a in w.items()}


def write_checkpoint(folder, cfg, w):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    table, blobs, off = {}, [], 0
    for name, t in tensors(w).items():
        ints = t.dtype == torch.int32
        b = (t if ints else t.view(torch.int16)).numpy().tobytes()
        table[name] = {"dtype": "I32" if ints else "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(b)]}
        off += len(b)
        blobs.append(b)
    head = json.dumps(table).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    return folder


def load(folder, cfg, w, dtype, max_tokens=256, max_seq_len=512):
    write_checkpoint(str(folder), cfg, w)
    return pkg().load_model(str(folder), dtype, max_tokens=max_tokens, max_seq_len=max_seq_len)


def expected(cfg, w, tokens, **faults):
    return ref.forward(cfg, w, tokens, **faults)


def spiked_latents(T, H, dim, rot, vdim, rank, at, targets, seed, gain=7.0):
    """q [T, H, dim + rot], latents [T, rank], key parts [T, rot] (unnormed, unrotated), W_uk, W_uv: the query
    at `at` scores high against the positions `targets`, through the latents alone."""
    rng = np.random.default_rng(seed)
    w_uk = bf16_round(rng.standard_normal((H * dim, rank)) / np.sqrt(rank))
    w_uv = bf16_round(rng.standard_normal((H * vdim, rank)) / np.sqrt(rank))
    q = rng.standard_normal((T, H, dim + rot))
    c = rng.standard_normal((T, rank))
    kr = rng.standard_normal((T, rot))
    for n, t in enumerate(targets):
        h = n % H      # head h finds this position
        c[t] = 3.0 * np.linalg.pinv(w_uk[h * dim:(h + 1) * dim]) @ rng.standard_normal(dim) + 0.3 * c[t]
        q[at, h, :dim] = gain * (w_uk[h * dim:(h + 1) * dim] @ c[t]) / np.linalg.norm(w_uk[h * dim:(h + 1) * dim] @ c[t])
    return [bf16_round(x) for x in (q, c, kr)] + [w_uk, w_uv]
