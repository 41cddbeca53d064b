"""Vipelix: a decoder of latent-attention layers with norms on both sides of every sublayer, of which a
run of layers is looped over with the same weights (the embedding and a step vector enter before a
pass), dense PolyNorm feed-forwards and mixtures whose experts the token id names, a head that is the
embedding table and capped logits.

This module maps a checkpoint folder (config.json, model.safetensors) to a ``StackConfig`` and
its weights; the layers themselves are those of ``StackModel``.
"""
from __future__ import annotations

import json
import os

import torch

from .checkpoint import CheckpointError, read_safetensors
from .model import LatentMixer, MoeFfn, PolyFfn, StackConfig, StackModel
from .qlinear import QuantLinear
from .registry import register


def _mixer(kind: str, m: dict):
    if kind != "latent_attention":
        raise CheckpointError(f"unknown mixer '{kind}'")
    if m["rot"]["dims"] != m["rot_dim"]:
        raise CheckpointError(f"{m['rot']['dims']} rotated dimensions of a rotated part of {m['rot_dim']}")
    return LatentMixer(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], m["rot"]["base"], True)


def _ffn(f, prefix: str, tensors: dict):
    if f is None:
        return None
    if f["kind"] == "dense":
        return PolyFfn(f["ff"], tuple(tensors[prefix + "act"].float().tolist()))
    if f["kind"] != "moe":
        raise CheckpointError(f"unknown feed-forward '{f['kind']}'")
    shared = f.get("shared")
    return MoeFfn(f["router"]["experts"], f["router"]["top"], f["expert"]["ff"], 0.0, "silu", "table", shared["ff"] if shared else 0)


def stack_config(config: dict, tensors: dict, max_seq_len: int) -> StackConfig:
    """``config`` is config.json; of ``tensors`` only the scalars that are constants of a layer are read."""
    layers = [(_mixer(e["type"], e["mixer"]), _ffn(e.get("mlp"), f"l{i}.mlp.", tensors)) for i, e in enumerate(config["layers"])]
    loop = config.get("loop")
    return StackConfig(config["width"], config["vocab"], layers, max_seq_len, config["norm"]["eps"], embed_norm=False, pre_norms=True,
                       loop=(loop["start"], loop["stop"], loop["times"]) if loop else None, logit_softcap=config.get("logit_softcap") or 0.0)


def stack_weights(cfg: StackConfig, tensors: dict) -> dict:
    """Checkpoint tensors -> the names and fused weights of ``StackModel``."""
    def get(name, *shape):
        if name not in tensors:
            raise CheckpointError(f"checkpoint lacks '{name}'")
        t = tensors[name]
        if tuple(t.shape) != shape:
            raise CheckpointError(f"'{name}' has shape {list(t.shape)}, expected {list(shape)}")
        return t

    d = cfg.d_model
    out = {"embedding": QuantLinear.from_bf16(get("embed", cfg.vocab_size, d)), "final_norm": get("final.norm", d)}
    if cfg.loop:
        out["loop_steps"] = get("loop.step", cfg.loop[2], d)
    for i, (mix, ffn) in enumerate(cfg.layers):
        p, q, H = f"l{i}.", f"layers.{i}.", mix.heads
        rows = [get(p + "mix.q", H * (mix.dim + mix.rot_dims), d), get(p + "mix.dkv", mix.kv_rank + mix.rot_dims, d), get(p + "mix.g", H, d)]
        n = sum(len(r) for r in rows)
        out[q + "in"] = QuantLinear.from_bf16(torch.cat(rows + [torch.zeros((-n % 8, d), dtype=torch.bfloat16)]))
        out[q + "ukv"] = QuantLinear.from_bf16(torch.cat([get(p + "mix.uk", H * mix.dim, mix.kv_rank).view(H, mix.dim, -1),
                                                          get(p + "mix.uv", H * mix.vdim, mix.kv_rank).view(H, mix.vdim, -1)], 1)
                                               .reshape(H * (mix.dim + mix.vdim), -1))
        out[q + "out"] = QuantLinear.from_bf16(get(p + "mix.o", d, H * mix.vdim))
        out[q + "mix_norm"] = get(p + "mix.dkv.norm", mix.kv_rank)
        out[q + "pre1"], out[q + "norm1"] = get(p + "norm1", d), get(p + "norm1b", d)
        if ffn is None:
            continue
        out[q + "pre2"], out[q + "norm2"] = get(p + "norm2", d), get(p + "norm2b", d)
        if isinstance(ffn, PolyFfn):
            out[q + "up"] = QuantLinear.from_bf16(get(p + "mlp.up", ffn.ff, d))
            out[q + "down"] = QuantLinear.from_bf16(get(p + "mlp.down", d, ffn.ff))
            continue
        out[q + "table"] = get(p + "mlp.table", cfg.vocab_size, ffn.top)
        for leaf, shape in (("gate", (ffn.ff, d)), ("up", (ffn.ff, d)), ("down", (d, ffn.ff))):
            out[q + leaf] = QuantLinear.from_bf16(torch.cat([get(f"{p}mlp.e{e}.{leaf}", *shape) for e in range(ffn.experts)]))
        if ffn.shared_ff:
            for leaf, shape in (("gate", (ffn.shared_ff, d)), ("up", (ffn.shared_ff, d)), ("down", (d, ffn.shared_ff))):
                out[q + "shared_" + leaf] = QuantLinear.from_bf16(get(f"{p}mlp.shared.{leaf}", *shape))
    return out


@register("Vipelix")
def load(path: str, dtype: torch.dtype = torch.bfloat16, max_tokens: int = 512, max_seq_len: int = 4096) -> StackModel:
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    tensors = read_safetensors(os.path.join(path, "model.safetensors"))
    cfg = stack_config(config, tensors, max_seq_len)
    return StackModel(cfg, stack_weights(cfg, tensors), dtype, max_tokens)
