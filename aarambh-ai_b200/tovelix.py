"""Tovelix: a decoder that mixes layers of sliding-window attention (q and k rotated, then scaled to
unit RMS; values blended with those of the first layer that does so) and of lightning attention, with
sparse experts whose router scores scale what an expert reads.  The residual stream enters every
sublayer unnormalised and each sublayer's result is RMS-normed before it is added; the head is the
embedding table.

This module maps a checkpoint folder (config.json, model.safetensors) to a ``StackConfig`` and
its weights; the layers themselves are those of ``StackModel``.
"""
from __future__ import annotations

import json
import os

import torch

from .checkpoint import CheckpointError, read_safetensors
from .model import AttentionMixer, LightningMixer, MoeFfn, StackConfig, StackModel
from .qlinear import QuantLinear
from .registry import register


def _mixer(kind: str, m: dict, v_lambda):
    if kind == "lightning":
        return LightningMixer(m["heads"], m["dim"], m["vdim"], tuple(m["decay"]))
    if kind != "attention":
        raise CheckpointError(f"unknown mixer '{kind}'")
    rot, mask = m.get("rot") or {}, m.get("mask") or {}
    return AttentionMixer(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], mask.get("size", 0), rot.get("dims", 0),
                          rot.get("base", 1.0), True, bool(m.get("v_mix")), v_lambda if m.get("v_mix") else 0.0)


def _ffn(f):
    if f is None:
        return None
    if f["kind"] != "moe":
        raise CheckpointError(f"unknown feed-forward '{f['kind']}'")
    return MoeFfn(f["router"]["experts"], f["router"]["top"], f["expert"]["ff"], f["expert"]["limit"])


def stack_config(config: dict, tensors: dict, max_seq_len: int) -> StackConfig:
    """``config`` is config.json; of ``tensors`` only the scalars that are constants of a layer are read."""
    layers = []
    for i, entry in enumerate(config["layers"]):
        lam = tensors.get(f"l{i}.mix.vmix")
        layers.append((_mixer(entry["type"], entry["mixer"], 0.0 if lam is None else float(lam)), _ffn(entry.get("mlp"))))
    return StackConfig(config["width"], config["vocab"], layers, max_seq_len, config["norm"]["eps"])


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
    out = {"embedding": QuantLinear.from_bf16(get("embed", cfg.vocab_size, d)), "embed_norm": get("embed.norm", d),
           "final_norm": get("final.norm", d)}
    for i, (mix, ffn) in enumerate(cfg.layers):
        p, q = f"l{i}.", f"layers.{i}."
        hd, hv = mix.heads * mix.dim, mix.heads * mix.vdim
        if isinstance(mix, LightningMixer):
            rows = [("q", hd), ("k", hd), ("v", hv), ("g", hv)]
            out[q + "mix_norm"] = get(p + "mix.norm", hv)
        else:
            rows = [("q", hd), ("k", mix.kv_heads * mix.dim), ("v", mix.kv_heads * mix.vdim)]
        out[q + "in"] = QuantLinear.from_bf16(torch.cat([get(f"{p}mix.{n}", r, d) for n, r in rows]))
        out[q + "out"] = QuantLinear.from_bf16(get(p + "mix.o", d, hv))
        out[q + "norm1"] = get(p + "norm1", d)
        if ffn is None:
            continue
        out[q + "norm2"] = get(p + "norm2", d)
        out[q + "router"] = QuantLinear.from_bf16(get(p + "mlp.router", ffn.experts, d))
        for leaf, shape in (("gate", (ffn.ff, d)), ("up", (ffn.ff, d)), ("down", (d, ffn.ff))):
            out[q + leaf] = QuantLinear.from_bf16(torch.cat([get(f"{p}mlp.e{e}.{leaf}", *shape) for e in range(ffn.experts)]))
    return out


@register("Tovelix")
def load(path: str, dtype: torch.dtype = torch.bfloat16, max_tokens: int = 512, max_seq_len: int = 4096) -> StackModel:
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    tensors = read_safetensors(os.path.join(path, "model.safetensors"))
    cfg = stack_config(config, tensors, max_seq_len)
    return StackModel(cfg, stack_weights(cfg, tensors), dtype, max_tokens)
