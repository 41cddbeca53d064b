"""Host-side mirror of the reference's model and engine entry points for the
dense grouped-query decoder: ``AarambhModel.forward_with_cache`` /
``forward_decode_batch`` / ``empty_kv_cache_with_capacity``
(crates/aarambh-studio-model/src/model.rs:508-662) and the greedy loop of
``InferenceEngine.generate_from_token_ids`` (crates/aarambh-studio-inference/src/
engine.rs:423-467) with ``Sampler`` argmax (sampler.rs:217-224).
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import torch

from . import _lib
from ._lib import ModelConfig as _CConfig, check, lib
from .kvcache import KVCache
from .qlinear import QuantLinear, dtype_code, stream_ptr

LAYER_LINEARS = ["wq", "wk", "wv", "wo", "w_gate", "w_up", "w_down"]


@dataclass
class ModelConfig:
    """The ModelConfig fields this path uses (crates/aarambh-studio-core/src/config.rs:734-868)."""
    n_layers: int
    d_model: int
    n_heads: int
    n_kv_heads: int
    head_dim: int
    ffn_hidden: int
    vocab_size: int
    max_seq_len: int
    rms_norm_eps: float = 1e-5
    rope_theta: float = 10000.0
    tie_embeddings: bool = True

    @classmethod
    def tiny_class(cls):
        return cls(6, 384, 6, 2, 64, 1024, 8192, 512)

    @classmethod
    def large_class(cls):
        return cls(32, 4096, 32, 8, 128, 14336, 32000, 1024, tie_embeddings=False)


class DecoderModel:
    """The step functions of a decoder handle (``ab2_model``), whatever layers it is made of.
    A subclass creates the handle and says what cache it takes."""

    dtype: torch.dtype            # activation type
    logits_dtype: torch.dtype     # element type of the logits

    def _create(self, fn, *args):
        h = C.c_void_p()
        check(fn(C.byref(h), *args))
        self._h = h

    def _norm(self, layer, which, w):
        w = w.detach().to(torch.float32).contiguous()
        check(lib.ab2_model_set_norm(self._h, layer, which, w.data_ptr()))

    def _ids(self, token_ids):
        ids = token_ids if isinstance(token_ids, torch.Tensor) else torch.tensor(token_ids)
        if ids.dim() != 2:
            raise _lib.Ab2Error(-1, f"token ids must have shape [batch, seq], got {list(ids.shape)}")
        if int(ids.max()) >= self.cfg.vocab_size or int(ids.min()) < 0:
            raise _lib.Ab2Error(-1, "token id outside the vocabulary")
        return ids.to(device="cuda", dtype=torch.int32).contiguous()

    def forward_with_cache(self, token_ids, seqlen_offset: int, cache: KVCache, row: int = 0,
                           last_only: bool = False) -> torch.Tensor:
        """ids [1, S] -> logits [1, S, vocab] (or [1, 1, vocab] with last_only)."""
        ids = self._ids(token_ids)
        if ids.shape[0] != 1:
            raise _lib.Ab2Error(-1, "forward_with_cache takes one sequence")
        S = ids.shape[1]
        out = torch.empty((1, 1 if last_only else S, self.cfg.vocab_size), dtype=self.logits_dtype, device="cuda")
        offs = (C.c_int * 1)(seqlen_offset)
        check(lib.ab2_model_forward(self._h, cache._h, ids.data_ptr(), S, row, 1, offs, 1 if last_only else 2,
                                    out.data_ptr(), None, stream_ptr()))
        return out

    def extend_cache(self, token_ids, cache: KVCache, row: int = 0) -> None:
        """Runs ids [1, S] from the row's cache length on for what they leave in the cache (no logits)."""
        ids = self._ids(token_ids)
        check(lib.ab2_model_forward(self._h, cache._h, ids.data_ptr(), ids.shape[1], row, 1, None, 0, None, None,
                                    stream_ptr()))

    def forward_decode_batch(self, token_ids, seqlen_offsets, cache: KVCache, row0: int = 0) -> torch.Tensor:
        """ids [B, 1], offsets [B] -> logits [B, 1, vocab]."""
        ids = self._ids(token_ids)
        if ids.shape[1] != 1:
            raise _lib.Ab2Error(-1, f"batched decode token ids must have shape [batch, 1], got {list(ids.shape)}")
        B = ids.shape[0]
        if len(seqlen_offsets) != B:
            raise _lib.Ab2Error(-1, f"batched decode received batch {B} and {len(seqlen_offsets)} offsets")
        out = torch.empty((B, 1, self.cfg.vocab_size), dtype=self.logits_dtype, device="cuda")
        offs = (C.c_int * B)(*[int(o) for o in seqlen_offsets])
        check(lib.ab2_model_forward(self._h, cache._h, ids.data_ptr(), 1, row0, B, offs, 1, out.data_ptr(), None,
                                    stream_ptr()))
        return out

    def forward_decode_rows(self, token_ids, rows, cache: KVCache) -> torch.Tensor:
        """One token for each of an arbitrary set of cache rows in ONE forward: ids [n, 1],
        rows [n] distinct cache rows; positions are the rows' cache lengths -> logits [n, 1, vocab]."""
        ids = self._ids(token_ids)
        rows = [int(r) for r in rows]
        if ids.shape[1] != 1 or ids.shape[0] != len(rows):
            raise _lib.Ab2Error(-1, f"expected ids [{len(rows)}, 1], got {list(ids.shape)}")
        n = len(rows)
        out = torch.empty((n, 1, self.cfg.vocab_size), dtype=self.logits_dtype, device="cuda")
        check(lib.ab2_model_forward_rows(self._h, cache._h, ids.data_ptr(), 1, (C.c_int * n)(*rows), n, 1,
                                         out.data_ptr(), None, stream_ptr()))
        return out

    def decode_step_rows(self, ids_dev: torch.Tensor, rows, cache: KVCache, logits: torch.Tensor | None,
                         argmax_dev: torch.Tensor | None):
        """Graph-replayed one-token step over an arbitrary set of cache rows (ids_dev [n] int32)."""
        rows = [int(r) for r in rows]
        n = len(rows)
        check(lib.ab2_model_decode_step_rows(self._h, cache._h, ids_dev.data_ptr(), (C.c_int * n)(*rows), n,
                                             logits.data_ptr() if logits is not None else None,
                                             argmax_dev.data_ptr() if argmax_dev is not None else None, stream_ptr()))

    def decode_step(self, ids_dev: torch.Tensor, cache: KVCache, logits: torch.Tensor | None,
                    argmax_dev: torch.Tensor | None, row0: int = 0):
        """Graph-replayed one-token step; ids_dev [B] int32 is read on the device."""
        check(lib.ab2_model_decode_step(self._h, cache._h, ids_dev.data_ptr(), row0, ids_dev.numel(),
                                        logits.data_ptr() if logits is not None else None,
                                        argmax_dev.data_ptr() if argmax_dev is not None else None, stream_ptr()))

    def decode_step_host(self, ids_host: torch.Tensor, cache: KVCache, out_host: torch.Tensor, row0: int = 0):
        """One greedy step with the tokens in host memory: ids_host [B] int32 in, out_host [B] int32
        out (pinned tensors make both copies asynchronous); returns when out_host is filled."""
        if ids_host.is_cuda or out_host.is_cuda or ids_host.dtype != torch.int32 or out_host.dtype != torch.int32:
            raise _lib.Ab2Error(-1, "decode_step_host takes int32 host tensors")
        if out_host.numel() < ids_host.numel() or not ids_host.is_contiguous() or not out_host.is_contiguous():
            raise _lib.Ab2Error(-1, "out_host must be contiguous and hold one token per row")
        check(lib.ab2_model_decode_step_host(self._h, cache._h, ids_host.data_ptr(), row0, ids_host.numel(),
                                             out_host.data_ptr(), stream_ptr()))

    def step_trace(self):
        """Phase timestamps (ns) of the last persistent one-row decode step as an int64
        array [3 CTAs, phases, 10]: phase start, prologue done, CTA done, barrier passed, then
        up to six points inside the phase (0 where unused)."""
        import numpy as np
        n = C.c_int(0)
        buf = np.zeros(3 * 4096 * 10, np.uint64)
        check(lib.ab2_model_step_trace(self._h, buf.ctypes.data, buf.size, C.byref(n)))
        return buf[:3 * n.value * 10].astype(np.int64).reshape(3, n.value, 10)

    def __del__(self):
        try:
            if self._h:
                lib.ab2_model_destroy(self._h)
                self._h = None
        except Exception:
            pass

class AarambhModel(DecoderModel):
    """weights: name -> QuantLinear for ``embedding``, optional ``lm_head`` and
    ``layers.{i}.{wq,wk,wv,wo,w_gate,w_up,w_down}``; name -> f32 tensor for
    ``final_norm`` and ``layers.{i}.{norm1,norm2}``."""

    def __init__(self, cfg: ModelConfig, weights: dict, dtype: torch.dtype = torch.float32,
                 max_tokens: int = 512, tp=None):
        """With ``tp`` (a ``parallel.TensorParallel``), ``cfg`` and ``weights`` are
        this rank's shard (``parallel.shard_config`` / ``shard_weight``)."""
        self.cfg, self.dtype, self.weights, self.tp = cfg, dtype, weights, tp
        c = _CConfig(cfg.n_layers, cfg.d_model, cfg.n_heads, cfg.n_kv_heads, cfg.head_dim, cfg.ffn_hidden,
                     cfg.vocab_size, cfg.max_seq_len, cfg.rms_norm_eps, cfg.rope_theta,
                     1 if cfg.tie_embeddings else 0)
        self.max_tokens, self.logits_dtype = max_tokens, dtype
        self._create(lib.ab2_model_create, C.byref(c), dtype_code(dtype), max_tokens)
        if tp is not None:
            check(lib.ab2_model_set_tp(self._h, tp._h))
        check(lib.ab2_model_set_linear(self._h, -1, 0, weights["embedding"]._h))
        if "lm_head" in weights:
            check(lib.ab2_model_set_linear(self._h, -1, 1, weights["lm_head"]._h))
        self._norm(-1, 0, weights["final_norm"])
        for l in range(cfg.n_layers):
            for which, name in enumerate(LAYER_LINEARS):
                check(lib.ab2_model_set_linear(self._h, l, which, weights[f"layers.{l}.{name}"]._h))
            self._norm(l, 0, weights[f"layers.{l}.norm1"])
            self._norm(l, 1, weights[f"layers.{l}.norm2"])
        check(lib.ab2_model_finalize(self._h))

    kv_dtype = "f32"   # of a cache that names none

    def empty_kv_cache_with_capacity(self, capacity: int, batch: int = 1, dtype: str = "f32") -> KVCache:
        c = self.cfg
        return KVCache(capacity, c.n_kv_heads, c.head_dim, c.n_heads, batch, c.n_layers, dtype)


@dataclass
class AttentionMixer:
    """Grouped-query softmax attention over a sliding window (``window`` keys, 0: all of them)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0
    rot_dims: int = 0             # leading dimensions rotated, in adjacent pairs
    rot_base: float = 10000.0
    qk_norm: bool = False         # q and k divided by their root mean square after the rotation
    v_mix: bool = False           # values mixed with those of the stack's first such layer
    v_lambda: float = 0.0


@dataclass
class LightningMixer:
    """Linear attention with one decay per head."""
    heads: int
    dim: int
    vdim: int
    decay: tuple


@dataclass
class LatentMixer:
    """Causal softmax attention whose keys and values are projections of one cached latent per token, plus
    a rotated key part that the heads share."""
    heads: int
    dim: int                      # unrotated dimensions of a query and key
    rot_dims: int                 # rotated ones besides, in adjacent pairs
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float = 10000.0
    head_gate: bool = False       # a head's output times the sigmoid of a gate value of its own


@dataclass
class MoeFfn:
    """Mixture of experts over gated units: ``clamped`` (with ``limit``) or ``silu``.  ``sigmoid`` routing: a
    router's largest scores, which multiply what the experts read.  ``table`` routing: the token id
    names the experts, each output weighs 1 / top."""
    experts: int
    top: int
    ff: int
    limit: float = 0.0
    glu: str = "clamped"
    routing: str = "sigmoid"
    shared_ff: int = 0            # width of an expert that runs for every token, 0: none


@dataclass
class PolyFfn:
    """W_down act(W_up x) with act(z) = a N(z) + b N(z^2) + c N(z^3) + e, N(z) = z / rms(z) over the row."""
    ff: int
    coef: tuple                   # a, b, c, e


@dataclass
class StackConfig:
    """A decoder listed layer by layer: ``layers`` holds (mixer, feed-forward or None) pairs."""
    d_model: int
    vocab_size: int
    layers: list
    max_seq_len: int
    rms_norm_eps: float = 1e-5
    tie_embeddings: bool = True
    embed_norm: bool = True       # the embedding is normed
    pre_norms: bool = False       # sublayers read a norm of the residual stream
    loop: tuple | None = None     # (start, stop, times): those layers run that often in a row
    logit_softcap: float = 0.0    # cap of tanh-capped logits, 0: none

    def runs(self) -> list:
        """Layer indices in the order in which a pass runs them; each run has a cache layer of its own."""
        start, stop, times = self.loop or (0, 0, 0)
        n = len(self.layers)
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    def c_specs(self, order=None):
        """The layers (or those of ``order``) as an array of ab2_layer_spec (and what it points to)."""
        order = range(len(self.layers)) if order is None else order
        arr = (_lib.LayerSpec * len(order))()
        keep = []
        for s, i in zip(arr, order):
            mix, ffn = self.layers[i]
            s.heads, s.dim, s.vdim = mix.heads, mix.dim, mix.vdim
            if isinstance(mix, LatentMixer):
                s.mixer = _lib.MIX_LATENT
                s.kv_rank, s.rot_dims, s.rot_base, s.scale, s.head_gate = mix.kv_rank, mix.rot_dims, mix.rot_base, mix.scale, int(mix.head_gate)
            elif isinstance(mix, LightningMixer):
                if len(mix.decay) != mix.heads:
                    raise _lib.Ab2Error(-1, f"{len(mix.decay)} decays for {mix.heads} heads")
                s.mixer = _lib.MIX_LIGHTNING
                keep.append((C.c_float * mix.heads)(*mix.decay))
                s.decay = C.cast(keep[-1], C.POINTER(C.c_float))
            else:
                s.mixer = _lib.MIX_ATTENTION
                s.kv_heads, s.window, s.scale = mix.kv_heads, mix.window, mix.scale
                s.rot_dims, s.rot_base, s.qk_norm = mix.rot_dims, mix.rot_base, int(mix.qk_norm)
                s.v_mix, s.v_lambda = int(mix.v_mix), mix.v_lambda
            if isinstance(ffn, PolyFfn):
                s.ffn, s.ff = _lib.FFN_POLY, ffn.ff
                s.poly[:] = ffn.coef
            elif ffn is not None:
                s.ffn, s.experts, s.top, s.ff, s.limit = _lib.FFN_MOE, ffn.experts, ffn.top, ffn.ff, ffn.limit
                s.glu, s.routing, s.shared_ff = _lib.GLU[ffn.glu], _lib.ROUTING[ffn.routing], ffn.shared_ff
        return arr, keep

    def c_form(self):
        start, stop, times = self.loop or (0, 0, 0)
        return _lib.StackForm(int(self.embed_norm), int(self.pre_norms), start, stop, times, self.logit_softcap)


class StackModel(DecoderModel):
    """A decoder made of layer specs (``StackConfig``) over dense bf16 weights.

    weights: name -> ``QuantLinear.from_bf16`` for ``embedding``, optional ``lm_head`` and
    ``layers.{i}.{in,out}`` (the mixer's input projections as one weight: q | k | v, lightning
    q | k | v | g, latent q | latent | key part | g and zero rows up to a multiple of 8), latent
    ``layers.{i}.ukv`` (head by head the rows of its keys and its values), ``layers.{i}.{gate,up,down,router}``
    (the experts one after the other) and ``layers.{i}.shared_{gate,up,down}``;
    name -> f32 tensor for ``embed_norm``, ``final_norm``, ``layers.{i}.{norm1,norm2}`` (after the mixer and the
    feed-forward), with ``pre_norms`` ``layers.{i}.{pre1,pre2}`` (before them), in lightning and latent layers
    ``layers.{i}.mix_norm``, with a loop ``loop_steps`` [times, d_model]; ``layers.{i}.table`` [vocab, top] int32 where
    the token id names the experts.  Logits are f32."""

    LINEARS = {"in": 0, "ukv": 1, "out": 3, "gate": 4, "up": 5, "down": 6, "router": 7, "shared_gate": 8, "shared_up": 9, "shared_down": 10}
    NORMS = {"norm1": 0, "norm2": 1, "mix_norm": 2, "pre1": 3, "pre2": 4}

    def __init__(self, cfg: StackConfig, weights: dict, dtype: torch.dtype = torch.bfloat16, max_tokens: int = 512):
        self.cfg, self.dtype, self.weights, self.tp = cfg, dtype, weights, None
        self.max_tokens, self.logits_dtype = max_tokens, torch.float32
        specs, _keep = cfg.c_specs()
        c = _CConfig(n_layers=len(cfg.layers), d_model=cfg.d_model, vocab=cfg.vocab_size, max_seq=cfg.max_seq_len,
                     rms_eps=cfg.rms_norm_eps, tied=1 if cfg.tie_embeddings else 0)
        self._create(lib.ab2_model_create_stack, C.byref(c), specs, dtype_code(dtype), max_tokens)
        check(lib.ab2_model_set_form(self._h, C.byref(cfg.c_form())))
        for name, w in weights.items():
            layer, leaf = -1, name
            if name.startswith("layers."):
                layer, leaf = int(name.split(".")[1]), name.split(".")[2]
            if layer < 0 and leaf in ("embedding", "lm_head"):
                check(lib.ab2_model_set_linear(self._h, -1, int(leaf == "lm_head"), w._h))
            elif leaf == "loop_steps":
                w = w.detach().to(torch.float32).contiguous()
                check(lib.ab2_model_set_loop_steps(self._h, w.data_ptr()))
            elif leaf == "table":
                w = w.detach().to(torch.int32).contiguous()
                check(lib.ab2_model_set_expert_table(self._h, layer, w.data_ptr()))
            elif layer < 0:
                self._norm(-1, int(leaf == "embed_norm"), w)
            elif leaf in self.NORMS:
                self._norm(layer, self.NORMS[leaf], w)
            else:
                check(lib.ab2_model_set_linear(self._h, layer, self.LINEARS[leaf], w._h))
        check(lib.ab2_model_finalize(self._h))

    @property
    def kv_dtype(self) -> str:
        return "f32" if self.dtype == torch.float32 else "bf16"

    def empty_kv_cache_with_capacity(self, capacity: int, batch: int = 1, dtype: str | None = None) -> KVCache:
        if dtype not in (None, self.kv_dtype):
            raise _lib.Ab2Error(-3, f"this model caches {self.kv_dtype}, not {dtype}")
        return KVCache.for_stack(self.cfg, capacity, batch, self.max_tokens, self.kv_dtype)


class InferenceEngine:
    """Greedy generation from raw token ids, at model level: exactly
    ``max_new_tokens`` steps, no end-of-text stop (the reference engine stops on
    token 0, crates/aarambh-studio-inference/src/engine.rs:898-911; ``eos_step``
    reports where it would have)."""

    def __init__(self, model: DecoderModel, kv_dtype: str | None = None):
        self.model, self.kv_dtype = model, kv_dtype or model.kv_dtype

    def generate_from_token_ids(self, prompt_ids, max_new_tokens: int, eos_token_id: int = 0,
                                on_device_sampling: bool = True):
        m = self.model
        prompt = torch.as_tensor(prompt_ids, dtype=torch.int64).view(1, -1)
        P = prompt.shape[1]
        if P + max_new_tokens > m.cfg.max_seq_len:
            raise _lib.Ab2Error(-1, "prompt plus new tokens exceed max_seq_len")
        cache = m.empty_kv_cache_with_capacity(P + max_new_tokens, 1, self.kv_dtype)
        from .dispatch import argmax
        stream = torch.cuda.Stream()   # a capturable (non-default) stream for the graph-replayed steps
        stream.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(stream):
            step = m.max_tokens        # a long prompt goes in as many portions as the workspace asks for
            for off in range(0, P, step):
                logits = m.forward_with_cache(prompt[:, off:off + step], off, cache, last_only=True)
            tokens = torch.empty(max_new_tokens, dtype=torch.int32, device="cuda")
            tokens[0:1] = argmax(logits.view(1, -1))
            if on_device_sampling:
                # two token buffers alternate as input and output, so two graphs
                # serve every step and no token visits the host
                bufs = [tokens[0:1].clone(), torch.empty(1, dtype=torch.int32, device="cuda")]
                for i in range(1, max_new_tokens):
                    m.decode_step(bufs[(i - 1) % 2], cache, None, bufs[i % 2])
                    tokens[i:i + 1].copy_(bufs[i % 2])
            else:
                for i in range(1, max_new_tokens):
                    lg = m.forward_decode_batch(tokens[i - 1:i].view(1, 1), [P + i - 1], cache)
                    tokens[i:i + 1] = argmax(lg.view(1, -1))
        torch.cuda.current_stream().wait_stream(stream)
        stream.synchronize()
        out = tokens.cpu().tolist()
        eos_step = next((i for i, t in enumerate(out) if t == eos_token_id), None)
        return {"token_ids": out, "eos_step": eos_step, "cache": cache}
