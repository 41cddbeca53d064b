"""Vipelix without a GPU: the registry, the configuration, the weights' layout, the ABI's structures, and
the oracle itself - a sequence cut in two gives what it gives whole, and the inputs of the GPU tests do
expose the faults they are meant to expose (planted in the oracle here)."""
import ctypes as C

import numpy as np
import pytest
import torch

import vipelix_fixtures as fx
from helpers import pkg
from oracle import vipelix_ref as ref


def test_registry_and_configuration(tmp_path):
    p = pkg()
    fx.write_checkpoint(str(tmp_path / "m"), fx.VARIED, {})
    assert p.registry.loader_for(str(tmp_path / "m")) is p.vipelix.load
    cfg = p.vipelix.stack_config(fx.VARIED, fx.tensors(fx.weights(fx.VARIED)), 700)
    assert (cfg.d_model, cfg.vocab_size, cfg.max_seq_len, cfg.rms_norm_eps) == (72, 211, 700, 3e-5)
    assert cfg.runs() == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    specs, _ = cfg.c_specs()
    a, b = specs[1], specs[0]
    assert (a.mixer, a.heads, a.dim, a.rot_dims, a.vdim, a.kv_rank, a.rot_base, a.head_gate) == (2, 5, 20, 6, 18, 44, 70.0, 1)
    assert a.scale == np.float32(0.3) and (a.ffn, a.ff) == (2, 88) and list(a.poly) == list(fx.bf16_round([0.6, -0.4, 0.3, 0.1]))
    assert (b.ffn, b.experts, b.top, b.ff, b.shared_ff, b.glu, b.routing) == (1, 5, 2, 48, 72, 1, 1)
    assert specs[2].shared_ff == 0 and specs[3].ffn == 0
    runs, _ = cfg.c_specs(cfg.runs())
    assert len(runs) == 9 and [r.kv_rank for r in runs] == [56, 44, 128, 44, 128, 44, 128, 16, 72]
    f = cfg.c_form()
    assert (f.embed_norm, f.pre_norms, f.loop_start, f.loop_stop, f.loop_times, f.logit_softcap) == (0, 1, 1, 3, 3, 9.0)
    assert C.sizeof(p._lib.StackForm) == 24
    plain = p.vipelix.stack_config(fx.PLAIN, fx.tensors(fx.weights(fx.PLAIN)), 700)
    assert plain.runs() == [0, 1] and plain.c_form().loop_times == 0
    bad = fx.config([(fx.latent(), None)])
    bad["layers"][0]["type"] = "other"
    with pytest.raises(p.checkpoint.CheckpointError):
        p.vipelix.stack_config(bad, {}, 1)


def test_runs_agree_with_the_oracle():
    p = pkg()
    for c in (fx.VARIED, fx.ROUND, fx.PLAIN, fx.config([(fx.latent(), None)] * 4, loop=(2, 4, 2)), fx.config([(fx.latent(), None)] * 3, loop=(0, 2, 1))):
        assert p.vipelix.stack_config(c, fx.tensors(fx.weights(c)), 9).runs() == [i for i, _ in ref.runs(c)]


def test_an_attention_cut_in_two_is_the_whole():
    q, c, kr, uk, uv = (x.astype(np.float64) for x in fx.spiked_latents(40, 3, 16, 8, 12, 24, 30, (2, 5, 29), 1))
    whole = ref.latent_attention(q, c, kr, uk, uv, 0.3)
    parts = [ref.latent_attention(q[a:b], c[:b], kr[:b], uk, uv, 0.3, first=a) for a, b in ((0, 17), (17, 18), (18, 40))]
    assert np.allclose(np.concatenate(parts), whole)


@pytest.mark.parametrize("at,targets", [(70, (0, 1, 69)), (131, (63, 64, 127)), (200, (0, 128, 191))])
def test_spiked_inputs_expose_a_lost_key(at, targets):
    q, c, kr, uk, uv = (x.astype(np.float64) for x in fx.spiked_latents(at + 1, 3, 16, 8, 12, 48, at, targets, 5))
    good = ref.latent_attention(q[at:], c, kr, uk, uv, 0.3, first=at)
    for t in targets:
        bad = ref.latent_attention(q[at:], c, kr, uk, uv, 0.3, first=at, lost=(t,))
        assert np.abs(bad - good).max() > 0.2 * np.abs(good).max(), t


def test_models_expose_a_wrong_loop():
    for cfg in (fx.VARIED, fx.ROUND):
        w = fx.weights(cfg, 3)
        toks = np.random.default_rng(4).integers(0, cfg["vocab"], 12).tolist()
        good = fx.expected(cfg, w, toks)
        for fault in ({"stale_pass": True}, {"no_inject": True}, {"lost": (3,)}):
            assert fx.errors(fx.expected(cfg, w, toks, **fault), good).max() > 0.05, fault


def test_oracle_rotation_activation_and_cap():
    x = np.array([[1.0, 0.0, 0.0, 1.0]])
    a1 = 3 * 10.0 ** -0.5
    assert np.allclose(ref.turn_pairs(x, [3], 10.0), [[np.cos(3), np.sin(3), -np.sin(a1), np.cos(a1)]])
    z = np.array([3.0, -4.0])
    want = 2 * z / np.sqrt(12.5) + 3 * z ** 2 / np.sqrt((81 + 256) / 2) + 5 * z ** 3 / np.sqrt((729 + 4096) / 2) + 7
    assert np.allclose(ref.poly_norm(z, (2, 3, 5, 7), 0.0), want)
    assert np.isclose(ref.softcap(np.float64(4.0), 2.0), 2 * np.tanh(2.0)) and ref.softcap(4.0, None) == 4.0
    assert np.isclose(ref.silu(np.float64(2.0)), 2 / (1 + np.exp(-2.0)))


def test_weights_are_laid_out_head_by_head(monkeypatch):
    p = pkg()
    monkeypatch.setattr(p.vipelix.QuantLinear, "from_bf16", classmethod(lambda cls, t: t))
    w = fx.tensors(fx.weights(fx.VARIED, 2))
    cfg = p.vipelix.stack_config(fx.VARIED, w, 64)
    out = p.vipelix.stack_weights(cfg, w)
    ukv = out["layers.1.ukv"].view(5, 20 + 18, 44)
    assert torch.equal(ukv[3, :20], w["l1.mix.uk"][60:80]) and torch.equal(ukv[3, 20:], w["l1.mix.uv"][54:72])
    rows = out["layers.1.in"]
    n = 5 * 26
    assert len(rows) % 8 == 0 and torch.equal(rows[:n], w["l1.mix.q"]) and torch.equal(rows[n:n + 50], w["l1.mix.dkv"])
    assert torch.equal(rows[n + 50:n + 55], w["l1.mix.g"]) and not rows[n + 55:].any()
    w["l0.mlp.table"] = w["l0.mlp.table"][:, :1]
    with pytest.raises(p.checkpoint.CheckpointError, match="table"):
        p.vipelix.stack_weights(cfg, w)
