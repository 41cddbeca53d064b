"""Tovelix without a GPU: the checkpoint reader, the registry, the configuration, the ABI's layer
spec, and the oracle itself - its two forms of every recurrence and window agree, and the inputs the
GPU tests use do expose the faults they are meant to expose (planted in the oracle here)."""
import ctypes as C
import json
import struct

import numpy as np
import pytest
import torch

import tovelix_fixtures as fx
from helpers import pkg
from oracle import tovelix_ref as ref


def test_safetensors_reader(tmp_path):
    p = pkg()
    a = np.arange(6, dtype=np.int32).reshape(2, 3)
    b = torch.tensor([1.5, -2.0], dtype=torch.bfloat16)
    head = json.dumps({"__metadata__": {"x": "y"}, "t": {"dtype": "I32", "shape": [2, 3], "data_offsets": [0, 24]},
                       "s": {"dtype": "BF16", "shape": [], "data_offsets": [24, 26]},
                       "b": {"dtype": "BF16", "shape": [2], "data_offsets": [24, 28]}}).encode()
    f = tmp_path / "m.safetensors"
    f.write_bytes(struct.pack("<Q", len(head)) + head + a.tobytes() + b.view(torch.int16).numpy().tobytes())
    t = p.checkpoint.read_safetensors(str(f))
    assert set(t) == {"t", "s", "b"} and np.array_equal(t["t"].numpy(), a) and torch.equal(t["b"], b)
    assert t["s"].shape == () and float(t["s"]) == 1.5
    f.write_bytes(struct.pack("<Q", 1 << 40))
    with pytest.raises(p.checkpoint.CheckpointError):
        p.checkpoint.read_safetensors(str(f))
    head = json.dumps({"t": {"dtype": "BF16", "shape": [4], "data_offsets": [0, 4]}}).encode()
    f.write_bytes(struct.pack("<Q", len(head)) + head + b"\0" * 8)
    with pytest.raises(p.checkpoint.CheckpointError):
        p.checkpoint.read_safetensors(str(f))


def test_registry_knows_its_architectures(tmp_path):
    p = pkg()
    assert "Tovelix" in p.registry.architectures()
    fx.write_checkpoint(str(tmp_path / "m"), fx.VARIED, {})
    assert p.registry.loader_for(str(tmp_path / "m")) is p.tovelix.load
    assert callable(p.registry.loader_for("x.gguf"))
    (tmp_path / "m" / "config.json").write_text('{"architecture": "Unheard"}')
    with pytest.raises(p.registry.UnknownModelError, match="Unheard"):
        p.registry.loader_for(str(tmp_path / "m"))
    with pytest.raises(p.registry.UnknownModelError):
        p.registry.loader_for(str(tmp_path / "nothing"))


def test_configuration_reads_every_constant():
    p = pkg()
    w = {k: torch.from_numpy(np.asarray(v)) for k, v in fx.weights(fx.VARIED).items()}
    cfg = p.tovelix.stack_config(fx.VARIED, w, 777)
    assert (cfg.d_model, cfg.vocab_size, cfg.max_seq_len, cfg.rms_norm_eps, cfg.tie_embeddings) == (96, 203, 777, 1e-4, True)
    specs, _keep = cfg.c_specs()
    assert [s.mixer for s in specs] == [1, 0, 0, 1, 0]
    assert [specs[0].decay[i] for i in range(3)] == [np.float32(x) for x in (0.5, 0.93, 0.997)]
    a = specs[1]
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.rot_dims, a.rot_base, a.qk_norm) == (4, 2, 32, 48, 9, 16, 500.0, 1)
    assert a.scale == np.float32(0.3) and a.v_mix == 1 and a.v_lambda == float(w["l1.mix.vmix"])
    assert (specs[2].v_mix, specs[2].v_lambda, specs[2].ffn) == (0, 0.0, 0)
    assert (specs[1].experts, specs[1].top, specs[1].ff, specs[1].limit) == (4, 1, 40, np.float32(0.7))
    assert C.sizeof(p._lib.LayerSpec) == 120
    with pytest.raises(p.checkpoint.CheckpointError):
        p.tovelix.stack_config(dict(fx.VARIED, layers=[{"type": "other", "mixer": {}}]), w, 1)
    with pytest.raises(p.Ab2Error):
        p.LightningMixer and p.StackConfig(8, 8, [(p.LightningMixer(2, 8, 8, (0.5,)), None)], 8).c_specs()


def test_oracle_state_carries_over_a_cut():
    rng = np.random.default_rng(1)
    q, k, v = (rng.standard_normal((50, 2, n)) for n in (8, 8, 5))
    whole, end = ref.lightning_attention(q, k, v, (0.9, 0.99))
    a, s = ref.lightning_attention(q[:17], k[:17], v[:17], (0.9, 0.99))
    b, s2 = ref.lightning_attention(q[17:], k[17:], v[17:], (0.9, 0.99), s)
    assert np.allclose(np.concatenate([a, b]), whole) and np.allclose(s2, end)
    lost, _ = ref.lightning_attention(q[17:], k[17:], v[17:], (0.9, 0.99), s, drop_state=True)
    assert np.abs(lost - whole[17:]).max() > 0.1 * np.abs(whole).max()


def spiked_attention(T, H, G, dim, vdim, window, at, seed):
    """q, k, v in which the query at `at` scores high against the keys at the window's last place, the
    place before it and the place outside, so that a window off by one shows."""
    rng = np.random.default_rng(seed)
    q, k, v = rng.standard_normal((T, H, dim)), rng.standard_normal((T, G, dim)), rng.standard_normal((T, G, vdim))
    for back in (window - 1, window):
        if at - back >= 0:
            for g in range(G):
                k[at - back, g] = q[at, g * (H // G)] * 1.5
    return [fx.bf16_round(x) for x in (q, k, v)]


def test_spiked_inputs_expose_a_shifted_window():
    q, k, v = (x.astype(np.float64) for x in spiked_attention(60, 4, 2, 32, 16, 13, 50, 3))
    good = ref.window_attention(q, k, v, 0.3, 13)
    for shift in (-1, 1):
        bad = ref.window_attention(q, k, v, 0.3, 13, window_shift=shift)
        assert np.abs(bad[50] - good[50]).max() > 0.2 * np.abs(good).max()


def test_oracle_rotation_and_router():
    x = np.array([1.0, 0.0, 0.0, 1.0, 5.0, 6.0])
    y = ref.rotate_interleaved(x, 3, 4, 10.0)
    a1 = 3 * 10.0 ** -0.5
    assert np.allclose(y, [np.cos(3), np.sin(3), -np.sin(a1), np.cos(a1), 5.0, 6.0])
    chosen = ref.route(np.array([1.0, 0.0]), np.array([[0.1, 0], [3.0, 0], [-1, 0], [2.0, 0]]), 2)
    assert [e for e, _ in chosen] == [1, 3] and np.isclose(chosen[0][1], 1 / (1 + np.exp(-3.0)))
    assert np.isclose(ref.clamped_glu(np.float64(9.0), np.float64(-9.0), 2.0), 2.0 / (1 + np.exp(-1.702 * 2)) * -1.0)
