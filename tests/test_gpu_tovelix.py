"""Tovelix on the GPU against the plain numpy restatement: every mechanism alone, then the model
through its own cache, portions, batches, sessions and generation."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import tovelix_fixtures as fx
from helpers import ROOT, pkg, rel_err
from oracle import tovelix_ref as ref
from test_tovelix_host import spiked_attention

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def tol(dtype, f32, b16):
    return f32 if dtype == torch.float32 else b16


def to_gpu(a, dtype):
    return torch.from_numpy(np.ascontiguousarray(a, np.float32)).to(dtype).cuda()


# ---------------------------------------------------------------- linears

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,K", [(16, 64), (203, 96), (130, 40), (77, 51), (640, 264)])
def test_dense_linear(dtype, N, K):
    rng = np.random.default_rng(N + K)
    w = fx.bf16_round(rng.standard_normal((N, K)))
    lin = pkg().QuantLinear.from_bf16(torch.from_numpy(w).to(torch.bfloat16))
    assert torch.equal(lin.dequantise().cpu(), torch.from_numpy(w))
    for M in (1, 3, 8, 9, 17, 32, 33, 100, 300, 700):
        x = fx.bf16_round(rng.standard_normal((M, K)))
        y = lin(to_gpu(x, dtype)).float().cpu().numpy()
        assert rel_err(y, x.astype(np.float64) @ w.T.astype(np.float64)) < tol(dtype, 1e-5, 5e-3), M
    assert pkg().device_status() == 0


def expert_weights(rng, E, ff, d):
    p = pkg()
    w = {"r": rng.standard_normal((E, d)) * 2 / np.sqrt(d), "g": rng.standard_normal((E * ff, d)) / np.sqrt(d) * 2,
         "u": rng.standard_normal((E * ff, d)) / np.sqrt(d) * 2, "d": rng.standard_normal((E * d, ff)) / np.sqrt(ff)}
    w = {k: fx.bf16_round(v) for k, v in w.items()}
    return w, [p.QuantLinear.from_bf16(torch.from_numpy(w[k]).to(torch.bfloat16)) for k in "rgud"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,top,ff,d", [(5, 2, 56, 96), (1, 1, 64, 64), (40, 3, 24, 72), (8, 8, 136, 128), (3, 1, 30, 50)])
def test_mixture_of_experts(dtype, E, top, ff, d):
    p = pkg()
    rng = np.random.default_rng(E * 100 + top)
    w, lin = expert_weights(rng, E, ff, d)
    limit = 0.8
    experts = p.dispatch.MoeExperts(p.MoeFfn(E, top, ff, limit), *lin)
    for T in (1, 2, 7, 16, 33, 70, 260):
        x = fx.bf16_round(rng.standard_normal((T, d)))
        got = experts(to_gpu(x, dtype)).cpu().numpy()
        x64 = x.astype(np.float64)
        bad = 0
        for t in range(T):
            chosen = ref.route(x64[t], w["r"].astype(np.float64), top)
            for slot, (e, s) in enumerate(chosen):
                want = ref.expert(s * x64[t], w["g"][e * ff:(e + 1) * ff].astype(np.float64), w["u"][e * ff:(e + 1) * ff].astype(np.float64),
                                  w["d"][e * d:(e + 1) * d].astype(np.float64), np.float64(limit))
                bad += not np.abs(got[t, slot] - want).max() <= tol(dtype, 1e-5, 1.5e-2) * np.abs(want).max()
        assert bad == 0, (T, bad)
    assert p.device_status() == 0


def test_router_takes_every_token_to_one_expert():
    """All pairs on one expert, the others empty, in the decode and the prompt kernels."""
    p = pkg()
    rng = np.random.default_rng(9)
    E, ff, d = 6, 64, 64
    w, lin = expert_weights(rng, E, ff, d)
    w["r"][:] = 0
    w["r"][4, 0] = 4.0
    lin[0] = p.QuantLinear.from_bf16(torch.from_numpy(w["r"]).to(torch.bfloat16))
    experts = p.dispatch.MoeExperts(p.MoeFfn(E, 1, ff, 2.0), *lin)
    for T in (5, 40, 300):
        x = fx.bf16_round(rng.standard_normal((T, d)))
        x[:, 0] = 1.0
        got = experts(to_gpu(x, torch.bfloat16)).cpu().numpy()[:, 0]
        s = 1 / (1 + np.exp(-4.0))
        want = np.stack([ref.expert(s * r, *(w[k][4 * n:5 * n].astype(np.float64) for k, n in (("g", ff), ("u", ff), ("d", d))), np.float64(2.0))
                         for r in x.astype(np.float64)])
        assert rel_err(got, want) < 1e-2


# ---------------------------------------------------------------- mixers alone

def feed_portions(T, sizes):
    """Cuts 0..T into portions whose sizes repeat `sizes`."""
    cuts, i = [0], 0
    while cuts[-1] < T:
        cuts.append(min(T, cuts[-1] + sizes[i % len(sizes)]))
        i += 1
    return list(zip(cuts, cuts[1:]))


PORTIONS = [[10**9], [1], [2, 3], [64, 1, 17, 5], [33, 40, 2]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,window,T", [(4, 2, 32, 48, 13, 120), (6, 6, 64, 64, 72, 150), (9, 1, 24, 40, 1, 50), (2, 1, 128, 80, 33, 140),
                                                   (16, 1, 8, 8, 30, 90), (2, 2, 160, 200, 17, 60), (3, 3, 20, 12, 0, 70)])
def test_window_attention(dtype, H, G, dim, vdim, window, T):
    p = pkg()
    W = window or T
    at = min(T - 1, W + 20)
    q, k, v = spiked_attention(T, H, G, dim, vdim, W, at, H * 100 + dim)
    want = ref.window_attention(*(x.astype(np.float64) for x in (q, k, v)), 0.3, W)
    qkv = np.concatenate([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1)
    mix = p.AttentionMixer(H, G, dim, vdim, 0.3, window)
    cfg = p.StackConfig(64, 64, [(mix, None)], 4 * T)
    for sizes in PORTIONS:
        parts = feed_portions(T, sizes)
        cache = p.KVCache.for_stack(cfg, 2 * T, 2, max(b - a for a, b in parts), "f32" if dtype == torch.float32 else "bf16")
        for row in (1, 0):
            got = []
            for a, b in parts:
                got.append(p.dispatch.window_attention(cache, cfg, 0, to_gpu(qkv[None, a:b], dtype), None, 1e-5, row0=row))
                cache.commit(b - a, row, 1)
            got = torch.cat(got, 1)[0].float().cpu().numpy().reshape(T, H, vdim)
            assert rel_err(got, want) < tol(dtype, 1e-5, 6e-3), sizes
            assert np.abs(got[at] - want[at]).max() < tol(dtype, 1e-5, 6e-3) * np.abs(want).max(), sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_normalisation_and_value_mixing(dtype):
    p = pkg()
    T, H, G, dim, vdim, rot, base, eps, lam = 90, 4, 2, 48, 24, 20, 700.0, 1e-3, 0.375
    rng = np.random.default_rng(2)
    q, k, v, first = (fx.bf16_round(rng.standard_normal((T, n, m))) for n, m in ((H, dim), (G, dim), (G, vdim), (G, vdim)))
    qr, kr = q.astype(np.float64), k.astype(np.float64)
    for t in range(T):
        qr[t], kr[t] = ref.rotate_interleaved(qr[t], t, rot, base), ref.rotate_interleaved(kr[t], t, rot, base)
    mixed = ref.mix_values(v.astype(np.float64), first.astype(np.float64), lam)
    want = ref.window_attention(ref.rms(qr, eps), ref.rms(kr, eps), mixed, 0.2, 30)
    mix = p.AttentionMixer(H, G, dim, vdim, 0.2, 30, rot, base, True, True, lam)
    cfg = p.StackConfig(64, 64, [(mix, None)], 256)
    cache = p.KVCache.for_stack(cfg, 128, 1, 64, "f32" if dtype == torch.float32 else "bf16")
    tables = p.dispatch.rotation_tables(256, rot, base)
    qkv = to_gpu(np.concatenate([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1)[None], dtype)
    got = []
    for a, b in feed_portions(T, [50, 1, 20]):
        f = to_gpu(first[a:b].reshape(b - a, -1), dtype)
        got.append(p.dispatch.window_attention(cache, cfg, 0, qkv[:, a:b].contiguous(), tables, eps, f, 2))
        cache.commit(b - a, 0, 1)
    got = torch.cat(got, 1)[0].float().cpu().numpy().reshape(T, H, vdim)
    assert rel_err(got, want) < tol(dtype, 1e-5, 1e-2)
    # mode 1 hands the values on as they are
    kept = torch.zeros((3, G * vdim), dtype=dtype, device="cuda")
    p.dispatch.window_attention(p.KVCache.for_stack(cfg, 128, 1, 64, "f32" if dtype == torch.float32 else "bf16"), cfg, 0,
                                qkv[:, :3].contiguous(), tables, eps, kept, 1)
    assert torch.equal(kept.float().cpu(), torch.from_numpy(v[:3].reshape(3, -1)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,vdim,decay", [(3, 40, 24, (0.5, 0.93, 0.997)), (2, 64, 72, (0.02, 1.0)), (1, 128, 128, (0.99,)), (2, 96, 64, (0.0, 0.9)),
                                              (2, 200, 33, (0.95, 0.7)), (1, 13, 9, (0.9,)), (40, 32, 64, (0.98,) * 40)])
def test_lightning_attention(dtype, H, dim, vdim, decay):
    p = pkg()
    T = 210
    rng = np.random.default_rng(H + dim)
    q, k, v = (fx.bf16_round(rng.standard_normal((T, H, n)) * 0.5 + 0.2) for n in (dim, dim, vdim))
    k[3] *= 8      # a far key that still shows at the end of a slow head
    want, _ = ref.lightning_attention(*(x.astype(np.float64) for x in (q, k, v)), np.float32(decay).astype(np.float64))
    qkv = np.concatenate([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1)
    cfg = p.StackConfig(64, 64, [(p.LightningMixer(H, dim, vdim, decay), None)], 256)
    cache = p.KVCache.for_stack(cfg, 256, 2, 256, "f32" if dtype == torch.float32 else "bf16")
    powers = p.dispatch.decay_powers(np.float32(decay).tolist())
    for sizes in PORTIONS:
        for row in (1, 0, 1):   # a row used again starts from nothing
            cache.truncate(0, row)
            got = []
            for a, b in feed_portions(T, sizes):
                got.append(p.dispatch.lightning_attention(cache, cfg, 0, to_gpu(qkv[None, a:b], dtype), powers, row0=row))
                cache.commit(b - a, row, 1)
            got = torch.cat(got, 1)[0].cpu().numpy().reshape(T, H, vdim)
            for h in range(H):
                assert rel_err(got[:, h], want[:, h]) < tol(dtype, 2e-5, 1e-4), (sizes, h)


@pytest.mark.parametrize("H,dim,vdim,T,rows", [(2, 64, 64, 1500, 1), (3, 128, 72, 700, 2), (1, 40, 24, 4100, 1)])
def test_lightning_segments(H, dim, vdim, T, rows):
    """Long prompts cut into segments that run side by side, on a row that already holds a state."""
    p = pkg()
    rng = np.random.default_rng(T)
    decay = np.float32([0.9985, 0.6, 1.0][:H])
    q, k, v = (fx.bf16_round(rng.standard_normal((rows, T, H, n)) * 0.3 + 0.1) for n in (dim, dim, vdim))
    want = np.stack([ref.lightning_attention(q[r].astype(np.float64), k[r].astype(np.float64), v[r].astype(np.float64), decay.astype(np.float64))[0]
                     for r in range(rows)])
    qkv = to_gpu(np.concatenate([x.reshape(rows, T, -1) for x in (q, k, v)], 2), torch.bfloat16)
    cfg = p.StackConfig(64, 64, [(p.LightningMixer(H, dim, vdim, decay.tolist()), None)], 2 * T)
    powers, scratch = p.dispatch.decay_powers(decay.tolist()), p.dispatch.lightning_scratch(cfg, 0)
    for cuts in ([0, T], [0, 19, T - 33, T], [0, 600, T]):
        cache = p.KVCache.for_stack(cfg, 2 * T, rows, T, "bf16")
        got = []
        for a, b in zip(cuts, cuts[1:]):
            got.append(p.dispatch.lightning_attention(cache, cfg, 0, qkv[:, a:b].contiguous(), powers, scratch=scratch))
            cache.commit(b - a)
        got = torch.cat(got, 1).cpu().numpy().reshape(want.shape)
        for r in range(rows):
            for h in range(H):
                assert rel_err(got[r, :, h], want[r, :, h]) < 1e-4, (cuts, r, h)


# ---------------------------------------------------------------- the model

def tokens_of(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def check_logits(got, want, dtype, steady=True):
    e = errors = fx.errors(got, want)
    if dtype == torch.float32:
        assert e.max() < 2e-4, (int(e.argmax()), e.max())
    elif steady:
        assert errors.max() < 4e-2, (int(e.argmax()), e.max())
    else:  # rounding may flip a close choice of experts at a few tokens
        assert np.median(e) < 4e-2 and (e > 8e-2).mean() < 0.15, (np.median(e), np.sort(e)[-8:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["VARIED", "STEADY"])
def test_prompt_portions_and_decoding(tmp_path, dtype, name):
    cfg = getattr(fx, name)
    w = fx.weights(cfg, 5)
    toks = tokens_of(190, cfg["vocab"], 6)
    want = fx.expected(cfg, w, toks)
    m = fx.load(tmp_path, cfg, w, dtype, max_tokens=256, max_seq_len=256)
    eng = pkg().sessions.SessionEngine(m, max_batch=2, capacity=256)
    alone = None
    for sizes in PORTIONS:
        row = eng.open_row()
        got = torch.cat([eng.feed(row, toks[a:b], range(b - a)).clone() for a, b in feed_portions(len(toks), sizes)])
        eng.close_row(row)
        check_logits(got, want, dtype, name == "STEADY")
        alone = got if alone is None else alone
    # a portion larger than the workspace goes in pieces
    small = fx.load(tmp_path, cfg, w, dtype, max_tokens=48, max_seq_len=256)
    eng = pkg().sessions.SessionEngine(small, max_batch=1, capacity=256)
    row = eng.open_row()
    want_at = [0, 1, 47, 48, 95, 130, 189]
    check_logits(eng.feed(row, toks, want_at), want[want_at], dtype, name == "STEADY")
    assert pkg().device_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_of_unequal_requests(tmp_path, dtype):
    """Requests of different lengths in the rows of one cache, decoded together in changing sets, rows
    given back and taken again: the logits are those of each request alone."""
    p, cfg = pkg(), fx.STEADY
    w = fx.weights(cfg, 11)
    m = fx.load(tmp_path, cfg, w, dtype, max_tokens=128, max_seq_len=256)
    cache = m.empty_kv_cache_with_capacity(200, batch=5)
    seqs = {r: tokens_of(n, cfg["vocab"], 20 + r) for r, n in enumerate((9, 1, 75, 40, 100))}
    want = {r: fx.expected(cfg, w, s + tokens_of(30, cfg["vocab"], 40 + r)) for r, s in seqs.items()}
    full = {r: s + tokens_of(30, cfg["vocab"], 40 + r) for r, s in seqs.items()}
    at = {}
    for r in (3, 0, 4, 1, 2):
        m.extend_cache(torch.tensor([full[r][:len(seqs[r])]]), cache, r)
        at[r] = len(seqs[r])
    for step, live in enumerate([[0, 1, 2, 3, 4], [4, 2, 0], [1], [3, 1, 4], [0, 1, 2, 3, 4], [2, 3]] * 3):
        ids = torch.tensor([[full[r][at[r]]] for r in live])
        lg = m.forward_decode_rows(ids, live, cache) if step % 2 else None
        if lg is None:
            lg = torch.empty((len(live), 1, cfg["vocab"]), device="cuda")
            stream = torch.cuda.Stream()
            stream.wait_stream(torch.cuda.current_stream())
            with torch.cuda.stream(stream):
                m.decode_step_rows(ids.to(torch.int32).cuda().view(-1), live, cache, lg, None)
            stream.synchronize()
        check_logits(lg[:, 0], np.stack([want[r][at[r]] for r in live]), dtype)
        for r in live:
            at[r] += 1
    # two rows at once through a prompt pass, then a row taken by a new request
    cache.truncate(0, 0)
    cache.truncate(0, 1)
    two = torch.tensor([full[2][:50], full[4][:50]])
    out = torch.empty((2, 50, cfg["vocab"]), device="cuda")
    p.check(p.lib.ab2_model_forward(m._h, cache._h, two.to(torch.int32).cuda().data_ptr(), 50, 0, 2, None, 2, out.data_ptr(), None,
                                    torch.cuda.current_stream().cuda_stream))
    check_logits(out[0], want[2][:50], dtype)
    check_logits(out[1], want[4][:50], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_past_every_ring(tmp_path, dtype):
    """Hundreds of decoded tokens: the windows' rings go round several times."""
    cfg = fx.STEADY
    w = fx.weights(cfg, 13)
    toks = tokens_of(330, cfg["vocab"], 14)
    m = fx.load(tmp_path, cfg, w, dtype, max_tokens=16, max_seq_len=400)
    eng = pkg().sessions.SessionEngine(m, max_batch=1, capacity=400)
    row = eng.open_row()
    eng.feed(row, toks[:11])
    got = torch.cat([eng.feed(row, [t], [0]).clone() for t in toks[11:]])
    check_logits(got, fx.expected(cfg, w, toks)[11:], dtype)


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        lg = fx.expected(cfg, w, toks)[-1]
        toks.append(int(len(lg) - 1 - np.argmax(lg[::-1])))
    return toks[len(prompt):]


def test_greedy_generation(tmp_path):
    """The engine and the session scheduler produce the restated model's tokens (f32)."""
    p, cfg = pkg(), fx.VARIED
    w = fx.weights(cfg, 17)
    m = fx.load(tmp_path, cfg, w, torch.float32, max_tokens=32, max_seq_len=128)
    prompts = [tokens_of(n, cfg["vocab"], 50 + n) for n in (41, 3)]
    want = [greedy(cfg, w, q, 12) for q in prompts]
    eng = p.InferenceEngine(m)
    for q, t in zip(prompts, want):
        assert eng.generate_from_token_ids(q, 12)["token_ids"] == t
        assert eng.generate_from_token_ids(q, 12, on_device_sampling=False)["token_ids"] == t
    se = p.sessions.SessionEngine(m, max_batch=2, capacity=100)
    live = [se.prepare_session_with_chunk_size(q, 12, chunk_size=7) for q in prompts]
    while any(not s.finished for s in live):
        for s in live:
            se.advance(s)
        se.decode_sessions([s for s in live if not s.finished])
    assert [s.generated_ids for s in live] == want


def run_program(name, args, text=""):
    exe = os.path.join(ROOT, "bin", name)
    res = subprocess.run([exe, *args], input=text, capture_output=True, text=True, timeout=240)
    assert res.returncode == 0, res.stderr[-2000:]
    return res.stdout


def test_command_line_programs(tmp_path):
    """bin/generate and bin/trace_run on a checkpoint folder."""
    cfg = fx.VARIED
    w = fx.weights(cfg, 17)
    folder = fx.write_checkpoint(str(tmp_path / "m"), cfg, w)
    prompts = [tokens_of(n, cfg["vocab"], 50 + n) for n in (21, 3)]
    want = [greedy(cfg, w, q, 5) for q in prompts]
    base = ["--model", folder, "--dtype", "float32", "--max-new-tokens", "5"]
    args = [["--tokens", ",".join(map(str, q))] for q in prompts]
    one = run_program("generate", base + args[0])
    two = run_program("generate", base + args[0] + args[1])
    assert [json.loads(x)["tokens"] for x in one.splitlines()] == want[:1]
    assert [json.loads(x)["tokens"] for x in two.splitlines()] == want
    q = prompts[0]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": q[:9], "want": [0, 8]}, {"id": "b", "tokens": q[:4], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": q[4:5], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": q[9:20], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": q[20:], "want": [0]}, {"id": "c", "tokens": q[:2], "want": [1]}], "end": ["a", "c"]}]
    out = run_program("trace_run", ["--model", folder, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "40"],
                      "\n".join(map(json.dumps, steps)) + "\n")
    assert [x for x in out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    full = fx.expected(cfg, w, q)
    for step, at in ((0, [0, 8]), (1, [4]), (3, [20, 1])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(at), cfg["vocab"])
        check_logits(got.astype(np.float64), full[at], torch.float32)
    assert not (tmp_path / "2.f32").exists()


def test_draft_verification_restores_the_state(tmp_path):
    p, cfg = pkg(), fx.VARIED
    w = fx.weights(cfg, 19)
    m = fx.load(tmp_path, cfg, w, torch.float32, max_tokens=64, max_seq_len=128)
    prompt = tokens_of(20, cfg["vocab"], 60)
    tail = greedy(cfg, w, prompt, 6)
    cache = m.empty_kv_cache_with_capacity(100)
    m.extend_cache(torch.tensor([prompt]), cache)
    wrong = [(t + 1) % cfg["vocab"] for t in tail]
    accepted, nxt, _ = p.sessions.verify_draft(m, cache, 0, 20, tail[0], [tail[1], tail[2], wrong[3], tail[4]])
    assert (accepted, nxt, cache.seq_len(0)) == (2, tail[3], 23)
    accepted, nxt, lg = p.sessions.verify_draft(m, cache, 0, 23, tail[3], [tail[4]])
    assert (accepted, nxt, cache.seq_len(0)) == (1, tail[5], 25)
    check_logits(lg, fx.expected(cfg, w, prompt + tail[:5])[-2:], torch.float32)


def test_cache_refuses_what_it_cannot_do(tmp_path):
    p, cfg = pkg(), fx.STEADY
    w = fx.weights(cfg, 23)
    m = fx.load(tmp_path, cfg, w, torch.float32, max_tokens=32, max_seq_len=64)
    cache = m.empty_kv_cache_with_capacity(40)
    assert cache.has_state()
    m.extend_cache(torch.tensor([tokens_of(20, cfg["vocab"], 1)]), cache)
    with pytest.raises(p.Ab2Error, match="recurrent state"):
        cache.truncate(10)
    with pytest.raises(p.Ab2Error, match="capacity"):
        m.extend_cache(torch.tensor([tokens_of(21, cfg["vocab"], 1)]), cache)
    with pytest.raises(p.Ab2Error, match="offsets"):
        m.forward_with_cache(torch.tensor([[1, 2]]), 5, cache)
    with pytest.raises(p.Ab2Error, match="workspace"):
        m.extend_cache(torch.tensor([tokens_of(33, cfg["vocab"], 1)]), m.empty_kv_cache_with_capacity(64))
    with pytest.raises(p.Ab2Error):
        m.empty_kv_cache_with_capacity(40, dtype="int8")
    # a snapshot carries rings and states
    snap = cache.snapshot()
    nxt = torch.tensor([[7]])
    a = m.forward_with_cache(nxt, 20, cache).clone()
    b = m.forward_with_cache(nxt, 20, snap)
    assert torch.equal(a, b)
    # windows only: cut back freely while the ring still holds the window before the cut
    wcfg = p.StackConfig(64, 64, [(p.AttentionMixer(1, 1, 8, 8, 1.0, 6), None)], 64)
    ring = p.KVCache.for_stack(wcfg, 64, 1, 4, "f32")
    for _ in range(5):
        p.dispatch.window_attention(ring, wcfg, 0, torch.zeros((1, 4, 24), device="cuda"), None, 1e-5)
        ring.commit(4)
    ring.truncate(17)
    with pytest.raises(p.Ab2Error, match="ring"):
        ring.truncate(10)
    ring.truncate(0)
