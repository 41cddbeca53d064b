"""Vipelix on the GPU against the plain numpy restatement: every mechanism alone, then the model
through its own cache, portions, batches, sessions and generation."""
import ctypes as C
import json

import numpy as np
import pytest
import torch

import vipelix_fixtures as fx
from helpers import pkg, rel_err
from oracle import vipelix_ref as ref
from test_gpu_tovelix import DTYPES, feed_portions, run_program, to_gpu, tokens_of, tol

pytestmark = pytest.mark.gpu

PORTIONS = [[10**9], [1], [2, 3], [64, 1, 17, 5], [130, 40, 2]]


# ---------------------------------------------------------------- latent attention alone

class LatentCase:
    """Inputs of one latent layer and what the restatement makes of them, position by position."""

    def __init__(self, H, dim, rot, vdim, rank, T, at, targets, seed, base=300.0, scale=0.35, gated=True, first=0):
        self.q, self.c, self.kr, uk, uv = fx.spiked_latents(T, H, dim, rot, vdim, rank, at, targets, seed)
        rng = np.random.default_rng(seed + 1)
        self.T, self.H, self.dim, self.rot, self.vdim, self.rank, self.eps = T, H, dim, rot, vdim, rank, 1e-4
        self.norm = fx.bf16_round(1 + 0.3 * rng.standard_normal(rank))
        self.gate = fx.bf16_round(rng.standard_normal((T, H)))
        f8 = [x.astype(np.float64) for x in (self.q, self.c, self.kr, uk, uv)]
        pos = np.arange(T)
        q = np.concatenate([f8[0][..., :dim], ref.turn_pairs(f8[0][..., dim:], pos, base) if rot else f8[0][..., dim:]], -1)
        c = ref.rms_norm(f8[1], self.norm.astype(np.float64), self.eps)
        kr = ref.turn_pairs(f8[2], pos, base) if rot else f8[2]
        self.want = ref.latent_attention(q[first:], c, kr, f8[3], f8[4], scale, first=first)
        if gated:
            self.want = self.want * ref.sigmoid(self.gate.astype(np.float64))[first:, :, None]
        p = pkg()
        self.cfg = p.StackConfig(64, 64, [(p.LatentMixer(H, dim, rot, vdim, rank, scale, base, gated), None)], 2 * T)
        self.ukv = p.QuantLinear.from_bf16(torch.from_numpy(np.concatenate([uk.reshape(H, dim, rank), uv.reshape(H, vdim, rank)], 1).reshape(-1, rank))
                                           .to(torch.bfloat16))
        self.tables = p.dispatch.rotation_tables(2 * T, rot, base) if rot else None
        n = H * (dim + rot) + rank + rot + (H if gated else 0)
        rows = [self.q.reshape(T, -1), self.c, self.kr] + ([self.gate] if gated else []) + [np.full((T, -n % 8), 9.0)]
        self.proj = np.concatenate(rows, 1)

    def cache(self, dtype, rows=1, step=None):
        return pkg().KVCache.for_stack(self.cfg, self.T + 3, rows, step or self.T, "f32" if dtype == torch.float32 else "bf16")

    def run(self, cache, parts, dtype, row=0, workspace=None):
        p, norm = pkg(), torch.from_numpy(self.norm).cuda()
        got = []
        for a, b in parts:
            got.append(p.dispatch.latent_attention(cache, self.cfg, 0, to_gpu(self.proj[None, a:b], dtype), norm, self.ukv, self.tables, self.eps,
                                                   row0=row, workspace=workspace))
            cache.commit(b - a, row, 1)
        assert p.device_status() == 0
        return torch.cat(got, 1)[0].float().cpu().numpy().reshape(-1, self.H, self.vdim)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,rot,vdim,rank,T", [(4, 40, 16, 56, 104, 200), (3, 16, 8, 24, 40, 150), (40, 24, 8, 16, 64, 140), (1, 128, 64, 128, 512, 150),
                                                   (5, 20, 6, 18, 44, 90), (2, 7, 2, 5, 9, 70), (2, 40, 0, 32, 128, 140), (33, 8, 8, 8, 72, 135),
                                                   (2, 64, 32, 64, 640, 70), (6, 144, 40, 72, 320, 133)])
def test_latent_attention(dtype, H, dim, rot, vdim, rank, T):
    at = T - 3
    x = LatentCase(H, dim, rot, vdim, rank, T, at, (0, 63, 64, at - 1)[:H], H * 100 + rank)
    for sizes in PORTIONS:
        if sizes == [1] and rank > 200:
            sizes = [T - 9, 1]
        parts = feed_portions(T, sizes)
        cache = x.cache(dtype, 2)
        for row in (1, 0, 1):   # a row used again starts from nothing
            cache.truncate(0, row)
            got = x.run(cache, parts, dtype, row)
            assert rel_err(got, x.want) < tol(dtype, 1e-5, 1.5e-2), sizes
            assert np.abs(got[at] - x.want[at]).max() < tol(dtype, 1e-5, 1.5e-2) * np.abs(x.want[at]).max(), sizes


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,rot,vdim,rank,T,gated", [(2, 64, 32, 32, 128, 1500, True), (3, 32, 64, 24, 512, 700, False), (16, 32, 16, 16, 224, 900, True)])
def test_far_keys_over_many_splits(dtype, H, dim, rot, vdim, rank, T, gated):
    """The last positions of a long context, decoded and in short portions: the keys are cut into runs,
    and a key's score that towers over the others sits at the ends of tiles and runs."""
    first = T - 8
    x = LatentCase(H, dim, rot, vdim, rank, T, T - 4, (0, 127, 128, 575, T - 70, T - 65, T - 5)[:max(2, min(H, 7))], 7, gated=gated, first=first)
    for tail in ([1] * 8, [2, 6], [3, 1, 4], [8]):
        cache = x.cache(dtype, step=T)
        cuts = [(0, first)]
        for n in tail:
            cuts.append((cuts[-1][1], cuts[-1][1] + n))
        got = x.run(cache, cuts, dtype)[first:]
        for i in range(8):
            assert np.abs(got[i] - x.want[i]).max() < tol(dtype, 1e-5, 1.5e-2) * np.abs(x.want[i]).max(), (tail, i)


@pytest.mark.parametrize("H,dim,rot,vdim,rank", [(64, 32, 8, 16, 64), (48, 48, 64, 16, 512), (50, 40, 16, 24, 200)])
def test_a_late_key_towers_over_the_others(H, dim, rot, vdim, rank):
    """Enough rows that every run walks many tiles, and every head's highest score comes late (a different
    tile for each): what was summed before has to be scaled down."""
    first, S = 420, 100
    x = LatentCase(H, dim, rot, vdim, rank, first + S, first + S - 2, [5 + 7 * h for h in range(H)], 9, first=first)
    got = x.run(x.cache(torch.bfloat16), [(0, first), (first, first + S)], torch.bfloat16)[first:]
    assert rel_err(got, x.want) < 1.5e-2
    for i in range(S):
        assert rel_err(got[i], x.want[i]) < 3e-2, i
    for h in range(H):
        assert rel_err(got[S - 2, h], x.want[S - 2, h]) < 3e-2, h


@pytest.mark.parametrize("H,dim,rot,vdim,rank,first", [(8, 128, 64, 128, 128, 0), (7, 40, 24, 72, 64, 0), (8, 64, 0, 64, 96, 133), (6, 136, 40, 64, 64, 5)])
def test_long_prompt_portions(H, dim, rot, vdim, rank, first):
    """Many key tiles per query, the highest scores in early, middle and late ones, at the tiles' edges."""
    T = 900
    at = T - 2
    x = LatentCase(H, dim, rot, vdim, rank, T, at, (0, 127, 128, 511, 640, 767, 895, at - 1)[:H], 21, first=T - 150)
    for cuts in ([(0, T)], [(0, first), (first, T)], [(0, 300), (300, 429), (429, T)]):
        cuts = [c for c in cuts if c[1] > c[0]]
        got = x.run(x.cache(torch.bfloat16), cuts, torch.bfloat16)[T - 150:]
        assert rel_err(got, x.want) < 1.5e-2, cuts
        for h in range(H):
            assert rel_err(got[at - T + 150, h], x.want[at - T + 150, h]) < 3e-2, (cuts, h)


@pytest.mark.parametrize("first", [0, 37])
def test_prompt_projected_some_heads_at_a_time(first):
    """A workspace that holds the keys and values of three heads only, and one that holds none."""
    x = LatentCase(7, 32, 16, 40, 64, 300, 250, (0, 100, 249), 3)
    cuts = ([(0, first)] if first else []) + [(first, 300)]
    p = pkg()
    specs, _ = x.cfg.c_specs()
    base = C.c_size_t()
    p.check(p.lib.ab2_latent_workspace(C.byref(specs[0]), 300, 1, p._lib.BF16, C.byref(base)))
    absorbed = (7 * 64 * 32 * 2 + 255) // 256 * 256
    for heads in (3, 0):
        n = max(base.value, absorbed + heads * 300 * 72 * 2) if heads else base.value
        got = x.run(x.cache(torch.bfloat16), cuts, torch.bfloat16, workspace=torch.empty(n, dtype=torch.uint8, device="cuda"))
        assert rel_err(got, x.want) < 1.5e-2


def test_latent_rows_of_unequal_length_together():
    """Rows of one cache at different lengths, decoded in one call and in a prompt portion for all."""
    p = pkg()
    lens = (3, 64, 131, 200)
    cases = [LatentCase(6, 32, 16, 24, 96, 340, 300, (0, 64, 299), 11 + r) for r in range(4)]
    for x in cases[1:]:   # one layer: the first case's weights serve all rows
        x.ukv, x.norm, x.cfg = cases[0].ukv, cases[0].norm, cases[0].cfg
    c0 = cases[0]
    cache = c0.cache(torch.bfloat16, rows=4)
    alone = []
    for r, x in enumerate(cases):
        one = c0.cache(torch.bfloat16)
        alone.append(x.run(one, [(0, lens[r]), (lens[r], lens[r] + 1), (lens[r] + 1, lens[r] + 6), (lens[r] + 6, lens[r] + 136)], torch.bfloat16))
        x.run(cache, [(0, lens[r])], torch.bfloat16, row=r)
    norm = torch.from_numpy(c0.norm).cuda()
    at = 0
    for S in (1, 5, 130):
        proj = np.stack([x.proj[n + at:n + at + S] for x, n in zip(cases, lens)])
        got = p.dispatch.latent_attention(cache, c0.cfg, 0, to_gpu(proj, torch.bfloat16), norm, c0.ukv, c0.tables, c0.eps)
        cache.commit(S)
        for r, n in enumerate(lens):
            w = alone[r][n + at:n + at + S]
            assert rel_err(got[r].float().cpu().numpy().reshape(w.shape), w) < 8e-3, (S, r)
        at += S
    assert p.device_status() == 0


# ---------------------------------------------------------------- feed-forwards alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [7, 64, 250, 1000, 11008])
def test_poly_norm(dtype, n):
    rng = np.random.default_rng(n)
    z = fx.bf16_round(rng.standard_normal((5, n)) * np.array([1e-3, 0.1, 1.0, 30.0, 300.0])[:, None])
    coef = (0.7, -0.5, 1.25, 0.2)
    got = pkg().dispatch.poly_norm(to_gpu(z, dtype), coef, 1e-5).float().cpu().numpy()
    want = ref.poly_norm(z.astype(np.float64), coef, 1e-5)
    for r in range(5):
        assert rel_err(got[r], want[r]) < tol(dtype, 1e-5, 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,top,ff,d", [(5, 2, 56, 96), (3, 3, 30, 50)])
def test_silu_experts(dtype, E, top, ff, d):
    """The SiLU unit in every kernel family of the expert linears (the router here scores what an expert reads)."""
    p = pkg()
    rng = np.random.default_rng(E)
    w = {k: fx.bf16_round(rng.standard_normal(s) / np.sqrt(s[1]) * 1.5) for k, s in (("r", (E, d)), ("g", (E * ff, d)), ("u", (E * ff, d)), ("d", (E * d, ff)))}
    experts = p.dispatch.MoeExperts(p.MoeFfn(E, top, ff, glu="silu"), *[p.QuantLinear.from_bf16(torch.from_numpy(w[k]).to(torch.bfloat16)) for k in "rgud"])
    w = {k: v.astype(np.float64) for k, v in w.items()}
    for T in (1, 9, 33, 200):
        x = fx.bf16_round(rng.standard_normal((T, d)))
        got = experts(to_gpu(x, dtype)).cpu().numpy()
        for t in range(T):
            s = ref.sigmoid(w["r"] @ x[t].astype(np.float64))
            for slot, e in enumerate(np.argsort(-s, kind="stable")[:top]):
                want = ref.gated_unit(s[e] * x[t].astype(np.float64), w["g"][e * ff:(e + 1) * ff], w["u"][e * ff:(e + 1) * ff], w["d"][e * d:(e + 1) * d])
                assert np.abs(got[t, slot] - want).max() <= tol(dtype, 1e-5, 1.5e-2) * np.abs(want).max(), (T, t)


# ---------------------------------------------------------------- the model

def check_logits(got, want, dtype):
    e = fx.errors(got, want)
    assert e.max() < tol(dtype, 1e-4, 4e-2), (int(e.argmax()), e.max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["VARIED", "ROUND", "PLAIN"])
def test_prompt_portions_and_decoding(tmp_path, dtype, name):
    cfg = getattr(fx, name)
    w = fx.weights(cfg, 5)
    toks = tokens_of(190, cfg["vocab"], 6)
    want = fx.expected(cfg, w, toks)
    m = fx.load(tmp_path, cfg, w, dtype, max_tokens=256, max_seq_len=256)
    eng = pkg().sessions.SessionEngine(m, max_batch=2, capacity=256)
    for sizes in PORTIONS:
        row = eng.open_row()
        got = torch.cat([eng.feed(row, toks[a:b], range(b - a)).clone() for a, b in feed_portions(len(toks), sizes)])
        eng.close_row(row)
        check_logits(got, want, dtype)
    # a portion larger than the workspace goes in pieces
    small = fx.load(tmp_path, cfg, w, dtype, max_tokens=48, max_seq_len=256)
    eng = pkg().sessions.SessionEngine(small, max_batch=1, capacity=256)
    row = eng.open_row()
    want_at = [0, 1, 47, 48, 95, 130, 189]
    check_logits(eng.feed(row, toks, want_at), want[want_at], dtype)
    assert pkg().device_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_of_unequal_requests(tmp_path, dtype):
    """Requests of different lengths in the rows of one cache, decoded together in changing sets, rows
    given back and taken again: the logits are those of each request alone."""
    p, cfg = pkg(), fx.VARIED
    w = fx.weights(cfg, 11)
    m = fx.load(tmp_path, cfg, w, dtype, max_tokens=128, max_seq_len=256)
    cache = m.empty_kv_cache_with_capacity(200, batch=5)
    start = {r: n for r, n in enumerate((9, 1, 75, 40, 100))}
    full = {r: tokens_of(n + 20, cfg["vocab"], 20 + r) for r, n in start.items()}
    want = {r: fx.expected(cfg, w, s) for r, s in full.items()}
    at = dict(start)
    for r in (3, 0, 4, 1, 2):
        m.extend_cache(torch.tensor([full[r][:at[r]]]), cache, r)
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
    # two rows at once through a prompt pass, taken by new requests
    cache.truncate(0, 0)
    cache.truncate(0, 1)
    two = torch.tensor([full[2][:50], full[4][:50]])
    out = torch.empty((2, 50, cfg["vocab"]), device="cuda")
    p.check(p.lib.ab2_model_forward(m._h, cache._h, two.to(torch.int32).cuda().data_ptr(), 50, 0, 2, None, 2, out.data_ptr(), None,
                                    torch.cuda.current_stream().cuda_stream))
    check_logits(out[0], want[2][:50], dtype)
    check_logits(out[1], want[4][:50], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(tmp_path, dtype):
    cfg = fx.ROUND
    w = fx.weights(cfg, 13)
    toks = tokens_of(330, cfg["vocab"], 14)
    m = fx.load(tmp_path, cfg, w, dtype, max_tokens=16, max_seq_len=400)
    eng = pkg().sessions.SessionEngine(m, max_batch=1, capacity=400)
    row = eng.open_row()
    eng.feed(row, toks[:11])
    got = torch.cat([eng.feed(row, [t], [0]).clone() for t in toks[11:]])
    check_logits(got, fx.expected(cfg, w, toks)[11:], dtype)


def test_wide_batches_take_the_prompt_linears(tmp_path):
    """40 sequences decoded together (more rows than the streaming linears take) and a prompt in one pass."""
    cfg = fx.PLAIN
    w = fx.weights(cfg, 15)
    m = fx.load(tmp_path, cfg, w, torch.bfloat16, max_tokens=64, max_seq_len=64)
    cache = m.empty_kv_cache_with_capacity(32, batch=40)
    seqs = [tokens_of(6, cfg["vocab"], 100 + r) for r in range(40)]
    for i in range(6):
        lg = m.forward_decode_batch(torch.tensor([[s[i]] for s in seqs]), [i] * 40, cache)
    check_logits(lg[:, 0], np.stack([fx.expected(cfg, w, s)[-1] for s in seqs]), torch.bfloat16)


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
    want = [greedy(cfg, w, q, 10) for q in prompts]
    eng = p.InferenceEngine(m)
    for q, t in zip(prompts, want):
        assert eng.generate_from_token_ids(q, 10)["token_ids"] == t
        assert eng.generate_from_token_ids(q, 10, on_device_sampling=False)["token_ids"] == t
    se = p.sessions.SessionEngine(m, max_batch=2, capacity=100)
    live = [se.prepare_session_with_chunk_size(q, 10, chunk_size=7) for q in prompts]
    while any(not s.finished for s in live):
        for s in live:
            se.advance(s)
        se.decode_sessions([s for s in live if not s.finished])
    assert [s.generated_ids for s in live] == want


def test_command_line_programs(tmp_path):
    """bin/generate and bin/trace_run on a checkpoint folder."""
    cfg = fx.VARIED
    w = fx.weights(cfg, 17)
    folder = fx.write_checkpoint(str(tmp_path / "m"), cfg, w)
    prompts = [tokens_of(n, cfg["vocab"], 50 + n) for n in (21, 3)]
    want = [greedy(cfg, w, q, 5) for q in prompts]
    args = ["--model", folder, "--dtype", "float32", "--max-new-tokens", "5"]
    for q in prompts:
        args += ["--tokens", ",".join(map(str, q))]
    assert [json.loads(x)["tokens"] for x in run_program("generate", args).splitlines()] == want
    q = prompts[0]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": q[:9], "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": q[9:20], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": q[20:], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": q[:2], "want": [1]}], "end": ["b"]}]
    run_program("trace_run", ["--model", folder, "--dtype", "bfloat16", "--out", str(tmp_path), "--max-tokens", "40"], "\n".join(map(json.dumps, steps)) + "\n")
    full = fx.expected(cfg, w, q)
    for step, at in ((0, [0, 8]), (2, [20]), (3, [1])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(at), cfg["vocab"])
        check_logits(got.astype(np.float64), full[at], torch.bfloat16)
    assert not (tmp_path / "1.f32").exists()


def test_draft_verification_cuts_the_cache_back(tmp_path):
    p, cfg = pkg(), fx.VARIED
    w = fx.weights(cfg, 19)
    m = fx.load(tmp_path, cfg, w, torch.float32, max_tokens=64, max_seq_len=128)
    prompt = tokens_of(20, cfg["vocab"], 60)
    tail = greedy(cfg, w, prompt, 6)
    cache = m.empty_kv_cache_with_capacity(100)
    assert not cache.has_state()
    m.extend_cache(torch.tensor([prompt]), cache)
    wrong = [(t + 1) % cfg["vocab"] for t in tail]
    accepted, nxt, _ = p.sessions.verify_draft(m, cache, 0, 20, tail[0], [tail[1], tail[2], wrong[3], tail[4]])
    assert (accepted, nxt, cache.seq_len(0)) == (2, tail[3], 23)
    snap = cache.snapshot()
    accepted, nxt, lg = p.sessions.verify_draft(m, cache, 0, 23, tail[3], [tail[4]])
    assert (accepted, nxt, cache.seq_len(0)) == (1, tail[5], 25)
    check_logits(lg, fx.expected(cfg, w, prompt + tail[:5])[-2:], torch.float32)
    accepted, nxt, lg2 = p.sessions.verify_draft(m, snap, 0, 23, tail[3], [tail[4]])
    assert torch.equal(lg, lg2)


def test_what_is_refused(tmp_path):
    p, cfg = pkg(), fx.VARIED
    w = fx.weights(cfg, 23)
    m = fx.load(tmp_path, cfg, w, torch.float32, max_tokens=32, max_seq_len=64)
    cache = m.empty_kv_cache_with_capacity(40)
    assert cache.n_layers == 9
    m.extend_cache(torch.tensor([tokens_of(20, cfg["vocab"], 1)]), cache)
    with pytest.raises(p.Ab2Error, match="capacity"):
        m.extend_cache(torch.tensor([tokens_of(21, cfg["vocab"], 1)]), cache)
    once = p.StackConfig(**dict(m.cfg.__dict__, loop=None))
    with pytest.raises(p.Ab2Error, match="cache layers"):
        m.extend_cache(torch.tensor([[1, 2]]), p.KVCache.for_stack(once, 40, 1, 8, "f32"))
    # a table that names an expert that is not there, or one twice
    for bad in (cfg["layers"][0]["mlp"]["router"]["experts"], int(w["l0.mlp.table"][7, 1])):
        broken = dict(w, **{"l0.mlp.table": w["l0.mlp.table"].copy()})
        broken["l0.mlp.table"][7, 0] = bad
        with pytest.raises(p.Ab2Error, match="names expert"):
            fx.load(tmp_path, cfg, broken, torch.float32)
    with pytest.raises(p.checkpoint.CheckpointError, match="loop.step"):
        fx.load(tmp_path, cfg, {k: v for k, v in w.items() if k != "loop.step"}, torch.float32)
    with pytest.raises(p.Ab2Error, match="loop"):
        fx.load(tmp_path, dict(cfg, loop={"start": 3, "stop": 9, "times": 1}), dict(w, **{"loop.step": w["loop.step"][:1]}), torch.float32)
