"""The algorithmic byte counts behind the reported roofline fractions, against constants worked
out by hand from the formats: W4A16 g128 stores K N / 2 bytes of codes, a bf16 scale and half a
byte of zero point per group of 128 weights; an INT8 KV token costs 2 x 8 x 128 code bytes and
2 x 8 f32 scales per layer."""
import os
import sys

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

import bench  # noqa: E402
import microbench  # noqa: E402


def test_weight_side_bytes_of_the_microbenchmark_shapes():
    assert bench.w4_bytes(4096, 4096) == 8_716_288
    assert bench.w4_bytes(14336, 4096) == bench.w4_bytes(4096, 14336) == 30_507_008
    assert bench.w4_bytes(128256, 4096) == 4096 * 128256 // 2 + 32 * 128256 * 2 + 32 * 128256 // 2
    for n, k in [(4096, 4096), (14336, 4096), (4096, 14336), (128256, 4096)]:
        assert microbench.w4_bytes(n, k) == bench.w4_bytes(n, k)


def test_bytes_and_flops_of_a_small_vipelix_step():
    c = dict(width=16, layers=3, loop=(1, 3, 2), heads=2, dim=4, rot=2, vdim=3, rank=5, experts=4, top=1, ff=6, shared=7, dense=9)
    assert bench.vipelix_runs(c) == (1, 4)
    mix = 2 * ((12 + 5 + 2 + 2) * 16 + 2 * 7 * 5 + 6 * 16)                     # weights of a mixer
    assert bench.vipelix_step_bytes(c, 1, 10, vocab=8) == 5 * (mix + 10 * 14) + 2 * 2 * 16 * 9 + 4 * 2 * 3 * 16 * (6 + 7) + 2 * 8 * 16
    per_token = 5 * mix + 4 * 16 * 9 + 4 * 6 * 16 * 13
    assert bench.vipelix_prefill_flops(c, 3, vocab=8) == 3 * per_token + 5 * 2 * 9 * 12 + 2 * 8 * 16


def test_bytes_of_one_large_decode_step():
    assert bench.step_weight_bytes(bench.LARGE) == 3_694_071_808
    assert bench.kv_bytes_per_token(bench.LARGE) == 32 * 2112
    shapes = bench.linear_shapes(bench.LARGE)
    assert shapes["wq"] == (4096, 4096) and shapes["wk"] == shapes["wv"] == (1024, 4096)
    assert shapes["w_gate"] == shapes["w_up"] == (14336, 4096) and shapes["w_down"] == (4096, 14336)
