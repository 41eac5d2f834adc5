"""Rofulorn on CUDA: the 32-bit residual norm, normed and rotated q / k with pages, windowed attention with kept first tokens, soft
cap and two maps (generic and tcgen05 kernels), the gated product, and the model through the engine, against the plain
float64 oracle.

float32 runs everything in true 32-bit (tight tolerance); bfloat16 is what serving uses (tolerance of 16-bit rounding).
"""
import pytest
import torch

import test_rofulorn_cpu as cases
from llmss_b200.utils.checkpoint import rofulorn_config

pytestmark = pytest.mark.gpu

F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16
MODES = [pytest.param(F32, 3e-4, id="f32"), pytest.param(BF16, 8e-2, id="bf16")]

# sizes the tensor-core kernels take, with tiles of 64, 128 and 256, partly filled ones, and many query heads per key/value head
cases.CONFIGS["wide"] = rofulorn_config(128, 211, [
    cases.dif(heads=4, kv_heads=2, dim=16, vdim=32, window=70, keep_first=5, rot_dims=8, mlp={"ff": 64}),
    cases.pln(heads=8, kv_heads=1, dim=40, vdim=72, window=33, rot_dims=24, mlp={"ff": 96}),
    cases.dif(heads=2, kv_heads=1, dim=64, vdim=128, window=100, keep_first=66, rot_dims=64, mlp=None),
    cases.dif(heads=4, kv_heads=2, dim=16, vdim=32, window=21, keep_first=9, rot_dims=8, kv_from=0, mlp={"ff": 128}),
    cases.pln(heads=2, kv_heads=2, dim=136, vdim=24, window=64, mlp={"ff": 64})], embed_scale=11.0)


def test_loaded_library_is_the_in_tree_one():
    from llmss_b200.ops import _lib

    _lib.load()
    assert _lib.LOADED_FROM.endswith("llmss_b200/_C/libllmss_b200.so")


@pytest.mark.parametrize("H,G,dk,dv,maps,cap", [(4, 2, 8, 12, 1, 0.0), (4, 2, 8, 12, 2, 9.0), (3, 3, 6, 10, 2, 0.0), (2, 1, 20, 5, 1, 12.0),
                                                (18, 1, 40, 72, 2, 20.0), (4, 2, 136, 24, 1, 0.0), (2, 1, 12, 300, 2, 4.0)])
def test_generic_attention(H, G, dk, dv, maps, cap):
    cases.test_window_edges_first_tokens_and_far_keys(H, G, dk, dv, maps, cap, "cuda", F32, 1e-4, bs=64)
    cases.test_window_edges_first_tokens_and_far_keys(H, G, dk, dv, maps, cap, "cuda", F32, 1e-4, bs=16, spans=[(20, 4), (33, 20)])


@pytest.mark.parametrize("H,G,dk,dv,maps,cap", [
    (4, 2, 16, 32, 2, 9.0), (6, 3, 24, 64, 2, 15.0), (4, 2, 64, 128, 2, 30.0), (2, 2, 128, 256, 2, 9.0),        # two maps: tiles 64, 64, 128, 256
    (4, 2, 64, 64, 1, 0.0), (8, 2, 128, 128, 1, 12.0), (3, 3, 104, 88, 1, 0.0), (4, 4, 40, 200, 1, 20.0), (2, 1, 8, 8, 1, 0.0),   # partly filled tiles
    (3, 1, 24, 8, 2, 0.0), (2, 1, 8, 136, 2, 3.0), (40, 1, 72, 24, 1, 0.0), (12, 1, 16, 32, 2, 9.0), (40, 1, 16, 32, 2, 0.0)])  # 24, 40, 80 rows per group
def test_tensor_core_attention(H, G, dk, dv, maps, cap):
    from llmss_b200.ops import cuda_impl as cu

    assert cu.span_uses_tc(BF16, dk, dv, maps, 64, 1.0)
    cases.test_window_edges_first_tokens_and_far_keys(H, G, dk, dv, maps, cap, "cuda", BF16, 6e-2, bs=64)
    cases.test_window_edges_first_tokens_and_far_keys(H, G, dk, dv, maps, cap, "cuda", F16, 2e-2, bs=32, spans=[(20, 4), (64, 65), (0, 0)])
    cases.test_window_edges_first_tokens_and_far_keys(H, G, dk, dv, maps, cap, "cuda", BF16, 6e-2, bs=16, spans=[(17, 3)])


def test_sizes_off_the_tensor_core_rules_in_16_bit():
    """Sizes that are no multiple of 8 run on the generic kernel; the two maps are combined from 32-bit outputs."""
    cases.test_window_edges_first_tokens_and_far_keys(3, 3, 6, 10, 2, 5.0, "cuda", BF16, 6e-2, bs=64)
    cases.test_window_edges_first_tokens_and_far_keys(2, 1, 20, 5, 1, 0.0, "cuda", BF16, 6e-2, bs=64)


def test_attention_into_columns_of_a_wider_row():
    cases.test_attention_into_columns_of_a_wider_row("cuda", F32, 1e-4)
    cases.test_attention_into_columns_of_a_wider_row("cuda", BF16, 5e-2)


def test_long_windows_over_many_splits():
    """1200 tokens: several key tiles per split of the decode kernel, a window that starts in the middle, kept tokens over two tiles."""
    for H, G, dk, dv, maps, cap in [(4, 2, 64, 128, 2, 30.0), (4, 1, 128, 128, 1, 0.0), (4, 2, 16, 32, 2, 0.0)]:
        torch.manual_seed(3)
        q, k, v = torch.randn(1200, H, maps, dk), torch.randn(1200, G, maps, dk), torch.randn(1200, G, dv)
        from llmss_b200 import ops
        from llmss_b200.engine.batch import BatchInput

        q, k, v = (x.to(BF16) for x in (q, k, v))
        table, bs = list(range(19, 0, -1)), 64
        for kdt, tol in ((F32, 1e-4), (BF16, 5e-2)):
            kc, vc = torch.zeros(20, G, bs, maps * dk, dtype=kdt), torch.zeros(20, G, bs, dv, dtype=kdt)
            for p in range(1200):
                kc[table[p // bs], :, p % bs], vc[table[p // bs], :, p % bs] = k[p].reshape(G, -1).to(kdt), v[p].to(kdt)
            kc, vc = kc.cuda(), vc.cuda()
            for window, keep in ((700, 70), (0, 0), (300, 3)):
                a = [cases.oracle.softmax_attention(q[:, :, m].double(), k[:, :, m].double().repeat_interleave(H // G, 1),
                                                    v.double().repeat_interleave(H // G, 1), dk ** -0.5,
                                                    {"size": window, "keep_first": keep} if window else None, cap or None) for m in range(maps)]
                size = lambda x: x.square().mean(-1).sqrt()
                ease = (((size(a[0]) + 0.5 * size(a[1])) / size(a[0] - 0.5 * a[1]) / 2.0).max(-1).values.clamp(min=1.0) if maps == 2
                        else torch.ones(1200))
                want = (a[0] if maps == 1 else cases.oracle.rms_div(a[0] - 0.5 * a[1], 1e-6) * 0.5).reshape(1200, -1)
                for lo, hi in ((0, 1200), (1199, 1200), (1000, 1130), (640, 641)):
                    batch = BatchInput.build([[0] * (hi - lo)], [lo], [table], bs, "cuda")
                    qq = cases._pad_maps(q[lo:hi].reshape(hi - lo, -1).to(kdt).cuda(), H, maps, dk, batch, kc, vc, dk ** -0.5)
                    got = ops.attention_bias(qq, kc, vc, batch, H, G, dk, dv, dk ** -0.5, None, out_dtype=kdt, window=window, keep_first=keep,
                                             softcap=cap, diff=(0.5, 1e-6, 0.5) if maps == 2 else None)
                    rms = size(want)[lo:hi, None]         # the first rows average few values and are larger
                    cases.close(got.double().cpu() / rms, want[lo:hi] / rms, tol, ease[lo:hi])


def test_row_kernels():
    for W, bias in [(32, False), (50, True), (1024, False), (7, False), (2048, True), (8192, False), (5001, True), (12288, False)]:
        cases.test_residual_norm(W, bias, "cuda", F32, 1e-5)
        cases.test_residual_norm(W, bias, "cuda", BF16, 2e-2)
    for T, W, F in [(5, 32, 24), (130, 50, 13), (1, 64, 128), (300, 256, 512)]:
        cases.test_gated_product(T, W, F, "cuda", F32, 1e-5)
        cases.test_gated_product(T, W, F, "cuda", BF16, 6e-2)   # products many times the spread, in 16-bit


@pytest.mark.parametrize("hq,hkv,dk,dv,maps,dims,norm", [(4, 2, 12, 8, 1, 8, False), (2, 1, 8, 20, 2, 8, True), (6, 3, 5, 7, 2, 4, True),
                                                         (1, 1, 20, 4, 1, 0, True), (4, 4, 64, 128, 2, 32, True), (16, 4, 128, 128, 1, 64, False),
                                                         (2, 1, 300, 260, 1, 300, True), (3, 3, 10, 6, 2, 6, True), (2, 2, 520, 8, 1, 500, True)])
def test_norm_rotation_and_pages(hq, hkv, dk, dv, maps, dims, norm):
    cases.test_norm_rotation_and_pages(hq, hkv, dk, dv, maps, dims, norm, "cuda", F32, 1e-5)
    cases.test_norm_rotation_and_pages(hq, hkv, dk, dv, maps, dims, norm, "cuda", BF16, 2e-2)


@pytest.mark.parametrize("dtype,tol", MODES)
@pytest.mark.parametrize("name", ["plain", "diff", "ffn", "mixed", "edges", "odd", "wide"])
def test_whole_prompt_and_residual_stream(tmp_path, name, dtype, tol):
    cases.test_whole_prompt_and_residual_stream(tmp_path, name, "cuda", dtype, tol)


@pytest.mark.parametrize("name", ["mixed", "edges", "odd", "wide"])
def test_decode_and_portions(tmp_path, name):
    cases.test_decode_token_by_token_and_portions(tmp_path, name, "cuda", F32, 3e-4)


def test_schedules_in_32_bit(tmp_path):
    cases.test_unequal_batches_against_each_alone(tmp_path / "a", "cuda", F32, 3e-4)
    cases.test_pages_are_used_again(tmp_path / "b", "cuda", F32, 3e-4)
    cases.test_steep_attention_far_back_and_over_page_borders(tmp_path / "c", "cuda", F32, 3e-4)
    cases.test_first_tokens(tmp_path / "d", "cuda", F32, 3e-4)
    cases.test_long_decoding(tmp_path / "e", "cuda", F32, 3e-4)
    cases.test_model_call_with_a_past(tmp_path / "f", "cuda", F32, 3e-4)


def test_schedules_in_16_bit(tmp_path):
    """bfloat16 on the tensor-core kernels: portions, single tokens, mixed batches and page reuse against the oracle."""
    cfg, W, eng = cases.build(tmp_path, "wide", "cuda", BF16)
    toks = cases.tokens_for(cfg, 200, 3)
    want = cases.want_logits(toks, cfg, W)
    for sizes in ([200], [150, 1], [31, 2, 36, 1, 1, 59, 2, 1], [64, 64, 1]):
        cases.close(cases.feed_in_portions(eng, "p", toks, sizes), want, 1e-1)


def test_decode_batch_of_unequal_requests_in_16_bit(tmp_path):
    """bfloat16: three requests of different lengths decode together, then beside a portion of a fourth; every request equals
    itself fed whole."""
    cfg, W, eng = cases.build(tmp_path, "wide", "cuda", BF16)
    reqs = {k: cases.tokens_for(cfg, n, 20 + i) for i, (k, n) in enumerate([("a", 90), ("b", 171), ("c", 40)])}
    whole = {k: cases.feed_in_portions(eng, "w" + k, t, [len(t)]).double().cpu() for k, t in reqs.items()}
    std = max(v.std().item() for v in whole.values())
    tail = 12
    out = eng.feed([(k, t[:-tail], [len(t) - tail - 1]) for k, t in reqs.items()])
    got = {k: [out[i:i + 1]] for i, k in enumerate(reqs)}
    for j in range(tail):
        last = j == tail - 1
        beside = [("x", cases.tokens_for(cfg, 9, j), [])] if j % 3 == 2 else []
        out = eng.feed([(k, [t[len(t) - tail + j]], [0]) for k, t in reqs.items()] + beside, list(reqs) + ["x"] if last else [])
        for i, k in enumerate(reqs):
            got[k].append(out[i:i + 1])
    for k, t in reqs.items():
        d = (torch.cat(got[k]).double().cpu() - whole[k][len(t) - tail - 1:]).abs().max(-1).values / std
        assert d.max() < 8e-2, (k, d)


@pytest.mark.parametrize("graph", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_generation(tmp_path, dtype, graph):
    cases.test_greedy_generation_through_engine_and_cli(tmp_path, "cuda", dtype, graph)


def test_generation_by_graph_equals_eager(tmp_path):
    """bfloat16 at tensor-core sizes: the captured decode step (padded batch, inert rows) and the eager one choose the same tokens
    past several page borders and windows."""
    cfg, W, a = cases.build(tmp_path, "wide", "cuda", BF16, max_batch=3, graph=True)
    _, _, b = cases.build(tmp_path, "wide", "cuda", BF16, max_batch=3, graph=False)
    prompts = [cases.tokens_for(cfg, n, 90 + n) for n in (60, 130, 5)]
    sp = cases.SamplingParams(max_new_tokens=80, is_greedy=True)
    ga, gb = a.generate(prompts, sp), b.generate(prompts, sp)
    assert ga == gb and a.runner.stats["graph_replays"] > 0
    lg = cases.want_logits(prompts[1] + ga[1], cfg, W)[len(prompts[1]) - 1:-1]
    for row, tok in zip(lg, ga[1]):
        assert row[tok] >= row.max() - 0.2 * lg.std()


def test_shared_prompt_prefix_and_prompt_rounds(tmp_path):
    cases.test_shared_prompt_prefix_and_prompt_rounds(tmp_path, "cuda", F32)
