"""Fipavik on CUDA: the residual norm with a factor, half-pair rotation with mixed values, latent rows and queries, attention with
chunks, windows and sinks (generic and tcgen05 kernels, values inside the key row), the expert forms beside a mixer, and the model
through the engine, against the plain float64 oracle.

float32 runs everything in true 32-bit (tight tolerance); bfloat16 is what serving uses (tolerance of 16-bit rounding).
"""
import pytest
import torch

import fipavik_oracle as oracle
import test_fipavik_cpu as cases
from llmss_b200.utils.checkpoint import fipavik_config

pytestmark = pytest.mark.gpu

F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16

# sizes the tensor-core kernels take: tiles of 64, 128 and 256, partly filled ones, groups of 4 to 40 query heads, unequal key and value
# sizes, a latent row that is not a multiple of 16
cases.CONFIGS["wide"] = fipavik_config(128, 211, [
    cases.att(heads=8, kv_heads=2, dim=40, vdim=72, chunk=50, rot_dims=24, mlp=cases.moe(experts=8, top=2, ff=32, shared=48)),
    cases.lat(heads=12, dim=32, rot_dim=16, vdim=24, kv_rank=56, window=70, mlp=cases.moe(experts=4, top=2, ff=40, shared=64)),
    cases.att(heads=4, kv_heads=2, dim=96, vdim=72, chunk=128, rot_dims=40, mlp=cases.moe(experts=6, top=4, ff=24, shared=None)),
    cases.lat(heads=4, dim=24, rot_dim=40, vdim=40, kv_rank=120, window=33),
    cases.att(heads=6, kv_heads=2, dim=136, vdim=72, chunk=23, rot_dims=8, mlp=cases.moe(experts=4, top=4, ff=16, shared=16))], residual_mult=0.45)


def test_loaded_library_is_the_in_tree_one():
    from llmss_b200.ops import _lib

    _lib.load()
    assert _lib.LOADED_FROM.endswith("llmss_b200/_C/libllmss_b200.so")


@pytest.mark.parametrize("H,G,dk,dv,shared", [(4, 2, 8, 12, 0), (3, 3, 6, 10, 0), (2, 1, 12, 300, 0), (18, 1, 40, 24, 1), (2, 1, 9, 5, 1)])
def test_generic_attention(H, G, dk, dv, shared):
    cases.test_chunk_and_window_edges_sinks_and_far_keys(H, G, dk, dv, shared, "cuda", F32, 1e-4, bs=64)
    cases.test_chunk_and_window_edges_sinks_and_far_keys(H, G, dk, dv, shared, "cuda", F32, 1e-4, bs=16, masks=[(20, 0), (0, 37), (30, 50)])


@pytest.mark.parametrize("H,G,dk,dv,shared", [
    (4, 2, 56, 48, 0), (4, 1, 64, 64, 0), (8, 2, 128, 128, 0), (6, 3, 40, 72, 0), (4, 4, 136, 24, 0), (2, 1, 8, 8, 0), (40, 1, 72, 24, 0),
    (2, 2, 256, 256, 0), (12, 2, 128, 64, 0), (20, 1, 96, 96, 0),
    (7, 1, 104, 72, 1), (12, 1, 72, 56, 1), (4, 1, 160, 120, 1), (16, 1, 256, 192, 1), (40, 1, 256, 192, 1), (6, 1, 24, 8, 1), (1, 1, 64, 64, 1)])
def test_tensor_core_attention(H, G, dk, dv, shared):
    from llmss_b200.ops import cuda_impl as cu

    assert cu.span_uses_tc(BF16, dk, dv, 1, 64, 1.0)
    cases.test_chunk_and_window_edges_sinks_and_far_keys(H, G, dk, dv, shared, "cuda", BF16, 6e-2, bs=64)
    cases.test_chunk_and_window_edges_sinks_and_far_keys(H, G, dk, dv, shared, "cuda", F16, 2e-2, bs=32, masks=[(20, 0), (0, 64), (0, 37), (64, 0)])
    cases.test_chunk_and_window_edges_sinks_and_far_keys(H, G, dk, dv, shared, "cuda", BF16, 6e-2, bs=16, masks=[(0, 16), (17, 0)])


def test_sizes_off_the_tensor_core_rules_in_16_bit():
    cases.test_chunk_and_window_edges_sinks_and_far_keys(3, 3, 6, 10, 0, "cuda", BF16, 6e-2, bs=64)
    cases.test_chunk_and_window_edges_sinks_and_far_keys(2, 1, 12, 9, 1, "cuda", BF16, 6e-2, bs=64)


def test_decode_groups_hold_all_heads():
    """Up to 32 query heads over one key / value head in one call at every tile size; more in groups."""
    from llmss_b200.ops import cuda_impl as cu

    for n, dk in ((9, 64), (16, 256), (32, 256), (32, 128)):
        assert cu._span_decode_groups(BF16, n, 1, dk, dk, 1, 64, 1.0) == [(0, n)]
    assert cu._span_decode_groups(BF16, 40, 1, 256, 192, 1, 64, 1.0) == [(0, 32), (32, 8)]


@pytest.mark.parametrize("H,G,dk,dv,shared", [(5, 1, 64, 40, 0), (16, 1, 256, 192, 1), (8, 2, 128, 128, 0)])
def test_long_masks_over_many_splits(H, G, dk, dv, shared):
    """1200 tokens: several key tiles per split of the decode kernel, windows and chunks that start in the middle of one, the sink once."""
    from llmss_b200 import ops
    from llmss_b200.engine.batch import BatchInput

    torch.manual_seed(3)
    L, bs, scale = 1200, 64, 1.5 * dk ** -0.5
    q, k, v = (x.to(BF16) for x in (torch.randn(L, H, dk), torch.randn(L, G, dk), torch.randn(L, G, dv)))
    v = k[..., :dv] if shared else v
    sink, table = torch.randn(H) + 2.0, list(range(19, 0, -1))
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(H // G, 1)) * scale
    for kdt, tol in ((F32, 1e-4), (BF16, 5e-2)):
        kc = torch.zeros(20, G, bs, dk, dtype=kdt)
        vc = kc[..., :dv] if shared else torch.zeros(20, G, bs, dv, dtype=kdt)
        for p in range(L):
            vc[table[p // bs], :, p % bs] = v[p].to(kdt)
            kc[table[p // bs], :, p % bs] = k[p].to(kdt)
        kc = kc.cuda()
        vc = kc[..., :dv] if shared else vc.cuda()
        for window, chunk in ((700, 0), (0, 0), (0, 1000), (0, 256), (300, 900)):
            a = oracle.sink_softmax(s, cases.visible(L, window, chunk), sink.double())
            want = torch.einsum("hij,jhd->ihd", a, v.double().repeat_interleave(H // G, 1)).reshape(L, -1)
            for lo, hi in ((0, L), (L - 1, L), (1000, 1130), (640, 641), (1023, 1025)):
                batch = BatchInput.build([[0] * (hi - lo)], [lo], [table], bs, "cuda")
                got = ops.attention_bias(q[lo:hi].reshape(hi - lo, -1).to(kdt).cuda(), kc, vc, batch, H, G, dk, dv, scale, None, out_dtype=kdt,
                                         window=window, chunk=chunk, sinks=sink.cuda())
                rms = want.square().mean(-1).sqrt()[lo:hi, None]         # the first rows average few values and are larger
                cases.close(got.double().cpu() / rms, want[lo:hi] / rms, tol)


def test_row_kernels():
    for W, bias in [(32, True), (50, True), (1024, False), (7, True), (2048, True), (5001, True), (12288, False)]:
        cases.test_residual_norm_with_a_factor(W, bias, "cuda", F32, 2e-5)
        cases.test_residual_norm_with_a_factor(W, bias, "cuda", BF16, 3e-2)


@pytest.mark.parametrize("hq,hkv,dk,dv,dims,extra", [
    (4, 2, 12, 8, 8, 0), (2, 1, 16, 20, 16, 6), (6, 3, 5, 7, 4, 3), (8, 2, 64, 32, 24, 8), (3, 3, 20, 4, 4, 4), (16, 4, 128, 128, 64, 16),
    (2, 1, 300, 260, 296, 4), (1, 1, 520, 8, 496, 4), (5, 5, 36, 128, 36, 0), (3, 1, 64, 96, 10, 1)])
def test_norm_half_rotation_and_mixed_values(hq, hkv, dk, dv, dims, extra):
    cases.test_norm_half_rotation_and_mixed_values(hq, hkv, dk, dv, dims, extra, "cuda", F32, 1e-5)
    cases.test_norm_half_rotation_and_mixed_values(hq, hkv, dk, dv, dims, extra, "cuda", BF16, 2e-2)


@pytest.mark.parametrize("H,d,r,R,pad,interleaved", [(4, 12, 8, 20, 0, False), (3, 5, 6, 11, 3, False), (2, 16, 8, 24, 8, True), (16, 128, 64, 192, 0, False),
                                                     (5, 8, 4, 40, 4, False), (33, 24, 10, 512, 6, False), (1, 200, 130, 8, 0, True)])
def test_latent_rows_and_queries(H, d, r, R, pad, interleaved):
    cases.test_latent_rows_and_queries(H, d, r, R, pad, interleaved, "cuda", F32, 1e-5)
    cases.test_latent_rows_and_queries(H, d, r, R, pad, interleaved, "cuda", BF16, 2e-2)


@pytest.mark.parametrize("T,W,E,top,ff,shared", [(5, 32, 6, 2, 12, 20), (40, 50, 3, 3, 7, 9), (1, 64, 8, 1, 16, 8), (9, 40, 4, 2, 24, None), (130, 256, 16, 4, 64, 96),
                                                 (3, 128, 7, 2, 8, 24)])
def test_expert_forms(T, W, E, top, ff, shared):
    cases.test_experts_beside_a_mixer(T, W, E, top, ff, shared, "cuda", F32, 2e-5)
    for form in ("gather", "dense", "grouped", None):
        cases.test_experts_beside_a_mixer(T, W, E, top, ff, shared, "cuda", BF16, 6e-2, form=form)


@pytest.mark.parametrize("name", ["latent", "chunk", "experts", "mixed", "edges", "odd", "wide"])
def test_whole_prompt_and_residual_stream(tmp_path, name):
    cases.test_whole_prompt_and_residual_stream(tmp_path / "a", name, "cuda", F32, 3e-4)
    cases.test_whole_prompt_and_residual_stream(tmp_path / "b", name, "cuda", BF16, 8e-2, margin=0.05 if name != "mixed" else 0.04)


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
    """bfloat16 on the tensor-core kernels: portions and single tokens against the oracle, in all expert forms."""
    cfg, W, eng = cases.build(tmp_path, "wide", "cuda", BF16)
    toks = cases.tokens_for(cfg, 200, 3)
    want, ok = cases.want_logits(toks, cfg, W), cases.clear_choices(toks, cfg, W, 0.05)
    assert ok.float().mean() > 0.5
    for sizes in ([200], [150, 1], [31, 2, 36, 1, 1, 59, 2, 1], [64, 64, 1]):
        cases.close(cases.feed_in_portions(eng, "p", toks, sizes).cpu()[ok], want[ok], 1e-1)


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
        ok = cases.clear_choices(t, cfg, W, 0.05)[len(t) - tail - 1:]
        d = (torch.cat(got[k]).double().cpu() - whole[k][len(t) - tail - 1:]).abs().max(-1).values / std
        assert d[ok].max() < 8e-2, (k, d)


@pytest.mark.parametrize("graph", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_generation(tmp_path, dtype, graph):
    cases.test_greedy_generation_through_engine_and_cli(tmp_path, "cuda", dtype, graph)


def test_generation_by_graph_equals_eager(tmp_path):
    """bfloat16 at tensor-core sizes: the captured decode step (padded batch, inert rows) and the eager one choose the same tokens
    past several page borders, windows and chunks."""
    cfg, W, a = cases.build(tmp_path, "wide", "cuda", BF16, max_batch=3, graph=True)
    _, _, b = cases.build(tmp_path, "wide", "cuda", BF16, max_batch=3, graph=False)
    prompts = [cases.tokens_for(cfg, n, 90 + n) for n in (60, 130, 5)]
    sp = cases.SamplingParams(max_new_tokens=80, is_greedy=True)
    ga, gb = a.generate(prompts, sp), b.generate(prompts, sp)
    assert ga == gb and a.runner.stats["graph_replays"] > 0
    seq = prompts[1] + ga[1]
    lg, ok = cases.want_logits(seq, cfg, W), cases.clear_choices(seq, cfg, W, 0.05)
    for t, tok in enumerate(ga[1]):
        row = lg[len(prompts[1]) + t - 1]
        assert row[tok] >= row.max() - 0.2 * lg.std() or not ok[len(prompts[1]) + t - 1]


def test_shared_prompt_prefix_and_prompt_rounds(tmp_path):
    cases.test_shared_prompt_prefix_and_prompt_rounds(tmp_path, "cuda", F32)
