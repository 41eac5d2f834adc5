"""Fipavik through the engine (CPU: the 32-bit PyTorch ops) against the plain float64 oracle in fipavik_oracle.py.

Own small configurations and random weights; the same cases run on CUDA in test_gpu_fipavik.py.
"""
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch
from safetensors.torch import load_file, save_file

import fipavik_oracle as oracle
from llmss_b200 import ops
from llmss_b200.engine.batch import BatchInput
from llmss_b200.engine.engine import Engine
from llmss_b200.engine.runner import SamplingParams
from llmss_b200.utils.checkpoint import fipavik_config, write_random_checkpoint

ROOT = Path(__file__).resolve().parents[1]
TOL = 2e-4
F64 = torch.float64


def lat(heads=4, dim=12, rot_dim=8, vdim=10, kv_rank=20, window=19, mlp=None, **kw):
    return dict(type="latent_attention", heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, window=window, mlp=mlp, **kw)


def att(heads=4, kv_heads=2, dim=12, vdim=8, chunk=13, rot_dims=8, mlp=None, **kw):
    return dict(type="attention", heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, chunk=chunk, rot_dims=rot_dims, mlp=mlp, **kw)


def moe(experts=5, top=2, ff=12, shared=20):
    return dict(experts=experts, top=top, ff=ff, shared=shared)


CONFIGS = {
    # each mechanism alone
    "latent": fipavik_config(32, 61, [lat()], residual_mult=0.7),
    "chunk": fipavik_config(32, 61, [att()], residual_mult=1.0),
    "experts": fipavik_config(32, 61, [att(heads=1, kv_heads=1, chunk=1, v_mix=False, mlp=moe())], residual_mult=0.4),
    # both kinds in an order of their own; a layer that does not mix between layers that do, layers without experts, without a shared
    # expert, different sizes per layer
    "mixed": fipavik_config(48, 97, [
        att(heads=6, kv_heads=3, dim=16, vdim=8, chunk=21, rot_dims=12, base=300.0, v_mix=False, mlp=moe(experts=7, top=3, ff=10, shared=14)),
        att(chunk=17, rot_dims=4, base=5000.0, mlp=moe(shared=None)),
        lat(heads=3, window=23, base=700.0, mlp=moe(experts=4, top=1)),
        att(heads=2, chunk=29, scale=0.4, mlp=None),
        lat(heads=5, dim=8, rot_dim=12, vdim=14, kv_rank=16, window=11, scale=0.3),
        att(heads=8, dim=8, rot_dims=6, chunk=40, mlp=moe(experts=6, top=2, ff=16, shared=8))], residual_mult=0.35),
    # ends of every range: one visible key, a chunk that is a page, one expert, all experts, one head, rotation of all or two channels
    "edges": fipavik_config(32, 61, [
        lat(heads=1, rot_dim=2, window=1, mlp=moe(experts=1, top=1, shared=None)),
        att(heads=3, kv_heads=3, chunk=16, rot_dims=12, mlp=moe(experts=3, top=3, ff=1, shared=1)),
        lat(heads=2, vdim=1, kv_rank=1, window=16, mlp=None),
        att(heads=3, kv_heads=3, dim=2, chunk=32, rot_dims=2),
        att(heads=2, kv_heads=1, vdim=20, chunk=400, rot_dims=2, v_mix=False, mlp=moe())], residual_mult=1.5, eps=1e-4),
    # nothing a multiple of 4: the scalar forms of the row kernels, products off the 16-byte rules
    "odd": fipavik_config(50, 101, [
        att(heads=3, kv_heads=1, dim=9, vdim=7, rot_dims=6, chunk=17, mlp=moe(experts=5, top=3, ff=13, shared=9)),
        lat(heads=3, dim=5, rot_dim=6, vdim=7, kv_rank=11, window=10, mlp=moe(experts=3, top=2, ff=7, shared=11)),
        att(heads=5, kv_heads=1, dim=6, vdim=7, rot_dims=2, chunk=31)], residual_mult=0.8),
}


def write_ckpt(tmp_path, cfg, seed=0, tweak=None):
    path = write_random_checkpoint(Path(tmp_path) / f"ckpt{seed}", cfg, dtype=torch.bfloat16, device="cpu", seed=seed)
    if tweak is not None:
        for f in sorted(path.glob("*.safetensors")):
            t = load_file(str(f))
            tweak(t)
            save_file({k: v.contiguous() for k, v in t.items()}, str(f), metadata={"format": "pt"})
    return path


def build(tmp_path, name, device="cpu", dtype=torch.float32, seed=0, tweak=None, **kw):
    cfg = CONFIGS[name] if isinstance(name, str) else name
    path = write_ckpt(tmp_path, cfg, seed, tweak)
    kw.setdefault("max_batch", 4)
    kw.setdefault("max_seq_len", 512)
    eng = Engine.from_pretrained(str(path), dtype=dtype, device=torch.device(device), use_cuda_graph=kw.pop("graph", False), **kw)
    return json.loads((path / "config.json").read_text()), oracle.load_weights(path), eng


def tokens_for(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def close(got, want, tol):
    """Largest difference per row relative to the spread of the expected values; every row is held."""
    got, want = torch.as_tensor(got).double().cpu(), torch.as_tensor(want).double().cpu()
    assert got.shape == want.shape
    spread = max(want.std(correction=0).item(), 1e-6)
    d = (got - want).abs().reshape(got.shape[0], -1).max(-1).values / spread
    assert d.max().item() < tol, f"relative error max {d.max().item():.3g} at row {int(d.argmax())} of {d.numel()}, tolerance {tol}"


def feed_in_portions(eng, key, toks, sizes):
    """Feed ``toks`` cut into ``sizes`` (the last size repeats); returns the logits of every position."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(i, len(sizes) - 1)], len(toks) - at)
        out.append(eng.feed([(key, toks[at:at + n], list(range(n)))], [key] if at + n == len(toks) else []))
        at, i = at + n, i + 1
    return torch.cat(out)


def clear_choices(toks, cfg, W, margin):
    """Positions at which no layer's choice of experts is a close call: routing may differ elsewhere by rounding alone."""
    _, layers = oracle.forward(toks, cfg, W, True)
    ok = torch.ones(len(toks), dtype=torch.bool)
    x = W["embed"][torch.as_tensor(toks)]
    for i, L in enumerate(cfg["layers"]):
        f = L.get("mlp")
        if f is not None and f["router"]["top"] < f["router"]["experts"]:
            h = oracle.layer_norm(x, W[f"l{i}.norm1"], W[f"l{i}.norm1.b"], cfg["norm"]["eps"])
            z = torch.sort(h @ W[f"l{i}.mlp.router"].T + W[f"l{i}.mlp.router.b"], dim=-1, descending=True).values
            k = f["router"]["top"]
            ok &= z[:, k - 1] - z[:, k] > margin
        x = layers[i]
    return ok


want_logits = oracle.forward


# ----------------------------------------------------------------------------- mechanisms alone (ops)
@pytest.mark.parametrize("W,bias", [(32, True), (50, True), (1024, False), (7, True)])
def test_residual_norm_with_a_factor(W, bias, device="cpu", out_dtype=torch.float32, tol=2e-5):
    torch.manual_seed(W)
    T, eps = 9, 1e-5
    x, y = torch.randn(T, W) + 20.0 * torch.randn(T, 1), torch.randn(T, W + 5)[:, 5:] * 4.0
    w, b = torch.rand(W) + 0.5, torch.randn(W) if bias else torch.zeros(W)
    d = lambda t: t.to(device)
    for mult in (0.3, 1.0, -2.5):
        h, r = ops.residual_norm(d(x), d(y), d(w), d(b) if bias else None, eps, ops.NORM_LAYER, out_dtype=out_dtype, mult=mult)
        s = x.double() + mult * y.double()
        close(r, s, 1e-6)
        close(h, oracle.layer_norm(s, w.double(), b.double(), eps), tol)


def _pages(bs, n_tokens_per_seq):
    tabs, nb = [], 1
    for n in n_tokens_per_seq:
        k = -(-n // bs)
        tabs.append(list(range(nb + k - 1, nb - 1, -1)))      # pages in falling order: position and page number differ
        nb += k
    return tabs, nb


@pytest.mark.parametrize("hq,hkv,dk,dv,dims,extra", [(4, 2, 12, 8, 8, 0), (2, 1, 16, 20, 16, 6), (6, 3, 5, 7, 4, 3), (8, 2, 64, 32, 24, 8), (3, 3, 20, 4, 4, 4),
                                                     (16, 4, 128, 128, 64, 16)])
def test_norm_half_rotation_and_mixed_values(hq, hkv, dk, dv, dims, extra, device="cpu", dtype=torch.float32, tol=1e-5):
    """Norm before rotation of the pairs (i, i + n) at positions up to thousands; values mixed with those of another projection
    (columns of a wider row), or as projected."""
    torch.manual_seed(hq * dk + dv)
    rot = {"base": 2000.0, "dims": dims}
    freq, _ = ops.rotary_frequencies(dims, rot["base"])
    bs, eps, lam = 16, 1e-3, 0.37
    lens, ctx = [5, 19, 1], [1000, 0, 4095]
    tabs, nb = _pages(bs, [c + n for c, n in zip(ctx, lens)])
    batch = BatchInput.build([[0] * n for n in lens], ctx, tabs, bs, device)
    T, nq, nk = sum(lens), hq * dk, hkv * dk
    wide, first = torch.randn(T, nq + nk + hkv * dv + extra) * 2.0, torch.randn(T, nq + nk + hkv * dv + extra) * 2.0
    qw, kw = torch.rand(dk) + 0.5, torch.rand(dk) + 0.5
    d = lambda t: t.to(device)
    pos = batch.positions.cpu()
    x, v1 = d(wide)[:, :nq + nk + hkv * dv], d(first)[:, nq + nk:nq + nk + hkv * dv]
    v = wide[:, nq + nk:nq + nk + hkv * dv].double().view(T, hkv, dv)
    vf = first[:, nq + nk:nq + nk + hkv * dv].double().view(T, hkv, dv)
    for mix in (True, False):
        kc, vc = torch.zeros(nb, hkv, bs, dk, dtype=dtype, device=device), torch.zeros(nb, hkv, bs, dv, dtype=dtype, device=device)
        q = ops.norm_rope_kv_write(x, hq, hkv, dk, dv, 1, d(qw), d(kw), eps, freq, 1.0, False, batch.positions, batch.slot_mapping, kc, vc,
                                   out_dtype=dtype, v_first=v1 if mix else None, v_lam=lam)
        wq = oracle.rotate(oracle.rms_norm(wide[:, :nq].double().view(T, hq, dk), qw.double(), eps), pos, rot)
        wk = oracle.rotate(oracle.rms_norm(wide[:, nq:nq + nk].double().view(T, hkv, dk), kw.double(), eps), pos, rot)
        wv = oracle.mix_values(v, vf, lam) if mix else v
        close(q, wq.reshape(T, nq), tol)
        s = batch.slot_mapping.long().cpu()
        close(kc.cpu()[s // bs, :, s % bs].reshape(T, -1), wk.reshape(T, -1), tol)
        close(vc.cpu()[s // bs, :, s % bs].reshape(T, -1), wv.reshape(T, -1), tol)
        assert float(kc[0].float().abs().sum()) == 0.0 and float(vc[0].float().abs().sum()) == 0.0


@pytest.mark.parametrize("H,d,r,R,pad,interleaved", [(4, 12, 8, 20, 0, False), (3, 5, 6, 11, 3, False), (2, 16, 8, 24, 8, True), (16, 128, 64, 192, 0, False),
                                                     (5, 8, 4, 40, 4, False)])
def test_latent_rows_and_queries(H, d, r, R, pad, interleaved, device="cpu", dtype=torch.float32, tol=1e-5):
    """Queries straight from the projection: the unrotated parts, the rotated ones in the absorbed-query buffer, the normed
    latent and the rotated key part side by side in the cache row, zeros behind; both pairings."""
    torch.manual_seed(H + d)
    freq, _ = ops.rotary_frequencies(r, 500.0)
    bs, eps, Wd = 16, 1e-3, R + r + pad
    lens, ctx = [7, 1, 18], [300, 2047, 0]
    tabs, nb = _pages(bs, [c + n for c, n in zip(ctx, lens)])
    batch = BatchInput.build([[0] * n for n in lens], ctx, tabs, bs, device)
    T, q_off, nq = sum(lens), 4, H * (d + r)
    y = torch.randn(T, q_off + nq + R + r + 5) * 2.0
    cn = torch.rand(R) + 0.5
    cache = torch.full((nb, bs, Wd), 7.0, dtype=dtype, device=device)
    qn, qa = ops.latent_rope_qkv(y.to(device), q_off, H, d, q_off + nq, R, r, cn.to(device), eps, freq, 1.0, interleaved, batch.positions,
                                 batch.slot_mapping, cache, dtype, dtype)
    pos, rot = batch.positions.cpu(), {"base": 500.0, "dims": r}

    def turned(x):          # neighbouring pairs are the half pairs of the de-interleaved channels
        if not interleaved:
            return oracle.rotate(x, pos, rot)
        o = oracle.rotate(torch.cat([x[..., 0::2], x[..., 1::2]], -1), pos, rot)
        return torch.stack([o[..., :r // 2], o[..., r // 2:]], -1).flatten(-2)

    q = y[:, q_off:q_off + nq].double().view(T, H, d + r)
    close(qn, q[..., :d].reshape(T, H * d), tol)
    tail = qa.view(T, H, Wd)[..., R:].cpu().double()
    close(tail[..., :r].reshape(T, -1), turned(q[..., d:]).reshape(T, -1), tol)
    assert float(tail[..., r:].abs().sum()) == 0.0
    dkv = y[:, q_off + nq:q_off + nq + R + r].double()
    row = torch.cat([oracle.rms_norm(dkv[:, :R], cn.double(), eps), turned(dkv[:, None, R:])[:, 0], torch.zeros(T, pad, dtype=F64)], -1)
    close(cache.view(-1, Wd).cpu()[batch.slot_mapping.long().cpu()], row, tol)
    assert bool((cache[0] == 7.0).all())


def visible(L, window, chunk):
    ok = torch.ones(L, L, dtype=torch.bool).tril()
    if window:
        ok &= oracle.visible_window(L, window)
    if chunk:
        ok &= oracle.visible_chunk(L, chunk)
    return ok


MASKS = [(0, 0), (20, 0), (1, 0), (64, 0), (0, 1), (0, 16), (0, 37), (0, 64), (0, 128), (30, 50), (0, 1000)]


@pytest.mark.parametrize("H,G,dk,dv,shared", [(4, 2, 8, 12, 0), (3, 3, 6, 10, 0), (4, 1, 20, 12, 1), (2, 1, 9, 5, 1)])
def test_chunk_and_window_edges_sinks_and_far_keys(H, G, dk, dv, shared, device="cpu", dtype=torch.float32, tol=1e-4, bs=16, L=150, masks=MASKS):
    """Attention over the pages with chunks, windows and sinks; ``shared``: the value is the first dv columns of the key row.  Keys just
    inside and just outside a chunk or window, at both sides of page borders, token 0 and far ones are made to dominate the
    softmax of chosen queries, so that one hidden or shown wrongly changes the row.  Prompt, portions down to two tokens,
    single tokens."""
    scale = 0.8 * 8 / dk ** 0.75
    for window, chunk in masks:
        torch.manual_seed(window * 7 + chunk)
        q, k, v = torch.randn(L, H, dk), torch.randn(L, G, dk), torch.randn(L, G, dv)
        sink = torch.randn(H) + torch.linspace(0.0, 3.0, H)
        w, c = window or 41, chunk or 45
        edge = lambda i: i // c * c
        pairs = [(149, 149 - w + 1), (148, 148 - w), (147, 147 - w - 1), (131, 131 - w + 1), (146, 0), (139, 15), (138, 16), (120, 63), (121, 64),
                 (100, 1), (64, 47), (33, 31), (17, 16), (145, 144), (128, 127)]
        pairs += [(i, j) for i in (144, 137, 119, 101, 80, 63, 40) for j in (edge(i), edge(i) - 1)]
        for i, j in pairs:
            if 0 <= j <= i:
                k[j] += 3.0 * q[i].view(G, H // G, dk).mean(1)
        if shared:
            v = k[..., :dv]
        q, k, v = (x.to(dtype).double() for x in (q, k, v))
        rep = H // G

        def expect(window, chunk, sink):
            s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, 1)) * scale
            a = oracle.sink_softmax(s, visible(L, window, chunk), sink.double())
            return torch.einsum("hij,jhd->ihd", a, v.repeat_interleave(rep, 1)).reshape(L, H * dv)

        want = expect(window, chunk, sink)
        if dtype == torch.float32:          # the edges and the sink show: one position more or less, or no sink, is far off
            others = [(window, chunk, sink - 50.0)] + ([(window + 1, chunk, sink)] if 0 < window < L - 2 else [])
            others += [(window, chunk + 1, sink)] if 0 < chunk < L - 2 else []
            for o in others:
                assert (expect(*o) - want).abs().max() > 30 * tol * want.std(), (window, chunk)
        pages = -(-L // bs)
        table = list(range(pages, 0, -1))
        kc = torch.zeros(1 + pages, G, bs, dk, dtype=dtype)
        vc = kc[..., :dv] if shared else torch.zeros(1 + pages, G, bs, dv, dtype=dtype)
        for p in range(L):
            vc[table[p // bs], :, p % bs] = v[p].to(dtype)
            kc[table[p // bs], :, p % bs] = k[p].to(dtype)
        kc = kc.to(device)
        vc = kc[..., :dv] if shared else vc.to(device)
        for cuts in ([L], [33, L - 33], [L - 40] + [1] * 40, [15, 2, 2, 30, 1, 64, L - 114]):
            at, rows = 0, []
            for n in cuts:
                batch = BatchInput.build([[0] * n], [at], [table], bs, device)
                rows.append(ops.attention_bias(q[at:at + n].reshape(n, -1).to(dtype).to(device), kc, vc, batch, H, G, dk, dv, scale, None,
                                               out_dtype=dtype, window=window, chunk=chunk, sinks=sink.to(device)))
                at += n
            close(torch.cat(rows), want, tol)


@pytest.mark.parametrize("T,W,E,top,ff,shared", [(5, 32, 6, 2, 12, 20), (40, 50, 3, 3, 7, 9), (1, 64, 8, 1, 16, 8), (9, 40, 4, 2, 24, None)])
def test_experts_beside_a_mixer(T, W, E, top, ff, shared, device="cpu", dtype=torch.float32, tol=1e-5, form=None):
    """The parallel block: a stand-in mixer that hands out known heads, routed experts (bias on the router, weights over the chosen
    logits only), the expert every token takes, one sum."""
    from llmss_b200.models.blocks import RoutedExperts
    from llmss_b200.models.decoder import interleave_gate_up
    from llmss_b200.models.mixers import GatedFFN, ParallelBlock

    torch.manual_seed(T + W)
    n_ctx = 24
    rnd = lambda *s: (torch.randn(*s) * s[-1] ** -0.5).to(dtype)
    p = {"router": 3.0 * rnd(E, W), "router.b": (torch.randn(E) * 0.7).to(dtype)}
    for e in [f"e{i}" for i in range(E)] + (["shared"] if shared else []):
        n = shared if e == "shared" else ff
        p.update({f"{e}.gate": 2 * rnd(n, W), f"{e}.up": rnd(n, W), f"{e}.down": 2 * rnd(W, n)})
    heads, w_o, w_in = torch.randn(T, n_ctx).to(dtype), rnd(W, n_ctx), rnd(10, W)
    d = lambda t: t.to(device)

    class Mixer:
        def __init__(self):
            self.w_in, self.b_in, self.w_o, self.b_o, self.n_out = d(w_in), None, d(w_o), None, n_ctx

        def context(self, h, batch, lc, dtype, out=None, y=None, carry=None):
            self.seen = y[:, :10]
            out.copy_(d(heads))

    ex = RoutedExperts(E, top, 1, 1, 1.0, ff, act=ops.ACT_SILU, gated=True)
    ex.w_router, ex.b_router = d(p["router"]), d(p["router.b"])
    ex.w_up = d(torch.stack([interleave_gate_up(p[f"e{i}.gate"], p[f"e{i}.up"]) for i in range(E)]))
    ex.w_down = d(torch.cat([p[f"e{i}.down"] for i in range(E)], dim=1))
    ffn = None
    if shared:
        ffn = GatedFFN(ops.ACT_SILU)
        ffn.set_weights(d(p["shared.gate"]), d(p["shared.up"]), d(p["shared.down"]))
    if form is not None:
        ex.form = lambda h: form
    block = ParallelBlock(Mixer(), ffn, ex)
    block.finalize()
    h = torch.randn(T, W).to(dtype)
    got = block.forward(d(h), None, None, dtype, {})
    p64, cfg = {k: v.double() for k, v in p.items()}, {"router": {"top": top}, "shared": {"ff": shared} if shared else None}
    want = heads.double() @ w_o.double().T + oracle.mixture(h.double(), p64, "", cfg)
    close(got, want, tol)
    close(block.mixer.seen, h.double() @ w_in.double().T, tol)
    assert got.dtype == torch.float32


def test_routing_weights_are_over_the_chosen_logits():
    z = torch.tensor([[1.0, 3.0, 2.0, -1.0, 2.5], [-4.0, 0.0, 60.0, -60.0, 1.0]])
    ids, w = ops.moe_route(z, 5, 3, 1, 1, 1.0)
    want = oracle.route(z.double(), 3)
    got = torch.zeros_like(want)
    got.scatter_(1, ids.long(), w.double())
    assert (got - want).abs().max() < 1e-6 and (want > 0).sum(-1).tolist() == [3, 3]


# ----------------------------------------------------------------------------- the model, whole prompts
def residual_stream(eng, toks):
    """The residual stream that leaves every layer for one whole prompt, through the core's own forward."""
    r = eng.runner
    n = -(-len(toks) // r.block_size)
    batch = BatchInput.build([toks], [0], [list(range(1, n + 1))], r.block_size, r.device, max_blocks=r.max_blocks_per_seq)
    taps = []
    with torch.no_grad():
        eng.core.forward_hidden(batch, r.kv, taps)
    return taps


@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_residual_stream(tmp_path, name, device="cpu", dtype=torch.float32, tol=TOL, margin=1e-4):
    cfg, W, eng = build(tmp_path, name, device, dtype)
    toks = tokens_for(cfg, 75, 1)
    want, layers = oracle.forward(toks, cfg, W, True)
    ok = clear_choices(toks, cfg, W, margin)
    assert ok.float().mean() > 0.6
    got = residual_stream(eng, toks)
    assert len(got) == len(layers)
    for i, g in enumerate(got):
        close(g.cpu()[ok], layers[i][ok], tol * (1 + i))
    close(eng.feed([("a", toks, list(range(len(toks))))], ["a"]).cpu()[ok], want[ok], tol * 2)


def test_each_mechanism_matters(tmp_path):
    """The oracle itself: leaving out one mechanism moves the logits far beyond any tolerance used here, so the comparisons do
    see it."""
    path = write_ckpt(tmp_path, CONFIGS["mixed"], 0)
    cfg, W = json.loads((path / "config.json").read_text()), oracle.load_weights(path)
    toks = tokens_for(cfg, 60, 1)
    want = oracle.forward(toks, cfg, W)

    def moved(change):
        W2, cfg2 = {k: v.clone() for k, v in W.items()}, json.loads(json.dumps(cfg))
        change(cfg2, W2)
        return (oracle.forward(toks, cfg2, W2) - want).abs().max() / want.std()

    def sized(kind, by):
        def f(c, w):
            for L in c["layers"]:
                if L["type"] == kind:
                    L["mixer"]["mask"]["size"] += by
        return f

    def ends(suffix, f):
        def g(c, w):
            for k in w:
                if k.endswith(suffix):
                    w[k] = f(w[k])
        return g

    def no_mixing(c, w):
        for L in c["layers"]:
            L["mixer"].pop("v_mix", None)

    def mix_with_the_first_layer(c, w):
        c["layers"][0]["mixer"].update(c["layers"][1]["mixer"], v_mix=True)
        for k in ("q", "k", "v", "o", "q.norm", "k.norm", "sink"):
            w[f"l0.mix.{k}"] = w[f"l1.mix.{k}"]

    def other_base(c, w):
        for L in c["layers"]:
            L["mixer"]["rot"]["base"] *= 2.0

    def no_shared(c, w):
        for L in c["layers"]:
            if L["mlp"] is not None:
                L["mlp"].pop("shared", None)

    def one_less(c, w):
        for L in c["layers"]:
            if L["mlp"] is not None and L["mlp"]["router"]["top"] > 1:
                L["mlp"]["router"]["top"] -= 1

    for name, change in {"window": sized("latent_attention", 1), "chunk": sized("attention", 1), "sink": ends(".sink", lambda t: t - 40.0),
                         "vmix": ends(".vmix", lambda t: t * 0.0), "no mixing": no_mixing, "first mixing layer": mix_with_the_first_layer,
                         "norm bias": ends("norm1.b", lambda t: t * 0.0), "final bias": ends("final.norm.b", lambda t: t * 0.0),
                         "latent norm": ends("dkv.norm", torch.ones_like), "key norm": ends("k.norm", torch.ones_like),
                         "router bias": ends("router.b", lambda t: t * 0.0), "base": other_base, "shared": no_shared, "top": one_less,
                         "mult": lambda c, w: c.update(residual_mult=c["residual_mult"] * 1.05)}.items():
        assert moved(change) > 20 * TOL, name


# ----------------------------------------------------------------------------- decoding, portions, batches
@pytest.mark.parametrize("name", ["mixed", "edges", "odd"])
def test_decode_token_by_token_and_portions(tmp_path, name, device="cpu", dtype=torch.float32, tol=TOL):
    """Prefill against token-by-token decoding, and portions down to two tokens that cut pages, windows and chunks."""
    cfg, W, eng = build(tmp_path, name, device, dtype)
    toks = tokens_for(cfg, 70, 2)
    want, ok = want_logits(toks, cfg, W), clear_choices(toks, cfg, W, 1e-4)
    for sizes in ([1], [2], [3, 1, 2, 7, 1, 1, 16, 5], [15, 1, 1, 17, 2], [33, 31, 1], [64, 1]):
        close(feed_in_portions(eng, "s", toks, sizes).cpu()[ok], want[ok], tol * 2)


def test_unequal_batches_against_each_alone(tmp_path, device="cpu", dtype=torch.float32, tol=TOL):
    """Portions of some requests beside single tokens of others in one step; every request equals itself alone."""
    cfg, W, eng = build(tmp_path, "mixed", device, dtype, max_batch=5)
    reqs = {k: tokens_for(cfg, n, 10 + i) for i, (k, n) in enumerate([("a", 61), ("b", 9), ("c", 33), ("d", 1), ("e", 20)])}
    want = {k: want_logits(t, cfg, W) for k, t in reqs.items()}
    plan = [[("a", 20), ("b", 1)], [("a", 1), ("b", 1), ("c", 17)], [("a", 2), ("c", 1), ("d", 1), ("b", 3)],
            [("a", 30), ("b", 1), ("c", 2), ("e", 5)], [("b", 3), ("c", 13), ("e", 1)], [("a", 8), ("e", 14)]]
    at, got = {k: 0 for k in reqs}, {k: [] for k in reqs}
    for step in plan:
        entries, end = [], []
        for k, n in step:
            entries.append((k, reqs[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
            if at[k] == len(reqs[k]):
                end.append(k)
        out = eng.feed(entries, end)
        o = 0
        for k, n in step:
            got[k].append(out[o:o + n])
            o += n
    for k in reqs:
        assert at[k] == len(reqs[k])
        ok = clear_choices(reqs[k], cfg, W, 1e-4)
        close(torch.cat(got[k]).cpu()[ok], want[k][ok], tol * 2)


def test_pages_are_used_again(tmp_path, device="cpu", dtype=torch.float32, tol=TOL):
    """A pool of a few pages serves six requests one after another and overlapping; what a page held before must not show.  A
    request beyond the pool, and one live request too many, are errors."""
    cfg, W, eng = build(tmp_path, "mixed", device, dtype, max_batch=2)
    bs = eng.runner.block_size
    _, _, small = build(tmp_path / "p", "mixed", device, dtype, max_batch=2, pool_tokens=4 * bs)

    def check(got, toks):
        ok = clear_choices(toks, cfg, W, 1e-4)
        close(got.cpu()[ok], want_logits(toks, cfg, W)[ok], tol * 2)

    for e in (eng, small):
        lens = [bs + 3, 2 * bs, 5, bs - 1, bs + 1, 7]
        reqs = [tokens_for(cfg, n, 30 + i) for i, n in enumerate(lens)]
        a = e.feed([(0, reqs[0][:5], list(range(5))), (1, reqs[1], list(range(lens[1])))], [1])
        check(a[5:], reqs[1])
        b = e.feed([(0, reqs[0][5:], list(range(lens[0] - 5))), (2, reqs[2], list(range(5)))], [0, 2])
        check(torch.cat([a[:5], b[:lens[0] - 5]]), reqs[0])
        check(b[lens[0] - 5:], reqs[2])
        for i in (3, 4, 5):
            check(feed_in_portions(e, i, reqs[i], [4, 1]), reqs[i])
        assert e.runner.alloc.num_free == e.runner.alloc.num_blocks - 1
    eng.feed([("x", [1, 2], []), ("y", [3], [])])
    with pytest.raises(RuntimeError):
        eng.feed([("z", [4], [])])
    eng.feed([], ["x", "y"])
    with pytest.raises((MemoryError, ValueError)):
        small.feed([("big", tokens_for(cfg, 5 * bs, 1), [])])


def steep_config():
    """Attention decided by single keys (a score scale several times the usual one): a key lost at a page border, a chunk's or window's
    edge, or a position rotated wrongly far from the start changes the result at once."""
    return fipavik_config(32, 71, [
        lat(heads=2, dim=8, rot_dim=8, vdim=8, kv_rank=12, scale=2.0, base=50.0, window=65),
        att(heads=2, kv_heads=1, dim=8, vdim=12, scale=2.5, base=50.0, chunk=48),
        lat(heads=4, dim=8, rot_dim=4, vdim=8, kv_rank=12, scale=2.0, base=20.0, window=32, mlp=moe(ff=16)),
        att(heads=2, kv_heads=1, dim=8, vdim=12, scale=2.5, base=50.0, chunk=128)], residual_mult=0.9)


def low_sinks(t):
    for k in t:
        if k.endswith(".sink"):
            t[k] = t[k] - 1.0


def test_steep_attention_far_back_and_over_page_borders(tmp_path, device="cpu", dtype=torch.float32, tol=TOL):
    cfg, W, eng = build(tmp_path, steep_config(), device, dtype, tweak=low_sinks)
    toks = tokens_for(cfg, 150, 4)
    want, ok = want_logits(toks, cfg, W), clear_choices(toks, cfg, W, 1e-3)
    for sizes in ([150], [31, 2, 36, 1, 1, 59, 2, 1], [100, 1]):
        close(feed_in_portions(eng, "w", toks, sizes).cpu()[ok], want[ok], tol * 4)
    # the first token of a chunk reaches the last one of it: another one there changes it
    toks2 = toks[:48] + [(toks[48] + 1) % cfg["vocab"]] + toks[49:]
    assert (want_logits(toks2, cfg, W)[95] - want[95]).abs().max() > 10 * tol * want.std()


def test_first_tokens(tmp_path, device="cpu", dtype=torch.float32, tol=TOL):
    """One-token and two-token requests, and the first tokens one by one, in pages that another request has just left."""
    cfg, W, eng = build(tmp_path, "mixed", device, dtype)
    feed_in_portions(eng, "warm", tokens_for(cfg, 40, 7), [40])          # leaves keys behind
    for n in (1, 2, 3, 6):
        toks = tokens_for(cfg, n, 50 + n)
        want, ok = want_logits(toks, cfg, W), clear_choices(toks, cfg, W, 1e-4)
        close(feed_in_portions(eng, "f", toks, [n]).cpu()[ok], want[ok], tol * 2)
        close(feed_in_portions(eng, "g", toks, [1]).cpu()[ok], want[ok], tol * 2)


def test_long_decoding(tmp_path, device="cpu", dtype=torch.float32, tol=TOL):
    cfg, W, eng = build(tmp_path, "mixed", device, dtype)
    toks = tokens_for(cfg, 160, 8)
    ok = clear_choices(toks, cfg, W, 2e-4)
    close(feed_in_portions(eng, "l", toks, [12, 1]).cpu()[ok], want_logits(toks, cfg, W)[ok], tol * 4)


# ----------------------------------------------------------------------------- generation through the public entry points
def oracle_greedy(W, cfg, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(want_logits(toks, cfg, W)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_engine_and_cli(tmp_path, device="cpu", dtype=torch.float32, graph=False):
    """Engine.generate: admission of more requests than the batch holds, packed prefill, decode steps, the sampler; then generate.py."""
    cfg, W, eng = build(tmp_path, "mixed", device, dtype, max_batch=2, graph=graph)
    prompts = [tokens_for(cfg, n, 60 + n) for n in (9, 1, 14)]
    got = eng.generate(prompts, SamplingParams(max_new_tokens=7, is_greedy=True))
    if dtype == torch.float32:
        assert got == [oracle_greedy(W, cfg, p, 7) for p in prompts]
    else:   # 16-bit: teacher-forced, every chosen token is the oracle's best or within rounding of it
        for p, g in zip(prompts, got):
            ok = clear_choices(p + g, cfg, W, 3e-2)
            lg = want_logits(p + g, cfg, W)
            for t, tok in enumerate(g):
                row = lg[len(p) + t - 1]
                assert row[tok] >= row.max() - 0.2 * lg.std() or not ok[len(p) + t - 1]
    if device == "cpu":
        path = tmp_path / "ckpt0"
        r = subprocess.run([sys.executable, str(ROOT / "generate.py"), "--pretrained_model_path", str(path), "--prompt_ids",
                            " ".join(map(str, prompts[0])), "--max_new_tokens", "5", "--is_greedy", "--use_cache"],
                           capture_output=True, text=True, timeout=300, cwd=str(ROOT), env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
        assert r.returncode == 0, r.stderr[-2000:]
        assert " ".join(map(str, got[0][:5])) in r.stdout.replace(",", " ").replace("  ", " "), r.stdout[-1000:]


def test_shared_prompt_prefix_and_prompt_rounds(tmp_path, device="cpu", dtype=torch.float32):
    """The cache holds pages only (the mixed values included), so a later prompt may continue on the pages of an earlier one with the
    same start; and prompts may be processed in rounds.  Eviction from the front is refused where chunks are counted from it."""
    cfg, W, plain = build(tmp_path, "mixed", device, dtype)
    _, _, shared = build(tmp_path, "mixed", device, dtype, prefix_cache=True)
    _, _, rounds = build(tmp_path, "mixed", device, dtype, prefill_chunk=7)
    bs = plain.runner.block_size
    head = tokens_for(cfg, 2 * bs + 3, 70)
    sp = SamplingParams(max_new_tokens=6, is_greedy=True)
    for tail in ([5, 6], [7], [5, 6, 8, 9]):
        want = plain.generate([head + tail], sp)
        assert shared.generate([head + tail], sp) == want
        assert rounds.generate([head + tail], sp) == want
    assert shared.runner.stats.get("prefix_hit_tokens", 0) >= 4 * bs
    _, _, e = build(tmp_path, "mixed", device, dtype, sliding_window=True)
    assert not e.runner.sliding
    _, _, e = build(tmp_path / "latent", "latent", device, dtype, sliding_window=True)
    assert e.runner.sliding


def test_model_call_with_a_past(tmp_path, device="cpu", dtype=torch.float32, tol=TOL):
    """The HF-shaped call: a prompt, then single tokens, with the cache object handed back."""
    from llmss_b200.models import MODEL_REGISTRY
    from llmss_b200.utils.config import load_config
    from llmss_b200.utils.dist import FakeGroup
    from llmss_b200.utils.hub import weight_files
    from llmss_b200.utils.weights import Weights

    path = write_ckpt(tmp_path, CONFIGS["mixed"], 0)
    cfg, W = json.loads((path / "config.json").read_text()), oracle.load_weights(path)
    config = load_config(str(path))
    weights = Weights(weight_files(str(path)), device=torch.device(device), dtype=dtype, process_group=FakeGroup(0, 1))
    model = MODEL_REGISTRY[config.model_type](config, weights).eval()
    assert model.core.num_parameters_local() == sum(v.numel() for k, v in W.items() if not k.endswith(".vmix"))
    seqs = [tokens_for(cfg, 30, 3), tokens_for(cfg, 30, 4)]
    ids = torch.tensor(seqs)
    out = model(ids[:, :21], use_cache=True)
    rows = [out.logits]
    for t in range(21, 30):
        out = model(ids[:, t:t + 1], past_key_values=out.past_key_values, use_cache=True)
        rows.append(out.logits)
    got = torch.cat(rows, dim=1)
    for b in (0, 1):
        ok = clear_choices(seqs[b], cfg, W, 1e-4)
        close(got[b].cpu()[ok], want_logits(seqs[b], cfg, W)[ok], tol * 2)


def test_trace_replay_writes_the_logits_it_is_asked_for(tmp_path):
    """bin/trace_run on CPU: two requests in portions and single tokens, logits files per step, `done` lines."""
    path = write_ckpt(tmp_path, CONFIGS["mixed"], 0)
    cfg, W = json.loads((path / "config.json").read_text()), oracle.load_weights(path)
    a, b = tokens_for(cfg, 21, 1), tokens_for(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": [0, 16]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[17:18], "want": []}, {"id": "b", "tokens": b[:7], "want": [6]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[7:], "want": [0, 1]}, {"id": "a", "tokens": a[18:], "want": [2]}],
              "end": ["a", "b"]}]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(path), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                       timeout=300, cwd=str(ROOT), env={**os.environ, "CUDA_VISIBLE_DEVICES": "", "LLMSS_TRACE_CPU": "1"})
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = want_logits(a, cfg, W), want_logits(b, cfg, W)
    read = lambda n: torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    close(read(0), wa[[0, 16]], TOL * 2)
    close(read(1), wb[[6]], TOL * 2)
    close(read(2), torch.cat([wb[[7, 8]], wa[[20]]]), TOL * 2)


def test_unknown_kinds_and_impossible_sizes_are_refused():
    from llmss_b200.models.fipavik import FipavikLM, fipavik_spec
    from llmss_b200.utils.dist import FakeGroup

    def bad(change):
        cfg = json.loads(json.dumps(CONFIGS["mixed"]))
        change(cfg["layers"])
        with pytest.raises(ValueError):
            FipavikLM(fipavik_spec(cfg), FakeGroup(0, 1), torch.device("cpu"), torch.float32)

    bad(lambda L: L[0].update(type="other"))
    bad(lambda L: L[0]["mlp"].update(kind="other"))
    bad(lambda L: L[3]["mixer"].update(vdim=9))                    # values of another size cannot mix
    bad(lambda L: L[0]["mlp"]["router"].update(top=8))             # more experts than there are
    bad(lambda L: L[2]["mixer"]["rot"].update(dims=10))            # more rotated channels than the key part has
