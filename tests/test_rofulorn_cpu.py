"""Rofulorn through the engine (CPU: the 32-bit PyTorch ops) against the plain float64 oracle in rofulorn_oracle.py.

Own small configurations and random weights; the same cases run on CUDA in test_gpu_rofulorn.py.
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

import rofulorn_oracle as oracle
from llmss_b200 import ops
from llmss_b200.engine.batch import BatchInput
from llmss_b200.engine.engine import Engine
from llmss_b200.engine.runner import SamplingParams
from llmss_b200.utils.checkpoint import rofulorn_config, write_random_checkpoint

ROOT = Path(__file__).resolve().parents[1]
TOL = 2e-4
F64 = torch.float64
WAVE = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 48}


def dif(heads=4, kv_heads=2, dim=12, vdim=20, window=19, keep_first=3, diff=0.4, softcap=6.0, mlp=None, rot_dims=8, scaling=WAVE, **kw):
    return dict(type="attention", heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, window=window, keep_first=keep_first, diff=diff,
                softcap=softcap, mlp=mlp, rot_dims=rot_dims, scaling=scaling, **kw)


def pln(heads=4, kv_heads=2, dim=12, vdim=8, window=13, mlp=None, **kw):
    return dict(type="attention_2", heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, window=window, mlp=mlp, **kw)


CONFIGS = {
    # each mechanism alone
    "plain": rofulorn_config(32, 61, [pln(rot_dims=6, base=300.0)], embed_scale=3.0),
    "diff": rofulorn_config(32, 61, [dif()], embed_scale=3.0),
    "ffn": rofulorn_config(32, 61, [pln(heads=1, kv_heads=1, window=1, mlp={"ff": 40})], embed_scale=2.0),
    # both kinds in an order of their own; two borrowers of different lenders, one with another window and more first tokens
    # than its lender; layers without a feed-forward
    "mixed": rofulorn_config(48, 97, [
        dif(mlp={"ff": 56}),
        pln(heads=6, kv_heads=3, dim=10, vdim=14, window=27, base=500.0, mlp={"ff": 24}),
        dif(heads=6, kv_heads=1, dim=8, vdim=12, window=9, keep_first=6, diff=0.8, softcap=None, scaling=None, rot_dims=4),
        dif(kv_from=0, window=31, keep_first=5, diff=0.2, mlp={"ff": 32}),
        pln(heads=2, kv_heads=2, dim=14, vdim=6, window=37),
        dif(heads=6, kv_heads=1, dim=8, vdim=12, window=12, keep_first=1, diff=0.5, softcap=3.0, scaling=None, rot_dims=4, kv_from=2,
            mlp={"ff": 40})], embed_scale=5.0),
    # values that are often 1 or equal: one head, one key, a window of one token, no first tokens or more of them than the window,
    # rotation of all or two channels, a scaling factor of 1, equal key and value sizes
    "edges": rofulorn_config(40, 53, [
        dif(heads=1, kv_heads=1, dim=8, vdim=8, window=1, keep_first=1, diff=0.1, rot_dims=8, scaling={"factor": 1.0, "low": 1.0, "high": 4.0, "original": 8}),
        pln(heads=5, kv_heads=5, dim=6, vdim=6, window=2, rot_dims=2, mlp={"ff": 8}),
        dif(heads=5, kv_heads=5, dim=4, vdim=8, window=3, keep_first=20, diff=0.9, rot_dims=2, scaling=None, softcap=1.0, mlp={"ff": 16}),
        dif(heads=2, kv_heads=1, dim=6, vdim=4, window=16, keep_first=0, diff=0.65, rot_dims=6, softcap=None),
        pln(heads=3, kv_heads=1, dim=16, vdim=4, window=16)], embed_scale=1.0, eps=1e-4),
    # nothing a multiple of 4: the scalar forms of the row kernels, products off the 16-byte rules
    "odd": rofulorn_config(50, 101, [
        pln(heads=3, kv_heads=1, dim=9, vdim=7, rot_dims=6, window=17, mlp={"ff": 13}),
        dif(heads=3, kv_heads=3, dim=5, vdim=11, rot_dims=2, window=10, keep_first=2, mlp={"ff": 9}),
        dif(heads=3, kv_heads=3, dim=5, vdim=11, rot_dims=2, window=23, keep_first=4, kv_from=1)], embed_scale=7.0),
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


def close(got, want, tol, ease=None):
    """Largest difference per row relative to the spread of the expected values; every row is held.  ``ease``: a factor >= 1 per
    row on the tolerance."""
    got, want = torch.as_tensor(got).double().cpu(), torch.as_tensor(want).double().cpu()
    assert got.shape == want.shape
    spread = max(want.std().item(), 1e-6)
    d = (got - want).abs().reshape(got.shape[0], -1).max(-1).values / spread
    if ease is not None:
        d = d / ease
    assert d.max().item() < tol, f"relative error max {d.max().item():.3g} at row {int(d.argmax())} of {d.numel()}, tolerance {tol}"


def feed_in_portions(eng, key, toks, sizes):
    """Feed ``toks`` cut into ``sizes`` (the last size repeats); returns the logits of every position."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(i, len(sizes) - 1)], len(toks) - at)
        out.append(eng.feed([(key, toks[at:at + n], list(range(n)))], [key] if at + n == len(toks) else []))
        at, i = at + n, i + 1
    return torch.cat(out)


def want_logits(toks, cfg, W):
    return oracle.forward(toks, cfg, W)


# ----------------------------------------------------------------------------- mechanisms alone (ops)
@pytest.mark.parametrize("rot", [{"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}},
                                 {"base": 300.0, "dims": 12, "scaling": {"factor": 3.0, "low": 0.5, "high": 9.0, "original": 100}},
                                 {"base": 50.0, "dims": 20, "scaling": {"factor": 16.0, "low": 2.0, "high": 2.5, "original": 64}},
                                 {"base": 77.0, "dims": 10}])
def test_frequency_tables(rot):
    f, mag = ops.rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    assert mag == 1.0 and f.dtype == F64
    assert torch.allclose(f, torch.tensor(oracle.rotary_frequencies(rot), dtype=F64), rtol=1e-12, atol=0)


def test_frequency_table_has_all_three_ranges():
    """Kept, blended and slowed frequencies all occur in the first table above, so each branch is compared."""
    base = oracle.rotary_frequencies({"base": 10000.0, "dims": 64})
    f = oracle.rotary_frequencies({"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}})
    r = [a / b for a, b in zip(f, base)]
    assert sum(x == 1.0 for x in r) > 3 and sum(abs(x - 0.125) < 1e-12 for x in r) > 2 and sum(0.13 < x < 0.99 for x in r) > 2


@pytest.mark.parametrize("W,bias", [(32, False), (50, True), (1024, False), (7, False), (2048, True)])
def test_residual_norm(W, bias, device="cpu", out_dtype=torch.float32, tol=1e-5):
    """Mean and mean square of rows with a large common offset, with and without a branch to add; the RMS kind of the same op."""
    torch.manual_seed(W)
    T, eps = 9, 1e-5
    x, y = torch.randn(T, W) + 30.0 * torch.randn(T, 1), torch.randn(T, W + 5)[:, 5:] * 4.0
    w, b = torch.rand(W) + 0.5, torch.randn(W) if bias else None
    d = lambda t: None if t is None else t.to(device)
    for add in (y, None):
        s = x.double() + (add.double() if add is not None else 0.0)
        for kind in (ops.NORM_LAYER, ops.NORM_RMS):
            h, r = ops.residual_norm(d(x), d(add), d(w), d(b), eps, kind, out_dtype=out_dtype)
            assert h.dtype == out_dtype and r.dtype == torch.float32
            close(r, s, 1e-6)
            want = oracle.layer_norm(s, w.double(), eps) if kind == ops.NORM_LAYER else oracle.rms_div(s, eps) * w.double()
            close(h, want + (b.double() if bias else 0.0), max(tol, 2e-5))


def _pages(bs, n_tokens_per_seq):
    tabs, nb = [], 1
    for n in n_tokens_per_seq:
        k = -(-n // bs)
        tabs.append(list(range(nb + k - 1, nb - 1, -1)))      # pages in falling order: position and page number differ
        nb += k
    return tabs, nb


@pytest.mark.parametrize("hq,hkv,dk,dv,maps,dims,norm", [(4, 2, 12, 8, 1, 8, False), (2, 1, 8, 20, 2, 8, True), (6, 3, 5, 7, 2, 4, True),
                                                         (1, 1, 20, 4, 1, 0, True), (4, 4, 64, 128, 2, 32, True)])
def test_norm_rotation_and_pages(hq, hkv, dk, dv, maps, dims, norm, device="cpu", dtype=torch.float32, tol=1e-5):
    """Norm before rotation, neighbouring pairs at positions up to thousands, both maps of a head in one key row, values as
    projected; then queries only, with the pages untouched."""
    torch.manual_seed(hq * dk + dv)
    rot = {"base": 2000.0, "dims": dims, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 512}} if dims else None
    freq, mag = ops.rotary_frequencies(dims, rot["base"], rot["scaling"]) if dims else (torch.zeros(0, dtype=F64), 1.0)
    bs, eps = 16, 1e-3
    lens, ctx = [5, 19, 1], [1000, 0, 4095]
    tabs, nb = _pages(bs, [c + n for c, n in zip(ctx, lens)])
    batch = BatchInput.build([[0] * n for n in lens], ctx, tabs, bs, device)
    T, nq, nk = sum(lens), hq * maps * dk, hkv * maps * dk
    x = torch.randn(T, nq + nk + hkv * dv) * 2.0
    qw, kw = (torch.rand(dk) + 0.5, torch.rand(dk) + 0.5) if norm else (None, None)
    d = lambda t: None if t is None else t.to(device)
    kc, vc = torch.zeros(nb, hkv, bs, maps * dk, dtype=dtype, device=device), torch.zeros(nb, hkv, bs, dv, dtype=dtype, device=device)

    def prepared(u, heads, w):
        u = u.double().reshape(T, heads * maps, dk)
        if w is not None:
            u = oracle.rms_div(u, eps) * w.double()
        return oracle.rotate(u, batch.positions.cpu(), rot)

    q = ops.norm_rope_kv_write(d(x), hq, hkv, dk, dv, maps, d(qw), d(kw), eps, freq, mag, True, batch.positions, batch.slot_mapping, kc, vc,
                               out_dtype=dtype)
    wq, wk = prepared(x[:, :nq], hq, qw), prepared(x[:, nq:nq + nk], hkv, kw).reshape(T, hkv, maps * dk)
    close(q, wq.reshape(T, nq), tol)
    for t, s in enumerate(batch.slot_mapping.tolist()):
        close(kc[s // bs, :, s % bs], wk[t], tol * 2)
        close(vc[s // bs, :, s % bs], x[t, nq + nk:].reshape(hkv, dv), tol * 2)
    assert float(kc[0].float().abs().sum()) == 0.0
    before = kc.clone()
    q2 = ops.norm_rope_kv_write(d(x[:, :nq].contiguous()), hq, 0, dk, dv, maps, d(qw), None, eps, freq, mag, True, batch.positions,
                                batch.slot_mapping, kc, vc, out_dtype=dtype)
    assert torch.equal(q2, q) and torch.equal(kc, before)


def _pad_maps(q, H, maps, dk, batch, kc, vc, scale):
    """The layout in which the CUDA decode kernel takes the queries of two-map heads (what norm_rope_kv_write produces there)."""
    if maps == 1 or not q.is_cuda or not batch.is_decode:
        return q
    from llmss_b200.ops import cuda_impl as cu

    if not cu.span_decode_uses_tc(q.dtype, H, kc.shape[1], dk, vc.shape[3], maps, kc.shape[2], scale):
        return q
    out = torch.zeros(q.shape[0], H, maps, maps, dk, dtype=q.dtype, device=q.device)
    for m in range(maps):
        out[:, :, m, m] = q.view(-1, H, maps, dk)[:, :, m]
    return out.reshape(q.shape[0], -1)


SPANS = [(0, 0), (20, 0), (20, 4), (1, 1), (33, 7), (64, 3), (7, 70)]


@pytest.mark.parametrize("H,G,dk,dv,maps,cap", [(4, 2, 8, 12, 1, 0.0), (4, 2, 8, 12, 2, 9.0), (3, 3, 6, 10, 2, 0.0), (2, 1, 20, 5, 1, 12.0)])
def test_window_edges_first_tokens_and_far_keys(H, G, dk, dv, maps, cap, device="cpu", dtype=torch.float32, tol=1e-4, bs=16, L=150, spans=SPANS):
    """Attention over the pages with a window, kept first tokens, soft cap and two maps.  Chosen keys -- just inside and just
    outside the window, the last kept and the first not kept token, token 0, both sides of page borders, far ones -- are made
    to dominate the softmax of chosen queries, so that one hidden or shown wrongly changes the row.  Prompt, portions down to
    two tokens, single tokens."""
    scale, lam, eps, factor = 0.8 * 8 / dk ** 0.75, 0.7, 1e-5, 0.6
    for window, keep in spans:
        torch.manual_seed(window * 7 + keep)
        q, k, v = torch.randn(L, H, maps, dk), torch.randn(L, G, maps, dk), torch.randn(L, G, dv)
        # (query, key): distances window - 1, window and window + 1; the last kept and the first not kept token; page borders
        w = window or 41
        pairs = [(149, 149 - w + 1), (148, 148 - w), (147, 147 - w - 1), (131, 131 - w + 1), (129, 129 - w), (140, keep - 1), (141, keep),
                 (146, 0), (139, 15), (138, 16), (120, 63), (121, 64), (100, 1), (64, 47), (33, 31), (17, 16), (145, 144), (128, 127)]
        for i, j in pairs:
            if 0 <= j <= i:
                k[j] += 3.0 * q[i].view(G, H // G, maps, dk).mean(1)
        q, k, v = (x.to(dtype).double() for x in (q, k, v))
        mask = {"size": window, "keep_first": keep} if window else None
        rep = H // G

        def expect(mask):
            a = [oracle.softmax_attention(q[:, :, m], k[:, :, m].repeat_interleave(rep, 1), v.repeat_interleave(rep, 1), scale, mask, cap or None)
                 for m in range(maps)]
            if maps == 1:
                return a[0].reshape(L, H * dv), None
            # rounding of the maps' outputs grows where they nearly cancel: by their sizes over the size of the difference
            size = lambda x: x.square().mean(-1).sqrt()
            ease = ((size(a[0]) + lam * size(a[1])) / size(a[0] - lam * a[1]) / 3.0).max(-1).values.clamp(min=1.0)
            return (oracle.rms_div(a[0] - lam * a[1], eps) * factor).reshape(L, H * dv), ease

        want, ease = expect(mask)
        if window and window + 2 < L and dtype == torch.float32:       # the edges show: one token more or less is far off
            for other in ({"size": window + 1, "keep_first": keep}, {"size": window, "keep_first": keep + 1}):
                if keep < L - window - 2:
                    assert (expect(other)[0] - want).abs().max() > 30 * tol * want.std(), other
        pages = -(-L // bs)
        table = list(range(pages, 0, -1))
        kc, vc = torch.zeros(1 + pages, G, bs, maps * dk, dtype=dtype), torch.zeros(1 + pages, G, bs, dv, dtype=dtype)
        for p in range(L):
            kc[table[p // bs], :, p % bs], vc[table[p // bs], :, p % bs] = k[p].reshape(G, -1).to(dtype), v[p].to(dtype)
        kc, vc = kc.to(device), vc.to(device)
        for cuts in ([L], [33, L - 33], [L - 40] + [1] * 40, [15, 2, 2, 30, 1, 64, L - 114]):
            at, rows = 0, []
            for n in cuts:
                batch = BatchInput.build([[0] * n], [at], [table], bs, device)
                qq = q[at:at + n].reshape(n, -1).to(dtype).to(device)
                rows.append(ops.attention_bias(_pad_maps(qq, H, maps, dk, batch, kc, vc, scale), kc, vc, batch, H, G, dk, dv, scale, None,
                                               out_dtype=dtype, window=window, keep_first=keep, softcap=cap,
                                               diff=(lam, eps, factor) if maps == 2 else None))
                at += n
            close(torch.cat(rows), want, tol, ease)


def test_attention_into_columns_of_a_wider_row(device="cpu", dtype=torch.float32, tol=1e-4):
    """The result lands in a column range of another product's operand and nothing beside it is touched; several sequences of
    unequal lengths, some of them single tokens, in one batch."""
    torch.manual_seed(5)
    H, G, dk, dv, bs, window, keep = 4, 2, 8, 16, 16, 11, 3
    lens, ctx = [30, 1, 2, 17], [0, 40, 63, 14]
    tabs, nb = _pages(bs, [c + n for c, n in zip(ctx, lens)])
    batch = BatchInput.build([[0] * n for n in lens], ctx, tabs, bs, device)
    kc, vc = torch.zeros(nb, G, bs, 2 * dk, dtype=dtype), torch.zeros(nb, G, bs, dv, dtype=dtype)
    qs, want = [], []
    for n, c, tab in zip(lens, ctx, tabs):
        L = n + c
        q, k, v = (torch.randn(L, *s).to(dtype).double() for s in ((H, 2, dk), (G, 2, dk), (G, dv)))
        for p in range(L):
            kc[tab[p // bs], :, p % bs], vc[tab[p // bs], :, p % bs] = k[p].reshape(G, -1).to(dtype), v[p].to(dtype)
        a = [oracle.softmax_attention(q[:, :, m], k[:, :, m].repeat_interleave(2, 1), v.repeat_interleave(2, 1), 0.5,
                                      {"size": window, "keep_first": keep}, 5.0) for m in (0, 1)]
        qs.append(q[c:].reshape(n, -1))
        want.append((oracle.rms_div(a[0] - 0.3 * a[1], 1e-6) * 0.5).reshape(L, -1)[c:])
    T = sum(lens)
    for lead, width in ((0, H * dv + 24), (0, H * dv + 5)):      # rows with and without 16-byte alignment
        buf = torch.full((T, width), 9.0, dtype=dtype, device=device)
        ops.attention_bias(torch.cat(qs).to(dtype).to(device), kc.to(device), vc.to(device), batch, H, G, dk, dv, 0.5, None, out_dtype=dtype,
                           window=window, keep_first=keep, softcap=5.0, diff=(0.3, 1e-6, 0.5), out=buf[:, lead:lead + H * dv])
        close(buf[:, lead:lead + H * dv], torch.cat(want), tol)
        assert bool((buf[:, lead + H * dv:] == 9.0).all())


@pytest.mark.parametrize("T,W,F", [(5, 32, 24), (130, 50, 13), (1, 64, 128)])
def test_gated_product(T, W, F, device="cpu", dtype=torch.float32, tol=1e-5):
    torch.manual_seed(T)
    from llmss_b200.models.mixers import GatedFFN

    h, g, u, dn = torch.randn(T, W), torch.randn(F, W) * W ** -0.5 * 2, torch.randn(F, W) * W ** -0.5, torch.randn(W, F) * F ** -0.5
    h, g, u, dn = (x.to(dtype) for x in (h, g, u, dn))
    f = GatedFFN()
    f.set_weights(g.to(device), u.to(device), dn.to(device))
    p = {"gate": g.double(), "up": u.double(), "down": dn.double()}
    close(f.forward(h.to(device)), oracle.gated_ffn(h.double(), p, ""), tol)
    buf = torch.zeros(T, F + 9, dtype=dtype, device=device)
    f.hidden(h.to(device), out=buf[:, 9:])
    close(buf[:, 9:], oracle.gelu_tanh(h.double() @ g.double().T) * (h.double() @ u.double().T), tol)
    assert float(buf[:, :9].float().abs().sum()) == 0.0


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
def test_whole_prompt_and_residual_stream(tmp_path, name, device="cpu", dtype=torch.float32, tol=TOL):
    cfg, W, eng = build(tmp_path, name, device, dtype)
    toks = tokens_for(cfg, 75, 1)
    want, layers = oracle.forward(toks, cfg, W, True)
    got = residual_stream(eng, toks)
    assert len(got) == len(layers)
    for i, g in enumerate(got):
        close(g, layers[i], tol * (1 + i))
    close(eng.feed([("a", toks, list(range(len(toks))))], ["a"]), want, tol * 2)


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

    def each(c, f):
        for L in c["layers"]:
            f(L["mixer"])

    def window_longer(c, w):
        each(c, lambda m: m["mask"].update(size=m["mask"]["size"] + 1))

    def first_fewer(c, w):
        each(c, lambda m: m["mask"].update(keep_first=max(0, m["mask"].get("keep_first", 0) - 1)))

    def no_cap(c, w):
        each(c, lambda m: m.pop("softcap", None))

    def no_scaling(c, w):
        each(c, lambda m: m["rot"].pop("scaling", None))

    def no_lambda(c, w):
        for k in w:
            if k.endswith(("lq1", "lq2")):
                w[k] *= 0.0

    def no_bias(c, w):
        for k in list(w):
            if k.endswith(".b"):
                del w[k]

    def no_qk_norm(c, w):
        for k in list(w):
            if k.endswith((".q.norm", ".k.norm")):
                del w[k]

    def own_pages(c, w):
        c["layers"][3]["mixer"].pop("kv_from")
        for s in ("k", "k.b", "v", "v.b", "k.norm"):
            w[f"l3.mix.{s}"] = w[f"l0.mix.{s}"].flip(0)

    for change in (window_longer, first_fewer, no_cap, no_scaling, no_lambda, no_bias, no_qk_norm, own_pages):
        assert moved(change) > 20 * TOL, change.__name__


# ----------------------------------------------------------------------------- decoding, portions, batches
@pytest.mark.parametrize("name", ["mixed", "edges", "odd"])
def test_decode_token_by_token_and_portions(tmp_path, name, device="cpu", dtype=torch.float32, tol=TOL):
    """Prefill against token-by-token decoding, and portions down to two tokens that cut pages and windows."""
    cfg, W, eng = build(tmp_path, name, device, dtype)
    toks = tokens_for(cfg, 70, 2)
    want = want_logits(toks, cfg, W)
    for sizes in ([1], [2], [3, 1, 2, 7, 1, 1, 16, 5], [15, 1, 1, 17, 2], [33, 31, 1], [64, 1]):
        close(feed_in_portions(eng, "s", toks, sizes), want, tol * 2)


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
        close(torch.cat(got[k]), want[k], tol * 2)


def test_pages_are_used_again(tmp_path, device="cpu", dtype=torch.float32, tol=TOL):
    """A pool of a few pages serves six requests one after another and overlapping; what a page held before must not show.  A
    request beyond the pool, and one live request too many, are errors."""
    cfg, W, eng = build(tmp_path, "mixed", device, dtype, max_batch=2)
    bs = eng.runner.block_size
    _, _, small = build(tmp_path / "p", "mixed", device, dtype, max_batch=2, pool_tokens=4 * bs)
    for e in (eng, small):
        lens = [bs + 3, 2 * bs, 5, bs - 1, bs + 1, 7]
        reqs = [tokens_for(cfg, n, 30 + i) for i, n in enumerate(lens)]
        want = [want_logits(t, cfg, W) for t in reqs]
        a = e.feed([(0, reqs[0][:5], list(range(5))), (1, reqs[1], list(range(lens[1])))], [1])
        close(a[5:], want[1], tol * 2)
        b = e.feed([(0, reqs[0][5:], list(range(lens[0] - 5))), (2, reqs[2], list(range(5)))], [0, 2])
        close(torch.cat([a[:5], b[:lens[0] - 5]]), want[0], tol * 2)
        close(b[lens[0] - 5:], want[2], tol * 2)
        for i in (3, 4, 5):
            close(feed_in_portions(e, i, reqs[i], [4, 1]), want[i], tol * 2)
        assert e.runner.alloc.num_free == e.runner.alloc.num_blocks - 1
    eng.feed([("x", [1, 2], []), ("y", [3], [])])
    with pytest.raises(RuntimeError):
        eng.feed([("z", [4], [])])
    eng.feed([], ["x", "y"])
    with pytest.raises((MemoryError, ValueError)):
        small.feed([("big", tokens_for(cfg, 5 * bs, 1), [])])


def steep_config():
    """Attention decided by single keys (a score scale several times the usual one): a key lost at a page border or a window's
    edge, a position rotated wrongly far from the start or a page read for the wrong layer changes the result at once."""
    return rofulorn_config(32, 71, [
        pln(heads=2, kv_heads=1, dim=8, vdim=8, scale=2.5, base=50.0, window=65),
        dif(heads=2, kv_heads=1, dim=8, vdim=12, scale=2.0, base=50.0, window=16, keep_first=17, softcap=25.0),
        pln(heads=4, kv_heads=4, dim=8, vdim=8, scale=2.5, rot_dims=4, base=20.0, window=32, mlp={"ff": 24}),
        dif(heads=2, kv_heads=1, dim=8, vdim=12, scale=2.0, base=50.0, window=63, keep_first=1, softcap=25.0, kv_from=1)], embed_scale=3.0)


def test_steep_attention_far_back_and_over_page_borders(tmp_path, device="cpu", dtype=torch.float32, tol=TOL):
    cfg, W, eng = build(tmp_path, steep_config(), device, dtype)
    toks = tokens_for(cfg, 150, 4)
    want = want_logits(toks, cfg, W)
    close(feed_in_portions(eng, "w", toks, [150]), want, tol * 3)
    close(feed_in_portions(eng, "p", toks, [31, 2, 36, 1, 1, 59, 2, 1]), want, tol * 3)
    close(feed_in_portions(eng, "d", toks, [100, 1]), want, tol * 3)
    # the first tokens reach the last ones through the kept keys: another first token changes them
    other = want_logits([(toks[0] + 1) % cfg["vocab"]] + toks[1:], cfg, W)
    assert (other[-5:] - want[-5:]).abs().max() > 100 * tol * want.std()


def test_first_tokens(tmp_path, device="cpu", dtype=torch.float32, tol=TOL):
    """One-token and two-token requests, and the first tokens one by one, in pages that another request has just left."""
    cfg, W, eng = build(tmp_path, "mixed", device, dtype)
    feed_in_portions(eng, "warm", tokens_for(cfg, 40, 7), [40])          # leaves keys behind
    for n in (1, 2, 3, 6):
        toks = tokens_for(cfg, n, 50 + n)
        want = want_logits(toks, cfg, W)
        close(feed_in_portions(eng, "f", toks, [n]), want, tol * 2)
        close(feed_in_portions(eng, "g", toks, [1]), want, tol * 2)


def test_long_decoding(tmp_path, device="cpu", dtype=torch.float32, tol=TOL):
    cfg, W, eng = build(tmp_path, "mixed", device, dtype)
    toks = tokens_for(cfg, 160, 8)
    close(feed_in_portions(eng, "l", toks, [12, 1]), want_logits(toks, cfg, W), tol * 4)


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
            lg = want_logits(p + g, cfg, W)[len(p) - 1:-1]
            for row, tok in zip(lg, g):
                assert row[tok] >= row.max() - 0.15 * lg.std()
    if device == "cpu":
        path = tmp_path / "ckpt0"
        r = subprocess.run([sys.executable, str(ROOT / "generate.py"), "--pretrained_model_path", str(path), "--prompt_ids",
                            " ".join(map(str, prompts[0])), "--max_new_tokens", "5", "--is_greedy", "--use_cache"],
                           capture_output=True, text=True, timeout=300, cwd=str(ROOT), env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
        assert r.returncode == 0, r.stderr[-2000:]
        assert " ".join(map(str, got[0][:5])) in r.stdout.replace(",", " ").replace("  ", " "), r.stdout[-1000:]


def test_shared_prompt_prefix_and_prompt_rounds(tmp_path, device="cpu", dtype=torch.float32):
    """The cache holds pages only, so a later prompt may continue on the pages of an earlier one with the same start; and
    prompts may be processed in rounds.  Eviction from the front is refused: kept first tokens are found by their place."""
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
    _, _, e = build(tmp_path / "plain", "plain", device, dtype, sliding_window=True)
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
    assert model.core.num_parameters_local() == sum(v.numel() for k, v in W.items() if not k.split(".")[-1].startswith(("lq", "lk")))
    seqs = [tokens_for(cfg, 30, 3), tokens_for(cfg, 30, 4)]
    ids = torch.tensor(seqs)
    out = model(ids[:, :21], use_cache=True)
    rows = [out.logits]
    for t in range(21, 30):
        out = model(ids[:, t:t + 1], past_key_values=out.past_key_values, use_cache=True)
        rows.append(out.logits)
    got = torch.cat(rows, dim=1)
    for b in (0, 1):
        close(got[b], want_logits(seqs[b], cfg, W), tol * 2)


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


def test_unknown_kinds_and_bad_lenders_are_refused():
    from llmss_b200.models.rofulorn import rofulorn_spec

    def bad(change):
        cfg = json.loads(json.dumps(CONFIGS["mixed"]))
        change(cfg["layers"])
        with pytest.raises(ValueError):
            rofulorn_spec(cfg)

    bad(lambda L: L[0].update(type="other"))
    bad(lambda L: L[0]["mlp"].update(kind="other"))
    bad(lambda L: L[3]["mixer"].update(kv_from=3))
    bad(lambda L: L[5]["mixer"].update(kv_from=3))       # a borrower lends nothing
    bad(lambda L: L[3]["mixer"].update(kv_from=2))       # other sizes
    bad(lambda L: L[3]["mixer"].update(kv_from=1))       # one map against two
