"""Fipavik: a decoder-only design whose layers run the mixer and a mixture of experts side by side on one normed input, with two
kinds of local attention that have a sink.

    x = embed[token]                                                             (32-bit from here on)
    layer:   h = layer_norm(x) * norm1 + norm1.b ;  x <- x + residual_mult * (mixer(h) + experts(h))     (experts may be absent)
    mixers:  "latent_attention" -- per-head keys and values from a normed latent, one rotated key part shared by the heads, a sliding
                                   window                                                    -> blocks.RotaryLatentAttention (span form)
             "attention"        -- grouped heads, normed q / k, a chunked mask, values mixed with those of the first mixing layer
                                                                                             -> mixers.RotaryAttention
    experts: the chosen W_down (silu(W_gate h) * (W_up h)), weighted by the softmax over the chosen router logits, plus one that
             every token takes                                                               -> blocks.RoutedExperts, mixers.GatedFFN
    logits = embed (layer_norm(x) * final.norm + final.norm.b)                   the embedding table is the output matrix

config.json keys: architecture, vocab, width, norm.eps, residual_mult, layers[i].{type, mixer{heads, dim, vdim, scale, rot{base, dims},
mask{size}, and kv_heads, v_mix | kv_rank, rot_dim}, mlp{kind, expert.ff, router{experts, top}, shared.ff} | null}.
Tensor names: embed, final.norm, l<i>.norm1 (each with .b), l<i>.mix.* (listed with each loader below),
l<i>.mlp.{router, router.b, e<j>.gate / up / down, shared.gate / up / down}.

The model is a graph over the framework's ops.  What a sequence carries between steps are pages -- keys and values of the attention
layers, latent rows of the others (engine.kv_cache.HybridCache without state slots) --, so prompt prefixes can be shared.  Runner,
block allocator, batching and sampler drive it like the other families.  It runs unsharded (TP = 1).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional

import torch
from torch import nn

from .. import ops
from ..engine.batch import BatchInput
from ..engine.kv_cache import HybridCache
from ..ops import ACT_SILU, NORM_LAYER
from ..parallel.comm import comm_for
from ..utils.tracing import trace
from .blocks import RotaryLatentAttention, RoutedExperts
from .decoder import interleave_gate_up
from .mixers import GatedFFN, LayerCacheView, ParallelBlock, RotaryAttention

MIXER_TYPES = ("latent_attention", "attention")
FFN_KINDS = ("moe",)
F32 = torch.float32


@dataclass
class FipavikSpec:
    hidden: int
    vocab: int
    eps: float
    residual_mult: float
    layers: List[dict] = field(default_factory=list)      # the config's layer entries, checked
    model_type: str = "fipavik"
    max_pos: int = 1 << 30       # rotary positions: no limit of its own
    default_seq_len: int = 4096  # block-table width when the caller names neither a length nor a pool
    learned_pos: bool = False

    @property
    def n_layers(self) -> int:
        return len(self.layers)


def _mixes(lc: dict) -> bool:
    return lc["type"] == "attention" and bool(lc["mixer"].get("v_mix"))


def fipavik_spec(config) -> FipavikSpec:
    c = config.raw if hasattr(config, "raw") else dict(config)
    layers = list(c["layers"])
    mixing = None                # the first layer that mixes values
    for i, lc in enumerate(layers):
        if lc["type"] not in MIXER_TYPES:
            raise ValueError(f"fipavik: layer {i} has unknown mixer type {lc['type']!r}; have {MIXER_TYPES}")
        f = lc.get("mlp")
        if f is not None and f.get("kind", "moe") not in FFN_KINDS:
            raise ValueError(f"fipavik: layer {i} has unknown feed-forward kind {f.get('kind')!r}; have {FFN_KINDS}")
        if _mixes(lc):
            m = lc["mixer"]
            mixing = m if mixing is None else mixing
            if int(m["kv_heads"]) * int(m["vdim"]) != int(mixing["kv_heads"]) * int(mixing["vdim"]):
                raise ValueError(f"fipavik: layer {i} mixes its values with a layer whose value heads or sizes differ")
    return FipavikSpec(int(c["width"]), int(c["vocab"]), float(c["norm"]["eps"]), float(c.get("residual_mult", 1.0)), layers)


def _build_mixer(lc: dict, width: int, eps: float, v_mix: Optional[str]):
    m = lc["mixer"]
    d, latent = int(m["dim"]), lc["type"] == "latent_attention"
    span = int(m["rot_dim"]) if latent else d              # the channels the rotation may use
    rot, size = m.get("rot"), int((m.get("mask") or {}).get("size") or 0)
    freq, mag = (ops.rotary_frequencies(int(rot.get("dims", span)), float(rot["base"])) if rot
                 else (torch.zeros(0, dtype=torch.float64), 1.0))
    if 2 * freq.numel() > span:
        raise ValueError(f"fipavik: {lc['type']} rotates {2 * freq.numel()} channels of {span}")
    if latent:
        return RotaryLatentAttention(int(m["heads"]), d, span, int(m["vdim"]), int(m["kv_rank"]), 0, float(m.get("scale", (d + span) ** -0.5)),
                                     eps, freq, mag, interleaved=False, gated=False, span=True, window=size)
    return RotaryAttention(width, int(m["heads"]), int(m["kv_heads"]), d, int(m["vdim"]), float(m.get("scale", d ** -0.5)), eps, freq, mag,
                           interleaved=False, chunk=size, v_mix=v_mix)


def _build_experts(f: Optional[dict]):
    """(the expert every token takes, the routed ones) of a layer's ``mlp`` entry."""
    if f is None:
        return None, None
    r = f["router"]
    return (GatedFFN(ACT_SILU) if f.get("shared") is not None else None,
            RoutedExperts(int(r["experts"]), int(r["top"]), 1, 1, 1.0, int(f["expert"]["ff"]), act=ACT_SILU, gated=True))


class FipavikLM(nn.Module):
    """The decoder core the engine drives (same surface as DecoderLM: forward / forward_hidden / logits / make_cache)."""

    def __init__(self, spec: FipavikSpec, process_group, device, dtype):
        super().__init__()
        self.spec = spec
        self.comm = comm_for(process_group, device)
        self.tp, self.rank = self.comm.size, self.comm.rank
        if self.tp != 1:
            raise NotImplementedError("fipavik runs unsharded: start it with one rank")
        self.device, self.dtype = torch.device(device), dtype
        self.vocab_blk = spec.vocab
        self.layers: List[ParallelBlock] = []
        mixed = False
        for lc in spec.layers:
            v_mix = None
            if _mixes(lc):
                v_mix, mixed = ("later" if mixed else "first"), True
            self.layers.append(ParallelBlock(_build_mixer(lc, spec.hidden, spec.eps, v_mix), *_build_experts(lc.get("mlp"))))
        self.norms: List[tuple] = []             # (weight, bias) of every layer's norm, then of the final one
        self.wte = None
        # a chunk is counted from the sequence's start: keys are found by their place in it, so no eviction from the front
        self.needs_first_pages = any(getattr(L.mixer, "chunk", 0) > 0 for L in self.layers)

    # ------------------------------------------------------------------ cache
    def default_block_size(self) -> int:
        return 64 if self.device.type == "cuda" else 16

    def make_cache(self, num_blocks: int, block_size: int, max_seqs: Optional[int] = None) -> HybridCache:
        kv, latents = {}, {}
        for i, L in enumerate(self.layers):
            if isinstance(L.mixer, RotaryLatentAttention):
                latents[i] = L.mixer.choose_width(self.device, self.dtype)
            else:
                kv[i] = L.mixer.kv_shape()
        return HybridCache(kv, {}, num_blocks, block_size, max_seqs or 1, self.dtype, self.device, latents=latents)

    def num_parameters_local(self) -> int:
        ts = [self.wte] + [t for wb in self.norms for t in wb]
        for L in self.layers:
            ts += L.weights()
        return sum(t.numel() for t in ts if t is not None)

    def finalize(self):
        for L in self.layers:
            if isinstance(L.mixer, RotaryLatentAttention):
                L.mixer.finalize()
            L.finalize()
        return self

    # ------------------------------------------------------------------ forward
    def forward_hidden(self, batch: BatchInput, kv: HybridCache, taps: Optional[list] = None) -> torch.Tensor:
        """Final-normed hidden states [T, width] of every packed token.  ``taps``: a list that receives the 32-bit
        residual stream that leaves every layer (debugging / tests)."""
        s, dt = self.spec, self.dtype
        with trace("embed"):
            x = ops.embed(batch.tokens, self.wte, out_dtype=F32)
        y, carry = None, {}      # the last layer's output, not yet added to the residual; what a layer leaves for later ones
        for i, L in enumerate(self.layers):
            with trace("residual_norm"):
                h, x = ops.residual_norm(x, y, *self.norms[i], s.eps, NORM_LAYER, out_dtype=dt, mult=s.residual_mult)
            if taps is not None and i > 0:
                taps.append(x.clone())
            y = L.forward(h, batch, LayerCacheView(kv, i), dt, carry)
        with trace("final_norm"):
            h, x = ops.residual_norm(x, y, *self.norms[-1], s.eps, NORM_LAYER, out_dtype=dt, mult=s.residual_mult)
        if taps is not None:
            taps.append(x.clone())
        return h

    def logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        with trace("lm_head"):
            return ops.linear(hidden_rows, self.wte, out_dtype=torch.float32)

    local_logits = logits

    def forward(self, batch: BatchInput, kv, last_only: bool = True, gather_logits: bool = True) -> torch.Tensor:
        h = self.forward_hidden(batch, kv)
        if last_only:
            h = h.index_select(0, batch.last_idx)
        return self.logits(h)


# ---------------------------------------------------------------------------------------------------- weights
def _f32(t):
    """Small per-channel parameters are kept in 32-bit whatever the compute type (the checkpoint's values are exact in it)."""
    return t.float().contiguous()


def _maybe(w, name):
    return _f32(w.get_tensor(name)) if w.has(name) else None


def _load_latent(mx: RotaryLatentAttention, w, p):
    """<p>.q [heads*(dim+rot_dim), W]; <p>.dkv [kv_rank+rot_dim, W] + .dkv.norm [kv_rank]; <p>.uk [heads*dim, kv_rank]; <p>.uv [heads*vdim,
    kv_rank]; <p>.sink [heads]; <p>.o [W, heads*vdim]."""
    get = w.get_tensor
    mx.w_q, mx.w_dkv, mx.cn_w = get(f"{p}.q"), get(f"{p}.dkv"), _f32(get(f"{p}.dkv.norm"))
    mx.w_uk, mx.w_uv, mx.w_o = get(f"{p}.uk").contiguous(), get(f"{p}.uv").contiguous(), get(f"{p}.o").contiguous()
    mx.sinks = _maybe(w, f"{p}.sink")
    rows = (mx.heads * (mx.dim + mx.rot), mx.rank + mx.rot, mx.heads * mx.dim, mx.heads * mx.vdim)
    if tuple(t.shape[0] for t in (mx.w_q, mx.w_dkv, mx.w_uk, mx.w_uv)) != rows or mx.w_o.shape[1] != mx.n_out:
        raise ValueError(f"{p}: projections do not fit the configured heads")


def _load_attention(mx: RotaryAttention, w, p):
    """<p>.q [heads*dim, W]; <p>.k [kv_heads*dim, W]; <p>.v [kv_heads*vdim, W]; <p>.q.norm / .k.norm [dim]; <p>.vmix (one number, value-mixing
    layers); <p>.sink [heads]; <p>.o [W, heads*vdim]."""
    get = w.get_tensor
    lam = float(get(f"{p}.vmix").float()) if mx.v_mix == "later" else 0.0
    mx.set_weights(get(f"{p}.q"), get(f"{p}.k"), get(f"{p}.v"), get(f"{p}.o"), q_norm=_maybe(w, f"{p}.q.norm"),
                   k_norm=_maybe(w, f"{p}.k.norm"), sinks=_maybe(w, f"{p}.sink"), v_lam=lam)
    if mx.w_in.shape[0] != (mx.heads + mx.kv_heads) * mx.dim + mx.kv_heads * mx.vdim or mx.w_o.shape[1] != mx.n_out:
        raise ValueError(f"{p}: projections do not fit the configured heads")


def _load_experts(L: ParallelBlock, w, p):
    get, ex = w.get_tensor, L.experts
    ex.w_router = get(f"{p}.router").contiguous()
    ex.b_router = get(f"{p}.router.b") if w.has(f"{p}.router.b") else None
    ex.w_up = torch.stack([interleave_gate_up(get(f"{p}.e{e}.gate"), get(f"{p}.e{e}.up")) for e in range(ex.experts)])   # [E, 2 F, W]
    ex.w_down = torch.cat([get(f"{p}.e{e}.down") for e in range(ex.experts)], dim=1)                                    # [W, E * F]
    if L.ffn is not None:
        L.ffn.set_weights(get(f"{p}.shared.gate"), get(f"{p}.shared.up"), get(f"{p}.shared.down"))


def load_fipavik(m: FipavikLM, w):
    get = w.get_tensor
    m.wte = get("embed").contiguous()
    for i, L in enumerate(m.layers):
        p = f"l{i}"
        m.norms.append((_f32(get(f"{p}.norm1")), _f32(get(f"{p}.norm1.b"))))
        (_load_latent if isinstance(L.mixer, RotaryLatentAttention) else _load_attention)(L.mixer, w, f"{p}.mix")
        if L.experts is not None:
            _load_experts(L, w, f"{p}.mlp")
    m.norms.append((_f32(get("final.norm")), _f32(get("final.norm.b"))))
