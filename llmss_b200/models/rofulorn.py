"""Rofulorn: a decoder-only design whose layers run the mixer and the feed-forward side by side on one normed input, with two
kinds of windowed rotary attention.

    x = embed[token] * scale                                                     (32-bit from here on)
    layer:   h = layer_norm(x) * norm1 ;  x <- x + (mixer(h) + ffn(h))           (a layer may have no feed-forward)
    mixers:  "attention"   -- differential: two query / key maps per head over one value, normed q / k, biases, soft-capped scores,
                              a window that keeps the first tokens; optionally ``kv_from`` an earlier layer
             "attention_2" -- plain, a window                                    both -> mixers.RotaryAttention
    ffn:     W_down (gelu_tanh(W_gate h) * (W_up h))                             -> mixers.GatedFFN
    logits = head (layer_norm(x) * final.norm)

config.json keys: architecture, vocab, width, norm.eps, embedding.scale, layers[i].{type, mixer{heads, kv_heads, dim, vdim,
scale, rot{base, dims, scaling{factor, low, high, original}}, mask{size, keep_first}, softcap, diff, kv_from}, mlp{kind, ff} | null}.
Tensor names: embed, head, final.norm, l<i>.norm1, l<i>.mix.*, l<i>.mlp.{gate, up, down} (mixer tensors: ``_load_mixer``).

The model is a graph over the framework's ops.  All a sequence carries between steps are the K / V pages of the layers with
projections of their own (engine.kv_cache.HybridCache without state slots), so prompt prefixes can be shared.  Runner, block
allocator, batching and sampler drive it like the other families.  It runs unsharded (TP = 1).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional

import torch
from torch import nn

from .. import ops
from ..engine.batch import BatchInput
from ..engine.kv_cache import HybridCache
from ..ops import ACT_GELU_TANH, NORM_LAYER
from ..parallel.comm import comm_for
from ..utils.tracing import trace
from .mixers import GatedFFN, LayerCacheView, ParallelBlock, RotaryAttention

MIXER_TYPES = ("attention", "attention_2")
FFN_KINDS = ("dense",)
F32 = torch.float32


@dataclass
class RofulornSpec:
    hidden: int
    vocab: int
    eps: float
    embed_scale: float
    layers: List[dict] = field(default_factory=list)      # the config's layer entries, checked
    model_type: str = "rofulorn"
    max_pos: int = 1 << 30       # rotary positions: no limit of its own
    default_seq_len: int = 4096  # block-table width when the caller names neither a length nor a pool
    learned_pos: bool = False

    @property
    def n_layers(self) -> int:
        return len(self.layers)


def _maps(m: dict) -> int:
    return 1 if m.get("diff") is None else 2


def rofulorn_spec(config) -> RofulornSpec:
    c = config.raw if hasattr(config, "raw") else dict(config)
    layers = list(c["layers"])
    for i, lc in enumerate(layers):
        if lc["type"] not in MIXER_TYPES:
            raise ValueError(f"rofulorn: layer {i} has unknown mixer type {lc['type']!r}; have {MIXER_TYPES}")
        f = lc.get("mlp")
        if f is not None and f.get("kind", "dense") not in FFN_KINDS:
            raise ValueError(f"rofulorn: layer {i} has unknown feed-forward kind {f.get('kind')!r}; have {FFN_KINDS}")
        m = lc["mixer"]
        j = m.get("kv_from")
        if j is not None:
            if not (0 <= int(j) < i) or layers[int(j)]["mixer"].get("kv_from") is not None:
                raise ValueError(f"rofulorn: layer {i} takes keys / values from layer {j}, which is not an earlier layer with "
                                 "projections of its own")
            o = layers[int(j)]["mixer"]
            if (int(o["kv_heads"]), int(o["dim"]), int(o["vdim"]), _maps(o)) != (int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), _maps(m)):
                raise ValueError(f"rofulorn: layer {i} and its lender {j} differ in key / value heads, sizes or maps")
    return RofulornSpec(int(c["width"]), int(c["vocab"]), float(c["norm"]["eps"]), float((c.get("embedding") or {}).get("scale", 1.0)), layers)


def _build_mixer(m: dict, width: int, eps: float) -> RotaryAttention:
    d = int(m["dim"])
    rot, mask, kv_from = m.get("rot"), m.get("mask") or {}, m.get("kv_from")
    freq, mag = (ops.rotary_frequencies(int(rot.get("dims", d)), float(rot["base"]), rot.get("scaling")) if rot
                 else (torch.zeros(0, dtype=torch.float64), 1.0))
    return RotaryAttention(width, int(m["heads"]), int(m["kv_heads"]), d, int(m["vdim"]), float(m.get("scale", d ** -0.5)), eps, freq, mag,
                           interleaved=True, window=mask.get("size"), keep_first=mask.get("keep_first"), softcap=m.get("softcap"),
                           diff=None if m.get("diff") is None else float(m["diff"]), kv_from=None if kv_from is None else int(kv_from))


class RofulornLM(nn.Module):
    """The decoder core the engine drives (same surface as DecoderLM: forward / forward_hidden / logits / make_cache)."""

    def __init__(self, spec: RofulornSpec, process_group, device, dtype):
        super().__init__()
        self.spec = spec
        self.comm = comm_for(process_group, device)
        self.tp, self.rank = self.comm.size, self.comm.rank
        if self.tp != 1:
            raise NotImplementedError("rofulorn runs unsharded: start it with one rank")
        self.device, self.dtype = torch.device(device), dtype
        self.vocab_blk = spec.vocab
        self.layers: List[ParallelBlock] = []
        for lc in spec.layers:
            self.layers.append(ParallelBlock(_build_mixer(lc["mixer"], spec.hidden, spec.eps),
                                             GatedFFN(ACT_GELU_TANH) if lc.get("mlp") is not None else None))
        self.norms: List[torch.Tensor] = []      # norm1 of every layer, then final.norm
        self.wte = self.w_head = None
        # a window that keeps the first tokens addresses keys by their place in the sequence: no eviction from the front
        self.needs_first_pages = any(L.mixer.keep_first > 0 for L in self.layers)

    # ------------------------------------------------------------------ cache
    def default_block_size(self) -> int:
        return 64 if self.device.type == "cuda" else 16

    def make_cache(self, num_blocks: int, block_size: int, max_seqs: Optional[int] = None) -> HybridCache:
        kv = {i: L.mixer.kv_shape() for i, L in enumerate(self.layers) if L.mixer.own_kv}
        return HybridCache(kv, {}, num_blocks, block_size, max_seqs or 1, self.dtype, self.device)

    def num_parameters_local(self) -> int:
        ts = [self.wte, self.w_head] + self.norms
        for L in self.layers:
            ts += L.weights()
        return sum(t.numel() for t in ts if t is not None)

    def finalize(self):
        for L in self.layers:
            L.finalize()
        return self

    # ------------------------------------------------------------------ forward
    def forward_hidden(self, batch: BatchInput, kv: HybridCache, taps: Optional[list] = None) -> torch.Tensor:
        """Final-normed hidden states [T, width] of every packed token.  ``taps``: a list that receives the 32-bit
        residual stream that leaves every layer (debugging / tests)."""
        s, dt = self.spec, self.dtype
        with trace("embed"):
            x = ops.embed(batch.tokens, self.wte, out_dtype=F32, scale=s.embed_scale)
        y = None                 # the last layer's output, not yet added to the residual
        for i, L in enumerate(self.layers):
            with trace("residual_norm"):
                h, x = ops.residual_norm(x, y, self.norms[i], None, s.eps, NORM_LAYER, out_dtype=dt)
            if taps is not None and i > 0:
                taps.append(x.clone())
            y = L.forward(h, batch, LayerCacheView(kv, i, pages_key=L.mixer.kv_from), dt)
        with trace("final_norm"):
            h, x = ops.residual_norm(x, y, self.norms[-1], None, s.eps, NORM_LAYER, out_dtype=dt)
        if taps is not None:
            taps.append(x.clone())
        return h

    def logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        with trace("lm_head"):
            return ops.linear(hidden_rows, self.w_head, out_dtype=torch.float32)

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


def _load_mixer(mx: RotaryAttention, w, p):
    """<p>.q [heads*maps*dim, W]; <p>.k [kv_heads*maps*dim, W] and <p>.v [kv_heads*vdim, W] unless the layer borrows them; <p>.o
    [W, heads*vdim]; where present a bias <name>.b for each, <p>.q.norm / .k.norm [dim]; differential: <p>.lq1 / .lk1 / .lq2 / .lk2
    [dim]."""
    get = w.get_tensor

    def maybe(name, f32=False):
        if not w.has(f"{p}.{name}"):
            return None
        return _f32(get(f"{p}.{name}")) if f32 else get(f"{p}.{name}")

    own = mx.own_kv
    mx.set_weights(get(f"{p}.q"), get(f"{p}.k") if own else None, get(f"{p}.v") if own else None, get(f"{p}.o"),
                   bq=maybe("q.b"), bk=maybe("k.b") if own else None, bv=maybe("v.b") if own else None, b_o=maybe("o.b"),
                   q_norm=maybe("q.norm", True), k_norm=maybe("k.norm", True) if own else None,
                   lam_vectors=tuple(_f32(get(f"{p}.{n}")) for n in ("lq1", "lk1", "lq2", "lk2")) if mx.diff is not None else None)
    n = (mx.heads + (mx.kv_heads if own else 0)) * mx.maps * mx.dim + (mx.kv_heads * mx.vdim if own else 0)
    if mx.w_in.shape[0] != n or mx.w_o.shape[1] != mx.n_out:
        raise ValueError(f"{p}: projections of {mx.w_in.shape[0]} rows and {mx.w_o.shape[1]} output columns do not fit the configured heads")


def load_rofulorn(m: RofulornLM, w):
    get = w.get_tensor
    m.wte, m.w_head = get("embed").contiguous(), get("head").contiguous()
    for i, L in enumerate(m.layers):
        p = f"l{i}"
        m.norms.append(_f32(get(f"{p}.norm1")))
        _load_mixer(L.mixer, w, f"{p}.mix")
        if L.ffn is not None:
            L.ffn.set_weights(get(f"{p}.mlp.gate"), get(f"{p}.mlp.up"), get(f"{p}.mlp.down"))
    m.norms.append(_f32(get("final.norm")))
