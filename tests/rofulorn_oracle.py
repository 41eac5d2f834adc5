"""Plain float64 implementation of the Rofulorn design: one function per mechanism, whole sequences, no cache, no state
objects, nothing imported from the package.  ``p`` maps tensor names to float64 tensors, ``cfg`` is the parsed config.json.
The tests compare the framework against these functions."""
import math

import torch

F64 = torch.float64


# ----------------------------------------------------------------------------------------------- norms
def layer_norm(x, w, eps):
    """Mean taken off, divided by the root of the mean squared deviation + eps, a weight and no bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms_div(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# ----------------------------------------------------------------------------------------------- rotary positions
def rotary_frequencies(rot):
    """One frequency per pair for a ``rot`` entry {base, dims, optionally scaling{factor, low, high, original}}: short
    wavelengths keep their frequency, long ones are slowed down by the factor, those between are blended."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            wavelength = 2.0 * math.pi / f
            factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            if wavelength > original / low:
                f = f / factor
            elif wavelength >= original / high:
                s = (original / wavelength - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate(x, positions, rot):
    """x [T, heads, d]: the neighbours (2i, 2i + 1) of the first rot.dims channels of every head turn by position * f_i."""
    if not rot:
        return x
    out = x.clone()
    for i, f in enumerate(rotary_frequencies(rot)):
        a = positions.to(F64) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


# ----------------------------------------------------------------------------------------------- softmax attention
def visible(T, mask):
    """[T, T] booleans, row = query: not ahead, and inside the window or among the kept first tokens."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    if mask and mask.get("size") is not None:
        ok = ok & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first") or 0)))
    return ok


def softmax_attention(q, k, v, scale, mask, softcap=None):
    """q, k [T, H, dk], v [T, H, dv]: already one key / value head per query head."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    s = s.masked_fill(~visible(T, mask)[None], float("-inf"))
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v)


def projection(h, p, name):
    y = h @ p[name].T
    return y + p[name + ".b"] if name + ".b" in p else y


def keys_and_values(h, positions, p, pre, m, eps):
    """(keys [T, G, maps, dim] after norm and rotation, values [T, G, vdim]) of a layer with projections of its own."""
    T, G, d, dv = h.shape[0], int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    maps = 2 if "diff" in m else 1
    k = projection(h, p, pre + "k").view(T, G * maps, d)
    if pre + "k.norm" in p:
        k = rms_div(k, eps) * p[pre + "k.norm"]
    return rotate(k, positions, m.get("rot")).view(T, G, maps, d), projection(h, p, pre + "v").view(T, G, dv)


def queries(h, positions, p, pre, m, eps):
    T, H, d = h.shape[0], int(m["heads"]), int(m["dim"])
    maps = 2 if "diff" in m else 1
    q = projection(h, p, pre + "q").view(T, H * maps, d)
    if pre + "q.norm" in p:
        q = rms_div(q, eps) * p[pre + "q.norm"]
    return rotate(q, positions, m.get("rot")).view(T, H, maps, d)


def diff_lambda(p, pre, diff):
    a = torch.exp((p[pre + "lq1"] * p[pre + "lk1"]).sum())
    b = torch.exp((p[pre + "lq2"] * p[pre + "lk2"]).sum())
    return a - b + diff


def attention(h, positions, p, pre, m, eps, lent=None):
    """``lent``: the (keys, values) of another layer, for a layer without its own.  Returns (output, keys, values)."""
    T, H, G = h.shape[0], int(m["heads"]), int(m["kv_heads"])
    k, v = keys_and_values(h, positions, p, pre, m, eps) if lent is None else lent
    q = queries(h, positions, p, pre, m, eps)
    rep = H // G
    kk, vv = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    a = [softmax_attention(q[:, :, i], kk[:, :, i], vv, float(m["scale"]), m.get("mask"), m.get("softcap")) for i in range(q.shape[2])]
    if "diff" in m:
        d = float(m["diff"])
        o = rms_div(a[0] - diff_lambda(p, pre, d) * a[1], eps) * (1.0 - d)
    else:
        o = a[0]
    return projection(o.reshape(T, -1), p, pre + "o"), k, v


# ----------------------------------------------------------------------------------------------- feed-forward
def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_ffn(h, p, pre):
    return (gelu_tanh(h @ p[pre + "gate"].T) * (h @ p[pre + "up"].T)) @ p[pre + "down"].T


# ----------------------------------------------------------------------------------------------- the model
def forward(tokens, cfg, p, return_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer)."""
    eps = float(cfg["norm"]["eps"])
    pos = torch.arange(len(tokens))
    x = p["embed"][torch.as_tensor(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    layers, kept = [], {}
    for i, L in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", L["mixer"]
        h = layer_norm(x, p[pre + "norm1"], eps)
        lent = kept[int(m["kv_from"])] if m.get("kv_from") is not None else None
        y, k, v = attention(h, pos, p, pre + "mix.", m, eps, lent)
        kept[i] = (k, v)
        if L.get("mlp") is not None:
            y = y + gated_ffn(h, p, pre + "mlp.")          # both sub-layers read the same normed input
        x = x + y
        layers.append(x)
    logits = layer_norm(x, p["final.norm"], eps) @ p["head"].T
    return (logits, layers) if return_layers else logits


def load_weights(path):
    """Every tensor of a checkpoint folder in float64."""
    from pathlib import Path

    from safetensors.torch import load_file

    out = {}
    for f in sorted(Path(path).glob("*.safetensors")):
        out.update({k: v.to(F64) for k, v in load_file(str(f)).items()})
    return out
