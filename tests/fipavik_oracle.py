"""Plain float64 implementation of the Fipavik design: one function per mechanism, whole sequences, no cache, no state
objects, nothing imported from the package.  ``p`` maps tensor names to float64 tensors, ``cfg`` is the parsed config.json.
The tests compare the framework against these functions."""
import torch

F64 = torch.float64


# ----------------------------------------------------------------------------------------------- norms
def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


# ----------------------------------------------------------------------------------------------- rotary positions
def rotate(x, positions, rot):
    """x [T, heads, d]: channels i and i + dims / 2 of every head turn by position * base^(-2 i / dims); the rest passes."""
    n = int(rot["dims"]) // 2
    out = x.clone()
    for i in range(n):
        a = positions.to(F64) * float(rot["base"]) ** (-2.0 * i / (2 * n))
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + n]
        out[..., i] = u * c - v * s
        out[..., i + n] = v * c + u * s
    return out


# ----------------------------------------------------------------------------------------------- softmax attention
def visible_chunk(T, size):
    """[T, T], row = query: not ahead, and in the query's own block of ``size`` positions."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def visible_window(T, size):
    """[T, T]: the query itself and the size - 1 tokens before it."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def sink_softmax(s, ok, sink):
    """s [H, T, T] scores, ok [T, T] visible, sink [H]: weights whose denominator also holds exp(sink)."""
    s = s.masked_fill(~ok[None], float("-inf"))
    m = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - m))


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, positions, p, pre, m, eps, v_first=None):
    """Grouped-query attention over chunks; ``v_first``: the values of the first mixing layer.  Returns (output, values)."""
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate(rms_norm((h @ p[pre + "q"].T).view(T, H, d), p[pre + "q.norm"], eps), positions, m["rot"])
    k = rotate(rms_norm((h @ p[pre + "k"].T).view(T, G, d), p[pre + "k.norm"], eps), positions, m["rot"])
    v = (h @ p[pre + "v"].T).view(T, G, dv)
    if v_first is not None:
        v = mix_values(v, v_first, p[pre + "vmix"])
    kk, vv = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * float(m["scale"])
    w = sink_softmax(s, visible_chunk(T, int(m["mask"]["size"])), p[pre + "sink"])
    return torch.einsum("hij,jhd->ihd", w, vv).reshape(T, H * dv) @ p[pre + "o"].T, v


def latent_attention(h, positions, p, pre, m, eps):
    """Per-head keys and values out of a normed latent, one rotated key part for all heads, a window."""
    T, H, d, r, dv, R = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    q = (h @ p[pre + "q"].T).view(T, H, d + r)
    q_n, q_r = q[..., :d], rotate(q[..., d:], positions, m["rot"])
    y = h @ p[pre + "dkv"].T
    c = rms_norm(y[:, :R], p[pre + "dkv.norm"], eps)
    k_r = rotate(y[:, None, R:], positions, m["rot"])[:, 0]
    k_n = (c @ p[pre + "uk"].T).view(T, H, d)
    v = (c @ p[pre + "uv"].T).view(T, H, dv)
    s = (torch.einsum("ihd,jhd->hij", q_n, k_n) + torch.einsum("ihd,jd->hij", q_r, k_r)) * float(m["scale"])
    w = sink_softmax(s, visible_window(T, int(m["mask"]["size"])), p[pre + "sink"])
    return torch.einsum("hij,jhd->ihd", w, v).reshape(T, H * dv) @ p[pre + "o"].T


# ----------------------------------------------------------------------------------------------- feed-forward
def silu(z):
    return z / (1.0 + torch.exp(-z))


def expert(h, p, pre):
    return (silu(h @ p[pre + "gate"].T) * (h @ p[pre + "up"].T)) @ p[pre + "down"].T


def route(z, top):
    """z [T, E] logits -> [T, E] weights: softmax over the ``top`` largest, 0 elsewhere."""
    chosen = torch.sort(z, dim=-1, descending=True, stable=True).indices[:, :top]
    e = torch.exp(z.gather(1, chosen) - z.max(-1, keepdim=True).values)
    return torch.zeros_like(z).scatter(1, chosen, e / e.sum(-1, keepdim=True))


def mixture(h, p, pre, f):
    w = route(h @ p[pre + "router"].T + p[pre + "router.b"], int(f["router"]["top"]))
    y = sum(w[:, e:e + 1] * expert(h, p, f"{pre}e{e}.") for e in range(w.shape[1]))
    return y + expert(h, p, pre + "shared.") if f.get("shared") is not None else y


# ----------------------------------------------------------------------------------------------- the model
def forward(tokens, cfg, p, return_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer)."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    pos = torch.arange(len(tokens))
    x = p["embed"][torch.as_tensor(tokens)]
    layers, v_first = [], None
    for i, L in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", L["mixer"]
        h = layer_norm(x, p[pre + "norm1"], p[pre + "norm1.b"], eps)
        if L["type"] == "attention":
            y, v = attention(h, pos, p, pre + "mix.", m, eps, v_first if m.get("v_mix") else None)
            if m.get("v_mix") and v_first is None:
                v_first = v
        else:
            y = latent_attention(h, pos, p, pre + "mix.", m, eps)
        if L.get("mlp") is not None:
            y = y + mixture(h, p, pre + "mlp.", L["mlp"])          # both sub-layers read the same normed input
        x = x + mult * y
        layers.append(x)
    logits = layer_norm(x, p["final.norm"], p["final.norm.b"], eps) @ p["embed"].T
    return (logits, layers) if return_layers else logits


def load_weights(path):
    """Every tensor of a checkpoint folder in float64."""
    from pathlib import Path

    from safetensors.torch import load_file

    out = {}
    for f in sorted(Path(path).glob("*.safetensors")):
        out.update({k: v.to(F64) for k, v in load_file(str(f)).items()})
    return out
