"""A plain, slow implementation of the Buguzen decoder, one function per mechanism, in float64.

It takes the configuration as the dictionary of config.json and the weights as a dictionary name -> tensor, runs ONE
sequence from its first token, and shares no code with the engine.  The tests compare the engine with it.

Notation: T tokens, E the width, H heads, G key/value heads, d the key size of a head, dv its value size.

The design: every layer is  x <- x + mixer(n1 x), x <- x + ff(n2 x)  (or the first alone), then a token input
x <- x + n_s(P (gelu(Gt x) * e_tok))  with the layer's own columns of a second table.  Mixers: differential attention (two
softmaxes over the same values, subtracted), attention whose values are its keys (sinks, a norm per head), and linear attention
with a fixed decay per head.  A span of layers may run several times; pass t first adds row t of a small table to the stream.
"""
import math

import torch

F64 = torch.float64


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def plain_frequencies(base, dims):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)


def linear_frequencies(base, dims, scaling):
    """Every frequency divided by one factor."""
    f = plain_frequencies(base, dims)
    return f / float(scaling["factor"]) if scaling else f


def banded_frequencies(base, dims, scaling):
    """Short waves as they are, long waves slowed by the factor, a blend between two wavelengths."""
    f = plain_frequencies(base, dims)
    if not scaling:
        return f
    factor, low, high = float(scaling["factor"]), float(scaling["low"]), float(scaling["high"])
    orig = float(scaling["original"])
    out = []
    for fi in f.tolist():
        wave = 2.0 * math.pi / fi
        if wave < orig / high:
            out.append(fi)
        elif wave > orig / low:
            out.append(fi / factor)
        else:
            s = (orig / wave - low) / (high - low)
            out.append((1.0 - s) * fi / factor + s * fi)
    return torch.tensor(out, dtype=F64)


def turn(u, v, positions, f):
    """The pairs (u, v) [T, heads, n] turned by the angles p * f."""
    ang = positions.to(F64)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    return u * c - v * s, v * c + u * s


def rotate_adjacent(x, positions, f):
    """x [T, heads, d]: entries (2i, 2i + 1) of the first 2 len(f) numbers are pairs."""
    dims, out = 2 * len(f), x.clone()
    out[..., 0:dims:2], out[..., 1:dims:2] = turn(x[..., 0:dims:2], x[..., 1:dims:2], positions, f)
    return out


def rotate_halves(x, positions, f):
    """x [T, heads, d]: entries (i, i + len(f)) are pairs."""
    n, out = len(f), x.clone()
    out[..., :n], out[..., n:2 * n] = turn(x[..., :n], x[..., n:2 * n], positions, f)
    return out


def visible(T, size):
    """visible[i, j]: 0 <= i - j < size (size None: every earlier key)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < size) if size is not None else d >= 0


def softmax_values(q, k, v, scale, mask, sink=None):
    """q [T, H, d], k [T, H, d], v [T, H, dv]: softmax over the visible keys, a sink per head in the denominator only."""
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~mask[None], float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(s - top)
    z = e.sum(-1, keepdim=True)
    if sink is not None:
        z = z + torch.exp(sink[:, None, None] - top)
    return torch.einsum("hij,jhd->ihd", e / z, v)


def window_size(m):
    return int(m["mask"]["size"]) if m.get("mask") else None


def map_weight(W, pre, diff):
    """What the second softmax is weighted with: one number for the layer."""
    dot = lambda a, b: torch.dot(W[pre + a].to(F64), W[pre + b].to(F64))
    return torch.exp(dot("lq1", "lk1")) - torch.exp(dot("lq2", "lk2")) + diff


def differential_attention(h, W, pre, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W[pre + "q"].T + W[pre + "q.b"]).view(T, H, 2, d)
    k = (h @ W[pre + "k"].T + W[pre + "k.b"]).view(T, G, 2, d)
    v = (h @ W[pre + "v"].T + W[pre + "v.b"]).view(T, G, dv).repeat_interleave(H // G, dim=1)
    maps = []
    for j in range(2):
        qj, kj = q[:, :, j], k[:, :, j].repeat_interleave(H // G, dim=1)
        if m.get("rot"):
            f = linear_frequencies(float(m["rot"]["base"]), int(m["rot"]["dims"]), m["rot"].get("scaling"))
            qj, kj = rotate_adjacent(qj, torch.arange(T), f), rotate_adjacent(kj, torch.arange(T), f)
        maps.append(softmax_values(qj, kj, v, float(m["scale"]), visible(T, window_size(m))))
    diff = float(m["diff"])
    o = maps[0] - map_weight(W, pre, diff) * maps[1]
    o = rms_norm(o, 1.0, eps) * (1.0 - diff)
    return o.reshape(T, H * dv) @ W[pre + "o"].T


def keys_as_values_attention(h, W, pre, m, eps):
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[pre + "q"].T + W[pre + "q.b"]).view(T, H, d)
    k = (h @ W[pre + "k"].T + W[pre + "k.b"]).view(T, G, d)
    v = k
    q, k = rms_norm(q, W[pre + "q.norm"], eps), rms_norm(k, W[pre + "k.norm"], eps)
    if m.get("rot"):
        f = banded_frequencies(float(m["rot"]["base"]), int(m["rot"]["dims"]), m["rot"].get("scaling"))
        q, k = rotate_halves(q, torch.arange(T), f), rotate_halves(k, torch.arange(T), f)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    o = softmax_values(q, k, v, float(m["scale"]), visible(T, window_size(m)), W[pre + "sink"])
    return o.reshape(T, H * d) @ W[pre + "o"].T


def decayed_sums(q, k, v, decay):
    """q, k [T, H, d], v [T, H, dv]: S <- decay S + k v^T from zero, o = S^T q."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = S * decay[:, None, None] + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hd,hdv->hv", q[t], S))
    return torch.stack(out)


def lightning(h, W, pre, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ W[pre + "q"].T).view(T, H, d)
    k = silu(h @ W[pre + "k"].T).view(T, H, d)
    v = silu(h @ W[pre + "v"].T).view(T, H, dv)
    o = decayed_sums(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)).reshape(T, H * dv)
    o = rms_norm(o, W[pre + "norm"], eps) * torch.sigmoid(h @ W[pre + "g"].T)
    return o @ W[pre + "o"].T


MIXERS = {"attention": differential_attention, "attention_2": keys_as_values_attention, "lightning": lightning}


def gated_ff(h, W, pre):
    return (torch.clamp(h @ W[pre + "gate"].T, min=0.0) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


def token_input(x, tokens, W, pre, i, dim, eps):
    e = W["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ W[pre + "gate"].T) * e) @ W[pre + "proj"].T
    return x + rms_norm(y, W[pre + "norm"], eps)


def order(cfg):
    """(layer, pass number or None): a number where a pass of the looped span begins."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, None) for i in range(a)]
    for t in range(times):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(cfg, W, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence from its first token (and, on request, the stream after every layer run)."""
    eps = float(cfg["norm"]["eps"])
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"][tokens].to(F64)
    side = (cfg.get("token_side") or {}).get("dim")
    streams = []
    for i, t in order(cfg):
        if t is not None:
            x = x + W["loop.step"][t]
        p, layer = f"l{i}.", cfg["layers"][i]
        x = x + MIXERS[layer["type"]](rms_norm(x, W[p + "norm1"], eps), W, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            x = x + gated_ff(rms_norm(x, W[p + "norm2"], eps), W, p + "mlp.")
        if side:
            x = token_input(x, tokens, W, p + "side.", i, side, eps)
        streams.append(x)
    logits = rms_norm(x, W["final.norm"], eps) @ W["head"].to(F64).T
    return (logits, torch.stack(streams)) if return_layers else logits
