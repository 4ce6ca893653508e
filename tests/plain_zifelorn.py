"""A plain, slow implementation of the Zifelorn decoder, one function per mechanism, in float64.

It takes the configuration as the dictionary of config.json and the weights as a dictionary name -> tensor, runs ONE
sequence from its first token, and shares no code with the engine.  The tests compare the engine with it.

Notation: T tokens, E the width, H heads, r the latent's size, dr the rotated part, C the channels of a recurrent block.
"""
import math

import torch

F64 = torch.float64


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def rotate_adjacent(x, positions, base):
    """x [T, heads, dr]: entries (2i, 2i + 1) turned by p * base^(-2i / dr)."""
    dr = x.shape[-1]
    f = torch.tensor([base ** (-2.0 * i / dr) for i in range(dr // 2)], dtype=F64)
    ang = positions.to(F64)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = a * c - b * s
    out[..., 1::2] = b * c + a * s
    return out


def latent_kv(h, W, pre, m, eps):
    """What a latent attention layer keeps a position: the normalised latent and the rotated key part."""
    T, r = h.shape[0], m["kv_rank"]
    u = h @ W[pre + "dkv"].T
    c = rms_norm(u[:, :r], W[pre + "dkv.norm"], eps)
    kr = rotate_adjacent(u[:, r:].reshape(T, 1, -1), torch.arange(T), float(m["rot"]["base"]))[:, 0]
    return c, kr


def latent_attention(h, W, pre, m, eps, kv):
    """kv: (latent c [T, r], rotated key part [T, dr]) - the layer's own or an earlier layer's."""
    T = h.shape[0]
    H, d, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = kv
    cq = rms_norm(h @ W[pre + "dq"].T, W[pre + "dq.norm"], eps)
    q = (cq @ W[pre + "uq"].T).view(T, H, d + dr)
    qn, qr = q[..., :d], rotate_adjacent(q[..., d:], torch.arange(T), float(m["rot"]["base"]))
    kn = (c @ W[pre + "uk"].T).view(T, H, d)
    v = (c @ W[pre + "uv"].T).view(T, H, dv)
    s = (torch.einsum("ihd,jhd->hij", qn, kn) + torch.einsum("ihd,jd->hij", qr, kr)) * float(m["scale"])
    hidden = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    p = torch.softmax(s.masked_fill(hidden[None], float("-inf")), -1)
    o = torch.einsum("hij,jhd->ihd", p, v).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def short_conv(u, w, bias):
    """u [T, C], w [C, taps]: y_t = bias + sum_j w[:, j] u_(t - taps + 1 + j), zeros in front of the sequence."""
    T, C = u.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=u.dtype), u], 0)
    y = bias[None, :].expand(T, C).clone()
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j][None, :]
    return y


def block_diagonal(u, w, b):
    """u [T, C] in equal parts, w [parts, out, in], b [parts, out]: each part through its own square matrix."""
    n, size = w.shape[0], w.shape[1]
    return (torch.einsum("tbi,boi->tbo", u.view(-1, n, size), w) + b.view(n, size)[None]).reshape(u.shape)


def rglru(u, r, i, lam):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a_t = -8 r_t softplus(lam), S = 0 in front of the sequence."""
    log_a = -8.0 * r * softplus(lam)[None, :]
    a = torch.exp(log_a)
    b = torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    S, out = torch.zeros_like(u[0]), []
    for t in range(u.shape[0]):
        S = a[t] * S + b[t]
        out.append(S)
    return torch.stack(out)


def recurrent_block(h, W, pre):
    y = gelu_tanh(h @ W[pre + "y"].T + W[pre + "y.b"])
    u = short_conv(h @ W[pre + "x"].T + W[pre + "x.b"], W[pre + "conv"], W[pre + "conv.b"])
    r = torch.sigmoid(block_diagonal(u, W[pre + "ra"], W[pre + "ra.b"]))
    i = torch.sigmoid(block_diagonal(u, W[pre + "ri"], W[pre + "ri.b"]))
    return (rglru(u, r, i, W[pre + "lam"]) * y) @ W[pre + "o"].T


def dense_ff(h, W, pre):
    return (gelu_tanh(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


def route(z, top):
    """The `top` largest logits and the softmax over those alone."""
    val, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(val, -1)


def experts_ff(h, W, pre, m):
    idx, w = route(h @ W[pre + "router"].T + W[pre + "router.b"], m["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k in range(idx.shape[1]):
            e = f"{pre}e{int(idx[t, k])}."
            up = torch.clamp(W[e + "up"] @ h[t], min=0.0) ** 2
            out[t] += w[t, k] * (W[e + "down"] @ up)
    return out


def forward(cfg, W, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence from its first token (and, on request, the stream after every layer)."""
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)].to(F64) * float(cfg["embedding"]["scale"])
    kept, streams = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                kept[i] = latent_kv(x, W, p + "mix.", m, eps)
            y = latent_attention(x, W, p + "mix.", m, eps, kept[i if src is None else src])
        else:
            y = recurrent_block(x, W, p + "mix.")
        x = x + rms_norm(y, W[p + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp:
            y = dense_ff(x, W, p + "mlp.") if mlp["kind"] == "dense" else experts_ff(x, W, p + "mlp.", mlp)
            x = x + rms_norm(y, W[p + "norm2"], eps)
        streams.append(x)
    logits = rms_norm(x, W["final.norm"], eps) @ W["embed"].to(F64).T * float(cfg["logit_scale"])
    return (logits, torch.stack(streams)) if return_layers else logits
