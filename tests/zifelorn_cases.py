"""Small Zifelorn configurations and random weights for the tests, made here (names and shapes written out by hand, so a
loader that expects other names or shapes fails).

The configurations differ from one another in every size and option: width, vocabulary, heads, latent sizes, key and value
sizes, rotated parts, layers that read an earlier layer's latents, channels of the recurrent blocks, blocks (one, some, of
sizes that are and are not multiples of eight), taps of the convolution (1 to 5), experts and how many of them a row uses (one,
some, all), dense feed-forwards and none, the two scales, and the order of layers.
"""
import json
import os

import torch

from plain_llama import write_safetensors


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def rglru(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, eps=1e-6, embed_scale=1.0, logit_scale=1.0):
    """layers: (mixer, mlp) pairs"""
    return {"architecture": "Zifelorn", "vocab": vocab, "width": width, "embedding": {"scale": embed_scale}, "norm": {"eps": eps},
            "logit_scale": logit_scale, "layers": [{"type": l["type"], "mixer": l["mixer"], "mlp": m} for l, m in layers]}


# every mixer and feed-forward, small everything, sizes that are no power of two; all experts used, one tap
CASE_A = config(96, 211, [
    (latent(3, 16, 8, 24, 40, 48, 0.2, 10000.0), dense(80)),
    (rglru(72, 3, 4), moe(40, 6, 2)),
    (latent(2, 24, 8, 16, 40, 32, 0.25, 10000.0, kv_from=0), None),
    (rglru(60, 1, 1), moe(24, 5, 5)),
], eps=2e-6, embed_scale=3.5, logit_scale=1.75)

# recurrent layers first; parts of 16, 12 and 7 channels; one expert a row; two owners of latents
CASE_B = config(128, 300, [
    (rglru(128, 8, 2), dense(96)),
    (latent(4, 24, 16, 40, 32, 72, 0.16, 50000.0), moe(56, 9, 1)),
    (rglru(48, 4, 3), None),
    (latent(4, 8, 16, 8, 32, 24, 0.3, 50000.0, kv_from=1), dense(64)),
    (latent(1, 16, 4, 12, 24, 20, 0.3, 700.0), moe(32, 3, 2)),
    (rglru(35, 5, 5), dense(48)),
], eps=3e-5, embed_scale=0.8, logit_scale=0.3)

# sizes the tensor-core kernels take: heads of 128 and 64 for whole prompts, parts of 128 and 256 channels
CASE_C = config(256, 333, [
    (latent(4, 64, 64, 128, 64, 64, 0.09, 10000.0), moe(128, 4, 2)),
    (rglru(256, 2, 4), dense(192)),
    (latent(2, 64, 64, 64, 64, 32, 0.1, 10000.0, kv_from=0), dense(64)),
    (rglru(512, 2, 2), moe(64, 12, 3)),
    (latent(3, 48, 16, 64, 128, 96, 0.12, 2000.0), dense(128)),
], embed_scale=6.0, logit_scale=2.5)

CASE_D = config(64, 90, [(rglru(40, 5, 3), dense(40)), (latent(2, 16, 16, 16, 24, 24, 0.25, 1000.0), moe(24, 4, 2))], eps=1e-4)

CASES = {"a": CASE_A, "b": CASE_B, "c": CASE_C, "d": CASE_D}


def tensor_shapes(cfg):
    E = cfg["width"]
    shapes = {"embed": (cfg["vocab"], E), "final.norm": (E,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        shapes[p + "norm1"] = (E,)
        x = p + "mix."
        if layer["type"] == "latent_attention":
            H = m["heads"]
            shapes[x + "dq"], shapes[x + "dq.norm"] = (m["q_rank"], E), (m["q_rank"],)
            shapes[x + "uq"] = (H * (m["dim"] + m["rot_dim"]), m["q_rank"])
            if "kv_from" not in m:
                shapes[x + "dkv"], shapes[x + "dkv.norm"] = (m["kv_rank"] + m["rot_dim"], E), (m["kv_rank"],)
            shapes[x + "uk"], shapes[x + "uv"] = (H * m["dim"], m["kv_rank"]), (H * m["vdim"], m["kv_rank"])
            shapes[x + "g"], shapes[x + "o"] = (H * m["vdim"], E), (E, H * m["vdim"])
        else:
            C, B = m["width"], m["blocks"]
            s = C // B
            for n in ("y", "x"):
                shapes[x + n], shapes[x + n + ".b"] = (C, E), (C,)
            shapes[x + "conv"], shapes[x + "conv.b"] = (C, m["conv"]), (C,)
            for n in ("ra", "ri"):
                shapes[x + n], shapes[x + n + ".b"] = (B, s, s), (B, s)
            shapes[x + "lam"], shapes[x + "o"] = (C,), (E, C)
        f = layer["mlp"]
        if f is None:
            continue
        shapes[p + "norm2"] = (E,)
        if f["kind"] == "dense":
            shapes[p + "mlp.gate"] = shapes[p + "mlp.up"] = (f["ff"], E)
            shapes[p + "mlp.down"] = (E, f["ff"])
        else:
            n, F = f["router"]["experts"], f["expert"]["ff"]
            shapes[p + "mlp.router"], shapes[p + "mlp.router.b"] = (n, E), (n,)
            for e in range(n):
                shapes[p + f"mlp.e{e}.up"], shapes[p + f"mlp.e{e}.down"] = (F, E), (E, F)
    return shapes


def random_weights(cfg, seed, sharp=1.0, lam=0.0, router=1.0):
    """bfloat16 tensors: matrices ~ N(0, 1/in), norm weights ~ 1 + N(0, 0.2), biases ~ N(0, 0.3), taps ~ N(0, 0.5), lam ~
    N(lam, 1), the table ~ N(0, 1) over its scale.  ``sharp`` multiplies the query and key maps of latent attention, so that a
    few keys carry each softmax; a low ``lam`` makes the recurrent states forget slowly; ``router`` multiplies the routers, so
    that the last of a row's choices - the one rounding may change - weighs little."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if last in ("norm", "norm1", "norm2"):
            t = 1.0 + torch.randn(shape, generator=g) * 0.2
        elif last == "lam":
            t = torch.randn(shape, generator=g) + lam
        elif last == "conv":
            t = torch.randn(shape, generator=g) * 0.5
        elif last == "b":
            t = torch.randn(shape, generator=g) * 0.3
        elif name == "embed":
            t = torch.randn(shape, generator=g) / cfg["embedding"]["scale"]
        else:
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
            if last in ("uq", "uk"):
                t = t * sharp
            if last == "router":
                t = t * router
        W[name] = t.to(torch.bfloat16)
    return W


def write_model(path, cfg, W):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), W)
    return str(path)


def make_model(tmp_path, cfg, seed, sharp=1.0, lam=0.0, router=1.0, change=None):
    """(model folder, float64 weights for the plain implementation); ``change(W)`` may edit the bfloat16 tensors first"""
    W = random_weights(cfg, seed, sharp, lam, router)
    if change:
        change(W)
    d = write_model(tmp_path, cfg, W)
    return d, {k: v.to(torch.float64) for k, v in W.items()}
