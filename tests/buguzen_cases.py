"""Small Buguzen configurations and random weights for the tests, made here (names and shapes written out by hand, so a
loader that expects other names or shapes fails).

The configurations differ from one another in every size and option: width, vocabulary, heads and key/value heads (one, some, as
many as heads), key and value sizes (also the sizes the tensor-core attention takes: 64, 128, and keys of 64 beside values of 128),
rotated dimensions (all, some, none) with and without slowed frequencies, windows (one token, shorter and longer than the
sequences, around a page's edge, none), decays (none at all, slow, one), feed-forwards of several sizes and none on every kind of
layer, the token input (with, without), the loop (none; once; three times over a span in the middle; twice over everything) and
the order of layers.
"""
import json
import os

import torch

from plain_llama import write_safetensors


def _attention(kind, heads, kv_heads, dim, vdim, scale, size, rot, scaling, keys):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(keys, scaling))
    return {"type": kind, "mixer": m}


def differential(heads, kv_heads, dim, vdim, scale, diff, size=None, rot=None, scaling=None):
    l = _attention("attention", heads, kv_heads, dim, vdim, scale, size, rot, scaling, ("factor",))
    l["mixer"]["diff"] = diff
    return l


def keys_as_values(heads, kv_heads, dim, scale, size=None, rot=None, scaling=None):
    return _attention("attention_2", heads, kv_heads, dim, dim, scale, size, rot, scaling, ("factor", "low", "high", "original"))


def lightning(heads, dim, vdim, decay):
    assert len(decay) == heads
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def config(width, vocab, layers, loop=None, side=None, eps=1e-5):
    """layers: (mixer, size of the feed-forward or None) pairs"""
    c = {"architecture": "Buguzen", "vocab": vocab, "width": width, "norm": {"eps": eps},
         "layers": [{"type": l["type"], "mixer": l["mixer"], "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for l, ff in layers]}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    if side is not None:
        c["token_side"] = {"dim": side}
    return c


# small everything, sizes that are no power of two; a span in the middle runs three times
CASE_A = config(96, 211, [
    (differential(4, 2, 20, 28, 0.3, 0.4, size=9, rot=(10000.0, 8), scaling=(3.0,)), 80),
    (keys_as_values(6, 3, 24, 0.2, size=21, rot=(700.0, 24), scaling=(4.0, 1.0, 3.0, 60)), None),
    (lightning(3, 16, 24, [0.5, 0.93, 0.999]), 56),
    (differential(3, 3, 12, 40, 0.25, 0.75, rot=(500.0, 12)), None),
], loop=(1, 3, 3), side=8, eps=2e-6)

# no loop, no token input; sizes the tensor-core attention takes; windows around a page's edge
CASE_B = config(128, 300, [
    (lightning(2, 64, 128, [0.8, 0.99]), 96),
    (differential(4, 2, 64, 128, 0.125, 0.55, size=65, rot=(300000.0, 16)), 128),
    (keys_as_values(6, 2, 128, 0.09, size=64, rot=(10000.0, 32), scaling=(16.0, 1.0, 4.0, 128)), None),
    (differential(3, 1, 64, 64, 0.2, 0.3, size=130, rot=(1000.0, 64), scaling=(2.0,)), 64),
    (keys_as_values(4, 4, 64, 0.15), 48),
    (lightning(1, 128, 64, [0.97]), None),
])

# a width the tensor-core contractions refuse, odd sizes everywhere, everything looped twice; a head that forgets at once, one that
# never forgets
CASE_C = config(100, 90, [
    (keys_as_values(5, 5, 10, 0.35, size=33, rot=(50.0, 6), scaling=(2.0, 0.5, 2.0, 16)), 28),
    (lightning(4, 9, 13, [0.0, 0.7, 1.0, 0.995]), None),
    (differential(2, 1, 7, 11, 0.5, 0.2, size=1), 20),
], loop=(0, 3, 2), side=5)

# a loop that runs once, in front of the last layers
CASE_D = config(64, 70, [(lightning(2, 8, 8, [0.9, 0.4]), None),
                         (keys_as_values(2, 1, 16, 0.25, size=8, rot=(1000.0, 16)), 40),
                         (differential(4, 4, 16, 32, 0.3, 0.5, size=40, rot=(100.0, 4), scaling=(1.5,)), 24)], loop=(1, 3, 1), side=12)

# layers without a token input inside a loop: the pass's vector has a kernel of its own
CASE_E = config(64, 80, [(differential(2, 2, 16, 16, 0.25, 0.6, size=17, rot=(1000.0, 8)), 40), (lightning(2, 16, 16, [0.95, 0.6]), 32)],
                loop=(0, 2, 3))

CASES = {"a": CASE_A, "b": CASE_B, "c": CASE_C, "d": CASE_D, "e": CASE_E}


def tensor_shapes(cfg):
    E = cfg["width"]
    shapes = {"embed": (cfg["vocab"], E), "head": (cfg["vocab"], E), "final.norm": (E,)}
    if "loop" in cfg:
        shapes["loop.step"] = (cfg["loop"]["times"], E)
    side = cfg.get("token_side", {}).get("dim")
    if side:
        shapes["side.embed"] = (cfg["vocab"], side * len(cfg["layers"]))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        shapes[p + "norm1"] = (E,)
        x, H, d, dv = p + "mix.", m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "lightning":
            rows, biased = {"q": H * d, "k": H * d, "v": H * dv, "g": H * dv}, ()
            shapes[x + "norm"] = (H * dv,)
        elif layer["type"] == "attention":
            rows, biased = {"q": H * 2 * d, "k": m["kv_heads"] * 2 * d, "v": m["kv_heads"] * dv}, "qkv"
            for n in ("lq1", "lk1", "lq2", "lk2"):
                shapes[x + n] = (d,)
        else:
            rows, biased = {"q": H * d, "k": m["kv_heads"] * d}, "qk"
            shapes[x + "q.norm"] = shapes[x + "k.norm"] = (d,)
            shapes[x + "sink"] = (H,)
        for n, r in rows.items():
            shapes[x + n] = (r, E)
            if n in biased:
                shapes[x + n + ".b"] = (r,)
        shapes[x + "o"] = (E, H * dv)
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            shapes[p + "norm2"] = (E,)
            shapes[p + "mlp.gate"] = shapes[p + "mlp.up"] = (F, E)
            shapes[p + "mlp.down"] = (E, F)
        if side:
            shapes[p + "side.gate"], shapes[p + "side.proj"], shapes[p + "side.norm"] = (side, E), (E, side), (E,)
    return shapes


def random_weights(cfg, seed, sharp=1.0):
    """bfloat16 tensors: matrices ~ N(0, 1/in), norm weights ~ 1 + N(0, 0.2), biases ~ N(0, 0.3), the vectors behind lambda ~
    N(0, 0.3), sinks ~ 1 + N(0, 1), tables and loop vectors ~ N(0, 1).  ``sharp`` multiplies the query and key maps, so that a few keys
    carry each softmax and a key that is wrongly seen or missed changes the result by much more than bfloat16 rounding does."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        t = torch.randn(shape, generator=g)
        if last in ("norm", "norm1", "norm2"):
            t = 1.0 + t * 0.2
        elif last == "b" or last in ("lq1", "lk1", "lq2", "lk2"):
            t = t * 0.3
        elif last == "sink":
            t = 1.0 + t
        elif last not in ("embed", "step"):
            t = t / shape[1] ** 0.5
            if name.endswith((".mix.q", ".mix.k")):
                t = t * sharp
        W[name] = t.to(torch.bfloat16)
    return W


def write_model(path, cfg, W):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), W)
    return str(path)


def make_model(tmp_path, cfg, seed, sharp=1.0, change=None):
    """(model folder, float64 weights for the plain implementation); ``change(W)`` may edit the bfloat16 tensors first"""
    W = random_weights(cfg, seed, sharp)
    if change:
        change(W)
    d = write_model(tmp_path, cfg, W)
    return d, {k: v.to(torch.float64) for k, v in W.items()}
