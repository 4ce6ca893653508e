"""The Buguzen decoder in the engine against the plain implementation (``plain_buguzen``): each mechanism alone, whole prompts,
portions, decoding, batches, reused slots and pages, and generation through the entry point.

Structure is tested in float32, where any key wrongly seen or missed, any state lost or kept too long is orders of
magnitude above the tolerance; the bfloat16 runs use sharpened attention (see ``buguzen_cases.random_weights``) so that the same
faults stay visible above rounding."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_buguzen as pb
from buguzen_cases import CASES, config, differential, keys_as_values, lightning, make_model, random_weights, write_model
from helpers import rel_err

pytestmark = pytest.mark.gpu

#: max |dlogit| / max |logit| against the float64 plain implementation.  float32: a key wrongly seen or a lost state is at 1e-3
#: and above.  bfloat16 with sharpened attention: rounding reaches a few 1e-2, a structural fault 0.3 and more
TOL = {"float32": 2e-5, "bfloat16": 8e-2}
EPS = 1e-6


def tokens_for(cfg, n, seed):
    rng = np.random.default_rng(seed)
    return [int(t) for t in rng.integers(0, cfg["vocab"], size=n)]


def engine_for(model_dir, dtype, **kw):
    from fastgguf_b200.engine.api import Engine
    args = dict(dtype=dtype, max_tokens=4096, max_batch=8)
    args.update(kw)
    return Engine.from_dir(model_dir, **args)


def entry(slot, toks, want=None):
    from fastgguf_b200.engine.batch import StepEntry
    return StepEntry(slot, toks, list(range(len(toks))) if want is None else want)


def plain_logits(cfg, W, toks):
    return pb.forward(cfg, W, toks).numpy()


def f32(x):
    return np.ascontiguousarray(x.numpy() if hasattr(x, "numpy") else x, dtype=np.float32)


def apart(a, b):
    """max |a - b| / max |b|: how far two results of the oracle, or of two models, lie apart (no error of the engine's)"""
    return float(np.abs(np.asarray(a) - np.asarray(b)).max() / np.abs(np.asarray(b)).max())


class Rows:
    """Collects the errors of a whole model's logits, row by row, and judges them.

    The difference of two maps, the recurrence's outputs and the token input are normalised whatever their size, so where one of
    them is short every rounding in it is amplified.  At most one row in fifty (or one row) may exceed the tolerance in float32,
    where none may exceed five times the tolerance; one in fifteen in bfloat16.  A key wrongly seen or a lost state moves most rows
    by far more."""

    def __init__(self, dtype):
        self.dtype, self.n, self.over = dtype, 0, []

    def add(self, got, want, what):
        e = rel_err(got, want)
        self.n += 1
        assert np.isfinite(e) and (self.dtype == "bfloat16" or e < 5 * TOL[self.dtype]), (what, e)
        if e >= TOL[self.dtype]:
            self.over.append((what, e))

    def done(self):
        assert len(self.over) <= max(1, self.n // (15 if self.dtype == "bfloat16" else 50)), (len(self.over), self.n, self.over[:20])


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """(case, dtype): for bfloat16 attention is sharpened"""
    out = {}
    for i, (name, cfg) in enumerate(CASES.items()):
        for dtype, sharp in (("float32", 1.0), ("bfloat16", 1.5)):
            d, W = make_model(tmp_path_factory.mktemp(f"b_{name}_{dtype}"), cfg, 100 + i, sharp)
            out[(name, dtype)] = (d, cfg, W)
    return out


# ------------------------------------------------------------------------------ mechanisms alone
MIXERS = {
    "two maps, small": differential(4, 2, 20, 28, 0.3, 0.4, size=9, rot=(10000.0, 8), scaling=(3.0,)),
    "two maps, one key head, odd sizes, one key seen": differential(3, 1, 7, 11, 0.5, 0.2, size=1),
    "two maps, as many key heads as heads, no window": differential(3, 3, 12, 40, 0.25, 0.75, rot=(500.0, 12)),
    "two maps, the constant zero": differential(2, 2, 16, 16, 0.25, 0.0, rot=(500.0, 4), scaling=(1.0,)),
    "keys as values, small": keys_as_values(6, 3, 24, 0.2, size=21, rot=(700.0, 24), scaling=(4.0, 1.0, 3.0, 60)),
    "keys as values, one head, no rotation": keys_as_values(1, 1, 10, 0.4),
    "keys as values, part rotated": keys_as_values(4, 2, 18, 0.3, size=40, rot=(50.0, 6)),
    "lightning, small": lightning(3, 16, 24, [0.5, 0.93, 0.999]),
    "lightning, odd sizes, one head that forgets at once": lightning(4, 9, 13, [0.0, 0.7, 1.0, 0.995]),
    "lightning, one head": lightning(1, 40, 8, [0.97]),
    "lightning, a state larger than a block holds": lightning(1, 180, 300, [0.9]),
    "lightning, values of more numbers than a block has threads": lightning(2, 9, 330, [0.97, 0.0]),
    "long two maps, keys of 64 beside values of 128": differential(4, 2, 64, 128, 0.125, 0.55, size=70, rot=(300000.0, 16)),
    "long two maps, 64 and 64, groups of three": differential(6, 2, 64, 64, 0.2, 0.3, rot=(1000.0, 64), scaling=(2.0,)),
    "long two maps, 128 and 128": differential(2, 1, 128, 128, 0.09, 0.45, size=129, rot=(1000.0, 32)),
    "long keys as values, 128": keys_as_values(6, 2, 128, 0.09, size=64, rot=(10000.0, 32), scaling=(16.0, 1.0, 4.0, 128)),
    "long keys as values, 64": keys_as_values(4, 4, 64, 0.15, size=100),
    "long lightning, heads of 64 and 128": lightning(2, 64, 128, [0.8, 0.99]),
    "long lightning, heads of 128 and 128": lightning(3, 128, 128, [0.3, 0.9, 0.9995]),
    "long lightning, heads of 24 and 40": lightning(3, 24, 40, [0.98, 0.6, 1.0]),
}


def one_layer(layer, ff=None, width=80, vocab=50, side=None):
    return config(width, vocab, [(layer, ff)], eps=EPS, side=side)


def mixer_alone(x, W, layer, eps=EPS):
    """what one layer without a feed-forward makes of the rows x"""
    return x + pb.MIXERS[layer["type"]](pb.rms_norm(x, W["l0.norm1"], eps), W, "l0.mix.", layer["mixer"], eps)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MIXERS))
def test_mixer_alone(tmp_path, name, dtype):
    """One layer of a mixer alone (norm, mixer, residual add) on rows given by the test: a portion of 37 rows, then one of 2,
    then single rows, so the second and later calls start from what the first left behind (the long cases: 160, 30 and 2
    rows, then 38 single ones)."""
    layer = MIXERS[name]
    cfg = one_layer(layer)
    d, W = make_model(tmp_path, cfg, 7, sharp=1.5)
    eng = engine_for(d, dtype)
    g = torch.Generator().manual_seed(8)
    cuts = [160, 30, 2] + [1] * 38 if name.startswith("long") else [37, 2, 1, 1, 1, 1, 1, 1]
    T = sum(cuts)
    x = torch.randn(T, cfg["width"], generator=g, dtype=torch.float64)
    want = mixer_alone(x, W, layer).numpy()
    assert np.abs(want - x.numpy()).max() > 0.1
    slot = eng.acquire()
    got, at = [], 0
    for n in cuts:
        got.append(eng.block_forward(0, [(slot, n)], f32(x[at:at + n])))
        at += n
    got = np.concatenate(got)
    tol = 2e-5 if dtype == "float32" else 4e-2
    bad = [(r, rel_err(got[r], want[r])) for r in range(T) if rel_err(got[r], want[r]) >= tol]
    assert len(bad) <= (0 if dtype == "float32" else T // 40), (name, bad[:8])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", [n for n in MIXERS if n.startswith("long")])
def test_a_wide_batch_of_prompts(tmp_path, name, dtype):
    """Prompts of 700, 300, 50 and 3 tokens in one step, then one more token each, then a portion of 5 for the last."""
    layer = MIXERS[name]
    cfg = one_layer(layer)
    d, W = make_model(tmp_path, cfg, 12, sharp=1.5)
    eng = engine_for(d, dtype, max_tokens=4096, max_batch=4)
    g = torch.Generator().manual_seed(9)
    lens = [700, 300, 50, 3]
    xs = [torch.randn(n + 6, cfg["width"], generator=g, dtype=torch.float64) for n in lens]
    want = [mixer_alone(x, W, layer).numpy() for x in xs]
    tol = 2e-5 if dtype == "float32" else 4e-2
    errs = []
    slots = [eng.acquire() for _ in lens]
    got = eng.block_forward(0, list(zip(slots, lens)), f32(torch.cat([x[:n] for x, n in zip(xs, lens)])))
    at = 0
    for b, n in enumerate(lens):
        errs += [(rel_err(got[at + r], want[b][r]), b, r) for r in range(n)]
        at += n
    got = eng.block_forward(0, [(s, 1) for s in slots], f32(torch.stack([x[n] for x, n in zip(xs, lens)])))
    errs += [(rel_err(got[b], want[b][n]), b, "decoded") for b, n in enumerate(lens)]
    got = eng.block_forward(0, [(slots[3], 5)], f32(xs[3][4:9]))
    errs += [(rel_err(got[i], want[3][4 + i]), 3, "portion", i) for i in range(5)]
    bad = [e for e in errs if e[0] >= tol]
    assert len(bad) <= (0 if dtype == "float32" else len(errs) // 40), (name, len(bad), bad[:8])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff,side,rows", [(56, None, 20), (64, 8, 5), (128, 5, 150), (100, 16, 33), (None, 24, 70), (192, 32, 300)])
def test_layer_with_everything(tmp_path, ff, side, rows, dtype):
    """x <- x + mixer(norm x), x <- x + ff(norm x), then the token input (the test's rows all carry token 0), for steps of few and
    many rows and sizes the tensor-core contractions take and refuse."""
    layer = lightning(2, 16, 24, [0.5, 0.9])
    cfg = one_layer(layer, ff, side=side)
    d, W = make_model(tmp_path, cfg, 9)
    eng = engine_for(d, dtype)
    x = torch.randn(rows, 80, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
    y = mixer_alone(x, W, layer)
    mid = y
    if ff:
        y = y + pb.gated_ff(pb.rms_norm(y, W["l0.norm2"], EPS), W, "l0.mlp.")
    if side:
        y = pb.token_input(y, torch.zeros(rows, dtype=torch.long), W, "l0.side.", 0, side, EPS)
    want = y.numpy()
    got = eng.block_forward(0, [(eng.acquire(), rows)], f32(x))
    err = np.array([rel_err(got[r], want[r]) for r in range(rows)])
    assert (err > (2e-5 if dtype == "float32" else 5e-2)).sum() <= rows // 25, np.sort(err)[-5:]
    assert apart(got, mid.numpy()) > 1e-2            # what stands behind the mixer is there


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [3, 40, 200, 1100])
def test_token_input_at_a_real_width(rows, dtype):
    """x + norm(P (gelu(G x) * e)) at sizes where the gate contraction runs on few rows, split along a cluster, and split along K
    through scratch memory, with the table's entry in its epilogue."""
    from fastgguf_b200.parts import run_part
    E, V, D, layer, n_layers = 2048, 90, 136, 1, 3
    g = torch.Generator().manual_seed(41)
    Wb = {"side.embed": torch.randn(V, D * n_layers, generator=g), "gate": torch.randn(D, E, generator=g) / E ** 0.5 * 2.0,
          "proj": torch.randn(E, D, generator=g) / D ** 0.5, "norm": 1.0 + 0.3 * torch.randn(E, generator=g)}
    Wb = {k: v.to(torch.bfloat16) for k, v in Wb.items()}
    W = {("s." + k if k != "side.embed" else k): v.double() for k, v in Wb.items()}
    x = torch.randn(rows, E, generator=g, dtype=torch.float64)
    toks = [int(v) for v in torch.randint(0, V, (rows,), generator=g)]
    want = pb.token_input(x, torch.tensor(toks), W, "s.", layer, D, 1e-4).numpy()
    params = dict(hidden_size=E, vocab_size=V, dim=D, column=layer * D, table_dim=n_layers * D, eps=1e-4)
    got = run_part("token_input", "gated_token_embedding", params, {"table": Wb["side.embed"], "gate": Wb["gate"], "proj": Wb["proj"], "norm": Wb["norm"]},
                   dtype, tokens=toks, x=f32(x))
    for r in range(rows):
        assert rel_err(got[r], want[r]) < (1e-5 if dtype == "float32" else 2e-2), r


@pytest.mark.parametrize("dim,vdim", [(64, 64), (64, 128), (128, 64), (128, 128)])
def test_the_tensor_core_recurrence_keeps_float32(tmp_path, dim, vdim):
    """In bfloat16, with projections that bfloat16 holds exactly, what the chunked and the single-token forms return differs from the
    float64 recurrence over the SAME rounded activations by float32 rounding only: state, decays and weighted scores are not rounded
    to bfloat16 on the way.  (o times a norm and a gate of one is read off the stream, whose sum is float32.)"""
    H = 2
    layer = lightning(H, dim, vdim, [0.9, 0.999])
    E, V = 256, H * vdim
    cfg = one_layer(layer, width=E)

    def change(W):
        g = torch.Generator().manual_seed(2)
        W["l0.norm1"] = torch.ones_like(W["l0.norm1"])
        for n in ("q", "k", "v"):
            # one input a row, so that a projection is one product: exact in bfloat16 for inputs and weights that are powers of two
            w = torch.zeros_like(W["l0.mix." + n])
            w[torch.arange(w.shape[0]), torch.randint(0, E, (w.shape[0],), generator=g)] = 1.0
            W["l0.mix." + n] = w
        W["l0.mix.g"] = torch.zeros_like(W["l0.mix.g"])
        W["l0.mix.norm"] = torch.ones_like(W["l0.mix.norm"])
        W["l0.mix.o"] = torch.zeros_like(W["l0.mix.o"])
        W["l0.mix.o"][torch.arange(V) % E, torch.arange(V)] = 1.0
    d, W = make_model(tmp_path, cfg, 4, change=change)
    T = 200
    g = torch.Generator().manual_seed(3)
    x = torch.randint(0, 2, (T, E), generator=g).double() * 2.0 - 1.0            # rows of +-1: the norm leaves them (1 / sqrt(1 + eps))
    act = lambda z: pb.silu(z).to(torch.bfloat16).double()
    h = x.to(torch.bfloat16).double()
    q, k, v = (act(h @ W["l0.mix." + n].T).view(T, H, -1) for n in ("q", "k", "v"))
    o = pb.decayed_sums(q, k, v, torch.tensor([0.9, 0.999], dtype=torch.float64)).reshape(T, V)
    y = (pb.rms_norm(o, 1.0, EPS) * 0.5).to(torch.bfloat16).double()             # what the output projection reads
    want = (x + y @ W["l0.mix.o"].T).numpy()
    for cuts in ([T], [70, 2, 100] + [1] * 28):
        eng = engine_for(d, "bfloat16")
        s, at, got = eng.acquire(), 0, []
        for n in cuts:
            got.append(eng.block_forward(0, [(s, n)], f32(x[at:at + n])))
            at += n
        got = np.concatenate(got)
        # a bfloat16 rounding of y may fall to the other side of a tie; nearly every number agrees to float32
        same = np.abs(got - want) < 1e-5 * np.abs(want).max()
        assert same.mean() > 0.995, (cuts[:3], same.mean())
        assert np.abs(got - want).max() < 2.0 ** -7 * np.abs(want).max()


def test_the_relu_gate_shuts(tmp_path):
    """A feed-forward whose gate is negative for every row adds nothing; with the gate's sign turned it adds up times gate."""
    layer = lightning(1, 8, 8, [0.5])
    for sign in (-1.0, 1.0):
        cfg = one_layer(layer, 64)

        def change(W):
            W["l0.norm2"] = torch.ones_like(W["l0.norm2"])
            W["l0.mix.o"] = torch.zeros_like(W["l0.mix.o"])
            W["l0.mlp.gate"] = (sign * torch.ones_like(W["l0.mlp.gate"])) * W["l0.mlp.gate"].abs()
        d, W = make_model(tmp_path / str(sign), cfg, 3, change=change)
        x = torch.rand(9, 80, generator=torch.Generator().manual_seed(1), dtype=torch.float64) + 0.1
        got = engine_for(d, "float32")
        got = got.block_forward(0, [(got.acquire(), 9)], f32(x))
        want = x + pb.gated_ff(pb.rms_norm(x, W["l0.norm2"], EPS), W, "l0.mlp.")
        assert rel_err(got, want.numpy()) < 1e-6
        assert bool((want == x).all()) == (sign < 0)


def test_the_second_map_is_subtracted_with_its_weight(tmp_path):
    """The four vectors behind lambda made so that it is 0, 0.5 or 2 (and the constant taken into account): each gives another
    output, the engine's follow the plain ones, and with lambda 0 the second map's projections do not matter."""
    layer = differential(2, 1, 8, 16, 0.5, 0.25, size=12, rot=(100.0, 8))
    outs = {}
    for lam in (0.0, 0.5, 2.0):
        cfg = one_layer(layer)

        def change(W):
            for n in ("lq1", "lk1", "lq2", "lk2"):
                W["l0.mix." + n] = torch.zeros_like(W["l0.mix." + n])
            want_exp = lam - 0.25 + 1.0                       # exp(lq1 . lk1), the other exponential being one
            W["l0.mix.lq1"][3] = 1.0
            W["l0.mix.lk1"][3] = float(np.log(want_exp))
        d, W = make_model(tmp_path / str(lam), cfg, 5, sharp=2.0, change=change)
        assert abs(float(pb.map_weight(W, "l0.mix.", 0.25)) - lam) < 2e-2
        x = torch.randn(30, 80, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
        eng = engine_for(d, "float32")
        got = eng.block_forward(0, [(eng.acquire(), 30)], f32(x))
        assert rel_err(got, mixer_alone(x, W, layer).numpy()) < 1e-5
        outs[lam] = got
    assert apart(outs[0.0], outs[0.5]) > 1e-2 and apart(outs[0.5], outs[2.0]) > 1e-2


def test_sinks_take_their_share(tmp_path):
    """Sinks far above every score leave almost nothing of the values, sinks far below change nothing, one per head."""
    layer = keys_as_values(2, 1, 16, 0.25, size=10)
    x = torch.randn(25, 80, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
    moved = {}
    for value in (-30.0, 0.0, 12.0):
        cfg = one_layer(layer)

        def change(W):
            W["l0.mix.sink"] = torch.tensor([value, -30.0], dtype=torch.bfloat16)
        d, W = make_model(tmp_path / str(value), cfg, 5, change=change)
        want = mixer_alone(x, W, layer).numpy()
        for dtype, tol in (("float32", 1e-5), ("bfloat16", 3e-2)):
            eng = engine_for(d, dtype)
            s = eng.acquire()
            got = np.concatenate([eng.block_forward(0, [(s, n)], f32(x[a:a + n])) for a, n in ((0, 20), (20, 2), (22, 1), (23, 1), (24, 1))])
            assert rel_err(got, want) < tol, (value, dtype)
        moved[value] = want
    assert apart(moved[0.0], moved[-30.0]) > 1e-2 and apart(moved[12.0], moved[0.0]) > 1e-2


def test_frequencies():
    """The rotation tables of both kinds of scaling against the plain implementation's frequencies."""
    from fastgguf_b200.registry import config_from_dict
    from fastgguf_b200.parts import position_tables
    case, positions = CASES["a"], np.arange(50)
    for layer, freq in ((case["layers"][0], pb.linear_frequencies), (case["layers"][1], pb.banded_frequencies), (case["layers"][3], pb.linear_frequencies)):
        rot = layer["mixer"]["rot"]
        f = freq(rot["base"], rot["dims"], rot.get("scaling")).numpy()
        part = next(l["mixer"]["params"]["position"] for l, src in zip(config_from_dict(case).spec_json()["layers"], case["layers"]) if src is layer)
        cos, sin, _ = position_tables("rope", part["params"], len(positions))
        ang = positions[:, None] * f[None, :]
        assert np.abs(cos[:, :len(f)] - np.cos(ang)).max() < 1e-6 and np.abs(sin[:, :len(f)] - np.sin(ang)).max() < 1e-6


# ------------------------------------------------------------------------------ windows, edges, far keys
def standout_model(tmp_path, layer, seed=11):
    """Weights made so that ONE key far outweighs all others for the rows that ask for it: keys are the queries' map of the row
    shifted back by one column, nothing is biased or rotated (and, with two maps, the second one is flat)."""
    cfg = one_layer(layer)
    W = random_weights(cfg, seed)
    m, p = layer["mixer"], "l0.mix."
    d, per = m["dim"], 2 if layer["type"] == "attention" else 1
    k = torch.randn(d, 80, generator=torch.Generator().manual_seed(1)) / 80 ** 0.5
    head = torch.cat([k] + [torch.zeros(d, 80)] * (per - 1))
    W[p + "q"] = head.repeat(m["heads"], 1).to(torch.bfloat16)
    W[p + "k"] = torch.roll(head, 1, dims=1).repeat(m["kv_heads"], 1).to(torch.bfloat16)
    for n in ("q.b", "k.b", "v.b"):
        if p + n in W:
            W[p + n] = torch.zeros_like(W[p + n])
    for n in ("l0.norm1", p + "q.norm", p + "k.norm"):
        if n in W:
            W[n] = torch.ones_like(W[n])
    if p + "sink" in W:
        W[p + "sink"] = torch.full_like(W[p + "sink"], -5.0)
    path = write_model(tmp_path, cfg, W)
    return path, {n: v.double() for n, v in W.items()}


WINDOWED = {
    "two maps, small": (lambda w: differential(4, 2, 24, 20, 1.0, 0.4, size=w), 6),
    "two maps, keys of 64 beside values of 128": (lambda w: differential(4, 2, 64, 128, 0.4, 0.4, size=w), 65),
    "two maps, 64 and 64": (lambda w: differential(2, 2, 64, 64, 0.4, 0.4, size=w), 100),
    "two maps, no window": (lambda w: differential(2, 1, 64, 128, 0.4, 0.4), None),
    "keys as values, small": (lambda w: keys_as_values(3, 1, 24, 1.0, size=w), 17),
    "keys as values, 128": (lambda w: keys_as_values(6, 2, 128, 0.2, size=w), 64),
    "keys as values, 64": (lambda w: keys_as_values(2, 2, 64, 0.4, size=w), 63),
    "keys as values, no window": (lambda w: keys_as_values(4, 2, 128, 0.2), None),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("special", [0, 1, 63, 64, 200])
@pytest.mark.parametrize("name", list(WINDOWED))
def test_one_key_stands_out_until_it_leaves_the_window(tmp_path, name, special, dtype):
    """One row's key far outweighs all others for every later row that sees it.  The rows inside the window return its value, the
    last of them too; the first one outside does not, nor any behind it - in a prompt, and decoded one by one from just behind the
    special row, and from inside the window on, past its edge and past pages' borders."""
    make, window = WINDOWED[name]
    layer = make(window)
    T = special + 140
    path, W = standout_model(tmp_path, layer)
    g = torch.Generator().manual_seed(3)
    rows = torch.randn(T, 80, generator=g, dtype=torch.float64)
    asked = torch.randn(80, generator=g, dtype=torch.float64)
    x = rows.clone()
    x[special] = torch.roll(asked, 1)
    x[special + 1:] = asked[None, :] + 0.1 * rows[special + 1:]
    other = x.clone()
    other[special] = rows[special]
    want, without = mixer_alone(x, W, layer).numpy(), mixer_alone(other, W, layer).numpy()
    moved = np.abs(want - without).max(1) / np.abs(want - x.numpy()).max(1)
    last_in = T - 1 if window is None else min(T - 1, special + window - 1)
    assert (moved[special + 1:last_in + 1] > 0.2).all() and (moved[last_in + 1:] < 1e-9).all()        # the window shows in the oracle
    for cuts in ([T], [special + 1] + [1] * (T - special - 1), [special + 50, 7, 2, 2] + [1] * (T - special - 61)):
        eng = engine_for(path, dtype)
        slot, at, got = eng.acquire(), 0, []
        for n in cuts:
            got.append(eng.block_forward(0, [(slot, n)], f32(x[at:at + n])))
            at += n
        got = np.concatenate(got)
        tol = 2e-5 if dtype == "float32" else 8e-2
        bad = [(r, rel_err(got[r], want[r])) for r in range(T) if rel_err(got[r], want[r]) > tol]
        assert len(bad) <= (0 if dtype == "float32" else T // 40), (name, special, len(cuts), bad[:8])


def test_a_head_that_never_forgets_carries_one_token(tmp_path):
    """One early row differs between two inputs of 300 rows: through decays of 1 and 0.999 the last rows differ by far more than
    rounding, in the engine exactly as in the plain implementation; through a decay of 0.5 they do not."""
    for decay, stays in (([1.0, 0.999], True), ([0.5, 0.0], False)):
        layer = lightning(2, 16, 20, decay)
        d, W = make_model(tmp_path / str(stays), one_layer(layer), 60)
        g = torch.Generator().manual_seed(4)
        xa = torch.randn(300, 80, generator=g, dtype=torch.float64)
        xb = xa.clone()
        xb[3] = 3.0 * torch.randn(80, generator=g, dtype=torch.float64)
        eng = engine_for(d, "float32")
        last = []
        for x in (xa, xb):
            want = mixer_alone(x, W, layer).numpy()
            s = eng.acquire()
            got = np.concatenate([eng.block_forward(0, [(s, n)], f32(x[a:a + n])) for a, n in ((0, 2), (2, 198), (200, 99), (299, 1))])
            eng.release(s)
            assert rel_err(got[-1], want[-1]) < 2e-5
            last.append(got[-1] - x[-1].numpy())
        moved = np.abs(last[0] - last[1]).max() / np.abs(last[0]).max()
        assert moved > 1e-4 if stays else moved < 1e-5, (decay, moved)


# ------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(CASES))
def test_whole_prompt(models, which, dtype):
    """Logits at every position of a prompt that passes pages, windows and the recurrence's chunks."""
    d, cfg, W = models[(which, dtype)]
    toks = tokens_for(cfg, 200, 12)
    want = plain_logits(cfg, W, toks)
    eng = engine_for(d, dtype)
    s = eng.acquire()
    got = eng.step_host([entry(s, toks)])
    judge = Rows(dtype)
    for p in range(len(toks)):
        judge.add(got[p], want[p], (which, p))
    judge.done()
    eng.release(s)
    eng.cache.check()


def test_the_first_tokens(models):
    """Sequences of one, two, three and five tokens, as a prompt and one by one: states start at zero, windows hold what there is."""
    for which in CASES:
        d, cfg, W = models[(which, "float32")]
        eng = engine_for(d, "float32")
        for n in (1, 2, 3, 5):
            toks = tokens_for(cfg, n, 30 + n)
            want = plain_logits(cfg, W, toks)
            s = eng.acquire()
            judge = Rows("float32")
            for p, row in enumerate(eng.step_host([entry(s, toks)])):
                judge.add(row, want[p], (which, n, p))
            eng.release(s)
            s = eng.acquire()
            for p, t in enumerate(toks):
                judge.add(eng.step_host([entry(s, [t])])[0], want[p], (which, n, p, "alone"))
            judge.done()
            eng.release(s)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which,cuts", [("a", [2, 2, 3, 17, 33, 64, 65, 2, 31]), ("b", [63, 2, 64, 1, 1, 70, 2, 16]),
                                        ("c", [100, 28, 1, 2, 64, 24]), ("d", [3, 2, 40, 2]), ("e", [31, 2, 32, 16, 15])])
def test_portions_and_decoding(models, which, cuts, dtype):
    """A prompt cut into portions of many sizes, down to two tokens and one, then 40 tokens one by one: the same logits
    as the whole sequence at every position."""
    d, cfg, W = models[(which, dtype)]
    toks = tokens_for(cfg, sum(cuts) + 40, 13)
    want = plain_logits(cfg, W, toks)
    eng = engine_for(d, dtype)
    s = eng.acquire()
    at = 0
    judge = Rows(dtype)
    for c in cuts + [1] * 40:
        got = eng.step_host([entry(s, toks[at:at + c])])
        for i in range(c):
            judge.add(got[i], want[at + i], (which, at + i, c))
        at += c
    judge.done()
    eng.release(s)
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(CASES))
def test_batch_of_unequal_requests(models, which, dtype):
    """Five requests of 1 to 140 tokens in one step, then decoded together while the shorter ones leave: every
    request's logits equal those it has alone."""
    d, cfg, W = models[(which, dtype)]
    lens, total = [1, 140, 64, 7, 65], [9, 150, 70, 30, 66]
    toks = [tokens_for(cfg, t, 20 + i) for i, t in enumerate(total)]
    want = [plain_logits(cfg, W, t) for t in toks]
    eng = engine_for(d, dtype)
    slots = [eng.acquire() for _ in toks]
    got = eng.step_host([entry(s, t[:n]) for s, t, n in zip(slots, toks, lens)])
    row = 0
    judge = Rows(dtype)
    for b, n in enumerate(lens):
        for p in range(n):
            judge.add(got[row], want[b][p], (which, b, p))
            row += 1
    at = list(lens)
    alive = list(range(len(toks)))
    while alive:
        got = eng.step_host([entry(slots[b], [toks[b][at[b]]]) for b in alive])
        for i, b in enumerate(alive):
            judge.add(got[i], want[b][at[b]], (which, b, at[b]))
            at[b] += 1
        for b in [b for b in alive if at[b] == total[b]]:
            eng.release(slots[b])
            alive.remove(b)
    judge.done()
    eng.cache.check()
    assert eng.cache.live_slots() == []


@pytest.mark.parametrize("which", ["a", "b"])
def test_portions_beside_decoding(models, which):
    """Steps in which one request is decoded while another brings a portion of its prompt and a third starts."""
    d, cfg, W = models[(which, "float32")]
    toks = [tokens_for(cfg, n, 120 + i) for i, n in enumerate((90, 150, 60))]
    want = [plain_logits(cfg, W, t) for t in toks]
    eng = engine_for(d, "float32")
    slots = [eng.acquire() for _ in toks]
    plan = [{0: 70}, {0: 1, 1: 50}, {0: 1, 1: 2, 2: 31}, {0: 1, 1: 66, 2: 1}, {1: 1, 2: 5}, {0: 4, 1: 20, 2: 1}]
    at = [0, 0, 0]
    judge = Rows("float32")
    for step in plan:
        got = eng.step_host([entry(slots[b], toks[b][at[b]:at[b] + n]) for b, n in step.items()])
        row = 0
        for b, n in step.items():
            for i in range(n):
                judge.add(got[row], want[b][at[b] + i], (which, b, at[b] + i))
                row += 1
            at[b] += n
    judge.done()
    eng.cache.check()


def test_slots_and_pages_used_again(models):
    """Sequences come and go in a cache of two slots and few pages: a new sequence starts from nothing (state rows are cleared,
    pages of the one before are not read), also after a sequence that was released halfway."""
    for which in ("a", "b"):
        d, cfg, W = models[(which, "float32")]
        eng = engine_for(d, "float32", max_tokens=512, max_batch=2)
        seqs = [tokens_for(cfg, n, 40 + i) for i, n in enumerate([200, 130, 90, 260, 70])]
        judge = Rows("float32")
        for k, toks in enumerate(seqs):
            s = eng.acquire()
            other = eng.acquire()
            eng.step_host([entry(other, seqs[(k + 1) % len(seqs)][:50], [])])       # a neighbour that is dropped halfway
            want = plain_logits(cfg, W, toks)
            head = len(toks) - 20
            got = eng.step_host([entry(s, toks[:head], [head - 1])])
            judge.add(got[0], want[head - 1], (which, k))
            eng.release(other)
            for p in range(head, len(toks)):
                judge.add(eng.step_host([entry(s, [toks[p]])])[0], want[p], (which, k, p))
            eng.release(s)
            eng.cache.check()
        judge.done()


def test_long_decoding_past_windows_and_pages(models):
    """300 tokens one by one after a short prompt: pages fill up and leave the windows, the recurrent states carry the first tokens
    all along."""
    for which in ("a", "b"):
        d, cfg, W = models[(which, "float32")]
        toks = tokens_for(cfg, 330, 50)
        want = plain_logits(cfg, W, toks)
        eng = engine_for(d, "float32")
        s = eng.acquire()
        eng.step_host([entry(s, toks[:30], [])])
        judge = Rows("float32")
        for p in range(30, 330):
            judge.add(eng.step_host([entry(s, [toks[p]])])[0], want[p], (which, p))
        judge.done()
        eng.release(s)
        eng.cache.check()


def test_each_pass_of_the_loop_has_its_vector(tmp_path):
    """The vectors added in front of the passes: swapping two of them changes the logits (they are used in order), with a token input in
    front of a pass (whose last kernel adds the vector) and without one."""
    for side in (None, 8):
        layers = [(lightning(2, 8, 8, [0.9, 0.5]), None), (differential(2, 1, 8, 12, 0.4, 0.3, size=6, rot=(100.0, 8)), 24)]
        cfg = config(64, 70, layers, loop=(0, 2, 3), side=side)
        toks = tokens_for(cfg, 40, 2)
        outs = []
        for swap in (False, True):
            def change(W):
                if swap:
                    W["loop.step"] = W["loop.step"][[1, 0, 2]].contiguous()
            d, W = make_model(tmp_path / f"{side}{swap}", cfg, 21, change=change)
            for dtype in ("float32", "bfloat16"):
                eng = engine_for(d, dtype)
                s = eng.acquire()
                got = np.concatenate([eng.step_host([entry(s, toks[:30])])] + [eng.step_host([entry(s, [t])]) for t in toks[30:]])
                want = plain_logits(cfg, W, toks)
                judge = Rows(dtype)
                for p in range(40):
                    judge.add(got[p], want[p], (side, swap, p))
                judge.done()
            outs.append(want)
        assert apart(outs[0], outs[1]) > 1e-2


def test_many_steps_back_to_back():
    """Ninety prompt steps of drawn shapes - one to three sequences of 2 to 2,048 tokens, every third step a prompt of 2,048 - each
    followed by three decode steps, at sizes where every contraction and attention runs on the tensor cores and the row-wise kernels
    between them are short against them: every step ends with finite logits, and a repeated prompt gives the same logits."""
    from fastgguf_b200.engine.api import Engine
    from fastgguf_b200.registry import config_from_dict
    cfg = config(1024, 4096, [
        (differential(8, 4, 64, 128, 0.125, 0.5, size=512, rot=(10000.0, 32), scaling=(2.0,)), 4096),
        (keys_as_values(8, 2, 128, 0.09, size=700, rot=(200000.0, 64), scaling=(16.0, 1.0, 3.0, 2048)), 4096),
        (lightning(8, 128, 128, [0.5, 0.8, 0.9, 0.95, 0.98, 0.99, 0.995, 0.999]), 4096),
        (lightning(8, 64, 128, [0.5, 0.8, 0.9, 0.95, 0.98, 0.99, 0.995, 0.999]), None),
    ], loop=(0, 4, 2), side=256)
    eng = Engine.from_random(config_from_dict(cfg), 3, dtype="bfloat16", max_tokens=8192, max_batch=4, max_seq_len=4096)
    rng = np.random.default_rng(5)
    fixed = tokens_for(cfg, 2048, 90)
    first = None
    for i in range(90):
        n_seq = int(rng.integers(1, 4))
        lens = [2048] if i % 3 == 0 else [int(rng.integers(2, 2049)) for _ in range(n_seq)]
        slots = [eng.acquire() for _ in lens]
        toks = [fixed if n == 2048 and i % 3 == 0 else tokens_for(cfg, n, 1000 + 7 * i + k) for k, n in enumerate(lens)]
        got = eng.step_host([entry(s, t, [len(t) - 1]) for s, t in zip(slots, toks)])
        assert np.isfinite(got).all()
        if i % 3 == 0:
            first = got if first is None else first
            assert np.array_equal(got, first)
        for _ in range(3):
            assert np.isfinite(eng.step_host([entry(s, [int(rng.integers(0, 4096))]) for s in slots])).all()
        for s in slots:
            eng.release(s)
    eng.check_device()
    eng.cache.check()


# ------------------------------------------------------------------------------ generation through the entry point
@pytest.mark.parametrize("use_graphs", [False, True])
@pytest.mark.parametrize("which", ["a", "b", "c"])
def test_greedy_generation(models, which, use_graphs):
    """Greedy decoding through Engine.generate - the scheduler's batches, the recorded decode step, slots that come
    back - follows the plain implementation: each token is the plain logits' best given the tokens before it (where the
    best two are closer than rounding, either counts)."""
    d, cfg, W = models[(which, "float32")]
    prompts = [tokens_for(cfg, n, 70 + i) for i, n in enumerate([5, 70, 1, 33, 12])]
    eng = engine_for(d, "float32", max_tokens=2048, max_batch=4, use_graphs=use_graphs)
    out = eng.generate(prompts, temp=0, max_tokens=24, ignore_eos=True, batch_size=3)
    for p, c in zip(prompts, out):
        assert len(c.tokens) == 24
        logits = plain_logits(cfg, W, p + c.tokens)
        for i, t in enumerate(c.tokens):
            row = logits[len(p) + i - 1]
            assert row[t] >= row.max() - 2e-4 * np.abs(row).max(), (which, i)
    eng.cache.check()
    assert eng.cache.live_slots() == []


def test_generation_in_bfloat16_runs_the_recorded_step(models):
    d, cfg, W = models[("b", "bfloat16")]
    prompts = [tokens_for(cfg, n, 80 + i) for i, n in enumerate([9, 40])]
    eng = engine_for(d, "bfloat16", max_tokens=1024, max_batch=2)
    out = eng.generate(prompts, temp=0, max_tokens=70, ignore_eos=True)
    for p, c in zip(prompts, out):
        logits = plain_logits(cfg, W, p + c.tokens)
        close = sum(logits[len(p) + i - 1][t] >= logits[len(p) + i - 1].max() - 0.05 * np.abs(logits[len(p) + i - 1]).max()
                    for i, t in enumerate(c.tokens))
        assert close >= 0.9 * len(c.tokens)
    eng.cache.check()


@pytest.mark.parametrize("which", ["a", "b"])
def test_trace_replay_three_cuts(tmp_path, models, which):
    """``bin/trace_run`` on a Buguzen folder in true 32-bit: the same requests whole, with their last 32 tokens one by one, and
    in batches of four unequal requests one batch after another (slots and pages are used again); a cache that holds just what
    the live requests need."""
    from trace_tools import batched_trace, collect, run_trace, tail_trace, whole_trace
    d, cfg, W = models[(which, "float32")]
    lengths = [5, 9, 1, 17, 3, 40, 11, 70, 33, 130]
    requests = {f"r{i}": tokens_for(cfg, n, 100 + i) for i, n in enumerate(lengths)}
    want = {rid: plain_logits(cfg, W, toks) for rid, toks in requests.items()}
    need = max(sum((len(requests[r]) + 63) // 64 * 64 for r in list(requests)[b:b + 4]) for b in range(0, 10, 4))
    for name, (steps, index), room in (("whole", whole_trace(requests), 192), ("tail", tail_trace(requests, 32), 192),
                                       ("batched", batched_trace(requests, 4), need)):
        run_trace(d, "float32", steps, str(tmp_path / name), max_tokens=room)
        rows = collect(str(tmp_path / name), steps, index, cfg["vocab"])
        assert len(rows) == sum(lengths), name
        judge = Rows("float32")
        for (rid, pos), row in rows.items():
            judge.add(row, want[rid][pos], (name, rid, pos))
        judge.done()


def test_command_line_generates(models):
    """``python -m fastgguf_b200 generate`` on a Buguzen folder: the model class comes from config.json, the tokens are
    those of Engine.generate."""
    d, cfg, W = models[("a", "float32")]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([sys.executable, "-m", "fastgguf_b200", "generate", d, "256", "--prompt", "5,17,3,200", "--prompt", "9",
                        "--temp", "0", "--max-tokens", "6", "--ignore-eos", "--dtype", "float32", "--json"],
                       cwd=root, capture_output=True, text=True)
    assert p.returncode == 0, p.stderr
    got = [r["tokens"] for r in json.loads(p.stdout)]
    eng = engine_for(d, "float32", max_tokens=512, max_batch=2)
    want = [c.tokens for c in eng.generate([[5, 17, 3, 200], [9]], temp=0, max_tokens=6, ignore_eos=True)]
    assert got == want
