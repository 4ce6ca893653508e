"""The Zifelorn decoder in the engine against the plain implementation (``plain_zifelorn``): each mechanism alone, whole
prompts, portions, decoding, batches, reused slots and pages, and generation through the entry point.

Structure is tested in float32, where any key wrongly seen or missed, any state lost or kept too long is orders of
magnitude above the tolerance; the bfloat16 runs use sharpened attention and routers (see ``zifelorn_cases.random_weights``)
so that the same faults stay visible above rounding."""
import copy

import numpy as np
import pytest
import torch

import plain_zifelorn as pz
from helpers import rel_err
from zifelorn_cases import CASES, config, dense, latent, make_model, moe, random_weights, rglru, write_model

pytestmark = pytest.mark.gpu

#: max |dlogit| / max |logit| against the float64 plain implementation.  float32: a key wrongly seen or a lost state is at 1e-3
#: and above.  bfloat16 with sharpened attention: rounding reaches a few 1e-2, a structural fault 0.3 and more
TOL = {"float32": 2e-5, "bfloat16": 1e-1}
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
    return pz.forward(cfg, W, toks).numpy()


def f32(x):
    return np.ascontiguousarray(x.numpy() if hasattr(x, "numpy") else x, dtype=np.float32)


class Rows:
    """Collects the errors of a whole model's logits, row by row, and judges them.

    Every sublayer's output is normalised whatever its size, so where one returns little every rounding in it is amplified; and
    in bfloat16 rounding may decide between two experts or two keys that compete closely.  At most one row in fifty (or one row)
    may exceed the tolerance in float32, where none may exceed three times the tolerance; one in fifteen in bfloat16.  A key
    wrongly seen or a lost state moves most rows by far more."""

    def __init__(self, dtype):
        self.dtype, self.n, self.over = dtype, 0, []

    def add(self, got, want, what):
        e = rel_err(got, want)
        self.n += 1
        assert np.isfinite(e) and (self.dtype == "bfloat16" or e < 3 * TOL[self.dtype]), (what, e)
        if e >= TOL[self.dtype]:
            self.over.append((what, e))

    def done(self):
        assert len(self.over) <= max(1, self.n // (15 if self.dtype == "bfloat16" else 50)), (len(self.over), self.n, self.over[:20])


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """(case, dtype): for bfloat16 attention and routers are sharpened, and where a row uses one expert it uses two (rounding
    that decides between two experts for a row's only choice changes all of what the row gets)"""
    out = {}
    for i, (name, case) in enumerate(CASES.items()):
        for dtype, sharp, router in (("float32", 1.0, 1.0), ("bfloat16", 1.5, 3.0)):
            cfg = copy.deepcopy(case)
            for layer in cfg["layers"]:
                if dtype == "bfloat16" and (layer["mlp"] or {}).get("kind") == "moe":
                    layer["mlp"]["router"]["top"] = max(2, layer["mlp"]["router"]["top"])
            d, W = make_model(tmp_path_factory.mktemp(f"z_{name}_{dtype}"), cfg, 100 + i, sharp, router=router)
            out[(name, dtype)] = (d, cfg, W)
    return out


# ------------------------------------------------------------------------------ mechanisms alone
MIXERS = {
    "latent attention, small": latent(3, 16, 8, 24, 40, 48, 0.2, 10000.0),
    "latent attention, one head, sizes that are no multiples of four": latent(1, 9, 6, 7, 13, 21, 0.3, 500.0),
    "latent attention, latent of 64, rotated part of 16 (tensor cores in decode)": latent(5, 24, 16, 40, 64, 32, 0.2, 3000.0),
    "rglru, small": rglru(72, 3, 4),
    "rglru, one block, one tap": rglru(60, 1, 1),
    "rglru, blocks of one channel": rglru(24, 24, 2),
    "rglru, blocks of seven, five taps": rglru(35, 5, 5),
    "rglru, more taps than a portion has tokens": rglru(48, 2, 7),
    "long latent attention, latent of 128, heads of 128 for whole prompts": latent(3, 96, 32, 128, 128, 80, 0.09, 50000.0),
    "long latent attention, heads of 64, values of 32": latent(4, 32, 32, 32, 192, 64, 0.12, 100.0),
    "long rglru, blocks of 128, four taps": rglru(256, 2, 4),
    "long rglru, blocks of 8 and two taps": rglru(104, 13, 2),
    "long rglru, one block of 320": rglru(320, 1, 3),
}


def mixer_alone(x, W, layer, eps=EPS):
    """what one layer without a feed-forward makes of the rows x"""
    if layer["type"] == "latent_attention":
        m = layer["mixer"]
        y = pz.latent_attention(x, W, "l0.mix.", m, eps, pz.latent_kv(x, W, "l0.mix.", m, eps))
    else:
        y = pz.recurrent_block(x, W, "l0.mix.")
    return x + pz.rms_norm(y, W["l0.norm1"], eps)


def one_layer(layer, mlp=None, width=80, vocab=50):
    return config(width, vocab, [(layer, mlp)], eps=EPS)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MIXERS))
def test_mixer_alone(tmp_path, name, dtype):
    """One layer of a mixer alone (mixer, norm, residual add) on rows given by the test: a portion of 37 rows, then one of 2,
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
    tol = 2e-5 if dtype == "float32" else 5e-2
    for r in range(T):
        assert rel_err(got[r], want[r]) < tol, (name, r)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["long rglru, blocks of 128, four taps", "rglru, blocks of seven, five taps",
                                  "long latent attention, latent of 128, heads of 128 for whole prompts"])
def test_a_wide_batch_of_prompts(tmp_path, name, dtype):
    """Prompts of 1,300, 300, 50 and 3 tokens in one step (the recurrence then walks two rounds of its cluster for the longest,
    part of one for the others), then one more token each, then a portion of 5 for the last."""
    layer = MIXERS[name]
    cfg = one_layer(layer)
    d, W = make_model(tmp_path, cfg, 12, sharp=1.5, lam=-2.0)
    eng = engine_for(d, dtype, max_tokens=4096, max_batch=4)
    g = torch.Generator().manual_seed(9)
    lens = [1300, 300, 50, 3]
    xs = [torch.randn(n + 6, cfg["width"], generator=g, dtype=torch.float64) for n in lens]
    want = [mixer_alone(x, W, layer).numpy() for x in xs]
    tol = 2e-5 if dtype == "float32" else 5e-2
    slots = [eng.acquire() for _ in lens]
    got = eng.block_forward(0, list(zip(slots, lens)), f32(torch.cat([x[:n] for x, n in zip(xs, lens)])))
    at = 0
    for b, n in enumerate(lens):
        for r in sorted({0, 1, 2, n // 2, n - 2, n - 1} | {p for p in (15, 16, 127, 128, 255, 256, 1023, 1024, 1025) if p < n}):
            assert rel_err(got[at + r], want[b][r]) < tol, (name, b, r)
        at += n
    got = eng.block_forward(0, [(s, 1) for s in slots], f32(torch.stack([x[n] for x, n in zip(xs, lens)])))
    for b, n in enumerate(lens):
        assert rel_err(got[b], want[b][n]) < tol, (name, b, "decoded")
    got = eng.block_forward(0, [(slots[3], 5)], f32(xs[3][4:9]))
    for i in range(5):
        assert rel_err(got[i], want[3][4 + i]) < tol, (name, "portion", i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_more_sequences_than_a_block_serves(tmp_path, dtype):
    """Nineteen sequences decoded together: the single-token kernel takes eight rows a block, the last block is not full."""
    layer = rglru(96, 4, 3)
    cfg = one_layer(layer)
    d, W = make_model(tmp_path, cfg, 13)
    eng = engine_for(d, dtype, max_tokens=4096, max_batch=19)
    g = torch.Generator().manual_seed(3)
    xs = [torch.randn(4, cfg["width"], generator=g, dtype=torch.float64) for _ in range(19)]
    want = [mixer_alone(x, W, layer).numpy() for x in xs]
    slots = [eng.acquire() for _ in xs]
    for t in range(4):
        got = eng.block_forward(0, [(s, 1) for s in slots], f32(torch.stack([x[t] for x in xs])))
        for b in range(19):
            assert rel_err(got[b], want[b][t]) < (1e-5 if dtype == "float32" else 3e-2), (b, t)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mlp,rows", [(dense(56), 20), (dense(64), 20), (dense(128), 150), (moe(40, 6, 2), 5), (moe(40, 6, 2), 33), (moe(48, 8, 3), 150),
                                      (moe(24, 5, 5), 12), (moe(20, 7, 1), 40), (moe(36, 3, 2), 200)],
                         ids=lambda v: str(v) if isinstance(v, int) else v["kind"] + str(v.get("ff") or (v["expert"]["ff"], *v["router"].values())))
def test_layer_with_both_sublayers(tmp_path, mlp, rows, dtype):
    """x <- x + norm(mixer(x)), then x <- x + norm(ff(x)), for feed-forwards of several sizes and steps of few and many rows
    (experts on the row kernels, on tiles, and grouped on the tensor cores)."""
    layer = rglru(24, 3, 2)
    cfg = one_layer(layer, mlp)
    d, W = make_model(tmp_path, cfg, 9, router=3.0)
    eng = engine_for(d, dtype)
    x = torch.randn(rows, 80, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
    mid = mixer_alone(x, W, layer)
    ff = pz.dense_ff(mid, W, "l0.mlp.") if mlp["kind"] == "dense" else pz.experts_ff(mid, W, "l0.mlp.", mlp)
    want = (mid + pz.rms_norm(ff, W["l0.norm2"], EPS)).numpy()
    got = eng.block_forward(0, [(eng.acquire(), rows)], f32(x))
    err = np.array([rel_err(got[r], want[r]) for r in range(rows)])
    if dtype == "float32":
        assert err.max() < 2e-5
    else:          # (rounding may decide between two experts at a rare row)
        assert (err > 4e-2).sum() <= rows // 25, np.sort(err)[-5:]
    assert rel_err(got, mid.numpy()) > 1e-2            # the feed-forward is there


def test_the_router_weighs_the_chosen_logits_alone(tmp_path):
    """A router whose logits come from its bias alone, far apart: rows use the experts of the two largest, with weights that sum
    to one over those two; a softmax over all experts, or a bias left out of the choice or the weights, gives something else."""
    cfg = one_layer(rglru(24, 3, 2), moe(40, 4, 2))

    def change(W):
        W["l0.mlp.router"] = torch.zeros_like(W["l0.mlp.router"])
        W["l0.mlp.router.b"] = torch.tensor([0.5, 2.0, -1.0, 1.0], dtype=torch.bfloat16)
    d, W = make_model(tmp_path, cfg, 14, change=change)
    x = torch.randn(9, 80, generator=torch.Generator().manual_seed(6), dtype=torch.float64)
    mid = mixer_alone(x, W, {"type": "rglru", "mixer": cfg["layers"][0]["mixer"]})

    def with_weights(w):
        y = sum(wk * (torch.clamp(mid @ W[f"l0.mlp.e{e}.up"].T, min=0.0) ** 2 @ W[f"l0.mlp.e{e}.down"].T) for e, wk in w.items())
        return (mid + pz.rms_norm(y, W["l0.norm2"], EPS)).numpy()
    p = 1.0 / (1.0 + np.exp(-1.0))                    # softmax of (2, 1)
    want = with_weights({1: p, 3: 1.0 - p})
    assert rel_err(with_weights({1: 0.5, 3: 0.5}), want) > 1e-2 and rel_err(with_weights({0: p, 1: 1.0 - p}), want) > 1e-2
    eng = engine_for(d, "float32")
    assert rel_err(eng.block_forward(0, [(eng.acquire(), 9)], f32(x)), want) < 1e-5


def test_recurrence_where_decay_is_close_to_one_and_to_zero(tmp_path):
    """lam far below zero: a is within 1e-6 of one and sqrt(1 - a^2) must not be the root of a cancelled difference; lam large:
    the state is almost the input.  The float32 engine follows the float64 equations in a prompt and decoded."""
    for lam, name in ((-12.0, "slow"), (6.0, "fast")):
        layer = rglru(48, 4, 3)
        cfg = one_layer(layer)
        d, W = make_model(tmp_path / name, cfg, 15, lam=lam)
        a_typical = torch.exp(-8.0 * 0.5 * pz.softplus(W["l0.mix.lam"]))
        assert bool((a_typical > 0.99).any()) if name == "slow" else bool((a_typical < 1e-3).all())
        x = torch.randn(90, 80, generator=torch.Generator().manual_seed(2), dtype=torch.float64)
        want = mixer_alone(x, W, layer).numpy()
        eng = engine_for(d, "float32")
        s = eng.acquire()
        got = np.concatenate([eng.block_forward(0, [(s, n)], f32(x[a:a + n])) for a, n in [(0, 60), (60, 20)] + [(80 + i, 1) for i in range(10)]])
        for r in range(90):
            assert rel_err(got[r], want[r]) < 2e-5, (name, r)


def test_a_state_that_forgets_slowly_carries_one_token(tmp_path):
    """One early row differs between two inputs of 300 rows: through the slowly decaying state the last rows differ by far more
    than rounding, in the engine exactly as in the plain implementation, in a prompt and across portions."""
    layer = rglru(40, 2, 3)
    cfg = one_layer(layer)
    d, W = make_model(tmp_path, cfg, 60, lam=-7.0)
    g = torch.Generator().manual_seed(4)
    xa = torch.randn(300, 80, generator=g, dtype=torch.float64)
    xb = xa.clone()
    xb[3] = torch.randn(80, generator=g, dtype=torch.float64)
    eng = engine_for(d, "float32")
    last = []
    for x in (xa, xb):
        want = mixer_alone(x, W, layer).numpy()
        s = eng.acquire()
        got = np.concatenate([eng.block_forward(0, [(s, n)], f32(x[a:a + n])) for a, n in ((0, 2), (2, 198), (200, 99), (299, 1))])
        eng.release(s)
        assert rel_err(got[-1], want[-1]) < 2e-5
        last.append(got[-1] - x[-1].numpy())
    assert np.abs(last[0] - last[1]).max() > 1e-3 * np.abs(last[0]).max()


@pytest.mark.parametrize("taps", [2, 3, 4, 6])
def test_the_convolution_reaches_taps_minus_one_tokens_back(tmp_path, taps):
    """An input that is nothing but one row: with the state's decay near zero (each token's state is its own input) the rows that
    still see it are the taps - 1 behind it, whether the rows come in one portion, in twos or one by one, on both sides of a page's
    border."""
    layer = rglru(32, 4, taps)
    cfg = one_layer(layer)

    def change(W):
        W["l0.mix.lam"] = torch.full_like(W["l0.mix.lam"], 40.0)           # a = exp(-8 r 40): nothing is kept
        W["l0.mix.x.b"] = torch.zeros_like(W["l0.mix.x.b"])
        W["l0.mix.conv"] = W["l0.mix.conv"].sign() * 0.5
    d, W = make_model(tmp_path, cfg, 16, change=change)
    T, at = 72, 62
    x = 0.02 * torch.randn(T, 80, generator=torch.Generator().manual_seed(5), dtype=torch.float64)
    y = x.clone()
    y[at] = torch.randn(80, generator=torch.Generator().manual_seed(6), dtype=torch.float64)
    want_x, want_y = mixer_alone(x, W, layer).numpy(), mixer_alone(y, W, layer).numpy()
    moved = np.abs(want_y - want_x).max(1) > 1e-6
    assert np.flatnonzero(moved).tolist() == list(range(at, at + taps))
    for cuts in ([T], [2] * (T // 2), [1] * T, [at + 1] + [1] * (T - at - 1)):
        eng = engine_for(d, "float32")
        s, p, got = eng.acquire(), 0, []
        for n in cuts:
            got.append(eng.block_forward(0, [(s, n)], f32(y[p:p + n])))
            p += n
        got = np.concatenate(got)
        for r in range(T):
            assert rel_err(got[r], want_y[r]) < 2e-5, (taps, cuts[0], r)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("special", [0, 1, 63, 64, 65, 127, 300])
def test_one_key_stands_out_among_hundreds(tmp_path, special, dtype):
    """Weights and inputs made so that ONE key far outweighs all others for every later query: the latent's map of a row is the
    queries' map of the row shifted back by one column, and the special row is the later rows' common direction shifted.  Rows
    behind it return its value, near and far, in a prompt and decoded one by one; without that key they would not."""
    H, d_, r_ = 2, 24, 32
    layer = latent(H, d_, 8, 16, r_, r_, 1.0, 1e6)
    cfg = one_layer(layer)
    T = special + 130
    W = random_weights(cfg, 11)
    k = torch.randn(r_, 80, generator=torch.Generator().manual_seed(1)) / 80 ** 0.5
    W["l0.mix.dq"] = k.to(torch.bfloat16)
    W["l0.mix.dkv"] = torch.cat([torch.roll(k, 1, dims=1), torch.zeros(8, 80)]).to(torch.bfloat16)        # no rotated part: positions do not matter
    for n in ("dq.norm", "dkv.norm"):
        W["l0.mix." + n] = torch.ones_like(W["l0.mix." + n])
    uk = torch.randn(H * d_, r_, generator=torch.Generator().manual_seed(2)) / r_ ** 0.5
    W["l0.mix.uk"] = uk.to(torch.bfloat16)
    W["l0.mix.uq"] = torch.cat([torch.cat([uk[h * d_:(h + 1) * d_], torch.zeros(8, r_)]) for h in range(H)]).to(torch.bfloat16)
    path = write_model(tmp_path, cfg, W)
    W = {n: v.double() for n, v in W.items()}
    g = torch.Generator().manual_seed(3)
    rows = torch.randn(T, 80, generator=g, dtype=torch.float64)
    asked = torch.randn(80, generator=g, dtype=torch.float64)
    x = rows.clone()
    x[special] = torch.roll(asked, 1)
    x[special + 1:] = asked[None, :] + 0.1 * rows[special + 1:]
    want = mixer_alone(x, W, layer).numpy()
    other = x.clone()
    other[special] = rows[special]
    without = mixer_alone(other, W, layer).numpy()
    seen = [r for r in range(special + 1, T) if np.abs(want[r] - without[r]).max() > 0.3 * np.abs(want[r] - x[r].numpy()).max()]
    assert len(seen) == T - special - 1              # the key shows
    for cuts in ([T], [special + 1] + [1] * 129, [special + 70] + [1] * 60):
        eng = engine_for(path, dtype)
        slot, at, got = eng.acquire(), 0, []
        for n in cuts:
            got.append(eng.block_forward(0, [(slot, n)], f32(x[at:at + n])))
            at += n
        got = np.concatenate(got)
        bad = [(r, rel_err(got[r], want[r])) for r in range(T) if rel_err(got[r], want[r]) > (3e-5 if dtype == "float32" else 8e-2)]
        assert len(bad) <= (0 if dtype == "float32" else T // 30), (special, cuts[0], bad[:8])


def test_the_gate_and_the_two_scales(tmp_path):
    """A gate that is shut (large negative logits) leaves the stream to the norm of almost nothing; the embedding's scale and the
    logits' scale are each used once: doubling the one with half the table changes the head only, doubling the other doubles the
    logits."""
    cfg = config(64, 70, [(latent(2, 16, 8, 16, 24, 24, 0.25, 1000.0), dense(40))], eps=EPS, embed_scale=2.0, logit_scale=0.75)
    d, W = make_model(tmp_path / "a", cfg, 17)
    toks = tokens_for(cfg, 20, 1)
    base = plain_logits(cfg, W, toks)
    other = dict(cfg, logit_scale=1.5)
    W2 = random_weights(cfg, 17)
    for name, c, w in (("a", cfg, W), ("b", other, W)):
        path = d if name == "a" else write_model(tmp_path / "b", c, W2)
        eng = engine_for(path, "float32")
        got = eng.step_host([entry(eng.acquire(), toks)])
        assert rel_err(got, plain_logits(c, w, toks)) < TOL["float32"]
        assert rel_err(got, base * (1.0 if name == "a" else 2.0)) < TOL["float32"]


# ------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(CASES))
def test_whole_prompt(models, which, dtype):
    """Logits at every position of a prompt that passes pages and the recurrence's runs of tokens."""
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
    """Sequences of one, two, three and five tokens, as a prompt and one by one: convolutions that reach in front of the
    sequence's start see zeros, states start at zero."""
    for which in CASES:
        d, cfg, W = models[(which, "float32")]
        eng = engine_for(d, "float32")
        for n in (1, 2, 3, 5):
            toks = tokens_for(cfg, n, 30 + n)
            want = plain_logits(cfg, W, toks)
            s = eng.acquire()
            assert rel_err(eng.step_host([entry(s, toks)]), want) < TOL["float32"], (which, n)
            eng.release(s)
            s = eng.acquire()
            got = np.concatenate([eng.step_host([entry(s, [t])]) for t in toks])
            assert rel_err(got, want) < TOL["float32"], (which, n)
            eng.release(s)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which,cuts", [("a", [2, 2, 3, 17, 33, 64, 65, 2, 31]), ("b", [63, 2, 64, 1, 1, 70, 2, 16]),
                                        ("c", [100, 28, 1, 2, 64, 24]), ("d", [3, 2, 40, 2])])
def test_portions_and_decoding(models, which, cuts, dtype):
    """A prompt cut into portions of many sizes, down to two tokens and one, then 40 tokens one by one: the same logits
    as the whole sequence at every position."""
    d, cfg, W = models[(which, dtype)]
    n = sum(cuts) + 40
    toks = tokens_for(cfg, n, 13)
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


def test_slots_and_pages_used_again(models):
    """Sequences come and go in a cache of two slots and few pages: a new sequence starts from nothing (state rows - the
    recurrences' and the convolutions' - are cleared, pages of the one before are not read), also after a sequence that
    was released halfway."""
    d, cfg, W = models[("b", "float32")]
    eng = engine_for(d, "float32", max_tokens=512, max_batch=2)
    seqs = [tokens_for(cfg, n, 40 + i) for i, n in enumerate([200, 130, 90, 260, 70, 140])]
    for k, toks in enumerate(seqs):
        s = eng.acquire()
        other = eng.acquire()
        eng.step_host([entry(other, seqs[(k + 1) % len(seqs)][:50], [])])       # a neighbour that is dropped halfway
        want = plain_logits(cfg, W, toks)
        head = len(toks) - 20
        got = eng.step_host([entry(s, toks[:head], [head - 1])])
        assert rel_err(got[0], want[head - 1]) < TOL["float32"], k
        eng.release(other)
        for p in range(head, len(toks)):
            got = eng.step_host([entry(s, [toks[p]])])
            assert rel_err(got[0], want[p]) < TOL["float32"], (k, p)
        eng.release(s)
        eng.cache.check()


def test_long_decoding_past_pages(models):
    """300 tokens one by one after a short prompt: pages fill up, the convolution's ring goes round and the recurrent states
    carry the first tokens all along."""
    d, cfg, W = models[("b", "float32")]
    toks = tokens_for(cfg, 330, 50)
    want = plain_logits(cfg, W, toks)
    eng = engine_for(d, "float32")
    s = eng.acquire()
    eng.step_host([entry(s, toks[:30], [])])
    for p in range(30, 330):
        got = eng.step_host([entry(s, [toks[p]])])
        assert rel_err(got[0], want[p]) < TOL["float32"], p
    eng.release(s)
    eng.cache.check()


def test_a_far_token_is_remembered(tmp_path):
    """One early token differs between two prompts of 400 tokens: through latent attention (its own latents and an earlier
    layer's), and through a state that forgets slowly, the last logits differ by far more than rounding, in the engine exactly as
    in the plain implementation; through a recurrent state that forgets at once they would not."""
    fast = (rglru(40, 2, 2), dense(40))
    for name, layers, lam in (("latent", [fast, (latent(2, 16, 8, 16, 24, 24, 0.4, 10000.0), dense(48)), (latent(3, 8, 8, 16, 24, 20, 0.4, 10000.0, kv_from=1), None)], 6.0),
                              ("state", [(rglru(40, 2, 3), dense(48))], -7.0), ("neither", [fast], 6.0)):
        cfg = config(64, 90, layers)
        d, W = make_model(tmp_path / name, cfg, 60, sharp=2.0, lam=lam)
        a = tokens_for(cfg, 400, 61)
        b = list(a)
        b[3] = (a[3] + 1) % cfg["vocab"]
        eng = engine_for(d, "float32")
        last = []
        for toks in (a, b):
            s = eng.acquire()
            got = eng.step_host([entry(s, toks[:380], [])])
            for p in range(380, 400):
                got = eng.step_host([entry(s, [toks[p]])])
            last.append(got[0])
            eng.release(s)
            assert rel_err(got[0], plain_logits(cfg, W, toks)[-1]) < TOL["float32"]
        # (rounding is at 1e-6 of the largest logit)
        moved = np.abs(last[0] - last[1]).max() / np.abs(last[0]).max()
        assert moved < 1e-5 if name == "neither" else moved > 1e-4, (name, moved)


def test_many_steps_back_to_back():
    """A hundred and twenty prompt steps of drawn shapes - one to three sequences of 2 to 2,048 tokens, every third step a prompt
    of 2,048 - each followed by three decode steps, at sizes where every contraction and attention runs on the tensor cores and
    the row-wise kernels between them are short against them: every step ends with finite logits, and a repeated prompt gives
    the same logits."""
    from fastgguf_b200.engine.api import Engine
    from fastgguf_b200.registry import config_from_dict
    cfg = config(1024, 4096, [
        (latent(16, 64, 64, 64, 256, 768, 0.09, 10000.0), dense(4096)),
        (rglru(1024, 8, 4), moe(1024, 8, 2)),
        (latent(16, 64, 64, 64, 256, 768, 0.09, 10000.0, kv_from=0), moe(1024, 8, 2)),
        (rglru(1280, 5, 3), dense(4096)),
    ])
    eng = Engine.from_random(config_from_dict(cfg), 3, dtype="bfloat16", max_tokens=8192, max_batch=4, max_seq_len=4096)
    rng = np.random.default_rng(5)
    fixed = tokens_for(cfg, 2048, 90)
    first = None
    for i in range(120):
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
@pytest.mark.parametrize("which", ["a", "b"])
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
            assert row[t] >= row.max() - 1e-4 * np.abs(row).max(), (which, i)
    eng.cache.check()
    assert eng.cache.live_slots() == []


def test_generation_in_bfloat16_runs_the_recorded_step(models):
    d, cfg, W = models[("c", "bfloat16")]
    prompts = [tokens_for(cfg, n, 80 + i) for i, n in enumerate([9, 40])]
    eng = engine_for(d, "bfloat16", max_tokens=1024, max_batch=2)
    out = eng.generate(prompts, temp=0, max_tokens=70, ignore_eos=True)
    for p, c in zip(prompts, out):
        logits = plain_logits(cfg, W, p + c.tokens)
        close = sum(logits[len(p) + i - 1][t] >= logits[len(p) + i - 1].max() - 0.05 * np.abs(logits[len(p) + i - 1]).max()
                    for i, t in enumerate(c.tokens))
        assert close >= 0.9 * len(c.tokens)
    eng.cache.check()


@pytest.mark.parametrize("which", ["a", "c"])
def test_trace_replay_three_cuts(tmp_path, models, which):
    """``bin/trace_run`` on a Zifelorn folder in true 32-bit: the same requests whole, with their last 32 tokens one by one, and
    in batches of four unequal requests one batch after another (slots and pages are used again); a cache that holds just what
    the live requests need."""
    from trace_tools import batched_trace, collect, run_trace, tail_trace, whole_trace
    d, cfg, W = models[(which, "float32")]
    lengths = [5, 9, 1, 17, 3, 40, 11, 70, 33, 130]
    requests = {f"r{i}": tokens_for(cfg, n, 100 + i) for i, n in enumerate(lengths)}
    want = {rid: plain_logits(cfg, W, toks) for rid, toks in requests.items()}
    need = max(sum((len(requests[r]) + 63) // 64 * 64 for r in list(requests)[b:b + 4]) for b in range(0, 10, 4))
    cuts = {}
    for name, (steps, index), room in (("whole", whole_trace(requests), 192), ("tail", tail_trace(requests, 32), 192),
                                       ("batched", batched_trace(requests, 4), need)):
        run_trace(d, "float32", steps, str(tmp_path / name), max_tokens=room)
        rows = collect(str(tmp_path / name), steps, index, cfg["vocab"])
        assert len(rows) == sum(lengths), name
        for (rid, pos), row in rows.items():
            assert rel_err(row, want[rid][pos]) < TOL["float32"], (name, rid, pos)
        cuts[name] = rows
    for key, row in cuts["whole"].items():
        scale = np.abs(row).max()
        assert np.abs(row - cuts["tail"][key]).max() < 2e-5 * scale and np.abs(row - cuts["batched"][key]).max() < 2e-5 * scale, key


def test_command_line_generates(models):
    """``python -m fastgguf_b200 generate`` on a Zifelorn folder: the model class comes from config.json, the tokens are
    those of Engine.generate."""
    import json
    import os
    import subprocess
    import sys
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
