"""Seeded random Buguzen configurations, engine against the plain implementation: every size, the order and mix of layers, heads,
windows, rotations and their scalings, decays, feed-forwards, the token input and the loop are drawn; then a batch of unequal
prompts, a portion, and decode steps during which sequences leave.  float32 engines are held to the float32 tolerance everywhere;
bfloat16 engines run the same model with sharpened attention."""
import numpy as np
import pytest

from buguzen_cases import config, differential, keys_as_values, lightning, make_model
from test_buguzen import Rows, engine_for, entry, plain_logits

pytestmark = pytest.mark.gpu


def draw_config(rng):
    width = int(rng.choice([64, 96, 128, 160, 200, 72, 256, 90]))
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        kv = int(rng.integers(1, 4))
        heads = kv * int(rng.integers(1, 5))
        size = None if rng.random() < 0.3 else int(rng.choice([1, 3, 17, 40, 64, 65, 100, 129]))
        scale = float(rng.uniform(0.05, 0.4))
        kind = rng.random()
        if kind < 0.35:
            dim, vdim = [(16, 24), (64, 128), (64, 64), (128, 128), (22, 40), (48, 16), (5, 9), (32, 128)][int(rng.integers(0, 8))]
            rot = None if dim % 2 or rng.random() < 0.2 else (float(rng.choice([50.0, 1e4, 5e5])), 2 * int(rng.integers(1, dim // 2 + 1)))
            mixer = differential(heads, kv, dim, vdim, scale, float(rng.uniform(0.0, 0.9)), size, rot,
                                 (float(rng.choice([1.0, 2.5, 8.0])),) if rng.random() < 0.6 else None)
        elif kind < 0.7:
            dim = int(rng.choice([16, 64, 128, 22, 48, 9]))
            rot = None if dim % 2 or rng.random() < 0.2 else (float(rng.choice([50.0, 1e4, 5e5])), 2 * int(rng.integers(1, dim // 2 + 1)))
            mixer = keys_as_values(heads, kv, dim, scale, size, rot,
                                   (float(rng.choice([2.0, 8.0])), 1.0, float(rng.choice([2.0, 4.0])), int(rng.choice([16, 64, 512]))) if rng.random() < 0.6 else None)
        else:
            heads = int(rng.integers(1, 6))
            mixer = lightning(heads, int(rng.choice([8, 16, 64, 128, 21])), int(rng.choice([8, 24, 64, 128, 13])),
                              [float(v) for v in rng.choice([0.2, 0.6, 0.9, 0.99, 0.999, 1.0], size=heads)])
        layers.append((mixer, None if rng.random() < 0.3 else int(rng.choice([64, 100, 192, 320]))))
    n = len(layers)
    loop = None
    if rng.random() < 0.6:
        start = int(rng.integers(0, n))
        loop = (start, int(rng.integers(start + 1, n + 1)), int(rng.integers(1, 4)))
    side = None if rng.random() < 0.3 else int(rng.choice([4, 8, 16, 24, 7]))
    return config(width, int(rng.integers(40, 500)), layers, loop=loop, side=side, eps=float(rng.choice([2e-5, 1e-6])))


@pytest.mark.parametrize("seed", list(range(31, 51)))
def test_random_configuration(tmp_path, seed):
    rng = np.random.default_rng(seed)
    cfg = draw_config(rng)
    dtype = "bfloat16" if seed % 3 == 0 else "float32"
    d, W = make_model(tmp_path, cfg, seed, sharp=1.5 if dtype == "bfloat16" else 1.0)
    B = int(rng.integers(1, 5))
    total = [int(rng.integers(3, 200)) for _ in range(B)]
    first = [int(rng.integers(1, t)) for t in total]
    toks = [[int(t) for t in rng.integers(0, cfg["vocab"], size=n)] for n in total]
    want = [plain_logits(cfg, W, t) for t in toks]
    eng = engine_for(d, dtype)
    slots = [eng.acquire() for _ in toks]
    got = eng.step_host([entry(s, t[:n]) for s, t, n in zip(slots, toks, first)])
    row = 0
    judge = Rows(dtype)
    for b, n in enumerate(first):
        for p in range(n):
            judge.add(got[row], want[b][p], (seed, b, p))
            row += 1
    at = list(first)
    # one more portion for the first sequence, then everyone token by token
    if total[0] - at[0] > 3:
        n = int(rng.integers(2, total[0] - at[0]))
        got = eng.step_host([entry(slots[0], toks[0][at[0]:at[0] + n])])
        for i in range(n):
            judge.add(got[i], want[0][at[0] + i], (seed, "portion", at[0] + i))
        at[0] += n
    alive = [b for b in range(B) if at[b] < total[b]]
    while alive:
        got = eng.step_host([entry(slots[b], [toks[b][at[b]]]) for b in alive])
        for i, b in enumerate(alive):
            judge.add(got[i], want[b][at[b]], (seed, b, at[b]))
            at[b] += 1
        for b in [b for b in alive if at[b] == total[b]]:
            eng.release(slots[b])
            alive.remove(b)
    judge.done()
    eng.cache.check()
