"""Gukosun at sizes drawn from a seed: widths that are no multiple of 16, key and value sizes with and without a fast attention
kernel and unequal in either direction, grouped heads or not, windows from 1 position to beyond the sequence, rotation of any even
part of a head or none, scaled or not, caps from one to a thousand or none, any decays, token inputs of any width, layers
without a feed-forward, blends in any of the attention layers, any order of layers. Each configuration runs a prompt whole, in
portions and token by token against the plain implementation, in both dtypes, and two requests side by side."""
import random
import warnings

import pytest
import torch

import plain_gukosun as P
from gukosun_configs import att, dense, left, make_weights, par, right, token_ids

pytestmark = pytest.mark.gpu


def random_config(seed: int) -> dict:
    rng = random.Random(11000 + seed)
    blend_kv, blend_v = rng.randint(1, 3), rng.choice([4, 7, 16, 24, 40, 64])
    layers = []
    for i in range(rng.randint(1, 5)):
        mlp = None if rng.random() < 0.25 else dense(rng.choice([8, 24, 37, 50, 72, 136, 256]))
        kv, dim, vdim = rng.randint(1, 3), rng.choice([4, 8, 12, 18, 24, 40, 64, 96, 128]), rng.choice([4, 7, 20, 32, 64, 80, 128])
        if rng.random() < 0.5:
            mix = rng.random() < 0.7
            if mix:
                kv, vdim = blend_kv, blend_v
            layers.append(att(kv * rng.randint(1, 4), kv, dim, vdim, round(rng.uniform(0.05, 0.4), 3), rng.choice([1, 2, 15, 16, 17, 32, 50, 1000]), mlp, mix))
            continue
        rot = None
        if rng.random() < 0.8:
            scaling = None if rng.random() < 0.25 else (rng.choice([1.5, 4.0, 32.0]), rng.choice([0.5, 1.0]), rng.choice([1.5, 4.0]), rng.choice([20, 64, 300, 4096]))
            rot = (2 * rng.randint(1, dim // 2), rng.choice([20.0, 1e4, 5e5]), scaling)
        lt = left(kv * rng.randint(1, 4), kv, dim, vdim, round(rng.uniform(0.05, 0.4), 3), rng.choice([None, 1.0, 5.0, 20.0, 1000.0]), rot)
        h = rng.randint(1, 4)
        rt = right(h, rng.choice([3, 8, 16, 24, 64, 100, 128]), rng.choice([4, 9, 16, 48, 64]), [rng.choice([0.2, 0.7, 0.95, 0.999, 1.0]) for _ in range(h)])
        layers.append(par(lt, rt, mlp))
    return {"architecture": "Gukosun", "vocab": rng.choice([50, 129, 333]), "width": rng.choice([40, 72, 74, 96, 100, 136, 200, 256]),
            "norm": {"eps": rng.choice([1e-6, 1e-5, 1e-3])}, "logit_scale": rng.choice([0.1, 1.0, 3.0]), "token_side": {"dim": rng.choice([4, 5, 8, 16, 30, 64])},
            "layers": layers}


def one_kind(kind: str) -> dict:
    """Models of a single kind of layer."""
    layers = {"windows": [att(2, 1, 16, 32, 0.25, 8, dense(40)), att(4, 4, 64, 64, 0.1, 30, None, v_mix=False)],
              "pairs": [par(left(4, 2, 16, 16, 0.3, 5.0, (16, 100.0, None)), right(2, 16, 16, (0.9, 0.99)), dense(40)),
                        par(left(2, 2, 32, 8, 0.2, None), right(1, 8, 40, (0.5,)), None)],
              "one layer": [par(left(1, 1, 64, 64, 0.2, 9.0, (64, 1e4, (2.0, 1.0, 4.0, 50))), right(8, 8, 8, [0.9] * 8), dense(24))]}[kind]
    return {"architecture": "Gukosun", "vocab": 97, "width": 64, "norm": {"eps": 1e-5}, "logit_scale": 1.0, "token_side": {"dim": 8}, "layers": layers}


KINDS = ["windows", "pairs", "one layer"]


def _err(got, ref):
    got, ref = got.double().cpu(), ref.double()
    got, ref = got - got.mean(dim=-1, keepdim=True), ref - ref.mean(dim=-1, keepdim=True)
    return (got - ref).pow(2).mean(dim=-1).sqrt() / ref.pow(2).mean(dim=-1).sqrt()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", list(range(24)) + KINDS)
def test_random_configuration(cuda_device, seed, dtype):
    from infinilm_b200.config import config_from_json
    from infinilm_b200.engine import Engine, StepEntry
    raw = random_config(seed) if isinstance(seed, int) else one_kind(seed)
    seed = seed if isinstance(seed, int) else 50 + KINDS.index(seed)
    w = make_weights(raw, seed, peak=3.0 if dtype == "float32" else 2.0)
    ids = token_ids(75, raw["vocab"], seed)
    other = token_ids(30, raw["vocab"], seed + 100)
    ref, ref_other = P.forward(raw, w, ids), P.forward(raw, w, other)
    with warnings.catch_warnings():
        warnings.simplefilter("ignore", RuntimeWarning)
        eng = Engine.from_tensors(config_from_json(raw), w, dtype=dtype, page_size=16, num_pages=8, max_seqs=2, max_batch_tokens=128)
    tol = 4e-5 if dtype == "float32" else 6e-2

    def judge(got, want, what):
        err = _err(got, want)
        n_bad = int((err > tol).sum())
        assert torch.isfinite(got).all()
        assert n_bad <= (0 if dtype == "float32" else len(err) // 15) and (dtype == "float32" or float(err.max()) <= 3 * tol), \
            f"seed {seed} {what}: {n_bad} positions over {tol:.0e}, worst {float(err.max()):.2e}; config {raw}"

    for cuts in ([75], [33, 2, 17, 1, 1, 21], [16] + [1] * 59):
        seq, outs, a = eng.open(str(cuts[0])), [], 0
        for c in cuts:
            outs.append(eng.step([StepEntry(seq, ids[a:a + c], list(range(c)))]).clone())
            a += c
        eng.close(seq)
        judge(torch.cat(outs, 0), ref, f"cuts {cuts[:3]}")
    # two requests side by side: a portion beside single tokens, then the other way round
    s1, s2 = eng.open("x"), eng.open("y")
    o1, o2 = [], []
    lg = eng.step([StepEntry(s1, ids[:40], list(range(40))), StepEntry(s2, other[:1], [0])]).clone()
    o1.append(lg[:40]), o2.append(lg[40:])
    for t in range(1, 6):
        lg = eng.step([StepEntry(s1, ids[39 + t:40 + t], [0]), StepEntry(s2, other[t:t + 1], [0])]).clone()
        o1.append(lg[:1]), o2.append(lg[1:])
    lg = eng.step([StepEntry(s1, ids[45:46], [0]), StepEntry(s2, other[6:30], list(range(24)))]).clone()
    o1.append(lg[:1]), o2.append(lg[1:])
    lg = eng.step([StepEntry(s1, ids[46:75], list(range(29)))]).clone()
    o1.append(lg)
    eng.close(s1), eng.close(s2)
    judge(torch.cat(o1, 0), ref, "side by side, first")
    judge(torch.cat(o2, 0), ref_other, "side by side, second")
    eng.synchronize()
    eng.cache.check_invariants()
