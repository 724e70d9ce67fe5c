"""Small Gukosun configurations that differ from one another in every size and option, and weights for them: drawn by the
framework's random-weights mode (values that bfloat16 holds exactly, so every path and the oracle compute with the same numbers),
then changed so that faults show: query norms scaled so that attention is peaked (a key that is lost, or a window's edge that is
one off, moves the output) and reaches the caps, sinks that take a share of the weight, blends far from 0 and 1, gates away from
one half, branches of the stream's own size."""
from __future__ import annotations

from typing import Dict

import torch


def dense(ff):
    return {"kind": "dense", "ff": ff}


def att(heads, kv_heads, dim, vdim, scale, window, mlp, v_mix=True):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                                       "mask": {"size": window}, "v_mix": v_mix}}


def par(left, right, mlp):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": right}}


def left(heads, kv_heads, dim, vdim, scale, cap, rot=None):
    """rot: None, (dims, base, None) or (dims, base, (factor, low, high, original)); cap None: scores as they are."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if cap is not None:
        m["softcap"] = cap
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if rot[2] is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), rot[2]))
    return m


def right(heads, dim, vdim, decay):
    assert len(decay) == heads
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def _model(vocab, width, eps, side, logit_scale, layers):
    return {"architecture": "Gukosun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "token_side": {"dim": side},
            "layers": layers}


def gk_a() -> dict:
    # grouped heads, a window of 20, value size above and below the key size; part of a head rotated, all three bands of the
    # frequencies' scaling; a layer without a feed-forward; a blend in the first and third attention layer, none in the second
    return _model(211, 96, 1e-5, 12, 0.7, [
        att(4, 2, 32, 48, 0.2, 20, dense(72)), par(left(6, 2, 16, 24, 0.3, 9.0, (12, 500.0, (4.0, 1.0, 6.0, 128))), right(3, 24, 16, (0.5, 0.93, 0.999)), dense(136)),
        att(3, 1, 24, 8, 0.3, 33, dense(40), v_mix=False), par(left(2, 2, 64, 32, 0.15, 30.0, (64, 1e4, (8.0, 1.0, 4.0, 64))), right(1, 16, 48, (0.8,)), None),
        att(8, 2, 16, 48, 0.25, 7, dense(64))])


def gk_b() -> dict:
    # parallel layers first; a width that is no multiple of 16, a side of 5 columns; a window of one page exactly; no rotation in
    # one layer, unscaled frequencies in another, no cap; one kv head; a decay of one and of (nearly) nothing
    return _model(300, 120, 1e-4, 5, 1.0, [
        par(left(3, 3, 20, 12, 0.22, None, (8, 50.0, None)), right(2, 10, 30, (1.0, 0.01)), dense(56)), att(6, 6, 16, 16, 0.25, 16, dense(72)),
        par(left(5, 1, 8, 40, 0.35, 4.0), right(4, 16, 8, (0.3, 0.9, 0.99, 0.7)), None), att(6, 6, 16, 16, 0.3, 50, None)])


def gk_c() -> dict:
    # head sizes of the tensor-memory prefill kernel (128; 64; 200 and 256 in one), a window longer than most test sequences and
    # one of 5, rotation of two dimensions alone, caps from low to high
    return _model(128, 128, 1e-6, 24, 0.25, [
        att(2, 1, 128, 128, 0.09, 400, dense(96)), par(left(4, 2, 64, 64, 0.12, 6.0, (2, 20.0, (3.0, 0.5, 2.0, 100))), right(2, 128, 64, (0.97, 0.6)), dense(256)),
        par(left(2, 2, 200, 256, 0.07, 50.0, (200, 1e6, (8.0, 1.0, 4.0, 512))), right(1, 64, 128, (0.995,)), dense(32)), att(8, 1, 128, 128, 0.1, 5, dense(96))])


def gk_d() -> dict:
    # odd sizes: a width of 74, key size 18 with 6 rotated, value size 7 and 13, a feed-forward of 37, windows of 1 and 11, a side of 3
    # columns; the only two attention layers blend, the first with the loudest values; a model that ends on a parallel layer
    return _model(64, 74, 1e-5, 3, 2.0, [
        att(2, 1, 18, 7, 0.3, 11, dense(37)), att(4, 1, 10, 7, 0.4, 1, None),
        par(left(3, 1, 18, 13, 0.25, 2.5, (6, 10.0, (16.0, 0.7, 1.9, 40))), right(3, 5, 9, (0.9, 0.5, 0.99)), dense(24))])


GUKOSUN = {"a": gk_a, "b": gk_b, "c": gk_c, "d": gk_d}


def make_weights(raw: dict, seed: int, peak: float = 4.0) -> Dict[str, torch.Tensor]:
    """`peak`: about the standard deviation the scaled scores of an attention layer are brought to, before any cap: a few keys then
    carry most of the weight, while rounding to bfloat16 does not yet decide which."""
    from infinilm_b200.config import config_from_json
    from infinilm_b200.weights import random_tensors
    w = random_tensors(config_from_json(raw), seed, "cpu")
    g = torch.Generator().manual_seed(seed + 77)
    unit = 1.0 / (0.02 * raw["width"] ** 0.5)     # brings the product of a drawn matrix with a normed row to size 1
    for name in sorted(w):
        x = w[name].float()
        L = raw["layers"][int(name[1:name.index(".")])] if name[0] == "l" and name[1].isdigit() else None
        m = None if L is None else L["mixer"]["left"] if L["type"] == "parallel" and ".left." in name else L["mixer"]
        if name == "embed":
            x = x * 50.0
        elif name.endswith(".q.norm"):
            x = (1.0 + (x - 1.0) * 4.0) * peak / (m["scale"] * m["dim"] ** 0.5)
        elif name.endswith((".norm1", ".norm", ".out", ".ls1", ".ls2")):
            x = 1.0 + (x - 1.0) * 5.0
        elif name.endswith(".vmix"):
            x = torch.tensor(0.3 + 0.5 * float(torch.rand((), generator=g)))
        elif name.endswith(".sink"):
            x = x * 1.5 + peak                    # beside a sum of exponentials of scores with that spread
        elif name.endswith((".mix.g", ".left.g", ".right.g")):
            x = x * unit * 1.5
        elif name.endswith((".mix.v", ".left.v", ".right.q", ".right.k", ".right.v", ".mlp.up")):
            x = x * unit
        elif name.endswith((".mix.o", ".left.o", ".right.o", ".mlp.down")):
            x = x * (1.0 / (0.02 * x.shape[1] ** 0.5))
        elif name.endswith(".side.gate"):
            x = x * unit * 0.4                    # (far on the negative side of GELU a norm would magnify what rounding left)
        else:
            continue
        w[name] = x.to(torch.bfloat16)
    return w


def token_ids(n: int, vocab: int, seed: int):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
