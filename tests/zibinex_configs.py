"""Small Zibinex configurations that differ from one another in every size and option, and weights for them: drawn by the
framework's random-weights mode (values that bfloat16 holds exactly, so every path and the oracle compute with the same
numbers), then changed so that faults show: query norms and projections scaled so that attention is peaked (a key that is
lost, or a window's edge that is one off, moves the output), the sigmoid's offsets low so that most keys weigh little,
penalties by distance from faint to strong, gate and up products that reach beyond the clamped gate's limit."""
from __future__ import annotations

import copy
from typing import Dict, Optional

import torch

GROUPS = 4                                        # groups of tokens that choose their experts apart (see `make_weights`)


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def lat(heads, dim, rot_dim, vdim, rank, scale, rot, mlp, weights_of=None):
    """rot: (base, None) or (base, (factor, original, fast, slow))."""
    r = {"dims": rot_dim, "base": rot[0]}
    if rot[1] is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[1]))
    L = {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": r},
         "mlp": mlp}
    return L if weights_of is None else dict(L, weights_of=weights_of)


def att(heads, kv_heads, dim, vdim, scale, window, mlp, weights_of=None):
    L = {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}},
         "mlp": mlp}
    return L if weights_of is None else dict(L, weights_of=weights_of)


def again(layers, i):
    """The layer that runs once more with layer i's weights."""
    return dict(copy.deepcopy(layers[i]), weights_of=i)


def _model(vocab, width, eps, layers):
    return {"architecture": "Zibinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def zb_a() -> dict:
    # grouped heads with a value size above the key size and a window of 20; a latent of 32 beside 8 rotated dimensions
    # (padded to 48); both kinds of layer run a second time with a cache of their own; two of five experts
    L = [lat(3, 16, 8, 24, 32, 0.3, (5000.0, (4.0, 128, 6.0, 0.5)), dense(72, 1.0)),
         att(4, 2, 32, 48, 0.2, 20, moe(40, 5, 2))]
    return _model(211, 96, 1e-5, L + [again(L, 1), again(L, 0), att(4, 4, 16, 16, 0.25, 33, None)])


def zb_b() -> dict:
    # a width that is no multiple of 16; a window of one page exactly; rotation without scaling; every expert chosen; a
    # layer without a feed-forward that runs three times, named through one another
    L = [att(6, 6, 16, 16, 0.25, 16, moe(56, 3, 3)), lat(2, 64, 16, 16, 48, 0.15, (300.0, None), None), att(6, 2, 24, 8, 0.3, 50, dense(64, 3.0))]
    return _model(300, 120, 1e-4, L + [again(L, 1), dict(again(L, 1), weights_of=3)])


def zb_c() -> dict:
    # head size 128 and a latent of 96 + 32 (the tensor-memory prefill kernel), a latent of 192 + 64 (its form for 256), a
    # window longer than most test sequences and one of 5
    L = [lat(2, 128, 32, 128, 96, 0.08, (20000.0, (8.0, 512, 16.0, 1.0)), moe(32, 7, 3)), att(2, 1, 128, 128, 0.09, 400, dense(96, 2.5)),
         att(8, 2, 128, 64, 0.11, 5, moe(32, 2, 1)), lat(4, 64, 64, 64, 192, 0.1, (1e6, (2.0, 64, 3.0, 1.5)), dense(48, 0.7))]
    return _model(128, 128, 1e-6, L + [again(L, 2)])


def zb_d() -> dict:
    # sizes without a fast attention kernel (a latent of 250 + 20), a latent of 24 + 4 with one head, key size 20 and value size
    # 12, windows of 7 and of 1 (a token sees itself alone), a single expert
    L = [lat(1, 12, 4, 20, 24, 0.35, (50.0, (16.0, 32, 2.0, 1.0)), moe(24, 1, 1)), att(3, 3, 20, 12, 0.22, 7, dense(40, 1.5)),
         lat(3, 8, 20, 12, 250, 0.3, (1000.0, (3.0, 400, 9.0, 2.0)), None), att(2, 1, 8, 40, 0.4, 1, moe(24, 6, 4))]
    return _model(64, 72, 1e-5, L)


ZIBINEX = {"a": zb_a, "b": zb_b, "c": zb_c, "d": zb_d}


def make_weights(raw: dict, seed: int, peak: float = 4.0, clear_choices: bool = False) -> Dict[str, torch.Tensor]:
    """`peak`: about the standard deviation the scaled scores of an attention layer are brought to: a few keys then carry
    most of the weight, while rounding to bfloat16 does not yet decide which.
    `clear_choices`: a token's experts follow from its group (token id mod 4) by margins that rounding cannot close, so that every
    position of a bfloat16 run can be compared: four columns of the residual stream carry the group alone (every branch norm
    writes nothing there, the final norm reads nothing there) and the routers' rows differ mostly in those columns, in
    another order for every group."""
    from infinilm_b200.config import config_from_json
    from infinilm_b200.weights import random_tensors
    w = random_tensors(config_from_json(raw), seed, "cpu")
    g = torch.Generator().manual_seed(seed + 77)
    W = raw["width"]

    def layer_of(name) -> Optional[dict]:
        return raw["layers"][int(name[1:name.index(".")])] if name.startswith("l") and "." in name and name[1].isdigit() else None
    for name in list(w):
        x, layer = w[name].float(), layer_of(name)
        typ, m = (layer["type"], layer["mixer"]) if layer else (None, None)
        if name == "embed":
            x = x * 50.0
            if clear_choices:
                x[:, :GROUPS] = 0.0
                x[torch.arange(x.shape[0]), torch.arange(x.shape[0]) % GROUPS] = 5.0
        elif name.endswith(("norm1", "norm2", "norm1b", "norm2b", "final.norm")):
            x = x * 4.0
            if clear_choices and not name.endswith(("norm1", "norm2")):
                x[:GROUPS] = -1.0
            elif clear_choices:
                x[:GROUPS] = 0.0
        elif name.endswith(".q.norm"):
            x = x * peak / (m["scale"] * m["dim"] ** 0.5)
        elif typ == "latent_attention" and name.endswith(".mix.q"):
            d, rd = m["dim"], m["rot_dim"]
            x = x.view(m["heads"], d + rd, W).clone()
            unit = 0.02 * W ** 0.5                # the size of a query column, and of the shared rotated key's
            x[:, :d] *= 0.6 * peak / (m["scale"] * unit * 0.08 * m["kv_rank"] ** 0.5 * d ** 0.5)
            x[:, d:] *= 0.6 * peak / (m["scale"] * unit * unit * 4.0 * rd ** 0.5)
            x = x.view(-1, W)
        elif typ == "latent_attention" and name.endswith(".mix.dkv"):
            x = x * 4.0
        elif name.endswith(".mix.g"):
            x = x * 6.0
        elif typ == "attention" and name.endswith((".mix.q", ".mix.k", ".mix.v")):
            x = x * 3.0
        elif name.endswith((".q.b", ".k.b", ".v.b")):
            x = x * 15.0
        elif name.endswith(".mix.pb"):
            x = x * 0.5 - 3.0
        elif name.endswith(".mix.r1"):
            x = torch.rand(x.shape, generator=g) * 1.5
        elif name.endswith(".mix.r2"):
            x = torch.rand(x.shape, generator=g) * 0.5 + 0.02
        elif layer is not None and layer.get("mlp") and layer["mlp"]["kind"] == "dense" and name.endswith((".mlp.gate", ".mlp.up")):
            x = x * layer["mlp"]["limit"] / (0.02 * W ** 0.5)             # products of the limit's own size
        elif name.endswith(".router"):
            x = x * (0.02 if clear_choices else 1.0 / W ** 0.5 * 3.0)
            if clear_choices:
                for c in range(GROUPS):
                    x[:, c] = torch.linspace(-2.0, 2.0, x.shape[0])[torch.randperm(x.shape[0], generator=g)]
        else:
            continue
        w[name] = x.to(torch.bfloat16)
    return w


def token_ids(n: int, vocab: int, seed: int):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
