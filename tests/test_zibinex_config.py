"""Zibinex on the CPU: configuration and its faults, run order (layers that run with another's weights), tensor names and cache
needs, the random-weights folder, the rotation's tables, and the plain implementation's own identities (a window's edge, the
penalty by distance, the rotation's pairs, the clamped gate, a weight on the expert's input)."""
import json
import math
import os

import pytest
import torch

import plain_zibinex as P
from zibinex_configs import ZIBINEX, make_weights, token_ids

from infinilm_b200.config import ConfigError, config_from_json, describe_model
from infinilm_b200.models.causal_lm import CausalLM
from infinilm_b200.weights import FolderSource, check_against, write_model_folder


def test_run_order_of_layers_that_run_with_anothers_weights():
    orders = {n: [s.layer for s in describe_model(config_from_json(ZIBINEX[n]())).order] for n in ZIBINEX}
    assert orders == {"a": [0, 1, 1, 0, 2], "b": [0, 1, 2, 1, 1], "c": [0, 1, 2, 3, 2], "d": [0, 1, 2, 3]}
    for n in ZIBINEX:
        spec = describe_model(config_from_json(ZIBINEX[n]()))
        assert all(s.cache_from is None for s in spec.order)              # every entry keeps a cache of its own
        assert all(l.arrangement == "sandwich_residual" for l in spec.layers)


@pytest.mark.parametrize("name", sorted(ZIBINEX))
def test_tensor_names_and_cache_needs(name):
    raw = ZIBINEX[name]()
    model = CausalLM(describe_model(config_from_json(raw)), torch.float32)
    specs = {p.full_name(ws.name): ws for p, ws in model.weight_specs()}
    names = {k: v.shape for k, v in specs.items()}
    W, needs = raw["width"], model.cache_needs()
    assert names["embed"] == (raw["vocab"], W) and names["final.norm"] == (W,) and specs["head"].fallback == "embed"
    assert len(needs) == len(raw["layers"]) and all(n.kind == "paged_kv" for n in needs)
    for i, L in enumerate(raw["layers"]):
        m, typ, f, px = L["mixer"], L["type"], L["mlp"], f"l{i}.mix"
        assert needs[i].window == (m["mask"]["size"] if typ == "attention" else None)
        assert needs[i].n_kv_heads == (m["kv_heads"] if typ == "attention" else 1)
        if typ == "latent_attention":
            assert m["kv_rank"] + m["rot_dim"] <= needs[i].head_dim < m["kv_rank"] + m["rot_dim"] + 16
        if "weights_of" in L:
            assert not any(k.startswith(f"l{i}.") for k in names)
            continue
        assert names[f"l{i}.norm1"] == names[f"l{i}.norm1b"] == (W,)
        assert (f"l{i}.norm2" in names) == (f"l{i}.norm2b" in names) == (f is not None)
        if f and f["kind"] == "moe":
            n = f["router"]["experts"]
            assert names[f"l{i}.mlp.router"] == (n, W) and names[f"l{i}.mlp.e{n - 1}.down"] == (W, f["expert"]["ff"])
            assert f"l{i}.mlp.e{n}.gate" not in names and f"l{i}.mlp.router.b" not in names
        elif f:
            assert names[f"l{i}.mlp.gate"] == names[f"l{i}.mlp.up"] == (f["ff"], W) and names[f"l{i}.mlp.down"] == (W, f["ff"])
        H = m["heads"]
        if typ == "latent_attention":
            assert names[f"{px}.q"] == (H * (m["dim"] + m["rot_dim"]), W) and names[f"{px}.dkv"] == (m["kv_rank"] + m["rot_dim"], W)
            assert names[f"{px}.dkv.norm"] == (m["kv_rank"],) and names[f"{px}.g"] == (H, W)
            assert names[f"{px}.uk"] == (H * m["dim"], m["kv_rank"]) and names[f"{px}.uv"] == (H * m["vdim"], m["kv_rank"])
        else:
            assert names[f"{px}.q"] == (H * m["dim"], W) and names[f"{px}.q.b"] == (H * m["dim"],) and names[f"{px}.q.norm"] == (m["dim"],)
            assert names[f"{px}.k"] == (m["kv_heads"] * m["dim"], W) and names[f"{px}.k.norm"] == (m["dim"],)
            assert names[f"{px}.v.b"] == (m["kv_heads"] * m["vdim"],)
            assert all(names[f"{px}.{x}"] == (H,) for x in ("r1", "r2", "pb"))
        assert names[f"{px}.o"] == (W, H * m["vdim"])


def test_config_faults_name_the_key():
    def broken(change, match, exc=ConfigError):
        raw = ZIBINEX["a"]()
        change(raw)
        with pytest.raises(exc, match=match):
            CausalLM(describe_model(config_from_json(raw)), torch.float32)
    broken(lambda r: r["layers"][0].update(type="something_else"), "something_else")
    broken(lambda r: r["layers"][0]["mixer"].pop("kv_rank"), "kv_rank")
    broken(lambda r: r["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims")
    broken(lambda r: r["layers"][0]["mixer"]["rot"].pop("base"), "base")
    broken(lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow")
    broken(lambda r: r["layers"][0]["mlp"].pop("limit"), "limit")
    broken(lambda r: r["layers"][0]["mlp"].update(kind="other"), "other")
    broken(lambda r: r["layers"][1]["mixer"].pop("mask"), "mask")
    broken(lambda r: r["layers"][1]["mixer"]["mask"].update(size=0), "mask.size")
    broken(lambda r: r["layers"][1]["mlp"]["router"].pop("top"), "top")
    broken(lambda r: r["layers"][2].update(weights_of=9), "weights_of")
    broken(lambda r: r["layers"][2].update(weights_of=2), "weights_of")
    broken(lambda r: r["layers"][2].update(weights_of=0), "weights")              # another kind of layer
    broken(lambda r: r["layers"][2]["mixer"].update(scale=0.5), "differs")
    broken(lambda r: r["norm"].pop("eps"), "eps")
    broken(lambda r: [r["layers"][i]["mlp"]["router"].update(top=6) for i in (1, 2)], "top", ValueError)
    broken(lambda r: [r["layers"][i]["mixer"].update(kv_heads=3) for i in (1, 2)], "kv heads", ValueError)


def test_random_folder_round_trip(tmp_path):
    raw = ZIBINEX["b"]()
    cfg = config_from_json(raw)
    folder = write_model_folder(cfg, 5, str(tmp_path / "m"))
    assert json.load(open(os.path.join(folder, "config.json"))) == raw
    src = FolderSource(folder)
    check_against(CausalLM(describe_model(cfg), torch.bfloat16), src)
    assert "head" not in src.names() and "l0.norm1b" in src.names() and not any(n.startswith("l3.") for n in src.names())
    src.close()


@pytest.mark.parametrize("dims,base,scaling", [(16, 1e4, (4.0, 256, 8.0, 1.0)), (8, 50.0, (16.0, 32, 2.0, 1.0)), (64, 1e6, (2.0, 64, 3.0, 1.5)),
                                               (4, 100.0, (1.0, 1000, 32.0, 1.0)), (32, 500.0, (8.0, 10, 32.0, 1.0)), (2, 10.0, (3.0, 5, 1.0, 1.0)),
                                               (128, 1e5, (40.0, 4096, 32.0, 1.0))])
def test_yarn_table(dims, base, scaling):
    from infinilm_b200.parts.position import YarnRope
    p = dict(zip(("factor", "original", "fast", "slow"), scaling))
    part = YarnRope({"rot_dim": dims, "theta": base, "interleaved": True, **p}, "", torch.float32)
    part.to_device(torch.device("cpu"))
    freq, mult = P.yarn_table(dims, base, p)
    assert part.interleaved and torch.allclose(part.freq64, freq, rtol=1e-13) and abs(part.mscale - mult) < 1e-14
    plain = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    assert ((freq <= plain * (1 + 1e-12)) & (freq >= plain / p["factor"] * (1 - 1e-12))).all()
    assert mult == 1.0 if p["factor"] == 1.0 else mult > 1.0


def test_yarn_keeps_fast_and_divides_slow_frequencies():
    # over 1,000 positions the wavelength of index i fits 1000 f_i / (2 pi) times
    freq, _ = P.yarn_table(32, 1e4, {"factor": 10.0, "original": 1000, "fast": 20.0, "slow": 2.0})
    plain = 1e4 ** (-2.0 * torch.arange(16, dtype=torch.float64) / 32)
    turns = 1000 * plain / (2 * math.pi)
    assert torch.allclose(freq[turns > 40], plain[turns > 40]) and int((turns > 40).sum()) >= 2
    dim = lambda t: 32 * math.log(1000 / (2 * math.pi * t)) / (2 * math.log(1e4))
    late = torch.arange(16) >= math.ceil(dim(2.0))
    assert torch.allclose(freq[late], plain[late] / 10.0) and int(late.sum()) >= 2
    mid = (torch.arange(16) > math.floor(dim(20.0))) & ~late
    assert (freq[mid] < plain[mid]).all() and (freq[mid] > plain[mid] / 10.0).all() and int(mid.sum()) >= 1


# ---- the plain implementation's own identities ----------------------------------------------------------------------
def test_rotation_pairs_and_angles():
    x = torch.zeros((3, 1, 8), dtype=torch.float64)
    x[:, 0, 2] = 1.0                                  # of two pairs, the second: dimensions 2 and 3
    x[:, 0, 6] = 2.0                                  # beyond the rotated part: passes
    f = torch.tensor([1.0, 0.3], dtype=torch.float64)
    y = P.rotate_pairs(x, f, 1.5)
    for p in range(3):
        want = [0, 0, 1.5 * math.cos(0.3 * p), 1.5 * math.sin(0.3 * p), 0, 0, 2.0, 0]
        assert torch.allclose(y[p, 0], torch.tensor(want, dtype=torch.float64))
    q, k = torch.randn((9, 1, 4), dtype=torch.float64), torch.randn((9, 1, 4), dtype=torch.float64)
    q[:], k[:] = q[:1], k[:1]                         # the same vector at every place: the product depends on the distance alone
    s = P.rotate_pairs(q, f, 1.0)[:, 0] @ P.rotate_pairs(k, f, 1.0)[:, 0].T
    assert torch.allclose(s[5, 2], s[8, 5]) and not torch.allclose(s[5, 2], s[5, 3])


def test_sigmoid_weights_window_and_distance():
    q = torch.zeros((10, 4), dtype=torch.float64)
    w = P.sigmoid_weights(q, q, 0.5, torch.tensor(0.0), torch.tensor(1.0), torch.tensor(-1.0), 4)
    one = 1.0 / (1.0 + math.e)
    assert torch.allclose(w[7], torch.tensor([0, 0, 0, 0, one, one, one, one, 0, 0], dtype=torch.float64))     # not normalised; four keys
    w = P.sigmoid_weights(q, q, 0.5, torch.tensor(2.0), torch.tensor(0.5), torch.tensor(0.0), 10)
    assert torch.allclose(w[9, 3], torch.tensor(1.0 / (1.0 + (1 + 0.5 * 6) ** 2.0), dtype=torch.float64))
    w = P.sigmoid_weights(q, q, 0.5, torch.tensor(2.0), torch.tensor(0.5), torch.tensor(0.0), 1)
    assert torch.allclose(w, torch.eye(10, dtype=torch.float64) * 0.5)


def test_clamped_unit():
    p = {"gate": torch.tensor([[1.0], [1.0], [1.0]], dtype=torch.float64), "up": torch.tensor([[1.0], [9.0], [-9.0]], dtype=torch.float64),
         "down": torch.eye(3, dtype=torch.float64)}
    y = P.clamped_unit(torch.tensor([[5.0], [-5.0]], dtype=torch.float64), p, 2.0)
    g = 2.0 / (1.0 + math.exp(-1.702 * 2.0))          # the gate is cut above only ...
    assert torch.allclose(y[0], torch.tensor([3.0 * g, 3.0 * g, -1.0 * g], dtype=torch.float64))
    g = -5.0 / (1.0 + math.exp(1.702 * 5.0))          # ... and passes below; up is cut on both sides
    assert torch.allclose(y[1], torch.tensor([-1.0 * g, -1.0 * g, 3.0 * g], dtype=torch.float64))


def test_a_choices_weight_goes_into_its_expert():
    g = torch.Generator().manual_seed(0)
    h = torch.randn((20, 8), generator=g, dtype=torch.float64) * 0.5
    p = {"router": torch.randn((3, 8), generator=g, dtype=torch.float64)}
    for e in range(3):
        p.update({f"e{e}.gate": torch.randn((5, 8), generator=g, dtype=torch.float64), f"e{e}.up": torch.randn((5, 8), generator=g, dtype=torch.float64),
                  f"e{e}.down": torch.randn((8, 5), generator=g, dtype=torch.float64)})
    idx, wt = P.route(h, p["router"], 2)
    assert ((wt > 0) & (wt < 1)).all() and not torch.allclose(wt.sum(-1), torch.ones(20, dtype=torch.float64))
    assert (wt[:, 0] >= wt[:, 1]).all()
    y = P.routed_feed_forward(h, p, {"router": {"top": 2}})
    t = int(torch.argmin(wt[:, 0]))
    by_hand = sum(P.expert((wt[t, j] * h[t])[None], *(p[f"e{int(idx[t, j])}.{n}"] for n in ("gate", "up", "down")))[0] for j in range(2))
    outside = sum(wt[t, j] * P.expert(h[t][None], *(p[f"e{int(idx[t, j])}.{n}"] for n in ("gate", "up", "down")))[0] for j in range(2))
    assert torch.allclose(y[t], by_hand) and not torch.allclose(y[t], outside, rtol=1e-2)


@pytest.mark.parametrize("name", sorted(ZIBINEX))
def test_test_weights_make_faults_visible(name):
    """The weights the device tests run with: a first token that is changed moves the last logits; every position's choice of
    experts is clear where that is asked for."""
    raw = ZIBINEX[name]()
    w = make_weights(raw, 3, clear_choices=True)
    ids, margins = token_ids(60, raw["vocab"], 1), []
    a = P.forward(raw, w, ids, margins=margins)
    b = P.forward(raw, w, [(ids[0] + 1) % raw["vocab"]] + ids[1:])
    assert min((float(m.min()) for m in margins), default=1.0) > 0.02
    assert float((a[-1] - b[-1]).abs().max()) > 1e-3 * float(a[-1].abs().max())
