"""Gukosun on the CPU: configuration and its faults, the description's parts, tensor names and cache needs, the random-weights
folder, tensors that a checkpoint may lack, the frequencies' scaling, and the plain implementation's own identities (a window's
edge, a sink's share, the cap, pairs of neighbours, blended values, the decayed sum, the token's own input)."""
import copy
import json
import math
import os

import pytest
import torch

import plain_gukosun as P
from gukosun_configs import GUKOSUN, att, dense, make_weights, token_ids

from infinilm_b200.config import ConfigError, config_from_json, describe_model
from infinilm_b200.models.causal_lm import CausalLM
from infinilm_b200.weights import FolderSource, check_against, write_model_folder


def _model(raw, dtype=torch.float32):
    return CausalLM(describe_model(config_from_json(raw)), dtype)


@pytest.mark.parametrize("name", sorted(GUKOSUN))
def test_tensor_names_and_cache_needs(name):
    raw = GUKOSUN[name]()
    model = _model(raw)
    specs = {p.full_name(ws.name): ws for p, ws in model.weight_specs()}
    names = {k: v.shape for k, v in specs.items()}
    W, V, sd, n = raw["width"], raw["vocab"], raw["token_side"]["dim"], len(raw["layers"])
    assert names["embed"] == names["head"] == (V, W) and names["final.norm"] == (W,) and names["side.embed"] == (V, n * sd)
    assert specs["head"].fallback is None and not any(".norm2" in k for k in names)
    needs = model.cache_needs()
    assert [s.layer for s in model.order] == list(range(n)) and len(needs) == n
    for i, L in enumerate(raw["layers"]):
        m, px, f = L["mixer"], f"l{i}.mix", L["mlp"]
        assert names[f"l{i}.norm1"] == names[f"l{i}.ls1"] == names[f"l{i}.side.norm"] == (W,)
        assert names[f"l{i}.side.gate"] == (sd, W) and names[f"l{i}.side.proj"] == (W, sd)
        assert specs[f"l{i}.ls2"].optional == (f is None) and not specs[f"l{i}.ls1"].optional
        if f is None:
            assert f"l{i}.mlp.up" not in names
        else:
            assert names[f"l{i}.mlp.up"] == (f["ff"], W) and names[f"l{i}.mlp.down"] == (W, f["ff"])
        if L["type"] == "parallel":
            l, r = m["left"], m["right"]
            assert names[f"{px}.left.q.norm"] == (l["heads"] * l["dim"],) and names[f"{px}.left.k.norm"] == (l["kv_heads"] * l["dim"],)
            assert names[f"{px}.left.g"] == (l["heads"], W) and names[f"{px}.left.sink"] == (l["heads"],)
            assert names[f"{px}.left.out"] == names[f"{px}.right.out"] == (W,)
            assert names[f"{px}.right.norm"] == (r["heads"] * r["vdim"],) and names[f"{px}.right.g"] == (r["heads"] * r["vdim"], W)
            assert f"{px}.left.vmix" not in names
            assert [x.kind for x in needs[i]] == ["paged_kv", "state"] and needs[i][0].window is None
            assert needs[i][1].shape == (r["heads"], r["vdim"], r["dim"]) and needs[i][1].dtype == "float32"
        else:
            assert names[f"{px}.q"] == (m["heads"] * m["dim"], W) and names[f"{px}.v"] == (m["kv_heads"] * m["vdim"], W)
            assert names[f"{px}.q.norm"] == names[f"{px}.k.norm"] == (m["dim"],) and names[f"{px}.sink"] == (m["heads"],)
            assert names[f"{px}.g"] == (m["heads"] * m["vdim"], W) and names[f"{px}.o"] == (W, m["heads"] * m["vdim"])
            assert (names.get(f"{px}.vmix") == ()) == m["v_mix"]
            assert needs[i].kind == "paged_kv" and needs[i].window == m["mask"]["size"] and needs[i].n_kv_heads == m["kv_heads"]
            assert max(m["dim"], m["vdim"]) <= needs[i].head_dim < max(m["dim"], m["vdim"]) + 16
    assert model.graph_safe


def test_the_first_layer_that_blends_is_where_the_values_come_from():
    roles = [b.mixer.mix_role for b in _model(GUKOSUN["a"]()).blocks if hasattr(b.mixer, "mix_role")]
    assert roles == ["first", None, "later"]
    raw = GUKOSUN["a"]()
    raw["layers"][0]["mixer"]["v_mix"] = False        # the next one that blends takes the place
    raw["layers"].append(copy.deepcopy(raw["layers"][4]))
    assert [b.mixer.mix_role for b in _model(raw).blocks if hasattr(b.mixer, "mix_role")] == [None, None, "first", "later"]


def test_config_faults_name_the_key():
    def broken(change, match, exc=ConfigError):
        raw = GUKOSUN["a"]()
        change(raw)
        with pytest.raises(exc, match=match):
            _model(raw)
    broken(lambda r: r["layers"][0].update(type="something_else"), "something_else")
    broken(lambda r: r["layers"][0].pop("mixer"), "mixer")
    broken(lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), "mask.size")
    broken(lambda r: r["layers"][0]["mixer"].pop("scale"), "scale")
    broken(lambda r: r["layers"][0]["mlp"].update(kind="other"), "other")
    broken(lambda r: r["layers"][0]["mlp"].pop("ff"), "ff")
    broken(lambda r: r["layers"][1]["mixer"].pop("right"), "right")
    broken(lambda r: r["layers"][1]["mixer"]["right"].update(decay=[0.5]), "decay")
    broken(lambda r: r["layers"][1]["mixer"]["right"].update(decay=[0.5, "x", 0.1]), "decay")
    broken(lambda r: r["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "rot.dims")
    broken(lambda r: r["layers"][1]["mixer"]["left"]["rot"].update(dims=18), "rot.dims")
    broken(lambda r: r["layers"][1]["mixer"]["left"]["rot"].pop("base"), "base")
    broken(lambda r: r["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("low"), "low")
    broken(lambda r: r["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(low=6.0), "low")
    broken(lambda r: r["layers"][1]["mixer"]["left"].update(softcap=-1.0), "softcap")
    broken(lambda r: r["layers"][4]["mixer"].update(vdim=40), "layout")
    broken(lambda r: r["norm"].pop("eps"), "eps")
    broken(lambda r: r.update(width=0), "width")
    broken(lambda r: r["layers"][0]["mixer"].update(heads=5), "kv heads", ValueError)


def test_random_folder_round_trip_and_tensors_that_may_be_absent(tmp_path):
    raw = GUKOSUN["b"]()
    cfg = config_from_json(raw)
    folder = write_model_folder(cfg, 5, str(tmp_path / "m"))
    assert json.load(open(os.path.join(folder, "config.json"))) == raw
    src = FolderSource(folder)
    check_against(_model(raw, torch.bfloat16), src)
    assert src.info("l1.mix.vmix")[1] == () and "l2.ls2" not in src.names() and "l0.ls2" in src.names()      # (layer 2 has no feed-forward)
    src.close()
    from infinilm_b200.weights.loader import DictSource, WeightError
    w = make_weights(raw, 0)
    check_against(_model(raw), DictSource(w))
    check_against(_model(raw), DictSource(dict(w, **{"l2.ls2": w["l0.ls2"]})))        # a factor nothing uses may be there
    with pytest.raises(WeightError, match="l0.ls2"):
        check_against(_model(raw), DictSource({k: v for k, v in w.items() if k != "l0.ls2"}))


def test_a_model_without_token_input():
    raw = GUKOSUN["a"]()
    raw.pop("token_side")
    names = {p.full_name(ws.name) for p, ws in _model(raw).weight_specs()}
    assert not any("side" in n for n in names)


@pytest.mark.parametrize("dims,base,scaling", [(16, 1e4, (4.0, 1.0, 4.0, 256)), (6, 10.0, (16.0, 0.7, 1.9, 40)), (64, 1e6, (2.0, 0.5, 3.0, 64)),
                                               (2, 20.0, (3.0, 1.0, 2.0, 100)), (128, 5e5, (8.0, 1.0, 4.0, 8192))])
def test_scaled_frequencies(dims, base, scaling):
    from infinilm_b200.parts.position import Llama3Rope
    sc = dict(zip(("factor", "low", "high", "original"), scaling))
    part = Llama3Rope({"rot_dim": dims, "theta": base, "interleaved": True, **sc}, "", torch.float32)
    part.to_device(torch.device("cpu"))
    freq = P.stretched_frequencies(dims, base, sc)
    assert part.interleaved and part.mscale == 1.0 and torch.allclose(part.freq64, freq, rtol=1e-13)
    plain = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    wave = 2 * math.pi / plain
    short, long = wave < sc["original"] / sc["high"], wave > sc["original"] / sc["low"]
    assert torch.allclose(freq[short], plain[short]) and torch.allclose(freq[long], plain[long] / sc["factor"])
    mid = ~short & ~long
    assert ((freq[mid] < plain[mid] * (1 + 1e-9)) & (freq[mid] > plain[mid] / sc["factor"] * (1 - 1e-9))).all()


# ---- the plain implementation's own identities ----------------------------------------------------------------------
def test_sink_cap_and_window_in_the_weights():
    q = torch.zeros((10, 4), dtype=torch.float64)
    w = P.weights_with_sink(q, q, 0.5, torch.tensor(math.log(3.0)), window=4)
    assert torch.allclose(w[7], torch.tensor([0, 0, 0, 0] + [1 / 7.0] * 4 + [0, 0], dtype=torch.float64))      # four keys of weight 1, a sink of 3
    assert torch.allclose(w[0, :1], torch.tensor([0.25], dtype=torch.float64))
    assert torch.allclose(P.weights_with_sink(q, q, 0.5, torch.tensor(-1e4), window=1), torch.eye(10, dtype=torch.float64))
    q = torch.tensor([[1000.0], [1000.0]], dtype=torch.float64)
    k = torch.tensor([[1.0], [-1.0]], dtype=torch.float64)
    w = P.weights_with_sink(q, k, 1.0, torch.tensor(-1e4), cap=2.0)           # scores of plus and minus 1,000 become 2 and -2; the sink is not capped
    assert torch.allclose(w[1], torch.softmax(torch.tensor([2.0, -2.0], dtype=torch.float64), 0))


def test_rotation_turns_neighbours():
    x = torch.zeros((3, 1, 8), dtype=torch.float64)
    x[:, 0, 2], x[:, 0, 6] = 1.0, 2.0                 # of two pairs the second; a dimension beyond the rotated part
    y = P.rotate_neighbours(x, torch.tensor([1.0, 0.3], dtype=torch.float64))
    for p in range(3):
        assert torch.allclose(y[p, 0], torch.tensor([0, 0, math.cos(0.3 * p), math.sin(0.3 * p), 0, 0, 2.0, 0], dtype=torch.float64))


def test_values_are_blended_with_the_first_layers():
    raw = GUKOSUN["a"]()
    W = raw["width"]
    raw["layers"] = [att(2, 1, 8, 16, 0.3, 5, None), att(2, 1, 8, 16, 0.3, 5, None)]
    w = make_weights(raw, 1)
    ids = token_ids(20, raw["vocab"], 2)
    w["l1.mix.vmix"] = torch.tensor(1.0)              # all of the first layer's values: the second layer's own do not matter ...
    a = P.forward(raw, w, ids)
    w["l1.mix.v"] = torch.zeros(16, W)
    assert torch.equal(P.forward(raw, w, ids), a)
    w["l0.mix.vmix"] = torch.tensor(0.9)              # ... and the first layer's blend is not used
    assert torch.equal(P.forward(raw, w, ids), a)
    w["l1.mix.vmix"] = torch.tensor(0.5)
    assert not torch.allclose(P.forward(raw, w, ids), a)


def test_decayed_sum_by_hand():
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn((6, 2, n), generator=g, dtype=torch.float64) for n in (3, 3, 5))
    dec = torch.tensor([0.5, 0.9], dtype=torch.float64)
    o = P.decayed_sum(q, k, v, dec)
    want = sum(dec[1] ** (5 - j) * (q[5, 1] @ k[j, 1]) * v[j, 1] for j in range(6))
    assert torch.allclose(o[5, 1], want)


def test_token_input_is_gated_by_the_stream():
    p = {"gate": torch.zeros((2, 3), dtype=torch.float64), "proj": torch.ones((3, 2), dtype=torch.float64), "norm": torch.ones(3, dtype=torch.float64)}
    x, e = torch.randn((4, 3), dtype=torch.float64), torch.randn((4, 2), dtype=torch.float64)
    assert float(P.token_input(x, e, p, 1e-5).abs().max()) == 0.0          # gelu(0) = 0
    p["gate"][0, 0] = 1.0
    y = P.token_input(x, e, p, 1e-5)
    s = P.gelu_tanh(x[:, 0]) * e[:, 0]
    assert torch.allclose(y[:, 0], s / torch.sqrt(s * s + 1e-5))


def _err(a, b):
    a, b = a - a.mean(-1, keepdim=True), b - b.mean(-1, keepdim=True)
    return (a - b).pow(2).mean(-1).sqrt() / b.pow(2).mean(-1).sqrt()


@pytest.mark.parametrize("name", sorted(GUKOSUN))
def test_test_weights_make_faults_visible(name):
    """The weights the device tests run with: a window one position off, scores without their cap, softmax without its sinks,
    values without their blend, frequencies without their scaling move the logits of most late positions far beyond what the
    device tests allow a float32 run, and a first token that is changed moves the last."""
    raw = GUKOSUN[name]()
    w = make_weights(raw, 3)
    ids = token_ids(90, raw["vocab"], 1)
    ref = P.forward(raw, w, ids)

    def moved(cfg, weights, at_least, what):
        err = _err(P.forward(cfg, weights, ids), ref)[-50:]
        assert float(err.median()) > at_least, f"{what}: {float(err.median()):.1e}"
    for d in (-1, 1):
        cfg = copy.deepcopy(raw)
        for L in cfg["layers"]:
            if L["type"] == "attention" and L["mixer"]["mask"]["size"] + d > 0:
                L["mixer"]["mask"]["size"] += d
        moved(cfg, w, 5e-3, f"window {d:+d}")
    moved(raw, {k: (v - 100 if k.endswith(".sink") else v) for k, v in w.items()}, 2e-2, "no sinks")
    moved(raw, {k: (v * 0 if k.endswith(".vmix") else v) for k, v in w.items()}, 1e-2, "no blend")
    moved(raw, {k: (v * 0 if k.endswith(".side.norm") else v) for k, v in w.items()}, 1e-1, "no token input")
    cfg = copy.deepcopy(raw)
    for L in cfg["layers"]:
        if L["type"] == "parallel":
            L["mixer"]["left"].pop("softcap", None)
    moved(cfg, w, 2e-2, "no cap")
    cfg, scaled = copy.deepcopy(raw), False
    for L in cfg["layers"]:
        if L["type"] == "parallel" and "scaling" in L["mixer"]["left"].get("rot", {}):
            scaled = bool(L["mixer"]["left"]["rot"].pop("scaling"))
    if scaled:
        moved(cfg, w, 5e-3, "no scaling")
    other = P.forward(raw, w, [(ids[0] + 1) % raw["vocab"]] + ids[1:])
    assert float(_err(other, ref)[-1]) > 1e-3
