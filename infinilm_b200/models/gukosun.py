"""Gukosun described as data: a decoder whose sublayers read one norm and join the stream together, each under a factor per
column, and whose layers end with an input of their own from the token (a row of a table, gated by the stream). A layer mixes
tokens in one of two ways - "attention": grouped-query attention over a sliding window without positions, queries and keys normed
per head, a learned sink per head, values blended with those of the first layer of this kind that blends, a gate per column;
"parallel": two mixers side by side, softmax attention over all positions (queries and keys normed over the whole projection,
neighbouring dimensions rotated as pairs, capped scores, a learned sink, a gate per head) and a decayed linear attention, half the
sum of both, each normed over the model width. Feed-forwards are down(relu(up(h))^2).

config.json: `vocab`, `width`, `norm.eps`, `logit_scale`, `token_side.dim` (absent or 0: no token input), `layers` (per layer `type`,
`mixer` with its sizes and constants - `left` and `right` in a parallel layer -, `mlp` - `kind` "dense" with `ff` - or null). Tensors:
`embed`, `side.embed` [vocab, layers * dim], `l<i>.norm1|ls1|ls2`, `l<i>.mix.*`, `l<i>.mlp.up|down`, `l<i>.side.gate|proj|norm`,
`final.norm`, `head`. The constants of the design that are not in config.json: the weight 1/2 of a parallel layer's two halves.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from ..config.model_config import ConfigError, ModelConfig, take
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunStep

HALF = 0.5
MIXERS = ("attention", "parallel")
FEED_FORWARDS = ("dense",)


def _obj(raw: Dict[str, Any], key: str, required: bool = True) -> Optional[Dict[str, Any]]:
    v = raw.get(key)
    if v is None:
        if required:
            raise ConfigError(f"config.json: required key '{key}' is missing")
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: key '{key}' must be an object")
    return v


def _heads(m: Dict[str, Any]) -> Dict[str, Any]:
    out = {"heads": take(m, "heads", int), "dim": take(m, "dim", int), "scale": take(m, "scale", float)}
    out["kv_heads"], out["vdim"] = take(m, "kv_heads", int, out["heads"]), take(m, "vdim", int, out["dim"])
    return out


def _rot(m: Dict[str, Any], dim: int) -> Optional[Dict[str, Any]]:
    rot = _obj(m, "rot", required=False)
    if rot is None or take(rot, "dims", int, dim) == 0:
        return None
    out = {"dims": take(rot, "dims", int, dim), "base": take(rot, "base", float), "scaling": None}
    if out["dims"] % 2 or not 0 < out["dims"] <= dim:
        raise ConfigError("config.json: rot.dims must be even and at most the head's dim")
    sc = _obj(rot, "scaling", required=False)
    if sc is not None:
        out["scaling"] = {k: take(sc, k, float) for k in ("factor", "original", "low", "high")}
        if min(out["scaling"]["factor"], out["scaling"]["original"]) <= 0.0 or not out["scaling"]["low"] < out["scaling"]["high"]:
            raise ConfigError("config.json: rot.scaling needs a positive factor and original, and low below high")
    return out


def _left(m: Dict[str, Any]) -> Dict[str, Any]:
    out = _heads(m)
    out["rot"] = _rot(m, out["dim"])
    cap = take(m, "softcap", float, None)
    if cap is not None and cap < 0.0:
        raise ConfigError("config.json: softcap must be positive")
    out["cap"] = cap or None
    return out


def _right(m: Dict[str, Any]) -> Dict[str, Any]:
    out = {k: take(m, k, int) for k in ("heads", "dim")}
    out["vdim"] = take(m, "vdim", int, out["dim"])
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != out["heads"] or not all(isinstance(x, (int, float)) and not isinstance(x, bool) for x in decay):
        raise ConfigError("config.json: 'decay' must list one number per head")
    out["decay"] = [float(x) for x in decay]
    return out


def _windowed(m: Dict[str, Any]) -> Dict[str, Any]:
    out = _heads(m)
    mask = _obj(m, "mask", required=False)
    out["window"] = None if mask is None else take(mask, "size", int)
    if out["window"] is not None and out["window"] < 1:
        raise ConfigError("config.json: mask.size must be positive")
    out["v_mix"] = take(m, "v_mix", bool, False)
    return out


@dataclass
class GukosunConfig(ModelConfig):
    norm_eps: float = 0.0
    logit_scale: float = 1.0
    side_dim: int = 0
    layers: List[Dict[str, Any]] = field(default_factory=list)

    @classmethod
    def from_json(cls, raw: Dict[str, Any]) -> "GukosunConfig":
        raw = dict(raw)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        out_layers, shared = [], None
        for i, L in enumerate(layers):
            typ = take(L, "type", str)
            if typ not in MIXERS:
                raise ConfigError(f"config.json: layer {i} has mixer type {typ!r} (known: {', '.join(MIXERS)})")
            m = _obj(L, "mixer")
            if typ == "parallel":
                mixer = {"left": _left(_obj(m, "left")), "right": _right(_obj(m, "right"))}
            else:
                mixer = _windowed(m)
                if mixer["v_mix"]:                # blended values are laid out alike
                    layout = (mixer["kv_heads"], mixer["vdim"])
                    if shared is not None and layout != shared:
                        raise ConfigError(f"config.json: layer {i} blends its values with an earlier layer's of another layout")
                    shared = layout
            f = _obj(L, "mlp", required=False)
            mlp = None
            if f is not None:
                kind = take(f, "kind", str)
                if kind not in FEED_FORWARDS:
                    raise ConfigError(f"config.json: layer {i} has feed-forward kind {kind!r} (known: {', '.join(FEED_FORWARDS)})")
                mlp = {"kind": kind, "ff": take(f, "ff", int)}
            out_layers.append({"type": typ, "mixer": mixer, "mlp": mlp})
        cfg = cls(architecture="Gukosun", model_type="gukosun", vocab_size=take(raw, "vocab", int), hidden_size=take(raw, "width", int),
                  max_position_embeddings=1 << 30, torch_dtype="bfloat16", eos_token_ids=[], raw=raw,
                  norm_eps=take(_obj(raw, "norm"), "eps", float), logit_scale=take(raw, "logit_scale", float, 1.0),
                  side_dim=take(_obj(raw, "token_side", required=False) or {}, "dim", int, 0), layers=out_layers)
        if cfg.vocab_size <= 0 or cfg.hidden_size <= 0 or cfg.side_dim < 0:
            raise ConfigError("config.json: vocab and width must be positive, token_side.dim not negative")
        return cfg


def describe(cfg: GukosunConfig) -> ModelSpec:
    W, eps, n_side = cfg.hidden_size, cfg.norm_eps, cfg.side_dim

    def norm(prefix: str, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": W, "eps": eps, "name": name}, prefix)

    def softmax(m: Dict[str, Any], **more) -> Dict[str, Any]:
        return dict({"hidden": W, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "qk_dim": m["dim"], "v_dim": m["vdim"], "scale": m["scale"],
                     "eps": eps, "sink": "learned", "output_gate": True}, **more)
    layers, blended = [], False
    for i, L in enumerate(cfg.layers):
        m, f = L["mixer"], L["mlp"]
        if L["type"] == "parallel":
            l, r = m["left"], m["right"]
            pos = None
            if l["rot"] is not None:
                rot = {"rot_dim": l["rot"]["dims"], "theta": l["rot"]["base"], "interleaved": True}
                pos = PartSpec("rope", rot) if l["rot"]["scaling"] is None else PartSpec("llama3", dict(rot, **l["rot"]["scaling"]))
            left = PartSpec("qk_norm_attention", softmax(l, norm_over="projection", position=pos, score_cap=l["cap"], gate_per="head"), "left")
            right = PartSpec("decay_linear_attention", {"hidden": W, "n_heads": r["heads"], "qk_dim": r["dim"], "v_dim": r["vdim"],
                                                        "decay": r["decay"], "eps": eps}, "right")
            mixer = PartSpec("parallel", {"branches": [(left, HALF), (right, HALF)], "branch_norm_eps": eps, "branch_norm_width": W}, f"l{i}.mix")
        else:
            mix = None
            if m["v_mix"]:
                mix, blended = {"role": "later" if blended else "first", "key": "values"}, True
            mixer = PartSpec("qk_norm_attention", softmax(m, window=m["window"], value_mix=mix), f"l{i}.mix")
        ffn = None
        if f is not None:
            ffn = PartSpec("squared_relu", {"hidden": W, "intermediate": f["ff"], "names": {"up": "up", "down": "down"}}, f"l{i}.mlp")
        side = None
        if n_side:
            side = PartSpec("token_input", {"hidden": W, "dim": n_side, "offset": i * n_side, "eps": eps}, f"l{i}.side")
        layers.append(LayerSpec("parallel_residual", norm(f"l{i}", "norm1"), mixer, None, ffn, {"scales": f"l{i}", "token_input": side}))
    table = None
    if n_side:
        table = PartSpec("token_table", {"vocab": cfg.vocab_size, "width": len(cfg.layers) * n_side, "name": "embed"}, "side")
    return ModelSpec(
        embedding=PartSpec("token_embedding", {"vocab": cfg.vocab_size, "hidden": W, "scale": 1.0, "name": "embed", "exact": True}, ""),
        layers=layers, order=[RunStep(i) for i in range(len(layers))], final_norm=norm("final", "norm"), token_table=table,
        head=PartSpec("linear_head", {"vocab": cfg.vocab_size, "hidden": W, "scale": cfg.logit_scale, "tied_to": None, "name": "head"}, ""))


register_architecture(["Gukosun", "gukosun"], GukosunConfig, describe)
