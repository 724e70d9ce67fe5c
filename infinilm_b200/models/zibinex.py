"""Zibinex described as data: a decoder with a norm in front of every sublayer and one on its output
(x += norm_b(sublayer(norm(x)))), whose layers mix tokens in one of two ways - "latent_attention": keys and values of every
head are up-projections of one normed latent per token, a rotated key part shared by the heads joins the scores (rotary
positions with YaRN scaling, dimension 2i paired with 2i + 1), one output gate per head; "attention": grouped-query attention
over a sliding window with biased projections, normed queries and keys, a penalty by the logarithm of the distance and
sigmoid weights in place of a softmax - and whose feed-forwards are a dense unit with a clamped gate or route each token to
the `top` of several small gated units by sigmoid scores, the score multiplying the unit's input. A layer may name an earlier
one whose weights it runs with (a cache of its own all the same).

config.json: `vocab`, `width`, `norm.eps`, `layers` (per layer `type`, `mixer` with its sizes and constants, `mlp` - `kind` "dense"
with `ff` and `limit`, "moe" with `expert.ff` and `router` {experts, top} - or null, and `weights_of`). Tensors: `embed` (also the
output head), `l<i>.norm1|norm1b|norm2|norm2b` (stored as deviations from one), `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`. The
constant of the design that is not in config.json: 1.702 in the clamped gate.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from ..config.model_config import ConfigError, ModelConfig, take
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunStep

GATE_ALPHA = 1.702
MIXERS = ("latent_attention", "attention")
FEED_FORWARDS = ("dense", "moe")


def _obj(raw: Dict[str, Any], key: str, required: bool = True) -> Optional[Dict[str, Any]]:
    v = raw.get(key)
    if v is None:
        if required:
            raise ConfigError(f"config.json: required key '{key}' is missing")
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: key '{key}' must be an object")
    return v


def _rot(m: Dict[str, Any], rot_dim: int) -> Optional[Dict[str, Any]]:
    if rot_dim == 0:
        return None
    rot = _obj(m, "rot")
    out = {"dims": take(rot, "dims", int, rot_dim), "base": take(rot, "base", float), "scaling": None}
    if out["dims"] % 2 or not 0 < out["dims"] <= rot_dim:
        raise ConfigError("config.json: rot.dims must be even and at most rot_dim")
    sc = _obj(rot, "scaling", required=False)
    if sc is not None:
        out["scaling"] = {k: take(sc, k, float) for k in ("factor", "original", "fast", "slow")}
        if min(out["scaling"].values()) <= 0.0:
            raise ConfigError("config.json: rot.scaling's numbers must be positive")
    return out


def _mixer(typ: str, m: Dict[str, Any]) -> Dict[str, Any]:
    out = {"heads": take(m, "heads", int), "dim": take(m, "dim", int), "scale": take(m, "scale", float)}
    out["vdim"] = take(m, "vdim", int, out["dim"])
    if typ == "latent_attention":
        out["kv_rank"], out["rot_dim"] = take(m, "kv_rank", int), take(m, "rot_dim", int, 0)
        out["rot"] = _rot(m, out["rot_dim"])
        return out
    out["kv_heads"] = take(m, "kv_heads", int, out["heads"])
    out["window"] = take(_obj(m, "mask"), "size", int)
    if out["window"] < 1:
        raise ConfigError("config.json: mask.size must be positive")
    return out


def _mlp(f: Dict[str, Any]) -> Dict[str, Any]:
    kind = take(f, "kind", str)
    if kind == "dense":
        return {"kind": kind, "ff": take(f, "ff", int), "limit": take(f, "limit", float)}
    if kind == "moe":
        r = _obj(f, "router")
        return {"kind": kind, "ff": take(_obj(f, "expert"), "ff", int), "experts": take(r, "experts", int), "top": take(r, "top", int)}
    raise ConfigError(f"config.json: feed-forward kind {kind!r} (known: {', '.join(FEED_FORWARDS)})")


@dataclass
class ZibinexConfig(ModelConfig):
    norm_eps: float = 0.0
    layers: List[Dict[str, Any]] = field(default_factory=list)
    tie_word_embeddings: bool = True              # the output head is the embedding table

    @classmethod
    def from_json(cls, raw: Dict[str, Any]) -> "ZibinexConfig":
        raw = dict(raw)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        out_layers = []
        for i, L in enumerate(layers):
            typ = take(L, "type", str)
            if typ not in MIXERS:
                raise ConfigError(f"config.json: layer {i} has mixer type {typ!r} (known: {', '.join(MIXERS)})")
            f = _obj(L, "mlp", required=False)
            out_layers.append({"type": typ, "mixer": _mixer(typ, _obj(L, "mixer")), "mlp": None if f is None else _mlp(f),
                               "weights_of": take(L, "weights_of", int, None)})
        for i, L in enumerate(out_layers):        # a layer that runs with another's weights is that layer in all else
            src, seen = L["weights_of"], {i}
            while src is not None:
                if not 0 <= src < len(out_layers) or src in seen:
                    raise ConfigError(f"config.json: layer {i}: weights_of must lead to a layer with weights of its own")
                seen.add(src)
                last, src = src, out_layers[src]["weights_of"]
            if L["weights_of"] is not None:
                if any(out_layers[last][k] != L[k] for k in ("type", "mixer", "mlp")):
                    raise ConfigError(f"config.json: layer {i} runs with layer {last}'s weights but differs from it")
                L["weights_of"] = last
        cfg = cls(architecture="Zibinex", model_type="zibinex", vocab_size=take(raw, "vocab", int), hidden_size=take(raw, "width", int),
                  max_position_embeddings=1 << 30, torch_dtype="bfloat16", eos_token_ids=[], raw=raw,
                  norm_eps=take(_obj(raw, "norm"), "eps", float), layers=out_layers)
        if cfg.vocab_size <= 0 or cfg.hidden_size <= 0:
            raise ConfigError("config.json: vocab and width must be positive")
        return cfg


def owned_layers(cfg: ZibinexConfig) -> List[int]:
    """The config's layers that have tensors of their own, in their order."""
    return [i for i, L in enumerate(cfg.layers) if L["weights_of"] is None]


def run_order(cfg: ZibinexConfig) -> List[RunStep]:
    """One entry - and so one cache - per layer of the config; a layer with `weights_of` runs that layer's block."""
    at = {i: n for n, i in enumerate(owned_layers(cfg))}
    return [RunStep(at[i if L["weights_of"] is None else L["weights_of"]]) for i, L in enumerate(cfg.layers)]


def describe(cfg: ZibinexConfig) -> ModelSpec:
    W, eps = cfg.hidden_size, cfg.norm_eps

    def norm(prefix: str, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": W, "eps": eps, "weight_offset": 1.0, "name": name}, prefix)
    layers = []
    for i in owned_layers(cfg):
        m, f, typ = cfg.layers[i]["mixer"], cfg.layers[i]["mlp"], cfg.layers[i]["type"]
        if typ == "latent_attention":
            pos = None
            if m["rot"] is not None:
                rot = {"rot_dim": m["rot"]["dims"], "theta": m["rot"]["base"], "interleaved": True}
                pos = PartSpec("rope", rot) if m["rot"]["scaling"] is None else PartSpec("yarn", dict(rot, **m["rot"]["scaling"]))
            mixer = PartSpec("latent_attention", {"hidden": W, "n_heads": m["heads"], "qk_dim": m["dim"], "v_dim": m["vdim"], "q_rank": None,
                                                  "kv_rank": m["kv_rank"], "scale": m["scale"], "eps": eps, "sink": False, "gate": True,
                                                  "gate_per": "head", "rot_part": m["rot_dim"], "position": pos}, f"l{i}.mix")
        else:
            mixer = PartSpec("qk_norm_attention", {"hidden": W, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "qk_dim": m["dim"],
                                                   "v_dim": m["vdim"], "scale": m["scale"], "eps": eps, "qkv_bias": True, "bias_in_norm": True,
                                                   "window": m["window"], "weights": "sigmoid", "distance_log": True}, f"l{i}.mix")
        ffn = ffn_norm = None
        branch_norms = {"mixer_branch_norm": norm(f"l{i}", "norm1b")}
        if f is not None:
            if f["kind"] == "dense":
                ffn = PartSpec("swiglu", {"hidden": W, "intermediate": f["ff"], "activation": "clamped", "limit": f["limit"], "alpha": GATE_ALPHA,
                                          "names": {"gate": "gate", "up": "up", "down": "down"}}, f"l{i}.mlp")
            else:
                ffn = PartSpec("routed_experts", {"hidden": W, "n_experts": f["experts"], "top": f["top"], "expert_ff": f["ff"], "shared_ff": None,
                                                  "router_bias": False, "route_rule": "sigmoid", "weight_on_input": True}, f"l{i}.mlp")
            ffn_norm = norm(f"l{i}", "norm2")
            branch_norms["ffn_branch_norm"] = norm(f"l{i}", "norm2b")
        layers.append(LayerSpec("sandwich_residual", norm(f"l{i}", "norm1"), mixer, ffn_norm, ffn, branch_norms))
    return ModelSpec(
        embedding=PartSpec("token_embedding", {"vocab": cfg.vocab_size, "hidden": W, "scale": 1.0, "name": "embed", "exact": True}, ""),
        layers=layers, order=run_order(cfg), final_norm=norm("final", "norm"),
        head=PartSpec("linear_head", {"vocab": cfg.vocab_size, "hidden": W, "scale": 1.0, "tied_to": "embed", "name": "head"}, ""))


register_architecture(["Zibinex", "zibinex"], ZibinexConfig, describe)
