"""A plain, slow implementation of the Gukosun design on whole sequences, one function per mechanism, written from the
design's equations in float64 (or any dtype given). It shares no code with the package: tensors in, tensors out.

Notation: T tokens, W width; a linear weight is [out, in] and applied as x @ w.T; positions count from 0.
"""
import math

import torch


def rms_norm(x, w, eps):
    """y = x / sqrt(mean(x^2) + eps) * w over the last axis (w None: no weight)."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


# ---- positions ----------------------------------------------------------------------------------------------------------
def stretched_frequencies(dims, base, scaling):
    """Frequencies [dims / 2] of a rotary encoding, base^(-2i / dims). With `scaling` those with a long wavelength are divided by
    `factor`, those with a short one stay, and those between take a blend that is linear in original / wavelength."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            turns = scaling["original"] * f / (2.0 * math.pi)          # how often it turns over the original length
            if turns < scaling["low"]:
                f = f / scaling["factor"]
            elif turns <= scaling["high"]:
                s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_neighbours(x, freq):
    """x [T, heads, d]: dimension 2i turns with dimension 2i + 1 by position * freq[i]; the dimensions behind pass."""
    T, n = x.shape[0], 2 * freq.numel()
    ang = torch.arange(T, dtype=torch.float64)[:, None] * freq[None, :]
    c, s = torch.cos(ang).to(x.dtype)[:, None, :], torch.sin(ang).to(x.dtype)[:, None, :]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


# ---- softmax attention ----------------------------------------------------------------------------------------------------
def weights_with_sink(q, k, scale, sink, window=None, cap=None):
    """Attention weights [T, T] of one head: softmax over the visible keys of cap * tanh(scale q.k / cap) (cap None: scale q.k),
    exp(sink) joining the denominator; visible are 0 <= i - j (< window)."""
    T = q.shape[0]
    n = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    s = (q @ k.T) * scale
    if cap is not None:
        s = cap * torch.tanh(s / cap)
    seen = (n >= 0) if window is None else (n >= 0) & (n < window)
    s = s.masked_fill(~seen, -math.inf)
    top = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attend(q, k, v, scale, sink, window=None, cap=None):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; head h reads key/value head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    return torch.stack([weights_with_sink(q[:, h], k[:, h // (H // G)], scale, sink[h], window, cap) @ v[:, h // (H // G)] for h in range(H)], dim=1)


def windowed_attention(h, p, m, eps, first_values=None):
    """Normed queries and keys (per head), no positions, a window, a sink, values blended with an earlier layer's, one gate per
    column. Returns (output, the layer's own values before any blending)."""
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads") or H
    q = rms_norm((h @ p["q"].T).view(T, H, d), p["q.norm"], eps)
    k = rms_norm((h @ p["k"].T).view(T, G, d), p["k.norm"], eps)
    v = own = h @ p["v"].T
    if first_values is not None:
        v = (1.0 - p["vmix"]) * v + p["vmix"] * first_values
    o = attend(q, k, v.view(T, G, e), m["scale"], p["sink"], window=m["mask"]["size"])
    o = o.reshape(T, H * e) * torch.sigmoid(h @ p["g"].T)
    return o @ p["o"].T, own


def rotated_attention(h, p, m, eps):
    """The left half of a parallel layer: queries and keys normed over the whole projection, rotated, capped scores, a sink, one
    gate per head, all positions up to the token's own."""
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads") or H
    q = rms_norm(h @ p["q"].T, p["q.norm"], eps).view(T, H, d)
    k = rms_norm(h @ p["k"].T, p["k.norm"], eps).view(T, G, d)
    if m.get("rot"):
        freq = stretched_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        q, k = rotate_neighbours(q, freq), rotate_neighbours(k, freq)
    v = (h @ p["v"].T).view(T, G, e)
    o = attend(q, k, v, m["scale"], p["sink"], cap=m.get("softcap"))
    o = o * torch.sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(T, H * e) @ p["o"].T


# ---- the decayed sum of outer products --------------------------------------------------------------------------------------
def silu(x):
    return x * torch.sigmoid(x)


def decayed_sum(q, k, v, decay):
    """Per head S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, from nothing. q, k [T, H, d], v [T, H, e] -> [T, H, e]."""
    T, H, d = q.shape
    S = torch.zeros((H, d, v.shape[2]), dtype=q.dtype)
    out = []
    for t in range(T):
        S = S * decay[:, None, None] + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def linear_attention(h, p, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(h @ p[n].T).view(T, H, -1) for n in ("q", "k", "v"))
    o = decayed_sum(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)).reshape(T, H * e)
    return (rms_norm(o, p["norm"], eps) * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def parallel_mixer(h, p, m, eps):
    """Half the sum of both halves, each normed over the width."""
    left = rms_norm(rotated_attention(h, sub(p, "left"), m["left"], eps), p["left.out"], eps)
    right = rms_norm(linear_attention(h, sub(p, "right"), m["right"], eps), p["right.out"], eps)
    return 0.5 * (left + right)


# ---- feed-forward and the token's own input -----------------------------------------------------------------------------------
def squared_relu_unit(h, p):
    z = (h @ p["up"].T).clamp(min=0.0)
    return (z * z) @ p["down"].T


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def token_input(x, e, p, eps):
    """What a layer adds at its end: the token's own row e [T, dim], gated by the stream, projected, normed."""
    return rms_norm((gelu_tanh(x @ p["gate"].T) * e) @ p["proj"].T, p["norm"], eps)


# ---- the model ------------------------------------------------------------------------------------------------------------
def sub(tensors, prefix):
    return {k[len(prefix) + 1:]: v for k, v in tensors.items() if k.startswith(prefix + ".")}


def forward(cfg, tensors, tokens, dtype=torch.float64, want_layers=False):
    """cfg: the parsed config.json; tensors: name -> tensor. Returns logits [T, vocab] (and the residual stream after every
    layer, [layers, T, W])."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][ids]
    n_side = (cfg.get("token_side") or {}).get("dim") or 0
    first_values = None
    kept = []
    for i, L in enumerate(cfg["layers"]):
        n, m, f = f"l{i}", L["mixer"], L.get("mlp")
        h = rms_norm(x, w[n + ".norm1"], eps)
        p = sub(w, n + ".mix")
        if L["type"] == "parallel":
            y = parallel_mixer(h, p, m, eps)
        else:
            y, own = windowed_attention(h, p, m, eps, first_values if m.get("v_mix") else None)
            if m.get("v_mix") and first_values is None:
                first_values = own
        y = y * w[n + ".ls1"]
        if f is not None:
            y = y + squared_relu_unit(h, sub(w, n + ".mlp")) * w[n + ".ls2"]
        x = x + y
        if n_side:
            x = x + token_input(x, w["side.embed"][ids][:, i * n_side:(i + 1) * n_side], sub(w, n + ".side"), eps)
        kept.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T * cfg.get("logit_scale", 1.0)
    return (logits, torch.stack(kept)) if want_layers else logits


def greedy_generate(cfg, tensors, prompt, n, dtype=torch.float64):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(torch.argmax(forward(cfg, tensors, ids, dtype)[-1])))
    return ids[len(prompt):]
