"""A plain, slow implementation of the Zibinex design on whole sequences, one function per mechanism, written from the
design's equations in float64 (or any dtype given). It shares no code with the package: tensors in, tensors out.

Notation: T tokens, W width; a linear weight is [out, in] and applied as x @ w.T; positions count from 0.
"""
import math

import torch


def rms_norm(x, w, eps, one_plus=False):
    """y = x / sqrt(mean(x^2) + eps) * w over the last axis (one_plus: the weight is 1 + w)."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y * (1.0 + w) if one_plus else y * w


# ---- positions ----------------------------------------------------------------------------------------------------------
def yarn_table(dims, base, scaling):
    """(frequencies [dims / 2], factor on cosine and sine). A frequency whose wavelength fits the original length often (more
    than `fast` turns) stays, one that turns less than `slow` times is divided by `factor`, those between are blended."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / dims)
    if scaling is None:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x, freq, mult):
    """x [T, heads, d]: dimension 2i turns with dimension 2i + 1 by position * freq[i]; cosine and sine times mult; dimensions
    from 2 * len(freq) on pass."""
    T = x.shape[0]
    n = 2 * freq.numel()
    ang = torch.arange(T, dtype=torch.float64)[:, None] * freq[None, :]
    c, s = (torch.cos(ang) * mult).to(x.dtype)[:, None, :], (torch.sin(ang) * mult).to(x.dtype)[:, None, :]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


# ---- mixers -------------------------------------------------------------------------------------------------------------
def latent_attention(h, p, m, eps):
    """Keys and values of every head are up-projections of one normed latent per token; a rotated key part, shared by the
    heads, joins each head's key; softmax over j <= i; one output gate per head."""
    T = h.shape[0]
    H, d, rd, e, r = m["heads"], m["dim"], m.get("rot_dim") or 0, m["vdim"], m["kv_rank"]
    q = (h @ p["q"].T).view(T, H, d + rd)
    ckr = h @ p["dkv"].T
    c = rms_norm(ckr[:, :r], p["dkv.norm"], eps)
    qn, qr, kr = q[..., :d], q[..., d:], ckr[:, None, r:]
    if rd:
        freq, mult = yarn_table(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        qr, kr = rotate_pairs(qr, freq, mult), rotate_pairs(kr, freq, mult)
    k = (c @ p["uk"].T).view(T, H, d)
    v = (c @ p["uv"].T).view(T, H, e)
    late = torch.triu(torch.ones(T, T, dtype=torch.bool), diagonal=1)
    out = []
    for j in range(H):
        s = (qn[:, j] @ k[:, j].T + qr[:, j] @ kr[:, 0].T) * m["scale"]
        out.append(torch.softmax(s.masked_fill(late, -math.inf), dim=-1) @ v[:, j])
    o = torch.stack(out, dim=1) * torch.sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(T, H * e) @ p["o"].T


def sigmoid_weights(q, k, scale, r1, r2, pb, window):
    """Weights [T, T] of one head: sigmoid(scale q_i.k_j - r1 ln(1 + r2 (i - j)) + pb) for 0 <= i - j < window, else 0."""
    T = q.shape[0]
    n = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    s = (q @ k.T) * scale - r1 * torch.log(1.0 + r2 * n.clamp(min=0).to(q.dtype)) + pb
    return torch.where((n >= 0) & (n < window), torch.sigmoid(s), torch.zeros((), dtype=q.dtype))


def sigmoid_attention(h, p, m, eps):
    """Grouped-query attention with normed queries and keys, biased projections, a penalty by the distance's logarithm, a
    sliding window, and weights that are each key's own sigmoid (they do not sum to one)."""
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads") or H
    q = rms_norm((h @ p["q"].T + p["q.b"]).view(T, H, d), p["q.norm"], eps)
    k = rms_norm((h @ p["k"].T + p["k.b"]).view(T, G, d), p["k.norm"], eps)
    v = (h @ p["v"].T + p["v.b"]).view(T, G, e)
    out = []
    for j in range(H):
        g = j // (H // G)
        out.append(sigmoid_weights(q[:, j], k[:, g], m["scale"], p["r1"][j], p["r2"][j], p["pb"][j], m["mask"]["size"]) @ v[:, g])
    return torch.stack(out, dim=1).reshape(T, H * e) @ p["o"].T


# ---- feed-forwards --------------------------------------------------------------------------------------------------------
def clamped_unit(h, p, limit):
    g = (h @ p["gate"].T).clamp(max=limit)
    u = (h @ p["up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ p["down"].T


def expert(x, w_gate, w_up, w_down):
    z = x @ w_gate.T
    return (z * torch.sigmoid(z) * (x @ w_up.T)) @ w_down.T


def route(h, w_router, top, margins=None):
    """Scores sigmoid(router logits); the `top` largest are chosen and are the weights as they stand. margins (a list or None)
    receives per token the gap between the last chosen and the first rejected logit."""
    z = h @ w_router.T
    full = torch.sort(z, dim=-1, descending=True, stable=True)
    if margins is not None:
        v = full.values
        margins.append(v[:, top - 1] - v[:, top] if top < v.shape[1] else torch.full((h.shape[0],), math.inf, dtype=h.dtype))
    idx = full.indices[:, :top]
    return idx, torch.sigmoid(torch.gather(z, 1, idx))


def routed_feed_forward(h, p, f, margins=None):
    """A chosen expert runs on its weight times the token's row; the outputs are summed as they come."""
    idx, wt = route(h, p["router"], f["router"]["top"], margins)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            n = int(idx[t, j])
            out[t] += expert(wt[t, j] * h[t][None], p[f"e{n}.gate"], p[f"e{n}.up"], p[f"e{n}.down"])[0]
    return out


# ---- the model ------------------------------------------------------------------------------------------------------------
def sub(tensors, prefix):
    return {k[len(prefix) + 1:]: v for k, v in tensors.items() if k.startswith(prefix + ".")}


def owner(cfg, i):
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, tensors, tokens, dtype=torch.float64, want_layers=False, margins=None):
    """cfg: the parsed config.json; tensors: name -> tensor. Returns logits [T, vocab] (and the residual stream after every
    layer, [layers, T, W])."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kept = []
    for i, L in enumerate(cfg["layers"]):
        n = f"l{owner(cfg, i)}"
        p, m = sub(w, n + ".mix"), L["mixer"]
        h = rms_norm(x, w[n + ".norm1"], eps, one_plus=True)
        y = latent_attention(h, p, m, eps) if L["type"] == "latent_attention" else sigmoid_attention(h, p, m, eps)
        x = x + rms_norm(y, w[n + ".norm1b"], eps, one_plus=True)
        f = L.get("mlp")
        if f is not None:
            h = rms_norm(x, w[n + ".norm2"], eps, one_plus=True)
            q = sub(w, n + ".mlp")
            y = clamped_unit(h, q, f["limit"]) if f["kind"] == "dense" else routed_feed_forward(h, q, f, margins)
            x = x + rms_norm(y, w[n + ".norm2b"], eps, one_plus=True)
        kept.append(x)
    logits = rms_norm(x, w["final.norm"], eps, one_plus=True) @ w["embed"].T
    return (logits, torch.stack(kept)) if want_layers else logits


def greedy_generate(cfg, tensors, prompt, n, dtype=torch.float64):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(torch.argmax(forward(cfg, tensors, ids, dtype)[-1])))
    return ids[len(prompt):]
