"""Each mechanism of the Zibinex parts alone, on the device, against the plain implementation: the norm of a branch, the add
and the next norm in one pass (rows and routed rows); the latent with a rotated part beside it and its cache write; sigmoid
weights with a penalty by distance over a window in each of the four attention kernels, with a key that stands out just inside
and just outside the window and at page borders; the clamped gate in its three kernels; the routing rule, weights on the
experts' inputs for few and many rows; the gate per head; the latent mixer's few-row and many-row paths."""
import math

import pytest
import torch

import plain_zibinex as P

pytestmark = pytest.mark.gpu

DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def _i32(x, dev="cuda"):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def _close(got, ref, dtype, what, tol=None):
    got, ref = got.double().cpu(), ref.double()
    assert got.shape == ref.shape and torch.isfinite(got).all(), what
    tol = tol or (3e-5 if dtype == "float32" else 2.5e-2)
    err = float((got - ref).abs().max()) / max(float(ref.abs().max()), 1e-9)
    assert err <= tol, f"{what}: relative error {err:.2e}"


# ---- between two sublayers ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H", [(1, 72), (5, 120), (33, 256), (3, 2048), (2, 13), (2, 4096), (2, 3001), (2, 8192), (4, 1028)])
@pytest.mark.parametrize("top,weighted", [(0, False), (1, False), (3, True), (32, False)])
def test_norm_add_norm(cuda_device, dtype, T, H, top, weighted):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(T * H + top)
    dt = DT[dtype]
    resid = torch.randn(T, H, generator=g) * 3
    wb, wn = 1.0 + 0.3 * torch.randn(H, generator=g), 1.0 + 0.3 * torch.randn(H, generator=g)
    if top:
        y = (torch.randn(T * top, H, generator=g) * 2).to(dt)
        pos = torch.randperm(T * top, generator=g).to(torch.int32)
        wt = torch.rand(T, top, generator=g) if weighted else None
        rows = y.double()[pos.long()].view(T, top, H)
        branch = (rows * (wt.double()[:, :, None] if weighted else 1.0)).sum(1)
        arg = ops.RoutedRows(y.cuda(), pos.cuda(), wt.cuda() if weighted else None, top)
    else:
        y = (torch.randn(T, H, generator=g) * 2).to(dt)
        branch, arg = y.double(), y.cuda()
    want = resid.double() + P.rms_norm(branch, wb.double(), 1e-3)
    r, out = resid.clone().cuda(), torch.empty(T, H, dtype=dt, device="cuda")
    ops.norm_add_norm(r, arg, wb.cuda(), 1e-3, wn.cuda(), 1e-2, out)
    _close(r, want, "float32", "stream")
    _close(out, P.rms_norm(want, wn.double(), 1e-2), dtype, "next input", None if dtype == "float32" else 5e-3)
    r2 = resid.clone().cuda()
    ops.norm_add_norm(r2, arg, wb.cuda(), 1e-3)       # only the add
    assert torch.equal(r2, r)


def test_norm_add_norm_of_a_row_does_not_depend_on_the_batch(cuda_device):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(1)
    T, H = 40, 520
    resid, y = torch.randn(T, H, generator=g).cuda(), torch.randn(T, H, generator=g).to(torch.bfloat16).cuda()
    w = (1.0 + 0.1 * torch.randn(H, generator=g)).cuda()
    r, out = resid.clone(), torch.empty(T, H, dtype=torch.bfloat16, device="cuda")
    ops.norm_add_norm(r, y, w, 1e-5, w, 1e-5, out)
    for t in (0, 17, 39):
        r1, o1 = resid[t:t + 1].clone(), torch.empty(1, H, dtype=torch.bfloat16, device="cuda")
        ops.norm_add_norm(r1, y[t:t + 1].contiguous(), w, 1e-5, w, 1e-5, o1)
        assert torch.equal(r1[0], r[t]) and torch.equal(o1[0], out[t])


# ---- a latent with a rotated part -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nh,qd,r,rp,rot,interleaved", [(3, 16, 32, 8, 8, True), (1, 12, 24, 4, 4, True), (4, 64, 192, 64, 64, True), (2, 10, 50, 20, 12, True),
                                                        (5, 8, 16, 6, 2, True), (2, 32, 96, 32, 32, False), (7, 128, 512, 64, 64, True), (2, 5, 7, 3, 2, False)])
def test_latent_and_rotated_part_to_the_cache(cuda_device, dtype, nh, qd, r, rp, rot, interleaved):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(nh * qd + rp)
    dt = DT[dtype]
    hd = (r + rp + 15) // 16 * 16
    pos, ent = list(range(29, 36)) + [0, 1, 2] + [2000], [0] * 7 + [1] * 3 + [2]       # over a page border; a sequence's start; far out
    bt = torch.full((3, 126), -1, dtype=torch.int32)
    bt[0, :3], bt[1, 0], bt[2, 125] = torch.tensor([5, 2, 7]), 3, 1
    bt = bt.cuda()
    T, lead = len(pos), 3
    nq = nh * (qd + rp)
    proj = (torch.randn(T, lead + nq + 2 + r + rp + 5, generator=g) * 2.0).to(dt)
    w = 1.0 + 0.2 * torch.randn(r, generator=g)
    freq, mult = P.yarn_table(rot, 777.0, {"factor": 5.0, "original": 100, "fast": 8.0, "slow": 0.5})
    cache = torch.full((9, 2, 1, 16, hd), 9.0, dtype=dt, device="cuda")
    q_out = torch.full((T, nh * hd), 9.0, dtype=dt, device="cuda")
    args = (lead, nh, qd, lead + nq + 2, r, rp, hd, w.cuda(), 1e-3, rot, freq.cuda(), mult, interleaved)
    ops.latent_rope_store(proj.cuda(), *args, q_out, _i32(pos), _i32(ent), bt, cache, 16)
    x = proj.double()

    def turned(cols):                             # [T, heads, rp] at the positions `pos`
        full = torch.zeros(2001, cols.shape[1], rp, dtype=torch.float64)
        full[pos] = cols
        if interleaved:
            return P.rotate_pairs(full, freq, mult)[pos]
        order = [j for i in range(rot // 2) for j in (i, i + rot // 2)] + list(range(rot, rp))      # pairs side by side, turned, put back
        out = torch.empty_like(full)
        out[..., order] = P.rotate_pairs(full[..., order], freq, mult)
        return out[pos]
    off_b = lead + nq + 2
    c = P.rms_norm(x[:, off_b:off_b + r], w.double(), 1e-3)
    k = turned(x[:, None, off_b + r:off_b + r + rp])[:, 0]
    q = turned(x[:, lead:lead + nq].view(T, nh, qd + rp)[:, :, qd:])
    tol = 2e-6 if dtype == "float32" else 6e-3        # (angles are made in double precision: position 2,000 is as good as position 1)
    got_q = q_out.view(T, nh, hd)
    _close(got_q[:, :, r:r + rp], q, dtype, "q", tol)
    assert float((got_q[:, :, :r].float() - 9.0).abs().max()) == 0.0      # not this kernel's business
    assert hd == r + rp or float(got_q[:, :, r + rp:].float().abs().max()) == 0.0
    for t_, (p, e) in enumerate(zip(pos, ent)):
        page = int(bt[e, p // 16])
        for plane in (0, 1):
            _close(cache[page, plane, 0, p % 16, :r], c[t_], dtype, f"latent of token {t_}", tol)
            _close(cache[page, plane, 0, p % 16, r:r + rp], k[t_], dtype, f"rotated part of token {t_}", tol)
            assert hd == r + rp or float(cache[page, plane, 0, p % 16, r + rp:].float().abs().max()) == 0.0
    untouched = cache.clone()
    for p, e in zip(pos, ent):
        untouched[int(bt[e, p // 16]), :, :, p % 16] = 9.0
    assert float((untouched.float() - 9.0).abs().max()) == 0.0


# ---- sigmoid weights over a window ------------------------------------------------------------------------------------------------
def _attn_case(nh, nkv, hd, starts, qlens, seed, marked=None):
    """Entries e with starts[e] cached tokens before their qlens[e] new ones; pages handed out in a scrambled order.
    marked (entry, key): that key is made to stand out for every query of the entry that may see it."""
    g = torch.Generator().manual_seed(seed)
    E = len(starts)
    lens = [s + q for s, q in zip(starts, qlens)]
    n_pages = sum((n + 15) // 16 for n in lens)
    perm = torch.randperm(n_pages + 3, generator=g).tolist()
    bt = torch.full((E, max((n + 15) // 16 for n in lens)), -1, dtype=torch.int32)
    ks = [torch.randn(n, nkv, hd, generator=g) for n in lens]
    vs = [torch.randn(n, nkv, hd, generator=g) for n in lens]
    qs = [torch.randn(ql, nh, hd, generator=g) for ql in qlens]
    if marked is not None:
        e, key = marked
        ks[e][key] *= 3.0
        qs[e] = qs[e] * 0.3 + ks[e][key].repeat_interleave(nh // nkv, 0)[None] * 0.4
        vs[e][key] *= 8.0
    cache = torch.zeros(n_pages + 4, 2, nkv, 16, hd)
    n = 0
    for e in range(E):
        for pi in range((lens[e] + 15) // 16):
            bt[e, pi] = perm[n]
            c = min(16, lens[e] - pi * 16)
            cache[perm[n], 0, :, :c] = ks[e][pi * 16: pi * 16 + c].transpose(0, 1)
            cache[perm[n], 1, :, :c] = vs[e][pi * 16: pi * 16 + c].transpose(0, 1)
            n += 1
    r1, r2, pb = torch.rand(nh, generator=g) * 1.5, torch.rand(nh, generator=g) + 0.05, torch.randn(nh, generator=g) * 0.5 - 2.0
    return dict(E=E, starts=starts, qlens=qlens, lens=lens, k=ks, v=vs, q=qs, bt=bt, cache=cache, r1=r1, r2=r2, pb=pb)


def _attn_reference(c, nh, nkv, scale, window, dtype):
    outs = []
    for e in range(c["E"]):
        k, v, q = (x.to(DT[dtype]).double() for x in (c["k"][e], c["v"][e], c["q"][e]))
        n, s0 = c["lens"][e], c["starts"][e]
        full = torch.zeros(n, nh, q.shape[2], dtype=torch.float64)        # rows before the portion: their queries do not matter
        full[s0:] = q
        heads = []
        for j in range(nh):
            gk = j // (nh // nkv)
            heads.append(P.sigmoid_weights(full[:, j], k[:, gk], scale, c["r1"][j].double(), c["r2"][j].double(), c["pb"][j].double(), window) @ v[:, gk])
        outs.append(torch.stack(heads, 1)[s0:])
    return torch.cat(outs, 0).reshape(sum(c["qlens"]), -1)


def _run_attention(kernel, c, nh, nkv, hd, scale, window, dtype, splits=1):
    from infinilm_b200 import ops
    dt = DT[dtype]
    q = torch.cat(c["q"], 0).reshape(-1, nh * hd).to(dt).cuda()
    cache, bt = c["cache"].to(dt).cuda(), c["bt"].cuda()
    n = torch.arange(window, dtype=torch.float64)[:, None]
    table = (c["pb"].double() - c["r1"].double() * torch.log1p(c["r2"].double() * n)).float().contiguous().cuda()
    kw = dict(dist_bias=table, sigmoid=True)
    T = q.shape[0]
    out = torch.full((T, nh * hd), float("nan"), device="cuda", dtype=dt)
    qstart = [0]
    for ql in c["qlens"]:
        qstart.append(qstart[-1] + ql)
    G = nh // nkv
    if kernel == "plain":
        pos = [s + i for s, ql in zip(c["starts"], c["qlens"]) for i in range(ql)]
        ent = [e for e, ql in enumerate(c["qlens"]) for _ in range(ql)]
        ops.attention_plain(q, out, cache, bt, _i32(pos), _i32(ent), 16, nh, nkv, hd, scale, window, **kw)
    elif kernel == "decode":
        rows = T * nh * splits
        ops.attention_decode(q, out, cache, bt, _i32(c["lens"]), T, 16, nh, nkv, hd, scale, window, 0, splits,
                             torch.empty(rows * hd, device="cuda"), torch.empty(rows * 2, device="cuda"), kv_map=ops.kv_tensor_map(cache), **kw)
    elif kernel == "prefill":
        tpt = max(1, 64 // G)
        ops.attention_prefill(q, out, cache, bt, _i32(qstart), _i32(c["lens"]), 0, c["E"], sum((x + tpt - 1) // tpt for x in c["qlens"]),
                              16, nh, nkv, hd, scale, window, **kw)
    else:
        tpt = max(1, ops.prefill_tc5_rows(hd) // G)
        if kernel == "tc5 log":                   # the bias by distance computed in the kernel
            kw = dict(sigmoid=True, log_bias=torch.stack([c["r1"], c["r2"], c["pb"]]).contiguous().cuda())
        ops.attention_prefill_tc5(q, out, ops.kv_tensor_map(cache), bt, _i32(qstart), _i32(c["lens"]), 0, c["E"],
                                  sum((x + tpt - 1) // tpt for x in c["qlens"]), 16, nh, nkv, hd, scale, window, **kw)
    torch.cuda.synchronize()
    ops.check_status("cuda:0")
    return out


WINDOWS = [20, 16, 17, 1, 2, 90, 300]


@pytest.mark.parametrize("kernel,dtype,nh,nkv,hd", [("plain", "float32", 3, 1, 40), ("plain", "bfloat16", 6, 3, 48), ("prefill", "bfloat16", 6, 3, 48),
                                                    ("prefill", "bfloat16", 8, 8, 80), ("tc5", "bfloat16", 4, 2, 64), ("tc5", "bfloat16", 9, 1, 128),
                                                    ("tc5", "bfloat16", 4, 1, 256), ("tc5 log", "bfloat16", 4, 2, 64), ("tc5 log", "bfloat16", 9, 1, 128),
                                                    ("tc5 log", "bfloat16", 4, 1, 256)])
def test_sigmoid_weights_over_portions(cuda_device, kernel, dtype, nh, nkv, hd):
    """Portions that start and end anywhere, with one key made to stand out: the oldest key a window shows, the one before it,
    and keys at page borders. A query that may see the key follows it; one that may not must not. (Without a marked key an
    entry's many small weights must add up: nothing normalises them.)"""
    starts, qlens = [0, 250, 31, 16, 0], [70, 9, 2, 33, 1]
    for size in WINDOWS:
        for mk in (None, (1, 255), (1, 240), (0, 0), (0, 15), (0, 16), (3, 31), (1, max(0, 258 - size)), (1, max(0, 259 - size)), (2, max(0, 32 - size))):
            c = _attn_case(nh, nkv, hd, starts, qlens, nh * hd + size, mk)
            got = _run_attention(kernel, c, nh, nkv, hd, 0.2, size, dtype)
            _close(got, _attn_reference(c, nh, nkv, 0.2, size, dtype), dtype, f"{kernel} window {size}, marked {mk}")


@pytest.mark.parametrize("kernel,dtype,nh,nkv,hd,splits", [("plain", "float32", 3, 1, 40, 1), ("decode", "bfloat16", 6, 3, 48, 1), ("decode", "bfloat16", 3, 1, 64, 4),
                                                           ("decode", "bfloat16", 8, 1, 80, 3), ("decode", "bfloat16", 4, 2, 128, 7), ("decode", "bfloat16", 2, 2, 256, 2),
                                                           ("decode", "bfloat16", 20, 1, 64, 12)])
def test_sigmoid_weights_of_single_tokens(cuda_device, kernel, dtype, nh, nkv, hd, splits):
    starts, qlens = [0, 15, 16, 17, 399, 63, 23, 24, 47, 48, 210, 19], [1] * 12
    for size in WINDOWS:
        for mk in (None, (4, 399), (4, 400 - size), (4, max(0, 399 - size)), (5, 48), (5, 47), (11, 0)):
            c = _attn_case(nh, nkv, hd, starts, qlens, nh * hd + size, mk)
            got = _run_attention(kernel, c, nh, nkv, hd, 0.2, size, dtype, splits)
            _close(got, _attn_reference(c, nh, nkv, 0.2, size, dtype), dtype, f"{kernel} window {size}, marked {mk}")


@pytest.mark.parametrize("kernel,hd", [("plain", 64), ("prefill", 64), ("tc5", 64), ("tc5 log", 64), ("decode", 64)])
def test_extreme_scores_and_masked_garbage(cuda_device, kernel, hd):
    """Scores far beyond where the exponential overflows (weights 0 and 1), with keys of neighbours' huge values outside the
    window: a masked key's weight is zero, not small."""
    c = _attn_case(2, 1, hd, [40, 100], [1, 1], 3)
    for e in range(2):
        c["q"][e] *= 60.0
        for j in range(c["lens"][e] - 10):        # outside the window of 10
            c["v"][e][j] = 1e30
            page, slot = int(c["bt"][e, j // 16]), j % 16
            c["cache"][page, 1, :, slot] = 1e30
    got = _run_attention(kernel, c, 2, 1, hd, 1.0, 10, "bfloat16" if kernel != "plain" else "float32")
    for e in range(2):                            # the reference: the window alone
        n = c["lens"][e]
        c["v"][e][: n - 10] = 0.0
    _close(got, _attn_reference(c, 2, 1, 1.0, 10, "bfloat16" if kernel != "plain" else "float32"), "bfloat16", kernel)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nh,nkv,dk,dv", [(4, 2, 32, 16), (3, 1, 20, 12), (2, 2, 7, 40)])
def test_norm_per_head_adds_the_biases_first(cuda_device, dtype, nh, nkv, dk, dv):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(dk)
    dt = DT[dtype]
    T, hd = 19, (max(dk, dv) + 15) // 16 * 16
    nq, nk, nv = nh * dk, nkv * dk, nkv * dv
    ld = (nq + nk + nv + 7) // 8 * 8
    proj, bias = torch.randn(T, ld, generator=g).to(dt), torch.randn(ld, generator=g) * 2
    wq, wk = 1.0 + 0.2 * torch.randn(dk, generator=g), 1.0 + 0.2 * torch.randn(dk, generator=g)
    cache, q_out = torch.zeros(2, 2, nkv, 16, hd, dtype=dt, device="cuda"), torch.empty(T, nh * hd, dtype=dt, device="cuda")
    ops.qk_norm_store(proj.cuda(), 0, nq, nq + nk, nh, nkv, dk, dv, hd, wq.cuda(), wk.cuda(), 1e-4, 0.0, 0, q_out, _i32(list(range(T))), _i32([0] * T),
                      _i32([[1, 0]]), cache, 16, bias=bias.cuda())
    x = proj.double() + bias.double()
    tol = 2e-6 if dtype == "float32" else 6e-3
    _close(q_out.view(T, nh, hd)[:, :, :dk], P.rms_norm(x[:, :nq].view(T, nh, dk), wq.double(), 1e-4), dtype, "q", tol)
    rows = torch.cat([cache[1], cache[0]], dim=2)[:, :, :T].transpose(1, 2)          # [plane, T, kv heads, hd]
    _close(rows[0, :, :, :dk], P.rms_norm(x[:, nq:nq + nk].view(T, nkv, dk), wk.double(), 1e-4), dtype, "k", tol)
    _close(rows[1, :, :, :dv], x[:, nq + nk:nq + nk + nv].view(T, nkv, dv), dtype, "v", tol)


# ---- the clamped gate ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("path,dtype,M,I,K", [("kernel", "float32", 5, 40, 24), ("kernel", "bfloat16", 300, 64, 48), ("kernel", "bfloat16", 3, 37, 16),
                                              ("skinny", "bfloat16", 1, 72, 96), ("skinny", "bfloat16", 8, 320, 200), ("skinny", "bfloat16", 16, 33, 128),
                                              ("mid", "bfloat16", 17, 96, 128), ("mid", "bfloat16", 100, 200, 192)])
@pytest.mark.parametrize("limit,alpha", [(1.0, 1.702), (3.5, 0.8)])
def test_clamped_gate(cuda_device, path, dtype, M, I, K, limit, alpha):
    """Products on both sides of both limits."""
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(M + I)
    dt = DT[dtype]
    x, w = torch.randn(M, K, generator=g).to(dt), (torch.randn(2 * I, K, generator=g) * 2.5 * limit / K ** 0.5).to(dt)
    z = x.double() @ w.double().T
    out = torch.empty(M, I, dtype=dt, device="cuda")
    if path == "kernel":
        zt = z.to(dt)
        z = zt.double()
        ops.swiglu(zt.cuda(), out, ops.ACT_CLAMPED, (limit, alpha))
    else:
        (ops.gemm_skinny if path == "skinny" else ops.gemm_mid)(x.cuda(), w.cuda(), out, 1.0, None, glu=ops.ACT_CLAMPED, act_params=(limit, alpha))
    assert float((z[:, :I] > limit).double().mean()) > 0.05 and float((z[:, I:].abs() > limit).double().mean()) > 0.1
    gt, up = z[:, :I].clamp(max=limit), z[:, I:].clamp(-limit, limit)
    _close(out, gt * torch.sigmoid(alpha * gt) * (up + 1.0), dtype, path, 1e-5 if dtype == "float32" else 1e-2)
    torch.cuda.synchronize()
    ops.check_status("cuda:0")


def test_clamped_gate_wants_its_limit(cuda_device):
    from infinilm_b200 import ops
    with pytest.raises(ops.KernelError, match="limit"):
        ops.swiglu(torch.zeros(2, 8, device="cuda"), torch.zeros(2, 4, device="cuda"), ops.ACT_CLAMPED)


# ---- routing ------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,E,top", [(1, 1, 1), (7, 12, 1), (16, 5, 5), (300, 64, 6), (3, 40, 32)])
def test_choice_by_sigmoid_scores(cuda_device, T, E, top):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(T + E)
    z = torch.randn(T, E + 3, generator=g) * 4
    z[0, 0] = 60.0                                # a score that rounds to one
    idx, wt = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
    ops.moe_select(z.cuda()[:, :E], None, idx, wt, top, rule=ops.ROUTE_SIGMOID, out_scale=1.5)
    order = torch.sort(z[:, :E].double(), dim=-1, descending=True, stable=True).indices[:, :top]
    assert torch.equal(idx.cpu().long(), order)
    _close(wt, 1.5 * torch.sigmoid(torch.gather(z.double(), 1, order)), "float32", "weights", 1e-6)
    corr = torch.zeros(E)
    corr[E - 1] = 5.0                             # a correction steers the choice, not the weights
    ops.moe_select(z.cuda()[:, :E], corr.cuda(), idx, wt, top, rule=ops.ROUTE_SIGMOID)
    assert (idx[:, 0] == E - 1).all()
    _close(wt[:, 0], torch.sigmoid(z[:, E - 1].double()), "float32", "weights beside a correction", 1e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,E,top,W,ff", [(1, 1, 1, 40, 24), (5, 6, 2, 72, 40), (16, 12, 1, 128, 64), (30, 4, 4, 96, 8), (300, 7, 3, 64, 32), (1100, 3, 2, 64, 32)])
@pytest.mark.parametrize("routed", [False, True])
def test_weights_on_the_experts_inputs(cuda_device, dtype, T, E, top, W, ff, routed):
    """The whole routed feed-forward: a few rows (two short kernels), some (product, choice, ragged products), many (the library's
    grouped product). The rows' own choices follow from four columns by clear margins."""
    from infinilm_b200.parts.moe import RoutedExperts
    from infinilm_b200.engine.step import Workspace
    g = torch.Generator().manual_seed(T + E)
    dt = DT[dtype]
    part = RoutedExperts({"hidden": W, "n_experts": E, "top": top, "expert_ff": ff, "shared_ff": None, "router_bias": False, "route_rule": "sigmoid",
                          "weight_on_input": True}, "m", dt)
    t = {}
    for ws in part.weight_specs():
        t[ws.name] = (torch.randn(*ws.shape, generator=g) * (0.02 if ws.name == "router" else 3.0 / W ** 0.5)).to(torch.bfloat16)
    x = torch.randn(T, W, generator=g)
    x[:, :4] = 0.0
    x[torch.arange(T), torch.arange(T) % 4] = 1.0
    for c in range(4):
        t["router"][:, c] = torch.linspace(-3.0, 3.0, E)[torch.randperm(E, generator=g)].to(torch.bfloat16)
    x = x.to(dt)
    part.set_weights({k: (v.cuda() if k.endswith("norm") else v.to(dt).cuda()) for k, v in t.items()})
    want = P.routed_feed_forward(x.double(), {k: v.double() for k, v in t.items()}, {"router": {"top": top}})

    class Ctx:
        pass
    ctx = Ctx()
    ctx.ws, ctx.dtype = Workspace("cuda:0", max(T, 64)), dt
    got = part.forward(x.cuda(), ctx, routed=routed)
    if routed:
        assert got.wt is None and got.top == top
        got = got.y.double()[got.pos.long()].view(T, top, W).sum(1)
    _close(got, want, dtype, f"T {T}")


# ---- a gate per head ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M,G,N,K", [(1, 3, 24, 32), (7, 6, 32, 64), (40, 2, 20, 12), (70, 4, 128, 192)])
def test_gate_per_group(cuda_device, dtype, M, G, N, K):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(M * G)
    dt = DT[dtype]
    ld = (G * (K + 16) + 7) // 8 * 8
    a = torch.randn(M, ld, generator=g).to(dt)
    w = (torch.randn(G, N, K, generator=g) / K ** 0.5).to(dt)
    gate = torch.randn(M, G + 5, generator=g).to(dt)
    out = torch.empty(M, G, N, dtype=dt, device="cuda")
    heads = a.cuda()[:, :G * (K + 16)].view(M, G, K + 16)[:, :, :K]       # columns in front of others that are not this product's
    ops.gemm_grouped(heads, w.cuda(), out, gate=gate.cuda()[:, 2:2 + G])
    want = torch.einsum("mgk,gnk->mgn", a[:, :G * (K + 16)].view(M, G, K + 16)[:, :, :K].double(), w.double())
    _close(out, want * torch.sigmoid(gate[:, 2:2 + G].double())[:, :, None], dtype, "gated", 1e-5 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("vdim,hd,ldg", [(24, 24, 9), (64, 64, 4), (20, 32, 4), (16, 48, 5)])
def test_head_gate_in_pieces_and_by_columns(cuda_device, vdim, hd, ldg):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(vdim)
    T, nh = 37, 3
    y, gate = torch.randn(T, nh * hd, generator=g).to(torch.bfloat16), torch.randn(T, ldg, generator=g).to(torch.bfloat16)
    out = torch.empty(T, nh * vdim, dtype=torch.bfloat16, device="cuda")
    ops.head_gate(y.cuda(), hd, gate.cuda(), 1, out, nh, vdim)
    want = y.double().view(T, nh, hd)[:, :, :vdim] * torch.sigmoid(gate.double()[:, 1:1 + nh])[:, :, None]
    _close(out.view(T, nh, vdim), want, "bfloat16", "gated", 6e-3)


@pytest.mark.parametrize("nh,d,rd,e,r", [(4, 32, 16, 24, 48), (2, 64, 32, 64, 96), (4, 64, 64, 64, 192)])
def test_latent_mixer_few_and_many_rows(cuda_device, nh, d, rd, e, r):
    """The mixer alone, in bfloat16, on a portion of 300 rows (the library's per-head products) and on the same rows with this
    package's products only."""
    from infinilm_b200.parts.latent_attention import LatentAttention
    from infinilm_b200.parts.spec import PartSpec
    from infinilm_b200.engine.step import Workspace
    g = torch.Generator().manual_seed(nh * d)
    W, T = 96, 300
    sc = {"factor": 4.0, "original": 128, "fast": 8.0, "slow": 1.0}
    base = {"hidden": W, "n_heads": nh, "qk_dim": d, "v_dim": e, "q_rank": None, "kv_rank": r, "scale": 0.15, "eps": 1e-5, "sink": False, "gate": True,
            "gate_per": "head", "rot_part": rd, "position": PartSpec("yarn", dict({"rot_dim": rd, "theta": 1e4, "interleaved": True}, **sc))}
    m = {"heads": nh, "dim": d, "rot_dim": rd, "vdim": e, "kv_rank": r, "scale": 0.15, "rot": {"dims": rd, "base": 1e4, "scaling": sc}}
    x = torch.randn(T, W, generator=g).to(torch.bfloat16)
    t, outs = None, []
    for own in (False, True):
        part = LatentAttention(dict(base, own_products_only=own), "m", torch.bfloat16)
        if t is None:
            t = {ws.name: (torch.randn(*ws.shape, generator=g) / ws.shape[-1] ** 0.5 if len(ws.shape) == 2 else 1.0 + 0.1 * torch.randn(*ws.shape, generator=g))
                 .to(torch.bfloat16) for ws in part.weight_specs()}
            want = P.latent_attention(x.double(), {k: v.double() for k, v in t.items()}, m, 1e-5)
        part.set_weights({k: v.cuda() for k, v in t.items()})
        n_pages = (T + 15) // 16
        storage = torch.zeros(n_pages, 2, 1, 16, part.hd, dtype=torch.bfloat16, device="cuda")
        from infinilm_b200 import ops

        class Ctx:
            def prompt_tiles(self, tpt):
                return (T + tpt - 1) // tpt

        class View:
            pass
        ctx, view = Ctx(), View()
        ctx.ws, ctx.dtype, ctx.tok_pos, ctx.tok_entry = Workspace("cuda:0", T), torch.bfloat16, _i32(list(range(T))), _i32([0] * T)
        ctx.entry_qstart, ctx.entry_kvlen, ctx.n_decode, ctx.n_entries, ctx.h_kvlen = _i32([0, T]), _i32([T]), 0, 1, [T]
        view.storage, view.block_table, view.page_size, view.writable = storage, _i32([list(range(n_pages))]), 16, True
        view.tma_map = ops.kv_tensor_map(storage)
        outs.append(part.forward(x.cuda(), ctx, view).clone())
        torch.cuda.synchronize()
        ops.check_status("cuda:0")
        _close(outs[-1], want, "bfloat16", f"own products {own}")
