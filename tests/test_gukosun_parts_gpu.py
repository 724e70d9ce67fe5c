"""Each mechanism of the Gukosun parts alone, on the device, against the plain implementation: capped scores and sinks over all
positions or a window in each of the four attention kernels, with a key that stands out just inside and just outside the window
and at page borders, and scores from far below the cap to far above it; the norm over the whole projection with neighbouring pairs
turned, near and far from the sequence's start; the norm per head with blended values; branches joined in one pass; the squared
relu in its three kernels; the token's gated row; the token input with few and many rows; the parallel mixer's two outputs."""
import math

import pytest
import torch

import plain_gukosun as P

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


# ---- capped scores and sinks ------------------------------------------------------------------------------------------------
def _attn_case(nh, nkv, hd, starts, qlens, seed, marked=None, size=1.0):
    """Entries e with starts[e] cached tokens before their qlens[e] new ones; pages handed out in a scrambled order. marked (entry,
    key): that key is made to stand out for every query of the entry that may see it. size: of the queries."""
    g = torch.Generator().manual_seed(seed)
    lens = [s + q for s, q in zip(starts, qlens)]
    n_pages = sum((n + 15) // 16 for n in lens)
    perm = torch.randperm(n_pages + 3, generator=g).tolist()
    bt = torch.full((len(starts), max((n + 15) // 16 for n in lens)), -1, dtype=torch.int32)
    ks = [torch.randn(n, nkv, hd, generator=g) for n in lens]
    vs = [torch.randn(n, nkv, hd, generator=g) for n in lens]
    qs = [torch.randn(ql, nh, hd, generator=g) * size for ql in qlens]
    if marked is not None:
        e, key = marked
        ks[e][key] *= 2.0
        qs[e] = qs[e] * 0.3 + ks[e][key].repeat_interleave(nh // nkv, 0)[None] * 0.3 * size
        vs[e][key] *= 8.0
    cache = torch.zeros(n_pages + 4, 2, nkv, 16, hd)
    n = 0
    for e in range(len(starts)):
        for pi in range((lens[e] + 15) // 16):
            bt[e, pi] = perm[n]
            c = min(16, lens[e] - pi * 16)
            cache[perm[n], 0, :, :c] = ks[e][pi * 16: pi * 16 + c].transpose(0, 1)
            cache[perm[n], 1, :, :c] = vs[e][pi * 16: pi * 16 + c].transpose(0, 1)
            n += 1
    return dict(E=len(starts), starts=starts, qlens=qlens, lens=lens, k=ks, v=vs, q=qs, bt=bt, cache=cache, sink=torch.randn(nh, generator=g) * 2 + 2)


def _attn_reference(c, nh, nkv, scale, window, cap, dtype):
    outs = []
    for e in range(c["E"]):
        k, v, q = (x.to(DT[dtype]).double() for x in (c["k"][e], c["v"][e], c["q"][e]))
        n, s0 = c["lens"][e], c["starts"][e]
        full = torch.zeros(n, nh, q.shape[2], dtype=torch.float64)        # rows before the portion: their queries do not matter
        full[s0:] = q
        outs.append(P.attend(full, k, v, scale, c["sink"].double(), window, cap)[s0:])
    return torch.cat(outs, 0).reshape(sum(c["qlens"]), -1)


def _run_attention(kernel, c, nh, nkv, hd, scale, window, cap, dtype, splits=1):
    from infinilm_b200 import ops
    dt = DT[dtype]
    q = torch.cat(c["q"], 0).reshape(-1, nh * hd).to(dt).cuda()
    cache, bt = c["cache"].to(dt).cuda(), c["bt"].cuda()
    kw = dict(sink=c["sink"].cuda(), cap=cap)
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
        ops.attention_prefill_tc5(q, out, ops.kv_tensor_map(cache), bt, _i32(qstart), _i32(c["lens"]), 0, c["E"],
                                  sum((x + tpt - 1) // tpt for x in c["qlens"]), 16, nh, nkv, hd, scale, window, **kw)
    torch.cuda.synchronize()
    ops.check_status("cuda:0")
    return out


PORTIONS = [("plain", "float32", 3, 1, 40), ("plain", "bfloat16", 6, 3, 48), ("prefill", "bfloat16", 6, 3, 48), ("prefill", "bfloat16", 8, 8, 80),
            ("tc5", "bfloat16", 4, 2, 64), ("tc5", "bfloat16", 9, 1, 128), ("tc5", "bfloat16", 4, 1, 256)]
SINGLES = [("plain", "float32", 3, 1, 40, 1), ("decode", "bfloat16", 6, 3, 48, 1), ("decode", "bfloat16", 3, 1, 64, 4), ("decode", "bfloat16", 8, 1, 80, 3),
           ("decode", "bfloat16", 4, 2, 128, 7), ("decode", "bfloat16", 2, 2, 256, 2), ("decode", "bfloat16", 20, 1, 64, 12)]


@pytest.mark.parametrize("kernel,dtype,nh,nkv,hd", PORTIONS)
def test_capped_scores_over_portions(cuda_device, kernel, dtype, nh, nkv, hd):
    """Portions that start and end anywhere over all positions, one key standing out: the first of all, keys at page borders."""
    starts, qlens = [0, 250, 31, 16, 0], [70, 9, 2, 33, 1]
    for cap, size in ((1.5, 1.0), (8.0, 3.0), (50.0, 1.0), (4.0, 12.0)):
        for mk in (None, (1, 0), (1, 240), (1, 255), (0, 0), (0, 15), (0, 16), (3, 31), (2, 31)):
            c = _attn_case(nh, nkv, hd, starts, qlens, nh * hd + int(cap), mk, size)
            got = _run_attention(kernel, c, nh, nkv, hd, hd ** -0.5, None, cap, dtype)
            _close(got, _attn_reference(c, nh, nkv, hd ** -0.5, None, cap, dtype), dtype, f"{kernel} cap {cap} size {size}, marked {mk}")


@pytest.mark.parametrize("kernel,dtype,nh,nkv,hd,splits", SINGLES)
def test_capped_scores_of_single_tokens(cuda_device, kernel, dtype, nh, nkv, hd, splits):
    starts, qlens = [0, 15, 16, 17, 399, 63, 23, 24, 47, 48, 210, 19], [1] * 12
    for cap, size in ((1.5, 1.0), (8.0, 3.0), (50.0, 1.0), (4.0, 12.0)):
        for mk in (None, (4, 0), (4, 399), (4, 208), (5, 48), (5, 47), (11, 0)):
            c = _attn_case(nh, nkv, hd, starts, qlens, nh * hd + int(cap), mk, size)
            got = _run_attention(kernel, c, nh, nkv, hd, hd ** -0.5, None, cap, dtype, splits)
            _close(got, _attn_reference(c, nh, nkv, hd ** -0.5, None, cap, dtype), dtype, f"{kernel} cap {cap} size {size}, marked {mk}")


@pytest.mark.parametrize("kernel,dtype,nh,nkv,hd", PORTIONS)
def test_sinks_over_a_window(cuda_device, kernel, dtype, nh, nkv, hd):
    """A learned sink per head, without and with a cap, over windows around the page size: a key just inside counts, the one before
    it does not."""
    starts, qlens = [0, 250, 31, 16, 0], [70, 9, 2, 33, 1]
    for size in (20, 16, 17, 1, 2, 90, 300):
        for mk in (None, (1, max(0, 258 - size)), (1, max(0, 259 - size)), (0, 16), (2, max(0, 32 - size))):
            for cap in (None, 5.0):
                c = _attn_case(nh, nkv, hd, starts, qlens, nh * hd + size, mk)
                got = _run_attention(kernel, c, nh, nkv, hd, hd ** -0.5, size, cap, dtype)
                _close(got, _attn_reference(c, nh, nkv, hd ** -0.5, size, cap, dtype), dtype, f"{kernel} window {size} cap {cap}, marked {mk}")


@pytest.mark.parametrize("kernel,dtype,nh,nkv,hd,splits", SINGLES)
def test_sinks_over_a_window_of_single_tokens(cuda_device, kernel, dtype, nh, nkv, hd, splits):
    starts, qlens = [0, 15, 16, 17, 399, 63, 23, 24, 47, 48, 210, 19], [1] * 12
    for size in (20, 16, 17, 1, 2, 90, 300):
        for mk in (None, (4, 400 - size), (4, max(0, 399 - size)), (5, 48), (11, 0)):
            c = _attn_case(nh, nkv, hd, starts, qlens, nh * hd + size, mk)
            got = _run_attention(kernel, c, nh, nkv, hd, hd ** -0.5, size, None, dtype, splits)
            _close(got, _attn_reference(c, nh, nkv, hd ** -0.5, size, None, dtype), dtype, f"{kernel} window {size}, marked {mk}")


@pytest.mark.parametrize("kernel,hd", [("plain", 64), ("prefill", 64), ("tc5", 64), ("tc5", 128), ("decode", 64)])
def test_scores_beyond_the_exponentials_range(cuda_device, kernel, hd):
    """Scores of some thousands, of both signs, become plus or minus the cap; a sink that towers over every score leaves nothing
    of the values; one far below leaves no trace."""
    for sink in (0.0, 60.0, -60.0):
        c = _attn_case(2, 1, hd, [40, 100], [1, 1], 3, size=400.0)
        c["sink"] = torch.full((2,), sink)
        dt = "bfloat16" if kernel != "plain" else "float32"
        got = _run_attention(kernel, c, 2, 1, hd, 1.0, None, 10.0, dt)
        want = _attn_reference(c, 2, 1, 1.0, None, 10.0, dt)
        if sink == 60.0:
            assert float(got.float().abs().max()) < 1e-12 and float(want.abs().max()) < 1e-12
        else:
            _close(got, want, dt, f"{kernel} sink {sink}")


@pytest.mark.parametrize("factor", [0.5, 0.97, 1.03, 2.0])
def test_both_sides_of_where_the_cap_changes_its_formula(cuda_device, factor):
    """The tensor-memory kernel takes a polynomial where a tile's scores lie below three quarters of the cap: queries and keys of
    one direction, so that every score is a number of our choosing around that border; the weights' ratios show the caps."""
    nh, hd, n, cap = 2, 64, 64, 10.0
    c = _attn_case(nh, 1, hd, [0], [n], 1)
    edge = 0.75 * cap * factor
    c["k"][0][:] = 0.0
    c["k"][0][:, 0, 0] = torch.linspace(-edge, edge, n).to(torch.bfloat16).float()
    c["q"][0][:] = 0.0
    c["q"][0][:, :, 0] = 1.0
    c["v"][0] = torch.eye(n).view(n, 1, n)[:, :, :hd].contiguous() * 8.0
    for pi in range(n // 16):
        c["cache"][int(c["bt"][0, pi]), 0, :, :] = c["k"][0][pi * 16:pi * 16 + 16].transpose(0, 1)
        c["cache"][int(c["bt"][0, pi]), 1, :, :] = c["v"][0][pi * 16:pi * 16 + 16].transpose(0, 1)
    got = _run_attention("tc5", c, nh, 1, hd, 1.0, None, cap, "bfloat16").double().cpu()
    want = _attn_reference(c, nh, 1, 1.0, None, cap, "bfloat16")
    big = want > 1e-3
    assert float(((got - want).abs() / want)[big].max()) < 1.2e-2      # (weights and outputs are rounded to bfloat16)


def test_a_cap_goes_with_softmax_alone(cuda_device):
    from infinilm_b200 import ops
    q = torch.zeros(1, 16, device="cuda")
    with pytest.raises(ops.KernelError, match="cap"):
        ops.attention_plain(q, q.clone(), torch.zeros(1, 2, 1, 16, 16, device="cuda"), _i32([[0]]), _i32([0]), _i32([0]), 16, 1, 1, 16, 1.0, cap=2.0, sigmoid=True)
    with pytest.raises(ops.KernelError, match="cap"):
        ops.attention_plain(q, q.clone(), torch.zeros(1, 2, 1, 16, 16, device="cuda"), _i32([[0]]), _i32([0]), _i32([0]), 16, 1, 1, 16, 1.0, cap=0.0)


# ---- norms in front of attention ----------------------------------------------------------------------------------------------------
def _pages(pos, ent):
    """A block table whose needed pages are named, one page each, in scrambled order."""
    need = sorted({(e, p // 16) for p, e in zip(pos, ent)})
    bt = torch.full((max(ent) + 1, max(p for _, p in need) + 1), -1, dtype=torch.int32)
    for n, (e, p) in enumerate(need):
        bt[e, p] = (n * 5 + 2) % (len(need) * 5 + 3)
    return bt, len(need) * 5 + 3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nh,nkv,dk,dv,rot", [(4, 2, 32, 16, 32), (6, 2, 16, 24, 12), (3, 1, 20, 12, 8), (2, 2, 64, 64, 2), (3, 1, 18, 13, 6), (5, 1, 7, 40, 4),
                                              (8, 2, 128, 128, 128), (16, 2, 64, 64, 64), (2, 1, 256, 200, 250), (1, 1, 4, 4, 4), (40, 8, 128, 128, 96)])
def test_norm_over_the_projection_and_neighbouring_pairs(cuda_device, dtype, nh, nkv, dk, dv, rot):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(nh * dk + rot)
    dt = DT[dtype]
    pos, ent = list(range(29, 36)) + [0, 1, 2] + [4000, 100000], [0] * 7 + [1] * 3 + [2, 2]      # over a page border; a start; far out
    bt, n_pages = _pages(pos, ent)
    T, lead, hd = len(pos), 4, (max(dk, dv) + 15) // 16 * 16
    nq, nk, nv = nh * dk, nkv * dk, nkv * dv
    ld = (lead + nq + nk + nv + 7) // 8 * 8
    proj = (torch.randn(T, ld, generator=g) * 2).to(dt)
    wq, wk = 1.0 + 0.2 * torch.randn(nq, generator=g), 1.0 + 0.2 * torch.randn(nk, generator=g)
    freq = P.stretched_frequencies(rot, 777.0, {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64})
    cache = torch.full((n_pages, 2, nkv, 16, hd), 9.0, dtype=dt, device="cuda")
    q_out = torch.full((T, nh * hd), 9.0, dtype=dt, device="cuda")
    ops.qk_rows_norm_rope_store(proj.cuda(), lead, lead + nq, lead + nq + nk, nh, nkv, dk, dv, hd, wq.cuda(), wk.cuda(), 1e-3, rot, None, q_out, _i32(pos),
                                _i32(ent), bt.cuda(), cache, 16, pair_freq=freq.cuda())
    x = proj.double()

    def turned(rows, w, heads):
        y = P.rms_norm(rows, w.double(), 1e-3).view(T, heads, dk)
        ang = torch.tensor(pos, dtype=torch.float64)[:, None] * freq[None]
        out = y.clone()
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        out[..., 0:rot:2] = y[..., 0:rot:2] * c - y[..., 1:rot:2] * s
        out[..., 1:rot:2] = y[..., 1:rot:2] * c + y[..., 0:rot:2] * s
        return out
    q, k = turned(x[:, lead:lead + nq], wq, nh), turned(x[:, lead + nq:lead + nq + nk], wk, nkv)
    v = x[:, lead + nq + nk:lead + nq + nk + nv].view(T, nkv, dv)
    tol = 2e-6 if dtype == "float32" else 6e-3        # (angles are made in double precision: position 100,000 is as good as position 1)
    got = q_out.view(T, nh, hd)
    _close(got[:, :, :dk], q, dtype, "q", tol)
    assert hd == dk or float(got[:, :, dk:].float().abs().max()) == 0.0
    untouched = cache.clone()
    for t, (p, e) in enumerate(zip(pos, ent)):
        page = int(bt[e, p // 16])
        _close(cache[page, 0, :, p % 16, :dk], k[t], dtype, f"key of token {t}", tol)
        _close(cache[page, 1, :, p % 16, :dv], v[t], dtype, f"value of token {t}", tol)
        assert hd == dk or float(cache[page, 0, :, p % 16, dk:].float().abs().max()) == 0.0
        assert hd == dv or float(cache[page, 1, :, p % 16, dv:].float().abs().max()) == 0.0
        untouched[page, :, :, p % 16] = 9.0
    assert float((untouched.float() - 9.0).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nh,nkv,dk,dv", [(4, 2, 32, 16), (3, 1, 20, 12), (2, 2, 7, 40), (8, 2, 128, 128), (3, 3, 18, 7)])
@pytest.mark.parametrize("mix", [0.0, 0.3, 1.0, -0.5, 1.75])
def test_norm_per_head_with_blended_values(cuda_device, dtype, nh, nkv, dk, dv, mix):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(dk)
    dt = DT[dtype]
    T, hd = 19, (max(dk, dv) + 15) // 16 * 16
    nq, nk, nv = nh * dk, nkv * dk, nkv * dv
    ld = (nq + nk + nv + 7) // 8 * 8
    proj, earlier = torch.randn(T, ld, generator=g).to(dt), (torch.randn(T, nv + 24, generator=g) * 3).to(dt)
    wq, wk = 1.0 + 0.2 * torch.randn(dk, generator=g), 1.0 + 0.2 * torch.randn(dk, generator=g)
    cache, q_out = torch.full((2, 2, nkv, 16, hd), 9.0, dtype=dt, device="cuda"), torch.empty(T, nh * hd, dtype=dt, device="cuda")
    first = earlier.cuda()[:, 8:8 + nv]               # a stretch of wider rows
    ops.qk_norm_store(proj.cuda(), 0, nq, nq + nk, nh, nkv, dk, dv, hd, wq.cuda(), wk.cuda(), 1e-4, 0.0, 0, q_out, _i32(list(range(T))), _i32([0] * T),
                      _i32([[1, 0]]), cache, 16, first=first, mix=mix)
    x = proj.double()
    tol = 2e-6 if dtype == "float32" else 6e-3
    _close(q_out.view(T, nh, hd)[:, :, :dk], P.rms_norm(x[:, :nq].view(T, nh, dk), wq.double(), 1e-4), dtype, "q", tol)
    rows = torch.cat([cache[1], cache[0]], dim=2)[:, :, :T].transpose(1, 2)          # [plane, T, kv heads, hd]
    _close(rows[0, :, :, :dk], P.rms_norm(x[:, nq:nq + nk].view(T, nkv, dk), wk.double(), 1e-4), dtype, "k", tol)
    want = (1.0 - mix) * x[:, nq + nk:nq + nk + nv] + mix * earlier.double()[:, 8:8 + nv]
    _close(rows[1, :, :, :dv], want.view(T, nkv, dv), dtype, "v", tol)
    assert hd == dv or float(rows[1, :, :, dv:].float().abs().max()) == 0.0


# ---- branches joined in one pass --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H", [(1, 72), (5, 120), (33, 256), (3, 2048), (2, 13), (2, 4096), (2, 3001), (2, 8192), (4, 1028), (2, 1500)])
@pytest.mark.parametrize("kinds", ["s", "ns", "nns", "pn", "nnps"])
def test_branch_sum(cuda_device, dtype, T, H, kinds):
    """kinds: of each branch - n: normed, with a factor per column; s: a factor per column; p: plain."""
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(T * H + len(kinds))
    dt = DT[dtype]
    resid, total, terms = torch.randn(T, H, generator=g) * 3, torch.zeros(T, H, dtype=torch.float64), []
    for i, k in enumerate(kinds):
        y, nw, cs = (torch.randn(T, H, generator=g) * (i + 1)).to(dt), 1.0 + 0.3 * torch.randn(H, generator=g), (torch.randn(H, generator=g)).to(torch.bfloat16)
        b = y.double()
        if k == "n":
            b = P.rms_norm(b, nw.double(), 1e-3)
        if k in "ns":
            b = b * cs.double()
        total += (0.5 + i) * b
        terms.append(ops.BranchTerm(y.cuda(), 0.5 + i, nw.cuda() if k == "n" else None, 1e-3, cs.cuda() if k in "ns" else None))
    wn = 1.0 + 0.3 * torch.randn(H, generator=g)
    r, copy, out = resid.clone().cuda(), torch.empty(T, H, dtype=dt, device="cuda"), torch.empty(T, H, dtype=dt, device="cuda")
    want = resid.double() + total
    ops.branch_sum(terms, r, copy=copy, next_weight=wn.cuda(), next_eps=1e-2, out=out)
    _close(r, want, "float32", "stream", 3e-6)
    _close(copy, want, dtype, "copy", 3e-6 if dtype == "float32" else 5e-3)
    _close(out, P.rms_norm(want, wn.double(), 1e-2), dtype, "next input", 1e-5 if dtype == "float32" else 5e-3)
    r2 = resid.clone().cuda()
    ops.branch_sum(terms, r2)                         # only the add
    assert torch.equal(r2, r)
    ops.branch_sum(terms, copy=copy)                  # only the sum
    _close(copy, total, dtype, "sum alone", 3e-6 if dtype == "float32" else 5e-3)
    if T > 1:                                         # a row does not depend on the others
        r1 = resid[1:2].clone().cuda()
        ops.branch_sum([ops.BranchTerm(t.y[1:2].clone(), t.scale, t.norm_weight, t.eps, t.col_scale) for t in terms], r1)
        assert torch.equal(r1[0], r[1])


def test_branch_sum_refuses_two_branches_in_one_buffer(cuda_device):
    from infinilm_b200 import ops
    y = torch.zeros(2, 8, device="cuda")
    with pytest.raises(ops.KernelError, match="one buffer"):
        ops.branch_sum([ops.BranchTerm(y), ops.BranchTerm(y)], torch.zeros(2, 8, device="cuda"))


# ---- squared relu, and the token's row ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("path,dtype,M,I,K", [("kernel", "float32", 5, 40, 24), ("kernel", "bfloat16", 300, 64, 48), ("kernel", "bfloat16", 3, 37, 16),
                                              ("kernel", "float32", 3, 37, 16), ("skinny", "bfloat16", 1, 72, 96), ("skinny", "bfloat16", 8, 320, 200),
                                              ("skinny", "bfloat16", 16, 33, 128), ("mid", "bfloat16", 17, 96, 128), ("mid", "bfloat16", 100, 200, 192),
                                              ("mid", "bfloat16", 64, 4096, 256), ("mid", "bfloat16", 128, 40, 72)])
def test_squared_relu(cuda_device, path, dtype, M, I, K):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(M + I)
    dt = DT[dtype]
    x, w = torch.randn(M, K, generator=g).to(dt), (torch.randn(I, K, generator=g) * 2.0 / K ** 0.5).to(dt)
    z = x.double() @ w.double().T
    out = torch.empty(M, I, dtype=dt, device="cuda")
    if path == "kernel":
        zt = z.to(dt)
        z = zt.double()
        ops.relu2(zt.cuda(), out)
    else:
        (ops.gemm_skinny if path == "skinny" else ops.gemm_mid)(x.cuda(), w.cuda(), out, glu=ops.ACT_RELU2)
    _close(out, z.clamp(min=0.0) ** 2, dtype, path, 1e-6 if dtype == "float32" else 6e-3)
    torch.cuda.synchronize()
    ops.check_status("cuda:0")


def test_squared_relu_behind_a_half_done_norm(cuda_device):
    """Rows that still want their 1 / rms: the product multiplies by it before the activation."""
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(2)
    M, H, I = 5, 96, 72
    x, wn, w = torch.randn(M, H, generator=g) * 3, 1.0 + 0.2 * torch.randn(H, generator=g), (torch.randn(I, H, generator=g) * 0.2).to(torch.bfloat16)
    xw = (x * wn).to(torch.bfloat16)
    sq = (x * x).view(M, 6, 16).sum(-1).contiguous()
    out = torch.empty(M, I, dtype=torch.bfloat16, device="cuda")
    xw_d = xw.cuda()
    ops.gemm_skinny(xw_d, w.cuda(), out, glu=ops.ACT_RELU2, norm_in=ops.NormedInput(xw_d, sq.cuda(), H, 1e-4))
    z = (xw.double() / torch.sqrt((x.double() ** 2).mean(-1, keepdim=True) + 1e-4)) @ w.double().T
    _close(out, z.clamp(min=0.0) ** 2, "bfloat16", "norm then squared relu", 6e-3)


@pytest.mark.parametrize("path,dtype,T,dim,W", [("kernel", "float32", 7, 12, 0), ("kernel", "bfloat16", 50, 5, 0), ("kernel", "bfloat16", 300, 256, 0),
                                                ("skinny", "bfloat16", 1, 5, 72), ("skinny", "bfloat16", 8, 24, 200), ("skinny", "bfloat16", 16, 250, 128)])
def test_gated_row_of_a_token(cuda_device, path, dtype, T, dim, W):
    from infinilm_b200 import ops
    g = torch.Generator().manual_seed(T + dim)
    dt = DT[dtype]
    V, off, pad = 40, 3, (dim + 7) // 8 * 8
    table, ids = torch.randn(V, off + dim + 6, generator=g).to(dt), torch.randint(0, V, (T,), generator=g)
    out = torch.full((T, pad), 9.0, dtype=dt, device="cuda")
    if path == "kernel":
        z = torch.randn(T, pad, generator=g) * 3
        ops.gelu_row(z.cuda(), _i32(ids.tolist()), table.cuda(), off, dim, out)
        z = z.double()
    else:
        x, w = torch.randn(T, W, generator=g).to(dt), (torch.randn(pad, W, generator=g) * 2.0 / W ** 0.5).to(dt)
        ops.gemm_skinny_gelu_row(x.cuda(), w.cuda(), _i32(ids.tolist()), table.cuda(), off, dim, out)
        z = x.double() @ w.double().T
    want = P.gelu_tanh(z[:, :dim]) * table.double()[ids][:, off:off + dim]
    _close(out[:, :dim], want, dtype, path, 2e-6 if dtype == "float32" else 6e-3)
    assert pad == dim or float(out[:, dim:].float().abs().max()) == 0.0


class _Ctx:
    """What a part reads of a step."""
    tap = None

    def __init__(self, dtype, T, ids=None):
        from infinilm_b200.engine.step import Workspace
        self.dtype, self.T, self.ws, self.shared = dtype, T, Workspace("cuda", T), {}
        self.token_ids = None if ids is None else _i32(ids)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,W,dim", [(1, 72, 5), (16, 128, 24), (17, 120, 1), (40, 256, 16), (200, 74, 12)])
def test_token_input(cuda_device, dtype, T, W, dim):
    from infinilm_b200.parts.token_input import TokenInput
    g = torch.Generator().manual_seed(T + W)
    dt = DT[dtype]
    part = TokenInput({"hidden": W, "dim": dim, "offset": dim, "eps": 1e-5}, "s", dt)
    t = {"gate": (torch.randn(dim, W, generator=g) / W ** 0.5).to(torch.bfloat16), "proj": torch.randn(W, dim, generator=g).to(torch.bfloat16),
         "norm": torch.ones(W)}
    part.set_weights({k: v.cuda().to(dt) for k, v in t.items()})
    table, ids = torch.randn(30, 3 * dim, generator=g).to(dt), torch.randint(0, 30, (T,), generator=g)
    x = torch.randn(T, W, generator=g).to(dt)
    y = part.branch(x.cuda(), table.cuda(), _Ctx(dt, T, ids.tolist()))
    want = (P.gelu_tanh(x.double() @ t["gate"].double().T) * table.double()[ids][:, dim:2 * dim]) @ t["proj"].double().T
    _close(y, want, dtype, "token input", 2e-6 if dtype == "float32" else 1.5e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_squared_relu_feed_forward_at_every_kind_of_row_count(cuda_device, dtype):
    from infinilm_b200.parts.feed_forward import SquaredReLU
    g = torch.Generator().manual_seed(4)
    dt = DT[dtype]
    for W, ff in ((96, 136), (74, 37)):
        part = SquaredReLU({"hidden": W, "intermediate": ff, "names": {"up": "up", "down": "down"}}, "f", dt)
        t = {"up": (torch.randn(ff, W, generator=g) / W ** 0.5).to(torch.bfloat16), "down": (torch.randn(W, ff, generator=g) / ff ** 0.5).to(torch.bfloat16)}
        part.set_weights({k: v.cuda().to(dt) for k, v in t.items()})
        for T in (1, 8, 16, 17, 100, 129, 300):
            x = torch.randn(T, W, generator=g).to(dt)
            y = part.forward(x.cuda(), _Ctx(dt, T))
            _close(y, P.squared_relu_unit(x.double(), {k: v.double() for k, v in t.items()}), dtype, f"{T} rows", 2e-6 if dtype == "float32" else 1.5e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n", [2, 3])
def test_normed_outputs_of_mixers_side_by_side(cuda_device, dtype, n):
    """Decayed linear attentions side by side, each with a norm on its output, summed by the part itself and handed out unsummed."""
    from infinilm_b200 import ops
    from infinilm_b200.cache.manager import StateView
    from infinilm_b200.parts.parallel import ParallelMixers
    from infinilm_b200.parts.spec import PartSpec
    g = torch.Generator().manual_seed(n)
    dt, W, T = DT[dtype], 64, 21
    m = {"heads": 2, "dim": 16, "vdim": 24, "decay": [0.9, 0.5]}
    part = ParallelMixers({"branches": [(PartSpec("decay_linear_attention", {"hidden": W, "n_heads": 2, "qk_dim": 16, "v_dim": 24, "decay": m["decay"], "eps": 1e-5},
                                                  f"b{i}"), 0.5 + i) for i in range(n)], "branch_norm_eps": 1e-4, "branch_norm_width": W}, "p", dt)
    t = {}
    for ws in part.weight_specs():
        t[ws.name] = (1.0 + 0.3 * torch.randn(*ws.shape, generator=g) if ws.role == "vector" else torch.randn(*ws.shape, generator=g) / ws.shape[-1] ** 0.5).to(torch.bfloat16)
    part.set_weights({k: v.cuda().to(dt) if v.dim() == 2 else v.cuda() for k, v in t.items()})
    x = torch.randn(T, W, generator=g).to(dt)
    want = torch.zeros(T, W, dtype=torch.float64)
    for i in range(n):
        p = {k[3:]: v.double() for k, v in t.items() if k.startswith(f"b{i}.")}
        want += (0.5 + i) * P.rms_norm(P.linear_attention(x.double(), p, m, 1e-5), p["out"], 1e-4)
    ctx = _Ctx(dt, T)
    ctx.n_decode, ctx.n_entries, ctx.entry_qstart = 0, 1, _i32([0, T])
    views = tuple(StateView(torch.zeros(3, 2, 24, 16, device="cuda"), _i32([0]), _i32([1]), writable=True) for _ in range(n))
    y = part.forward(x.cuda(), ctx, views)
    _close(y, want, dtype, "summed", 3e-5 if dtype == "float32" else 2e-2)
    terms = part.forward(x.cuda(), ctx, views, terms=True)
    assert len(terms) == n
    r = torch.zeros(T, W, device="cuda")
    ops.branch_sum(terms, r)
    _close(r, want, dtype, "unsummed", 3e-5 if dtype == "float32" else 2e-2)
