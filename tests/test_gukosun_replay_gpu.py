"""Gukosun through the engine against the plain implementation under every way of cutting the work: whole prompts; every layer's
stream in 32-bit; a prompt and then its last tokens one by one (long decoding, with and without replayed graphs); decoding from
the first token; portions of changing size down to two tokens and one; up to three live requests mixed, unequal, with so few
pages that they are used again; tokens changed one by one around the windows' edges and page borders, and the first tokens of a
sequence; a first token that must still count at position 300; greedy generation through `LLM.generate` and the scheduler; the
command line; and the trace runner as a process."""
import json
import os
import subprocess
import sys
import warnings

import pytest
import torch

import plain_gukosun as P
from gukosun_configs import GUKOSUN, make_weights, token_ids

pytestmark = pytest.mark.gpu

TOL = {"float32": 4e-5, "bfloat16": 6e-2}
LENGTHS = {"a": [1, 2, 15, 16, 17, 41, 130], "b": [3, 33, 131, 140], "c": [1, 16, 17, 90, 290], "d": [2, 6, 50, 150]}
CASES = [("a", 0), ("b", 1), ("c", 2), ("d", 3)]
DTYPES = ["float32", "bfloat16"]
PEAK = {"float32": 4.0, "bfloat16": 2.5}


def _engine(raw, w, dtype, num_pages=48, max_seqs=4, max_batch_tokens=512):
    from infinilm_b200.config import config_from_json
    from infinilm_b200.engine import Engine
    with warnings.catch_warnings():
        warnings.simplefilter("ignore", RuntimeWarning)
        return Engine.from_tensors(config_from_json(raw), w, dtype=dtype, page_size=16, num_pages=num_pages, max_seqs=max_seqs,
                                   max_batch_tokens=max_batch_tokens)


_oracle_cache = {}


def _weights(name, seed, dtype):
    return make_weights(GUKOSUN[name](), seed, peak=PEAK[dtype])


def _oracle(name, seed, ids, dtype):
    key = (name, seed, tuple(ids), PEAK[dtype])
    if key not in _oracle_cache:
        _oracle_cache[key] = P.forward(GUKOSUN[name](), _weights(name, seed, dtype), ids)
    return _oracle_cache[key]


def _err(got, ref):
    got, ref = got.double().cpu(), ref.double()
    got, ref = got - got.mean(dim=-1, keepdim=True), ref - ref.mean(dim=-1, keepdim=True)
    return (got - ref).pow(2).mean(dim=-1).sqrt() / ref.pow(2).mean(dim=-1).sqrt()


def _check(got, ref, dtype, what):
    """Per position: the root mean square over the vocabulary of the logits' difference (each side's mean taken off), relative
    to that of the expected logits."""
    assert got.shape == ref.shape and torch.isfinite(got).all(), what
    err = _err(got, ref)
    bad = torch.nonzero(err > TOL[dtype])
    allowed = 0 if dtype == "float32" else max(1, len(err) // 25)
    assert bad.numel() <= allowed and (dtype == "float32" or float(err.max()) <= 2 * TOL[dtype]), \
        f"{what}: first wrong position {int(bad[0])} of {ref.shape[0]} (rel err {float(err[int(bad[0])]):.2e}, worst {float(err.max()):.2e}, {bad.numel()} wrong)"


def _run_cut(eng, ids, cuts, seq_id="r"):
    from infinilm_b200.engine import StepEntry
    assert sum(cuts) == len(ids)
    seq, outs, a = eng.open(seq_id), [], 0
    for c in cuts:
        outs.append(eng.step([StepEntry(seq, ids[a:a + c], list(range(c)))]).clone())
        a += c
    eng.close(seq)
    return torch.cat(outs, 0)


def _run_schedule(eng, requests, schedule):
    from infinilm_b200.engine import StepEntry
    done, seqs, outs = {k: 0 for k in requests}, {}, {k: [] for k in requests}
    for step in schedule:
        entries = []
        for rid, n in step:
            if rid not in seqs:
                seqs[rid] = eng.open(rid)
            entries.append(StepEntry(seqs[rid], requests[rid][done[rid]:done[rid] + n], list(range(n))))
            done[rid] += n
        logits, r = eng.step(entries).clone(), 0
        for rid, n in step:
            outs[rid].append(logits[r:r + n])
            r += n
            if done[rid] == len(requests[rid]):
                eng.close(seqs.pop(rid))
        eng.cache.check_invariants()
    assert all(done[k] == len(requests[k]) for k in requests)
    return {k: torch.cat(v, 0) for k, v in outs.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,seed", CASES)
def test_whole_prompts(cuda_device, name, seed, dtype):
    raw = GUKOSUN[name]()
    eng = _engine(raw, _weights(name, seed, dtype), dtype)
    for n in LENGTHS[name]:
        ids = token_ids(n, raw["vocab"], 100 + n)
        _check(_run_cut(eng, ids, [n]), _oracle(name, seed, ids, dtype), dtype, f"{name} whole prompt of {n}")
    eng.synchronize()
    eng.cache.check_invariants()


@pytest.mark.parametrize("name,seed", CASES)
def test_every_layer_in_32_bit(cuda_device, name, seed):
    """The residual stream after every layer run, against the plain implementation."""
    from infinilm_b200.engine import StepEntry
    raw = GUKOSUN[name]()
    w = _weights(name, seed, "float32")
    eng = _engine(raw, w, "float32")
    ids = token_ids(70, raw["vocab"], 5)
    _, want = P.forward(raw, w, ids, want_layers=True)
    got = []
    eng.runner.tap = lambda nm, resid, pending: got.append(resid.detach().clone().cpu())
    seq = eng.open("x")
    eng.step([StepEntry(seq, ids, [69])])
    eng.close(seq)
    eng.runner.tap = None
    assert len(got) == len(raw["layers"])
    for i, g in enumerate(got):
        err = float((g.double() - want[i]).abs().max()) / float(want[i].abs().max())
        assert err < 2e-5, f"layer {i}: {err:.2e}"


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,seed", CASES)
def test_prompt_then_token_by_token(cuda_device, name, seed, dtype, graphs):
    """Prefill against decoding through the caches: the last 60 tokens one by one, and a sequence decoded from
    its very first token on. With `graphs` the single-token steps are captured and replayed as CUDA graphs."""
    raw = GUKOSUN[name]()
    eng = _engine(raw, _weights(name, seed, dtype), dtype)
    if graphs:
        eng.enable_graphs()
        assert eng.model.graph_safe
    ids = token_ids(110, raw["vocab"], 7)
    _check(_run_cut(eng, ids, [50] + [1] * 60), _oracle(name, seed, ids, dtype), dtype, f"{name} 50 + 60 x 1")
    ids = token_ids(45, raw["vocab"], 8)
    _check(_run_cut(eng, ids, [1] * 45), _oracle(name, seed, ids, dtype), dtype, f"{name} 45 x 1")
    eng.synchronize()
    eng.cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,seed", CASES)
def test_portions_of_changing_size(cuda_device, name, seed, dtype):
    raw = GUKOSUN[name]()
    eng = _engine(raw, _weights(name, seed, dtype), dtype)
    ids = token_ids(131, raw["vocab"], 9)
    ref = _oracle(name, seed, ids, dtype)
    for cuts in ([2, 2, 3, 16, 1, 31, 17, 2, 40, 15, 2], [64, 64, 3], [5] * 26 + [1], [15, 1, 16, 32, 33, 34], [23, 2, 24, 1, 25, 56]):
        _check(_run_cut(eng, ids, cuts), ref, dtype, f"{name} portions {cuts[:6]}")
    eng.synchronize()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,seed", CASES)
def test_mixed_batches_reuse_pages(cuda_device, name, seed, dtype):
    """Five unequal requests through three live places and a pool that cannot hold them all at once: single tokens beside
    portions, requests that pause, pages given back and taken again."""
    raw = GUKOSUN[name]()
    eng = _engine(raw, _weights(name, seed, dtype), dtype, num_pages=14, max_seqs=3)
    req = {k: token_ids(n, raw["vocab"], 20 + i) for i, (k, n) in enumerate((("p", 90), ("q", 37), ("r", 3), ("s", 70), ("t", 18)))}
    schedule = [[("p", 40), ("q", 2)], [("p", 1), ("q", 1), ("r", 2)], [("q", 30), ("p", 1)], [("r", 1), ("p", 17), ("q", 1)],
                [("p", 1), ("q", 1), ("s", 33)], [("s", 1), ("p", 20), ("q", 2)], [("s", 2), ("p", 10), ("t", 17)], [("s", 34), ("t", 1)]]
    got = _run_schedule(eng, req, schedule)
    for k, ids in req.items():
        _check(got[k], _oracle(name, seed, ids, dtype), dtype, f"{name} mixed, request {k}")
    eng.synchronize()
    assert len(eng.cache.live) == 0 and all(n == grp.pool.n_pages for grp in eng.cache.groups if grp.pool for n in [grp.pool.n_free])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,seed", [("a", 11), ("d", 12), ("c", 15)])
def test_a_changed_token_at_the_windows_edges_and_at_page_borders(cuda_device, name, seed, dtype):
    """One token is another at every distance around the windows' edges (20, 33 and 7 in "a", 11 and 1 in "d", 5 in "c"), around
    page borders and among the first tokens, in a prompt, in portions and decoded alone: a key that is seen one position too long,
    or lost one too early, moves the logits (tests of the weights show by how much), and so does the token's own input."""
    raw = GUKOSUN[name]()
    w = make_weights(raw, seed, peak=PEAK[dtype])
    eng = _engine(raw, w, dtype)
    base = [t if t != 5 else 6 for t in token_ids(64, raw["vocab"], 12)]
    for at in (63, 62, 60, 59, 58, 57, 56, 53, 52, 48, 47, 44, 43, 42, 32, 31, 30, 29, 16, 15, 2, 1, 0):
        ids = list(base)
        ids[at] = 5
        ref = P.forward(raw, w, ids)
        for cuts in ([64], [at + 1] + [1] * (63 - at), [at, 2] + [1] * (62 - at) if at + 2 <= 64 else [64], [33, 15, 16]):
            if sum(cuts) != 64 or min(cuts) < 1:
                continue
            _check(_run_cut(eng, ids, cuts), ref, dtype, f"changed at {at}, cuts {cuts[:3]}")
    eng.synchronize()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_reaches_the_end(cuda_device, dtype):
    """A change of the first token must still move the logits 300 tokens later - through the attention over all positions alone: the
    windows have left it behind and the decays forgotten it - and the engine must follow there, whole, decoded and in portions."""
    raw = GUKOSUN["a"]()
    for L in raw["layers"]:
        if L["type"] == "parallel":
            L["mixer"]["right"]["decay"] = [0.6] * L["mixer"]["right"]["heads"]
    w = make_weights(raw, 13, peak=PEAK[dtype])
    for i in (1, 3):                              # the first token's key: one that queries look for
        w[f"l{i}.mix.left.q.norm"] = (w[f"l{i}.mix.left.q.norm"].float() * 1.5).to(torch.bfloat16)
    ids = token_ids(300, raw["vocab"], 14)
    other = [(ids[0] + 3) % raw["vocab"]] + ids[1:]
    ref, ref2 = P.forward(raw, w, ids), P.forward(raw, w, other)
    assert float(_err(ref2, ref)[-40:].max()) > 20 * TOL["float32"]
    eng = _engine(raw, w, dtype)
    _check(_run_cut(eng, ids, [300])[-40:], ref[-40:], dtype, "far token, whole")
    _check(_run_cut(eng, other, [260] + [1] * 40)[-40:], ref2[-40:], dtype, "far token, decoded")
    _check(_run_cut(eng, ids, [7, 130, 2, 121] + [1] * 40)[-40:], ref[-40:], dtype, "far token, portions then decoded")
    eng.synchronize()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_portion_walks_its_recurrence_in_segments(cuda_device, dtype):
    """Portions of several hundred tokens (the recurrence is walked in segments at once), also beside other entries, then decoding."""
    raw = GUKOSUN["b"]()
    w = make_weights(raw, 5, peak=PEAK[dtype])
    ids, short = token_ids(430, raw["vocab"], 2), token_ids(60, raw["vocab"], 3)
    ref, ref_short = P.forward(raw, w, ids), P.forward(raw, w, short)
    eng = _engine(raw, w, dtype)
    _check(_run_cut(eng, ids, [430]), ref, dtype, "430 at once")
    _check(_run_cut(eng, ids, [3, 400] + [1] * 27), ref, dtype, "3 + 400 + single tokens")
    got = _run_schedule(eng, {"l": ids, "s": short}, [[("s", 30)], [("l", 380), ("s", 1)], [("s", 29), ("l", 50)]])
    _check(got["l"], ref, dtype, "long beside short")
    _check(got["s"], ref_short, dtype, "short beside long")
    eng.synchronize()


@pytest.mark.parametrize("graphs", [False, True])
def test_windows_pages_are_given_back(cuda_device, graphs):
    """A model of windowed layers alone decodes far longer than its pool could hold: the pages behind the window come back."""
    raw = GUKOSUN["a"]()
    raw["layers"] = [raw["layers"][0], raw["layers"][2], raw["layers"][4]]
    w = make_weights(raw, 8)
    eng = _engine(raw, w, "bfloat16", num_pages=6)
    if graphs:                                    # a replayed step made from the step before gives pages back as any other
        eng.enable_graphs()
    ids = token_ids(400, raw["vocab"], 3)
    _check(_run_cut(eng, ids, [40] + [1] * 300 + [33, 27]), P.forward(raw, w, ids), "bfloat16", "400 tokens through 6 pages a group")
    assert not graphs or eng.runner.fast_steps > 200
    eng.synchronize()
    eng.cache.check_invariants()


@pytest.mark.parametrize("drop", ["token_side", "mlp", "cap", "mask"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_models_without_an_option(cuda_device, drop, dtype):
    """No token input at all (the branches' sum makes the next norm itself), no feed-forward anywhere, no caps, no windows."""
    raw = GUKOSUN["a"]()
    if drop == "token_side":
        raw.pop(drop)
    for L in raw["layers"]:
        if drop == "mlp":
            L["mlp"] = None
        if drop == "cap" and L["type"] == "parallel":
            L["mixer"]["left"].pop("softcap")
        if drop == "mask" and L["type"] == "attention":
            L["mixer"]["mask"]["size"] = 10 ** 6
    w = make_weights(raw, 21, peak=PEAK[dtype])
    eng = _engine(raw, w, dtype)
    ids = token_ids(75, raw["vocab"], 4)
    ref = P.forward(raw, w, ids)
    for cuts in ([75], [30, 2, 17] + [1] * 26):
        _check(_run_cut(eng, ids, cuts), ref, dtype, f"without {drop}, cuts {cuts[:3]}")
    eng.synchronize()


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_llm(cuda_device, dtype):
    from infinilm_b200.config import config_from_json
    from infinilm_b200.llm import LLM, SamplingParams
    raw = GUKOSUN["c"]()
    w = make_weights(raw, 4, peak=PEAK[dtype])
    prompts = [token_ids(n, raw["vocab"], 30 + n) for n in (5, 21, 40)]
    with warnings.catch_warnings():
        warnings.simplefilter("ignore", RuntimeWarning)
        llm = LLM.from_tensors(config_from_json(raw), w, dtype=dtype, num_blocks=40, block_size=16, max_batch_size=3)
    outs = llm.generate(prompt_token_ids=prompts, sampling_params=SamplingParams(top_k=1, max_tokens=24, ignore_eos=True))
    for p, o in zip(prompts, outs):
        got = list(o.outputs[0].token_ids)
        assert len(got) == 24
        if dtype == "float32":
            assert got == P.greedy_generate(raw, w, p, 24)
            continue
        lg = P.forward(raw, w, list(p) + got)[len(p) - 1:-1]      # every token is the plain implementation's argmax, where that is clear
        top2 = torch.topk(lg, 2).values
        for t, row, gap in zip(got, lg, top2[:, 0] - top2[:, 1]):
            assert float(gap) < 0.2 * float(row.abs().max()) or t == int(torch.argmax(row))
    llm.close()


def test_command_line_on_a_random_folder(cuda_device, tmp_path):
    """The package's command line: write a folder of random weights for a configuration, then generate from it."""
    from infinilm_b200 import cli
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(GUKOSUN["a"]()))
    folder = str(tmp_path / "m")
    assert cli.main(["--write-random-model", folder, "--config", str(cfg_path), "--seed", "3"]) == 0
    with warnings.catch_warnings():
        warnings.simplefilter("ignore", RuntimeWarning)
        rc = cli.main(["--model", folder, "--enable-paged-attn", "--block-size", "16", "--num-blocks", "32", "--prompt-len", "21",
                       "--max-new-tokens", "9", "--batch-size", "2", "--ignore-eos", "--enable-graph", "--log-level", "ERROR"])
    assert rc == 0


def test_trace_runner_as_a_process(cuda_device, tmp_path):
    """A model folder replayed step by step by the runner."""
    from infinilm_b200.weights.safetensors_io import write_safetensors
    raw = GUKOSUN["b"]()
    w = make_weights(raw, 6, peak=PEAK["bfloat16"])
    folder = str(tmp_path / "m")
    os.makedirs(folder)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(raw, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), w)
    req = {k: token_ids(n, raw["vocab"], 40 + n) for k, n in (("a", 70), ("b", 9), ("c", 33), ("d", 50), ("e", 20))}
    steps = [[("a", 30), ("b", 2)], [("a", 1), ("b", 7), ("c", 3)], [("a", 39), ("c", 30), ("d", 1)], [("d", 49), ("e", 20)]]
    done, lines, wants = {k: 0 for k in req}, [], []
    for n, st in enumerate(steps):
        entries, end = [], []
        for rid, c in st:
            a = done[rid]
            entries.append({"id": rid, "tokens": req[rid][a:a + c], "want": [0, c - 1] if c > 1 else [0]})
            wants.append([(rid, a), (rid, a + c - 1)] if c > 1 else [(rid, a)])
            done[rid] = a + c
            if done[rid] == len(req[rid]):
                end.append(rid)
        lines.append(json.dumps({"step": n, "entries": entries, "end": end}))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out_dir = str(tmp_path / "out")
    ref = {k: P.forward(raw, w, ids) for k, ids in req.items()}
    for dtype in ("float32", "bfloat16"):
        p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out_dir,
                            "--max-tokens", "192"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=900)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {n}" for n in range(len(steps))]
        k0 = 0
        for n, st in enumerate(steps):
            rows = [x for e in wants[k0:k0 + len(st)] for x in e]
            k0 += len(st)
            got = torch.frombuffer(bytearray(open(os.path.join(out_dir, f"{n}.f32"), "rb").read()), dtype=torch.float32).view(len(rows), raw["vocab"])
            want = torch.stack([ref[rid][pos] for rid, pos in rows])
            _check(got, want, dtype, f"trace step {n} ({dtype})")


@pytest.mark.parametrize("name,seed", [("a", 0), ("d", 3)])
def test_a_batch_decodes_in_replayed_steps_past_its_windows(cuda_device, name, seed):
    """Three unequal requests decode side by side in replayed steps, each made from the step before, while every one's windows
    leave pages behind at steps of its own and others take those pages; a fourth joins in between."""
    from infinilm_b200.engine import StepEntry
    raw = GUKOSUN[name]()
    w = _weights(name, seed, "bfloat16")
    eng = _engine(raw, w, "bfloat16", num_pages=36)
    eng.enable_graphs()
    req = {k: token_ids(n, raw["vocab"], 60 + n) for k, n in (("p", 150), ("q", 131), ("r", 137), ("s", 40))}
    first = {"p": 30, "q": 11, "r": 17, "s": 20}
    seqs, at, out = {}, {}, {k: [] for k in req}

    def step(who):
        ent = [StepEntry(seqs[k], req[k][at[k]:at[k] + n], list(range(n)) if n == 1 else [n - 1]) for k, n in who]
        lg = eng.step(ent).clone()
        for i, (k, n) in enumerate(who):
            at[k] += n
            out[k].append((at[k] - 1, lg[i]))
    for k in "pqr":
        seqs[k], at[k] = eng.open(k), 0
        step([(k, first[k])])
    for n in range(60):
        step([(k, 1) for k in "pqr"])
        eng.cache.check_invariants()
    seqs["s"], at["s"] = eng.open("s"), 0
    step([("p", 1), ("s", 20), ("q", 1), ("r", 1)])
    for n in range(20):
        step([(k, 1) for k in "pqrs"])
    eng.close(seqs.pop("s"))
    for n in range(39):
        step([(k, 1) for k in "pqr"])
        eng.cache.check_invariants()
    assert eng.runner.fast_steps > 90
    for k in req:
        lg = P.forward(raw, w, req[k])
        pos = torch.tensor([p for p, _ in out[k]])
        _check(torch.stack([x for _, x in out[k]]), lg[pos], "bfloat16", f"request {k}")
    eng.synchronize()
