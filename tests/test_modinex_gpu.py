"""Modinex on the GPU against the plain implementation (tests/plain/modinex_plain.py), in 32-bit and bfloat16: each
mechanism's kernel alone, the replay families (whole, last tokens one by one, portions down to two tokens, mixed batches with
pages and slots used again), a far key among hundreds, marked keys at the first and last place of every stretch, a far token
carried by the state, the first tokens of a sequence, long decoding, long portions, and greedy generation through
Engine.generate, the command line and bin/trace_run."""
import functools
import json
import os
import subprocess
import sys
import tempfile

import numpy as np
import pytest

from tests import modinex_cases as C
from tests import traces
from tests.modinex_configs import ALL, PAGE
from tests.plain import modinex_plain as P
from tests.plain.lfm2_plain import read_safetensors

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# Fractions of the largest |logit| of the compared requests.  float32 is the sharp test.  bfloat16: nine places in ten stay
# within TOL and none leaves WORST (a wrong key, state or stretch moves a place by the scale itself).
TOL = {"float32": 3e-5, "bfloat16": 4e-2}
WORST = {"float32": 3e-5, "bfloat16": 0.2}
_tmp = tempfile.TemporaryDirectory(prefix="imparo_b200_modinex_")


def rescale(path):
    """The drawn matrices are small, and then every token looks alike to the layers.  Matrices are scaled to a standard
    deviation of 1 / sqrt(columns) (the embedding to 1, position vectors to 0.5), so that tokens, positions, scores and gates
    all weigh in."""
    import torch
    from imparo_b200.weights.safetensors_io import write_safetensors
    out = {}
    for k, v in read_safetensors(path).items():
        t = torch.as_tensor(np.asarray(v))
        if v.ndim == 2:
            std = {"embed": 1.0, "pos": 0.5}.get(k, 1.0 / np.sqrt(v.shape[1]))
            t = (t.float() / t.float().std() * std).to(t.dtype)
        elif k.endswith((".up.b", ".down.b")):
            t = t * 10.0
        out[k] = t
    write_safetensors(path, out)


@functools.lru_cache(maxsize=None)
def model_dir(name, seed=1):
    from imparo_b200.weights import write_random_model
    d = os.path.join(_tmp.name, f"{name}_{seed}")
    write_random_model(d, ALL[name], seed=seed, dtype="bfloat16", norm_jitter=0.3)
    rescale(os.path.join(d, "model.safetensors"))
    # the decay's inner size is the stored tensor's: the configuration of the folder does not name it
    with open(os.path.join(d, "config.json")) as f:
        cfg = json.load(f)
    for L in cfg["layers"]:
        L["mixer"].pop("rank", None)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    return d


@functools.lru_cache(maxsize=None)
def weights(name, seed=1):
    return read_safetensors(os.path.join(model_dir(name, seed), "model.safetensors"))


def make_requests(name, lengths, seed=0):
    rng = np.random.default_rng(seed)
    return {f"r{i}": rng.integers(0, ALL[name]["vocab"], n).tolist() for i, n in enumerate(lengths)}


_plain = {}


def plain_logits(name, requests, seed=1):
    out = {}
    for rid, toks in requests.items():
        key = (name, seed, tuple(toks))
        if key not in _plain:
            _plain[key] = P.forward(ALL[name], weights(name, seed), toks)
        out[rid] = _plain[key]
    return out


def engine_for(name, dtype, steps, parallel=4, page=None, **kw):
    from imparo_b200.engine import Engine
    page = page or PAGE[name]
    max_tokens = traces.max_live_tokens(steps, max(64, page))
    return Engine(model_dir(name), dtype=dtype, ctx=max_tokens, parallel=parallel, page_size=page,
                  num_pages=(max_tokens + page - 1) // page, max_step_tokens=max(256, max_tokens), **kw)


def all_errors(steps, got, want):
    at, out = {}, []
    for s in steps:
        r = 0
        for e in s["entries"]:
            start = at.get(e["id"], 0)
            for w in e["want"]:
                out.append((s["step"], e["id"], start + w, float(np.abs(got[s["step"]][r] - want[s["step"]][r]).max())))
                r += 1
            at[e["id"]] = start + len(e["tokens"])
        for name in s["end"]:
            at.pop(name, None)
    return out


def check_trace(engine, steps, name, requests, dtype, share=0.1):
    from tests.gpu_helpers import run_trace
    ref = plain_logits(name, requests)
    want = traces.expected(steps, ref)
    got = run_trace(engine, steps)
    assert sorted(got) == sorted(want)
    scale = max(float(np.abs(v).max()) for v in ref.values())
    errs = all_errors(steps, got, want)
    bad = next((e for e in errs if not e[3] <= WORST[dtype] * scale), None)
    assert bad is None, (f"first wrong place: step {bad[0]}, request {bad[1]}, position {bad[2]}, "
                         f"error {bad[3]:.3e} > {WORST[dtype] * scale:.3e}")
    over = [e for e in errs if not e[3] <= TOL[dtype] * scale]
    assert len(over) <= share * len(errs), f"{len(over)} of {len(errs)} places beyond {TOL[dtype] * scale:.3e}; the first: {over[0]}"
    assert engine.cache.n_requests() == 0
    return got


LENGTHS = {"A": [70, 45, 96, 33, 64, 51], "B": [5, 23, 140, 67, 90, 34], "C": [81, 40, 201, 97, 58], "D": [150, 47, 96, 300, 64],
           "E": [60, 75, 40, 104, 52, 83]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALL))
@pytest.mark.parametrize("family", ["whole", "tail", "portions", "mixed"])
def test_family(name, dtype, family):
    reqs = make_requests(name, LENGTHS[name])
    steps = {"whole": traces.whole, "tail": lambda r: traces.tail_one_by_one(r, tail=44), "portions": traces.portions,
             "mixed": lambda r: traces.mixed(r, seed=3)}[family](reqs)
    check_trace(engine_for(name, dtype, steps), steps, name, reqs, dtype)
    if family == "mixed":
        assert traces.max_live_tokens(steps) < sum(traces.round_up(len(t), 64) for t in reqs.values())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_cutting_does_not_change_logits_beyond_rounding(name, dtype):
    from tests.gpu_helpers import run_trace
    reqs = make_requests(name, [61, 47, 75], seed=5)
    outs = []
    for build in (traces.whole, traces.tail_one_by_one, traces.portions, lambda r: traces.mixed(r, seed=9)):
        steps = build(reqs)
        got = run_trace(engine_for(name, dtype, steps), steps)
        by_pos, at = {}, {}
        for s in steps:
            r = 0
            for e in s["entries"]:
                start = at.get(e["id"], 0)
                for w in e["want"]:
                    by_pos[(e["id"], start + w)] = got[s["step"]][r]
                    r += 1
                at[e["id"]] = start + len(e["tokens"])
        outs.append(by_pos)
    keys = set(outs[1]) & set(outs[0])
    assert len(keys) > 90
    scale = max(float(np.abs(v).max()) for v in outs[0].values())
    tol = (2e-5 if dtype == "float32" else 0.1) * scale
    for k in keys:
        for o in outs[1:]:
            if k in o:
                assert np.abs(o[k] - outs[0][k]).max() <= tol, k


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["B", "C", "D"])
def test_long_portions(name, dtype):
    """Prompts of several hundred tokens, whole and in portions of 71 to 300 tokens beside another request's single tokens:
    whole tiles of the tensor-core attention, stretches that begin and end inside tiles, the recurrence in chunks."""
    reqs = make_requests(name, [700, 333], seed=13)
    steps = traces.whole(reqs)
    check_trace(engine_for(name, dtype, steps), steps, name, reqs, dtype)
    a, b = reqs["r0"], reqs["r1"]
    steps, at_a, at_b = [], 0, 0
    steps.append({"step": 0, "entries": [{"id": "b", "tokens": b[:300], "want": [0, 150, 299]}], "end": []})
    at_b = 300
    for n in (300, 129, 200, 71):
        steps.append({"step": len(steps), "entries": [{"id": "a", "tokens": a[at_a:at_a + n], "want": [0, n // 2, n - 1]},
                                                     {"id": "b", "tokens": [b[at_b]], "want": [0]}],
                      "end": ["a"] if at_a + n == 700 else []})
        at_a += n
        at_b += 1
    steps.append({"step": len(steps), "entries": [{"id": "b", "tokens": b[at_b:], "want": [0, len(b) - at_b - 1]}], "end": ["b"]})
    check_trace(engine_for(name, dtype, steps), steps, name, {"a": a, "b": b}, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "D"])
def test_long_decoding(name, dtype):
    """390 tokens one by one: stretches end and begin, their pages go back, the states are carried through every step."""
    reqs = make_requests(name, [400], seed=8)
    steps = traces.tail_one_by_one(reqs, tail=390)
    check_trace(engine_for(name, dtype, steps), steps, name, reqs, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "D", "E"])
def test_first_tokens_of_a_sequence(name, dtype):
    reqs = make_requests(name, [1, 2, 3, 6], seed=11)
    for build in (traces.whole, lambda r: traces.tail_one_by_one(r, tail=8)):
        steps = build(reqs)
        check_trace(engine_for(name, dtype, steps), steps, name, reqs, dtype, share=0.5 if dtype == "bfloat16" else 0.0)


@pytest.mark.parametrize("name", ["A", "B"])
def test_state_slots_and_pages_start_clean_when_used_again(name):
    a = make_requests(name, [50], seed=20)
    b = {"other": make_requests(name, [37], seed=21)["r0"]}
    steps = traces.whole(a) + [dict(s, step=s["step"] + 1) for s in traces.portions(b, sizes=(1, 2, 3))]
    eng = engine_for(name, "float32", steps, parallel=1)       # one slot: it must be reused
    check_trace(eng, steps, name, dict(a, **b), "float32")


@pytest.mark.parametrize("page", [16, 64, 128])
def test_page_sizes_of_the_tensor_core_attention(page):
    reqs = make_requests("C", [310, 77], seed=31)
    steps = traces.tail_one_by_one(reqs, tail=9)
    check_trace(engine_for("C", "bfloat16", steps, page=page), steps, "C", reqs, "bfloat16")


# ---- each mechanism's kernel alone ------------------------------------------------------------------------------

def _dev(a, dtype=None):
    import torch
    t = torch.as_tensor(np.ascontiguousarray(a)).cuda()
    return t if dtype is None else t.to(dtype)


def _f32(a):
    import torch
    return _dev(np.asarray(a, dtype=np.float32), torch.float32)


def _bf16_round(a):
    import torch
    return torch.as_tensor(np.asarray(a, dtype=np.float32)).to(torch.bfloat16).float().numpy().astype(np.float64)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,width,groups", [(7, 72, 3), (7, 40, 20), (7, 52, 1), (7, 52, 4), (7, 128, 8), (7, 2048, 4), (7, 1024, 1), (7, 4100, 2), (7, 96, 96),
                                            (7, 6144, 3), (300, 2048, 4), (257, 72, 3), (260, 96, 12), (256, 1000, 1), (300, 768, 2), (270, 2100, 2)])
def test_group_norms_and_the_normed_add(T, width, groups, dtype):
    """The norm in groups (rows in place and picked), the add of a normed output alone and with the next norm in the same
    pass, with a bias and with split partials of the output."""
    import torch
    from imparo_b200.kernels import ops
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    tol = 1e-5 if dtype == "float32" else 1e-2
    rng = np.random.default_rng(width + groups)
    x, y, w, wn, bias = rng.standard_normal((T, width)) * 3, rng.standard_normal((T, width)) * 1e-2, rng.uniform(0.5, 1.5, width), rng.uniform(0.5, 1.5, width), rng.standard_normal(width) * 1e-2
    eps = 1e-5
    out = torch.empty(T, width, dtype=tdt, device="cuda")
    ops.group_rmsnorm(_f32(x), _f32(w), eps, groups, out)
    want = P.group_rms(x, groups, eps) * w
    assert np.abs(out.float().cpu().numpy() - want).max() <= tol * np.abs(want).max()
    rows = [4, 0, 6]
    picked = torch.empty(3, width, dtype=tdt, device="cuda")
    ops.group_rmsnorm(_f32(x), _f32(w), eps, groups, picked, rows=_dev(np.array(rows, dtype=np.int32)))
    assert np.abs(picked.float().cpu().numpy() - want[rows]).max() <= tol * np.abs(want).max()
    new = x + P.group_rms(y, groups, eps) * w
    xd = _f32(x)
    ops.group_norm_add(xd, _f32(y), _f32(w), eps, groups)
    assert np.abs(xd.cpu().numpy() - new).max() <= 1e-5 * np.abs(new).max()
    # left pending, with a bias noted on the output: the next norm does all of it
    xd, yd = _f32(x), _f32(y)
    ops.allow_unfinished(yd)
    ops.add_bias(yd, _f32(bias))
    ops.disallow_unfinished(yd)
    ops.group_norm_add(xd, yd, _f32(w), eps, groups, defer=True)
    assert np.abs(xd.cpu().numpy() - x).max() <= 1e-6 * 10
    ops.group_rmsnorm(xd, _f32(wn), eps, groups, out)
    new = x + P.group_rms(y + bias, groups, eps) * w
    want = P.group_rms(new, groups, eps) * wn
    assert np.abs(xd.cpu().numpy() - new).max() <= 1e-5 * np.abs(new).max()
    assert np.abs(out.float().cpu().numpy() - want).max() <= tol * np.abs(want).max()


@pytest.mark.parametrize("T,K,width,groups", [(3, 512, 256, 4), (8, 2048, 192, 2), (1, 1024, 128, 1)])
def test_an_unfinished_product_is_finished_by_the_add(T, K, width, groups):
    """A product of few rows may leave split partials and its bias to the normed add; whoever else reads the buffer finds it
    whole."""
    import torch
    from imparo_b200.kernels import ops
    rng = np.random.default_rng(T + K)
    a, wm = _bf16_round(rng.standard_normal((T, K))), _bf16_round(rng.standard_normal((width, K)) / np.sqrt(K))
    bias, x, w = rng.standard_normal(width), rng.standard_normal((T, width)), rng.uniform(0.5, 1.5, width)
    y = a @ wm.T + bias
    for settled in (False, True):
        xd, yd = _f32(x), torch.full((T, width), 9.0, device="cuda")
        ops.allow_unfinished(yd)
        ops.linear(_dev(a, torch.bfloat16), _dev(wm, torch.bfloat16), yd)
        ops.add_bias(yd, _f32(bias))
        ops.disallow_unfinished(yd)
        if settled:
            ops.settle(yd)
            assert np.abs(yd.cpu().numpy() - y).max() <= 1e-4
        ops.group_norm_add(xd, yd, _f32(w), 1e-5, groups)
        want = x + P.group_rms(y, groups, 1e-5) * w
        assert np.abs(xd.cpu().numpy() - want).max() <= 1e-4


def _attention_by_kernels(dtype, m, rows, q_norm, k_norm, pb, cuts, page, eps=1e-5, expect=None):
    """Head norms, rotation, cache write and the attention on one request cut as `cuts`; rows: the product [T, q | k | v].
    expect: "tensor" asserts that the tensor-core kernels take the launches."""
    import torch
    from imparo_b200.kernels import ops
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    nh, nkv, hd, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = len(rows)
    n_blocks = -(-T // page)
    n_pages = n_blocks + 3
    table = torch.arange(n_pages - 1, n_pages - 1 - n_blocks, -1, dtype=torch.int32, device="cuda").reshape(1, -1)
    kc = torch.zeros(n_pages * page * nkv * hd, dtype=tdt, device="cuda")
    vc = torch.zeros(n_pages * page * nkv * vd, dtype=tdt, device="cuda")
    status = ops.new_status("cuda")
    chunk = m["mask"]["size"] if m.get("mask") else None
    n_rot = m["rot"]["dims"] if m.get("rot") else 0
    inv_freq = _f32([float(m["rot"]["base"]) ** (-2.0 * i / n_rot) for i in range(n_rot // 2)]) if n_rot else None
    bias = _f32(pb)
    out_all, at = np.zeros((T, nh * vd)), 0
    for n in cuts:
        pos, iot = _dev(np.arange(at, at + n, dtype=np.int32)), _dev(np.zeros(n, dtype=np.int32))
        q = torch.empty(n, nh * hd, dtype=tdt, device="cuda")
        ops.qkv_norm_rotate_store(_dev(rows[at:at + n], tdt), pos, iot, _f32(q_norm), _f32(k_norm), eps, inv_freq, n_rot, q, kc, vc, table,
                                  page, n_pages, nh, nkv, hd, vd, status)
        if chunk and at // chunk:                            # pages of earlier stretches are gone
            table[0, :at // chunk * chunk // page] = -1
        out = torch.full((n, nh * vd), 7.0, dtype=tdt, device="cuda")
        done = False
        if expect == "tensor" and n >= 8:
            done = ops.attention_sigmoid_prefill(q, kc, vc, _dev(np.array([0, n], dtype=np.int32)), _dev(np.array([at], dtype=np.int32)), 1, table,
                                                 page, n_pages, None, chunk, m["scale"], bias, out, nh, nkv, hd, vd, status)
            assert done, "the tensor-core prompt kernel declined a shape it is said to take"
        elif expect == "tensor" and nh // nkv <= 8:
            range_, n_splits = ops.split_plan(n, nkv, min(table.shape[1] * page, chunk or 1 << 30))
            done = ops.attention_sigmoid_split(q, kc, vc, pos, iot, table, page, n_pages, None, chunk, m["scale"], bias, out,
                                               torch.empty(n * nh * n_splits * vd, device="cuda"), torch.empty(n * nh * n_splits * 2, device="cuda"),
                                               range_, n_splits, nh, nkv, hd, vd, status)
            assert done, "the split-key kernel declined a shape it is said to take"
        if not done:
            ops.attention_any(q, kc, vc, pos, iot, table, page, n_pages, None, m["scale"], False, out, nh, nkv, hd, vd, status, chunk=chunk,
                              score_bias=bias)
        out_all[at:at + n] = out.float().cpu().numpy()
        at += n
    ops.read_status(status)
    return out_all


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nh,nkv,hd,vd,size,rot", [(6, 2, 12, 20, 9, 8), (4, 2, 16, 16, 33, 16), (3, 3, 24, 8, 70, None), (5, 1, 7, 5, None, 4), (2, 2, 250, 256, 19, 64)])
def test_sigmoid_attention_on_the_general_kernels(dtype, nh, nkv, hd, vd, size, rot):
    """Head norms with weights, rotation of a part, value sizes of their own, stretches of any size: a prompt of 45 tokens, then
    30 tokens one by one (pages of 4: every border is crossed; pages of earlier stretches unmapped)."""
    rng = np.random.default_rng(hd + vd)
    m = {"heads": nh, "kv_heads": nkv, "dim": hd, "vdim": vd, "scale": 2.5 / hd}
    if size:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = {"base": 300.0, "dims": rot}
    rows = rng.standard_normal((75, nh * hd + nkv * (hd + vd))) * 1.5
    if dtype == "bfloat16":
        rows = _bf16_round(rows)
    qn, kn, pb = rng.uniform(0.5, 1.5, hd), rng.uniform(0.5, 1.5, hd), rng.uniform(-3.0, 1.0, nh)
    want = C.attention_rows_plain(m, 1e-5, rows, qn, kn, pb)
    got = _attention_by_kernels(dtype, m, rows, qn, kn, pb, [45] + [1] * 30, 4)
    assert np.abs(got - want).max() <= (2e-5 if dtype == "float32" else 2e-2) * np.abs(want).max()


@pytest.mark.parametrize("nh,nkv,hd,vd,size,page", [(4, 2, 64, 64, 48, 16), (7, 1, 64, 96, 50, 16), (6, 3, 48, 112, None, 32), (16, 2, 128, 128, 200, 64),
                                                    (3, 1, 112, 16, 129, 128), (5, 5, 16, 48, 31, 16), (24, 1, 32, 64, 100, 16), (8, 8, 80, 64, 37, 32)])
def test_sigmoid_attention_on_tensor_cores(nh, nkv, hd, vd, size, page):
    """Portions of 300, 9, 130 and 60 tokens on the tcgen05 kernel, a portion of 3 and single tokens on the split-key kernel (more
    than 8 heads per key head: the general kernel)."""
    rng = np.random.default_rng(hd + vd + nh)
    m = {"heads": nh, "kv_heads": nkv, "dim": hd, "vdim": vd, "scale": 2.5 / hd, "rot": {"base": 10000.0, "dims": hd // 2 // 2 * 2}}
    if size:
        m["mask"] = {"size": size}
    T = 300 + 9 + 3 + 130 + 60 + 20
    rows = _bf16_round(rng.standard_normal((T, nh * hd + nkv * (hd + vd))) * 1.5)
    qn, kn, pb = rng.uniform(0.5, 1.5, hd), rng.uniform(0.5, 1.5, hd), rng.uniform(-4.0, 1.0, nh)
    want = C.attention_rows_plain(m, 1e-5, rows, qn, kn, pb)
    got = _attention_by_kernels("bfloat16", m, rows, qn, kn, pb, [300, 9, 3, 130, 60] + [1] * 20, page, expect="tensor")
    assert np.abs(got - want).max() <= 2e-2 * np.abs(want).max()


def test_sigmoid_attention_of_several_requests_and_windows():
    """A ragged batch (portions of unequal length at unequal positions) on the tcgen05 kernel, and a sliding window in place of
    stretches on all three kernels."""
    import torch
    from imparo_b200.kernels import ops
    rng = np.random.default_rng(4)
    nh, nkv, hd, vd, page, scale = 6, 2, 64, 48, 16, 0.06
    pb = rng.uniform(-4.0, 1.0, nh)
    starts, lens = [0, 37, 200], [150, 9, 77]
    n_pages = 64
    kc = _dev(rng.standard_normal((n_pages * page, nkv * hd)), torch.bfloat16)
    vc = _dev(rng.standard_normal((n_pages * page, nkv * vd)), torch.bfloat16)
    perm = rng.permutation(n_pages)
    tab = np.full((3, 32), -1, dtype=np.int32)
    at = 0
    for i in range(3):
        nb = -(-(starts[i] + lens[i]) // page)
        tab[i, :nb] = perm[at:at + nb]
        at += nb
    T = sum(lens)
    q = _dev(rng.standard_normal((T, nh * hd)), torch.bfloat16)
    row_start = np.concatenate([[0], np.cumsum(lens)]).astype(np.int32)
    pos = np.concatenate([np.arange(s, s + n) for s, n in zip(starts, lens)]).astype(np.int32)
    iot = np.repeat(np.arange(3), lens).astype(np.int32)
    K, V = kc.float().cpu().numpy().astype(np.float64), vc.float().cpu().numpy().astype(np.float64)
    Q = q.float().cpu().numpy().astype(np.float64).reshape(T, nh, hd)
    status = ops.new_status("cuda")
    for window, chunk in ((None, None), (45, None), (None, 50)):
        want = np.zeros((T, nh, vd))
        for t in range(T):
            p, i = int(pos[t]), int(iot[t])
            lo = 0 if window is None and chunk is None else (max(0, p - window + 1) if window else p // chunk * chunk)
            rows = tab[i][np.arange(lo, p + 1) // page] * page + np.arange(lo, p + 1) % page
            for h in range(nh):
                g = h // (nh // nkv)
                s = K[rows, g * hd:(g + 1) * hd] @ Q[t, h] * scale + pb[h]
                want[t, h] = P.sigmoid(s) @ V[rows, g * vd:(g + 1) * vd]
        want = want.reshape(T, nh * vd)
        args = (_dev(tab), page, n_pages)
        out = torch.zeros(T, nh * vd, dtype=torch.bfloat16, device="cuda")
        assert ops.attention_sigmoid_prefill(q, kc, vc, _dev(row_start), _dev(np.array(starts, dtype=np.int32)), 3, *args, window, chunk, scale,
                                             _f32(pb), out, nh, nkv, hd, vd, status)
        assert np.abs(out.float().cpu().numpy() - want).max() <= 2e-2 * np.abs(want).max()
        out.zero_()
        range_, ns = ops.split_plan(T, nkv, min([512] + [x for x in (window, chunk) if x]))
        assert ops.attention_sigmoid_split(q, kc, vc, _dev(pos), _dev(iot), *args, window, chunk, scale, _f32(pb), out,
                                           torch.empty(T * nh * ns * vd, device="cuda"), torch.empty(T * nh * ns * 2, device="cuda"), range_, ns,
                                           nh, nkv, hd, vd, status)
        assert np.abs(out.float().cpu().numpy() - want).max() <= 2e-2 * np.abs(want).max()
        ops.attention_any(q, kc, vc, _dev(pos), _dev(iot), *args, window, scale, False, out, nh, nkv, hd, vd, status, chunk=chunk, score_bias=_f32(pb))
        assert np.abs(out.float().cpu().numpy() - want).max() <= 2e-2 * np.abs(want).max()
    ops.read_status(status)
    # a softmax over stretches on the general kernel
    out = torch.zeros(T, nh * vd, dtype=torch.bfloat16, device="cuda")
    ops.attention_any(q, kc, vc, _dev(pos), _dev(iot), _dev(tab), page, n_pages, None, scale, False, out, nh, nkv, hd, vd, status, chunk=50)
    t = 140
    rows = tab[0][np.arange(100, 141) // page] * page + np.arange(100, 141) % page
    s = K[rows, :hd] @ Q[t, 0] * scale
    p = np.exp(s - s.max())
    assert np.abs(out.float().cpu().numpy()[t, :vd] - p @ V[rows, :vd] / p.sum()).max() <= 2e-2


@pytest.mark.parametrize("dtype,D,V,H,G,expect", [("float32", 32, 32, 4, 2, None), ("bfloat16", 32, 32, 4, 2, "tensor"), ("bfloat16", 64, 112, 6, 1, "tensor"),
                                                  ("bfloat16", 24, 12, 4, 2, None)])
@pytest.mark.parametrize("far,page", [(0, 16), (15, 16), (16, 16), (31, 32), (127, 32), (128, 64)])
def test_a_far_key_among_hundreds(dtype, D, V, H, G, expect, far, page):
    """One key, before, at or after a page border, weighs nearly 1 for the queries that look for it and the hundreds of others
    nearly nothing, in a prompt of 600 and in 20 single tokens (tests/modinex_cases.py: far_key_case)."""
    for rot in (D, D // 2 // 2 * 2):
        m, rows, qn, kn, pb, seekers, v_far, want = C.far_key_case(far, seed=far * 31 + page, D=D, V=V, H=H, G=G, rot=rot)
        got = _attention_by_kernels(dtype, m, rows, qn, kn, pb, [600] + [1] * 20, page, expect=expect)
        assert np.abs(got - want).max() <= (5e-5 if dtype == "float32" else 4e-2) * np.abs(want).max()
        for t in seekers:
            assert np.abs(got[t].reshape(G, H // G, V) - v_far[:, None, :]).max() < 0.3


@pytest.mark.parametrize("dtype,D,V,H,G,expect", [("float32", 32, 16, 4, 1, None), ("bfloat16", 32, 16, 4, 1, "tensor"), ("bfloat16", 64, 112, 6, 1, "tensor"),
                                                  ("bfloat16", 128, 64, 2, 2, "tensor"), ("bfloat16", 20, 12, 4, 2, None)])
@pytest.mark.parametrize("size,page", [(16, 16), (17, 16), (33, 16), (5, 4), (64, 16), (45, 32), (128, 64), (1, 16)])
def test_keys_at_the_first_and_last_place_of_every_stretch(dtype, D, V, H, G, expect, size, page):
    """A query sees exactly the marks of its own stretch, in a prompt of 230 and decoded one by one; the pages of earlier
    stretches are unmapped (tests/modinex_cases.py: chunk_edge_case)."""
    m, rows, qn, kn, pb, places, want = C.chunk_edge_case(size, D, V, seed=size * 7 + page + D, H=H, G=G)
    if expect and page not in (16, 32, 64, 128):
        expect = None
    got = _attention_by_kernels(dtype, m, rows, qn, kn, pb, [230] + [1] * 30, page, expect=expect)
    assert np.abs(got - want).max() <= (5e-5 if dtype == "float32" else 4e-2) * np.abs(want).max()
    for p, marks in places.items():
        assert np.abs(got[p] - 5.0 * marks).max() < 0.5


def _run_gla(rows, g, lens, cuts, slots, H, D, V, dtype="float32", n_slots=6, chunked=False, w_norm=None, gate=None, eps=1e-5):
    """rows, g: per request the product's rows [q | k | v] and log decays.  -> (outputs per request [T, H * V], states);
    chunked: gla_chunked (bfloat16), whose outputs are normed and gated up to 128 value columns."""
    import torch
    from imparo_b200.kernels import ops
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    S = torch.full((n_slots, H, D, V), 7.0, device="cuda")
    S[slots] = 0.0
    status = ops.new_status("cuda")
    qk, vv = H * D, H * V
    got, at = [np.zeros((k, vv)) for k in lens], [0] * len(lens)
    for cut in cuts:
        items = [i for i in range(len(lens)) if cut[i]]
        starts = np.concatenate([[0], np.cumsum([cut[i] for i in items])]).astype(np.int32)
        x = np.concatenate([np.concatenate([rows[i][at[i]:at[i] + cut[i]], gate[i][at[i]:at[i] + cut[i]]], axis=1) for i in items])
        gg = _f32(np.concatenate([g[i][at[i]:at[i] + cut[i]] for i in items]))
        T = len(x)
        proj = torch.zeros(T, 2 * qk + 2 * vv, dtype=tdt, device="cuda")
        proj[:] = _dev(x, tdt)
        sl = _dev(np.array([slots[i] for i in items], dtype=np.int32))
        o = torch.empty(T, vv, device="cuda")
        if chunked:
            offs = (0, qk, 2 * qk, 2 * qk + vv)
            assert ops.gla_chunked_takes(proj, offs, D, V)
            n = T // ops.GLA_CHUNK + len(items)
            y = torch.empty(T, vv, dtype=tdt, device="cuda")
            done = ops.gla_chunked(proj, offs, gg, D ** -0.5, _f32(w_norm), eps, S, _dev(starts), sl, len(items),
                                   torch.empty(n * H * D * V, device="cuda"), torch.empty(n * H * D, device="cuda"), o, y, H, D, V, status)
            assert done == (V <= 128)
            if not done:
                ops.head_norm_gate(o, _f32(w_norm), eps, proj[:, 2 * qk + vv:], y, H, V, act="silu")
            oc = y.float().cpu().numpy()
        else:
            ops.gla_scan(proj, 0, qk, 2 * qk, gg, D ** -0.5, S, _dev(starts), sl, len(items), o, H, D, V, status)
            oc = o.cpu().numpy()
        for k, i in enumerate(items):
            got[i][at[i]:at[i] + cut[i]] = oc[starts[k]:starts[k + 1]]
            at[i] += cut[i]
    ops.read_status(status)
    return got, S


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,V", [(4, 32, 40), (2, 16, 24), (3, 8, 40), (1, 40, 70), (2, 136, 20), (1, 7, 5), (2, 64, 64), (1, 200, 33), (2, 16, 200), (1, 72, 264)])
def test_recurrence_kernel(H, D, V, dtype):
    """Three requests of unequal length: a launch of portions, then their next portions and single tokens from the states the
    launches before left (slots in no particular order), against the plain recurrence on each whole sequence; the final states."""
    rng = np.random.default_rng(H * 100 + D)
    lens, slots = [137, 5, 90], [4, 0, 2]
    made = [C.memory_inputs(rng, n, H, D, V, strength=0.1) for n in lens]
    rows = [m[0] if dtype == "float32" else _bf16_round(m[0]) for m in made]
    g = [np.asarray(m[1], dtype=np.float32).astype(np.float64) for m in made]
    gate = [np.zeros((n, H * V)) for n in lens]
    got, S = _run_gla(rows, g, lens, ([120, 2, 31], [16, 1, 2], [1, 1, 1], [0, 1, 56]), slots, H, D, V, dtype, gate=gate)
    assert float(S[1].min()) == 7.0 and float(S[3].max()) == 7.0                     # other slots untouched
    for i, r in enumerate(rows):
        want, Sw = C.memory_plain(r, g[i], H, D, V)
        assert np.abs(got[i] - want.reshape(lens[i], -1)).max() <= 3e-5 * np.abs(want).max()
        assert np.abs(S[slots[i]].cpu().numpy() - Sw).max() <= 3e-5 * np.abs(Sw).max()


@pytest.mark.parametrize("strength", [0.02, 0.3, 3.0])
@pytest.mark.parametrize("H,D,V", [(2, 64, 64), (3, 32, 128), (1, 128, 80), (2, 16, 16), (1, 96, 208), (2, 48, 256), (1, 128, 128)])
def test_recurrence_in_chunks(H, D, V, strength):
    """The tensor-core chunks (bfloat16) on requests of 1 to 300 rows, portion after portion, from weak decays to decays that
    leave nothing of a row after a few steps (where growing factors would leave the range of numbers)."""
    rng = np.random.default_rng(H * 100 + D)
    lens, slots = [300, 5, 190], [4, 0, 2]
    made = [C.memory_inputs(rng, n, H, D, V, strength=strength) for n in lens]
    rows = [_bf16_round(m[0]) for m in made]
    g = [np.asarray(m[1], dtype=np.float32).astype(np.float64) for m in made]
    gate = [_bf16_round(rng.standard_normal((n, H * V))) for n in lens]
    w = rng.uniform(0.5, 1.5, V)
    got, S = _run_gla(rows, g, lens, ([200, 2, 131], [99, 1, 2], [1, 1, 1], [0, 1, 56]), slots, H, D, V, "bfloat16", chunked=True, w_norm=w, gate=gate)
    assert float(S[1].min()) == 7.0 and float(S[3].max()) == 7.0
    for i, r in enumerate(rows):
        o, Sw = C.memory_plain(r, g[i], H, D, V)
        want = (P.unit_rms(o, 1e-5) * w).reshape(lens[i], -1) * P.silu(gate[i])
        assert np.abs(S[slots[i]].cpu().numpy() - Sw).max() <= 1e-4 * np.abs(Sw).max()
        assert np.abs(got[i] - want).max() <= 6e-3 * np.abs(want).max()


@pytest.mark.parametrize("dtype,chunked", [("float32", False), ("bfloat16", False), ("bfloat16", True)])
def test_state_carries_a_far_token(dtype, chunked):
    """A key channel that never decays and that only the first token writes to is read back hundreds of tokens later, in a prompt
    and in single tokens (tests/modinex_cases.py: far_memory_case)."""
    (H, D, V), rows, g, seekers, want = C.far_memory_case()
    if dtype == "bfloat16":
        rows = _bf16_round(rows)
        want, _ = C.memory_plain(rows, g, H, D, V)
    gate = np.full((420, H * V), 1.0)
    got, _ = _run_gla([rows], [g], [420], [[400]] + [[1]] * 20, [1], H, D, V, dtype, n_slots=2, chunked=chunked, w_norm=np.ones(V), gate=[gate])
    if chunked:
        o = want
        want = (P.unit_rms(o, 1e-5)).reshape(420, -1) * P.silu(gate)
        assert np.abs(got[0] - want).max() <= 6e-3 * np.abs(want).max()
        return
    assert np.abs(got[0] - want.reshape(420, -1)).max() <= 5e-5 * np.abs(want).max()
    assert all(abs(got[0][t, 0] - 5.0) < 0.05 for t in seekers)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,V,rank,tau", [(4, 32, 40, 12, 11.0), (2, 64, 128, 5, 1.0), (3, 100, 48, 20, 4.0), (1, 200, 100, 33, 9.0), (2, 7, 300, 1, 2.0),
                                            (2, 128, 256, 16, 16.0)])
def test_one_row_step_with_decay_norm_and_gate(H, D, V, rank, tau, dtype):
    """gla_step against gla_decay + gla_scan + head_norm_gate and against the plain formulas, over five steps of four requests."""
    import torch
    from imparo_b200.kernels import ops
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    rnd = (lambda a: a) if dtype == "float32" else _bf16_round
    rng = np.random.default_rng(H + D + V)
    n, steps, qk, vv = 4, 5, H * D, H * V
    cols = (0, qk, 2 * qk, 2 * qk + vv, 2 * qk + 2 * vv)
    x = rnd(rng.standard_normal((steps, n, cols[4] + rank)))
    w2, b, w = rnd(rng.standard_normal((qk, rank)) / np.sqrt(rank)), rng.uniform(-2.0, 4.0, qk), rng.uniform(0.5, 1.5, V)
    slots, starts = _dev(np.array([3, 0, 4, 1], dtype=np.int32)), _dev(np.arange(n + 1, dtype=np.int32))
    status = ops.new_status("cuda")
    S1, S2 = torch.zeros(5, H, D, V, device="cuda"), torch.zeros(5, H, D, V, device="cuda")
    S1[2] = 3.0
    Sw = [np.zeros((H, D, V)) for _ in range(n)]
    for t in range(steps):
        proj = _dev(x[t], tdt)
        y1, y2 = torch.empty(n, vv, dtype=tdt, device="cuda"), torch.empty(n, vv, dtype=tdt, device="cuda")
        took = ops.gla_step(proj, cols, rank, _dev(w2, tdt), _f32(b), tau, _f32(w), 1e-5, D ** -0.5, S1, starts, slots, n, y1, H, D, V, status)
        assert took
        g, o = torch.empty(n, qk, device="cuda"), torch.empty(n, vv, device="cuda")
        ops.gla_decay(proj[:, cols[4]:], _dev(w2, tdt), _f32(b), tau, g)
        ops.gla_scan(proj, 0, qk, 2 * qk, g, D ** -0.5, S2, starts, slots, n, o, H, D, V, status)
        ops.head_norm_gate(o, _f32(w), 1e-5, proj[:, cols[3]:cols[4]], y2, H, V, act="silu")
        z = x[t][:, cols[4]:] @ w2.T + b
        gw = np.log(P.channel_decay(z, tau))
        assert np.abs(g.cpu().numpy() - gw).max() <= 2e-6 * max(np.abs(gw).max(), 1.0)
        want = np.zeros((n, vv))
        for i in range(n):
            ow, Sw[i] = C.memory_plain(x[t][i:i + 1, :cols[3]], gw[i:i + 1], H, D, V, Sw[i])
            want[i] = (P.unit_rms(ow, 1e-5) * w).reshape(-1) * P.silu(x[t][i, cols[3]:cols[4]])
        tol = (3e-5 if dtype == "float32" else 1e-2) * np.abs(want).max()
        for y in (y1, y2):
            assert np.abs(y.float().cpu().numpy() - want).max() <= tol
    ops.read_status(status)
    assert float((S1[[0, 1, 3, 4]] - S2[[0, 1, 3, 4]]).abs().max()) <= 1e-4 and float(S1[2].min()) == 3.0


@pytest.mark.parametrize("H,D,V,rank,tau", [(2, 64, 64, 16, 16.0), (1, 128, 128, 5, 1.0), (3, 48, 32, 32, 4.0), (2, 16, 144, 1, 2.0), (1, 96, 80, 27, 0.3)])
def test_chunks_make_their_decays(H, D, V, rank, tau):
    """The first launch of the chunked form makes the log decays from the inner columns: the same as gla_decay's, and the same
    outputs and states as with decays given."""
    import torch
    from imparo_b200.kernels import ops
    rng = np.random.default_rng(H + D + V + rank)
    qk, vv = H * D, H * V
    l_at = (2 * qk + 2 * vv + 7) // 8 * 8
    T, starts = 333, np.array([0, 130, 133, 333], dtype=np.int32)
    proj = _dev(rng.standard_normal((T, (l_at + rank + 7) // 8 * 8)), torch.bfloat16)
    w2, b = _dev(rng.standard_normal((qk, rank)) / np.sqrt(rank), torch.bfloat16), _f32(rng.uniform(-1.0, 4.0, qk))
    offs = (0, qk, 2 * qk, 2 * qk + vv, l_at)
    slots, w = _dev(np.array([2, 0, 1], dtype=np.int32)), _f32(rng.uniform(0.5, 1.5, V))
    status = ops.new_status("cuda")
    g1, g2 = torch.empty(T, qk, device="cuda"), torch.full((T, qk), 5.0, device="cuda")
    ops.gla_decay(proj[:, l_at:l_at + rank], w2, b, tau, g1)
    n = T // ops.GLA_CHUNK + 3
    res = []
    for g, decay in ((g1, None), (g2, (w2, b, tau, rank))):
        S = torch.ones(3, H, D, V, device="cuda")
        o, y = torch.zeros(T, vv, device="cuda"), torch.zeros(T, vv, dtype=torch.bfloat16, device="cuda")
        ops.gla_chunked(proj, offs, g, D ** -0.5, w, 1e-5, S, _dev(starts), slots, 3, torch.empty(n * H * D * V, device="cuda"),
                        torch.empty(n * H * D, device="cuda"), o, y, H, D, V, status, decay=decay)
        res.append((S, o if V > 128 else y.float()))
    ops.read_status(status)
    assert float((g1 - g2).abs().max()) <= 1e-5 * max(1.0, float(g1.abs().max()))
    for x, y in zip(*res):
        assert float((x - y).abs().max()) <= 1e-2 * float(x.abs().max())


@pytest.mark.parametrize("T,width,F,kind,biased,dtype", [(300, 128, 256, "gelu_tanh", True, "bfloat16"), (700, 64, 136, "gelu_tanh", True, "bfloat16"),
                                                         (256, 192, 80, "relu2", False, "bfloat16"), (5, 256, 64, "gelu_tanh", True, "bfloat16"),
                                                         (33, 52, 30, "silu", True, "bfloat16"), (19, 52, 37, "gelu_tanh", True, "float32"),
                                                         (1, 1024, 512, "gelu_tanh", True, "bfloat16"), (40, 128, 200, "silu", False, "bfloat16")])
def test_product_with_bias_and_activation(T, width, F, kind, biased, dtype):
    import torch
    from imparo_b200.kernels import ops
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    rng = np.random.default_rng(T + F)
    x, w = _bf16_round(rng.standard_normal((T, width))), _bf16_round(rng.standard_normal((F, width)) / np.sqrt(width) * 2.0)
    bias = rng.standard_normal(F) if biased else None
    z = x @ w.T + (bias if biased else 0.0)
    want = {"gelu_tanh": P.gelu_tanh, "silu": P.silu, "relu2": lambda v: np.maximum(v, 0.0) ** 2}[kind](z)
    out = torch.empty(T, F, dtype=tdt, device="cuda")
    status = ops.new_status("cuda")
    ops.linear_act(_dev(x, tdt), _dev(w, tdt), out, kind, bias=None if bias is None else _f32(bias), status=status)
    ops.read_status(status)
    assert np.abs(out.float().cpu().numpy() - want).max() <= (1e-5 if dtype == "float32" else 1.5e-2) * np.abs(want).max()


# ---- generation ------------------------------------------------------------------------------------------------

def plain_generate(name, prompt, n_new):
    toks, out, margins = list(prompt), [], []
    for _ in range(n_new):
        row = plain_logits(name, {"g": toks})["g"][-1]
        t = int(np.argmax(row))
        top2 = np.partition(row, -2)[-2:]
        out.append(t)
        margins.append(float(top2[1] - top2[0]))
        toks.append(t)
    return out, margins


@pytest.mark.parametrize("dtype,min_margin", [("float32", 1e-3), ("bfloat16", 0.3)])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_greedy_generation_through_the_scheduler(name, dtype, min_margin):
    """Three prompts through Engine.generate: continuous batching with prompt portions of at most 8 tokens beside
    decoding requests, two state slots for three requests, pages used again."""
    from imparo_b200.engine import Engine
    from tests.test_generate_gpu import agree
    prompts = list(make_requests(name, [5, 23, 40], seed=1).values())
    page = PAGE[name]
    eng = Engine(model_dir(name), dtype=dtype, ctx=64, parallel=2, page_size=page, num_pages=2 * (64 // page), max_step_tokens=8)
    got = eng.generate(prompts, max_tokens=10)
    for i, p in enumerate(prompts):
        want, margins = plain_generate(name, p, 10)
        agree(got[i], want, margins, min_margin)
    assert eng.cache.n_requests() == 0
    eng.cache.check()


def test_command_line_and_trace_runner(tmp_path):
    from tests.test_trace_run_gpu import replay
    name = "A"
    prompt = make_requests(name, [16], seed=0)["r0"]
    want, _ = plain_generate(name, prompt, 6)
    tf = tmp_path / "tokens.txt"
    tf.write_text(" ".join(map(str, prompt)))
    r = subprocess.run([sys.executable, "-m", "imparo_b200", "-m", model_dir(name), "--dtype", "float32", "--decode", "6",
                        "-c", "64", "-t", str(tf), "--json"], cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(r.stdout.strip().splitlines()[-1])["tokens"] == [want]
    reqs = make_requests(name, [70, 33, 90, 41, 64, 52], seed=7)
    steps = traces.mixed(reqs, seed=1)
    max_tokens = traces.max_live_tokens(steps, 64)
    out = tmp_path / "out"
    replay(model_dir(name), "bfloat16", steps, out, max_tokens)
    ref = plain_logits(name, reqs)
    want = traces.expected(steps, ref)
    got = {s["step"]: np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, ALL[name]["vocab"]) for s in steps if s["step"] in want}
    scale = max(float(np.abs(v).max()) for v in ref.values())
    errs = all_errors(steps, got, want)
    assert max(e[3] for e in errs) <= WORST["bfloat16"] * scale
    assert sum(e[3] > TOL["bfloat16"] * scale for e in errs) <= 0.1 * len(errs)
