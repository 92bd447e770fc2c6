"""Modinex configurations drawn from a seeded generator: widths, the number and order of the two layer types, feed-forwards on
either or none, heads per key head, key and value sizes (also those the tensor-core kernels take, next to sizes they decline),
rotation of the whole head, a part or none, stretches shorter and longer than a page, of one position or no mask, decay powers
and inner sizes, norm groups, page sizes, ways of cutting; each replayed as a mixed trace in 32-bit (every position) and
bfloat16 against the plain implementation."""
import json
import os
import tempfile

import numpy as np
import pytest

from tests import traces
from tests.plain import modinex_plain as P
from tests.plain.lfm2_plain import read_safetensors

pytestmark = pytest.mark.gpu
_tmp = tempfile.TemporaryDirectory(prefix="imparo_b200_modinex_random_")


def draw_config(seed, fast=False):
    """fast: key and value sizes in multiples of 16 and widths in multiples of 8 (what the tensor-core kernels take)."""
    rng = np.random.default_rng(7000 + seed + (5000 if fast else 0))
    pick = lambda xs: xs[int(rng.integers(0, len(xs)))]
    width = pick([64, 128, 192, 256]) if fast else pick([36, 48, 64, 96, 100, 120, 128, 160])
    groups = pick([g for g in (1, 2, 3, 4, 5, 6, 8, 10) if width % g == 0 and width // g >= 8])

    def attention():
        heads = pick([1, 2, 3, 4, 6, 8, 12])
        kv = pick([k for k in (1, 2, 3, 4, 6, 8, 12) if heads % k == 0])
        dim, vdim = pick([6, 8, 12, 16, 24, 32, 50, 64, 80, 136]), pick([5, 8, 12, 16, 24, 40, 64, 80, 130])
        if fast:
            heads = pick([1, 2, 4, 8, 16, 24])
            kv = pick([k for k in (1, 2, 4, 8) if heads % k == 0])
            dim, vdim = pick([16, 32, 48, 64, 80, 96, 128]), pick([16, 32, 48, 64, 80, 96, 112, 128])
        m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": float(rng.uniform(0.5, 3.0)) / dim}
        if rng.random() < 0.9:
            m["mask"] = {"size": int(pick([1, 2, 5, 16, 17, 31, 45, 64, 100, 128, 300]))}
        if rng.random() < 0.85:
            m["rot"] = {"base": float(pick([50.0, 10000.0, 1000000.0])), "dims": dim if rng.random() < 0.5 else 2 * int(rng.integers(1, dim // 2 + 1))}
        return {"type": "attention", "mixer": m}

    def gla():
        dim, vdim = pick([4, 7, 8, 16, 24, 32, 64, 100, 128, 200]), pick([4, 8, 12, 20, 32, 33, 48, 64, 70, 128, 260])
        if fast:
            dim, vdim = pick([16, 32, 48, 64, 96, 128]), pick([16, 32, 48, 64, 96, 128, 160, 256])
        return {"type": "gla", "mixer": {"heads": pick([1, 2, 3, 4, 6]), "dim": dim, "vdim": vdim, "tau": float(pick([0.5, 1.0, 3.0, 8.0, 16.0, 40.0])),
                                         "rank": pick([1, 3, 8, 16, 20, 40])}}

    def layer():
        L = attention() if rng.random() < 0.55 else gla()
        L["mlp"] = {"kind": "dense", "ff": int(pick([16, 30, 64, 100, 128]))} if rng.random() < 0.6 else None
        return L
    cfg = {"architecture": "Modinex", "vocab": int(rng.integers(100, 700)), "width": width, "max_positions": 640,
           "norm": {"eps": float(pick([1e-6, 1e-5, 3e-6])), "groups": groups}, "layers": [layer() for _ in range(int(rng.integers(2, 7)))]}
    return cfg, rng


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", list(range(14)) + [f"fast{i}" for i in range(10)])
def test_drawn_configuration_mixed_trace(seed, dtype):
    from imparo_b200.engine import Engine
    from imparo_b200.weights import write_random_model
    from tests.gpu_helpers import run_trace
    from tests.test_modinex_gpu import TOL, WORST, all_errors, rescale
    fast = isinstance(seed, str)
    seed = int(seed[4:]) if fast else seed
    cfg, rng = draw_config(seed, fast)
    folder = os.path.join(_tmp.name, f"m{seed}{'f' if fast else ''}")
    if not os.path.isdir(folder):
        write_random_model(folder, cfg, seed=seed, dtype="bfloat16", norm_jitter=0.3)
        rescale(os.path.join(folder, "model.safetensors"))
        with open(os.path.join(folder, "config.json"), "w") as f:          # the inner sizes are the stored tensors'
            json.dump(dict(cfg, layers=[dict(L, mixer={k: v for k, v in L["mixer"].items() if k != "rank"}) for L in cfg["layers"]]), f)
    w = read_safetensors(os.path.join(folder, "model.safetensors"))
    lengths = [int(x) for x in rng.integers(3, 200, 3)] + ([int(rng.integers(300, 520))] if fast else [int(rng.integers(3, 200))]) + [1]
    reqs = {f"r{i}": rng.integers(0, cfg["vocab"], n).tolist() for i, n in enumerate(lengths)}
    steps = traces.mixed(reqs, seed=seed, max_portion=int(rng.choice([3, 17, 70, 200])))
    page = int(rng.choice([16, 16, 32, 64])) if fast else int(rng.choice([4, 8, 16, 16, 32, 64]))
    max_tokens = traces.max_live_tokens(steps, max(64, page))
    eng = Engine(folder, dtype=dtype, ctx=max_tokens, parallel=4, page_size=page, num_pages=(max_tokens + page - 1) // page,
                 max_step_tokens=max(256, max_tokens))
    ref = {k: P.forward(cfg, w, t) for k, t in reqs.items()}
    # How much this draw amplifies rounding, place by place: the plain implementation in 32-bit against itself in 64-bit.  (A
    # normed read-out of the recurrence's first tokens is the sign of a dot product, whatever its size; a group of a sublayer's
    # output that is nearly zero is scaled up by its norm.)
    scale = max(float(np.abs(v).max()) for v in ref.values())
    cond = {k: np.abs(P.forward(cfg, w, t, dtype=np.float32) - ref[k]).max(axis=1) / scale for k, t in reqs.items()}
    usual = float(np.median(np.concatenate(list(cond.values()))))
    got = run_trace(eng, steps)
    errs = all_errors(steps, got, traces.expected(steps, ref))
    if dtype == "float32":
        over = [e for e in errs if not e[3] <= max(WORST[dtype], 20 * float(cond[e[1]][e[2]])) * scale]
        assert not over, (cfg, page, over[0], scale)
    else:
        kept = [e for e in errs if float(cond[e[1]][e[2]]) <= 10 * max(usual, 1e-7)]
        assert len(kept) >= 0.5 * len(errs)
        loose = max(1.0, usual / 5e-7)
        assert float(np.median([e[3] for e in kept])) <= TOL[dtype] * loose * scale, (cfg, page, scale)
        assert sum(e[3] > 2 * TOL[dtype] * loose * scale for e in kept) <= 0.1 * len(kept), (cfg, page, max(kept, key=lambda e: e[3]), scale)
    assert eng.cache.n_requests() == 0
