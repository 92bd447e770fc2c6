"""The plain Zinunex implementation checked by hand on small inputs (closed forms that share nothing with its loops), the
made-up cases of tests/zinunex_cases.py checked for what they claim, and the host side of the design: configuration errors,
the tensors a model declares, its schedule, what it asks of the cache manager and what the manager keeps for readers."""
import copy

import numpy as np
import pytest

from tests import zinunex_cases as C
from tests.plain import zinunex_plain as P
from tests.zinunex_configs import ALL


def test_rotations_depend_on_distance_only_and_leave_the_rest():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 12)), rng.standard_normal((1, 12))
    freq = P.plain_frequencies(50.0, 8)
    for turn in (P.turn_neighbours, P.turn_halves):
        dots = [float((turn(q, [p + d], freq) * turn(k, [p], freq)).sum()) for p, d in ((0, 7), (100, 7), (31, 7))]
        assert np.allclose(dots, dots[0])
        assert np.array_equal(turn(q, [9], freq)[:, 8:], q[:, 8:])           # dimensions beyond rot.dims pass unchanged
        assert np.array_equal(turn(q, [0], freq), q)
    a = 9 * 50.0 ** (-2 * 1 / 8)                                              # the second pair's angle
    r = P.turn_neighbours(q, [9], freq)
    assert np.allclose(r[0, 2], q[0, 2] * np.cos(a) - q[0, 3] * np.sin(a)) and np.allclose(r[0, 3], q[0, 3] * np.cos(a) + q[0, 2] * np.sin(a))
    r = P.turn_halves(q, [9], freq)
    assert np.allclose(r[0, 1], q[0, 1] * np.cos(a) - q[0, 5] * np.sin(a)) and np.allclose(r[0, 5], q[0, 5] * np.cos(a) + q[0, 1] * np.sin(a))


def test_blended_frequencies():
    base, n, sc = 10000.0, 32, {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}
    f, mag = P.blended_frequencies(base, n, sc)
    plain = P.plain_frequencies(base, n)
    assert np.isclose(mag, 0.1 * np.log(8.0) + 1.0)
    # pairs below the dimension at which `fast` turns fit keep their frequency, those above that of `slow` are divided
    where = lambda t: n * np.log(2048 / (2 * np.pi * t)) / (2 * np.log(base))
    lo, hi = np.floor(where(32.0)), np.ceil(where(1.0))
    assert 0 < lo < hi < n / 2
    for i in range(n // 2):
        if i <= lo:
            assert np.isclose(f[i], plain[i])
        elif i >= hi:
            assert np.isclose(f[i], plain[i] / 8.0)
        else:
            assert plain[i] / 8.0 < f[i] < plain[i]
    assert np.array_equal(P.blended_frequencies(base, n, None)[0], plain) and P.blended_frequencies(base, n, None)[1] == 1.0


def test_window_and_sink():
    T, size = 12, 4
    q, k, v = np.ones((T, 1, 2)), np.zeros((T, 1, 2)), np.arange(T, dtype=float).reshape(T, 1, 1)
    out = P.softmax_attention(q, k, v, 1.0, size)[:, 0, 0]
    for i in range(T):
        assert np.isclose(out[i], np.mean(range(max(0, i - size + 1), i + 1)))
    with_sink = P.softmax_attention(q, k, v, 1.0, None, np.array([np.log(3.0)]))[:, 0, 0]
    assert np.allclose(with_sink, [sum(range(i + 1)) / (i + 1 + 3.0) for i in range(T)])


def test_router_groups_correction_and_scale():
    s = np.array([[0.9, 0.1, 0.6, 0.55, 0.3, 0.2]])
    z = np.log(s / (1.0 - s))
    zero = np.zeros(6)
    ids, w = P.route(z, zero, 2, 3, 1, 2.0)                     # pair sums 1.0, 1.15, 0.5: not the group with the largest single
    assert ids.tolist() == [[2, 3]] and np.allclose(w, [[1.2, 1.1]])
    ids, w = P.route(z, zero, 2, 3, 2, 1.0)
    assert ids.tolist() == [[0, 2]]
    corr = np.array([-2.0, -2.0, -0.5, 0.0, 0.9, 0.9])
    ids, w = P.route(z, corr, 2, 3, 2, 1.0)                     # choice: -1.1, -1.9, 0.1, 0.55, 1.2, 1.1
    assert ids.tolist() == [[4, 5]] and np.allclose(w, [[0.3, 0.2]])      # weights are the scores without the correction
    ids, w = P.route(z, np.full(6, -5.0), 3, 2, 1, 1.0)         # all choice scores negative: a group left out stays out
    assert sorted(ids.tolist()[0]) == [0, 1, 2]
    ids, _ = P.route(z, zero, 1, 6, 2, 1.0)                     # groups of one expert
    assert ids.tolist() == [[0]]


def test_expert_shared_factor_and_side_input():
    W = {"e0.up": np.array([[1.0], [-1.0]]), "e0.down": np.array([[2.0, 10.0]]), "router": np.array([[0.0]]), "correction": np.zeros(1),
         "shared.up": np.array([[1.0]]), "shared.down": np.array([[1.0]]), "shared.sg": np.array([[np.log(3.0)]])}
    mlp = {"router": {"experts": 1, "top": 1, "scale": 4.0}, "expert": {"ff": 2}, "shared": {"ff": 1}}
    out = P.moe_ff(np.array([[3.0], [1.0], [-1.0]]), W, "", mlp)
    routed = lambda x: 4.0 * 0.5 * (2.0 * max(x, 0.0) ** 2 + 10.0 * max(-x, 0.0) ** 2)
    shared = lambda x: 1.0 / (1.0 + 3.0 ** -x) * max(x, 0.0) ** 2
    assert np.allclose(out[:, 0], [routed(x) + shared(x) for x in (3.0, 1.0, -1.0)])
    x, e = np.array([[1.0, 2.0]]), np.array([[0.5]])
    W = {"side.gate": np.array([[1.0, -1.0]]), "side.proj": np.array([[3.0], [4.0]]), "side.norm": np.array([2.0, 1.0])}
    g = float(P.gelu_tanh(np.array(-1.0))) * 0.5
    assert np.isclose(P.gelu_tanh(np.array(-1.0)), -0.158808, atol=1e-6)
    y = np.array([3.0 * g, 4.0 * g])
    want = x[0] + y / np.sqrt((y @ y) / 2 + 1e-6) * W["side.norm"]
    assert np.allclose(P.token_side(x, e, W, "", 1e-6)[0], want)


def tiny_weights(cfg, seed=0):
    from imparo_b200.weights.random_init import draw_random_tensors, model_on_cpu
    _, _, model = model_on_cpu(cfg)
    return {k: v.float().numpy().astype(np.float64) for k, v in draw_random_tensors(model.weight_specs(), seed, "float32", "cpu", matrix_std=0.3).items()}


def test_causality_side_table_and_shared_latents():
    cfg = ALL["A"]
    W = tiny_weights(cfg)
    toks = [5, 9, 5, 100, 7, 5]
    base = P.forward(cfg, W, toks)
    assert np.allclose(P.forward(cfg, W, toks[:4]), base[:4])                # later tokens change nothing before them
    moved = dict(W, **{"side.embed": W["side.embed"].copy()})
    moved["side.embed"][100, 3 * 12:4 * 12] += 1.0                           # one token's entries of layer 3
    layers0, layers1 = [], []
    P.forward(cfg, W, toks, layer_outputs=layers0)
    P.forward(cfg, moved, toks, layer_outputs=layers1)
    assert len(layers0) == len(cfg["layers"])
    assert all(np.array_equal(layers0[i], layers1[i]) for i in range(3))
    assert np.abs(layers0[3][3] - layers1[3][3]).max() > 1e-3 and np.array_equal(layers0[3][:3], layers1[3][:3])
    latents = dict(W, **{"l1.mix.dkv.norm": W["l1.mix.dkv.norm"] * 1.5})     # the source's latent reaches its readers
    lay = []
    P.forward(cfg, latents, toks, layer_outputs=lay)
    assert np.array_equal(lay[0], layers0[0]) and np.abs(lay[4] - layers0[4]).max() > 1e-6


def test_made_up_cases_are_decided_by_their_far_element():
    for through in ("latent", "rotated"):
        for window in (None, 37):
            m, W, proj, seen, unseen, v_far, want = C.far_latent_case(15, 1, through=through, window=window)
            w = want.reshape(len(want), m["heads"], m["vdim"])
            assert len(seen) >= 3 and bool(unseen) == (window is not None)
            for t in seen:
                assert np.abs(w[t] - v_far).max() < 0.05 * np.abs(v_far).max()
            for t in unseen:
                assert np.abs(w[t] - v_far).max() > 0.3 * np.abs(v_far).max()
    m, rows, sink, seekers, v_far, want = C.far_key_case(16, 32, 3, n_rot=20)
    assert len(seekers) == 5
    for t in seekers:
        assert np.abs(want[t, :32] - v_far).max() < 0.05 * np.abs(v_far).max()
    assert np.abs(want[301, :32] - v_far).max() > 0.5 * np.abs(v_far).max()
    # leaving the sinks out changes the first tokens by more than half of what they are
    m, rows, sink, want = C.sink_case(16, 5)
    without = C.attention_rows_plain(m, rows, np.full(4, -50.0))
    for t in (0, 1, 5):
        assert np.abs(want[t] - without[t]).max() > 0.5 * np.abs(without[t]).max()
    assert np.abs(want[149] - without[149]).max() > 0.3 * np.abs(without[149]).max()


# ---- the host side ---------------------------------------------------------------------------------------------------

def test_configuration_reads_every_size_and_names_what_is_wrong():
    from imparo_b200.config import ConfigError, load_config
    arch, cfg = load_config(ALL["A"])
    assert arch.name == "Zinunex" and cfg.width == 64 and cfg.eps == 1e-5 and cfg.side_dim == 12
    a = cfg.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.rot_dims, a.rot_factor) == (4, 2, 16, 16, 3.0)
    lat = cfg.layers[2].mixer
    assert (lat.heads, lat.dim, lat.rot_dim, lat.vdim, lat.kv_rank, lat.window, lat.kv_from, lat.rot_base) == (2, 8, 8, 20, 24, 21, 1, 300.0)
    assert (lat.rot_scaling.factor, lat.rot_scaling.original, lat.rot_scaling.fast, lat.rot_scaling.slow) == (4.0, 64.0, 8.0, 1.0)
    moe = cfg.layers[0].mlp
    assert (moe.experts, moe.top, moe.groups, moe.keep, moe.scale, moe.ff, moe.shared_ff) == (6, 2, 3, 2, 1.7, 24, 24)
    assert cfg.layers[2].mlp is None and cfg.layers[3].mlp.shared_ff is None
    e = load_config(ALL["E"])[1]
    assert e.side_dim is None and e.layers[0].mixer.rot_dims == 0 and e.layers[1].mixer.rot_dim == 0 and e.layers[1].mixer.window == 1
    b = load_config(ALL["B"])[1]
    assert b.layers[2].mixer.window is None and b.layers[0].mixer.rot_scaling is None and b.layers[1].mixer.rot_dims == 10

    def broken(change):
        c = copy.deepcopy(ALL["A"])
        change(c)
        return c
    for change, word in ((lambda c: c["layers"][0].update(type="conv"), "unknown type"),
                         (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
                         (lambda c: c["layers"][0]["mixer"].update(vdim=8), "vdim"),
                         (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
                         (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "dims"),
                         (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
                         (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "kv_from"),
                         (lambda c: c["layers"][2]["mixer"].update(kv_from=4), "kv_from"),
                         (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "kv_from"),
                         (lambda c: c["layers"][2]["mixer"].update(kv_rank=32), "kv_rank"),
                         (lambda c: c["layers"][2]["mixer"]["rot"].update(base=10.0), "rotation"),
                         (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "count"),
                         (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "top"),
                         (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "unknown kind"),
                         (lambda c: c["layers"][0]["mlp"].pop("expert"), "expert"),
                         (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
                         (lambda c: c.pop("norm"), "norm")):
        with pytest.raises(ConfigError, match=word):
            load_config(broken(change))


def test_tensors_schedule_and_cache_needs():
    from imparo_b200.parts.spec import PagedKV
    from imparo_b200.weights.random_init import model_on_cpu
    _, _, model = model_on_cpu(ALL["A"])
    names = {w.name: w.shapes[0] for w in model.weight_specs()}
    assert names["embed"] == (211, 64) and names["head"] == (211, 64) and names["side.embed"] == (211, 5 * 12)
    assert names["l0.mix.q"] == (64, 64) and names["l0.mix.k"] == (32, 64) and names["l0.mix.sink"] == (4,) and "l0.mix.v" not in names
    assert names["l1.mix.q"] == (3 * 24, 64) and names["l1.mix.dkv"] == (32, 64) and names["l1.mix.dkv.norm"] == (24,)
    assert names["l2.mix.q"] == (2 * 16, 64) and names["l2.mix.uk"] == (16, 24) and names["l2.mix.uv"] == (40, 24) and "l2.mix.dkv" not in names
    assert names["l0.mlp.router"] == (6, 64) and names["l0.mlp.correction"] == (6,) and names["l0.mlp.e5.down"] == (64, 24)
    assert "l0.mlp.e0.gate" not in names and names["l1.mlp.shared.up"] == (20, 64) and names["l1.mlp.shared.sg"] == (1, 64)
    assert "l3.mlp.shared.up" not in names and "l2.norm2" not in names and "l2.mlp.router" not in names
    assert names["l4.side.gate"] == (12, 64) and names["l4.side.proj"] == (64, 12) and names["l4.side.norm"] == (64,)
    assert [(e.layer, e.cache_from) for e in model.schedule] == [(0, None), (1, None), (2, 1), (3, None), (4, 1)]
    needs = dict(model.cache_requirements())
    # the source keeps what its longest reader sees
    assert needs == {0: (PagedKV(2, 16),), 1: (PagedKV(1, 32, 21, None, values_are_keys=True),), 3: (PagedKV(3, 8),)}
    _, _, model = model_on_cpu(ALL["B"])
    assert dict(model.cache_requirements())[0] == (PagedKV(1, 40, None, None, values_are_keys=True),)      # a reader without a window
    _, _, model = model_on_cpu(ALL["E"])
    assert "side.embed" not in {w.name for w in model.weight_specs()}


def test_cached_rows_are_padded_in_bfloat16_only_where_it_pays():
    import torch
    from imparo_b200.parts.base import Runtime, Workspace, make_part
    from imparo_b200.parts.spec import PartSpec
    for rank, rot, precision, row in ((48, 16, "bfloat16", 64), (60, 32, "bfloat16", 128), (24, 8, "bfloat16", 32), (28, 12, "bfloat16", 64),
                                      (60, 32, "float32", 92), (200, 16, "bfloat16", 216), (96, 32, "bfloat16", 128)):
        rt = Runtime(precision=precision, device=torch.device("cpu"), workspace=Workspace("cpu"))
        part = make_part("mixer", PartSpec("latent_attention", {
            "hidden": 32, "heads": 2, "dim": 8, "vdim": 8, "kv_rank": rank, "rot_dim": rot, "scale": 0.1, "eps": 1e-6, "pad_row": True,
            "position": PartSpec("rope_interleaved", {"head_dim": rot, "theta": 100.0})}), "", rt)
        assert part.cache_specs()[0].head_dim == row
        assert [w.shapes[0] for w in part.weight_specs() if w.name == "dkv"] == [(rank + rot, 32)]


def test_the_cache_manager_keeps_what_a_reader_with_a_longer_window_sees():
    from imparo_b200.cache import CacheManager
    from imparo_b200.weights.random_init import model_on_cpu
    _, _, model = model_on_cpu(ALL["A"])
    reqs = model.cache_requirements()
    cm = CacheManager(reqs, page_size=4, num_pages=40, num_slots=2)
    g = [k.window for k in cm.group_keys].index(21)
    cm.add(1)
    for n in (30, 1, 1, 1):
        cm.reserve(1, n)
        cm.commit(1, n)
    # 33 positions cached; the next query (33) of the longest reader sees 13..33: pages from 12 // 4 = 3 on are still there
    table = cm.table(1, g)
    assert (table[:3] < 0).all() and (table[3:9] >= 0).all()
    cm.release(1)
    assert cm.free_pages(g) == 40


def test_a_reader_of_other_rows_is_refused():
    from imparo_b200.parts.spec import PagedKV, SlotState, keeping_for, reads_as
    a = PagedKV(1, 32, 9, None, values_are_keys=True)
    assert reads_as(PagedKV(1, 32, None, None, values_are_keys=True), a) and not reads_as(PagedKV(1, 40, 9, None, values_are_keys=True), a)
    assert not reads_as(SlotState((3,)), a) and reads_as(SlotState((3,)), SlotState((3,)))
    assert keeping_for(a, PagedKV(1, 32, 4, None, values_are_keys=True)) == a
    assert keeping_for(a, PagedKV(1, 32, 12, None, values_are_keys=True)).window == 12
    assert keeping_for(PagedKV(2, 8, chunk=5), PagedKV(2, 8, chunk=5)).chunk == 5
    assert keeping_for(PagedKV(2, 8, chunk=5), PagedKV(2, 8)).chunk is None
