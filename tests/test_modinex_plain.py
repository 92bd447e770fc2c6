"""The plain Modinex implementation checked by hand on small inputs (closed forms that share nothing with its loops), the
made-up cases of tests/modinex_cases.py checked for what they claim, and the host side of the design: configuration errors,
the tensors a model declares, its schedule, what it asks of the cache manager and how that gives stretches back."""
import numpy as np
import pytest

from tests import modinex_cases as C
from tests.modinex_configs import ALL
from tests.plain import modinex_plain as P


def test_norm_in_groups():
    x = np.array([[3.0, 4.0, 0.0, 0.0, 1.0, 1.0]])
    y = P.group_rms(x, 3, 1e-9)
    assert np.allclose(y, [[3 / np.sqrt(12.5), 4 / np.sqrt(12.5), 0, 0, 1, 1]])
    assert np.allclose(P.group_rms(x, 1, 0.0), x / np.sqrt(np.mean(x ** 2)))
    tiny = np.full((1, 4), 1e-4)
    assert np.allclose(P.group_rms(tiny, 2, 1e-5), 1e-4 / np.sqrt(1e-8 + 1e-5))          # eps inside the root


def test_rotation_depends_on_distance_only_and_leaves_the_rest():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 12)), rng.standard_normal((1, 12))
    dots = [float((P.rotate_half_pairs(q, [p + d], 50.0, 8) * P.rotate_half_pairs(k, [p], 50.0, 8)).sum()) for p, d in ((0, 7), (100, 7), (31, 7))]
    assert np.allclose(dots, dots[0])
    r = P.rotate_half_pairs(q, [9], 50.0, 8)
    assert np.array_equal(r[:, 8:], q[:, 8:])
    a = 9 * 50.0 ** (-2 * 1 / 8)                                   # pair (1, 5)
    assert np.allclose(r[0, 1], q[0, 1] * np.cos(a) - q[0, 5] * np.sin(a)) and np.allclose(r[0, 5], q[0, 5] * np.cos(a) + q[0, 1] * np.sin(a))


def test_sigmoid_weights_are_not_normalised_and_stretches_start_at_multiples():
    T, size = 13, 4
    q, k, v = np.zeros((T, 2, 3)), np.zeros((T, 1, 3)), np.ones((T, 1, 1))
    out = P.sigmoid_attention(q, k, v, 1.0, np.array([0.0, -2.0]), size)
    for i in range(T):
        assert np.isclose(out[i, 0, 0], 0.5 * (i % size + 1)) and np.isclose(out[i, 1, 0], (i % size + 1) / (1 + np.exp(2.0)))
    assert np.allclose(P.sigmoid_attention(q, k, v, 1.0, np.zeros(2))[:, 0, 0], 0.5 * np.arange(1, T + 1))


def test_recurrence_against_its_unrolled_form():
    rng = np.random.default_rng(1)
    T, H, D, V = 9, 2, 3, 4
    rows, g = C.memory_inputs(rng, T, H, D, V, strength=0.5)
    o, S = C.memory_plain(rows, g, H, D, V)
    q, k, v = rows[:, :6].reshape(T, H, D) / np.sqrt(D), rows[:, 6:12].reshape(T, H, D), rows[:, 12:].reshape(T, H, V)
    G = np.cumsum(g, axis=0).reshape(T, H, D)
    for t in range(T):
        want = sum(((q[t] * k[s] * np.exp(G[t] - G[s])).sum(axis=1))[:, None] * v[s] for s in range(t + 1))
        assert np.allclose(o[t], want)
    assert np.allclose(S, sum((k[s] * np.exp(G[-1] - G[s]))[:, :, None] * v[s][:, None, :] for s in range(T)))
    o2, _ = C.memory_plain(rows[5:], g[5:], H, D, V, C.memory_plain(rows[:5], g[:5], H, D, V)[1])
    assert np.allclose(o2, o[5:])                                  # the state carries a cut
    z = np.array([-30.0, 0.0, 5.0])
    assert np.allclose(P.channel_decay(z, 1.0), 1 / (1 + np.exp(-z))) and np.allclose(P.channel_decay(z, 16.0) ** 16, 1 / (1 + np.exp(-z)))


def _tiny_weights(cfg, seed=0):
    from imparo_b200.weights.random_init import draw_random_tensors, model_on_cpu
    _, _, model = model_on_cpu(cfg)
    return {k: v.float().numpy().astype(np.float64) for k, v in draw_random_tensors(model.weight_specs(), seed, "float32", "cpu", matrix_std=0.3).items()}


def test_position_vectors_causality_and_norms_on_both_sides():
    cfg = ALL["A"]
    W = _tiny_weights(cfg)
    toks = [5, 9, 5, 100, 7, 5]
    layers = []
    base = P.forward(cfg, W, toks, layer_outputs=layers)
    assert len(layers) == len(cfg["layers"]) and np.abs(base[0] - base[2]).max() > 1e-6
    assert np.allclose(P.forward(cfg, W, toks[:4]), base[:4])
    W2 = dict(W, pos=W["pos"].copy())
    W2["pos"][4:] += 1.0
    moved = P.forward(cfg, W2, toks)
    assert np.array_equal(moved[:4], base[:4]) and np.abs(moved[4] - base[4]).max() > 1e-6
    # a sublayer's output enters by its direction only: scaling the mixer's output matrix changes (nearly) nothing
    W3 = dict(W, **{"l0.mix.o": W["l0.mix.o"] * 1e3, "l1.mix.o": W["l1.mix.o"] * 1e3})
    W4 = dict(W, **{"l0.mix.o": W["l0.mix.o"] * 1e6, "l1.mix.o": W["l1.mix.o"] * 1e6})
    assert np.abs(P.forward(cfg, W3, toks) - P.forward(cfg, W4, toks)).max() < 1e-4


@pytest.mark.parametrize("rot", [32, 12, 0])
def test_far_key_case_is_decided_by_the_far_key(rot):
    m, rows, qn, kn, pb, seekers, v_far, want = C.far_key_case(15, 1, rot=rot)
    w = want.reshape(len(want), 2, 2, -1)                            # [T, key head, heads per key head, V]
    for t in seekers:
        assert np.abs(w[t] - v_far[:, None, :]).max() < 0.15
    assert np.abs(w[301] - v_far[:, None, :]).max() > 2.0


@pytest.mark.parametrize("size", [5, 16, 17, 64])
def test_chunk_edge_case_counts_the_marks_that_are_seen(size):
    m, rows, qn, kn, pb, places, want = C.chunk_edge_case(size, 32, 16, 3)
    assert any(p % size == 0 for p in places) and any(p % size == size - 1 for p in places)
    for p, marks in places.items():
        assert np.abs(want[p] - 5.0 * marks).max() < 0.3


def test_far_memory_case_is_read_back():
    _, _, _, seekers, want = C.far_memory_case()
    assert all(abs(want[t, 0, 0] - 5.0) < 1e-6 for t in seekers) and abs(want[150, 0, 0] - 5.0) > 0.5


# ---- the host side ---------------------------------------------------------------------------------------------------

def test_configuration_reads_every_size_and_names_what_is_wrong():
    from imparo_b200.config import ConfigError, load_config
    arch, cfg = load_config(ALL["A"])
    assert arch.name == "Modinex" and cfg.width == 72 and cfg.groups == 3 and cfg.max_positions == 700 and cfg.eps == 1e-5
    a = cfg.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.rot_dims, a.rot_base, a.scale) == (6, 2, 12, 20, 9, 8, 300.0, 0.35)
    g = cfg.layers[3].mixer
    assert (g.heads, g.dim, g.vdim, g.tau) == (2, 20, 12, 1.0) and cfg.layers[3].mlp.ff == 30 and cfg.layers[1].mlp is None
    b = load_config(ALL["B"])[1]
    assert b.groups == 1 and b.layers[1].mixer.kv_heads == 3 and b.layers[1].mixer.vdim == 24 and b.layers[1].mixer.rot_dims == 0
    assert b.layers[3].mixer.chunk is None

    def broken(change):
        import copy
        c = copy.deepcopy(ALL["A"])
        change(c)
        return c
    for change, word in ((lambda c: c["layers"][0].update(type="conv"), "unknown type"),
                         (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
                         (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "dims"),
                         (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
                         (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
                         (lambda c: c["layers"][1]["mixer"].update(tau=0.0), "tau"),
                         (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown kind"),
                         (lambda c: c["norm"].update(groups=5), "groups"),
                         (lambda c: c.pop("norm"), "norm")):
        with pytest.raises(ConfigError, match=word):
            load_config(broken(change))


def test_tensors_schedule_and_cache_needs():
    from imparo_b200.models.modinex import modinex_model_spec
    from imparo_b200.config import load_config
    from imparo_b200.parts.spec import PagedKV, SlotState
    from imparo_b200.weights.random_init import model_on_cpu
    _, _, model = model_on_cpu(ALL["A"])
    names = {w.name: w.shapes[0] for w in model.weight_specs()}
    assert names["pos"] == (700, 72) and names["embed"] == (211, 72) and names["head"] == (211, 72) and names["final.norm"] == (72,)
    assert names["l0.mix.q"] == (72, 72) and names["l0.mix.k"] == (24, 72) and names["l0.mix.v"] == (40, 72) and names["l0.mix.o"] == (72, 120)
    assert names["l0.mix.q.norm"] == (12,) and names["l0.mix.pb"] == (6,) and names["l0.mlp.up.b"] == (40,) and names["l0.mlp.down"] == (72, 40)
    assert names["l1.mix.a1"] == (5, 72) and names["l1.mix.a2"] == (24, 5) and names["l1.mix.a2.b"] == (24,) and names["l1.mix.norm"] == (24,)
    assert all(f"l0.{n}" in names for n in ("norm1", "norm1b", "norm2", "norm2b")) and "l1.norm2" not in names and "l1.norm2b" not in names
    needs = dict(model.cache_requirements())
    assert needs[0] == (PagedKV(2, 12, None, 20, chunk=9),) and needs[1] == (SlotState((3, 8, 24)),)
    assert needs[2] == (PagedKV(1, 16, None, None, chunk=21),)
    # sizes that only a stored tensor gives: its shape wins over anything else
    spec = modinex_model_spec(load_config(ALL["A"])[1], tensor_shapes={"pos": (555, 72), "l1.mix.a1": (11, 72)})
    assert spec.max_positions == 555 and spec.layers[1].mixer.params["decay_rank"] == 11 and spec.layers[3].mixer.params["decay_rank"] == 12


def test_stretches_go_back_when_the_next_position_cannot_see_them():
    from imparo_b200.cache import CacheManager
    from imparo_b200.parts.spec import PagedKV
    full, chunked = PagedKV(1, 8), PagedKV(1, 8, chunk=10)
    cm = CacheManager([(0, (full,)), (1, (chunked,))], page_size=4, num_pages=16, num_slots=2, device=None)
    cm.add(7)
    cached = 0
    for n in (3, 9, 1, 7, 2, 11, 1, 1):
        cm.reserve(7, n)
        first = cached // 10 * 10 // 4                       # pages the step's own rows may read are there while it runs
        assert all(cm.table(7, 1)[b] >= 0 for b in range(first, (cached + n - 1) // 4 + 1))
        cm.commit(7, n)
        cached += n
        keep = cached // 10 * 10 // 4                        # the first page the next position can see
        table = cm.table(7, 1)
        assert all(table[b] < 0 for b in range(min(keep, len(table)))) and all(table[b] >= 0 for b in range(keep, len(table)))
        assert cm.blocks_in_use(7, 0) == -(-cached // 4)
        cm.check()
    cm.release(7)
    assert cm.free_pages(1) == 16
