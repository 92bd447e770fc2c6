"""Made-up inputs for single Modinex mechanisms in which one far or edge element decides the output, with what the plain
implementation says about them.  Random weights and inputs would hide a lost far key, a stretch that starts one position off
or a state that was not carried among hundreds of ordinary terms; here one score stands out by construction.  The builders
run on the CPU (tests/test_modinex_plain.py checks what they claim); the GPU tests feed the same inputs to the kernels."""
import numpy as np

from tests.plain import modinex_plain as P


def attention_rows_plain(m, eps, rows, q_norm, k_norm, pb, first=0):
    """The plain attention fed with rows that already are the product [q | k | v]; `first`: the position of the first row."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    eye = np.eye(rows.shape[1])
    a, b, c = H * D, H * D + G * D, H * D + G * (D + V)
    W = {"q": eye[:a], "k": eye[a:b], "v": eye[b:c], "q.norm": q_norm, "k.norm": k_norm, "pb": pb, "o": np.eye(H * V)}
    return P.attention(rows, W, "", m, eps, np.arange(first, first + len(rows)))


def _marked(rng, T, H, G, D, V, rot, base, score, bias):
    """Ordinary rows [q | k | v] whose keys are orthogonal to a direction (per key head the same), with no rotation-dependent
    part of it: the direction lies in the unrotated dimensions where there are any; otherwise queries are turned to meet it."""
    rows = rng.standard_normal((T, H * D + G * (D + V)))
    direction = rng.standard_normal(D)
    if rot < D:
        direction[:rot] = 0.0
    direction /= np.sqrt(np.mean(direction ** 2))
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": score / D}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
    k = rows[:, H * D:H * D + G * D].reshape(T, G, D)
    turned = P.rotate_half_pairs(k, np.arange(T), base, rot)                     # ordinary keys as cached: no part along the direction
    turned -= (turned @ direction)[..., None] * direction / (direction @ direction)
    rows[:, H * D:H * D + G * D] = P.rotate_half_pairs(turned, -np.arange(T), base, rot).reshape(T, G * D)
    return m, rows, direction, np.full(H, bias)


def _point(rows, m, t, direction, at, what):
    """Row t's queries (or keys) such that after the rotation by t they lie along `direction` (as a key at position `at` would
    after its own rotation, when `at` is given)."""
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    rot, base = (m["rot"]["dims"], m["rot"]["base"]) if m.get("rot") else (0, 1.0)
    n, off = (H, 0) if what == "q" else (G, H * D)
    vec = P.rotate_half_pairs(np.tile(direction, (1, n, 1)) * 2.0, [-t], base, rot)
    rows[t, off:off + n * D] = vec.reshape(-1)


def far_key_case(far, seed, T=620, prompt=600, H=4, G=2, D=32, V=32, rot=32):
    """The key at position `far` lies, as cached, along a direction to which every other key is orthogonal; the seeking queries
    lie along it too and weigh it with sigmoid(18 - 9), every other key with about sigmoid(-9): they return its value.
    -> (m, rows [T, q | k | v], q_norm, k_norm, pb, seekers, v_far [G, V], want [T, H * V])"""
    rng = np.random.default_rng(seed)
    m, rows, direction, pb = _marked(rng, T, H, G, D, V, rot, 300.0, 18.0, -9.0)
    v_far = np.tile(np.linspace(3.0, 5.0, V), (G, 1))
    _point(rows, m, far, direction, None, "k")
    rows[far, H * D + G * D:] = v_far.reshape(-1)
    seekers = [t for t in (far + 1, 300, prompt - 1, prompt, T - 1) if t > far]
    for t in seekers:
        _point(rows, m, t, direction, None, "q")
    one = np.ones(D)
    return m, rows, one, one, pb, seekers, v_far, attention_rows_plain(m, 1e-5, rows, one, one, pb)


def chunk_edge_case(size, D, V, seed, T=260, H=4, G=1):
    """Stretches of `size` positions: in each the first and the last key are marked (along the direction, value 5).  The last
    query of a stretch sees both of its own, the first query of the next one sees its own mark only, and the queries in between
    look for marks too; a mark of another stretch that is seen (or one of the own stretch that is lost) moves the output by 5.
    -> (m, rows, q_norm, k_norm, pb, places, want): places = {position: marks it sees}"""
    rng = np.random.default_rng(seed)
    m, rows, direction, pb = _marked(rng, T, H, G, D, V, min(D, 16) // 2 * 2, 100.0, 18.0, -9.0)
    m["mask"] = {"size": size}
    marks = sorted({p for c in range(0, T, size) for p in (c, c + size - 1) if p < T})
    for p in marks:
        _point(rows, m, p, direction, None, "k")
        rows[p, H * D + G * D:] = 5.0
    places = {}
    for p in range(T):
        if p % size in (0, 1, size // 2, size - 1):
            _point(rows, m, p, direction, None, "q")
            places[p] = sum(1 for x in marks if p // size * size <= x <= p)
    one = np.ones(D)
    return m, rows, one, one, pb, places, attention_rows_plain(m, 1e-5, rows, one, one, pb)


def memory_inputs(rng, T, H, D, V, strength=0.05):
    """Rows [q | k | v] of the recurrence and log decays [T, H * D] (about -strength each)."""
    rows = rng.standard_normal((T, 2 * H * D + H * V))
    g = -strength * rng.uniform(0.2, 2.0, (T, H * D))
    return rows, g


def memory_plain(rows, g, H, D, V, state=None):
    """The plain recurrence on rows that already are the projections.  -> (o [T, H, V], S [H, D, V])"""
    T = len(rows)
    q = rows[:, :H * D].reshape(T, H, D) * D ** -0.5
    k = rows[:, H * D:2 * H * D].reshape(T, H, D)
    v = rows[:, 2 * H * D:].reshape(T, H, V)
    return P.decayed_memory(q, k, v, np.exp(g).reshape(T, H, D), state)


def far_memory_case(seed=3, T=420, prompt=400, H=2, D=64, V=16):
    """One key channel of head 0 never decays and only the first token writes to it: queries on that channel read its value
    back hundreds of tokens later, while every other channel forgets.
    -> ((H, D, V), rows, g, seekers, want [T, H, V])"""
    rng = np.random.default_rng(seed)
    rows, g = memory_inputs(rng, T, H, D, V, strength=0.3)
    ch = 17
    rows[:, H * D + ch] = 0.0
    g[:, ch] = 0.0
    rows[0, H * D + ch] = 2.0
    rows[0, 2 * H * D:2 * H * D + V] = 5.0
    seekers = [1, 200, prompt - 1, prompt, T - 1]
    for t in seekers:
        rows[t, :D] = 0.0
        rows[t, ch] = 0.5 * D ** 0.5
    want, _ = memory_plain(rows, g, H, D, V)
    return (H, D, V), rows, g, seekers, want
