"""Made-up inputs for single Zinunex mechanisms in which one far or edge element decides the output, with what the plain
implementation says about them.  Random weights and inputs would hide a lost far key, a window that is one position off, a
rotation that pairs the wrong dimensions or a sink that is left out among hundreds of ordinary terms; here one score stands
out by construction.  The builders run on the CPU (tests/test_zinunex_plain.py checks what they claim); the GPU tests feed the
same inputs to the kernels."""
import numpy as np

from tests.plain import zinunex_plain as P

SCALING = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}


def latent_rows_plain(m, eps, proj, W, queries=None):
    """The plain latent attention fed with rows that already are the product [q | latent | key part].  queries: rows [q] of
    another layer that reads these latents (m then holds that layer's sizes)."""
    D, R, C = m["dim"], m["rot_dim"], m["kv_rank"]
    T = len(proj)
    a = proj.shape[1] - C - R
    positions = np.arange(T)
    eye = np.eye(C + R)
    c, kr = P.latent_of(proj[:, a:], {"dkv": eye, "dkv.norm": W["dkv.norm"]}, "", m, eps, positions)
    q = proj[:, :a] if queries is None else queries
    Wp = {"q": np.eye(m["heads"] * (D + R)), "uk": W["uk"], "uv": W["uv"], "o": np.eye(m["heads"] * m["vdim"])}
    return P.latent_attention(q, Wp, "", m, positions, c, kr)


def far_latent_case(far, seed, T=620, prompt=600, C=16, R=8, H=2, through="latent", window=None):
    """One position `far` stands out for the queries that look for it, through the latent part of the score (its latent
    points along `direction`, every other latent is orthogonal to it) or through the rotated part (only it and the seeking
    queries carry a rotated part at all; the seekers' is the far key's before rotation, turned by their distance, so that it
    lines up with the far key's after both are rotated).  Without a window every seeker returns the far position's value; with
    one only those at most window - 1 positions behind it (`seen`).
    -> (m, W, proj rows [T, q | latent | key part], seen, unseen, v_far [heads, vdim], want [T, heads * vdim])"""
    rng = np.random.default_rng(seed)
    D, V = C, 8
    m = {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": C, "scale": 8.0 / C, "rot": {"base": 100.0, "dims": R, "scaling": SCALING}}
    if window is not None:
        m["mask"] = {"size": window}
    W = {"uk": np.concatenate([np.eye(D, C)] * H) * 1.5, "uv": rng.standard_normal((H * V, C)) / np.sqrt(C), "dkv.norm": np.ones(C)}
    direction = rng.standard_normal(C)
    direction /= np.sqrt(np.mean(direction ** 2))
    a = H * (D + R)
    proj = rng.standard_normal((T, a + C + R))
    lat = proj[:, a:a + C]
    lat -= np.outer(lat @ direction, direction) / (direction @ direction)
    proj[:, a + C:] = 0.0                                        # no rotated key part ...
    q = proj[:, :a].reshape(T, H, D + R)
    q[:, :, D:] = 0.0                                            # ... and no rotated query part, but for the marked ones
    places = {far + 1, 300, prompt - 1, prompt, T - 1}
    if window is not None:
        places |= {far + window - 1, far + window, far + window // 2}
    seekers = sorted(t for t in places if far < t < T)
    freq, mag = P.blended_frequencies(100.0, R, SCALING)
    if through == "latent":
        proj[far, a:a + C] = direction * 3.0
        for t in seekers:
            q[t, :, :D] = direction * 0.3 / 1.5 * 4.0
    else:
        key = rng.standard_normal(R)
        key *= 3.0 / np.sqrt(np.mean(key ** 2))
        proj[far, a + C:] = key
        for t in seekers:
            # turned by far - t before the rotation by t: both parts end at the angle of position far
            q[t, :, D:] = P.turn_neighbours(np.repeat(key[None, None, :], H, axis=1), [far - t], freq)[0]
            q[t, :, :D] = 0.0
    proj[:, :a] = q.reshape(T, a)
    want = latent_rows_plain(m, 1e-5, proj, W)
    c_far = P.unit_rms(proj[far, a:a + C][None], 1e-5)[0]
    v_far = (W["uv"] @ c_far).reshape(H, V)
    seen = [t for t in seekers if window is None or t - far < window]
    return m, W, proj, seen, [t for t in seekers if t not in seen], v_far, want


def attention_rows_plain(m, rows, sink):
    """The plain attention fed with rows that already are the products [q | k]."""
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    eye = np.eye(rows.shape[1])
    W = {"q": eye[:H * D], "k": eye[H * D:H * D + G * D], "sink": np.asarray(sink, dtype=rows.dtype), "o": np.eye(H * D)}
    return P.sink_attention(rows, W, "", m, np.arange(len(rows)))


def far_key_case(far, hd, seed, H=2, G=1, T=620, prompt=600, n_rot=None):
    """Keys are values, so the far key is what the seekers return: the key at `far` is large, every other key is orthogonal to
    it in each rotated pair's span at equal length (here: small), and the seekers' queries are that key turned by their
    distance, so that only the right rotation (frequencies divided by the factor) lines them up.  Sinks are far below.
    -> (m, rows [T, q | k], sink, seekers, v_far [hd], want [T, heads * hd])"""
    rng = np.random.default_rng(seed)
    n_rot = hd if n_rot is None else n_rot
    m = {"heads": H, "kv_heads": G, "dim": hd, "vdim": hd, "scale": 12.0 / hd, "rot": {"base": 1000.0, "dims": n_rot, "scaling": {"factor": 3.0}}}
    rows = rng.standard_normal((T, (H + G) * hd)) * 0.3
    key = rng.standard_normal(hd)
    key *= 2.0 / np.sqrt(np.mean(key ** 2))
    k = rows[:, H * hd:].reshape(T, G, hd)
    k[far] = key
    rows[:, H * hd:] = k.reshape(T, G * hd)
    freq = P.plain_frequencies(1000.0, n_rot) / 3.0
    seekers = sorted({t for t in (far + 1, 300, prompt - 1, prompt, T - 1) if t > far})
    q = rows[:, :H * hd].reshape(T, H, hd)
    for t in seekers:
        q[t] = P.turn_halves(np.repeat(key[None, None, :], H, axis=1), [far - t], freq)[0]
    rows[:, :H * hd] = q.reshape(T, H * hd)
    sink = np.full(H, -3.0)
    return m, rows, sink, seekers, key, attention_rows_plain(m, rows, sink)


def sink_case(hd, seed, H=4, G=2, T=150, n_rot=None):
    """Sinks as strong as all the keys together: with scores near zero a query at position i has i + 1 keys of weight about one,
    and the sinks' exponentials are those of 0, 3, 5 and a negative number, so that the first tokens are cut to small fractions.
    -> (m, rows, sink, want)"""
    rng = np.random.default_rng(seed)
    m = {"heads": H, "kv_heads": G, "dim": hd, "vdim": hd, "scale": 0.2 / hd, "rot": {"base": 100.0, "dims": hd if n_rot is None else n_rot}}
    rows = rng.standard_normal((T, (H + G) * hd)) + 1.0
    sink = np.resize([0.0, 3.0, 5.0, -2.0], H)
    return m, rows, sink, attention_rows_plain(m, rows, sink)
