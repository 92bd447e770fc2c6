"""Plain Zinunex forward: whole sequences, no cache, one function per mechanism.

Written from the design's equations alone; it shares no code with the engine (own config
reading, plain numpy arithmetic, a loop per token where the engine has kernels).  All
arithmetic runs in the numpy dtype given (float64 by default: a ground truth for judging
rounding).

The design in this file's notation (one sequence of T tokens at positions 0..T-1, width W):

  x = embed[tokens]
  layer i:  x = x + mixer(rms(x) * norm1);  x = x + ff(rms(x) * norm2)  (ff absent: skipped);
            e = side.embed[tokens, i * n : (i + 1) * n];  y = P (gelu_tanh(G x) * e);  x = x + rms(y) * side.norm
  mixer "latent_attention": q = W_q h, per head [dim plain | rot_dim turned]; W_dkv h = [c_raw (kv_rank) | kr (rot_dim)];
          c = rms(c_raw) * dkv.norm; per head k = W_uk c, v = W_uv c; the turned parts by position, pairs (2i, 2i + 1),
          frequencies blended between the plain and the stretched ones, sines and cosines times a magnitude;
          score = scale * (q_plain . k + q_turned . kr); keys i - size < j <= i; softmax; W_o.
          With kv_from = j: c and kr are those that layer j made.
  mixer "attention": grouped queries; q = W_q h, k = W_k h, v = k before the rotation; the first rot.dims dimensions
          turn, pairs (i, i + dims/2), frequencies divided by scaling.factor; score = scale * q . k; keys j <= i;
          p_j = exp(s_j) / (exp(sink_h) + sum exp(s)); W_o
  ff "moe": s = sigmoid(W_router h); choice scores s + correction; experts in groups.count equal groups of neighbours, a
          group's score the sum of its two largest choice scores, only the groups.keep best groups' experts are candidates;
          the `top` candidates with the largest choice scores, weighted by s * router.scale; expert: W_down relu(W_up h)^2;
          plus sigmoid(W_sg h) times the shared expert (same form)
  out:    logits = head (rms(x) * final.norm)
"""
from __future__ import annotations

import numpy as np


# ----------------------------------------------------------------------------
# small pieces
# ----------------------------------------------------------------------------

def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


# ----------------------------------------------------------------------------
# rotations
# ----------------------------------------------------------------------------

def plain_frequencies(base, n):
    return np.asarray(base, dtype=np.float64) ** (-2.0 * np.arange(n // 2) / n)


def blended_frequencies(base, n, scaling):
    """-> (frequencies [n/2], magnitude).  scaling: factor, original, fast, slow (None: plain, 1)."""
    f = plain_frequencies(base, n)
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def dim_of(turns):
        return n * np.log(original / (2.0 * np.pi * turns)) / (2.0 * np.log(base))
    lo = max(np.floor(dim_of(float(scaling["fast"]))), 0.0)
    hi = min(np.ceil(dim_of(float(scaling["slow"]))), n - 1.0)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * np.log(factor) + 1.0


def _cos_sin(x, positions, freq, magnitude):
    a = (np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]).astype(x.dtype)
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (len(freq),)
    m = x.dtype.type(magnitude)
    return (np.cos(a) * m).reshape(shape), (np.sin(a) * m).reshape(shape)


def turn_neighbours(x, positions, freq, magnitude=1.0):
    """x [T, ..., D]: dimension 2i turns with 2i + 1 by position * freq[i]; dimensions beyond 2 len(freq) pass."""
    n = 2 * len(freq)
    c, s = _cos_sin(x, positions, freq, magnitude)
    out = x.copy()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


def turn_halves(x, positions, freq):
    """x [T, ..., D]: dimension i turns with i + len(freq) by position * freq[i]; dimensions beyond 2 len(freq) pass."""
    half = len(freq)
    c, s = _cos_sin(x, positions, freq, 1.0)
    out = x.copy()
    u, v = x[..., :half], x[..., half:2 * half]
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


# ----------------------------------------------------------------------------
# mixers
# ----------------------------------------------------------------------------

def softmax_attention(q, k, v, scale, window=None, sink=None):
    """q [T, H, D], k [T, H, D], v [T, H, V] (keys already spread over the query heads): position i sees j <= i, with a
    window only i - j < window; sink [H]: one more term exp(sink_h) in the denominator."""
    T = q.shape[0]
    out = np.zeros((T, q.shape[1], v.shape[2]), dtype=q.dtype)
    for i in range(T):
        lo = 0 if window is None else max(0, i - window + 1)
        s = np.einsum("hd,jhd->hj", q[i], k[lo:i + 1]) * scale
        top = s.max(axis=1)
        if sink is not None:
            top = np.maximum(top, sink)
        e = np.exp(s - top[:, None])
        den = e.sum(axis=1)
        if sink is not None:
            den = den + np.exp(sink - top)
        out[i] = np.einsum("hj,jhv->hv", e / den[:, None], v[lo:i + 1])
    return out


def latent_of(h, W, p, m, eps, positions):
    """What a latent layer caches: (c [T, kv_rank], kr [T, rot_dim] turned)."""
    C = int(m["kv_rank"])
    down = h @ W[p + "dkv"].T
    c = unit_rms(down[:, :C], eps) * W[p + "dkv.norm"]
    kr = down[:, C:]
    rot = m.get("rot")
    if rot:
        freq, mag = blended_frequencies(float(rot["base"]), int(rot["dims"]), rot.get("scaling"))
        kr = turn_neighbours(kr, positions, freq, mag)
    return c, kr


def latent_attention(h, W, p, m, positions, c, kr):
    T = h.shape[0]
    H, D, R, V = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"])
    q = (h @ W[p + "q"].T).reshape(T, H, D + R)
    qr = q[..., D:]
    rot = m.get("rot")
    if rot:
        freq, mag = blended_frequencies(float(rot["base"]), int(rot["dims"]), rot.get("scaling"))
        qr = turn_neighbours(qr, positions, freq, mag)
    k = (c @ W[p + "uk"].T).reshape(T, H, D)
    v = (c @ W[p + "uv"].T).reshape(T, H, V)
    qf = np.concatenate([q[..., :D], qr], axis=-1)
    kf = np.concatenate([k, np.repeat(kr[:, None, :], H, axis=1)], axis=-1)
    window = int(m["mask"]["size"]) if m.get("mask") else None
    o = softmax_attention(qf, kf, v, float(m["scale"]), window)
    return o.reshape(T, H * V) @ W[p + "o"].T


def sink_attention(h, W, p, m, positions):
    T = h.shape[0]
    H, D = int(m["heads"]), int(m["dim"])
    G = int(m.get("kv_heads", H))
    q = (h @ W[p + "q"].T).reshape(T, H, D)
    k = (h @ W[p + "k"].T).reshape(T, G, D)
    v = k
    rot = m.get("rot")
    if rot:
        freq = plain_frequencies(float(rot["base"]), int(rot["dims"]))
        if rot.get("scaling"):
            freq = freq / float(rot["scaling"]["factor"])
        q, k = turn_halves(q, positions, freq), turn_halves(k, positions, freq)
    per = H // G
    k, v = np.repeat(k, per, axis=1), np.repeat(v, per, axis=1)        # query head j reads key head j // per
    o = softmax_attention(q, k, v, float(m["scale"]), sink=W[p + "sink"])
    return o.reshape(T, H * D) @ W[p + "o"].T


# ----------------------------------------------------------------------------
# feed-forward
# ----------------------------------------------------------------------------

def expert(h, W, p):
    return relu_squared(h @ W[p + "up"].T) @ W[p + "down"].T


def route(z, correction, top, groups, keep, scale, gaps=None):
    """z [T, E] router logits -> (ids [T, top], weights [T, top]).  gaps: a list that receives, per row, by how much (in
    choice scores) the closest decision was made: the last kept group against the first one left out, the last chosen
    expert against the best candidate that was not chosen."""
    T, E = z.shape
    s = sigmoid(z)
    choice = s + correction
    ids = np.zeros((T, top), dtype=np.int64)
    gap = np.full(T, np.inf)
    per = E // groups
    for t in range(T):
        cand = choice[t].copy()
        if groups > 1 and keep < groups:
            score = np.array([np.sort(cand[g * per:(g + 1) * per])[-2:].sum() for g in range(groups)])
            order = np.argsort(-score, kind="stable")
            gap[t] = score[order[keep - 1]] - score[order[keep]]
            for g in order[keep:]:
                cand[g * per:(g + 1) * per] = -np.inf
        order = np.argsort(-cand, kind="stable")
        ids[t] = order[:top]
        if top < E:
            gap[t] = min(gap[t], cand[order[top - 1]] - cand[order[top]])
    if gaps is not None:
        gaps.append(gap)
    return ids, np.take_along_axis(s, ids, axis=1) * scale


def moe_ff(h, W, p, mlp, gaps=None):
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ W[p + "router"].T
    ids, w = route(z, W[p + "correction"], int(r["top"]), int(groups["count"]), int(groups["keep"]), float(r.get("scale", 1.0)), gaps)
    out = np.zeros((h.shape[0], W[p + "e0.down"].shape[0]), dtype=h.dtype)
    for t in range(h.shape[0]):
        for j in range(ids.shape[1]):
            out[t] += w[t, j] * expert(h[t:t + 1], W, f"{p}e{int(ids[t, j])}.")[0]
    if mlp.get("shared"):
        out = out + sigmoid(h @ W[p + "shared.sg"].T) * expert(h, W, p + "shared.")
    return out


# ----------------------------------------------------------------------------
# the model
# ----------------------------------------------------------------------------

def token_side(x, e, W, p, eps):
    """The per-layer token input: e [T, n] are the layer's columns of the side table at the tokens."""
    y = (gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T
    return x + unit_rms(y, eps) * W[p + "side.norm"]


def forward(cfg, W, tokens, dtype=np.float64, layer_outputs=None, gaps=None):
    """cfg: the config.json dictionary; W: name -> array; tokens: one sequence.  Returns logits [T, vocab].
    layer_outputs: a list that receives the stream after every layer; gaps: a list that receives every routed layer's
    per-row decision gaps (route)."""
    W = {k: np.asarray(v, dtype=dtype) for k, v in W.items()}
    eps = float(cfg["norm"]["eps"])
    tokens = np.asarray(tokens)
    positions = np.arange(len(tokens))
    x = W["embed"][tokens]
    made = {}                                # layer -> (c, kr) of the latent layers that make their own
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = unit_rms(x, eps) * W[p + "norm1"]
        if L["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                made[i] = latent_of(h, W, p + "mix.", m, eps, positions)
                src = i
            y = latent_attention(h, W, p + "mix.", m, positions, *made[src])
        elif L["type"] == "attention":
            y = sink_attention(h, W, p + "mix.", m, positions)
        else:
            raise ValueError(f"unknown layer type {L['type']!r}")
        x = x + y
        if L.get("mlp"):
            x = x + moe_ff(unit_rms(x, eps) * W[p + "norm2"], W, p + "mlp.", L["mlp"], gaps)
        if cfg.get("token_side"):
            n = int(cfg["token_side"]["dim"])
            x = token_side(x, W["side.embed"][tokens, i * n:(i + 1) * n], W, p, eps)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return (unit_rms(x, eps) * W["final.norm"]) @ W["head"].T
