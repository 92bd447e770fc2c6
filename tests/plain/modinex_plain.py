"""Plain Modinex forward: whole sequences, no cache, one function per mechanism.

Written from the design's equations alone; it shares no code with the engine (own config
reading, plain numpy arithmetic, a loop per token where the engine has kernels).  All
arithmetic runs in the numpy dtype given (float64 by default: a ground truth for judging
rounding).

The design in this file's notation (one sequence of T tokens at positions 0..T-1, width W; grms: the row in norm.groups
equal stretches, each by its own root mean square, then times the weight):

  x = embed[tokens] + pos[positions]
  layer:  x = x + grms1b(mixer(grms1(x)));   x = x + grms2b(ff(grms2(x)))       (no ff: the second line is left out)
  mixer "attention": q = rms(W_q h) * q.norm, k = rms(W_k h) * k.norm per head, both turned by position over the first
          rot.dims dimensions (pairs (i, i + n/2), angle p * base^(-2i/n)); v = W_v h; query head j reads key head
          j // (heads / kv_heads); position i sees j <= i of its own stretch of mask.size positions (stretches counted
          from 0); a seen key weighs sigmoid(scale * q . k + pb_head), nothing is divided; heads side by side; W_o
  mixer "gla": q = W_q h * dim^-1/2, k = W_k h, v = W_v h; alpha = sigmoid(W_a2 (W_a1 h) + a2.b)^(1/tau) per head and key
          channel; S_0 = 0, S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t; rms(o) per head * norm, heads side
          by side times silu(W_g h); W_o
  ff "dense": W_down gelu_tanh(W_up h + b) + b
  logits = head grms_final(x)
"""
from __future__ import annotations

import numpy as np


# ----------------------------------------------------------------------------
# small pieces
# ----------------------------------------------------------------------------

def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def group_rms(x, groups, eps):
    """The last axis in `groups` equal stretches, each divided by its own root mean square."""
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return unit_rms(parts, eps).reshape(x.shape)


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rotate_half_pairs(x, positions, base, n):
    """x [T, ..., D]: the first n dimensions turn, dimension i with i + n/2, by the angle p * base^(-2i/n)."""
    if not n:
        return x
    half = n // 2
    f = np.asarray(base, dtype=np.float64) ** (-2.0 * np.arange(half) / n)
    a = (np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]).astype(x.dtype)
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (half,)
    c, s = np.cos(a).reshape(shape), np.sin(a).reshape(shape)
    u, v = x[..., :half], x[..., half:n]
    out = x.copy()
    out[..., :half] = u * c - v * s
    out[..., half:n] = v * c + u * s
    return out


# ----------------------------------------------------------------------------
# mixers
# ----------------------------------------------------------------------------

def chunk_start(i, size):
    """The first position that position i sees: its stretch's first (size None: all)."""
    return 0 if size is None else (i // size) * size


def sigmoid_attention(q, k, v, scale, bias, size=None):
    """q [T, H, D], k [T, G, D], v [T, G, V], bias [H].  Position i sees chunk_start(i) <= j <= i."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for i in range(T):
        lo = chunk_start(i, size)
        for h in range(H):
            s = k[lo:i + 1, h // per] @ q[i, h] * scale + bias[h]
            out[i, h] = sigmoid(s) @ v[lo:i + 1, h // per]
    return out


def attention(h, W, p, m, eps, positions):
    T = h.shape[0]
    H, D = int(m["heads"]), int(m["dim"])
    G, V = int(m.get("kv_heads", H)), int(m.get("vdim", D))
    q = unit_rms((h @ W[p + "q"].T).reshape(T, H, D), eps) * W[p + "q.norm"]
    k = unit_rms((h @ W[p + "k"].T).reshape(T, G, D), eps) * W[p + "k.norm"]
    v = (h @ W[p + "v"].T).reshape(T, G, V)
    rot = m.get("rot")
    if rot:
        q = rotate_half_pairs(q, positions, rot["base"], int(rot["dims"]))
        k = rotate_half_pairs(k, positions, rot["base"], int(rot["dims"]))
    size = int(m["mask"]["size"]) if m.get("mask") else None
    o = sigmoid_attention(q, k, v, float(m["scale"]), W[p + "pb"], size)
    return o.reshape(T, H * V) @ W[p + "o"].T


def decayed_memory(q, k, v, alpha, state=None):
    """The recurrence alone.  q, k, alpha [T, H, D], v [T, H, V].  Returns o [T, H, V] and the final S [H, D, V]."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]), q.dtype) if state is None else state.copy()
    o = np.zeros(v.shape, q.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o, S


def channel_decay(z, tau):
    """sigmoid(z)^(1/tau)."""
    return sigmoid(z) ** (1.0 / tau)


def gla(h, W, p, m, eps):
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ W[p + "q"].T).reshape(T, H, D) * h.dtype.type(D ** -0.5)
    k = (h @ W[p + "k"].T).reshape(T, H, D)
    v = (h @ W[p + "v"].T).reshape(T, H, V)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    o, _ = decayed_memory(q, k, v, channel_decay(z, float(m["tau"])).reshape(T, H, D).astype(h.dtype))
    o = (unit_rms(o, eps) * W[p + "norm"]).reshape(T, H * V)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ----------------------------------------------------------------------------
# the model
# ----------------------------------------------------------------------------

def dense_ff(h, W, p):
    return gelu_tanh(h @ W[p + "up"].T + W[p + "up.b"]) @ W[p + "down"].T + W[p + "down.b"]


def layer_output(x, W, L, p, eps, groups, positions):
    h = group_rms(x, groups, eps) * W[p + "norm1"]
    kind, m = L["type"], L["mixer"]
    if kind == "attention":
        y = attention(h, W, p + "mix.", m, eps, positions)
    elif kind == "gla":
        y = gla(h, W, p + "mix.", m, eps)
    else:
        raise ValueError(f"unknown layer type {kind!r}")
    x = x + group_rms(y, groups, eps) * W[p + "norm1b"]
    if L.get("mlp") is not None:
        h = group_rms(x, groups, eps) * W[p + "norm2"]
        x = x + group_rms(dense_ff(h, W, p + "mlp."), groups, eps) * W[p + "norm2b"]
    return x


def forward(cfg, W, tokens, dtype=np.float64, layer_outputs=None):
    """cfg: the config.json dictionary; W: name -> array; tokens: one sequence.  Returns logits [T, vocab].
    layer_outputs: a list that receives the stream after every layer."""
    W = {k: np.asarray(v, dtype=dtype) for k, v in W.items()}
    eps, groups = float(cfg["norm"]["eps"]), int(cfg["norm"].get("groups", 1))
    positions = np.arange(len(tokens))
    x = W["embed"][np.asarray(tokens)] + W["pos"][positions]
    for i, L in enumerate(cfg["layers"]):
        x = layer_output(x, W, L, f"l{i}.", eps, groups, positions)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return (group_rms(x, groups, eps) * W["final.norm"]) @ W["head"].T
