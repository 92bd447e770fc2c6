"""Gated linear attention with a decay per key channel and token, as a part (mixer "gated_linear_attention").

With q = W_q h * dim^(-1/2), k = W_k h (heads x dim) and v = W_v h (heads x vdim), every head keeps a matrix S [dim, vdim] per
request:  S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t,  alpha = sigmoid(W_a2 (W_a1 h) + b)^(1/tau) per head and
key channel.  Each head's o is divided by its root mean square over vdim, times a weight [vdim] shared by the heads; the heads
side by side are multiplied by silu(W_g h) and projected by W_o.  The state starts at zero for a new request, is 32-bit and
lives in the request's state slot; decays, their logarithms, the recurrence and the norm are 32-bit in both precisions.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Part
from .spec import SlotState, WeightSpec


class GatedLinearAttention(Part):
    """params: hidden, heads, dim, vdim, tau, decay_rank (inner size of the decay's two-step projection), eps (of the per-head
    output norm), names (optional dict of tensor names after the prefix: q, k, v, g, o, norm, a1, a2, a2_bias).

    forward(..., accumulate=False) overwrites `residual` (then any float32 [tokens, hidden] buffer)."""
    adds_with_linear = True
    CHUNK_FROM = 128          # portions from this many tokens on (rounded up to a power of two) run in chunks

    NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm", "a1": "a1", "a2": "a2", "a2_bias": "a2.b"}

    def __init__(self, params, prefix, rt):
        super().__init__(params, prefix, rt)
        p = params
        self.hidden = int(p["hidden"])
        self.heads = int(p["heads"])
        self.dim = int(p["dim"])
        self.vdim = int(p["vdim"])
        self.tau = float(p["tau"])
        self.rank = int(p["decay_rank"])
        self.eps = float(p["eps"])
        if not 1 <= self.dim <= 256:
            raise ValueError(f"gated linear attention: key size {self.dim} is not supported by the kernel (1 to 256)")
        if not 1 <= self.rank <= 1024:
            raise ValueError(f"gated linear attention: decay rank {self.rank} is not supported by the kernel (1 to 1024)")
        if not self.tau > 0.0:
            raise ValueError("gated linear attention: tau must be positive")
        self.qk = self.heads * self.dim
        self.vv = self.heads * self.vdim
        self.names = {k: prefix + v for k, v in {**self.NAMES, **p.get("names", {})}.items()}
        self.w_in = self.w_a2 = self.b_a2 = self.w_o = self.w_norm = None

    def weight_specs(self):
        n, H = self.names, self.hidden
        return [WeightSpec(n["q"], ((self.qk, H),)), WeightSpec(n["k"], ((self.qk, H),)), WeightSpec(n["v"], ((self.vv, H),)),
                WeightSpec(n["g"], ((self.vv, H),)), WeightSpec(n["o"], ((H, self.vv),)),
                WeightSpec(n["norm"], ((self.vdim,),), role="vector", init=("norm",)),
                WeightSpec(n["a1"], ((self.rank, H),)), WeightSpec(n["a2"], ((self.qk, self.rank),)),
                WeightSpec(n["a2_bias"], ((self.qk,),), role="vector", init=("uniform", 0.0, 4.0))]

    def bind(self, tensors):
        n = self.names
        # one fused projection [q | k | v | g | a1], every stretch starting at a multiple of 8 columns: a layout choice
        at, parts = 0, []
        for key in ("q", "k", "v", "g", "a1"):
            at = (at + 7) // 8 * 8
            parts.append((at, tensors[n[key]]))
            at += tensors[n[key]].shape[0]
        first = parts[0][1]
        self.w_in = torch.zeros(((at + 7) // 8 * 8, first.shape[1]), dtype=first.dtype, device=first.device)
        for a, w in parts:
            self.w_in[a:a + w.shape[0]] = w
        self.columns = tuple(a for a, _ in parts)
        self.w_a2, self.b_a2 = tensors[n["a2"]], tensors[n["a2_bias"]]
        self.w_o = tensors[n["o"]]
        self.w_norm = tensors[n["norm"]]

    def cache_specs(self):
        return (SlotState((self.heads, self.dim, self.vdim)),)

    def forward(self, x, batch, caches, residual, accumulate=True):
        st = caches[0]
        rt, T = self.rt, x.shape[0]
        ws = rt.workspace
        H, D, V = self.heads, self.dim, self.vdim
        proj = ws.get("gla_in", (T, self.w_in.shape[0]), rt.act_dtype, first="tokens")
        ops.linear(x, self.w_in, proj, status=rt.status)
        q_at, k_at, v_at, g_at, a_at = self.columns
        q_scale = float(D) ** -0.5
        y = ws.get("gla_y", (T, self.vv), rt.act_dtype, first="tokens")
        # one row per request: decay, recurrence, norm and gate are one kernel
        done = batch.decode_only and ops.gla_step(proj, self.columns, self.rank, self.w_a2, self.b_a2, self.tau, self.w_norm, self.eps,
                                                  q_scale, st.state, batch.item_row_start, batch.item_slot, batch.n_items, y, H, D, V,
                                                  rt.status)
        if not done:
            g = ws.get("gla_decay", (T, self.qk), torch.float32, first="tokens")
            in_chunks = batch.max_tokens_per_item >= self.CHUNK_FROM and ops.gla_chunked_takes(proj, self.columns, D, V)
            decay = None
            if in_chunks and self.rank <= ops.GLA_CHUNK_RANK:
                decay = (self.w_a2, self.b_a2, self.tau, self.rank)
            else:
                ops.gla_decay(proj[:, a_at:a_at + self.rank], self.w_a2, self.b_a2, self.tau, g)
            o = None
            if not in_chunks or V > ops.GLA_CHUNK_COLUMNS:
                o = ws.get("gla_o", (T, self.vv), torch.float32, first="tokens")
            if in_chunks:
                chunks = T // ops.GLA_CHUNK + batch.n_items
                done = ops.gla_chunked(proj, self.columns, g, q_scale, self.w_norm, self.eps, st.state, batch.item_row_start,
                                       batch.item_slot, batch.n_items, ws.get("gla_chunk_state", (chunks * H * D * V,), torch.float32),
                                       ws.get("gla_chunk_decay", (chunks * H * D,), torch.float32), o, y, H, D, V, rt.status,
                                       decay=decay)
            else:
                ops.gla_scan(proj, q_at, k_at, v_at, g, q_scale, st.state, batch.item_row_start, batch.item_slot, batch.n_items, o, H, D,
                             V, rt.status)
            if not done:
                ops.head_norm_gate(o, self.w_norm, self.eps, proj[:, g_at:g_at + self.vv], y, H, V, act="silu")
        ops.linear(y, self.w_o, residual, accumulate=accumulate, status=rt.status)
