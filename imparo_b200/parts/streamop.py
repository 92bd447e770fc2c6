"""Parts that work on the residual stream between layers (kind "stream_op"): a schedule entry may name
one that runs right before it (ScheduleEntry.before), a layer of the pre-norm arrangement one behind its sublayers
(LayerSpec.params["after"]).

StretchEntry: what a repeated stretch of layers gets at the start of each of its passes: a learned vector
of that pass, row `index` of a [passes, width] tensor, and — from the second pass on — the tokens' embedding
rows once more (the embedding's output is the plain table row, so it is gathered again, not kept).

TokenSideInput: a layer's own input from the token: g = gelu_tanh(G x) * e with e the layer's columns of the token's row of a
side table, y = P g, x += y / rms(y) * weight."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Part
from .spec import WeightSpec


class StretchEntry(Part):
    """params: width, passes, index (which pass), vector (tensor name [passes, width], or None),
    embedding (tensor name of the token table to add again, or None), vocab."""

    def __init__(self, params, prefix, rt):
        super().__init__(params, prefix, rt)
        self.width = int(params["width"])
        self.passes = int(params["passes"])
        self.index = int(params["index"])
        self.vector_name = params.get("vector")
        self.embedding_name = params.get("embedding")
        self.vocab = int(params.get("vocab", 0))
        if not 0 <= self.index < self.passes:
            raise ValueError(f"stretch entry: pass {self.index} of {self.passes}")
        self.vec = self.table = None

    def weight_specs(self):
        specs = []
        if self.vector_name:
            specs.append(WeightSpec(self.vector_name, ((self.passes, self.width),), role="vector", init=("normal", 0.02)))
        if self.embedding_name:
            specs.append(WeightSpec(self.embedding_name, ((self.vocab, self.width),)))
        return specs

    def bind(self, tensors):
        if self.vector_name:
            self.vec = tensors[self.vector_name][self.index].contiguous()
        if self.embedding_name:
            self.table = tensors[self.embedding_name]

    def forward(self, x, batch):
        ops.stream_inject(x, self.table, batch.token_ids if self.table is not None else None, self.vec, self.rt.status)


class TokenSideInput(Part):
    """params: width, dim, index (which stretch of dim columns of the table's rows), columns (of the table), vocab, eps, table
    (the table's tensor name, without the layer's prefix), names (optional: gate [dim, width], proj [width, dim], norm [width],
    after the prefix).

    forward(x, batch, rows=None, copy=None): x the float32 stream, rows (int32) which of the step's tokens its rows are, copy
    the stream in the activation dtype when the caller has it (wants_copy(rows) says whether it would be read).  The normed add
    is left to the next reader of the stream."""
    reads_copy = True
    NAMES = {"gate": "side.gate", "proj": "side.proj", "norm": "side.norm"}

    def __init__(self, params, prefix, rt):
        super().__init__(params, prefix, rt)
        self.width, self.dim = int(params["width"]), int(params["dim"])
        self.vocab, self.columns = int(params["vocab"]), int(params["columns"])
        self.col0 = int(params["index"]) * self.dim
        if not 0 <= self.col0 <= self.columns - self.dim:
            raise ValueError(f"token side input: stretch {params['index']} of {self.dim} columns is not in a table of {self.columns}")
        self.eps = float(params["eps"])
        self.table_name = params["table"]
        self.names = {k: prefix + v for k, v in {**self.NAMES, **params.get("names", {})}.items()}
        self.table = self.w_gate = self.w_proj = self.w_norm = None

    def weight_specs(self):
        n = self.names
        return [WeightSpec(self.table_name, ((self.vocab, self.columns),)), WeightSpec(n["gate"], ((self.dim, self.width),)),
                WeightSpec(n["proj"], ((self.width, self.dim),)), WeightSpec(n["norm"], ((self.width,),), role="vector", init=("norm",))]

    def bind(self, tensors):
        n = self.names
        self.table, self.w_gate, self.w_proj, self.w_norm = tensors[self.table_name], tensors[n["gate"]], tensors[n["proj"]], tensors[n["norm"]]

    def wants_copy(self, n_rows: int) -> bool:
        return self.rt.act_dtype != torch.float32 and n_rows > ops.SIDE_GATE_ROWS

    def forward(self, x, batch, rows=None, copy=None):
        rt, n = self.rt, x.shape[0]
        ws = rt.workspace
        first = "tokens" if rows is None else "rows"
        g = ws.get("side_g", (n, self.dim), rt.act_dtype, first=first)

        def tmp(what):
            if what == "copy":
                return ws.get("stream_copy", (n, self.width), rt.act_dtype, first=first)
            return ws.get("side_z", (n, self.dim), torch.float32, first=first)
        ops.token_side_gate(x, self.w_gate, self.table, self.col0, batch.token_ids, g, rt.status, rows=rows, copy=copy, tmp=tmp)
        y = ws.get("side_y", (n, self.width), torch.float32, first=first)
        ops.allow_unfinished(y)
        try:
            ops.linear(g, self.w_proj, y, status=rt.status)
        finally:
            ops.disallow_unfinished(y)
        ops.group_norm_add(x, y, self.w_norm, self.eps, 1, defer=True)
