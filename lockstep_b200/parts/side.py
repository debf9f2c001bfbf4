"""Inputs a layer takes besides the residual stream: a row of the token's own for every layer.

"token_table" (category ``table``, shared by the layers: ``ModelSpec.shared``): a table [vocabulary, layers x dim] whose
row of a token holds ``dim`` elements for every layer.

"token_input" (category ``side``): with e the layer's part of the token's row and x the residual stream,
    h <- h + rms(y) gain,  y = W_proj (gelu(W_gate x) e)
(the tanh form of gelu; rms divides by the root mean square over the width).  ``table``: the name of the shared table,
``at``: the first of the layer's columns.
"""

from __future__ import annotations

import torch

from .. import kernels as K
from .base import Part, Runtime, WeightSpec, register_part


class TokenTable(Part):
    def __init__(self, vocab_size: int, columns: int, tensor: str, runtime: Runtime):
        self.vocab, self.columns, self.tensor = int(vocab_size), int(columns), str(tensor)
        self.table = None

    def weight_specs(self):
        return {self.tensor: WeightSpec((self.vocab, self.columns), "table", ("normal", 0.0, 1.0))}

    def bind(self, tensors):
        self.table = tensors[self.tensor]


class TokenInput(Part):
    graph_safe = True

    def __init__(self, hidden_size: int, dim: int, at: int, table: str, norm_eps: float, runtime: Runtime, names=None):
        self.w, self.dim, self.at, self.table = int(hidden_size), int(dim), int(at), str(table)
        self.eps, self.rt = float(norm_eps), runtime
        self.names = {"gate": "gate", "proj": "proj", "norm": "norm"}
        self.names.update(names or {})
        if self.table not in runtime.shared or self.at + self.dim > runtime.shared[self.table].columns:
            raise ValueError(f"token_input: no shared table {self.table!r} with columns {self.at} to {self.at + self.dim}")

    def weight_specs(self):
        n = self.names
        return {n["gate"]: WeightSpec((self.dim, self.w)), n["proj"]: WeightSpec((self.w, self.dim)),
                n["norm"]: WeightSpec((self.w,), "gain")}

    def bind(self, tensors):
        n = self.names
        self.w_gate, self.w_proj = tensors[n["gate"]], tensors[n["proj"]]
        self.gain = tensors[n["norm"]].to(torch.float32).reshape(1, self.w).contiguous()

    def forward(self, h: torch.Tensor, ctx) -> None:
        rt, tokens = self.rt, h.shape[0]
        table = rt.shared[self.table].table
        g = rt.rows(tokens, self.dim)
        # few tokens: the gate's product, its activation and the token's row in one kernel
        if not (rt.dtype == torch.bfloat16 and tokens <= K.FEW_TOKENS
                and K.side_gate_few(h, self.w_gate, ctx.token_ids, table, self.at, g, rt.err)):
            x = h
            if rt.dtype != torch.float32:
                x = rt.rows(tokens, self.w)
                K.rows_cast(h, x)
            z = rt.rows(tokens, self.dim, dtype=torch.float32)
            K.gemm_nt(x, self.w_gate, z, err=rt.err)
            K.side_gate(z, ctx.token_ids, table, self.at, g, rt.err)
        y = rt.rows(tokens, self.w, dtype=torch.float32)
        K.gemm_nt(g, self.w_proj, y, err=rt.err)
        K.norm_merge_add(h, y.view(1, tokens, self.w), self.gain, 1.0, None, self.eps, 0.0)


@register_part("table", "token_table")
def _build_table(spec, runtime, **_):
    return TokenTable(spec["vocab_size"], spec["columns"], spec.get("tensor", "weight"), runtime)


@register_part("side", "token_input")
def _build_input(spec, runtime, **_):
    return TokenInput(spec["hidden_size"], spec["dim"], spec["at"], spec["table"], spec["norm_eps"], runtime,
                      names=spec.get("names"))
