"""What a layer adds to the residual stream of the token itself.

Kind ``gated_token_row``: the model has a table with a row per token of the vocabulary (``table``), of which layer i owns the
columns ``column .. column + dim - 1``.  With e the token's part of the row and x the residual stream,

    g = gelu(W_gate x) * e                   (the tanh form of gelu)
    x <- x + rms(W_proj g) * w               (rms: divided by its root mean square; w a stored weight)

The gate reads the stream itself, without a norm before it.  Its logits and the gelu are float32, the opened row is rounded once;
the norm and the sum are part of the pass over the stream that also applies the next layer's first norm.
"""

from __future__ import annotations

from typing import Dict, List

import torch

from .. import kernels as K
from ..config.spec import PartSpec
from ..weights.loader import ParamSpec
from .base import NORMS, TOKEN_INPUTS, TokenInput
from .linear import FusedLinear


@TOKEN_INPUTS.register("gated_token_row")
class GatedTokenRow(TokenInput):
    def __init__(self, spec, prefix, dtype, device):
        super().__init__(spec, prefix, dtype, device)
        self.hidden = int(spec["hidden_size"])
        self.dim = int(spec["dim"])
        self.column = int(spec["column"])
        self.table_name = str(spec["table"])
        n = dict(spec.get("names", {}))
        suffixes = tuple(spec.get("suffixes", (".weight", ".bias")))
        self.gate = FusedLinear(prefix, [n.get("gate", "gate_proj")], self.hidden, [self.dim], False, dtype, suffixes=suffixes)
        self.proj = FusedLinear(prefix, [n.get("proj", "proj")], self.dim, [self.hidden], False, dtype, suffixes=suffixes)
        self.norm = NORMS.build(PartSpec("rmsnorm", {"size": self.hidden, "eps": float(spec["eps"]), "tensor": n.get("norm", "norm.weight")}), prefix, dtype, device)
        self.table = None

    def parts(self):
        return [self.norm]

    def params(self) -> List[ParamSpec]:
        return self.gate.params() + self.proj.params()

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.gate.bind(tensors)
        self.proj.bind(tensors)

    def take_tables(self, tables: Dict[str, torch.Tensor]) -> None:
        self.table = tables[self.table_name]
        if self.column + self.dim > self.table.shape[1]:
            raise ValueError(f"{self.prefix!r}: columns {self.column} .. {self.column + self.dim} of a table of {self.table.shape[1]}")

    def post_norm(self):
        return self.norm

    def forward(self, x, ctx):
        g = torch.empty((x.shape[0], self.dim), dtype=self.dtype, device=x.device)
        if K.token_gate_accepts(x):
            # few tokens: the gate's product opens the row itself
            K.token_gate(x, self.gate.weight, self.table, self.column, ctx.token_ids, g)
            return self.proj(g)
        z = self.gate(x, out_dtype=torch.float32)
        K.gelu_token_rows(z, self.table, self.column, ctx.token_ids, g)
        return self.proj(g)
