"""A second input of the tokens, given to every layer."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import kernels
from ..weights.spec import ParamSpec
from .base import Part
from .linear import Linear


class SideTable(Part):
    """A table [vocab, layers * dim]: a token's row holds ``dim`` numbers for each layer.  The layers' ``TokenSideInput`` parts
    read it."""

    def __init__(self, vocab: int, layers: int, dim: int, param_name: str = "weight"):
        self.vocab, self.layers, self.dim, self.param_name = vocab, layers, dim, param_name
        self.table: Optional[torch.Tensor] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {self.param_name: ParamSpec((self.vocab, self.layers * self.dim), std=1.0)}

    def bind(self, params, compute_dtype):
        self.table = params[self.param_name]


class TokenSideInput(Part):
    """x += rms(W_proj (gelu(W_gate x) * e)) * w with e the token's ``dim`` numbers for this layer (``table``, part ``index``),
    gelu by tanh, rms(y) = y / sqrt(mean(y^2) + eps).  The first product reads the stream rounded to the compute dtype, whose
    32-bit rows the block's last update leaves beside the stream; the sum and the norm are 32-bit and happen in the pass that
    also computes the norm that reads the stream next (kernels.stream_update).
    ``names``: the tensors' names below the part's prefix (keys gate, proj, norm)."""

    def __init__(self, hidden: int, table: SideTable, index: int, eps: float, names: Optional[Dict[str, str]] = None):
        if not 0 <= index < table.layers:
            raise ValueError(f"token side input: the table has {table.layers} parts, not part {index}")
        self.hidden, self.table, self.index, self.dim, self.eps = hidden, table, int(index), table.dim, float(eps)
        self.names = {"gate": "gate.weight", "proj": "proj.weight", "norm": "norm.weight"}
        self.names.update(names or {})
        self.gate: Optional[Linear] = None
        self.proj: Optional[Linear] = None
        self.norm_w = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        n = self.names
        return {n["gate"]: ParamSpec((self.dim, self.hidden)), n["proj"]: ParamSpec((self.hidden, self.dim)),
                n["norm"]: ParamSpec((self.hidden,), kind="vector", init="ones")}

    def bind(self, params, compute_dtype):
        n = self.names
        # padded to a multiple of 8 (zeros): rows of 16 bytes for the second product
        self.padded = (self.dim + 7) // 8 * 8
        gate, proj = params[n["gate"]], params[n["proj"]]
        if self.padded != self.dim:
            gate = torch.cat([gate, gate.new_zeros((self.padded - self.dim, self.hidden))], dim=0)
            proj = torch.cat([proj, proj.new_zeros((self.hidden, self.padded - self.dim))], dim=1)
        self.gate, self.proj = Linear(gate.contiguous()), Linear(proj.contiguous())
        self.norm_w = params[n["norm"]].contiguous()

    def cuda_modules(self, compute_dtype):
        return ["layernorm"]

    def addend(self, ctx, x: torch.Tensor):
        """(the update before its norm: float32 [T, H] or a stack of partial sums, (norm weight, eps)); ``x`` [T, H] is the stream
        in the compute dtype."""
        z = ctx.matmul_rows_or_parts(x, self.gate.weight)
        g = kernels.side_gate(z, self.table.table, self.index * self.dim, self.dim, ctx.tokens, self.padded)
        return self.proj.f32_parts(ctx, g), (self.norm_w, self.eps)
