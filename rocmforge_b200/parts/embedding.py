"""Token embedding and output head."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import kernels
from ..cache.requests import StateRequest
from ..weights.spec import ParamSpec
from .base import Part
from .linear import Linear


class TokenEmbedding(Part):
    """x = E[token], no scaling (maeddesg/ROCmForge src/gpu/forward.rs:826-883); with ``scale``, x = E[token] * scale
    (formed in 32-bit on the way into the stream; a head tied to the table reads the table itself)."""

    def __init__(self, vocab: int, hidden: int, param_name: str = "weight", scale: Optional[float] = None):
        self.vocab, self.hidden, self.param_name = vocab, hidden, param_name
        self.scale = None if scale is None or float(scale) == 1.0 else float(scale)
        self.weight: Optional[torch.Tensor] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {self.param_name: ParamSpec((self.vocab, self.hidden))}

    def bind(self, params, compute_dtype):
        self.weight = params[self.param_name]

    def cuda_modules(self, compute_dtype):
        return ["elementwise"]

    def forward(self, ctx, token_ids: torch.Tensor) -> torch.Tensor:
        return kernels.embed(self.weight, token_ids, scale=self.scale)

    def forward_with(self, ctx, token_ids: torch.Tensor, positions: "LearnedPositions" = None, rounded: bool = False):
        """(x, y): x = E[token] (+ positions' vector of the token's position), and y = x in the compute dtype if
        ``rounded`` (for a first layer that reads the stream itself), else None; one kernel."""
        if self.scale is not None:
            raise NotImplementedError("a scaled embedding does not go with learned positions or a first layer that reads the stream")
        return kernels.embed_positions(self.weight, token_ids, positions.table if positions is not None else None,
                                       ctx.tok_pos if positions is not None else None,
                                       rounded=rounded and ctx.compute_dtype != torch.float32)


class LearnedPositions(Part):
    """A learned vector per position, [positions, hidden], added to the embedding (not scaled).  Sequences cannot grow
    beyond the table (the model's longest sequence is set from it)."""

    def __init__(self, positions: int, hidden: int, param_name: str = "weight"):
        self.positions, self.hidden, self.param_name = positions, hidden, param_name
        self.table: Optional[torch.Tensor] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {self.param_name: ParamSpec((self.positions, self.hidden))}

    def bind(self, params, compute_dtype):
        self.table = params[self.param_name]

    def cuda_modules(self, compute_dtype):
        return ["elementwise"]


class PairEmbedding(Part):
    """x = norm(E[token] * scale + P[row]): the row of a second table is (previous token * mul_prev + token * mul_cur) mod
    ``buckets``, and row ``buckets`` (the last one) for a sequence's first token; an RMS norm with a weight behind it.  All in
    32-bit.  ``buckets`` None: no second table.

    The previous token of a step's first token is per-sequence state.  It is kept by the parity of its position, so that a step of
    one token per sequence that runs a second time finds what the first run found (``StateRequest.repeatable``)."""

    def __init__(self, vocab: int, hidden: int, *, scale: float = 1.0, eps: float, buckets: Optional[int] = None, mul_prev: int = 0,
                 mul_cur: int = 0, names: Optional[Dict[str, str]] = None):
        """``names``: the tensors' names below the part's prefix (keys table, pairs, norm)."""
        self.vocab, self.hidden, self.scale, self.eps = vocab, hidden, float(scale), float(eps)
        self.buckets = None if buckets is None else int(buckets)
        self.mul_prev, self.mul_cur = int(mul_prev), int(mul_cur)
        self.names = {"table": "weight", "pairs": "pairs.weight", "norm": "norm.weight"}
        self.names.update(names or {})
        self.table = self.pairs = self.norm_w = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        n = self.names
        s = {n["table"]: ParamSpec((self.vocab, self.hidden)), n["norm"]: ParamSpec((self.hidden,), kind="vector", init="ones")}
        if self.buckets is not None:
            s[n["pairs"]] = ParamSpec((self.buckets + 1, self.hidden))
        return s

    def bind(self, params, compute_dtype):
        n = self.names
        self.table, self.norm_w = params[n["table"]], params[n["norm"]].contiguous()
        self.pairs = params[n["pairs"]] if self.buckets is not None else None

    def cuda_modules(self, compute_dtype):
        return ["streams"]

    def cache_request(self):
        if self.buckets is None:
            return None
        return StateRequest((("last", (2,), torch.int32),), repeatable=True)

    def forward(self, ctx, token_ids: torch.Tensor, view=None) -> torch.Tensor:
        return kernels.pair_embed(self.table, self.pairs, token_ids, ctx.tok_seq, ctx.tok_pos, ctx.seq_slot, ctx.cu_q,
                                  view["last"] if view is not None else None, scale=self.scale, mul_prev=self.mul_prev,
                                  mul_cur=self.mul_cur, buckets=self.buckets or 1, norm=(self.norm_w, self.eps))


class OutputHead(Part):
    """logits = W y in float32; with tied embeddings W is the embedding matrix itself
    (maeddesg/ROCmForge src/gpu/forward.rs:1313-1338; tie: src/gpu/weights.rs:868-886)."""

    def __init__(self, vocab: int, hidden: int, tied_to: Optional[str] = None, param_name: str = "weight",
                 softcap: Optional[float] = None, scale: Optional[float] = None):
        """``scale``: logits <- scale * logits, and ``softcap``: logits <- softcap * tanh(logits / softcap), in 32-bit."""
        self.vocab, self.hidden, self.tied_to, self.param_name = vocab, hidden, tied_to, param_name
        self.softcap = float(softcap) if softcap else None
        self.scale = None if scale is None or float(scale) == 1.0 else float(scale)
        self.linear: Optional[Linear] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {self.param_name: ParamSpec((self.vocab, self.hidden), tied_to=self.tied_to)}

    def bind(self, params, compute_dtype):
        self.linear = Linear(params[self.param_name])

    def cuda_modules(self, compute_dtype):
        return (["elementwise"] if self.softcap is not None else []) + (["streams"] if self.scale is not None else [])

    def forward(self, ctx, y: torch.Tensor) -> torch.Tensor:
        logits = self.linear(ctx, y, out_f32=True)
        if self.scale is not None:
            logits = kernels.scale_(logits, self.scale)
        return kernels.softcap_(logits, self.softcap) if self.softcap is not None else logits
