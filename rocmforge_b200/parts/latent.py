"""Attention whose queries, keys and values are made from narrow latents of the token."""
from __future__ import annotations

from typing import Dict, Optional

import numpy as np
import torch

from .. import kernels
from ..cache.requests import KVRequest
from ..engine.stream import ScaledRows
from ..weights.spec import ParamSpec
from .attention import GQAAttention, query_tiles
from .base import MIXERS, Mixer
from .linear import Linear


def stacked_on_boundaries(blocks, hidden):
    """The matrices ``blocks`` [n, hidden] stacked with every block's first row on a 16-byte boundary of the product's output
    rows (8 columns of bfloat16), and the columns at which they start."""
    out, cols, at = [], [], 0
    for b in blocks:
        pad = (-at) % 8
        if pad:
            out.append(b.new_zeros((pad, hidden)))
            at += pad
        cols.append(at)
        out.append(b)
        at += b.shape[0]
    if at % 8:
        out.append(blocks[0].new_zeros(((-at) % 8, hidden)))
    return torch.cat(out, dim=0).contiguous(), cols


@MIXERS.register("latent_attention")
class LatentAttention(Mixer):
    """Softmax attention without positions whose heads are expanded from two latents of the mixer's input x:

        c_q = rms(W_dq x) * w_q            (``q_rank`` numbers)        q_h = W_uq c_q       (``dim`` per head)
        c   = rms(W_dkv x) * w_kv          (``kv_rank`` numbers)       k_h = W_uk c,  v_h = W_uv c   (``dim``, ``vdim`` per head)
        score = scale q_h . k_h over the last ``window`` positions (None: all earlier ones), ordinary softmax
        out = W_o concat_h(o_h * sigmoid(W_g x)_h)                     (``gate`` "sigmoid_head"; None: no gate)

    rms(x) = x / sqrt(mean(x^2) + eps), in 32-bit.  One product makes W_dq x | W_dkv x | W_g x, one kernel norms the two
    latents, two products expand them, and from there on the mixer is grouped-query attention with as many kv heads as
    heads: the expanded keys and values of the window go into the paged cache through the per-head writer, and the
    attention kernels, the gate and the output product are those of ``gqa_attention`` (an inner part without projections
    of its own).  Caching the expanded heads rather than c costs heads * (dim + vdim) instead of kv_rank numbers a
    position; a window bounds both.
    ``names``: the tensors' names below the part's prefix (keys dq, dq_norm, uq, dkv, dkv_norm, uk, uv, g, o).
    """

    def __init__(self, hidden: int, n_heads: int, head_dim: int, v_head_dim: int, q_rank: int, kv_rank: int, eps: float, *,
                 scale: Optional[float] = None, window: Optional[int] = None, gate: Optional[str] = "sigmoid_head",
                 names: Optional[Dict[str, str]] = None):
        if gate not in (None, "sigmoid_head"):
            raise ValueError(f"latent_attention: gate {gate!r} has no kernel (sigmoid_head)")
        self.hidden, self.n_heads, self.head_dim, self.v_head_dim = hidden, n_heads, head_dim, v_head_dim
        self.q_rank, self.kv_rank, self.eps, self.gate = int(q_rank), int(kv_rank), float(eps), gate
        self.names = {"dq": "q_a_proj.weight", "dq_norm": "q_a_norm.weight", "uq": "q_b_proj.weight",
                      "dkv": "kv_a_proj.weight", "dkv_norm": "kv_a_norm.weight", "uk": "k_b_proj.weight",
                      "uv": "v_b_proj.weight", "g": "g_proj.weight", "o": "o_proj.weight"}
        self.names.update(names or {})
        # the attention over the expanded heads: masks, kernel choice and tile tables are gqa_attention's
        self.inner = GQAAttention(hidden, n_heads, n_heads, head_dim, qkv_bias=False, window=window, position=None,
                                  scale=scale, v_head_dim=v_head_dim)
        self.q_size, self.k_size, self.v_size = n_heads * head_dim, n_heads * head_dim, n_heads * v_head_dim
        self.down: Optional[Linear] = None
        self.uq: Optional[Linear] = None
        self.ukv: Optional[Linear] = None
        self.o: Optional[Linear] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        n = self.names
        s = {n["dq"]: ParamSpec((self.q_rank, self.hidden)), n["dq_norm"]: ParamSpec((self.q_rank,), kind="vector", init="ones"),
             n["uq"]: ParamSpec((self.q_size, self.q_rank)),
             n["dkv"]: ParamSpec((self.kv_rank, self.hidden)), n["dkv_norm"]: ParamSpec((self.kv_rank,), kind="vector", init="ones"),
             n["uk"]: ParamSpec((self.k_size, self.kv_rank)), n["uv"]: ParamSpec((self.v_size, self.kv_rank)),
             n["o"]: ParamSpec((self.hidden, self.v_size))}
        if self.gate is not None:
            s[n["g"]] = ParamSpec((self.n_heads, self.hidden))
        return s

    def bind(self, params, compute_dtype):
        n = self.names
        blocks = [params[n["dq"]], params[n["dkv"]]] + ([params[n["g"]]] if self.gate is not None else [])
        w, cols = stacked_on_boundaries(blocks, self.hidden)
        self.down = Linear(w)
        self.cq_col, self.c_col = cols[0], cols[1]
        self.gate_col = cols[2] if self.gate is not None else None
        self.dq_norm_w = params[n["dq_norm"]].contiguous()
        self.dkv_norm_w = params[n["dkv_norm"]].to(self.dq_norm_w.dtype).contiguous()
        self.uq = Linear(params[n["uq"]])
        self.ukv = Linear(torch.cat([params[n["uk"]], params[n["uv"]]], dim=0).contiguous())
        self.o = Linear(params[n["o"]])

    def cuda_modules(self, compute_dtype):
        return list(dict.fromkeys(["elementwise"] + self.inner.cuda_modules(compute_dtype)))

    def cache_request(self):
        return self.inner.cache_request()

    def step_table_names(self):
        return self.inner.step_table_names()

    def step_table(self, name, batch):
        return self.inner.step_table(name, batch)

    def heads_out(self, ctx, y, view):
        if isinstance(y, ScaledRows):
            y = y.materialize()
        p = self.down(ctx, y)                                                # [T, W_dq x | W_dkv x | W_g x]
        c_q, c = kernels.stretch_norm(p, [(self.cq_col, self.q_rank, self.dq_norm_w), (self.c_col, self.kv_rank, self.dkv_norm_w)],
                                      self.eps)
        q = self.uq(ctx, c_q)                                                # the queries need nothing more
        kv = self.ukv(ctx, c)                                                # [T, k heads | v heads]
        # keys and values into their pages, head by head (rows without query heads: nothing is normed or turned)
        kernels.head_norm_kv_write(kv, 0, self.n_heads, self.head_dim, self.v_head_dim, None, ctx.tok_seq, ctx.tok_pos,
                                   ctx.seq_slot, view.block_table, view.k_pages, view.v_pages, view.writes,
                                   compute_dtype=ctx.compute_dtype)
        o = self.inner.attend(ctx, q, view)
        if self.gate is not None:
            o = kernels.sigmoid_gate(o, p[:, self.gate_col:self.gate_col + self.n_heads], group=self.v_head_dim)
        return o

    def forward(self, ctx, y, cache_view, stream):
        self.o.add_to_stream(ctx, self.heads_out(ctx, y, cache_view), stream)

    def output(self, ctx, y, cache_view):
        return self.o.f32_parts(ctx, self.heads_out(ctx, y, cache_view))


@MIXERS.register("latent_cache_attention")
class LatentCacheAttention(Mixer):
    """Causal softmax attention whose cache holds, for every position, one latent and one rotated key part for all heads:

        c, r  = the first ``kv_rank`` and the last ``rot_dim`` rows of W_dkv x;  c <- rms(c) * w,  r <- turned by the position
        q_h   = [q_h', q_h''] (``head_dim`` and ``rot_dim``) of W_q x;           q_h'' <- turned by the position
        k_h   = W_uk,h c,  v_h = W_uv,h c                                        (``head_dim``, ``v_head_dim``)
        score = scale (q_h' . k_h + q_h'' . r),  ordinary softmax over all positions up to the query's
        out   = W_o (concat_h(o_h) * sigmoid(W_g x))                             (``gate`` "sigmoid"; None: no gate)

    One product makes W_q x | W_dkv x | W_g x; one kernel norms, turns and writes the cache row [c | r].  Then two forms:

    * prompts (more than ``SHORT`` new tokens in a sequence, bfloat16): the latents of the step's sequences are expanded by one
      product into k and v of all heads, and the tcgen05 prompt attention reads both where the product left them, the rotated part
      from the latents' rows (``kernels.attention_latent_prefill``; a score costs head_dim + rot_dim multiplications).  A prompt
      that continues a context gathers the context's rows from the pages first.
    * decoding and short portions: q_h' is folded into the latent's space, q_h' . W_uk,h c = (W_uk,h^T q_h') . c, so attention runs on
      the cache rows themselves as ONE key-value head whose values are the rows' first ``kv_rank`` numbers, and W_uv is applied
      to the result (``kernels.attention_latent_decode``, or the generic attention in 32-bit and for sizes it does not take).
    ``names``: the tensors' names below the part's prefix (keys q, dkv, dkv_norm, uk, uv, g, o)."""

    SHORT = 4            # new tokens of a sequence up to which a portion is worked on like single tokens
    TILE = 128           # rows of the prompt kernel's query tiles

    def __init__(self, hidden: int, n_heads: int, head_dim: int, rot_dim: int, v_head_dim: int, kv_rank: int, eps: float, *,
                 scale: float, position=None, gate: Optional[str] = None, names: Optional[Dict[str, str]] = None):
        if gate not in (None, "sigmoid"):
            raise ValueError(f"latent_cache_attention: gate {gate!r} has no kernel (sigmoid)")
        if (rot_dim > 0) != (position is not None):
            raise ValueError("latent_cache_attention: a rotated part goes with a position encoding")
        if position is not None and position.rotation()["rot_dim"] != rot_dim:
            raise ValueError("latent_cache_attention: the rotated part turns as a whole")
        self.hidden, self.n_heads, self.head_dim, self.rot_dim, self.v_head_dim = hidden, n_heads, head_dim, int(rot_dim), v_head_dim
        self.kv_rank, self.eps, self.scale, self.position, self.gate = int(kv_rank), float(eps), float(scale), position, gate
        self.names = {"q": "q_proj.weight", "dkv": "kv_a_proj.weight", "dkv_norm": "kv_a_norm.weight", "uk": "k_b_proj.weight",
                      "uv": "v_b_proj.weight", "g": "g_proj.weight", "o": "o_proj.weight"}
        self.names.update(names or {})
        self.q_size, self.k_size, self.v_size = n_heads * (head_dim + self.rot_dim), n_heads * head_dim, n_heads * v_head_dim
        self.row = (self.kv_rank + self.rot_dim + 7) // 8 * 8          # a cache row: [c | r | zeros], whole 16-byte pieces
        self.down = self.o = self.ukv = self.fold = self.unfold = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        n = self.names
        s = {n["q"]: ParamSpec((self.q_size, self.hidden)), n["dkv"]: ParamSpec((self.kv_rank + self.rot_dim, self.hidden)),
             n["dkv_norm"]: ParamSpec((self.kv_rank,), kind="vector", init="ones"),
             n["uk"]: ParamSpec((self.k_size, self.kv_rank)), n["uv"]: ParamSpec((self.v_size, self.kv_rank)),
             n["o"]: ParamSpec((self.hidden, self.v_size))}
        if self.gate is not None:
            s[n["g"]] = ParamSpec((self.v_size, self.hidden))
        return s

    def bind(self, params, compute_dtype):
        n, H = self.names, self.n_heads
        blocks = [params[n["q"]], params[n["dkv"]]] + ([params[n["g"]]] if self.gate is not None else [])
        w, cols = stacked_on_boundaries(blocks, self.hidden)
        self.down = Linear(w)
        self.down_col, self.gate_col = cols[1], cols[2] if self.gate is not None else None
        self.norm_w = params[n["dkv_norm"]].contiguous()
        uk, uv = params[n["uk"]], params[n["uv"]]
        self.fold = uk.view(H, self.head_dim, self.kv_rank).transpose(1, 2).contiguous()      # [H, rank, dim]: W_uk,h^T
        self.unfold = uv.view(H, self.v_head_dim, self.kv_rank).contiguous()                   # [H, vdim, rank]
        if compute_dtype == torch.bfloat16:
            self.ukv = Linear(torch.cat([uk, uv], dim=0).contiguous())
        self.o = Linear(params[n["o"]])
        if self.position is not None:
            self.position.prepare(w.device)

    def cuda_modules(self, compute_dtype):
        return ["latent", "attention_generic"] + (["attention_latent_prefill", "attention_latent_decode"]
                                                  if compute_dtype == torch.bfloat16 else [])

    def cache_request(self):
        return KVRequest(1, self.row, v_head_dim=self.kv_rank, values_are_keys=True)

    def step_table_names(self):
        return ("attention_tiles128", "context_rows")

    def step_table(self, name, batch):
        """The prompt kernel's query tiles; and where every sequence's positions start when all of them (the new ones included)
        lie in one matrix, sequence after sequence."""
        if name == "attention_tiles128":
            return query_tiles(batch, self.TILE)
        if batch.is_decode:
            return np.zeros((0,), dtype=np.int32)
        return np.concatenate([[0], np.cumsum(batch.starts + batch.n_new)]).astype(np.int32)

    def _expands(self, ctx) -> bool:
        return (ctx.compute_dtype == torch.bfloat16 and not ctx.is_decode and ctx.max_new > self.SHORT and ctx.host is not None
                and ctx.options.tuned_attention and ctx.options.tcgen05_attention
                and kernels.attention_latent_prefill_supported(self.n_heads, self.head_dim, self.rot_dim, self.v_head_dim, self.kv_rank))

    def heads_out(self, ctx, y, view):
        """The concatenated (gated) heads [T, heads * v_head_dim]: the output projection's input."""
        H, D, R, V, K = self.n_heads, self.head_dim, self.rot_dim, self.v_head_dim, self.kv_rank
        p = ctx.matmul_rows_or_parts(y, self.down.weight)                  # q | c, r | gate
        T, parts = p.shape[-2], p.dim() == 3
        new = dict(dtype=ctx.compute_dtype, device=p.device)
        gate = None
        if self.gate is not None:
            gate = torch.empty((T, self.v_size), **new) if parts else p[:, self.gate_col:self.gate_col + self.v_size]
        common = dict(q_col=0, down_col=self.down_col, heads=H, dim=D, rot=R, rank=K, norm_weight=self.norm_w, eps=self.eps,
                      rotation=self.position.rotation() if self.position is not None else None, tok_seq=ctx.tok_seq,
                      tok_pos=ctx.tok_pos, seq_slot=ctx.seq_slot, block_table=view.block_table, pages=view.k_pages,
                      compute_dtype=ctx.compute_dtype, gate_col=self.gate_col or 0, gate=gate if parts else None)
        if self._expands(ctx):
            fresh = not ctx.host.starts.any()                              # every sequence starts here: no context to gather
            lat = torch.empty((T, self.row), **new) if fresh else None
            q = torch.empty((T, self.q_size), **new) if parts else p[:, :self.q_size]
            heads = q.unflatten(1, (H, D + R))
            kernels.latent_write(p, rows=lat, q_dim=heads[:, :, :D] if parts else None, q_rot=heads[:, :, D:] if R else None, **common)
            cu_k = ctx.tables["context_rows"]
            if not fresh:
                lat = kernels.latent_gather(view.k_pages, cu_k, ctx.seq_slot, view.block_table,
                                            int((ctx.host.starts + ctx.host.n_new).sum()))
            kv = ctx.matmul(lat[:, :K], self.ukv.weight)                   # [keys, k of all heads | v of all heads]
            return kernels.attention_latent_prefill(q, kv, lat, ctx.tables["attention_tiles128"], ctx.seq_start, ctx.seq_nnew,
                                                    ctx.cu_q, cu_k, heads=H, dim=D, rot=R, vdim=V, rank=K, scale=self.scale, gate=gate)
        folded = torch.empty((T, H, self.row), **new)                      # [W_uk^T q' | turned q'' | zeros]
        q_dim = torch.empty((T, H, D), **new) if parts else p[:, :self.q_size].unflatten(1, (H, D + R))[:, :, :D]
        kernels.latent_write(p, q_dim=q_dim if parts else None, q_rot=folded[:, :, K:] if self.row > K else None, **common)
        kernels.head_product(q_dim, self.fold, out=folded)
        if (ctx.compute_dtype == torch.bfloat16 and ctx.options.tuned_attention
                and kernels.attention_latent_decode_groups(H, K, self.row) > 0):
            o = kernels.attention_latent_decode(folded, view.k_pages, ctx.tok_seq, ctx.tok_pos, ctx.seq_slot, ctx.seq_start,
                                                view.block_table, rank=K, scale=self.scale,
                                                longest=ctx.model_cache_limit if ctx.replayed else ctx.max_end)
        else:
            o = kernels.attention_generic(folded.view(T, H * self.row), H, 1, self.row, view.k_pages, view.v_pages, ctx.tok_seq,
                                          ctx.tok_pos, ctx.seq_slot, view.block_table, self.scale, None, v_head_dim=K).view(T, H, K)
        return kernels.head_product(o, self.unfold, gate=gate).view(T, self.v_size)

    def forward(self, ctx, y, cache_view, stream):
        self.o.add_to_stream(ctx, self.heads_out(ctx, y, cache_view), stream)

    def output(self, ctx, y, cache_view):
        return self.o.f32_parts(ctx, self.heads_out(ctx, y, cache_view))
