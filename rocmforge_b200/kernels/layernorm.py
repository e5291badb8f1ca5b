"""Python faces of csrc/layernorm.cu: the residual update with a layer norm behind it, and the token table's gate."""
from __future__ import annotations

import functools

import torch

from ._ffi import c_float, c_int, c_ll, c_void_p, check, dtype_code, fn, need, need_cuda, ptr, stream
from .basic import _rows_or_parts


@functools.lru_cache(None)
def _f(name, *argtypes):
    return fn("layernorm", name, list(argtypes))


class RoutedSum:
    """The result of routed experts before it is summed: per token the weighted sum of the rows of ``y`` (float32 [pairs, H],
    sorted by expert) that ``inv`` names, in the order of the choices; a choice whose expert (``idx``) is not below ``experts``
    contributes the feed-forward's input ``x`` itself."""

    def __init__(self, y, inv, idx, w, x, experts: int):
        self.y, self.inv, self.idx, self.w, self.x, self.experts = y, inv, idx, w, x, int(experts)


class GatedRows:
    """A result (float32 [T, H] or a stack of partial sums) whose rows are multiplied by sigmoid(``logits``), a float32 [T]
    view."""

    def __init__(self, rows, logits):
        self.rows, self.logits = rows, logits


def stream_update(h: torch.Tensor, addends, compute_dtype: torch.dtype, *, post=None, next_norm=None, rounded: bool = False,
                  rows: torch.Tensor | None = None):
    """One pass over the float32 stream ``h`` [T, H], everything in 32-bit:

        m = the sum of ``addends`` (up to one RoutedSum and one dense one: a float32 [T, H], a stack [S, T, H] of partial sums
            added in index order, or GatedRows of such)
        m <- m / sqrt(mean(m^2) + eps) * w          with ``post`` = (w, eps)
        h += m
        returns (h - mean) / sqrt(mean((h - mean)^2) + eps) * w + b in the compute dtype with ``next_norm`` = (w, b, eps);
        with ``rounded`` h itself in the compute dtype; else None

    Without addends ``rows`` (int32) may list the rows to norm; h is then left alone."""
    routed, dense, logits = None, None, None
    for a in addends:
        if isinstance(a, RoutedSum):
            need(routed is None, "stream_update: one routed addend")
            routed = a
        else:
            need(dense is None, "stream_update: one dense addend")
            dense, logits = (a.rows, a.logits) if isinstance(a, GatedRows) else (a, None)
    need(h.dtype == torch.float32 and h.dim() == 2 and h.is_contiguous(), "stream_update: h must be contiguous float32 [T, H]")
    need(rows is None or (not addends and rows.dtype == torch.int32 and rows.dim() == 1), "stream_update: rows (int32) go without addends")
    need(not (rounded and next_norm is not None) and (addends or rounded or next_norm is not None), "stream_update: nothing to do")
    T, H = h.shape
    w_post, post_eps = post if post is not None else (None, 0.0)
    w, b, eps = next_norm if next_norm is not None else (None, None, 0.0)
    need_cuda(h, dense, logits, w_post, w, b, rows)
    vecs = [v for v in (w_post, w, b) if v is not None]
    need(all(v.shape == (H,) and v.is_contiguous() and v.dtype in (torch.float32, torch.bfloat16) for v in vecs)
         and (w is None or w.dtype == b.dtype), "stream_update: norm vectors must be [H] in float32 or bfloat16, w and b alike")
    n = 0
    if dense is not None:
        need(dense.dtype == torch.float32 and dense.is_contiguous() and dense.dim() in (2, 3) and tuple(dense.shape[-2:]) == (T, H),
             "stream_update: the dense addend must be contiguous float32 [T, H] or [S, T, H]")
        n = dense.shape[0] if dense.dim() == 3 else 1
    need(logits is None or (logits.dtype == torch.float32 and logits.shape == (T,)), "stream_update: gate logits must be float32 [T]")
    rargs = [ptr(None), ptr(None), ptr(None), ptr(None), ptr(None), 0, 1, 0]
    if routed is not None:
        top = routed.w.shape[1]
        need_cuda(routed.y, routed.inv, routed.idx, routed.w, routed.x)
        need(routed.y.dtype == torch.float32 and routed.y.is_contiguous() and routed.y.shape == (T * top, H)
             and routed.inv.numel() == T * top and routed.idx.shape == (T, top) and routed.w.shape == (T, top)
             and routed.inv.dtype == torch.int32 and routed.idx.dtype == torch.int32 and routed.w.dtype == torch.float32
             and routed.x.dtype == compute_dtype and routed.x.shape == (T, H) and routed.x.stride(1) == 1,
             "stream_update: the routed addend's tensors do not fit h")
        rargs = [ptr(routed.y), ptr(routed.inv), ptr(routed.idx), ptr(routed.w), ptr(routed.x), routed.x.stride(0), top, routed.experts]
    R = T if rows is None else rows.shape[0]
    y = torch.empty((R, H), dtype=compute_dtype, device=h.device) if rounded or next_norm is not None else None
    f = _f("rf_stream_update", c_int, c_void_p, c_void_p, c_void_p, c_int, c_ll, c_void_p, c_int, c_void_p, c_void_p, c_void_p,
           c_void_p, c_void_p, c_ll, c_int, c_int, c_void_p, c_int, c_float, c_void_p, c_void_p, c_int, c_float, c_void_p, c_int,
           c_int, c_void_p)
    check(f(dtype_code(compute_dtype), ptr(h), ptr(rows), ptr(dense), n, T * H, ptr(logits),
            logits.stride(0) if logits is not None else 0, *rargs, ptr(w_post),
            int(w_post is not None and w_post.dtype == torch.float32), float(post_eps), ptr(w), ptr(b),
            int(w is not None and w.dtype == torch.float32), float(eps), ptr(y), R, H, stream()), f"stream_update (H={H})")
    return y


def side_gate(z: torch.Tensor, table: torch.Tensor, col0: int, dim: int, tokens: torch.Tensor, width: int) -> torch.Tensor:
    """gelu(z) * table[token, col0 : col0 + dim] in the table's dtype as [T, width], zeros from column ``dim`` on (gelu by tanh,
    evaluated in 32-bit).  z [T, >= dim] in the table's dtype, or float32 partial sums [S, T, >= dim]."""
    need_cuda(z, table, tokens)
    T, W, S, ps, rs = _rows_or_parts(z, "side_gate")
    need(W >= dim and width >= dim and (S > 0 or z.dtype == table.dtype), "side_gate: z must be [T, >= dim] in the table's dtype")
    need(table.dim() == 2 and table.stride(1) == 1 and 0 <= col0 and col0 + dim <= table.shape[1], "side_gate: the columns leave the table")
    need(tokens.dtype == torch.int32 and tokens.shape == (T,), "side_gate: tokens must be int32 [T]")
    out = torch.empty((T, width), dtype=table.dtype, device=z.device)
    f = _f("rf_side_gate", c_int, c_void_p, c_int, c_ll, c_int, c_void_p, c_ll, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
           c_void_p)
    check(f(dtype_code(table.dtype), ptr(z), S, ps, rs, ptr(table), table.stride(0), int(col0), ptr(tokens), ptr(out), int(width),
            int(dim), table.shape[0], T, stream()), "side_gate")
    return out
