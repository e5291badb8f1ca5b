"""Python faces of the kernels of latent-caching attention (csrc/latent.cu, attention_latent_prefill.cu,
attention_latent_decode.cu) and of several residual streams (csrc/streams.cu).

Each function checks shapes and dtypes, then launches on torch's current stream.
"""
from __future__ import annotations

import functools

import torch

from ._ffi import c_float, c_int, c_ll, c_void_p, check, dtype_code, fn, need, need_cuda, ptr, stream
from .basic import PAGE, decode_splits, key_span


@functools.lru_cache(None)
def _f(module, name, *argtypes):
    return fn(module, name, list(argtypes))


def _is_f32(t) -> int:
    return int(t is not None and t.dtype == torch.float32)


# ---------------------------------------------------------------- several residual streams

def streams_update(x: torch.Tensor, streams: int, compute_dtype: torch.dtype, *, y: torch.Tensor | None = None,
                   mix: torch.Tensor | None = None, out: torch.Tensor | None = None, in_: torch.Tensor | None = None,
                   next_norm=None, rows: torch.Tensor | None = None):
    """The streams of every token after a sub-layer, and the next sub-layer's input, in one pass and in 32-bit:

        x_t <- sum_s mix[s, t] x_s + out[t] y         (all from the old streams; without ``y`` nothing is updated)
        next = rms(sum_t in_[t] x_t) * weight          (``next_norm`` = (weight, eps); ``in_`` None: the plain sum)

    ``x`` float32 [T, streams, W], or [T, 1, W] while all streams are still equal; ``y`` float32 [T, W] or a stack [n, T, W]
    of partial sums, added in index order; ``rows`` (int32, without ``y``): only those tokens.  Returns (x, next or None); an
    ``x`` with all streams is updated in place."""
    need_cuda(x, y, mix, out, in_, rows)
    need(x.dtype == torch.float32 and x.dim() == 3 and x.is_contiguous() and x.shape[1] in (1, streams),
         "streams_update: x must be contiguous float32 [T, 1 or streams, W]")
    T, have, W = x.shape
    for v, shape in ((mix, (streams, streams)), (out, (streams,)), (in_, (streams,))):
        need(v is None or (v.dtype == torch.float32 and tuple(v.shape) == shape and v.is_contiguous()),
             f"streams_update: coefficients must be float32 {shape}")
    x_new, n_y = x, 0
    if y is not None:
        need(y.dtype == torch.float32 and y.is_contiguous() and tuple(y.shape[-2:]) == (T, W) and y.dim() in (2, 3)
             and mix is not None and out is not None and rows is None,
             "streams_update: y must be contiguous float32 [T, W] or [n, T, W], with mix and out")
        n_y = y.shape[0] if y.dim() == 3 else 1
        if have != streams:
            x_new = torch.empty((T, streams, W), dtype=torch.float32, device=x.device)
    weight, eps, nxt, n_rows = None, 0.0, None, T
    if rows is not None:
        need(rows.dtype == torch.int32 and rows.dim() == 1 and next_norm is not None, "streams_update: rows must be 1-d int32")
        n_rows = rows.shape[0]
    if next_norm is not None:
        weight, eps = next_norm
        need(weight.is_cuda and weight.shape == (W,) and weight.dtype in (torch.float32, torch.bfloat16) and weight.is_contiguous(),
             "streams_update: the norm's weight must be [W]")
        nxt = torch.empty((n_rows, W), dtype=compute_dtype, device=x.device)
    f = _f("streams", "rf_streams_update", c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
           c_void_p, c_int, c_float, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p)
    check(f(dtype_code(compute_dtype), ptr(x), have, ptr(y), n_y, ptr(mix), ptr(out), ptr(x_new) if y is not None else ptr(None),
            ptr(in_), ptr(weight), _is_f32(weight), float(eps), ptr(nxt), ptr(rows), streams, W, n_rows, stream()),
          f"streams_update (streams={streams}, W={W})")
    return x_new, nxt


def pair_embed(table: torch.Tensor, pairs: torch.Tensor | None, ids, tok_seq, tok_pos, seq_slot, cu_q, state, *, scale: float,
               mul_prev: int = 0, mul_cur: int = 0, buckets: int = 1, norm=None) -> torch.Tensor:
    """x = table[id] * scale + pairs[(previous id * mul_prev + id * mul_cur) mod buckets] (row ``buckets`` for a sequence's
    first token), RMS-normed with ``norm`` = (weight, eps) if given; float32 [T, W].  ``state`` int32 [slots, 2]: the token of
    position p is kept at p % 2, so that a step's first token finds the one before it."""
    need_cuda(table, pairs, ids, tok_seq, tok_pos, seq_slot, cu_q, state)
    need(table.dim() == 2 and table.is_contiguous() and ids.dtype == torch.int32, "pair_embed: table must be a contiguous matrix")
    V, W = table.shape
    T = ids.shape[0]
    weight, eps = norm if norm is not None else (None, 0.0)
    if pairs is not None:
        need(pairs.is_contiguous() and pairs.dtype == table.dtype and tuple(pairs.shape) == (buckets + 1, W),
             "pair_embed: the pair table must be [buckets + 1, W] of the embedding's dtype")
        need(state is not None and state.dtype == torch.int32 and state.dim() == 2 and state.shape[1] == 2 and state.is_contiguous(),
             "pair_embed: state must be int32 [slots, 2]")
    h = torch.empty((T, W), dtype=torch.float32, device=table.device)
    f = _f("streams", "rf_pair_embed", c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
           c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_float, c_ll, c_ll, c_ll, c_float, c_void_p)
    check(f(dtype_code(table.dtype), ptr(table), ptr(pairs), ptr(ids), ptr(tok_seq), ptr(tok_pos), ptr(seq_slot), ptr(cu_q),
            ptr(state), ptr(weight), _is_f32(weight), ptr(h), T, W, V, float(scale), int(mul_prev) % buckets, int(mul_cur) % buckets,
            int(buckets), float(eps), stream()), f"pair_embed (W={W})")
    return h


def scale_(x: torch.Tensor, factor: float) -> torch.Tensor:
    """x <- factor * x in place (float32 logits)."""
    need_cuda(x)
    need(x.dtype == torch.float32 and x.is_contiguous(), "scale: a contiguous float32 tensor")
    f = _f("streams", "rf_scale", c_void_p, c_ll, c_float, c_void_p)
    check(f(ptr(x), x.numel(), float(factor), stream()), "scale")
    return x


# ---------------------------------------------------------------- latents on their way into the cache

def latent_write(src: torch.Tensor, *, q_col: int, down_col: int, heads: int, dim: int, rot: int, rank: int, norm_weight, eps: float,
                 rotation, tok_seq, tok_pos, seq_slot, block_table, pages: torch.Tensor, compute_dtype: torch.dtype,
                 rows: torch.Tensor | None = None, q_dim: torch.Tensor | None = None, q_rot: torch.Tensor | None = None,
                 gate_col: int = 0, gate: torch.Tensor | None = None) -> None:
    """The projection's rows q (``heads`` x [dim | rot], at column ``q_col``) | down (rank + rot, at ``down_col``) | gate.

    ``src`` [T, columns] in the compute dtype, or a float32 stack [n, T, columns] of partial sums.  down's first ``rank``
    numbers, RMS-normed with ``norm_weight``, and its last ``rot``, turned by the position (``rotation``: inv_freq,
    interleaved, magnitude of a position encoding; None with rot 0), become the position's row of ``pages``
    [n_pages, 1, 64, ld >= rank + rot] (zeros behind them), and of ``rows`` [T, ld] if given.  The queries' rotated parts go to
    ``q_rot`` [T, heads, >= rot] (zeros behind them; it may be a view of ``src`` itself), their first parts to ``q_dim``
    [T, heads, dim] if given, and the gate's columns to ``gate`` [T, n] if given."""
    need_cuda(src, norm_weight, tok_seq, tok_pos, seq_slot, block_table, pages, rows, q_dim, q_rot, gate)
    parts = src.dim() == 3
    need(src.stride(-1) == 1 and (src.dtype == torch.float32 and src.is_contiguous() if parts else src.dim() == 2 and src.dtype == compute_dtype),
         "latent_write: src must be [T, columns] of the compute dtype or a float32 stack of partial sums")
    T = src.shape[-2]
    ld = pages.shape[-1]
    need(pages.dtype == compute_dtype and pages.is_contiguous() and tuple(pages.shape[1:3]) == (1, PAGE) and ld >= rank + rot,
         "latent_write: pages must be [n_pages, 1, 64, >= rank + rot] of the compute dtype")
    need(norm_weight.shape == (rank,) and norm_weight.is_contiguous(), "latent_write: the norm's weight must be [rank]")
    need(rows is None or (tuple(rows.shape) == (T, ld) and rows.is_contiguous() and rows.dtype == compute_dtype), "latent_write: rows must be [T, ld]")
    need(rot == 0 or (q_rot is not None and rotation is not None), "latent_write: rotated parts need a place and a rotation")
    for v, n in ((q_dim, dim), (q_rot, rot)):
        need(v is None or (v.dim() == 3 and v.shape[0] == T and v.shape[1] == heads and v.shape[2] >= n and v.stride(2) == 1
                           and v.dtype == compute_dtype), "latent_write: query parts must be [T, heads, n] views")
    need(gate is None or (gate.dim() == 2 and gate.shape[0] == T and gate.is_contiguous() and gate.dtype == compute_dtype), "latent_write: gate must be [T, n]")
    rotation = rotation or {}
    inv_freq = rotation.get("inv_freq")
    need(rot == 0 or (inv_freq is not None and inv_freq.dtype == torch.float32 and inv_freq.numel() == rot // 2),
         "latent_write: inv_freq must hold rot / 2 float32 frequencies")

    def st(v, i):
        return v.stride(i) if v is not None else 0
    f = _f("latent", "rf_latent_write", c_int, c_void_p, c_int, c_int, c_ll, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p,
           c_int, c_float, c_void_p, c_int, c_float, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p,
           c_ll, c_ll, c_void_p, c_ll, c_ll, c_int, c_void_p, c_int, c_int, c_void_p)
    check(f(dtype_code(compute_dtype), ptr(src), src.stride(-2), src.shape[0] if parts else 0, src.stride(0) if parts else 0, q_col,
            down_col, gate_col, heads, dim, rot, rank, ptr(norm_weight), _is_f32(norm_weight), float(eps), ptr(inv_freq),
            int(bool(rotation.get("interleaved", False))), float(rotation.get("magnitude", 1.0)), ptr(tok_seq), ptr(tok_pos), ptr(seq_slot),
            ptr(block_table), block_table.shape[1], ptr(pages), ld, ptr(rows), ptr(q_dim), st(q_dim, 0), st(q_dim, 1), ptr(q_rot),
            st(q_rot, 0), st(q_rot, 1), q_rot.shape[2] - rot if q_rot is not None else 0, ptr(gate), gate.shape[1] if gate is not None else 0,
            T, stream()), f"latent_write (heads={heads}, dim={dim}, rot={rot}, rank={rank})")


def latent_gather(pages: torch.Tensor, cu_k: torch.Tensor, seq_slot, block_table, n_rows: int) -> torch.Tensor:
    """The cache rows of whole sequences as one matrix [n_rows, ld]: position j of sequence i in row cu_k[i] + j (``cu_k`` int32
    [B + 1], n_rows = cu_k[B])."""
    need_cuda(pages, cu_k, seq_slot, block_table)
    need(pages.is_contiguous() and tuple(pages.shape[1:3]) == (1, PAGE) and (pages.shape[3] * pages.element_size()) % 16 == 0,
         "latent_gather: rows of whole 16-byte pieces")
    B = seq_slot.shape[0]
    need(cu_k.dtype == torch.int32 and cu_k.numel() == B + 1, "latent_gather: cu_k must be int32 [B + 1]")
    out = torch.empty((n_rows, pages.shape[3]), dtype=pages.dtype, device=pages.device)
    f = _f("latent", "rf_latent_gather", c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_void_p)
    check(f(ptr(pages), pages.shape[3] * pages.element_size(), ptr(cu_k), ptr(seq_slot), ptr(block_table), block_table.shape[1],
            ptr(out), n_rows, B, stream()), "latent_gather")
    return out


def head_product(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor | None = None, gate: torch.Tensor | None = None) -> torch.Tensor:
    """out[t, h, :] = W_h x[t, h, :] with a matrix per head, ``w`` [heads, N, K]; ``x`` [T, heads, K] and ``out`` [T, heads, >= N]
    may be strided; ``gate`` [T, heads * N] (rows may be strided): the results are multiplied by sigmoid(gate)."""
    need_cuda(x, w, out, gate)
    H, N, K = w.shape
    T = x.shape[0]
    need(w.is_contiguous() and x.dim() == 3 and x.shape[1:] == (H, K) and x.stride(2) == 1 and x.dtype == w.dtype,
         "head_product: x [T, heads, K] and w [heads, N, K] must share a dtype")
    if out is None:
        out = torch.empty((T, H, N), dtype=x.dtype, device=x.device)
    need(out.dim() == 3 and out.shape[:2] == (T, H) and out.shape[2] >= N and out.stride(2) == 1 and out.dtype == x.dtype,
         "head_product: out must be [T, heads, >= N]")
    need(gate is None or (gate.shape == (T, H * N) and gate.stride(1) == 1 and gate.dtype == x.dtype), "head_product: gate must be [T, heads * N]")
    f = _f("latent", "rf_head_product", c_int, c_void_p, c_ll, c_ll, c_void_p, c_int, c_int, c_int, c_void_p, c_ll, c_ll, c_void_p, c_ll,
           c_int, c_void_p)
    check(f(dtype_code(x.dtype), ptr(x), x.stride(0), x.stride(1), ptr(w), H, N, K, ptr(out), out.stride(0), out.stride(1), ptr(gate),
            gate.stride(0) if gate is not None else 0, T, stream()), f"head_product (heads={H}, N={N}, K={K})")
    return out


# ---------------------------------------------------------------- attention

@functools.lru_cache(None)
def attention_latent_prefill_supported(heads: int, dim: int, rot: int, vdim: int, rank: int) -> bool:
    f = _f("attention_latent_prefill", "rf_attention_latent_prefill_supported", c_int, c_int, c_int, c_int, c_int)
    return bool(f(heads, dim, rot, vdim, rank))


def attention_latent_prefill(q: torch.Tensor, kv: torch.Tensor, lat: torch.Tensor, q_tiles, seq_start, seq_nnew, cu_q, cu_k, *,
                             heads: int, dim: int, rot: int, vdim: int, rank: int, scale: float, window: int | None = None,
                             gate: torch.Tensor | None = None) -> torch.Tensor:
    """Causal attention of the step's new tokens over expanded latents, with tcgen05.mma: ``q`` [T, >= heads * (dim + rot)];
    ``kv`` [n, heads * dim | heads * vdim] and ``lat`` [n, >= rank + rot] hold position j of sequence i in row cu_k[i] + j (unrotated
    key parts and values; latents and, from column ``rank`` on, the rotated key part all heads share); ``q_tiles`` (sequence, first
    row) pairs of 128-row tiles.  ``gate`` [T, heads * vdim]: the result is multiplied by sigmoid(gate).  bfloat16."""
    need_cuda(q, kv, lat, q_tiles, seq_start, seq_nnew, cu_q, cu_k, gate)
    need(all(t.dtype == torch.bfloat16 and t.dim() == 2 and t.stride(1) == 1 and t.data_ptr() % 16 == 0 and t.stride(0) % 8 == 0
             for t in (q, kv, lat)), "attention_latent_prefill: bfloat16 matrices with 16-byte aligned rows")
    need(kv.shape[0] == lat.shape[0] and kv.shape[1] == heads * (dim + vdim), "attention_latent_prefill: kv must be [n, heads * (dim + vdim)]")
    need(gate is None or (gate.dtype == torch.bfloat16 and gate.shape == (q.shape[0], heads * vdim) and gate.stride(1) == 1),
         "attention_latent_prefill: gate must be [T, heads * vdim]")
    T = q.shape[0]
    out = torch.empty((T, heads * vdim), dtype=torch.bfloat16, device=q.device)
    from .tensor_core import status_word
    f = _f("attention_latent_prefill", "rf_attention_latent_prefill", c_void_p, c_int, c_int, c_void_p, c_int, c_void_p, c_int, c_int,
           c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
           c_int, c_float, c_int, c_void_p, c_void_p)
    check(f(ptr(q), q.stride(0), T, ptr(kv), kv.stride(0), ptr(lat), lat.stride(0), kv.shape[0], heads * dim, ptr(out), out.stride(0),
            ptr(gate), gate.stride(0) if gate is not None else 0, ptr(q_tiles), q_tiles.numel() // 2, ptr(seq_start), ptr(seq_nnew),
            ptr(cu_q), ptr(cu_k), heads, dim, rot, vdim, rank, float(scale), key_span(window), ptr(status_word(q.device)), stream()),
          f"attention_latent_prefill (heads={heads}, dim={dim}, rot={rot}, vdim={vdim})")
    return out


@functools.lru_cache(None)
def attention_latent_decode_groups(heads: int, rank: int, ld: int) -> int:
    """How many groups of heads the latent decode attention cuts ``heads`` into; 0: it does not take these sizes."""
    if not _f("attention_latent_decode", "rf_attention_latent_decode_supported", c_int, c_int, c_int)(heads, rank, ld):
        return 0
    return _f("attention_latent_decode", "rf_attention_latent_decode_groups", c_int, c_int, c_int)(heads, rank, ld)


def attention_latent_decode(q: torch.Tensor, pages: torch.Tensor, tok_seq, tok_pos, seq_slot, seq_start, block_table, *, rank: int,
                            scale: float, window: int | None = None, splits: int | None = None,
                            longest: int | None = None) -> torch.Tensor:
    """Attention of single tokens in the latents' space, with tcgen05.mma: ``q`` [T, heads, ld] (folded queries | rotated parts |
    zeros), ``pages`` [n_pages, 1, 64, ld]; scores over whole rows, values = the rows' first ``rank`` numbers; [T, heads, rank].
    A cluster of ``splits`` CTAs per (token, group of heads) shares the pages (chosen from T and ``longest`` if not given)."""
    need_cuda(q, pages, tok_seq, tok_pos, seq_slot, seq_start, block_table)
    T, heads, ld = q.shape
    groups = attention_latent_decode_groups(heads, rank, ld)
    need(groups > 0, f"attention_latent_decode: heads={heads}, rank={rank}, row={ld} is not supported")
    need(q.dtype == torch.bfloat16 and q.is_contiguous() and q.data_ptr() % 16 == 0, "attention_latent_decode: q must be contiguous bfloat16")
    need(pages.dtype == torch.bfloat16 and pages.is_contiguous() and tuple(pages.shape[1:]) == (1, PAGE, ld),
         "attention_latent_decode: pages must be [n_pages, 1, 64, ld] in bfloat16")
    if splits is None:
        splits = decode_splits(T, groups, longest, window)
    out = torch.empty((T, heads, rank), dtype=torch.bfloat16, device=q.device)
    from .tensor_core import status_word
    f = _f("attention_latent_decode", "rf_attention_latent_decode", c_void_p, c_void_p, c_ll, c_void_p, c_void_p, c_void_p, c_void_p,
           c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_float, c_int, c_int, c_int, c_void_p, c_void_p)
    check(f(ptr(q), ptr(pages), pages.shape[0], ptr(out), ptr(tok_seq), ptr(tok_pos), ptr(seq_slot), ptr(seq_start), ptr(block_table),
            block_table.shape[1], heads, rank, ld, float(scale), key_span(window), int(splits), T, ptr(status_word(q.device)), stream()),
          f"attention_latent_decode (heads={heads}, rank={rank}, row={ld}, splits={splits})")
    return out
