"""The kernels of the Gedilorn decoder alone (needs a GPU), against the plain functions or the sums written out, with inputs made
so that a key one place off, a swapped index, a lost token or a missing gate shows."""
import math

import pytest
import torch

from plain import gedilorn_plain as P

pytestmark = pytest.mark.gpu
DEV = "cuda"
F32, BF16 = torch.float32, torch.bfloat16


def ints(x):
    return torch.tensor(list(x), dtype=torch.int32, device=DEV)


def status_clean():
    from rocmforge_b200 import kernels
    kernels.tensor_core.check_status(torch.device(DEV))


# --------------------------------------------------------------------------- streams

@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 6, 7, 8, 9, 12])
@pytest.mark.parametrize("T,W,n", [(1, 2048, 3), (3, 64, 1), (200, 100, 2), (5, 1024, 10), (150, 516, 1), (8, 4096, 4)])
def test_new_streams_and_the_next_input(S, T, W, n):
    """x_t <- sum_s mix[s, t] x_s + out[t] y with a mix that is not symmetric, y as partial sums; the normed sum of the NEW streams;
    from equal streams held once and from S of them (in place); the sum alone, and for chosen rows."""
    from rocmforge_b200 import kernels
    g = torch.Generator(device=DEV).manual_seed(S * 1000 + T)
    r = lambda *shape: torch.randn(*shape, generator=g, device=DEV)
    mix, out, inn, w = r(S, S), r(S), r(S), r(W)
    parts = r(n, T, W)
    for first in (True, False):
        x = r(T, 1 if first else S, W)
        full = x.expand(T, S, W).double().transpose(0, 1)
        want = P.spread(full, mix.double(), out.double(), parts.double().sum(0))
        u = P.rms_norm(P.collect(want, inn.double()), w.double(), 1e-5)
        for dt in (F32, BF16):
            x_new, y = kernels.streams_update(x.clone(), S, dt, y=parts if n > 1 else parts[0], mix=mix, out=out, in_=inn,
                                              next_norm=(w.to(dt), 1e-5))
            assert (x_new.double().transpose(0, 1) - want).abs().max() < 2e-5 * want.abs().max()
            tol = 2e-5 if dt == F32 else 2e-2
            assert y.dtype == dt and (y.double() - u).abs().max() < tol * u.abs().max()
        x_new, y = kernels.streams_update(x.clone(), S, F32, y=parts, mix=mix, out=out)
        assert y is None and (x_new.double().transpose(0, 1) - want).abs().max() < 2e-5 * want.abs().max()
        rows = ints([T - 1, 0, T // 2])
        _, y = kernels.streams_update(x, S, F32, next_norm=(w, 1e-5), rows=rows)
        ref = P.rms_norm(full.sum(0), w.double(), 1e-5)[rows.long()]
        assert (y.double() - ref).abs().max() < 2e-5 * ref.abs().max()
        _, y = kernels.streams_update(x, S, F32, in_=inn, next_norm=(w, 1e-5))
        ref = P.rms_norm(P.collect(full, inn.double()), w.double(), 1e-5)
        assert (y.double() - ref).abs().max() < 2e-5 * ref.abs().max()


# --------------------------------------------------------------------------- embedding of pairs

@pytest.mark.parametrize("V,W,buckets,mp,mc", [(50, 64, 37, 1009, 53), (120000, 36, 99991, 2147483647, 1999999973), (30, 10, 1, 3, 5),
                                               (90, 1028, 4000, 31, 17)])
def test_rows_of_pairs_over_portions_of_every_parity(V, W, buckets, mp, mc):
    """Two sequences side by side in portions of odd and even length: the previous token comes from the step's own tokens or from
    the state; multipliers whose products leave 32 bits; a slot used again starts without a previous token; a step of one token
    that runs twice (with another token first) finds what it found."""
    from rocmforge_b200 import kernels
    g = torch.Generator().manual_seed(V)
    E, B = torch.randn(V, W, generator=g), torch.randn(buckets + 1, W, generator=g)
    w = torch.rand(W, generator=g) + 0.5
    cfg = {"embedding": {"scale": 3.0, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}}
    Wd = {"embed": E.double(), "bigram": B.double(), "embed.norm": w.double()}
    seqs = [torch.randint(0, V, (40,), generator=g).tolist() for _ in range(2)]
    if V == 120000:
        seqs[0][3:6] = [V - 1, V - 1, V - 2]
    refs = [P.embedding(cfg, Wd, s, 1e-6) for s in seqs]
    state = torch.full((5, 2), -7, dtype=torch.int32, device=DEV)          # what an earlier holder of the slots left
    Ed, Bd, wd = E.to(DEV), B.to(DEV), w.to(DEV)

    def step(chunks, slots, starts):
        toks = [t for c in chunks for t in c]
        cu = [0]
        for c in chunks:
            cu.append(cu[-1] + len(c))
        seq = [i for i, c in enumerate(chunks) for _ in c]
        pos = [st + k for st, c in zip(starts, chunks) for k in range(len(c))]
        return kernels.pair_embed(Ed, Bd, ints(toks), ints(seq), ints(pos), ints(slots), ints(cu), state, scale=3.0, mul_prev=mp,
                                  mul_cur=mc, buckets=buckets, norm=(wd, 1e-6)).double().cpu()
    at = 0
    for n in (1, 2, 3, 1, 1, 4, 5, 2, 1, 7, 6, 1):
        if at + n > 40:
            break
        if n == 1:
            step([[(seqs[0][at] + 1) % V], [(seqs[1][at] + 2) % V]], [3, 1], [at, at])          # a step that will be dropped
        got = step([seqs[0][at:at + n], seqs[1][at:at + n]], [3, 1], [at, at])
        want = torch.cat([refs[0][at:at + n], refs[1][at:at + n]])
        assert (got - want).abs().max() < 1e-5 * want.abs().max(), f"portion of {n} tokens at {at}"
        at += n
    got = step([seqs[1][:3]], [3], [0])
    assert (got - refs[1][:3]).abs().max() < 1e-5 * refs[1].abs().max(), "a slot used again"


# --------------------------------------------------------------------------- the gated unit with relu

@pytest.mark.parametrize("M,N,K", [(1, 80, 64), (7, 200, 72), (40, 256, 128), (128, 272, 64), (130, 512, 192), (300, 320, 136), (9, 34, 30)])
def test_relu_gated_product(M, N, K):
    """relu(gate) * up from row-interleaved weights: the products' epilogues (few tokens, many tokens, clustered) and the separate
    kernel, on values of both signs."""
    from rocmforge_b200 import kernels
    tc = kernels.tensor_core
    torch.manual_seed(M)
    x, w = torch.randn(M, K, device=DEV).to(BF16), (torch.randn(N, K, device=DEV) / K ** 0.5).to(BF16)
    p = x.double() @ w.double().T
    want = torch.relu(p[:, 0::2]) * p[:, 1::2]
    got = [kernels.swiglu(kernels.gemm_simt(x.float(), w.float()), activation="relu")]
    if tc.supported(M, N, K, tc.REGLU):
        if M <= tc.SKINNY_MAX_TOKENS:
            got.append(tc.gemm_tc_skinny(x, w, mode=tc.REGLU))
        got += [tc.gemm_tc(x, w, mode=tc.REGLU), tc.gemm_tc(x, w, mode=tc.REGLU, cluster=0)]
    for y in got:
        tol = 1e-4 if y.dtype == F32 else 1e-2
        assert y.shape == want.shape and (y.double() - want).abs().max() < tol * want.abs().max()
    status_clean()


# --------------------------------------------------------------------------- latents on their way into the cache

def _positions(lens, starts, extra=3, seed=0):
    """(tok_seq, tok_pos, seq_slot, block_table, n_pages) of sequences that bring lens[i] tokens from starts[i] on; pages shuffled."""
    g = torch.Generator().manual_seed(seed)
    B = len(lens)
    need = [(s + n + 63) // 64 for s, n in zip(starts, lens)]
    n_pages = sum(need) + extra
    order = torch.randperm(n_pages, generator=g).tolist()
    bt = torch.full((B + 2, max(need)), -1, dtype=torch.int32)
    slots = [(2 * i + 1) % (B + 2) for i in range(B)] if (B + 2) % 2 else list(range(1, B + 1))
    at = 0
    for i in range(B):
        bt[slots[i], :need[i]] = torch.tensor(order[at:at + need[i]], dtype=torch.int32)
        at += need[i]
    seq = [i for i, n in enumerate(lens) for _ in range(n)]
    pos = [s + k for s, n in zip(starts, lens) for k in range(n)]
    return ints(seq), ints(pos), ints(slots), bt.to(DEV), n_pages


@pytest.mark.parametrize("H,D,R,K", [(3, 10, 6, 21), (1, 16, 0, 12), (5, 48, 24, 136), (20, 128, 64, 512), (2, 8, 2, 3)])
@pytest.mark.parametrize("dt", [F32, BF16])
def test_the_cache_row_and_the_query_parts(H, D, R, K, dt):
    """Norm of the latent's part only, rotation of neighbouring pairs with stretched frequencies and a magnitude, zeros behind; rows
    at the right places of shuffled pages and nothing else touched; from the product's matrix and from partial sums; queries left
    in place (turned where they lie) and taken out; the gate's columns."""
    from rocmforge_b200 import kernels
    from rocmforge_b200.parts import POSITIONS
    torch.manual_seed(H)
    lens, starts = [5, 1, 70], [0, 63, 3]
    seq, pos, slots, bt, n_pages = _positions(lens, starts)
    T, G = sum(lens), 24
    q_n, ld = H * (D + R), (K + R + 7) // 8 * 8
    down_col = (q_n + 7) // 8 * 8
    gate_col = (down_col + K + R + 7) // 8 * 8
    src = torch.randn(T, gate_col + G, device=DEV).to(dt)
    w = (torch.rand(K, device=DEV) + 0.5).to(dt)
    rot = None
    if R:
        enc = POSITIONS.build("rope_yarn", head_dim=R, theta=100.0, interleaved=True, factor=4.0, original=64, fast=8.0, slow=1.0)
        enc.prepare(DEV)
        rot = enc.rotation()
    x = src.double().cpu()
    c = P.rms_norm(x[:, down_col:down_col + K], w.double().cpu(), 1e-5)
    heads = x[:, :q_n].reshape(T, H, D + R)
    kr, qr = x[:, down_col + K:down_col + K + R], heads[..., D:]
    if R:
        f, mag = P.stretched_frequencies(R, 100.0, dict(factor=4.0, original=64, fast=8.0, slow=1.0))
        kr, qr = P.turn_neighbours(kr, pos.cpu(), f, mag), P.turn_neighbours(qr, pos.cpu(), f, mag)
    want = torch.cat([c, kr, torch.zeros(T, ld - K - R, dtype=torch.float64)], dim=1)
    tol = 2e-5 if dt == F32 else 1e-2

    def near(got, ref):
        assert got.numel() == 0 or (got.double().cpu() - ref).abs().max() <= tol * max(1.0, float(ref.abs().max()))
    for form in ("matrix", "parts", "in place"):
        pages = torch.full((n_pages, 1, 64, ld), 7.0, device=DEV, dtype=dt)
        a = src.clone()
        if form == "parts":
            half = torch.randn_like(a.float())
            a = torch.stack([a.float() - half, half])
        rows = torch.full((T, ld), 3.0, device=DEV, dtype=dt)
        q_dim = torch.zeros(T, H, D, device=DEV, dtype=dt)
        folded = torch.full((T, H, ld), 5.0, device=DEV, dtype=dt)
        q_rot = folded[:, :, K:] if form != "in place" else a[:, :q_n].unflatten(1, (H, D + R))[:, :, D:]
        gate = torch.zeros(T, G, device=DEV, dtype=dt)
        kernels.latent_write(a, q_col=0, down_col=down_col, heads=H, dim=D, rot=R, rank=K, norm_weight=w, eps=1e-5, rotation=rot,
                             tok_seq=seq, tok_pos=pos, seq_slot=slots, block_table=bt, pages=pages, compute_dtype=dt, rows=rows,
                             q_dim=q_dim if form != "in place" else None,
                             q_rot=q_rot if q_rot.shape[2] else None, gate_col=gate_col, gate=gate)
        near(rows, want)
        flat = pages.view(n_pages * 64, ld)
        at = bt[slots.long()[seq.long()], (pos // 64).long()].long() * 64 + (pos % 64).long()
        assert torch.equal(flat[at], rows)
        untouched = torch.ones(n_pages * 64, dtype=torch.bool, device=DEV)
        untouched[at] = False
        assert (flat[untouched] == 7.0).all()
        near(gate, x[:, gate_col:gate_col + G])
        near(q_rot[:, :, :R], qr)
        if form == "in place":
            assert torch.equal(a[:, :q_n].unflatten(1, (H, D + R))[:, :, :D], src[:, :q_n].unflatten(1, (H, D + R))[:, :, :D])
        else:
            near(q_dim, heads[..., :D])
            assert (folded[:, :, :K] == 5.0).all() and (folded[:, :, K + R:] == 0).all()


def test_rows_of_whole_sequences_are_gathered_in_order():
    from rocmforge_b200 import kernels
    lens = [1, 64, 65, 200]
    seq, pos, slots, bt, n_pages = _positions(lens, [0] * 4)
    pages = torch.randn(n_pages, 1, 64, 24, device=DEV).to(BF16)
    cu = ints([0] + torch.tensor(lens).cumsum(0).tolist())
    got = kernels.latent_gather(pages, cu, slots, bt, sum(lens))
    at = bt[slots.long()[seq.long()], (pos // 64).long()].long() * 64 + (pos % 64).long()
    assert torch.equal(got, pages.view(-1, 24)[at])


@pytest.mark.parametrize("T", [1, 5, 16, 17, 70, 130])
@pytest.mark.parametrize("H,N,K", [(1, 8, 12), (3, 21, 10), (5, 136, 48), (16, 512, 128), (16, 128, 512), (2, 100, 72)])
def test_a_matrix_per_head(T, H, N, K):
    """Strided inputs and outputs (other columns untouched), with and without the gate, sizes that are no multiple of a tile."""
    from rocmforge_b200 import kernels
    torch.manual_seed(T)
    for dt in (F32, BF16):
        pad = 8 - K % 8 if K % 8 else 8
        x = torch.randn(T, H, K + pad, device=DEV).to(dt)[:, :, :K]
        w = (torch.randn(H, N, K, device=DEV) / K ** 0.5).to(dt)
        out = torch.full((T, H, N + 3), 9.0, device=DEV, dtype=dt)
        gate = torch.randn(T, H * N + 8, device=DEV).to(dt)[:, :H * N]
        want = torch.einsum("thk,hnk->thn", x.double(), w.double())
        tol = 1e-5 if dt == F32 else 1e-2
        kernels.head_product(x, w, out=out)
        assert (out[:, :, :N].double() - want).abs().max() < tol * want.abs().max() and (out[:, :, N:] == 9.0).all()
        got = kernels.head_product(x, w, gate=gate)
        want = want * torch.sigmoid(gate.double()).view(T, H, N)
        assert (got.double() - want).abs().max() < tol * want.abs().max()


# --------------------------------------------------------------------------- attention

def _softmax_rows(q, keys, vals, scale, upto):
    """q [n, H, L], keys [T, H or 1, L], vals [T, H or 1, V]: row r sees keys 0 .. upto[r]; float64."""
    n, H, _ = q.shape
    out = []
    for h in range(H):
        k, v = keys[:, h % keys.shape[1]], vals[:, h % vals.shape[1]]
        s = (q[:, h] @ k.T) * scale
        hidden = torch.arange(k.shape[0], device=s.device)[None, :] > torch.as_tensor(upto, device=s.device)[:, None]
        out.append(torch.softmax(s.masked_fill(hidden, float("-inf")), dim=-1) @ v)
    return torch.stack(out, dim=1)


DECODE_SIZES = [(1, 64, 16), (3, 21, 6), (16, 512, 64), (17, 136, 24), (32, 200, 0), (40, 64, 8), (70, 56, 8), (128, 128, 64), (6, 192, 0),
                (2, 1024, 64)]


@pytest.mark.parametrize("H,K,R", DECODE_SIZES)
def test_single_tokens_over_cached_latents(H, K, R):
    """Sequences of 1 to 700 positions in shuffled pages whose other rows are NaN (pages not owned, positions not written), every
    number of CTAs a token, against the softmax written out in float64; the generic kernel on the same rows in 32-bit."""
    from rocmforge_b200 import kernels
    torch.manual_seed(H + K)
    ends = [1, 2, 16, 17, 63, 64, 65, 128, 130, 321, 700]
    ld = (K + R + 7) // 8 * 8
    B = len(ends)
    seq, pos, slots, bt, n_pages = _positions(ends, [0] * B)
    at = bt[slots.long()[seq.long()], (pos // 64).long()].long() * 64 + (pos % 64).long()
    for dt in (F32, BF16):
        pages = torch.full((n_pages, 1, 64, ld), float("nan"), device=DEV, dtype=dt)
        rows = torch.randn(sum(ends), ld, device=DEV).to(dt)
        rows[:, K + R:] = 0
        pages.view(-1, ld)[at] = rows
        q = (torch.randn(B, H, ld, device=DEV) * 0.6).to(dt)
        scale = 2.0 / (K + R) ** 0.5
        tok_seq, tok_pos, start = ints(range(B)), ints(e - 1 for e in ends), ints(max(e - 1, 0) for e in ends)
        want, a = [], 0
        for i, e in enumerate(ends):
            k = rows[a:a + e].double()[:, None]
            want.append(_softmax_rows(q[i:i + 1].double(), k, k[..., :K], scale, [e - 1])[0])
            a += e
        want = torch.stack(want)
        got = kernels.attention_generic(q.view(B, H * ld), H, 1, ld, pages, pages[..., :K], tok_seq, tok_pos, slots, bt, scale, None,
                                        v_head_dim=K).view(B, H, K).double()
        assert (got - want).abs().max() < (1e-5 if dt == F32 else 2e-2) * want.abs().max(), "generic"
        if dt == F32:
            continue
        assert kernels.attention_latent_decode_groups(H, K, ld) == -(-H // (16 if H <= 16 else 32 if H <= 32 else 64)) or K > 512
        for splits in (1, 2, 3, 4, 8, None):
            got = kernels.attention_latent_decode(q, pages, tok_seq, tok_pos, slots, start, bt, rank=K, scale=scale, splits=splits,
                                                  longest=max(ends)).double()
            err = (got - want).abs().amax(dim=(1, 2))
            assert err.max() < 2e-2 * want.abs().max(), f"{splits} CTAs a token: context of {ends[int(err.argmax())]}"
    status_clean()


@pytest.mark.parametrize("splits", [1, 2, 8])
@pytest.mark.parametrize("i,j", [(699, 0), (699, 63), (699, 64), (699, 639), (699, 640), (130, 1), (255, 128), (256, 127), (64, 0), (63, 63)])
def test_a_far_latent_among_hundreds(i, j, splits):
    """One position's row stands out and is found, with its own values; the row just behind the query would stand out more."""
    from rocmforge_b200 import kernels
    torch.manual_seed(i * 1000 + j)
    T, H, K, R = 702, 5, 96, 16
    rows = torch.randn(T, K + R, device=DEV) * 0.05
    rows[:, 0] = 0
    rows[j, 0], rows[i + 1, 0] = 4.0, 8.0
    rows[j, 1:K] = torch.randn(K - 1, device=DEV)
    rows[i + 1, 1:K] = 1000.0
    q = torch.zeros(1, H, K + R, device=DEV)
    q[..., 0] = 8.0
    rows, q = rows.to(BF16), q.to(BF16)
    seq, pos, slots, bt, n_pages = _positions([T], [0])
    pages = torch.full((n_pages, 1, 64, K + R), float("nan"), device=DEV, dtype=BF16)
    at = bt[slots.long()[seq.long()], (pos // 64).long()].long() * 64 + (pos % 64).long()
    pages.view(-1, K + R)[at] = rows
    got = kernels.attention_latent_decode(q, pages, ints([0]), ints([i]), slots, ints([i]), bt, rank=K, scale=1.0, splits=splits)
    assert (got[0].float() - rows[j, :K].float()).abs().max() < 2e-2 * float(rows[j, :K].float().abs().max())
    status_clean()


def test_scores_that_grow_from_page_to_page():
    """The reference of the exponentials has to move several times, by little and by much, up and (in effect) never down, for some heads
    and not for others, with earlier results rescaled; one to eight CTAs a token."""
    from rocmforge_b200 import kernels
    torch.manual_seed(3)
    T, H, K = 640, 20, 128
    rows = torch.randn(T, K, device=DEV) * 0.3
    rows[:, 0] = torch.linspace(-20, 20, T, device=DEV)
    rows[:, 1] = torch.where(torch.arange(T, device=DEV) % 130 == 77, 30.0, 0.0)
    q = torch.randn(1, H, K, device=DEV) * 0.3
    q[0, :, 0] = torch.linspace(-3, 3, H, device=DEV)
    q[0, ::3, 1] = 2.0
    rows, q = rows.to(BF16), q.to(BF16)
    seq, pos, slots, bt, n_pages = _positions([T], [0])
    pages = torch.zeros(n_pages, 1, 64, K, device=DEV, dtype=BF16)
    at = bt[slots.long()[seq.long()], (pos // 64).long()].long() * 64 + (pos % 64).long()
    pages.view(-1, K)[at] = rows
    want = _softmax_rows(q.double(), rows.double()[:, None], rows.double()[:, None], 1.0, [T - 1])[0]
    for splits in (1, 2, 4, 8):
        got = kernels.attention_latent_decode(q, pages, ints([0]), ints([T - 1]), slots, ints([T - 1]), bt, rank=K, scale=1.0, splits=splits)
        assert (got[0].double() - want).abs().max() < 2e-2 * want.abs().max(), f"{splits} CTAs"
    status_clean()


PREFILL_SIZES = [(4, 32, 16, 32, 64), (5, 48, 24, 96, 136), (3, 128, 64, 128, 512), (2, 16, 8, 144, 40), (2, 80, 0, 16, 64), (3, 64, 40, 112, 320),
                 (1, 192, 64, 256, 72), (2, 256, 128, 64, 64)]


def _expanded(H, D, R, V, K, n, seed):
    g = torch.Generator(device=DEV).manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g, device=DEV)
    ld = (K + R + 7) // 8 * 8
    kv, lat = (r(n, H * (D + V)) * 0.7).to(BF16), (r(n, ld) * 0.7).to(BF16)
    keys = torch.cat([kv[:, :H * D].double().view(n, H, D), lat[:, K:K + R].double()[:, None].expand(n, H, R)], dim=-1)
    return kv, lat, keys, kv[:, H * D:].double().view(n, H, V)


@pytest.mark.parametrize("gated", [False, True])
@pytest.mark.parametrize("H,D,R,V,K", PREFILL_SIZES)
def test_prompts_over_expanded_latents(H, D, R, V, K, gated):
    """Unequal sequences in one launch, some that start in the middle of a context, query tiles on and off borders of 128 and key
    tiles on and off borders of 64, against the softmax written out in float64."""
    from rocmforge_b200 import kernels
    assert kernels.attention_latent_prefill_supported(H, D, R, V, K)
    lens, starts = [1, 129, 300, 64, 7], [0, 0, 61, 256, 500]
    ends = [a + b for a, b in zip(lens, starts)]
    T, n = sum(lens), sum(ends)
    kv, lat, keys, vals = _expanded(H, D, R, V, K, n, H + D)
    torch.manual_seed(D)
    q = torch.randn(T, H * (D + R) + 16, device=DEV).to(BF16)[:, :H * (D + R)]
    gate = torch.randn(T, H * V + 8, device=DEV).to(BF16)[:, :H * V] if gated else None
    tiles = sorted([(i, r) for i, m in enumerate(lens) for r in range(0, m, 128)], key=lambda t: starts[t[0]] + t[1])
    cu_q, cu_k = [0], [0]
    for a, e in zip(lens, ends):
        cu_q.append(cu_q[-1] + a); cu_k.append(cu_k[-1] + e)
    scale = 1.5 / (D + R) ** 0.5
    got = kernels.attention_latent_prefill(q, kv, lat, ints(x for t in tiles for x in t), ints(starts), ints(lens), ints(cu_q), ints(cu_k),
                                           heads=H, dim=D, rot=R, vdim=V, rank=K, scale=scale, gate=gate).double().view(T, H, V)
    status_clean()
    for i in range(len(lens)):
        rows, ctx = slice(cu_q[i], cu_q[i + 1]), slice(cu_k[i], cu_k[i + 1])
        want = _softmax_rows(q[rows].double().view(-1, H, D + R), keys[ctx], vals[ctx], scale, range(starts[i], ends[i]))
        if gated:
            want = want * torch.sigmoid(gate[rows].double()).view(-1, H, V)
        err = (got[rows] - want).abs().amax(dim=(1, 2))
        assert err.max() < 2e-2 * max(1.0, float(want.abs().max())), f"sequence {i}, row {int(err.argmax())}"


@pytest.mark.parametrize("part", ["unrotated", "rotated"])
@pytest.mark.parametrize("i,j", [(299, 0), (299, 63), (299, 64), (130, 1), (255, 128), (256, 127), (64, 0), (63, 63), (127, 126), (128, 0)])
def test_a_far_key_in_a_prompt(i, j, part):
    """The query at i scores the key at j far above all others, through its unrotated part (one head alone) or through the shared rotated
    part (all heads), and the key just behind i higher still; whole prompts and a portion that begins at i - 1."""
    from rocmforge_b200 import kernels
    H, D, R, V, K, T = 3, 48, 24, 32, 40, 302
    kv, lat, _, _ = _expanded(H, D, R, V, K, T, i + j)
    kv, lat = kv.float() * 0.1, lat.float() * 0.1
    q = torch.randn(T, H, D + R, device=DEV) * 0.1
    vals = kv[:, H * D:].view(T, H, V)
    if part == "unrotated":
        q[i, 1, 0] = 30.0
        kv[j, D], kv[i + 1, D] = 3.0, 6.0
        found = [1]
    else:
        q[i, :, D] = 30.0
        lat[j, K], lat[i + 1, K] = 3.0, 6.0
        found = [0, 1, 2]
    vals[j], vals[i + 1] = torch.randn(H, V, device=DEV), 1000.0
    kv, lat, q = kv.to(BF16), lat.to(BF16), q.to(BF16).view(T, -1)
    for lo in (0, i - 1):
        n = T - lo
        tiles = [(0, r) for r in range(0, n, 128)]
        got = kernels.attention_latent_prefill(q[lo:].contiguous(), kv, lat, ints(x for t in tiles for x in t), ints([lo]), ints([n]), ints([0, n]),
                                               ints([0, T]), heads=H, dim=D, rot=R, vdim=V, rank=K, scale=1.0).view(n, H, V)
        want = kv[j, H * D:].view(H, V)
        for h in found:
            assert (got[i - lo, h].float() - want[h].float()).abs().max() < 3e-2, f"head {h}, from {lo} on"
    status_clean()


@pytest.mark.parametrize("D,R,V,K", [(576, 0, 576, 8), (600, 40, 700, 8), (1152, 0, 64, 8)])
def test_the_generic_attention_with_wide_heads(D, R, V, K):
    """Heads above 512 elements (chunks of 32 keys, a head a pass) against the softmax written out."""
    from rocmforge_b200 import kernels
    torch.manual_seed(D)
    T, H, L = 70, 3, D + R
    k, v = torch.randn(T, 1, L, device=DEV), torch.randn(T, 1, V, device=DEV)
    seq, pos, slots, bt, n_pages = _positions([T], [0])
    at = bt[slots.long()[seq.long()], (pos // 64).long()].long() * 64 + (pos % 64).long()
    kp, vp = torch.zeros(n_pages, 1, 64, L, device=DEV), torch.zeros(n_pages, 1, 64, V, device=DEV)
    kp.view(-1, L)[at], vp.view(-1, V)[at] = k[:, 0], v[:, 0]
    q = torch.randn(T, H, L, device=DEV)
    got = kernels.attention_generic(q.view(T, H * L), H, 1, L, kp, vp, seq, pos, slots, bt, 0.05, None, v_head_dim=V).view(T, H, V)
    want = _softmax_rows(q.double(), k.double(), v.double(), 0.05, range(T))
    assert (got.double() - want).abs().max() < 1e-4
