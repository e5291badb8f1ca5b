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
