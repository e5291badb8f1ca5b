"""Each mechanism of the Dubodra decoder on its own kernels (needs a GPU), against the plain functions or the same sums in
float64, with inputs made so that a key one place off, a lost state, a group or a choice that should not count shows."""
import math

import pytest
import torch

from plain import dubodra_plain as P

pytestmark = pytest.mark.gpu
DEV = "cuda"


def i32(*values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def rel(got, want):
    return float((got.double() - want.double()).abs().max() / want.double().abs().max().clamp_min(1e-30))


# --------------------------------------------------------------------------- layer norm and the residual update

def ref_layer_norm(x, w, b, eps):
    x, w, b = x.double(), w.double(), b.double()
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * w + b


@pytest.mark.parametrize("T,H", [(1, 64), (5, 100), (3, 33), (300, 256), (7, 2048), (320, 1030), (2, 14000), (3, 5000), (310, 2100), (300, 5120), (299, 1996)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_layer_norm_of_all_and_of_listed_rows(T, H, dtype):
    """A row far from zero mean (an RMS norm, or a variance taken around zero, is far off), a nearly constant one (eps counts)."""
    from rocmforge_b200 import kernels
    torch.manual_seed(T * 7 + H)
    h = torch.randn(T, H, device=DEV) + 3.0
    h[0] = 5.0 + 1e-3 * torch.randn(H, device=DEV)
    w, b = (torch.randn(H, device=DEV).to(dtype) for _ in range(2))
    before = h.clone()
    y = kernels.stream_update(h, [], dtype, next_norm=(w, b, 1e-3))
    tol = 3e-5 if dtype == torch.float32 else 6e-3
    want = ref_layer_norm(h, w, b, 1e-3)
    assert rel(y, want) < tol and torch.equal(h, before)
    rows = torch.tensor([T - 1, 0], dtype=torch.int32, device=DEV)
    y2 = kernels.stream_update(h, [], dtype, next_norm=(w, b, 1e-3), rows=rows)
    assert rel(y2, want[rows.long()]) < tol


@pytest.mark.parametrize("T,H,parts", [(1, 64, 3), (4, 99, 1), (40, 256, 11), (310, 1024, 1), (3, 2048, 15), (300, 1500, 2), (305, 3000, 1), (2, 4104, 3), (300, 4200, 1)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_update_sums_gates_norms_and_hands_on(T, H, parts, dtype):
    """The routed rows with identity experts, a gated stack of partial sums, both together, an update normed before it is added,
    the three things left for the next reader."""
    from rocmforge_b200 import kernels
    torch.manual_seed(H + parts)
    top, experts = 3, 4
    h0 = torch.randn(T, H, device=DEV)
    dense = torch.randn(parts, T, H, device=DEV)
    logits = torch.randn(T, 5, device=DEV)[:, 2]
    idx = torch.randint(0, experts + 2, (T, top), dtype=torch.int32, device=DEV)
    idx[0] = i32(experts, experts + 1, 0)[:top]
    order = torch.argsort(idx.reshape(-1), stable=True)
    inv = torch.empty_like(order)
    inv[order] = torch.arange(T * top, device=DEV)
    inv = inv.to(torch.int32)
    rows = torch.randn(T * top, H, device=DEV)
    rows[idx.reshape(-1)[order] >= experts] = float("nan")        # identity experts have no rows
    wts = torch.rand(T, top, device=DEV)
    x = torch.randn(T, H + 8, device=DEV).to(dtype)[:, :H]
    routed = kernels.RoutedSum(rows, inv, idx, wts, x, experts)
    per = torch.where((idx < experts)[:, :, None], rows[inv.long()].view(T, top, H).double(), x.double()[:, None, :])
    want_routed = (per * wts.double()[:, :, None]).sum(1)
    gate = torch.sigmoid(logits.double())[:, None]
    w, b, wp = (torch.randn(H, device=DEV).to(dtype) for _ in range(3))
    tol, ytol = 2e-6, (3e-5 if dtype == torch.float32 else 6e-3)
    for addends, want in (([routed], want_routed), ([kernels.GatedRows(dense, logits)], gate * dense.double().sum(0)),
                          ([routed, kernels.GatedRows(dense, logits)], want_routed + gate * dense.double().sum(0)), ([dense], dense.double().sum(0))):
        h = h0.clone()
        y = kernels.stream_update(h, addends, dtype, next_norm=(w, b, 1e-5))
        assert rel(h, h0.double() + want) < tol
        assert rel(y, ref_layer_norm(h0.double() + want, w, b, 1e-5)) < ytol
    h = h0.clone()
    y = kernels.stream_update(h, [dense], dtype, post=(wp, 1e-2), rounded=True)
    want = h0.double() + P.unit_rms(dense.double().sum(0), 1e-2) * wp.double()
    assert rel(h, want) < tol and torch.equal(y, h.to(dtype))
    h = h0.clone()
    assert kernels.stream_update(h, [dense], dtype, post=(wp, 1e-2)) is None and rel(h, want) < tol
    h = h0.clone()
    y = kernels.stream_update(h, [dense], dtype, post=(wp, 1e-2), next_norm=(w, b, 1e-5))
    assert rel(y, ref_layer_norm(want, w, b, 1e-5)) < ytol


@pytest.mark.parametrize("dim,width,layers,index", [(5, 8, 3, 2), (16, 16, 4, 0), (1, 8, 2, 1), (24, 24, 1, 0)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_side_gate(dim, width, layers, index, dtype):
    from rocmforge_b200 import kernels
    torch.manual_seed(dim)
    T, vocab = 37, 50
    table = torch.randn(vocab, layers * dim, device=DEV).to(dtype)
    tokens = torch.randint(0, vocab, (T,), dtype=torch.int32, device=DEV)
    e = table[tokens.long()][:, index * dim:(index + 1) * dim].double()
    z = (2.0 * torch.randn(T, width, device=DEV)).to(dtype)
    parts = torch.randn(4, T, width, device=DEV)
    for src, x in ((z, z.double()), (parts, parts.double().sum(0))):
        got = kernels.side_gate(src, table, index * dim, dim, tokens, width)
        want = P.gelu_by_tanh(x[:, :dim]) * e
        assert got.shape == (T, width) and rel(got[:, :dim], want) < (2e-6 if dtype == torch.float32 else 5e-3)
        assert not got[:, dim:].any()


# --------------------------------------------------------------------------- gated units

@pytest.mark.parametrize("M,K,ff", [(1, 64, 40), (9, 256, 136), (70, 512, 300), (128, 128, 64), (200, 256, 512), (600, 320, 384), (5, 100, 30)])
@pytest.mark.parametrize("activation", ["gelu_tanh", "clamped_glu"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_units_in_every_product(M, K, ff, activation, dtype):
    """Few tokens, up to 128, more; widths that the clustered product takes and does not; limits that bite on both sides."""
    from rocmforge_b200 import kernels
    from rocmforge_b200.engine.context import Options, StepContext
    from rocmforge_b200.parts.linear import Linear
    torch.manual_seed(M + K)
    x = torch.randn(M, K, device=DEV).to(dtype)
    g, u = ((2.0 * torch.randn(ff, K, device=DEV) / math.sqrt(K)).to(dtype) for _ in range(2))
    ctx = StepContext.__new__(StepContext)
    ctx.options, ctx.compute_dtype = Options(), dtype
    w = Linear(torch.stack([g, u], dim=1).reshape(2 * ff, K).contiguous())
    kw = dict(limit=1.3, alpha=1.702) if activation == "clamped_glu" else {}
    got = ctx.gated_activation(x, w, activation, **kw)
    zg, zu = x.double() @ g.double().T, x.double() @ u.double().T
    if activation == "gelu_tanh":
        want = P.gelu_by_tanh(zg) * zu
    else:
        c = torch.clamp(zg, max=1.3)
        want = c * torch.sigmoid(1.702 * c) * (torch.clamp(zu, -1.3, 1.3) + 1.0)
    assert (zg > 1.3).any() and (zu < -1.3).any()
    assert rel(got, want) < (1e-5 if dtype == torch.float32 else 8e-3)
    if dtype == torch.bfloat16:
        kernels.tensor_core.check_status("cuda:0")


# --------------------------------------------------------------------------- routing

ROUTES = [(6, 2, 3, 2, 1.7), (18, 4, 6, 2, 0.5), (12, 3, 4, 1, 1.0), (64, 8, 8, 4, 2.5), (7, 7, 1, 1, 1.0), (8, 2, 8, 2, 3.0),
          (100, 16, 20, 7, 1.0), (1024, 5, 64, 3, 1.0), (1000, 16, 1000, 16, 1.0)]


@pytest.mark.parametrize("E,top,groups,keep,scale", ROUTES)
def test_choice_among_the_best_groups(E, top, groups, keep, scale):
    """Choice scores that are mostly negative (an excluded expert that counted as 0 would be chosen), corrections that change
    the choice but not the weights, rows with a stride."""
    from rocmforge_b200 import kernels
    torch.manual_seed(E + top)
    T = 203
    z = (2.0 * torch.randn(T, E + 3, device=DEV))[:, :E]
    corr = torch.randn(E, device=DEV) * 0.3 - 1.0
    idx, w = kernels.moe_route_grouped(z, corr, top, groups=groups, keep=keep, scale=scale)
    s = torch.softmax(z.double().cpu(), dim=-1)
    c = s + corr.double().cpu()
    margin = P.choice_margin(c, top, {"count": groups, "keep": keep})
    chosen = P.limit_to_groups(c, groups, keep).topk(top, dim=-1).indices
    clear = margin > 1e-6
    assert clear.double().mean() > 0.9
    assert torch.equal(idx.cpu().long()[clear].sort(-1).values, chosen[clear].sort(-1).values)
    own = s.gather(1, idx.cpu().long())
    want = own / (own.sum(-1, keepdim=True) + 1e-20) * scale
    assert float((w.cpu().double() - want).abs().max()) < 2e-6 * scale
    order = c.gather(1, idx.cpu().long())
    assert (order[:, :-1] - order[:, 1:] > -1e-6).all()              # the choices come best first


def test_equal_choice_scores_take_the_lower_index():
    from rocmforge_b200 import kernels
    idx, w = kernels.moe_route_grouped(torch.zeros(2, 12, device=DEV), torch.zeros(12, device=DEV), 3, groups=4, keep=2)
    assert idx.tolist() == [[0, 1, 2]] * 2 and torch.allclose(w, torch.full_like(w, 1 / 3))


def test_a_group_counts_by_its_largest_member():
    """Group 1 holds the largest sum but not the largest member, so it is closed."""
    from rocmforge_b200 import kernels
    corr = torch.tensor([-0.1, -5.0, -0.2, -0.21, -4.0, 0.3], device=DEV)
    idx, _ = kernels.moe_route_grouped(torch.zeros(1, 6, device=DEV), corr, 2, groups=3, keep=2)
    assert idx.tolist() == [[5, 0]]


@pytest.mark.parametrize("T,E,identity,top", [(1, 3, 1, 2), (40, 5, 2, 3), (300, 12, 4, 2), (17, 1, 7, 2), (9, 4, 0, 1)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sorted_pairs_leave_identity_experts_out(T, E, identity, top, dtype):
    from rocmforge_b200 import kernels
    torch.manual_seed(T + E)
    idx = torch.stack([torch.randperm(E + identity, device=DEV)[:top] for _ in range(T)]).to(torch.int32)
    if T == 40:
        idx[:] = torch.arange(E, E + identity, device=DEV).repeat(2)[:top].to(torch.int32)      # nobody uses a real expert
    perm, inv, tiles, max_tiles, n_active = kernels.moe_sort_passive(idx, E, identity, 16)
    flat = idx.reshape(-1)
    real = int((flat < E).sum())
    assert int(n_active) == real
    assert torch.equal(flat[perm.long()].sort().values, flat[perm.long()]) and torch.equal(perm[inv.long()].cpu(), torch.arange(T * top, dtype=torch.int32))
    tl = tiles.cpu().tolist()
    covered = []
    for e, a, b in zip(*[iter(tl[1:1 + 3 * tl[0]])] * 3):
        assert e < E and 0 < b - a <= 16 and (flat[perm[a:b].long()] == e).all()
        covered += range(a, b)
    assert covered == list(range(real)) and tl[0] <= max_tiles
    H = 24
    x = torch.randn(T, H, device=DEV).to(dtype)
    y = torch.full((T * top, H), float("nan"), device=DEV)
    y[:real] = torch.randn(real, H, device=DEV)
    w = torch.rand(T, top, device=DEV)
    got = kernels.moe_combine(y, inv, w, identity=(idx, E, x))
    want = torch.zeros(T, H, dtype=torch.float64, device=DEV)
    for k in range(top):
        row = torch.where((idx[:, k] < E)[:, None], y[inv.view(T, top)[:, k].long()].double(), x.double())
        want += w[:, k].double()[:, None] * row
    assert rel(got, want) < 1e-6
    g = kernels.moe_gather(x, perm, top, n_active=n_active)
    assert torch.equal(g[:real], x[perm.long()[:real] // top])


# --------------------------------------------------------------------------- linear attention with a fixed decay

@pytest.mark.parametrize("W", [64, 100, 33])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_silu_columns_and_the_joint_norm(W, dtype):
    from rocmforge_b200 import kernels
    torch.manual_seed(W)
    T = 21
    p = (3.0 * torch.randn(T, W + 40, device=DEV)).to(dtype)
    parts = torch.randn(5, T, W + 40, device=DEV)
    for src, x in ((p, p.double()), (parts, parts.double().sum(0))):
        assert rel(kernels.silu_columns(src[..., :W]), P.silu(x[:, :W])) < 1e-6
        o = torch.randn(T, W, device=DEV) * torch.rand(T, 1, device=DEV)
        w = torch.randn(W, device=DEV).to(dtype)
        for fn, gate in (("sigmoid", torch.sigmoid), ("silu", P.silu)):
            got = kernels.row_norm_gate(o, src[..., 40:], 1e-4, w, dtype, gate_fn=fn)
            want = P.unit_rms(o.double(), 1e-4) * w.double() * gate(x[:, 40:])
            assert rel(got, want) < (3e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("heads,dim,vdim,decay", [(2, 24, 12, [0.5, 1.0]), (3, 64, 64, [0.0, 0.9, 0.999]), (1, 256, 20, [0.97])])
def test_fixed_decay_in_portions_and_chunks(heads, dim, vdim, decay):
    """q, k and v as neighbouring columns of one matrix (rows with a stride), two sequences of unequal length, the state carried
    from portion to portion, decays of 0 and 1: the scan and the chunked kernels against the recurrence in float64."""
    from rocmforge_b200 import kernels
    torch.manual_seed(dim)
    qk, vs = heads * dim, heads * vdim
    lens = [150, 7]
    a = torch.randn(sum(lens), 2 * qk + vs, device=DEV) * 0.5
    dec = torch.tensor(decay, dtype=torch.float32, device=DEV)
    want = []
    at = 0
    for n in lens:
        r = a[at:at + n].double().cpu()
        want.append(torch.cat([P.fixed_decay_recurrence(r[:, h * dim:(h + 1) * dim], r[:, qk + h * dim: qk + (h + 1) * dim],
                                                        r[:, 2 * qk + h * vdim: 2 * qk + (h + 1) * vdim], decay[h])[0] for h in range(heads)], dim=1))
        at += n

    def run(rows, cu, state, slots, table):
        q, k, v = a[rows, :qk], a[rows, qk:2 * qk], a[rows, 2 * qk:]
        sub = a[rows]
        q, k, v = sub[:, :qk], sub[:, qk:2 * qk], sub[:, 2 * qk:]
        if table is None:
            return kernels.retention_scan((q, k), v, state, dec, i32(*cu), i32(*slots), heads, dim, vdim)
        return kernels.retention_chunked((q, k), v, state, dec, i32(*table), i32(*cu), i32(*slots), heads, dim, vdim)
    for chunked in (False, True):
        state = torch.zeros(3, heads, vdim, dim, device=DEV)
        got0, got1 = [], []
        # the first sequence in portions of 70, 1, 64 and 15 tokens, the second beside the first portion
        table = [0, 2, 3, 0, 0, 0, 64, 1, 0] if chunked else None
        o = run(torch.cat([torch.arange(70), torch.arange(150, 157)]).to(DEV), [0, 70, 77], state, [2, 0], table)
        got0.append(o[:70]); got1.append(o[70:])
        for s, e in ((70, 71), (71, 135), (135, 150)):
            got0.append(run(torch.arange(s, e, device=DEV), [0, e - s], state, [2], [0, 1, 0, 0] if chunked else None))
        assert rel(torch.cat(got0).cpu(), want[0]) < 2e-5 and rel(torch.cat(got1).cpu(), want[1]) < 2e-5, f"chunked {chunked}"
        assert not state[1].any()


# --------------------------------------------------------------------------- the delta rule with one decay per head

@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 24, 12), (3, 3, 64, 40), (1, 1, 256, 8), (2, 1, 128, 128), (2, 2, 1, 5)])
def test_per_head_decays(H, G, dim, vdim):
    """The prepared inputs, and the scan in portions, against the recurrence in float64; decays of exactly 0 and 1 among them;
    one token a sequence on the other kernel form."""
    from rocmforge_b200 import kernels
    torch.manual_seed(dim + H)
    lens = [61, 9]
    T = sum(lens)
    qkv = torch.randn(T, 2 * G * dim + H * vdim, device=DEV)
    ab = torch.randn(T, 2 * H + 3, device=DEV) * 2.0
    dt, al = torch.randn(H, device=DEV), torch.randn(H, device=DEV)
    qn, kn, kq, decay, beta = kernels.delta_prepare(qkv, ab[:, H:2 * H], dt, al, ab[:, :H], H, G, dim, dim ** -0.5, 1e-6)
    q = P.unit_vector(qkv[:, :G * dim].double().view(T, G, dim)) * dim ** -0.5
    k = P.unit_vector(qkv[:, G * dim:2 * G * dim].double().view(T, G, dim))
    want_g = torch.exp(-torch.exp(al.double()) * torch.nn.functional.softplus(ab[:, H:2 * H].double() + dt.double()))
    assert decay.shape == (T, H) and rel(decay, want_g) < 1e-5 and rel(beta, torch.sigmoid(ab[:, :H].double())) < 1e-6
    assert rel(qn.view(T, G, dim), q) < 1e-5 and rel(kn.view(T, G, dim), k) < 1e-5 and float((kq.double() - (q * k).sum(-1)).abs().max()) < 1e-5
    decay[5], decay[40] = 0.0, 1.0
    v = qkv[:, 2 * G * dim:]
    want, ends = [], []
    for a, b in ((0, 61), (61, 70)):
        pairs = [P.corrected_recurrence(q[a:b, h // (H // G)].cpu(), k[a:b, h // (H // G)].cpu(), v[a:b, h * vdim:(h + 1) * vdim].double().cpu(),
                                        beta[a:b, h].double().cpu(), decay[a:b, h].double().cpu()) for h in range(H)]
        want.append(torch.cat([o for o, _ in pairs], dim=1)); ends.append(torch.stack([s for _, s in pairs]))

    def run(rows, cu, slots, state, one=False):
        r = rows.to(DEV)
        return kernels.delta_scan(qn[r], kn[r], kq[r], decay[r], beta[r], v[r], state, i32(*cu), i32(*slots), H, G, dim, vdim, one_token=one)
    state = torch.zeros(3, H, dim, vdim, device=DEV)
    got0, got1 = [], []
    o = run(torch.cat([torch.arange(30), torch.arange(61, 70)]), [0, 30, 39], [1, 2], state)
    got0.append(o[:30]); got1.append(o[30:])
    got0.append(run(torch.arange(30, 31), [0, 1], [1], state, one=True))
    got0.append(run(torch.arange(31, 33), [0, 2], [1], state))
    got0.append(run(torch.arange(33, 61), [0, 28], [1], state))
    assert rel(torch.cat(got0).cpu(), want[0]) < 2e-5 and rel(torch.cat(got1).cpu(), want[1]) < 2e-5
    assert rel(state[1].cpu(), ends[0]) < 2e-5 and rel(state[2].cpu(), ends[1]) < 2e-5 and not state[0].any()


@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 24, 12), (3, 3, 64, 40), (1, 1, 256, 8), (2, 1, 128, 128), (2, 2, 1, 5), (1, 1, 130, 70), (2, 1, 30, 33), (1, 1, 200, 20),
                                          (2, 2, 128, 36)])
def test_the_delta_rule_in_chunks(H, G, dim, vdim):
    """Prompts in chunks of 64 against the recurrence in float64: sequences of a whole number of chunks, of one token more, of a
    few tokens, side by side; a continued state; decays of exactly 0 and 1 and tiny ones at chunk borders; keys that repeat (the
    system is then far from the identity)."""
    from rocmforge_b200 import kernels
    torch.manual_seed(dim + H)
    lens = [129, 64, 3, 200]
    T = sum(lens)
    q = torch.randn(T, G * dim, device=DEV) * dim ** -0.5
    k = P.unit_vector(torch.randn(T, G, dim, device=DEV))
    k[20:60] = k[20:21]
    k[150:158] = k[150:151]
    k = k.reshape(T, G * dim).contiguous()
    wide = torch.randn(T, 3 + H * vdim, device=DEV)
    v = wide[:, 3:]
    beta = torch.rand(T, H, device=DEV)
    decay = torch.rand(T, H, device=DEV) ** 0.2
    for t, g in ((0, 0.0), (5, 1.0), (63, 0.0), (64, 1e-30), (65, 1e-30), (128, 1.0), (193, 0.0), (260, 1.0)):
        decay[t] = g
    decay[300:340] = 1.0
    starts = [sum(lens[:i]) for i in range(4)]
    state = torch.zeros(6, H, dim, vdim, device=DEV)
    begin = torch.randn(H, dim, vdim, device=DEV)
    state[4] = begin
    slots = [1, 4, 0, 3]

    def reference(i):
        a, b = starts[i], starts[i] + lens[i]
        outs, ends = [], []
        for h in range(H):
            g = h // (H // G)
            o, S = P.corrected_recurrence(q[a:b, g * dim:(g + 1) * dim].double().cpu(), k[a:b, g * dim:(g + 1) * dim].double().cpu(),
                                          v[a:b, h * vdim:(h + 1) * vdim].double().cpu(), beta[a:b, h].double().cpu(), decay[a:b, h].double().cpu(),
                                          begin[h].double().cpu() if slots[i] == 4 else None)
            outs.append(o); ends.append(S)
        return torch.cat(outs, dim=1), torch.stack(ends)
    refs = [reference(i) for i in range(4)]
    scan_state = state.clone()

    def run(parts, cut):
        """The sequences' tokens cut[i] .. parts[i] as one step."""
        rows = torch.cat([torch.arange(starts[i] + cut[i], starts[i] + parts[i]) for i in range(4) if parts[i] > cut[i]]).to(DEV)
        live = [i for i in range(4) if parts[i] > cut[i]]
        ns = [parts[i] - cut[i] for i in live]
        counts = [(n + 63) // 64 for n in ns]
        table = [sum(counts[:j]) for j in range(len(live) + 1)] + [x for j, n in enumerate(ns) for r in range(0, n, 64) for x in (j, r)]
        cu = [sum(ns[:j]) for j in range(len(ns) + 1)]
        o = kernels.delta_chunked(q[rows], k[rows], decay[rows], beta[rows], v[rows], state, i32(*table), i32(*cu), i32(*[slots[i] for i in live]),
                                  H, G, dim, vdim)
        return {i: o[cu[j]:cu[j + 1]] for j, i in enumerate(live)}
    first = run([70, 64, 3, 100], [0, 0, 0, 0])
    second = run([129, 64, 3, 200], [70, 64, 3, 100])
    for i in range(4):
        got = torch.cat([first[i]] + ([second[i]] if i in second else [])).cpu()
        assert rel(got, refs[i][0]) < 5e-5, f"sequence {i}: {rel(got, refs[i][0]):.1e}"
        assert rel(state[slots[i]].cpu(), refs[i][1]) < 5e-5, f"state of sequence {i}"
    assert not state[2].any() and not state[5].any()
    kernels.tensor_core.check_status("cuda:0")
    kq = (q.view(T, G, dim) * k.view(T, G, dim)).sum(-1).contiguous()
    scan = kernels.delta_scan(q, k, kq, decay, beta, v, scan_state, i32(0, 129, 193, 196, 396), i32(*slots), H, G, dim, vdim)
    assert rel(scan.cpu(), torch.cat([r[0] for r in refs])) < 5e-5


# --------------------------------------------------------------------------- attention with capped scores, every key visible

def paged(k, v, extra=2):
    T, nkv, d = k.shape
    n = (T + 63) // 64
    order = torch.randperm(n + extra)[:n]
    kp = torch.full((n + extra, nkv, 64, d), float("nan"), device=DEV, dtype=k.dtype)
    vp = torch.full((n + extra, nkv, 64, v.shape[2]), float("nan"), device=DEV, dtype=v.dtype)
    for p in range(n):
        a, b = 64 * p, min(T, 64 * p + 64)
        kp[order[p], :, :b - a], vp[order[p], :, :b - a] = k[a:b].transpose(0, 1), v[a:b].transpose(0, 1)
    return kp, vp, order.to(torch.int32).to(DEV).reshape(1, n)


@pytest.mark.parametrize("d,dv,dtype", [(64, 64, torch.bfloat16), (128, 128, torch.bfloat16), (20, 12, torch.float32), (64, 128, torch.bfloat16)])
@pytest.mark.parametrize("i,far", [(299, 0), (299, 63), (299, 64), (64, 0), (191, 127), (128, 128), (299, 298), (63, 1)])
def test_one_far_key_stands_out(d, dv, dtype, i, far):
    """A key among up to three hundred holds a query's whole weight, and the key after the query would win if it were seen: in
    a prompt (every query of it) and as a step of its own, on the prompt, the decode and the generic kernel."""
    from rocmforge_b200 import kernels
    nh, nkv, T, cap, scale = 8, 2, 300, 12.0, 0.3
    torch.manual_seed(i * 301 + far)
    q, k, v = torch.randn(T, nh, d, device=DEV) * 0.1, torch.randn(T, nkv, d, device=DEV) * 0.1, torch.randn(T, nkv, dv, device=DEV)
    q[i] = 0.0
    q[i, :, 0] = 30.0
    k[far, :, 0] = 4.0                                    # a score far in the cap's flat part
    if i + 1 < T:
        k[i + 1, :, 0], v[i + 1] = 8.0, 1000.0
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    kp, vp, bt = paged(k, v)
    see = torch.arange(T, device=DEV)[None, :] <= torch.arange(T, device=DEV)[:, None]

    def reference(rows):
        out = []
        for h in range(nh):
            s = P.capped(q[rows, h].double() @ k[:, h // 4].double().T * scale, cap).masked_fill(~see[rows], float("-inf"))
            out.append(torch.softmax(s, dim=-1) @ v[:, h // 4].double())
        return torch.stack(out, dim=1)
    tol = 1e-5 if dtype == torch.float32 else 2e-2
    zero = i32(0)
    n = i + 1
    rows = torch.arange(n, device=DEV)
    pos, seq = rows.to(torch.int32), torch.zeros(n, dtype=torch.int32, device=DEV)
    flat = q[:n].reshape(n, nh * d).contiguous()
    want = reference(rows)
    assert float((want[-1] - v[far].double().repeat_interleave(4, 0)).abs().max()) < 0.1
    outs = [kernels.attention_generic(flat, nh, nkv, d, kp, vp, seq, pos, zero, bt, scale, None, v_head_dim=dv, softcap=cap)]
    if d == dv and dtype == torch.bfloat16:
        tiles = i32(*[x for r in range(0, n, 128) for x in (0, r)])
        outs.append(kernels.attention_prefill_tc(flat, nh, nkv, d, kp, vp, tiles, zero, zero, i32(n), i32(0, n), bt, scale, None, softcap=cap))
    for o in outs:
        assert rel(o.reshape(n, nh, dv), want) < tol
    one = q[i:i + 1].reshape(1, nh * d).contiguous()
    outs = [kernels.attention_generic(one, nh, nkv, d, kp, vp, zero, i32(i), zero, bt, scale, None, v_head_dim=dv, softcap=cap)]
    if d == dv and dtype == torch.bfloat16:
        for splits in (1, 4):
            outs.append(kernels.attention_decode_warps(one, nh, nkv, d, kp, vp, zero, i32(i), zero, bt, scale, None, splits=splits, softcap=cap))
    for o in outs:
        assert rel(o.reshape(1, nh, dv), want[-1:]) < tol
    kernels.tensor_core.check_status("cuda:0")


@pytest.mark.parametrize("hd,rot,partials", [(16, 8, False), (64, 64, True), (20, 20, False), (12, 0, True)])
def test_heads_are_normed_before_their_rotation(hd, rot, partials):
    """RMS norm with a weight each for q and k, then the first ``rot`` elements turn as pairs (i, i + rot/2); values untouched."""
    from rocmforge_b200 import kernels
    torch.manual_seed(hd)
    T, nh, nkv, hv = 9, 4, 2, 10
    x = torch.randn(3 if partials else 1, T, (nh + nkv) * hd + nkv * hv, device=DEV)
    wq, wk = torch.randn(hd, device=DEV), torch.randn(hd, device=DEV)
    pos = torch.randint(0, 120, (T,), device=DEV).to(torch.int32).sort().values
    pos[:] = torch.arange(50, 50 + T, device=DEV)
    kp, vp = torch.zeros(3, nkv, 64, hd, device=DEV), torch.zeros(3, nkv, 64, hv, device=DEV)
    bt = i32(2, 0).view(1, 2)
    inv = torch.tensor([1000.0 ** (-2.0 * j / rot) for j in range(rot // 2)], dtype=torch.float32, device=DEV) if rot else None
    got = kernels.head_norm_kv_write(x if partials else x[0], nh, nkv, hd, hv, inv, torch.zeros(T, dtype=torch.int32, device=DEV), pos, i32(0),
                                     bt, kp, vp, True, compute_dtype=torch.float32, rot_dim=rot, interleaved=False, unit_norm_eps=1e-3,
                                     q_norm_weight=wq, k_norm_weight=wk)
    r = x.double().sum(0).cpu()
    cut = [nh * hd, (nh + nkv) * hd]

    def turned(y, w):
        return P.turn_pairs(P.unit_rms(y, 1e-3) * w.double().cpu(), pos.cpu(), rot, 1000.0)
    q = turned(r[:, :cut[0]].view(T, nh, hd), wq)
    k = turned(r[:, cut[0]:cut[1]].view(T, nkv, hd), wk)
    v = r[:, cut[1]:].view(T, nkv, hv)
    assert rel(got.cpu().view(T, nh, hd), q) < 1e-5
    for t in range(T):
        p = int(pos[t])
        page = int(bt[0, p // 64])
        assert float((kp[page, :, p % 64].cpu().double() - k[t]).abs().max()) < 1e-5
        assert float((vp[page, :, p % 64].cpu().double() - v[t]).abs().max()) < 1e-6
