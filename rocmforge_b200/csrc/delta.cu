// The gated delta rule: a matrix state per head that decays per key channel and is corrected, not just added to:
//   S <- diag(g_t) S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t      (S is [dim, vdim])
// so the read-out sees the token's own write.  With S' = diag(g_t) S both products that a token needs are taken from S'
// in one pass over the state, r_k = S'^T k_t and r_q = S'^T q_t, because o_t = r_q + (k_t . q_t) u_t; the state is read
// once and written once per token.  Everything here is 32-bit.
//
//   delta_prepare  q and k heads made unit vectors (x / sqrt(sum x^2 + unit_eps), q also times q_scale), their dot
//                  products k . q, beta = sigmoid of the projection's columns, and the decays
//                  g = exp(-exp(A_log_h) softplus(a + dt_bias)) per head and key channel (or one per head)
//   delta_scan     the recurrence, token by token.  A block owns (sequence, head, 32 value columns): the columns of S are
//                  independent of each other, so blocks never talk.  Four lanes share a column, each with a quarter of
//                  its rows in registers over the step's tokens; per token their partial r_k and r_q meet by shuffles.
//                  The order of every sum is fixed by (dim, position) alone: how a prompt is cut into steps and what
//                  else is in the batch change no bit.
//   delta_chunk_*  the same recurrence for prompts, with one decay per head and token: chunks of 64 tokens, see below
#include <type_traits>
#include "tcgen05_common.cuh"

#define DL_WARPS 4

template <typename T>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const float* __restrict__ qkv, int qkv_stride, const float* __restrict__ a, int a_stride, const void* __restrict__ dt_bias,
                     const void* __restrict__ a_log, int vec_is_f32, const T* __restrict__ beta_src, int beta_stride,
                     float* __restrict__ qn, float* __restrict__ kn, float* __restrict__ kq, float* __restrict__ decay,
                     float* __restrict__ beta, int H, int G, int D, int per_head, float q_scale, float unit_eps) {
    pdl_trigger();
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
    pdl_wait();
    const float* row = qkv + (size_t)t * qkv_stride;
    // few tokens: a token's heads and channels are spread over gridDim.y blocks
    for (int g = blockIdx.y * nwarp + warp; g < G; g += gridDim.y * nwarp) {                 // a warp per q/k head
        const float* q = row + g * D;
        const float* k = row + (G + g) * D;
        float sq = 0.f, sk = 0.f, dot = 0.f;
        for (int e = lane; e < D; e += 32) { const float x = q[e], y = k[e]; sq += x * x; sk += y * y; dot += x * y; }
        sq = warp_sum(sq); sk = warp_sum(sk); dot = warp_sum(dot);
        const float rq = q_scale / sqrtf(sq + unit_eps), rk = 1.f / sqrtf(sk + unit_eps);
        for (int e = lane; e < D; e += 32) {
            qn[((size_t)t * G + g) * D + e] = q[e] * rq;
            kn[((size_t)t * G + g) * D + e] = k[e] * rk;
        }
        if (lane == 0) kq[(size_t)t * G + g] = dot * rq * rk;
    }
    const int ND = per_head ? H : H * D;                 // decays of a token
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < ND; i += gridDim.y * blockDim.x) {
        const int h = per_head ? i : i / D;
        const float x = a[(size_t)t * a_stride + i] + load_vec(dt_bias, vec_is_f32, i);
        const float sp = fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
        decay[(size_t)t * ND + i] = expf(-expf(load_vec(a_log, vec_is_f32, h)) * sp);
    }
    for (int h = blockIdx.y * blockDim.x + threadIdx.x; h < H; h += gridDim.y * blockDim.x)
        beta[(size_t)t * H + h] = 1.f / (1.f + expf(-Cvt<T>::to_f32(beta_src[(size_t)t * beta_stride + h])));
}

// grid (ceil(vdim / COLS), heads, sequences); 128 threads.  LPC lanes share a value column (a warp owns 32 / LPC columns, a
// block COLS = 128 / LPC); DP = LPC * ROWS >= dim, a multiple of 4 LPC; rows beyond dim hold zeros.  Of every 4 LPC rows of
// the state the lane with number rg inside its column holds rows 4 rg .. 4 rg + 3, so that the lanes' 16-byte reads of q, k
// and the decays from shared memory lie in a row.  A column's partial products meet by log2(LPC) shuffles; the warps of a block never wait for each other
// inside a stage.  The tokens' q, k, decays, values, beta and k . q are copied asynchronously, a stage of TOK tokens
// ahead of the arithmetic.
__device__ __forceinline__ void dl_copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void dl_copy4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// PER_HEAD: the decay is one number per (token, head) instead of one per key channel.
template <int ROWS, int LPC, bool PER_HEAD>
__global__ void __launch_bounds__(DL_WARPS * 32)
delta_scan_kernel(const float* __restrict__ qn, const float* __restrict__ kn, const float* __restrict__ kq,
                  const float* __restrict__ decay, const float* __restrict__ beta, const float* __restrict__ v, int v_stride,
                  float* __restrict__ state, float* __restrict__ o, const int* __restrict__ cu_q,
                  const int* __restrict__ seq_slot, int H, int G, int D, int V) {
    constexpr int DP = LPC * ROWS;                                   // rows of the padded state
    constexpr int COLS = DL_WARPS * 32 / LPC;                        // value columns of a block
    constexpr int TOK = DP <= 64 ? 16 : (DP <= 128 ? 8 : 4);         // tokens of a stage
    constexpr int NT = DL_WARPS * 32;
    constexpr int GP = PER_HEAD ? 4 : DP;                            // decays of a token
    __shared__ __align__(16) float sk[2][TOK][DP], sq[2][TOK][DP], sg[2][TOK][GP];
    __shared__ __align__(16) float sv[2][TOK][COLS];
    __shared__ float sb[2][TOK], skq[2][TOK];
    pdl_trigger();
    const int b = blockIdx.z, h = blockIdx.y, j0 = blockIdx.x * COLS;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int rg = lane % LPC, cl = warp * (32 / LPC) + lane / LPC;            // this lane's rows inside every 16, its column in the block
    const int hg = h / (H / G);
    const int t0 = cu_q[b], n = cu_q[b + 1] - t0;
    const int col = j0 + cl;
    const bool live = col < V;
    float* S = state + ((size_t)seq_slot[b] * H + h) * D * V;
    // what no copy ever writes: rows beyond dim (k = q = 0, decay 1) and columns beyond vdim (value 0)
    for (int i = tid; i < 2 * TOK * DP; i += NT) {
        const int d = i % DP;
        if (d >= D) {
            (&sk[0][0][0])[i] = 0.f; (&sq[0][0][0])[i] = 0.f;
            if constexpr (!PER_HEAD) (&sg[0][0][0])[i] = 1.f;
        }
    }
    for (int i = tid; i < 2 * TOK * COLS; i += NT)
        if (j0 + i % COLS >= V) (&sv[0][0][0])[i] = 0.f;
    const bool vec = (D & 3) == 0;
    pdl_wait();
    auto stage_in = [&](int base, int buf) {
        const int cnt = min(TOK, n - base);
        if (vec) {
            const int dq = D >> 2;
            for (int i = tid; i < cnt * dq; i += NT) {
                const int tt = i / dq, d = (i - tt * dq) * 4;
                const size_t t = (size_t)(t0 + base + tt);
                dl_copy16(&sk[buf][tt][d], kn + (t * G + hg) * D + d);
                dl_copy16(&sq[buf][tt][d], qn + (t * G + hg) * D + d);
                if constexpr (!PER_HEAD) dl_copy16(&sg[buf][tt][d], decay + (t * H + h) * D + d);
            }
        } else {
            for (int i = tid; i < cnt * D; i += NT) {
                const int tt = i / D, d = i - tt * D;
                const size_t t = (size_t)(t0 + base + tt);
                dl_copy4(&sk[buf][tt][d], kn + (t * G + hg) * D + d);
                dl_copy4(&sq[buf][tt][d], qn + (t * G + hg) * D + d);
                if constexpr (!PER_HEAD) dl_copy4(&sg[buf][tt][d], decay + (t * H + h) * D + d);
            }
        }
        const int nc = min(COLS, V - j0);
        for (int i = tid; i < cnt * nc; i += NT) {
            const int tt = i / nc, c = i - tt * nc;
            dl_copy4(&sv[buf][tt][c], v + (size_t)(t0 + base + tt) * v_stride + h * V + j0 + c);
        }
        if (tid < cnt) {
            dl_copy4(&sb[buf][tid], beta + (size_t)(t0 + base + tid) * H + h);
            dl_copy4(&skq[buf][tid], kq + (size_t)(t0 + base + tid) * G + hg);
            if constexpr (PER_HEAD) dl_copy4(&sg[buf][tid][0], decay + (size_t)(t0 + base + tid) * H + h);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float s[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const int i = (r >> 2) * (4 * LPC) + rg * 4 + (r & 3);
        s[r] = (live && i < D) ? S[(size_t)i * V + col] : 0.f;
    }
    if (n > 0) stage_in(0, 0);
    for (int base = 0, buf = 0; base < n; base += TOK, buf ^= 1) {
        const int cnt = min(TOK, n - base);
        if (base + TOK < n) {
            stage_in(base + TOK, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();                                    // this stage's copies of every thread have landed
        float4 g4[ROWS / 4], k4[ROWS / 4], q4[ROWS / 4];
        auto fetch = [&](int tt) {
#pragma unroll
            for (int r = 0; r < ROWS / 4; ++r) {
                if constexpr (PER_HEAD) { const float g = sg[buf][tt][0]; g4[r] = make_float4(g, g, g, g); }
                else g4[r] = *reinterpret_cast<const float4*>(&sg[buf][tt][rg * 4 + r * 4 * LPC]);
                k4[r] = *reinterpret_cast<const float4*>(&sk[buf][tt][rg * 4 + r * 4 * LPC]);
                q4[r] = *reinterpret_cast<const float4*>(&sq[buf][tt][rg * 4 + r * 4 * LPC]);
            }
        };
        for (int tt = 0; tt < cnt; ++tt) {
            fetch(tt);
            float pk[4] = {0.f, 0.f, 0.f, 0.f}, pq[4] = {0.f, 0.f, 0.f, 0.f};
            float4 kc[ROWS / 4];
#pragma unroll
            for (int r = 0; r < ROWS / 4; ++r) {
                kc[r] = k4[r];
                s[4 * r + 0] *= g4[r].x; pk[0] = fmaf(s[4 * r + 0], k4[r].x, pk[0]); pq[0] = fmaf(s[4 * r + 0], q4[r].x, pq[0]);
                s[4 * r + 1] *= g4[r].y; pk[1] = fmaf(s[4 * r + 1], k4[r].y, pk[1]); pq[1] = fmaf(s[4 * r + 1], q4[r].y, pq[1]);
                s[4 * r + 2] *= g4[r].z; pk[2] = fmaf(s[4 * r + 2], k4[r].z, pk[2]); pq[2] = fmaf(s[4 * r + 2], q4[r].z, pq[2]);
                s[4 * r + 3] *= g4[r].w; pk[3] = fmaf(s[4 * r + 3], k4[r].w, pk[3]); pq[3] = fmaf(s[4 * r + 3], q4[r].w, pq[3]);
            }
            float rk = (pk[0] + pk[1]) + (pk[2] + pk[3]), rq = (pq[0] + pq[1]) + (pq[2] + pq[3]);
            const float bt = sb[buf][tt], vt = sv[buf][tt][cl], kqt = skq[buf][tt];
#pragma unroll
            for (int m = 1; m < LPC; m <<= 1) { rk += __shfl_xor_sync(0xffffffffu, rk, m); rq += __shfl_xor_sync(0xffffffffu, rq, m); }
            const float u = bt * (vt - rk);
#pragma unroll
            for (int r = 0; r < ROWS / 4; ++r) {
                s[4 * r + 0] = fmaf(kc[r].x, u, s[4 * r + 0]);
                s[4 * r + 1] = fmaf(kc[r].y, u, s[4 * r + 1]);
                s[4 * r + 2] = fmaf(kc[r].z, u, s[4 * r + 2]);
                s[4 * r + 3] = fmaf(kc[r].w, u, s[4 * r + 3]);
            }
            if (rg == 0 && live) o[(size_t)(t0 + base + tt) * H * V + h * V + col] = fmaf(kqt, u, rq);
        }
        __syncthreads();                                    // the stage is used up: the stage after next may land in it
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const int i = (r >> 2) * (4 * LPC) + rg * 4 + (r & 3);
        if (live && i < D) S[(size_t)i * V + col] = s[r];
    }
}

template <int ROWS, int LPC, bool PER_HEAD>
static int launch_scan(const float* qn, const float* kn, const float* kq, const float* decay, const float* beta, const float* v,
                       int v_stride, float* state, float* o, const int* cu_q, const int* seq_slot, int B, int H, int G, int D,
                       int V, cudaStream_t st) {
    constexpr int COLS = DL_WARPS * 32 / LPC;
    rf_launch(delta_scan_kernel<ROWS, LPC, PER_HEAD>, dim3((V + COLS - 1) / COLS, H, B), dim3(DL_WARPS * 32), 0, st, qn, kn, kq, decay,
              beta, v, v_stride, state, o, cu_q, seq_slot, H, G, D, V);
    RF_LAUNCH_CHECK();
    return 0;
}

extern "C" {
// qkv float [T, qkv_stride]: q heads (G x D), k heads (G x D), then values; a float rows of a_stride, H*D columns; dt_bias [H*D]
// and a_log [H] of one dtype (vec_is_f32); beta_src [T, beta_stride] of dtype, H columns.  Out: qn, kn float [T, G*D], kq float
// [T, G], decay float [T, H*D], beta float [T, H].  per_head: one decay a head, so a, dt_bias and decay have H columns.
int rf_delta_prepare(int dtype, const float* qkv, int qkv_stride, const float* a, int a_stride, const void* dt_bias, const void* a_log,
                     int vec_is_f32, const void* beta_src, int beta_stride, float* qn, float* kn, float* kq, float* decay,
                     float* beta, int H, int G, int D, int per_head, float q_scale, float unit_eps, int T_, cudaStream_t st) {
    if (T_ <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || D <= 0) return RF_ERR_BAD_ARG;
    int by = T_ >= 512 ? 1 : per_head ? (G + 3) / 4 : (H * D + 511) / 512;           // about four decays a thread when there are few tokens
    if (by > 32) by = 32;
    if (dtype == 0)
        rf_launch(delta_prepare_kernel<float>, dim3(T_, by), dim3(128), 0, st, qkv, qkv_stride, a, a_stride, dt_bias, a_log, vec_is_f32,
                  reinterpret_cast<const float*>(beta_src), beta_stride, qn, kn, kq, decay, beta, H, G, D, per_head, q_scale, unit_eps);
    else
        rf_launch(delta_prepare_kernel<__nv_bfloat16>, dim3(T_, by), dim3(128), 0, st, qkv, qkv_stride, a, a_stride, dt_bias, a_log, vec_is_f32,
                  reinterpret_cast<const __nv_bfloat16*>(beta_src), beta_stride, qn, kn, kq, decay, beta, H, G, D, per_head, q_scale, unit_eps);
    RF_LAUNCH_CHECK();
    return 0;
}
// decay float [T, H*D], or (per_head) [T, H]; state float [slots, H, D, V]; v float [T, v_stride] with head h's values at columns h*V..; o float [T, H*V]; cu_q [B+1]
int rf_delta_scan(const float* qn, const float* kn, const float* kq, const float* decay, const float* beta, const float* v,
                  int v_stride, float* state, float* o, const int* cu_q, const int* seq_slot, int B, int H, int G, int D, int V,
                  int per_head, int one_token, int lanes, cudaStream_t st) {
    if (B <= 0) return 0;
    if (lanes != 0 && lanes != 4 && lanes != 8) return RF_ERR_BAD_ARG;
    if (H <= 0 || G <= 0 || H % G || D <= 0 || V <= 0 || H > 65535 || B > 65535) return RF_ERR_BAD_ARG;
#define DL_GO(ROWS, LPC) return (per_head ? launch_scan<ROWS, LPC, true> : launch_scan<ROWS, LPC, false>)(qn, kn, kq, decay, beta, v, v_stride, state, o, cu_q, seq_slot, B, H, G, D, V, st)
    // Steps of one token a sequence (the state is read and written once, nothing else): four lanes a column.  Steps with
    // longer portions: eight lanes a column (twice the blocks, half the chain of each; fetching the next token's operands
    // into registers ahead of the chain was measured and cost more in registers than it hid).  The two forms add a column's products in another order: a difference of rounding between a token
    // decoded alone and the same token inside a portion, none between two cuts into portions.
    const int lpc = lanes > 0 ? lanes : (one_token ? 4 : 8);
    const int rows = (D + 4 * lpc - 1) / (4 * lpc) * 4;        // rows a lane, a multiple of 4
    if (lpc == 4) { if (rows <= 8) DL_GO(8, 4); if (rows <= 16) DL_GO(16, 4); if (rows <= 32) DL_GO(32, 4); if (rows <= 64) DL_GO(64, 4); }
    if (lpc == 8) { if (rows <= 4) DL_GO(4, 8); if (rows <= 8) DL_GO(8, 8); if (rows <= 16) DL_GO(16, 8); if (rows <= 32) DL_GO(32, 8); }
#undef DL_GO
    return RF_ERR_UNSUPPORTED;
}
}

// ---------------------------------------------------------------- prompts: chunks of 64 tokens, one decay per head and token
// With positions t, s inside a chunk of cnt tokens, S0 the state before it, P(s, t) = g_(s+1) ... g_t (P(t, t) = 1) and
// G_t = g_0 ... g_t, the recurrence above says
//     u_t = beta_t v_t - beta_t G_t S0^T k_t - sum_(s<t) A_ts u_s,      A_ts = beta_t P(s, t) (k_s . k_t)
//     o_t = G_t S0^T q_t + sum_(s<=t) P(s, t) (k_s . q_t) u_s,          S_end = G_end S0 + sum_s P(s, end) k_s u_s^T
// so a chunk's u follow from one unit lower triangular system: U = U0 - W S0 with (1 + A) U0 = diag(beta) V and
// (1 + A) W = diag(beta G) K, neither of which needs S0.
//   delta_chunk_solve   (chunks side by side)  A and the scores M_ts = P(s, t) (k_s . q_t); U0 and W by forward substitution, a
//                       thread a column, sixteen rows at a time
//   delta_chunk_carry   (chunk after chunk, a block per sequence, head and 16 value columns)  U = U0 - W S, then the state;
//                       leaves every chunk's start state and U
//   delta_chunk_out     (chunks side by side)  o = [M | G q] [U ; S0]
// Decays are multiplied on as running products, never divided by and never taken the logarithm of: 0 and 1 need no special case.
// Everything is 32-bit.  The chunk table (built on the host with the step) is first[B+1] (index of each sequence's first
// chunk), then (sequence, first row) per chunk.
#define DC 64                 // tokens of a chunk
#define DC_LD 68              // row stride of A: rows start on 16-byte boundaries
#define DC_PLD 17             // row stride of the products inside a block of 16 tokens
#define DC_COLS 256           // columns of a substitution pass
#define DV 16                 // value columns of a carry block
#define DO 64                 // value columns of an out block

struct ChunkPlace { int b, row0, cnt; };
__device__ __forceinline__ ChunkPlace chunk_place(const int* table, const int* cu_q, int B, int c) {
    ChunkPlace p;
    p.b = table[B + 1 + 2 * c];
    p.row0 = cu_q[p.b] + table[B + 2 + 2 * c];
    p.cnt = min(DC, cu_q[p.b + 1] - p.row0);
    return p;
}
// rows [0, 64) x columns [0, n) of src (row stride given) into dst (row stride ld, a multiple of 4), asynchronously; rows from
// cnt on and columns from n to n4 (the next multiple of 4) become zeros.  vec: every row of src starts on a 16-byte boundary.
__device__ __forceinline__ void chunk_tile(float* dst, int ld, const float* src, size_t stride, int cnt, int n, bool vec, int tid, int nt) {
    const int n4 = (n + 3) & ~3, per = vec ? n4 >> 2 : n4;       // pieces of a row
    int r = tid / per, c = tid - r * per;
    const int dr = nt / per, dc = nt - dr * per;
    for (int i = tid; i < DC * per; i += nt) {
        if (vec) {
            if (r < cnt) dl_copy16(dst + r * ld + 4 * c, src + (size_t)r * stride + 4 * c);
            else *reinterpret_cast<float4*>(dst + r * ld + 4 * c) = make_float4(0.f, 0.f, 0.f, 0.f);
        } else {
            if (r < cnt && c < n) dl_copy4(dst + r * ld + c, src + (size_t)r * stride + c);
            else dst[r * ld + c] = 0.f;
        }
        r += dr; c += dc;
        if (c >= per) { c -= per; ++r; }
    }
}
__device__ __forceinline__ void copies_done() {
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 0;" ::: "memory");
}

// grid (chunk, head); 256 threads.  Thread (ty, tx) owns rows t = ty + 16 x and columns s = tx + 16 y, x, y = 0 .. 3, of the
// two score matrices: with y > x every s lies after every t, so ten of the sixteen pairs (x, y) are formed.
// M [chunk][head][t][s]; gw [chunk][head][2][64]: G_t, then P(s, cnt - 1); and what the carry kernel fetches with one bulk copy
// each: Kc [chunk][q/k head][64][KD], U0 [chunk][head][ceil(V/DV)][64][DV], Wt [chunk][head][d][64], zeros beyond the chunk's
// tokens, D and V.
__global__ void __launch_bounds__(256, 2)
delta_chunk_solve_kernel(const float* __restrict__ qn, const float* __restrict__ kn, const float* __restrict__ decay,
                         const float* __restrict__ beta, const float* __restrict__ v, int v_stride, float* __restrict__ M,
                         float* __restrict__ gw, float* __restrict__ Kc, float* __restrict__ U0, float* __restrict__ Wt,
                         const int* __restrict__ table,
                         const int* __restrict__ cu_q, int B, int H, int G, int D, int V, int region) {
    extern __shared__ __align__(16) float sh[];
    const int ld = ((D + 3) & ~3) + 4;
    float* ks = sh;                                   // [64][ld], and later X [64][256]
    float* qs = ks + DC * ld;                         // [64][ld]
    float* X = sh;
    float* at = sh + region;                          // [64 s][DC_LD]: A_ts, zeros for s >= t
    float* ps = at + DC * DC_LD;                      // [64 s][DC_PLD]: P(s, t) for the tokens t >= s of s's own block of 16
    __shared__ float sg[DC], sb[DC], sG[DC], sF[DC];  // g, beta, G, and the products from a block's first token on
    pdl_trigger();
    const int c = blockIdx.x, h = blockIdx.y, hg = h / (H / G), tid = threadIdx.x;
    const ChunkPlace p = chunk_place(table, cu_q, B, c);
    pdl_wait();
    if (tid < DC) {
        const bool in = tid < p.cnt;
        sg[tid] = in ? decay[(size_t)(p.row0 + tid) * H + h] : 1.f;
        sb[tid] = in ? beta[(size_t)(p.row0 + tid) * H + h] : 0.f;
    }
    const size_t qk0 = ((size_t)p.row0 * G + hg) * D;
    chunk_tile(ks, ld, kn + qk0, (size_t)G * D, p.cnt, D, (D & 3) == 0, tid, 256);
    chunk_tile(qs, ld, qn + qk0, (size_t)G * D, p.cnt, D, (D & 3) == 0, tid, 256);
    __syncthreads();
    if (tid < DC) {                                   // thread s multiplies g_(s+1), g_(s+2), ... on, to its block's end
        const int e = tid | 15;
        float run = 1.f;
        ps[tid * DC_PLD + (tid & 15)] = 1.f;
        for (int t = tid + 1; t <= e; ++t) { run *= sg[t]; ps[tid * DC_PLD + (t & 15)] = run; }
    } else if (tid < DC + 4) {
        float run = 1.f;
        for (int t = (tid - DC) * 16; t < (tid - DC) * 16 + 16; ++t) { run *= sg[t]; sF[t] = run; }
    }
    copies_done();
    __syncthreads();
    // P(s, t) across blocks: from s to its block's end, the whole blocks between, from t's block's start to t
    auto between = [&](int s, int t) {
        const int bs = s >> 4, bt = t >> 4;
        if (bs == bt) return ps[s * DC_PLD + (t & 15)];
        float w = ps[s * DC_PLD + 15];
        for (int b = bs + 1; b < bt; ++b) w *= sF[16 * b + 15];
        return w * sF[t];
    };
    if (tid < DC) {
        sG[tid] = sg[0] * between(0, tid);
        float* o = gw + ((size_t)c * H + h) * 2 * DC;
        o[tid] = sG[tid];
        o[DC + tid] = tid < p.cnt ? between(tid, p.cnt - 1) : 0.f;
    }
    const int tx = tid & 15, ty = tid >> 4;
    float a[4][4], m[4][4];
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) { a[x][y] = 0.f; m[x][y] = 0.f; }
    const int D4 = (D + 3) & ~3;
    if (h % (H / G) == 0) {                               // one of the heads that share these keys leaves them for the carry kernel
        float* o = Kc + ((size_t)c * G + hg) * DC * D4;
        for (int i = tid; i < DC * D4 / 4; i += 256) {
            const int r = i / (D4 >> 2);
            *reinterpret_cast<float4*>(o + 4 * i) = *reinterpret_cast<const float4*>(ks + r * ld + 4 * (i - r * (D4 >> 2)));
        }
    }
#pragma unroll 2
    for (int i = 0; i < D4; i += 4) {
        float4 kt[4], qt[4], kk[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            kt[x] = *reinterpret_cast<const float4*>(ks + (ty + 16 * x) * ld + i);
            qt[x] = *reinterpret_cast<const float4*>(qs + (ty + 16 * x) * ld + i);
            kk[x] = *reinterpret_cast<const float4*>(ks + (tx + 16 * x) * ld + i);
        }
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int y = 0; y <= x; ++y) {
                a[x][y] = fmaf(kt[x].x, kk[y].x, a[x][y]); a[x][y] = fmaf(kt[x].y, kk[y].y, a[x][y]);
                a[x][y] = fmaf(kt[x].z, kk[y].z, a[x][y]); a[x][y] = fmaf(kt[x].w, kk[y].w, a[x][y]);
                m[x][y] = fmaf(qt[x].x, kk[y].x, m[x][y]); m[x][y] = fmaf(qt[x].y, kk[y].y, m[x][y]);
                m[x][y] = fmaf(qt[x].z, kk[y].z, m[x][y]); m[x][y] = fmaf(qt[x].w, kk[y].w, m[x][y]);
            }
    }
    float* Mo = M + ((size_t)c * H + h) * DC * DC;
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) {
            const int t = ty + 16 * x, s = tx + 16 * y;
            const float w = y <= x && s <= t ? between(s, t) : 0.f;
            at[s * DC_LD + t] = s < t ? sb[t] * w * a[x][y] : 0.f;
            Mo[t * DC + s] = s <= t ? w * m[x][y] : 0.f;
        }
    __syncthreads();                                  // A is in place, the tiles of k and q are used up
    const int VP = (V + DV - 1) / DV * DV;
    for (int j0 = 0; j0 < VP + D; j0 += DC_COLS) {
        const int j = j0 + tid;
        if (j < VP + D) {                             // (a thread reads only what it wrote: no barrier between the row blocks)
            const bool is_v = j < VP;                 // (columns from V to VP repeat the last one, times zero)
            const float* src = is_v ? v + (size_t)p.row0 * v_stride + h * V + min(j, V - 1) : kn + qk0 + (j - VP);
            const size_t stride = is_v ? (size_t)v_stride : (size_t)G * D;
            const float live = is_v && j >= V ? 0.f : 1.f;
            float* wo = is_v ? U0 + (((size_t)c * H + h) * (VP / DV) + j / DV) * DC * DV + j % DV
                             : Wt + (((size_t)c * H + h) * D + (j - VP)) * DC;
            // a block's sixteen inputs are asked for while the block before is worked on; rows beyond the chunk's tokens repeat the
            // last one and are multiplied by a beta of zero
            float next[16];
            auto ask = [&](int t0) {
#pragma unroll
                for (int r = 0; r < 16; ++r) next[r] = src[(size_t)min(t0 + r, p.cnt - 1) * stride];
            };
            ask(0);
            for (int t0 = 0; t0 < DC; t0 += 16) {
                float x[16];
                if (t0 >= p.cnt) {
                    for (int r = 0; r < 16; ++r) wo[is_v ? (t0 + r) * DV : t0 + r] = 0.f;
                    continue;
                }
#pragma unroll
                for (int r = 0; r < 16; ++r) x[r] = next[r] * (is_v ? live * sb[t0 + r] : sb[t0 + r] * sG[t0 + r]);
                if (t0 + 16 < p.cnt) ask(t0 + 16);
                for (int s = 0; s < t0; ++s) {
                    const float xs = X[s * DC_COLS + tid];
#pragma unroll
                    for (int r = 0; r < 16; r += 4) {
                        const float4 av = *reinterpret_cast<const float4*>(at + s * DC_LD + t0 + r);
                        x[r] = fmaf(-av.x, xs, x[r]); x[r + 1] = fmaf(-av.y, xs, x[r + 1]);
                        x[r + 2] = fmaf(-av.z, xs, x[r + 2]); x[r + 3] = fmaf(-av.w, xs, x[r + 3]);
                    }
                }
#pragma unroll
                for (int s = 0; s < 15; ++s) {
                    float av[16];
#pragma unroll
                    for (int r = (s + 1) & ~3; r < 16; r += 4) {
                        const float4 f = *reinterpret_cast<const float4*>(at + (t0 + s) * DC_LD + t0 + r);
                        av[r] = f.x; av[r + 1] = f.y; av[r + 2] = f.z; av[r + 3] = f.w;
                    }
#pragma unroll
                    for (int r = s + 1; r < 16; ++r) x[r] = fmaf(-av[r], x[s], x[r]);
                }
#pragma unroll
                for (int r = 0; r < 16; ++r) X[(t0 + r) * DC_COLS + tid] = x[r];
                if (is_v) {
#pragma unroll
                    for (int r = 0; r < 16; ++r) wo[(t0 + r) * DV] = x[r];
                } else {
#pragma unroll
                    for (int r = 0; r < 16; r += 4)
                        *reinterpret_cast<float4*>(wo + t0 + r) = make_float4(x[r], x[r + 1], x[r + 2], x[r + 3]);
                }
            }
        }
    }
}

// grid (ceil(V / DV), head, sequence); 256 threads.  The state's columns live in the registers of the first four warps (a thread:
// four rows of every 128, four columns) and, for the product with W, in shared memory.  U = U0 - W S: warp w forms the share of
// rows d of its eighth, the eight shares are added in order.  The state's update is cut in two by tokens: the last four warps sum
// over tokens 32 .. 63 and hand their sums over through shared memory.  A chunk's inputs come as four bulk copies on a barrier per
// stage, awaited with a limit (issued row by row, as small copies, their issue alone took longer than the arithmetic).
// LS [chunk][head][d][V]: the state before each chunk; U rows of H*V.
__device__ __forceinline__ void bulk_copy(float* dst, const float* src, uint32_t floats, uint32_t bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(smem_u32(dst)), "l"(src), "r"(4 * floats), "r"(bar) : "memory");
}
template <int TILES>                                  // row tiles of 128 a thread holds: 1 (D <= 128, two stages), 2 (one stage)
__global__ void __launch_bounds__(256, 1)
delta_chunk_carry_kernel(const float* __restrict__ Kc, const float* __restrict__ U0, const float* __restrict__ Wt,
                         const float* __restrict__ gw, float* __restrict__ state, float* __restrict__ U, float* __restrict__ LS,
                         const int* __restrict__ table, const int* __restrict__ cu_q, const int* __restrict__ seq_slot, int B, int H,
                         int G, int D, int V, int* __restrict__ status) {
    constexpr int STAGES = TILES == 1 ? 2 : 1;
    extern __shared__ __align__(16) float sh[];
    const int KD = (D + 3) & ~3;
    const int stage = D * DC + DC * KD + DC * DV + 2 * DC;      // W, keys, U0, the decays' products
    float* Ss = sh + STAGES * stage;                  // [KD][DV]
    float* red = Ss + KD * DV;                        // [8][(64 + 16) * DV]
    float* Us = red + 8 * 80 * DV;                    // [64][DV]
    __shared__ __align__(8) uint64_t bars[STAGES];
    __shared__ int abort_flag;
    pdl_trigger();
    const int h = blockIdx.y, b = blockIdx.z, j0 = blockIdx.x * DV, hg = h / (H / G);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nc = min(DV, V - j0);
    const int c0 = table[b], c1 = table[b + 1];
    const int n_new = cu_q[b + 1] - cu_q[b];
    const bool owner = tid < 128;                     // holds state
    const int cc = (tid & 3) * 4, dg = ((tid & 127) >> 2) * 4;  // this thread's four columns and its first row
    const bool quad = (V & 3) == 0 && cc + 3 < nc;
    float* S = state + ((size_t)seq_slot[b] * H + h) * D * V + j0;
    if (tid == 0) {
        abort_flag = 0;
#pragma unroll
        for (int i = 0; i < STAGES; ++i) mbar_init(smem_u32(&bars[i]), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    pdl_wait();
    auto fetch = [&](int c, int buf) {                // by one thread
        float* w = sh + buf * stage;
        const uint32_t bar = smem_u32(&bars[buf]);
        mbar_expect_tx(bar, 4u * (uint32_t)stage);
        bulk_copy(w, Wt + ((size_t)c * H + h) * D * DC, D * DC, bar);
        bulk_copy(w + D * DC, Kc + ((size_t)c * G + hg) * DC * KD, DC * KD, bar);
        bulk_copy(w + D * DC + DC * KD, U0 + (((size_t)c * H + h) * gridDim.x + blockIdx.x) * DC * DV, DC * DV, bar);
        bulk_copy(w + D * DC + DC * KD + DC * DV, gw + ((size_t)c * H + h) * 2 * DC, 2 * DC, bar);
    };
    float s[TILES][4][4];
#pragma unroll
    for (int i = 0; i < TILES; ++i)
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int d = dg + r + 128 * i;
#pragma unroll
            for (int u = 0; u < 4; ++u) s[i][r][u] = (owner && d < D && cc + u < nc) ? S[(size_t)d * V + cc + u] : 0.f;
            if (owner && d < KD) *reinterpret_cast<float4*>(Ss + d * DV + cc) = make_float4(s[i][r][0], s[i][r][1], s[i][r][2], s[i][r][3]);
        }
    if (STAGES == 2 && c0 < c1 && tid == 0) fetch(c0, 0);
    const int dper = (D + 7) / 8, d0 = warp * dper, d1 = min(D, d0 + dper);
    const int rg = (lane >> 2) * 4, cg = (lane & 3) * 4;
    for (int c = c0; c < c1; ++c) {
        const int buf = STAGES == 2 ? (c - c0) & 1 : 0;
        const uint32_t parity = ((c - c0) / STAGES) & 1;
        if (STAGES == 1) {
            __syncthreads();                              // the chunk before is used up
            if (tid == 0) fetch(c, 0);
        }
        mbar_wait(smem_u32(&bars[buf]), parity, &abort_flag);
        __syncthreads();
        if (*(volatile int*)&abort_flag) {                // the copies never arrived: say so, give them one more limit, leave
            if (tid == 0) {
                atomicExch(status, 10);
                abort_flag = 0;
                mbar_wait(smem_u32(&bars[buf]), parity, &abort_flag);
            }
            return;
        }
        if (STAGES == 2 && c + 1 < c1 && tid == 0) fetch(c + 1, buf ^ 1);
        const float* w = sh + buf * stage;
        const float* k = w + D * DC;
        const float* u0 = k + DC * KD;
        const float* g = u0 + DC * DV;
        const int row0 = cu_q[b] + (c - c0) * DC, cnt = min(DC, n_new - (c - c0) * DC);
        if (owner) {
            float* ls = LS + ((size_t)c * H + h) * D * V + j0 + cc;
#pragma unroll
            for (int i = 0; i < TILES; ++i)
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    const int d = dg + r + 128 * i;
                    if (d >= D) continue;
                    if (quad) *reinterpret_cast<float4*>(ls + (size_t)d * V) = make_float4(s[i][r][0], s[i][r][1], s[i][r][2], s[i][r][3]);
                    else
#pragma unroll
                        for (int u = 0; u < 4; ++u)
                            if (cc + u < nc) ls[(size_t)d * V + u] = s[i][r][u];
                }
        }
        float acc[8][4];
#pragma unroll
        for (int r = 0; r < 8; ++r) { acc[r][0] = acc[r][1] = acc[r][2] = acc[r][3] = 0.f; }
#pragma unroll 4
        for (int d = d0; d < d1; ++d) {
            const float4 w0 = *reinterpret_cast<const float4*>(w + d * DC + rg), w1 = *reinterpret_cast<const float4*>(w + d * DC + 32 + rg);
            const float4 sv = *reinterpret_cast<const float4*>(Ss + d * DV + cg);
            const float wr[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                acc[r][0] = fmaf(wr[r], sv.x, acc[r][0]); acc[r][1] = fmaf(wr[r], sv.y, acc[r][1]);
                acc[r][2] = fmaf(wr[r], sv.z, acc[r][2]); acc[r][3] = fmaf(wr[r], sv.w, acc[r][3]);
            }
        }
        // a row's place in red leaves a gap of one row after every four: the warp's 16-byte stores then spread over all banks
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            const int t = (r < 4 ? 0 : 32) + rg + (r & 3);
            *reinterpret_cast<float4*>(red + (warp * 80 + t + (t >> 2)) * DV + cg) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
        }
        __syncthreads();
        {
            const int t = tid >> 2;
            float4 x = *reinterpret_cast<const float4*>(u0 + t * DV + cc);
#pragma unroll
            for (int q = 0; q < 8; ++q) {
                const float4 y = *reinterpret_cast<const float4*>(red + (q * 80 + t + (t >> 2)) * DV + cc);
                x.x -= y.x; x.y -= y.y; x.z -= y.z; x.w -= y.w;
            }
            if (t < cnt) {
                float* uo = U + (size_t)(row0 + t) * H * V + h * V + j0 + cc;
                if (quad) *reinterpret_cast<float4*>(uo) = x;
                else {
                    const float xs[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
                    for (int q = 0; q < 4; ++q)
                        if (cc + q < nc) uo[q] = xs[q];
                }
            }
            const float wt = g[DC + t];                   // P(t, end); 0 beyond the chunk's tokens
            *reinterpret_cast<float4*>(Us + t * DV + cc) = make_float4(x.x * wt, x.y * wt, x.z * wt, x.w * wt);
        }
        __syncthreads();
        const float gend = g[cnt - 1];
        float x[TILES][4][4];
#pragma unroll
        for (int i = 0; i < TILES; ++i) {
            const int d = dg + 128 * i;
#pragma unroll
            for (int r = 0; r < 4; ++r) { x[i][r][0] = x[i][r][1] = x[i][r][2] = x[i][r][3] = 0.f; }
            if (d < KD) {
                const int t0 = owner ? 0 : DC / 2;
#pragma unroll 8
                for (int t = t0; t < t0 + DC / 2; ++t) {
                    const float4 kk = *reinterpret_cast<const float4*>(k + t * KD + d);
                    const float4 uu = *reinterpret_cast<const float4*>(Us + t * DV + cc);
                    const float kv[4] = {kk.x, kk.y, kk.z, kk.w};
#pragma unroll
                    for (int r = 0; r < 4; ++r) {
                        x[i][r][0] = fmaf(kv[r], uu.x, x[i][r][0]); x[i][r][1] = fmaf(kv[r], uu.y, x[i][r][1]);
                        x[i][r][2] = fmaf(kv[r], uu.z, x[i][r][2]); x[i][r][3] = fmaf(kv[r], uu.w, x[i][r][3]);
                    }
                }
                if (!owner)                               // (the shares of W S are used up: their place takes these sums)
#pragma unroll
                    for (int r = 0; r < 4; ++r)
                        *reinterpret_cast<float4*>(red + (d + r) * DV + cc) = make_float4(x[i][r][0], x[i][r][1], x[i][r][2], x[i][r][3]);
            }
        }
        __syncthreads();
        if (owner)
#pragma unroll
            for (int i = 0; i < TILES; ++i)
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    const int d = dg + r + 128 * i;
                    if (d >= KD) continue;
                    const float4 y = *reinterpret_cast<const float4*>(red + d * DV + cc);
                    s[i][r][0] = fmaf(gend, s[i][r][0], x[i][r][0] + y.x); s[i][r][1] = fmaf(gend, s[i][r][1], x[i][r][1] + y.y);
                    s[i][r][2] = fmaf(gend, s[i][r][2], x[i][r][2] + y.z); s[i][r][3] = fmaf(gend, s[i][r][3], x[i][r][3] + y.w);
                    *reinterpret_cast<float4*>(Ss + d * DV + cc) = make_float4(s[i][r][0], s[i][r][1], s[i][r][2], s[i][r][3]);
                }
    }
    if (owner)
#pragma unroll
        for (int i = 0; i < TILES; ++i)
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                const int d = dg + r + 128 * i;
#pragma unroll
                for (int u = 0; u < 4; ++u)
                    if (d < D && cc + u < nc) S[(size_t)d * V + cc + u] = s[i][r][u];
            }
}

// grid (chunk, head, ceil(V / DO)); 256 threads: thread (ty, tx) owns rows ty + 16 x and columns 4 tx .. 4 tx + 3.
__global__ void __launch_bounds__(256)
delta_chunk_out_kernel(const float* __restrict__ qn, const float* __restrict__ M, const float* __restrict__ gw,
                       const float* __restrict__ U, const float* __restrict__ LS, float* __restrict__ o, const int* __restrict__ table,
                       const int* __restrict__ cu_q, int B, int H, int G, int D, int V) {
    extern __shared__ __align__(16) float sh[];
    const int D4 = (D + 3) & ~3, ld = DC + D4 + 4;
    float* lhs = sh;                                  // [64][ld]: M_ts, then q
    float* rhs = lhs + DC * ld;                       // [64 + D4][DO]: U, then the state before the chunk
    __shared__ float sG[DC];
    pdl_trigger();
    const int c = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * DO, hg = h / (H / G), tid = threadIdx.x;
    const ChunkPlace p = chunk_place(table, cu_q, B, c);
    const int nc = min(DO, V - j0);
    pdl_wait();
    chunk_tile(lhs, ld, M + ((size_t)c * H + h) * DC * DC, DC, p.cnt, DC, true, tid, 256);
    chunk_tile(lhs + DC, ld, qn + ((size_t)p.row0 * G + hg) * D, (size_t)G * D, p.cnt, D, (D & 3) == 0, tid, 256);
    if (tid < DC) sG[tid] = gw[((size_t)c * H + h) * 2 * DC + tid];
    const bool vec = (V & 3) == 0;
    const float* us = U + (size_t)p.row0 * H * V + h * V + j0;
    const float* ss = LS + ((size_t)c * H + h) * D * V + j0;
    const int per = vec ? DO / 4 : DO, step = vec ? 4 : 1;
    for (int i = tid; i < (DC + D4) * per; i += 256) {
        const int r = i / per, cc = (i - r * per) * step;
        const bool in = cc < nc && (r < DC ? r < p.cnt : r - DC < D);
        const float* src = r < DC ? us + (size_t)r * H * V + cc : ss + (size_t)(r - DC) * V + cc;
        float* dst = rhs + r * DO + cc;
        if (vec) {
            if (in) dl_copy16(dst, src); else *reinterpret_cast<float4*>(dst) = make_float4(0.f, 0.f, 0.f, 0.f);
        } else {
            if (in) dl_copy4(dst, src); else *dst = 0.f;
        }
    }
    copies_done();
    __syncthreads();
    const int tx = tid & 15, ty = tid >> 4;
    float a[4][4], e[4][4];
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) { a[x][y] = 0.f; e[x][y] = 0.f; }
    // four inner positions i .. i + 3 for the rows x >= x0: 4 (4 - x0) + 16 loads' worth of FMAs
    auto block = [&](float (&acc)[4][4], int i, auto x0) {
        float4 r[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) r[q] = *reinterpret_cast<const float4*>(rhs + (i + q) * DO + 4 * tx);
#pragma unroll
        for (int x = decltype(x0)::value; x < 4; ++x) {
            const float4 l = *reinterpret_cast<const float4*>(lhs + (ty + 16 * x) * ld + i);
            acc[x][0] = fmaf(l.x, r[0].x, acc[x][0]); acc[x][1] = fmaf(l.x, r[0].y, acc[x][1]); acc[x][2] = fmaf(l.x, r[0].z, acc[x][2]); acc[x][3] = fmaf(l.x, r[0].w, acc[x][3]);
            acc[x][0] = fmaf(l.y, r[1].x, acc[x][0]); acc[x][1] = fmaf(l.y, r[1].y, acc[x][1]); acc[x][2] = fmaf(l.y, r[1].z, acc[x][2]); acc[x][3] = fmaf(l.y, r[1].w, acc[x][3]);
            acc[x][0] = fmaf(l.z, r[2].x, acc[x][0]); acc[x][1] = fmaf(l.z, r[2].y, acc[x][1]); acc[x][2] = fmaf(l.z, r[2].z, acc[x][2]); acc[x][3] = fmaf(l.z, r[2].w, acc[x][3]);
            acc[x][0] = fmaf(l.w, r[3].x, acc[x][0]); acc[x][1] = fmaf(l.w, r[3].y, acc[x][1]); acc[x][2] = fmaf(l.w, r[3].z, acc[x][2]); acc[x][3] = fmaf(l.w, r[3].w, acc[x][3]);
        }
    };
    // the scores of tokens s in 16 y .. 16 y + 15 are zero for the rows x < y
    for (int i = 0; i < 16; i += 4) block(a, i, std::integral_constant<int, 0>{});
    for (int i = 16; i < 32; i += 4) block(a, i, std::integral_constant<int, 1>{});
    for (int i = 32; i < 48; i += 4) block(a, i, std::integral_constant<int, 2>{});
    for (int i = 48; i < 64; i += 4) block(a, i, std::integral_constant<int, 3>{});
    for (int i = DC; i < DC + D4; i += 4) block(e, i, std::integral_constant<int, 0>{});
#pragma unroll
    for (int x = 0; x < 4; ++x) {
        const int t = ty + 16 * x;
        if (t >= p.cnt) continue;
        float* out = o + (size_t)(p.row0 + t) * H * V + h * V + j0 + 4 * tx;
        const float g = sG[t];
#pragma unroll
        for (int y = 0; y < 4; ++y)
            if (4 * tx + y < nc) out[y] = fmaf(g, e[x][y], a[x][y]);
    }
}

static int chunk_smem(const void* kernel, size_t bytes, size_t* configured) {
    if (bytes <= *configured) return 0;
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (e != cudaSuccess) return (int)e;
    *configured = bytes;
    return 0;
}

extern "C" {
// Floats of scratch memory that rf_delta_chunked needs for T_ tokens in n_chunks chunks.
long long rf_delta_chunked_scratch(int n_chunks, int H, int G, int D, int V, int T_) {
    const long long D4 = (D + 3) & ~3, VP = (V + DV - 1) / DV * DV;
    return (long long)n_chunks * H * (DC * DC + 2 * DC + (long long)D * DC + VP * DC + (long long)D * V) + n_chunks * G * DC * D4 +
           (long long)T_ * H * V + 16;
}
// What rf_delta_scan computes with per_head decays, for prompts (see above).  table: first[B+1], then n_chunks pairs (sequence,
// first row of the chunk among the sequence's new tokens), in the order of the sequences.
int rf_delta_chunked(const float* qn, const float* kn, const float* decay, const float* beta, const float* v, int v_stride,
                     float* state, float* o, float* scratch, const int* table, int n_chunks, const int* cu_q, const int* seq_slot,
                     int B, int H, int G, int D, int V, int T_, int* status, cudaStream_t st) {
    if (B <= 0 || n_chunks <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || D <= 0 || V <= 0 || H > 65535 || B > 65535) return RF_ERR_BAD_ARG;
    if (D > 256 || status == nullptr || (reinterpret_cast<uintptr_t>(scratch) & 15) || (reinterpret_cast<uintptr_t>(kn) & 15) ||
        (reinterpret_cast<uintptr_t>(qn) & 15))
        return RF_ERR_UNSUPPORTED;
    const size_t ch = (size_t)n_chunks * H;
    const int D4 = (D + 3) & ~3, VP = (V + DV - 1) / DV * DV;
    float* M = scratch;
    float* gw = M + ch * DC * DC;
    float* Wt = gw + ch * 2 * DC;
    float* U0 = Wt + ch * D * DC;
    float* Kc = U0 + ch * VP * DC;
    float* U = Kc + (size_t)n_chunks * G * DC * D4;
    float* LS = U + ((size_t)T_ * H * V + 3) / 4 * 4;
    int region = 2 * DC * (D4 + 4);
    if (region < DC * DC_COLS) region = DC * DC_COLS;
    const size_t smem1 = ((size_t)region + DC * DC_LD + DC * DC_PLD) * sizeof(float);
    const int tiles = D4 <= 128 ? 1 : 2;
    const size_t smem2 = ((size_t)(tiles == 1 ? 2 : 1) * (D * DC + DC * D4 + DC * DV + 2 * DC) + D4 * DV + 8 * 80 * DV + DC * DV) * sizeof(float);
    const size_t smem3 = ((size_t)DC * (DC + D4 + 4) + (DC + D4) * DO) * sizeof(float);
    static size_t set1 = 48 * 1024, set2[2] = {48 * 1024, 48 * 1024}, set3 = 48 * 1024;
    const auto carry = tiles == 1 ? delta_chunk_carry_kernel<1> : delta_chunk_carry_kernel<2>;
    int e;
    if ((e = chunk_smem((const void*)delta_chunk_solve_kernel, smem1, &set1)) ||
        (e = chunk_smem((const void*)carry, smem2, &set2[tiles - 1])) ||
        (e = chunk_smem((const void*)delta_chunk_out_kernel, smem3, &set3)))
        return e;
    rf_launch(delta_chunk_solve_kernel, dim3(n_chunks, H), dim3(256), smem1, st, qn, kn, decay, beta, v, v_stride, M, gw, Kc, U0, Wt, table,
              cu_q, B, H, G, D, V, region);
    RF_LAUNCH_CHECK();
    rf_launch(carry, dim3(VP / DV, H, B), dim3(256), smem2, st, (const float*)Kc, (const float*)U0, (const float*)Wt, (const float*)gw,
              state, U, LS, table, cu_q, seq_slot, B, H, G, D, V, status);
    RF_LAUNCH_CHECK();
    rf_launch(delta_chunk_out_kernel, dim3(n_chunks, H, (V + DO - 1) / DO), dim3(256), smem3, st, qn, (const float*)M, (const float*)gw,
              (const float*)U, (const float*)LS, o, table, cu_q, B, H, G, D, V);
    RF_LAUNCH_CHECK();
    return 0;
}
}
