// Attention that caches a narrow latent of every position and one rotated key part shared by the heads.
//
//   latent_write      the projection's row  q (heads x [dim | rot]) | down (rank + rot) | gate  on its way into the step:
//                     the first `rank` numbers of `down` are RMS-normed with a weight, the last `rot` turn with the
//                     position, and both go to the position's cache row [latent | rotated part | zeros]; the rotated parts
//                     of the queries turn and go wherever the attention wants them.
//   latent_gather     cache rows of whole sequences, position after position, into one matrix (prompts that continue a
//                     context expand its latents again).
//   head_product      y[t, h, :] = W_h x[t, h, :] with a matrix per head: queries folded into the latent's space, and
//                     attention results out of it (optionally times sigmoid(gate)).
#include "common.cuh"

struct LatentWrite {
    const void* src;             // [T][src_stride], or n_parts float32 partial sums [n_parts][T][src_stride]
    int src_stride, n_parts;
    long long part_stride;
    int q_col, down_col, gate_col;
    int heads, dim, rot, rank;
    const void* norm_w;          // [rank]
    int norm_w_is_f32;
    float eps;
    const float* inv_freq;       // [rot / 2]
    int interleaved;
    float magnitude;
    const int *tok_seq, *tok_pos, *seq_slot, *block_table;
    int max_pages;
    void* pages;                 // [n_pages][RF_PAGE][ld]
    int ld;
    void* rows;                  // [T][ld] copy of the cache rows, or null
    void* qn;                    // unrotated query parts, or null (they stay where they are)
    long long qn_tok, qn_head;   // strides in elements
    void* qr;                    // rotated query parts
    long long qr_tok, qr_head;
    int qr_pad;                  // zeros behind every rotated part
    void* gate;                  // [T][gate_n], or null
    int gate_n;
};

template <typename T, bool PARTS>
__device__ __forceinline__ float lw_load(const LatentWrite& a, int t, int col) {
    if constexpr (PARTS) {
        const float* p = reinterpret_cast<const float*>(a.src) + (size_t)t * a.src_stride + col;
        float v = 0.f;
#pragma unroll 8
        for (int s = 0; s < a.n_parts; ++s) v += p[(size_t)s * a.part_stride];
        return v;
    } else {
        return Cvt<T>::to_f32(reinterpret_cast<const T*>(a.src)[(size_t)t * a.src_stride + col]);
    }
}
__device__ __forceinline__ void lw_turn(const LatentWrite& a, int pos, int i, float& u, float& v) {
    float s, c;
    sincosf((float)pos * a.inv_freq[i], &s, &c);
    s *= a.magnitude; c *= a.magnitude;
    const float x = u * c - v * s;
    v = v * c + u * s;
    u = x;
}

#define LW_UNIT 512              // columns of one unit of work

// units of a token: 0 the cache row; then the rotated query parts, the unrotated ones (if they move) and the gate (if it
// moves), LW_UNIT at a time
template <typename T, bool PARTS>
__global__ void __launch_bounds__(256)
latent_write_kernel(LatentWrite a) {
    __shared__ float red[34];
    extern __shared__ float lat[];                   // [rank]
    pdl_trigger();
    const int t = blockIdx.x;
    const int pos = a.tok_pos[t];
    const int slot = a.seq_slot[a.tok_seq[t]];
    const int page = a.block_table[(size_t)slot * a.max_pages + pos / RF_PAGE];
    const int half = a.rot >> 1, hq = a.dim + a.rot;
    const int n_rot = (a.heads * half + LW_UNIT - 1) / LW_UNIT;
    const int n_nope = a.qn != nullptr ? (a.heads * a.dim + LW_UNIT - 1) / LW_UNIT : 0;
    const int n_gate = a.gate != nullptr ? (a.gate_n + LW_UNIT - 1) / LW_UNIT : 0;
    const int n_units = 1 + n_rot + n_nope + n_gate;
    pdl_wait();
    for (int unit = blockIdx.y; unit < n_units; unit += gridDim.y) {
        if (unit == 0) {
            float ss = 0.f;
            for (int c = threadIdx.x; c < a.rank; c += blockDim.x) {
                const float v = lw_load<T, PARTS>(a, t, a.down_col + c);
                lat[c] = v;
                ss = fmaf(v, v, ss);
            }
            const float r = rsqrtf(block_sum(ss, red) / (float)a.rank + a.eps);
            T* dst = reinterpret_cast<T*>(a.pages) + ((size_t)page * RF_PAGE + pos % RF_PAGE) * a.ld;
            T* copy = a.rows != nullptr ? reinterpret_cast<T*>(a.rows) + (size_t)t * a.ld : nullptr;
            for (int c = threadIdx.x; c < a.rank; c += blockDim.x) {      // a thread reads what it wrote
                const T v = Cvt<T>::from_f32(lat[c] * r * load_vec(a.norm_w, a.norm_w_is_f32, c));
                dst[c] = v;
                if (copy != nullptr) copy[c] = v;
            }
            for (int i = threadIdx.x; i < half; i += blockDim.x) {
                const int e0 = a.interleaved ? 2 * i : i, e1 = a.interleaved ? 2 * i + 1 : i + half;
                float u = lw_load<T, PARTS>(a, t, a.down_col + a.rank + e0), v = lw_load<T, PARTS>(a, t, a.down_col + a.rank + e1);
                lw_turn(a, pos, i, u, v);
                dst[a.rank + e0] = Cvt<T>::from_f32(u);
                dst[a.rank + e1] = Cvt<T>::from_f32(v);
                if (copy != nullptr) { copy[a.rank + e0] = Cvt<T>::from_f32(u); copy[a.rank + e1] = Cvt<T>::from_f32(v); }
            }
            for (int c = a.rank + a.rot + threadIdx.x; c < a.ld; c += blockDim.x) {
                dst[c] = Cvt<T>::from_f32(0.f);
                if (copy != nullptr) copy[c] = Cvt<T>::from_f32(0.f);
            }
            // zeros behind the rotated query parts (the same rows' padding)
            if (a.qr_pad > 0)
                for (int c = threadIdx.x; c < a.heads * a.qr_pad; c += blockDim.x)
                    reinterpret_cast<T*>(a.qr)[t * a.qr_tok + (c / a.qr_pad) * a.qr_head + a.rot + c % a.qr_pad] = Cvt<T>::from_f32(0.f);
            continue;
        }
        int base = unit - 1;
        if (base < n_rot) {
            const int end = min(a.heads * half, (base + 1) * LW_UNIT);
            for (int p = base * LW_UNIT + threadIdx.x; p < end; p += blockDim.x) {
                const int h = p / half, i = p - h * half;
                const int e0 = a.interleaved ? 2 * i : i, e1 = a.interleaved ? 2 * i + 1 : i + half;
                const int col = a.q_col + h * hq + a.dim;
                float u = lw_load<T, PARTS>(a, t, col + e0), v = lw_load<T, PARTS>(a, t, col + e1);
                lw_turn(a, pos, i, u, v);
                T* dst = reinterpret_cast<T*>(a.qr) + t * a.qr_tok + h * a.qr_head;
                dst[e0] = Cvt<T>::from_f32(u);
                dst[e1] = Cvt<T>::from_f32(v);
            }
            continue;
        }
        base -= n_rot;
        if (base < n_nope) {
            const int end = min(a.heads * a.dim, (base + 1) * LW_UNIT);
            for (int p = base * LW_UNIT + threadIdx.x; p < end; p += blockDim.x) {
                const int h = p / a.dim, c = p - h * a.dim;
                reinterpret_cast<T*>(a.qn)[t * a.qn_tok + h * a.qn_head + c] = Cvt<T>::from_f32(lw_load<T, PARTS>(a, t, a.q_col + h * hq + c));
            }
            continue;
        }
        base -= n_nope;
        const int end = min(a.gate_n, (base + 1) * LW_UNIT);
        for (int c = base * LW_UNIT + threadIdx.x; c < end; c += blockDim.x)
            reinterpret_cast<T*>(a.gate)[(size_t)t * a.gate_n + c] = Cvt<T>::from_f32(lw_load<T, PARTS>(a, t, a.gate_col + c));
    }
}

// ---------------------------------------------------------------- cache rows of whole sequences into one matrix
// cu [B + 1]: first row of every sequence in out; row cu[i] + j is position j of sequence i.  16 bytes a thread and step.
__global__ void __launch_bounds__(128)
latent_gather_kernel(const uint4* __restrict__ pages, const int* __restrict__ cu, const int* __restrict__ seq_slot,
                     const int* __restrict__ block_table, int max_pages, uint4* __restrict__ out, int n16, int B) {
    pdl_trigger();
    const int row = blockIdx.x;
    int lo = 0, hi = B - 1;                          // the last sequence whose first row is not behind this one
    while (lo < hi) { const int mid = (lo + hi + 1) >> 1; if (cu[mid] <= row) lo = mid; else hi = mid - 1; }
    const int pos = row - cu[lo];
    const int page = block_table[(size_t)seq_slot[lo] * max_pages + pos / RF_PAGE];
    const uint4* src = pages + ((size_t)page * RF_PAGE + pos % RF_PAGE) * n16;
    pdl_wait();
    for (int i = threadIdx.x; i < n16; i += blockDim.x) out[(size_t)row * n16 + i] = src[i];
}

// ---------------------------------------------------------------- a matrix per head
// y[t][h][n] = sum_k W[h][n][k] x[t][h][k] (* sigmoid(gate[t][h * N + n]))
struct HeadProduct {
    const void* x; long long x_tok, x_head;
    const void* w;               // [heads][N][K]
    void* y; long long y_tok, y_head;
    const void* gate; long long gate_tok;
    int T_, N, K;
};

// FFMA: a block owns 32 tokens x 64 outputs of one head, K in steps of 16 through shared memory; a thread 2 x 4 results.
template <typename T>
__global__ void __launch_bounds__(256)
head_product_simt_kernel(HeadProduct a) {
    __shared__ float xs[16][33], ws[16][65];
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.z, t0 = blockIdx.y * 32, n0 = blockIdx.x * 64, tid = threadIdx.x;
    const int tx = tid & 15, ty = tid >> 4;          // outputs tx + 16 j, tokens ty + 16 i
    const T* x = reinterpret_cast<const T*>(a.x) + h * a.x_head;
    const T* w = reinterpret_cast<const T*>(a.w) + (size_t)h * a.N * a.K;
    float acc[2][4] = {};
    for (int k0 = 0; k0 < a.K; k0 += 16) {
        for (int i = tid; i < 32 * 16; i += 256) {
            const int r = i >> 4, k = i & 15, t = t0 + r;
            xs[k][r] = (t < a.T_ && k0 + k < a.K) ? Cvt<T>::to_f32(x[t * a.x_tok + k0 + k]) : 0.f;
        }
        for (int i = tid; i < 64 * 16; i += 256) {
            const int r = i >> 4, k = i & 15, n = n0 + r;
            ws[k][r] = (n < a.N && k0 + k < a.K) ? Cvt<T>::to_f32(w[(size_t)n * a.K + k0 + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k)
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xs[k][ty + 16 * i], ws[k][tx + 16 * j], acc[i][j]);
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = t0 + ty + 16 * i, n = n0 + tx + 16 * j;
            if (t >= a.T_ || n >= a.N) continue;
            float v = acc[i][j];
            if (a.gate != nullptr)
                v /= 1.f + expf(-Cvt<T>::to_f32(reinterpret_cast<const T*>(a.gate)[t * a.gate_tok + (size_t)h * a.N + n]));
            reinterpret_cast<T*>(a.y)[t * a.y_tok + h * a.y_head + n] = Cvt<T>::from_f32(v);
        }
}

// bfloat16, few tokens: a block owns 16 outputs of one head and up to MT * 16 tokens; its four warps share K, and their
// partial results meet in shared memory in a fixed order.  mma.sync with tokens on the rows and outputs on the columns.
// A lane takes 8 neighbouring k of a row at a time (16 bytes): the k's of a 32-wide block are dealt to the two MMA steps in
// the same permuted order for both operands, which leaves the sum unchanged.  K a multiple of 8; all strides of x, w too.
__device__ __forceinline__ void hp_mma(float* d, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
template <int MT>
__global__ void __launch_bounds__(128)
head_product_mma_kernel(HeadProduct a) {
    __shared__ float part[4][MT * 16][17];
    pdl_trigger();
    const int h = blockIdx.z, n0 = blockIdx.x * 16, t0 = blockIdx.y * (MT * 16);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
    const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(a.x) + h * a.x_head;
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.w) + (size_t)h * a.N * a.K;
    const int kb_all = (a.K + 31) / 32, per = (kb_all + 3) / 4;
    const int kb0 = warp * per, kb1 = min(kb_all, kb0 + per);
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float acc[MT][2][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
    bool waited = false;
    for (int kb = kb0; kb < kb1; kb += 4) {
        uint4 wf[4][2];
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int n = n0 + 8 * j + g, k = (kb + u) * 32 + 8 * q;
                wf[u][j] = (kb + u < kb1 && n < a.N && k < a.K) ? *reinterpret_cast<const uint4*>(w + (size_t)n * a.K + k) : zero;
            }
        if (!waited) { pdl_wait(); waited = true; }   // the weights are nobody's result; x is
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            if (kb + u >= kb1) break;
            const int k = (kb + u) * 32 + 8 * q;
#pragma unroll
            for (int i = 0; i < MT; ++i) {
                const int ta = t0 + 16 * i + g, tb = ta + 8;
                const uint4 xa = (ta < a.T_ && k < a.K) ? *reinterpret_cast<const uint4*>(x + ta * a.x_tok + k) : zero;
                const uint4 xb = (tb < a.T_ && k < a.K) ? *reinterpret_cast<const uint4*>(x + tb * a.x_tok + k) : zero;
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    hp_mma(acc[i][j], xa.x, xb.x, xa.y, xb.y, wf[u][j].x, wf[u][j].y);
                    hp_mma(acc[i][j], xa.z, xb.z, xa.w, xb.w, wf[u][j].z, wf[u][j].w);
                }
            }
        }
    }
    if (!waited) pdl_wait();
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            part[warp][16 * i + g][8 * j + 2 * q] = acc[i][j][0];
            part[warp][16 * i + g][8 * j + 2 * q + 1] = acc[i][j][1];
            part[warp][16 * i + g + 8][8 * j + 2 * q] = acc[i][j][2];
            part[warp][16 * i + g + 8][8 * j + 2 * q + 1] = acc[i][j][3];
        }
    __syncthreads();
    for (int e = threadIdx.x; e < MT * 16 * 16; e += 128) {
        const int r = e >> 4, c = e & 15, t = t0 + r, n = n0 + c;
        if (t >= a.T_ || n >= a.N) continue;
        float v = (part[0][r][c] + part[1][r][c]) + (part[2][r][c] + part[3][r][c]);
        if (a.gate != nullptr) {
            const float gt = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(a.gate)[t * a.gate_tok + (size_t)h * a.N + n]);
            v = __fdividef(v, 1.f + __expf(-gt));
        }
        reinterpret_cast<__nv_bfloat16*>(a.y)[t * a.y_tok + h * a.y_head + n] = __float2bfloat16_rn(v);
    }
}

template <typename T>
static int launch_latent_write(const LatentWrite& a, int T_, cudaStream_t st) {
    const int units = 1 + (a.heads * (a.rot / 2) + LW_UNIT - 1) / LW_UNIT + (a.qn ? (a.heads * a.dim + LW_UNIT - 1) / LW_UNIT : 0) +
                      (a.gate ? (a.gate_n + LW_UNIT - 1) / LW_UNIT : 0);
    int by = 1;                                      // few tokens: a token's units over several blocks
    while (by < units && (long long)T_ * by < 2 * 148) ++by;
    const size_t smem = (size_t)a.rank * sizeof(float);
    if (smem > 40 * 1024) return RF_ERR_UNSUPPORTED;
    if (a.n_parts > 0) rf_launch(latent_write_kernel<T, true>, dim3(T_, by), dim3(256), smem, st, a);
    else rf_launch(latent_write_kernel<T, false>, dim3(T_, by), dim3(256), smem, st, a);
    RF_LAUNCH_CHECK();
    return 0;
}

extern "C" {

// n_parts 0: src [T][src_stride] in the compute dtype, else float32 partial sums; qn / gate / rows may be null.
int rf_latent_write(int dtype, const void* src, int src_stride, int n_parts, long long part_stride, int q_col, int down_col,
                    int gate_col, int heads, int dim, int rot, int rank, const void* norm_w, int norm_w_is_f32, float eps,
                    const float* inv_freq, int interleaved, float magnitude, const int* tok_seq, const int* tok_pos,
                    const int* seq_slot, const int* block_table, int max_pages, void* pages, int ld, void* rows, void* qn,
                    long long qn_tok, long long qn_head, void* qr, long long qr_tok, long long qr_head, int qr_pad, void* gate,
                    int gate_n, int T_, cudaStream_t st) {
    if (T_ <= 0) return 0;
    if (heads < 1 || dim < 0 || rot < 0 || rot % 2 || rank < 1 || ld < rank + rot || (rot > 0 && (!inv_freq || !qr))) return RF_ERR_BAD_ARG;
    if (qr_pad > 0 && !qr) return RF_ERR_BAD_ARG;
    const LatentWrite a{src, src_stride, n_parts, part_stride, q_col, down_col, gate_col, heads, dim, rot, rank, norm_w, norm_w_is_f32,
                        eps, inv_freq, interleaved, magnitude, tok_seq, tok_pos, seq_slot, block_table, max_pages, pages, ld, rows, qn,
                        qn_tok, qn_head, qr, qr_tok, qr_head, qr_pad, gate, gate_n};
    return dtype == 0 ? launch_latent_write<float>(a, T_, st) : launch_latent_write<__nv_bfloat16>(a, T_, st);
}

// rows of `row_bytes` (a multiple of 16) each
int rf_latent_gather(const void* pages, int row_bytes, const int* cu, const int* seq_slot, const int* block_table, int max_pages,
                     void* out, int n_rows, int B, cudaStream_t st) {
    if (n_rows <= 0) return 0;
    if (row_bytes % 16 || B < 1) return RF_ERR_BAD_ARG;
    rf_launch(latent_gather_kernel, dim3(n_rows), dim3(row_bytes >= 16 * 128 ? 128 : 64), 0, st, reinterpret_cast<const uint4*>(pages),
              cu, seq_slot, block_table, max_pages, reinterpret_cast<uint4*>(out), row_bytes / 16, B);
    RF_LAUNCH_CHECK();
    return 0;
}

int rf_head_product(int dtype, const void* x, long long x_tok, long long x_head, const void* w, int heads, int N, int K, void* y,
                    long long y_tok, long long y_head, const void* gate, long long gate_tok, int T_, cudaStream_t st) {
    if (T_ <= 0) return 0;
    if (heads < 1 || heads > 65535 || N < 1 || K < 1) return RF_ERR_BAD_ARG;
    const HeadProduct a{x, x_tok, x_head, w, y, y_tok, y_head, gate, gate_tok, T_, N, K};
    auto whole = [](const void* p, long long s) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && s % 8 == 0; };
    if (dtype != 0 && K % 8 == 0 && whole(x, x_tok) && whole(w, x_head)) {
        const int nb = (N + 15) / 16;
        const int rows = T_ <= 16 ? 16 : 64;
        const int tb = (T_ + rows - 1) / rows;
        if (tb > 65535) return RF_ERR_UNSUPPORTED;
        if (rows == 16) rf_launch(head_product_mma_kernel<1>, dim3(nb, tb, heads), dim3(128), 0, st, a);
        else rf_launch(head_product_mma_kernel<4>, dim3(nb, tb, heads), dim3(128), 0, st, a);
        RF_LAUNCH_CHECK();
        return 0;
    }
    const dim3 grid((N + 63) / 64, (T_ + 31) / 32, heads);
    if (grid.y > 65535) return RF_ERR_UNSUPPORTED;
    if (dtype == 0) rf_launch(head_product_simt_kernel<float>, grid, dim3(256), 0, st, a);
    else rf_launch(head_product_simt_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, a);
    RF_LAUNCH_CHECK();
    return 0;
}

}
