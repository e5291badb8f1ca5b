// Several residual streams instead of one (hyper-connections), and an embedding that looks at pairs of tokens.
//
//   streams_update    for every token, from S old streams x_1 .. x_S and a sub-layer's result y:
//                         x_t <- sum_s mix[s, t] x_s + out[t] y                     (all streams at once from the old ones)
//                         next = rms(sum_t in[t] x_t) * w                           (the next sub-layer's input, if asked)
//                     in one pass over the token's streams.  y comes as 32-bit partial sums of a K-split product, added
//                     here in index order.  Without y it only collects: next = rms(sum_s in[s] x_s) * w.
//   pair_embed        x = E[token] * scale + P[row of (previous token, token)], RMS-normed with a weight; the previous
//                     token of a step's first token comes from a per-sequence state.
// Everything is evaluated in 32-bit; T is the compute dtype of the weights tables and of next.
#include "common.cuh"

#define ST_MAX_CLUSTER 8

struct StreamsArgs {
    const float* x;              // [rows][S][W], or [rows][W] when all streams are still equal (x_streams == 1)
    int x_streams;               // 1 or S
    const float* y;              // n_y partial sums [n_y][rows][W], or null
    int n_y;
    const float* mix;            // [S][S] from, to
    const float* out;            // [S]
    float* x_new;                // [rows][S][W] (may be x when x_streams == S)
    const float* in;             // [S], null: ones
    const void* w;               // [W] norm weight
    int w_is_f32;
    float eps;
    void* next;                  // [rows][W] in the compute dtype, or null
    const int* pick;             // row r of the launch reads token row pick[r] (null: r); only without y
    int S, W;
};

__device__ __forceinline__ uint32_t st_rank() { uint32_t r; asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ void st_cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

template <int V> struct StVec;
template <> struct StVec<4> {
    static __device__ __forceinline__ void load(const float* p, float* v) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    }
    static __device__ __forceinline__ void store(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
    static __device__ __forceinline__ void put(float* p, const float* v) { store(p, v); }
    static __device__ __forceinline__ void put(__nv_bfloat16* p, const float* v) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 x;
        x.x = *reinterpret_cast<const uint32_t*>(&a); x.y = *reinterpret_cast<const uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = x;
    }
    static __device__ __forceinline__ void weight(const void* w, int f32, int c, float* v) {
        if (f32) load(reinterpret_cast<const float*>(w) + c, v);
        else {
            const uint2 x = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(w) + c);
            v[0] = __uint_as_float(x.x << 16); v[1] = __uint_as_float(x.x & 0xffff0000u);
            v[2] = __uint_as_float(x.y << 16); v[3] = __uint_as_float(x.y & 0xffff0000u);
        }
    }
};
template <> struct StVec<1> {
    static __device__ __forceinline__ void load(const float* p, float* v) { v[0] = *p; }
    static __device__ __forceinline__ void store(float* p, const float* v) { *p = v[0]; }
    static __device__ __forceinline__ void put(float* p, const float* v) { *p = v[0]; }
    static __device__ __forceinline__ void put(__nv_bfloat16* p, const float* v) { *p = __float2bfloat16_rn(v[0]); }
    static __device__ __forceinline__ void weight(const void* w, int f32, int c, float* v) { v[0] = load_vec(w, f32, c); }
};

// S_: the number of streams when it is small (their elements stay in registers), 0: any number.
// A row is one block, or a cluster of blocks with a share of the columns each whose sums of squares meet through shared
// memory (few rows).
template <typename T, int V, int S_>
__global__ void __launch_bounds__(512)
streams_update_kernel(StreamsArgs a, int cluster) {
    extern __shared__ float sm[];                    // [share] of the collected row, then 34 for sums, then the cluster's sums
    pdl_trigger();
    const int S = S_ ? S_ : a.S;
    const int rank = cluster > 1 ? (int)st_rank() : 0;
    const int row = blockIdx.x / cluster;
    const int share = ((a.W / V + cluster - 1) / cluster) * V;
    const int c_lo = rank * share, c_hi = min(a.W, c_lo + share);
    float* u_s = sm;
    float* red = sm + share;
    float* sums = red + 34;                          // [ST_MAX_CLUSTER]
    // every block of the row must be running before its shared memory is written from another
    const bool meet = cluster > 1 && a.next != nullptr;
    if (meet) asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    // weights: no kernel of a step writes them
    constexpr int SR = S_ ? S_ : 1;
    float mix_r[SR * SR], out_r[SR], in_r[SR];
    if (S_) {
#pragma unroll
        for (int i = 0; i < SR; ++i) {
            in_r[i] = a.in != nullptr ? a.in[i] : 1.f;
            out_r[i] = a.y != nullptr ? a.out[i] : 0.f;
#pragma unroll
            for (int j = 0; j < SR; ++j) mix_r[i * SR + j] = a.y != nullptr ? a.mix[i * SR + j] : 0.f;
        }
    }
    pdl_wait();
    const int src = a.pick != nullptr ? a.pick[row] : row;
    const float* x = a.x + (size_t)src * a.x_streams * a.W;
    const size_t s_step = a.x_streams == 1 ? 0 : (size_t)a.W;
    const size_t y_stride = (size_t)(gridDim.x / cluster) * a.W;
    float ss = 0.f;
    for (int c = c_lo + V * (int)threadIdx.x; c < c_hi; c += V * (int)blockDim.x) {
        float u[V];
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = 0.f;
        float y[V];
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = 0.f;
        if constexpr (S_ > 0) {
            float xs[SR][V];
#pragma unroll
            for (int s = 0; s < SR; ++s) StVec<V>::load(x + s * s_step + c, xs[s]);
            if (a.y != nullptr) {
                const float* yp = a.y + (size_t)row * a.W + c;
#pragma unroll 8
                for (int p = 0; p < a.n_y; ++p) {
                    float t[V];
                    StVec<V>::load(yp + (size_t)p * y_stride, t);
#pragma unroll
                    for (int e = 0; e < V; ++e) y[e] += t[e];
                }
                float* xn = a.x_new + (size_t)row * S * a.W + c;
#pragma unroll
                for (int t = 0; t < SR; ++t) {
                    float v[V];
#pragma unroll
                    for (int e = 0; e < V; ++e) v[e] = out_r[t] * y[e];
#pragma unroll
                    for (int s = 0; s < SR; ++s)
#pragma unroll
                        for (int e = 0; e < V; ++e) v[e] = fmaf(mix_r[s * SR + t], xs[s][e], v[e]);
                    StVec<V>::store(xn + (size_t)t * a.W, v);
#pragma unroll
                    for (int e = 0; e < V; ++e) u[e] = fmaf(in_r[t], v[e], u[e]);
                }
            } else {
#pragma unroll
                for (int s = 0; s < SR; ++s)
#pragma unroll
                    for (int e = 0; e < V; ++e) u[e] = fmaf(in_r[s], xs[s][e], u[e]);
            }
        } else {
            // any number of streams (V == 1): the old elements are read again for every new one, so they must not be
            // overwritten before all are formed: the new ones go through shared memory, one column of S a thread
            if (a.y != nullptr) {
                for (int p = 0; p < a.n_y; ++p) y[0] += a.y[(size_t)p * y_stride + (size_t)row * a.W + c];
                float* col = sums + ST_MAX_CLUSTER + threadIdx.x;
                for (int t = 0; t < S; ++t) {
                    float v = a.out[t] * y[0];
                    for (int s = 0; s < S; ++s) v = fmaf(a.mix[s * S + t], x[s * s_step + c], v);
                    col[t * blockDim.x] = v;
                }
                for (int t = 0; t < S; ++t) {
                    const float v = col[t * blockDim.x];
                    a.x_new[((size_t)row * S + t) * a.W + c] = v;
                    u[0] = fmaf(a.in != nullptr ? a.in[t] : 1.f, v, u[0]);
                }
            } else {
                for (int s = 0; s < S; ++s) u[0] = fmaf(a.in != nullptr ? a.in[s] : 1.f, x[s * s_step + c], u[0]);
            }
        }
        if (a.next != nullptr) {
            StVec<V>::store(u_s + (c - c_lo), u);
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(u[e], u[e], ss);
        }
    }
    if (a.next == nullptr) return;                   // (the whole cluster returns)
    float total = block_sum(ss, red);
    if (meet) {
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
        if (threadIdx.x < cluster) {                 // this block's sum to every block of the row
            uint32_t remote;
            const uint32_t mine = (uint32_t)__cvta_generic_to_shared(sums + rank);
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(mine), "r"((int)threadIdx.x));
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(total) : "memory");
        }
        st_cluster_sync();
        total = 0.f;
        for (int r = 0; r < cluster; ++r) total += sums[r];
    }
    const float r = rsqrtf(total / (float)a.W + a.eps);
    T* out = reinterpret_cast<T*>(a.next) + (size_t)row * a.W;
    for (int c = c_lo + V * (int)threadIdx.x; c < c_hi; c += V * (int)blockDim.x) {       // a thread reads what it wrote
        float u[V], w[V];
        StVec<V>::load(u_s + (c - c_lo), u);
        StVec<V>::weight(a.w, a.w_is_f32, c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = u[e] * r * w[e];
        StVec<V>::put(out + c, u);
    }
}

template <typename T, int V, int S_>
static int st_launch(const StreamsArgs& a, int rows, int cluster, int threads, cudaStream_t st) {
    const int share = ((a.W / V + cluster - 1) / cluster) * V;
    const size_t smem = (size_t)(share + 34 + ST_MAX_CLUSTER + (S_ == 0 ? a.S * threads : 0)) * sizeof(float);
    if (smem > 200 * 1024) return RF_ERR_UNSUPPORTED;
    static size_t configured = 48 * 1024;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(streams_update_kernel<T, V, S_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = smem;
    }
    if (cluster > 1) rf_launch_cluster(streams_update_kernel<T, V, S_>, dim3(rows * cluster), dim3(threads), smem, st, cluster, a, cluster);
    else rf_launch(streams_update_kernel<T, V, S_>, dim3(rows), dim3(threads), smem, st, a, 1);
    RF_LAUNCH_CHECK();
    return 0;
}

template <typename T>
static int st_dispatch(const StreamsArgs& a, int rows, cudaStream_t st) {
    auto whole = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = a.W % 4 == 0 && whole(a.x) && whole(a.y) && whole(a.x_new) && whole(a.w) && whole(a.next) && a.S <= 8;
    if (!vec) {
        return st_launch<T, 1, 0>(a, rows, 1, 128, st);
    }
    // few rows: a row's columns over several blocks, so that the row's streams are fetched by several multiprocessors
    int cluster = 1;
    while (cluster < ST_MAX_CLUSTER && rows * cluster * 2 <= 148 && a.W / (cluster * 2) >= 256) cluster *= 2;
    const int per = (a.W / 4 + cluster - 1) / cluster;
    int threads = (per + 31) / 32 * 32;
    if (threads > 256) threads = rows >= 148 ? 256 : 512;
    if (threads > (per + 31) / 32 * 32) threads = (per + 31) / 32 * 32;
    if (threads < 64) threads = 64;
    switch (a.S) {
        case 1: return st_launch<T, 4, 1>(a, rows, cluster, threads, st);
        case 2: return st_launch<T, 4, 2>(a, rows, cluster, threads, st);
        case 3: return st_launch<T, 4, 3>(a, rows, cluster, threads, st);
        case 4: return st_launch<T, 4, 4>(a, rows, cluster, threads, st);
        case 5: return st_launch<T, 4, 5>(a, rows, cluster, threads, st);
        case 6: return st_launch<T, 4, 6>(a, rows, cluster, threads, st);
        case 7: return st_launch<T, 4, 7>(a, rows, cluster, threads, st);
        default: return st_launch<T, 4, 8>(a, rows, cluster, threads, st);
    }
}

// ---------------------------------------------------------------- embedding of a token and of the pair it ends
// The row of a pair is (previous * mul_prev + current * mul_cur) mod buckets, the multipliers given modulo buckets, the
// products in 64-bit; a sequence's first token takes row `buckets`.  state [slots][2]: the token at position p lies at
// p & 1, so a step of one token that runs again (launched ahead of the host and dropped) finds its previous token still
// there.  The block of a sequence's first new token reads the state and then writes it.
template <typename T, int V4>
__global__ void __launch_bounds__(512)
pair_embed_kernel(const T* __restrict__ table, const T* __restrict__ pairs, const int* __restrict__ ids,
                  const int* __restrict__ tok_seq, const int* __restrict__ tok_pos, const int* __restrict__ seq_slot,
                  const int* __restrict__ cu_q, int* __restrict__ state, const void* __restrict__ w, int w_is_f32,
                  float* __restrict__ out, int H, int V, float scale, long long mul_prev, long long mul_cur,
                  long long buckets, float eps) {
    extern __shared__ float sm[];                    // [H], 34
    __shared__ int row_s;
    float* red = sm + H;
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    int id = ids[t];
    id = id < 0 ? 0 : (id >= V ? V - 1 : id);        // ids are validated on the host; never read outside
    if (threadIdx.x == 0 && pairs != nullptr) {
        const int seq = tok_seq[t], pos = tok_pos[t], first = cu_q[seq], slot = seq_slot[seq];
        long long row = buckets;
        if (pos > 0) {
            int prev = t > first ? ids[t - 1] : state[2 * slot + ((pos - 1) & 1)];
            prev = prev < 0 ? 0 : (prev >= V ? V - 1 : prev);
            row = ((long long)prev * mul_prev + (long long)id * mul_cur) % buckets;
        }
        row_s = (int)row;
        if (t == first) {
            const int last = cu_q[seq + 1] - 1;
            state[2 * slot + ((pos + last - first) & 1)] = ids[last];
        }
    }
    __syncthreads();
    const T* e = table + (size_t)id * H;
    const T* p = pairs != nullptr ? pairs + (size_t)row_s * H : nullptr;
    float ss = 0.f;
    for (int c = V4 * threadIdx.x; c < H; c += V4 * blockDim.x) {
        float v[V4], x[V4];
        StVec<V4>::weight(e, sizeof(T) == 4, c, v);
        if (p != nullptr) StVec<V4>::weight(p, sizeof(T) == 4, c, x);
#pragma unroll
        for (int i = 0; i < V4; ++i) {
            v[i] *= scale;
            if (p != nullptr) v[i] += x[i];
            ss = fmaf(v[i], v[i], ss);
        }
        StVec<V4>::store(sm + c, v);
    }
    const float r = w != nullptr ? rsqrtf(block_sum(ss, red) / (float)H + eps) : 1.f;
    float* o = out + (size_t)t * H;
    for (int c = V4 * threadIdx.x; c < H; c += V4 * blockDim.x) {      // a thread reads what it wrote
        float v[V4], x[V4];
        StVec<V4>::load(sm + c, v);
        if (w != nullptr) {
            StVec<V4>::weight(w, w_is_f32, c, x);
#pragma unroll
            for (int i = 0; i < V4; ++i) v[i] *= r * x[i];
        }
        StVec<V4>::store(o + c, v);
    }
}

template <typename T>
static int launch_pair_embed(const void* table, const void* pairs, const int* ids, const int* tok_seq, const int* tok_pos,
                             const int* seq_slot, const int* cu_q, int* state, const void* w, int w_is_f32, float* out, int T_,
                             int H, int V, float scale, long long mul_prev, long long mul_cur, long long buckets, float eps,
                             cudaStream_t st) {
    if (T_ <= 0) return 0;
    if (pairs != nullptr && (state == nullptr || buckets <= 0 || buckets >= (1ll << 31) || mul_prev < 0 || mul_prev >= buckets ||
                             mul_cur < 0 || mul_cur >= buckets))
        return RF_ERR_BAD_ARG;
    const size_t smem = (size_t)(H + 34) * sizeof(float);
    if (smem > 200 * 1024) return RF_ERR_UNSUPPORTED;
    auto whole = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
    const bool vec = H % 4 == 0 && whole(table) && whole(pairs) && whole(w) && whole(out);
    auto kernel = vec ? pair_embed_kernel<T, 4> : pair_embed_kernel<T, 1>;
    static size_t configured[2] = {48 * 1024, 48 * 1024};
    if (smem > configured[vec]) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured[vec] = smem;
    }
    int threads = ((vec ? H / 4 : H) + 31) / 32 * 32;
    threads = threads < 64 ? 64 : (threads > 512 ? 512 : threads);
    rf_launch(kernel, dim3(T_), dim3(threads), smem, st, reinterpret_cast<const T*>(table), reinterpret_cast<const T*>(pairs),
              ids, tok_seq, tok_pos, seq_slot, cu_q, state, w, w_is_f32, out, H, V, scale, mul_prev, mul_cur, buckets, eps);
    RF_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------- x <- factor * x, in place (logits)
__global__ void scale_kernel(float* __restrict__ x, size_t n, float factor) {
    pdl_trigger();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) x[i] *= factor;
}

extern "C" {

// x [rows or more][x_streams][W] float32 with x_streams 1 (all S streams equal) or S; y: n_y partial sums [n_y][rows][W]
// or null (then nothing is updated and pick may choose the rows); x_new [rows][S][W]; next [rows][W] in the compute dtype
// (dtype 0 float32, 1 bfloat16) or null; in null: the plain sum of the streams.
int rf_streams_update(int dtype, const float* x, int x_streams, const float* y, int n_y, const float* mix, const float* out,
                      float* x_new, const float* in, const void* w, int w_is_f32, float eps, void* next, const int* pick, int S,
                      int W, int rows, cudaStream_t st) {
    if (rows <= 0) return 0;
    if (S < 1 || W < 1 || (x_streams != 1 && x_streams != S)) return RF_ERR_BAD_ARG;
    if (y != nullptr && (n_y < 1 || mix == nullptr || out == nullptr || x_new == nullptr || pick != nullptr)) return RF_ERR_BAD_ARG;
    if (y == nullptr && next == nullptr) return RF_ERR_BAD_ARG;
    if (next != nullptr && w == nullptr) return RF_ERR_BAD_ARG;
    const StreamsArgs a{x, x_streams, y, n_y, mix, out, x_new, in, w, w_is_f32, eps, next, pick, S, W};
    return dtype == 0 ? st_dispatch<float>(a, rows, st) : st_dispatch<__nv_bfloat16>(a, rows, st);
}

int rf_pair_embed(int dtype, const void* table, const void* pairs, const int* ids, const int* tok_seq, const int* tok_pos,
                  const int* seq_slot, const int* cu_q, int* state, const void* w, int w_is_f32, float* out, int T_, int H, int V,
                  float scale, long long mul_prev, long long mul_cur, long long buckets, float eps, cudaStream_t st) {
    return dtype == 0 ? launch_pair_embed<float>(table, pairs, ids, tok_seq, tok_pos, seq_slot, cu_q, state, w, w_is_f32, out, T_,
                                                 H, V, scale, mul_prev, mul_cur, buckets, eps, st)
                      : launch_pair_embed<__nv_bfloat16>(table, pairs, ids, tok_seq, tok_pos, seq_slot, cu_q, state, w, w_is_f32,
                                                         out, T_, H, V, scale, mul_prev, mul_cur, buckets, eps, st);
}

int rf_scale(float* x, long long n, float factor, cudaStream_t st) {
    if (n <= 0) return 0;
    const long long blocks = (n + 255) / 256;
    rf_launch(scale_kernel, dim3((unsigned)(blocks > 148 * 16 ? 148 * 16 : blocks)), dim3(256), 0, st, x, (size_t)n, factor);
    RF_LAUNCH_CHECK();
    return 0;
}

}
