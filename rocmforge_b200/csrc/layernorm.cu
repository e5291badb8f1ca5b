// Layer norm, and the residual update of blocks whose norms are layer norms.
//
//   stream_update   one pass over the rows of the 32-bit residual stream h [rows][H]:
//                     m = routed + gate * dense                      (either may be missing)
//                       routed  sum over a token's choices, in their order, of weight_k * row_k, where row_k is a row of
//                               the experts' sorted outputs or, for an identity expert, the feed-forward's input itself
//                       dense   [n][rows][H] partial sums of a K-split product, added in index order; gate (optional) is
//                               sigmoid of one number per row
//                     m <- m / sqrt(mean(m^2) + post_eps) * w_post   (with w_post)
//                     h += m
//                     y = (h - mean) / sqrt(mean((h - mean)^2) + eps) * w + b   in the compute dtype (with w, b), or
//                     y = h in the compute dtype (without)
//                   Without addends it norms the rows that `rows` lists (null: all) and leaves h alone.
//   side_gate       g[t, j] = gelu(z[t, j]) * table[token_t, col0 + j] (gelu by tanh), in the compute dtype; z comes as
//                   the product's matrix or as its partial sums
// All sums and statistics are 32-bit.  A row's result depends on the row alone.
#include "common.cuh"

struct RoutedRows {
    const float* y;          // [pairs][H], sorted by expert
    const int* inv;          // [rows * top]: the sorted row of a pair
    const int* idx;          // [rows * top]: a pair's expert
    const float* w;          // [rows * top]
    const void* x;           // the feed-forward's input, of the compute dtype
    long long x_stride;
    int top, experts;        // a pair whose expert is not below `experts` is an identity expert's
};
struct DenseRows {
    const float* p;
    long long part_stride;
    int n;
    const float* gate;       // logits, one per row, gate_stride apart
    int gate_stride;
};
struct UpdateNorms {
    const void* w_post;
    const void* w;
    const void* b;
    int post_is_f32, w_is_f32;
    float post_eps, eps;
};

template <int V> struct Pack { float v[V]; };

template <int V> __device__ __forceinline__ Pack<V> ld_f32(const float* p) {
    Pack<V> r;
    if constexpr (V == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
    } else r.v[0] = *p;
    return r;
}
template <int V> __device__ __forceinline__ void st_f32(float* p, const Pack<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int V, typename T> __device__ __forceinline__ Pack<V> ld_any(const T* p) {
    Pack<V> r;
    if constexpr (V == 4 && sizeof(T) == 2) {
        const uint2 x = *reinterpret_cast<const uint2*>(p);
        r.v[0] = __uint_as_float(x.x << 16); r.v[1] = __uint_as_float(x.x & 0xffff0000u);
        r.v[2] = __uint_as_float(x.y << 16); r.v[3] = __uint_as_float(x.y & 0xffff0000u);
    } else if constexpr (V == 4) {
        r = ld_f32<4>(reinterpret_cast<const float*>(p));
    } else r.v[0] = Cvt<T>::to_f32(*p);
    return r;
}
template <int V> __device__ __forceinline__ Pack<V> ld_vec(const void* p, int is_f32, int c) {
    return is_f32 ? ld_any<V>(reinterpret_cast<const float*>(p) + c) : ld_any<V>(reinterpret_cast<const __nv_bfloat16*>(p) + c);
}
template <int V, typename T> __device__ __forceinline__ void st_any(T* p, const Pack<V>& r) {
    if constexpr (V == 4 && sizeof(T) == 2) {
        __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 x;
        x.x = *reinterpret_cast<uint32_t*>(&a); x.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = x;
    } else if constexpr (V == 4) {
        st_f32<4>(reinterpret_cast<float*>(p), r);
    } else *p = Cvt<T>::from_f32(r.v[0]);
}

// A block per row.  V elements a thread at a time: 4 where every row starts on a 16-byte boundary, else 1.  (Rows of widths that the
// kernel below does not take; the row stays in shared memory between the passes.)
template <typename T, int V>
__global__ void __launch_bounds__(1024)
stream_update_kernel(float* __restrict__ h, const int* __restrict__ rows, RoutedRows rt, DenseRows dn, UpdateNorms nm,
                     T* __restrict__ y, int H) {
    extern __shared__ __align__(16) float row[];     // [H], 34 for the sums behind it
    float* red = row + (H + 3) / 4 * 4;
    pdl_trigger();
    const float invH = 1.f / (float)H;
    pdl_wait();
    const size_t t = blockIdx.x;
    const size_t src = (size_t)(rows != nullptr ? rows[t] : (int)t) * H;
    const bool adds = rt.y != nullptr || dn.p != nullptr;
    const float gate = dn.gate != nullptr ? 1.f / (1.f + expf(-dn.gate[t * dn.gate_stride])) : 1.f;
    float acc = 0.f;                                 // of m^2 (with w_post) or of h
    for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
        Pack<V> m;
#pragma unroll
        for (int u = 0; u < V; ++u) m.v[u] = 0.f;
        if (dn.p != nullptr) {
            const float* p = dn.p + t * H + c;
#pragma unroll 8
            for (int s = 0; s < dn.n; ++s) {
                const Pack<V> a = ld_f32<V>(p + (size_t)s * dn.part_stride);
#pragma unroll
                for (int u = 0; u < V; ++u) m.v[u] += a.v[u];
            }
#pragma unroll
            for (int u = 0; u < V; ++u) m.v[u] *= gate;
        }
        if (rt.y != nullptr) {
            Pack<V> r;
#pragma unroll
            for (int u = 0; u < V; ++u) r.v[u] = 0.f;
#pragma unroll 4
            for (int k = 0; k < rt.top; ++k) {
                const size_t pr = t * rt.top + k;
                const float w = rt.w[pr];
                const Pack<V> a = rt.idx[pr] < rt.experts
                    ? ld_f32<V>(rt.y + (size_t)rt.inv[pr] * H + c)
                    : ld_any<V>(reinterpret_cast<const T*>(rt.x) + t * rt.x_stride + c);
#pragma unroll
                for (int u = 0; u < V; ++u) r.v[u] = fmaf(w, a.v[u], r.v[u]);
            }
#pragma unroll
            for (int u = 0; u < V; ++u) m.v[u] = r.v[u] + m.v[u];
        }
        if (nm.w_post != nullptr) {
#pragma unroll
            for (int u = 0; u < V; ++u) acc += m.v[u] * m.v[u];
        } else {
            const Pack<V> old = ld_f32<V>(h + src + c);
#pragma unroll
            for (int u = 0; u < V; ++u) { m.v[u] += old.v[u]; acc += m.v[u]; }
            if (adds) st_f32<V>(h + src + c, m);
        }
        st_f32<V>(row + c, m);
    }
    if (nm.w_post != nullptr) {
        const float r = rsqrtf(block_sum(acc, red) * invH + nm.post_eps);
        acc = 0.f;
        for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {          // a thread reads what it wrote
            Pack<V> m = ld_f32<V>(row + c);
            const Pack<V> w = ld_vec<V>(nm.w_post, nm.post_is_f32, c), old = ld_f32<V>(h + src + c);
#pragma unroll
            for (int u = 0; u < V; ++u) { m.v[u] = fmaf(m.v[u] * r, w.v[u], old.v[u]); acc += m.v[u]; }
            st_f32<V>(h + src + c, m);
            st_f32<V>(row + c, m);
        }
    }
    if (y == nullptr) return;
    if (nm.w == nullptr) {
        for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) st_any<V>(y + t * H + c, ld_f32<V>(row + c));
        return;
    }
    const float mean = block_sum(acc, red) * invH;
    float dev = 0.f;
    for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
        const Pack<V> m = ld_f32<V>(row + c);
#pragma unroll
        for (int u = 0; u < V; ++u) { const float d = m.v[u] - mean; dev = fmaf(d, d, dev); }
    }
    const float r = rsqrtf(block_sum(dev, red) * invH + nm.eps);
    for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
        Pack<V> m = ld_f32<V>(row + c);
        const Pack<V> w = ld_vec<V>(nm.w, nm.w_is_f32, c), b = ld_vec<V>(nm.b, nm.w_is_f32, c);
#pragma unroll
        for (int u = 0; u < V; ++u) m.v[u] = fmaf((m.v[u] - mean) * r, w.v[u], b.v[u]);
        st_any<V>(y + t * H + c, m);
    }
}

// The same with a row in registers: NV groups of four elements a thread, asked for all at once, and one barrier a sum (every warp
// adds the warps' sums up for itself, always by the same tree).  Rows of H = 4 * NV * threads elements at most.
template <typename T, int NV, int MAXT>
__global__ void __launch_bounds__(MAXT)
stream_update_regs_kernel(float* __restrict__ h, const int* __restrict__ rows, RoutedRows rt, DenseRows dn, UpdateNorms nm,
                          T* __restrict__ y, int H) {
    __shared__ float red[3][32];
    pdl_trigger();
    const float invH = 1.f / (float)H;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5, step = blockDim.x * 4, c0 = threadIdx.x * 4;
    auto row_sum = [&](float v, int i) {
        v = warp_sum(v);
        if (lane == 0) red[i][warp] = v;
        __syncthreads();
        return warp_sum(lane < n_warps ? red[i][lane] : 0.f);
    };
    pdl_wait();
    const size_t t = blockIdx.x;
    const size_t src = (size_t)(rows != nullptr ? rows[t] : (int)t) * H;
    const bool adds = rt.y != nullptr || dn.p != nullptr;
    Pack<4> m[NV], old[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * step;
        m[i].v[0] = m[i].v[1] = m[i].v[2] = m[i].v[3] = 0.f;
        old[i] = m[i];
        if (c < H) old[i] = ld_f32<4>(h + src + c);
    }
    if (dn.p != nullptr) {
        const float* p = dn.p + t * H + c0;
#pragma unroll 4
        for (int s = 0; s < dn.n; ++s, p += dn.part_stride) {
#pragma unroll
            for (int i = 0; i < NV; ++i)
                if (c0 + i * step < H) {
                    const Pack<4> a = ld_f32<4>(p + i * step);
#pragma unroll
                    for (int u = 0; u < 4; ++u) m[i].v[u] += a.v[u];
                }
        }
        if (dn.gate != nullptr) {
            const float gate = 1.f / (1.f + expf(-dn.gate[t * dn.gate_stride]));
#pragma unroll
            for (int i = 0; i < NV; ++i)
#pragma unroll
                for (int u = 0; u < 4; ++u) m[i].v[u] *= gate;
        }
    }
    if (rt.y != nullptr) {
        Pack<4> r[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) r[i].v[0] = r[i].v[1] = r[i].v[2] = r[i].v[3] = 0.f;
        for (int k = 0; k < rt.top; ++k) {
            const size_t pr = t * rt.top + k;
            const float w = rt.w[pr];
            const bool real = rt.idx[pr] < rt.experts;
            const float* yr = rt.y + (size_t)rt.inv[pr] * H + c0;
            const T* xr = reinterpret_cast<const T*>(rt.x) + t * rt.x_stride + c0;
#pragma unroll
            for (int i = 0; i < NV; ++i)
                if (c0 + i * step < H) {
                    const Pack<4> a = real ? ld_f32<4>(yr + i * step) : ld_any<4>(xr + i * step);
#pragma unroll
                    for (int u = 0; u < 4; ++u) r[i].v[u] = fmaf(w, a.v[u], r[i].v[u]);
                }
        }
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int u = 0; u < 4; ++u) m[i].v[u] = r[i].v[u] + m[i].v[u];
    }
    if (nm.w_post != nullptr) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int u = 0; u < 4; ++u) ss += m[i].v[u] * m[i].v[u];
        const float r = rsqrtf(row_sum(ss, 0) * invH + nm.post_eps);
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (c0 + i * step < H) {
                const Pack<4> w = ld_vec<4>(nm.w_post, nm.post_is_f32, c0 + i * step);
#pragma unroll
                for (int u = 0; u < 4; ++u) m[i].v[u] = fmaf(m[i].v[u] * r, w.v[u], old[i].v[u]);
            }
    } else {
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int u = 0; u < 4; ++u) m[i].v[u] += old[i].v[u];
    }
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        if (c0 + i * step < H && adds) st_f32<4>(h + src + c0 + i * step, m[i]);
#pragma unroll
        for (int u = 0; u < 4; ++u) sum += m[i].v[u];
    }
    if (y == nullptr) return;
    if (nm.w == nullptr) {
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (c0 + i * step < H) st_any<4>(y + t * H + c0 + i * step, m[i]);
        return;
    }
    const float mean = row_sum(sum, 1) * invH;
    float dev = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
        if (c0 + i * step < H)
#pragma unroll
            for (int u = 0; u < 4; ++u) { const float d = m[i].v[u] - mean; dev = fmaf(d, d, dev); }
    const float r = rsqrtf(row_sum(dev, 2) * invH + nm.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i)
        if (c0 + i * step < H) {
            const Pack<4> w = ld_vec<4>(nm.w, nm.w_is_f32, c0 + i * step), b = ld_vec<4>(nm.b, nm.w_is_f32, c0 + i * step);
#pragma unroll
            for (int u = 0; u < 4; ++u) m[i].v[u] = fmaf((m[i].v[u] - mean) * r, w.v[u], b.v[u]);
            st_any<4>(y + t * H + c0 + i * step, m[i]);
        }
}

template <typename T, int NV, int MAXT>
static int go_regs(float* h, const int* rows, const RoutedRows& rt, const DenseRows& dn, const UpdateNorms& nm, void* y, int R, int H,
                   cudaStream_t st) {
    const int threads = ((H / 4 + NV - 1) / NV + 31) / 32 * 32;
    rf_launch(stream_update_regs_kernel<T, NV, MAXT>, dim3(R), dim3(threads), 0, st, h, rows, rt, dn, nm, reinterpret_cast<T*>(y), H);
    RF_LAUNCH_CHECK();
    return 0;
}

template <typename T, int V>
static int go_update(float* h, const int* rows, const RoutedRows& rt, const DenseRows& dn, const UpdateNorms& nm, void* y, int R,
                     int H, cudaStream_t st) {
    const size_t smem = ((size_t)(H + 3) / 4 * 4 + 34) * sizeof(float);
    if (smem > 200 * 1024) return RF_ERR_UNSUPPORTED;
    static size_t configured = 48 * 1024;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(stream_update_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = smem;
    }
    // few rows: as many threads as there are groups of elements (the pass is a chain of loads); many: small blocks, several
    // on a multiprocessor.  Which of the two it is follows the number of rows, and only the order of a row's sums with it.
    int threads = (H / V + 31) / 32 * 32;
    const int most = R <= 296 ? 1024 : 256;
    threads = threads < 64 ? 64 : (threads > most ? most : threads);
    rf_launch(stream_update_kernel<T, V>, dim3(R), dim3(threads), smem, st, h, rows, rt, dn, nm, reinterpret_cast<T*>(y), H);
    RF_LAUNCH_CHECK();
    return 0;
}

template <typename T>
static int launch_update(float* h, const int* rows, const RoutedRows& rt, const DenseRows& dn, const UpdateNorms& nm, void* y,
                         int R, int H, cudaStream_t st) {
    if (R <= 0) return 0;
    const bool adds = rt.y != nullptr || dn.p != nullptr;
    if (H <= 0 || (rows != nullptr && adds) || (!adds && y == nullptr) || (dn.p != nullptr && dn.n < 1)) return RF_ERR_BAD_ARG;
    if (rt.y != nullptr && (!rt.inv || !rt.idx || !rt.w || !rt.x || rt.top < 1)) return RF_ERR_BAD_ARG;
    if ((nm.w_post != nullptr && !adds) || ((nm.w == nullptr) != (nm.b == nullptr))) return RF_ERR_BAD_ARG;
    auto on16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = H % 4 == 0 && on16(h) && on16(rt.y) && on16(rt.x) && rt.x_stride % 4 == 0 && on16(dn.p) &&
                     dn.part_stride % 4 == 0 && on16(nm.w_post) && on16(nm.w) && on16(nm.b) && on16(y);
    if (vec && R <= 296) {                               // few rows: a group of elements a thread (the pass is a chain of loads)
        if (H <= 4096) return go_regs<T, 1, 1024>(h, rows, rt, dn, nm, y, R, H, st);
        if (H <= 8192) return go_regs<T, 2, 1024>(h, rows, rt, dn, nm, y, R, H, st);
    } else if (vec) {                                    // many: small blocks, several on a multiprocessor
        if (H <= 1024) return go_regs<T, 1, 256>(h, rows, rt, dn, nm, y, R, H, st);
        if (H <= 2048) return go_regs<T, 2, 256>(h, rows, rt, dn, nm, y, R, H, st);
        if (H <= 4096) return go_regs<T, 4, 256>(h, rows, rt, dn, nm, y, R, H, st);
        if (H <= 8192) return go_regs<T, 8, 256>(h, rows, rt, dn, nm, y, R, H, st);
    }
    return vec ? go_update<T, 4>(h, rows, rt, dn, nm, y, R, H, st) : go_update<T, 1>(h, rows, rt, dn, nm, y, R, H, st);
}

// ---------------------------------------------------------------- a gated part of the token's row of a table
template <typename T>
__global__ void __launch_bounds__(256)
side_gate_kernel(const void* __restrict__ z, int n_partials, long long part_stride, int z_stride, const T* __restrict__ table,
                 long long table_stride, int col0, const int* __restrict__ tokens, T* __restrict__ out, int out_stride, int dim,
                 int vocab, size_t n) {
    pdl_trigger();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / out_stride;
        const int j = (int)(i - t * out_stride);
        float g = 0.f;                                // columns from dim on: padding of the product that follows
        if (j < dim) {
            float x = 0.f;
            if (n_partials > 0) {
                const float* p = reinterpret_cast<const float*>(z) + t * z_stride + j;
#pragma unroll 4
                for (int s = 0; s < n_partials; ++s) x += p[(size_t)s * part_stride];
            } else x = Cvt<T>::to_f32(reinterpret_cast<const T*>(z)[t * z_stride + j]);
            const int id = min(max(tokens[t], 0), vocab - 1);
            const float e = Cvt<T>::to_f32(table[(size_t)id * table_stride + col0 + j]);
            g = 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x))) * e;
        }
        out[i] = Cvt<T>::from_f32(g);
    }
}

template <typename T>
static int launch_side(const void* z, int n_partials, long long part_stride, int z_stride, const void* table, long long table_stride,
                       int col0, const int* tokens, void* out, int out_stride, int dim, int vocab, int T_, cudaStream_t st) {
    const size_t n = (size_t)T_ * out_stride;
    if (n == 0) return 0;
    if (dim < 1 || dim > out_stride || vocab < 1 || n_partials < 0 || col0 < 0 || col0 + dim > table_stride) return RF_ERR_BAD_ARG;
    const size_t blocks = (n + 255) / 256;
    rf_launch(side_gate_kernel<T>, dim3((unsigned)(blocks > 148 * 16 ? 148 * 16 : blocks)), dim3(256), 0, st, z, n_partials,
              part_stride, z_stride, reinterpret_cast<const T*>(table), table_stride, col0, tokens, reinterpret_cast<T*>(out),
              out_stride, dim, vocab, n);
    RF_LAUNCH_CHECK();
    return 0;
}

extern "C" {
// dtype: 0 = float32, 1 = bfloat16 (of y and of the routed rows' input).  See the top of the file; null pointers switch a part
// off.  rows: only without addends.  w and b are of one dtype (w_is_f32, else bfloat16).
int rf_stream_update(int dtype, float* h, const int* rows, const float* dense, int n_dense, long long part_stride,
                     const float* gate, int gate_stride, const float* routed, const int* inv, const int* idx, const float* rw,
                     const void* x, long long x_stride, int top, int experts, const void* w_post, int post_is_f32, float post_eps,
                     const void* w, const void* b, int w_is_f32, float eps, void* y, int R, int H, cudaStream_t st) {
    const RoutedRows rt{routed, inv, idx, rw, x, x_stride, top, experts};
    const DenseRows dn{dense, part_stride, n_dense, gate, gate_stride};
    const UpdateNorms nm{w_post, w, b, post_is_f32, w_is_f32, post_eps, eps};
    return dtype == 0 ? launch_update<float>(h, rows, rt, dn, nm, y, R, H, st)
                      : launch_update<__nv_bfloat16>(h, rows, rt, dn, nm, y, R, H, st);
}
// z: [T, z_stride] of dtype (n_partials 0) or n_partials float32 matrices [T, z_stride], part_stride apart; table [vocab,
// table_stride] of dtype; out [T, out_stride], zeros from column dim on.
int rf_side_gate(int dtype, const void* z, int n_partials, long long part_stride, int z_stride, const void* table,
                 long long table_stride, int col0, const int* tokens, void* out, int out_stride, int dim, int vocab, int T_,
                 cudaStream_t st) {
    return dtype == 0
        ? launch_side<float>(z, n_partials, part_stride, z_stride, table, table_stride, col0, tokens, out, out_stride, dim, vocab, T_, st)
        : launch_side<__nv_bfloat16>(z, n_partials, part_stride, z_stride, table, table_stride, col0, tokens, out, out_stride, dim, vocab, T_, st);
}
}
