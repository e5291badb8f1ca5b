// Prompt attention of a latent-caching mixer on the 5th-generation tensor cores.
//
// The step's sequences have their latents expanded into one matrix (a product before this kernel):
//     kv   [keys, ldkv]   a head's unrotated key part at column head * dim, its values at v_col + head * vdim
//     lat  [keys, ldl]    the cache rows themselves; columns rank .. rank + rot hold the rotated key part that all heads share
// The keys of sequence i are rows cu_k[i] .. cu_k[i + 1), position after position.  A query head is [dim | rot].
//
// A CTA owns 128 consecutive new tokens of one sequence and one head, as in attention_prefill_tc.cu, whose division of
// labour this kernel has (TMA producer, one MMA thread, four softmax warps with a row a thread, S in two buffers and O in
// tensor memory, P written back over the scores it was made from).  What differs: S is the sum of two products over the
// same accumulator, Q_dim K_dim^T out of kv's column block of the head and Q_rot K_rot^T out of the shared columns of lat, so
// the concatenated key never exists in memory; the three head sizes are free (dim and vdim multiples of 16, rot of 8) and
// independent; keys come from a matrix, not from pages; the epilogue may multiply by sigmoid(gate).
#include "tcgen05_common.cuh"

#define LP_THREADS 192
#define LP_BM 128
#define LP_BN 64

struct LatentPrefill {
    __nv_bfloat16* out; int out_stride;
    const __nv_bfloat16* gate; int gate_stride;      // [T][>= heads * vdim] or null
    const int* tiles;                                // (sequence, first new row) of every query tile
    const int *seq_start, *seq_nnew, *cu_q, *cu_k;
    int dim, rot, vdim, rank, v_col;
    int nq, nr, nv;                                  // 64-column blocks of a head's unrotated part, rotated part, values
    int k_stages, v_stages;
    int tmem_cols;
    float scale;
    int span;
    int* status;
};

// bf16 x bf16 -> f32, M = 128, N = n, A K-major, B K-major (b_mn = 0) or MN-major (b_mn = 1)
__device__ __forceinline__ uint32_t lp_idesc(int n, int b_mn) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)b_mn << 16) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(LP_BM >> 4) << 24);
}

__global__ void __launch_bounds__(LP_THREADS, 2)
attention_latent_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv,
                                const __grid_constant__ CUtensorMap map_lat, LatentPrefill a) {
    constexpr uint32_t QB = LP_BM * 128, KB = LP_BN * 128;             // bytes of a 64-column block of queries / keys
    extern __shared__ __align__(1024) uint8_t smem[];                  // no static shared memory: the window starts aligned
    const int nb = a.nq + a.nr;
    uint8_t* q_s = smem;                                               // [nb][128][128 B]
    uint8_t* k_s = q_s + (size_t)nb * QB;                              // [k_stages][nb][64][128 B]
    uint8_t* v_s = k_s + (size_t)a.k_stages * nb * KB;                 // [v_stages][nv][64][128 B]
    uint64_t* bars = reinterpret_cast<uint64_t*>(v_s + (size_t)a.v_stages * a.nv * KB);
    // q_full, k_full[2], k_free[2], s_full[2], p_ready[2], pv_done[2], v_full[2], v_free[2]; p_ready and pv_done alternate
    // from tile to tile so that no barrier completes two phases between two looks of one of its waiters
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
    int& abort_flag = *reinterpret_cast<int*>(tmem_slot + 1);
    const uint32_t b_q = smem_u32(&bars[0]), b_kfull = smem_u32(&bars[1]), b_kfree = smem_u32(&bars[3]);
    const uint32_t b_sfull = smem_u32(&bars[5]), b_pready = smem_u32(&bars[7]), b_pvdone = smem_u32(&bars[9]);
    const uint32_t b_vfull = smem_u32(&bars[11]), b_vfree = smem_u32(&bars[13]);

    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // the table is sorted by the keys a tile sees and walked backwards, heads fastest: the heaviest tiles start first
    const int tile_idx = gridDim.y - 1 - blockIdx.y;
    const int seq = a.tiles[2 * tile_idx], q0 = a.tiles[2 * tile_idx + 1];
    const int head = blockIdx.x;
    const int start = a.seq_start[seq], n_new = a.seq_nnew[seq];
    const int row_base = a.cu_q[seq] + q0, key_base = a.cu_k[seq];
    int rows_here = n_new - q0; if (rows_here > LP_BM) rows_here = LP_BM;
    const int pos_first = start + q0, pos_last = pos_first + rows_here - 1;
    const int kt_lo = rf_first_key(pos_first, a.span) / LP_BN, kt_hi = pos_last / LP_BN;
    const int n_kt = kt_hi - kt_lo + 1;

    if (threadIdx.x == 0) {
        abort_flag = 0;
        mbar_init(b_q, 1);
        for (int s = 0; s < 2; ++s) {
            mbar_init(b_kfull + 8 * s, 1); mbar_init(b_kfree + 8 * s, 1);
            mbar_init(b_vfull + 8 * s, 1); mbar_init(b_vfree + 8 * s, 1);
            mbar_init(b_sfull + 8 * s, 1); mbar_init(b_pready + 8 * s, 128); mbar_init(b_pvdone + 8 * s, 1);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_q) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_kv) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_lat) : "memory");
    }
    if (warp == 1) {
        tcgen05_alloc(smem_u32(tmem_slot), a.tmem_cols);
        tcgen05_relinquish();
    }
    tcgen05_fence_before();
    __syncthreads();
    tcgen05_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    const uint32_t tmem_s = tmem_base, tmem_o = tmem_base + 2 * LP_BN;
    pdl_wait();

    if (warp == 0) {
        // ---------------- producer
        if (lane == 0) {
            const int qc = head * (a.dim + a.rot);
            mbar_expect_tx(b_q, nb * QB);
            for (int b = 0; b < a.nq; ++b) tma_load_2d(smem_u32(q_s + b * QB), &map_q, qc + b * 64, row_base, b_q);
            for (int b = 0; b < a.nr; ++b) tma_load_2d(smem_u32(q_s + (a.nq + b) * QB), &map_q, qc + a.dim + b * 64, row_base, b_q);
            for (int t = 0; t < n_kt; ++t) {
                const int row = key_base + (kt_lo + t) * LP_BN;
                const int sk = a.k_stages == 2 ? t & 1 : 0, use_k = a.k_stages == 2 ? t >> 1 : t;
                uint8_t* kd = k_s + (size_t)sk * nb * KB;
                if (!mbar_wait(b_kfree + 8 * sk, (use_k & 1) ^ 1, &abort_flag)) break;
                mbar_expect_tx(b_kfull + 8 * sk, nb * KB);
                for (int b = 0; b < a.nq; ++b)
                    tma_load_2d(smem_u32(kd + b * KB), &map_kv, head * a.dim + b * 64, row, b_kfull + 8 * sk);
                for (int b = 0; b < a.nr; ++b)
                    tma_load_2d(smem_u32(kd + (a.nq + b) * KB), &map_lat, a.rank + b * 64, row, b_kfull + 8 * sk);
                const int sv = a.v_stages == 2 ? t & 1 : 0, use = a.v_stages == 2 ? t >> 1 : t;
                uint8_t* vd = v_s + (size_t)sv * a.nv * KB;
                if (!mbar_wait(b_vfree + 8 * sv, (use & 1) ^ 1, &abort_flag)) break;
                mbar_expect_tx(b_vfull + 8 * sv, a.nv * KB);
                for (int b = 0; b < a.nv; ++b)
                    tma_load_2d(smem_u32(vd + b * KB), &map_kv, a.v_col + head * a.vdim + b * 64, row, b_vfull + 8 * sv);
            }
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer
        if (elect_one()) {
            const uint32_t idesc_s = lp_idesc(LP_BN, 0), idesc_o = lp_idesc(a.vdim, 1);
            const int ks_dim = a.dim >> 4, ks_all = ks_dim + ((a.rot + 15) >> 4);
            auto issue_s = [&](int t) -> bool {          // the scores of tile t + 1 are computed under the softmax of tile t
                const int st = t & 1, sk = a.k_stages == 2 ? st : 0, use_k = a.k_stages == 2 ? t >> 1 : t;
                if (!mbar_wait(b_kfull + 8 * sk, use_k & 1, &abort_flag)) return false;
                tcgen05_fence_after();
                uint64_t kd = make_smem_desc(smem_u32(k_s + (size_t)sk * nb * KB)), qd = make_smem_desc(smem_u32(q_s));
                const uint32_t d = tmem_s + st * LP_BN;
                // block after block: the unrotated columns' steps, then the rotated ones' (a step is 32 bytes, 2 descriptor units)
                for (int b = 0; b < nb; ++b, qd += QB >> 4, kd += KB >> 4) {
                    const int left = b < a.nq ? ks_dim - 4 * b : ks_all - ks_dim - 4 * (b - a.nq);
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        if (k < left) tcgen05_mma_bf16(d, qd + 2 * k, kd + 2 * k, idesc_s, (b | k) ? 1u : 0u);
                }
                tcgen05_commit(b_sfull + 8 * st);
                tcgen05_commit(b_kfree + 8 * sk);
                return true;
            };
            bool ok = mbar_wait(b_q, 0, &abort_flag);
            if (ok && n_kt > 0) ok = issue_s(0);
            for (int t = 0; t < n_kt && ok; ++t) {
                const int st = t & 1;
                if (t + 1 < n_kt) { ok = issue_s(t + 1); if (!ok) break; }
                const int sv = a.v_stages == 2 ? st : 0, use = a.v_stages == 2 ? t >> 1 : t;
                ok = mbar_wait(b_pready + 8 * st, (t >> 1) & 1, &abort_flag);
                if (!ok) break;
                ok = mbar_wait(b_vfull + 8 * sv, use & 1, &abort_flag);
                if (!ok) break;
                tcgen05_fence_after();
                const uint32_t v_t = smem_u32(v_s + (size_t)sv * a.nv * KB);
#pragma unroll
                for (int ks = 0; ks < LP_BN / 16; ++ks)
                    tcgen05_mma_bf16_ts(tmem_o, tmem_s + st * LP_BN + ks * 8, make_smem_desc_mn(v_t + ks * 16 * 128, KB), idesc_o,
                                        (t | ks) ? 1u : 0u);
                tcgen05_commit(b_vfree + 8 * sv);
                tcgen05_commit(b_pvdone + 8 * st);
            }
        }
    } else {
        // ---------------- softmax, correction, epilogue: one thread per query row
        const int quarter = warp & 3, row = quarter * 32 + lane;
        const uint32_t lane_base = (uint32_t)(quarter * 32) << 16;
        const int pos_i = pos_first + row, lo_i = rf_first_key(pos_i, a.span);
        const bool row_ok = row < rows_here;
        const float sl2 = a.scale * 1.4426950408889634f;
        float m_ref = -INFINITY, l = 0.f;
        bool ok = true;
        for (int t = 0; t < n_kt; ++t) {
            const int st = t & 1, key0 = (kt_lo + t) * LP_BN;
            ok = mbar_wait(b_sfull + 8 * st, (t >> 1) & 1, &abort_flag);
            if (!ok) break;
            tcgen05_fence_after();
            const bool no_mask = key0 + LP_BN - 1 <= pos_first && rows_here == LP_BM && key0 >= rf_first_key(pos_last, a.span);
            float sc[LP_BN];
            {
                uint32_t r[32];
#pragma unroll
                for (int c0 = 0; c0 < LP_BN; c0 += 32) {
                    tcgen05_ld32(tmem_s + st * LP_BN + lane_base + c0, r);
                    tcgen05_wait_ld();
#pragma unroll
                    for (int j = 0; j < 32; ++j) sc[c0 + j] = __uint_as_float(r[j]);
                }
            }
            if (!no_mask) {
#pragma unroll
                for (int j = 0; j < LP_BN; ++j) {
                    const int key = key0 + j;
                    if (!(row_ok && key <= pos_i && key >= lo_i)) sc[j] = -INFINITY;
                }
            }
            float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int j = 0; j < LP_BN; j += 4) {
                mx4[0] = fmaxf(mx4[0], sc[j]); mx4[1] = fmaxf(mx4[1], sc[j + 1]);
                mx4[2] = fmaxf(mx4[2], sc[j + 2]); mx4[3] = fmaxf(mx4[3], sc[j + 3]);
            }
            const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * sl2;
            float corr = 1.f;                            // the reference moves only when a maximum grew by more than 8 (log2)
            if (mx > m_ref + 8.f) {
                corr = (m_ref == -INFINITY) ? 0.f : at_exp2(m_ref - mx);
                m_ref = mx;
            }
            const float nref = (m_ref == -INFINITY) ? 0.f : -m_ref;
            float sum4[4] = {0.f, 0.f, 0.f, 0.f};
            uint32_t pk[LP_BN / 2];
#pragma unroll
            for (int j = 0; j < LP_BN; j += 4) {
                const float p0 = at_exp2(fmaf(sc[j], sl2, nref)), p1 = at_exp2(fmaf(sc[j + 1], sl2, nref));
                const float p2 = at_exp2(fmaf(sc[j + 2], sl2, nref)), p3 = at_exp2(fmaf(sc[j + 3], sl2, nref));
                sum4[0] += p0; sum4[1] += p1; sum4[2] += p2; sum4[3] += p3;
                pk[j >> 1] = at_pack_bf16x2(p0, p1);
                pk[(j >> 1) + 1] = at_pack_bf16x2(p2, p3);
            }
            const float sum = (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
            tcgen05_st32(tmem_s + st * LP_BN + lane_base, pk);
            bool seen = false;
            if (t > 0 && __any_sync(0xffffffffu, corr != 1.f)) {
                ok = mbar_wait(b_pvdone + 8 * ((t - 1) & 1), ((t - 1) >> 1) & 1, &abort_flag);
                if (!ok) break;
                seen = true;
                tcgen05_fence_after();
#pragma unroll 1
                for (int c0 = 0; c0 < a.vdim; c0 += 16) {
                    uint32_t r[16];
                    tcgen05_ld16(tmem_o + lane_base + c0, r);
                    tcgen05_wait_ld();
#pragma unroll
                    for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * corr);
                    tcgen05_st16(tmem_o + lane_base + c0, r);
                }
            }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            l = l * corr + sum;
            tcgen05_fence_before();
            at_arrive(b_pready + 8 * st);
            if (t > 0 && !seen) {                        // every phase of a barrier is seen once
                ok = mbar_wait(b_pvdone + 8 * ((t - 1) & 1), ((t - 1) >> 1) & 1, &abort_flag);
                if (!ok) break;
            }
        }
        if (ok && n_kt > 0) ok = mbar_wait(b_pvdone + 8 * ((n_kt - 1) & 1), ((n_kt - 1) >> 1) & 1, &abort_flag);
        if (ok) {
            tcgen05_fence_after();
            const float inv = l > 0.f ? 1.f / l : 0.f;
            __nv_bfloat16* orow = a.out + (size_t)(row_base + row) * a.out_stride + (size_t)head * a.vdim;
            const __nv_bfloat16* grow = a.gate != nullptr ? a.gate + (size_t)(row_base + row) * a.gate_stride + (size_t)head * a.vdim : nullptr;
#pragma unroll 1
            for (int c0 = 0; c0 < a.vdim; c0 += 16) {
                uint32_t r[16];
                tcgen05_ld16(tmem_o + lane_base + c0, r);
                uint4 g[2];
                if (row_ok && grow != nullptr) {
                    g[0] = *reinterpret_cast<const uint4*>(grow + c0);
                    g[1] = *reinterpret_cast<const uint4*>(grow + c0 + 8);
                }
                tcgen05_wait_ld();
                if (row_ok) {
                    float v[16];
#pragma unroll
                    for (int j = 0; j < 16; ++j) v[j] = __uint_as_float(r[j]) * inv;
                    if (grow != nullptr) {
                        const uint32_t gw[8] = {g[0].x, g[0].y, g[0].z, g[0].w, g[1].x, g[1].y, g[1].z, g[1].w};
#pragma unroll
                        for (int j = 0; j < 8; ++j) {
                            v[2 * j] = __fdividef(v[2 * j], 1.f + __expf(-__uint_as_float(gw[j] << 16)));
                            v[2 * j + 1] = __fdividef(v[2 * j + 1], 1.f + __expf(-__uint_as_float(gw[j] & 0xffff0000u)));
                        }
                    }
#pragma unroll
                    for (int q = 0; q < 2; ++q)
                        *reinterpret_cast<uint4*>(orow + c0 + 8 * q) =
                            make_uint4(pack_bf16x2(v[8 * q], v[8 * q + 1]), pack_bf16x2(v[8 * q + 2], v[8 * q + 3]),
                                       pack_bf16x2(v[8 * q + 4], v[8 * q + 5]), pack_bf16x2(v[8 * q + 6], v[8 * q + 7]));
                }
            }
        }
    }
    tcgen05_fence_before();
    __syncthreads();
    if (warp == 1) {
        tcgen05_fence_after();
        tcgen05_dealloc(tmem_base, a.tmem_cols);
    }
    if (threadIdx.x == 0 && abort_flag && a.status) atomicExch(a.status, 8);
}

// ---------------------------------------------------------------- host side
static size_t lp_smem(int nb, int nv, int k_stages, int v_stages) {
    return (size_t)nb * LP_BM * 128 + (size_t)k_stages * nb * LP_BN * 128 + (size_t)v_stages * nv * LP_BN * 128 + 15 * 8 + 16;
}

extern "C" {

int rf_attention_latent_prefill_supported(int heads, int dim, int rot, int vdim, int rank) {
    if (heads < 1 || heads > 65535 || dim < 16 || dim % 16 || rot < 0 || rot % 8 || vdim < 16 || vdim % 16 || vdim > 256 || rank % 8) return 0;
    if (lp_smem((dim + 63) / 64 + (rot + 63) / 64, (vdim + 63) / 64, 1, 1) > 227 * 1024) return 0;
    return encode_fn() != nullptr;
}

// q [T][q_stride]: heads x [dim | rot] first; kv [n_keys][ldkv], lat [n_keys][ldl]; out [T][out_stride] (heads x vdim).
// span as in rf_first_key; gate null: none.
int rf_attention_latent_prefill(const void* q, int q_stride, int T, const void* kv, int ldkv, const void* lat, int ldl, int n_keys,
                                int v_col, void* out, int out_stride, const void* gate, int gate_stride, const int* tiles,
                                int n_tiles, const int* seq_start, const int* seq_nnew, const int* cu_q, const int* cu_k, int heads,
                                int dim, int rot, int vdim, int rank, float scale, int span, int* status, cudaStream_t st) {
    if (n_tiles <= 0) return 0;
    if (!rf_attention_latent_prefill_supported(heads, dim, rot, vdim, rank) || n_tiles > 65535) return RF_ERR_UNSUPPORTED;
    if ((reinterpret_cast<uintptr_t>(out) & 15) || out_stride % 8 || v_col % 8 || n_keys < 1 || rank + rot > ldl ||
        heads * dim > v_col || v_col + heads * vdim > ldkv || heads * (dim + rot) > q_stride)
        return RF_ERR_BAD_ARG;
    if (gate != nullptr && ((reinterpret_cast<uintptr_t>(gate) & 15) || gate_stride % 8)) return RF_ERR_BAD_ARG;
    CUtensorMap mq, mkv, ml;
    int e;
    if ((e = make_map(&mq, q, T, (long long)heads * (dim + rot), q_stride, LP_BM)) ||
        (e = make_map(&mkv, kv, n_keys, v_col + heads * vdim, ldkv, LP_BN)) ||
        (e = make_map(&ml, lat, n_keys, rank + rot, ldl, LP_BN)))
        return e;
    LatentPrefill a{};
    a.out = reinterpret_cast<__nv_bfloat16*>(out); a.out_stride = out_stride;
    a.gate = reinterpret_cast<const __nv_bfloat16*>(gate); a.gate_stride = gate_stride;
    a.tiles = tiles; a.seq_start = seq_start; a.seq_nnew = seq_nnew; a.cu_q = cu_q; a.cu_k = cu_k;
    a.dim = dim; a.rot = rot; a.vdim = vdim; a.rank = rank; a.v_col = v_col;
    a.nq = (dim + 63) / 64; a.nr = (rot + 63) / 64; a.nv = (vdim + 63) / 64;
    a.tmem_cols = vdim <= 128 ? 256 : 512;
    a.scale = scale; a.span = span; a.status = status;
    // Stages: as many as leave room for two CTAs on a multiprocessor (half of 228 KB less the 1 KB the system keeps for each),
    // or, where one CTA is all that fits, as many as fit.  Values come first: a tile's keys are used up a whole tile before its
    // values are, so one stage of keys is refilled in time and one of values is not.
    const int nb = a.nq + a.nr;
    const int forms[4][2] = {{2, 2}, {1, 2}, {2, 1}, {1, 1}};
    a.k_stages = 0;
    for (size_t limit : {(size_t)(113 * 1024), (size_t)(227 * 1024)})
        for (int f = 0; f < 4 && a.k_stages == 0; ++f)
            if (lp_smem(nb, a.nv, forms[f][0], forms[f][1]) <= limit) { a.k_stages = forms[f][0]; a.v_stages = forms[f][1]; }
    const size_t smem = lp_smem(nb, a.nv, a.k_stages, a.v_stages);
    static size_t configured = 0;
    if (smem > configured) {
        cudaError_t ce = cudaFuncSetAttribute(attention_latent_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (ce != cudaSuccess) return (int)ce;
        configured = smem;
    }
    cudaError_t ce = rf_launch(attention_latent_prefill_kernel, dim3(heads, n_tiles), dim3(LP_THREADS), smem, st, mq, mkv, ml, a);
    if (ce != cudaSuccess) return (int)ce;
    RF_LAUNCH_CHECK();
    return 0;
}

}
