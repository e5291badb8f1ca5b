// Attention of single tokens over cached latents (one row [latent | rotated part] a position, shared by all heads) on the
// 5th-generation tensor cores.
//
// Every head's query has been folded into the latent's space (q = [W_uk^T q_dim | q_rot], as long as a cache row), so the
// scores of all heads are products with the SAME rows, and so are the values (the rows' first `rank` numbers): attention
// with one key-value head whose cache is read once for all heads.  Heads are few (16 to 64 at a time), keys and latent
// dimensions many, so the products run transposed, with the cache row tile as the A operand both times and the heads as
// the MMA's N:
//     S^T [64 keys x heads]  = C Q^T         A: the page's tile, K-major; B: the queries, K-major
//     O^T [rank x heads]    += C^T P^T       A: the SAME tile read as an MN-major operand (dimensions on the rows); B: the
//                                            weights, written to shared memory by the softmax warps
// so a page comes into shared memory once (TMA, 128-byte swizzle, two or more stages) and is used for both.
// A CTA owns (token, group of heads) and every splits-th page; the CTAs of a token are a thread-block cluster and merge
// their (reference, sum, O) through distributed shared memory: no scratch memory, no atomics.
//   warp 0  TMA producer (pages older than the step are asked for before the dependency wait)
//   warp 1  issues the MMAs, scores up to two pages ahead of the softmax
//   warps 2-5  softmax: the 64 rows of an M = 64 accumulator lie in the first 16 lanes of each 32-lane quarter of tensor
//           memory, so a lane below 16 owns one key and all heads.  The exponentials' reference of a head moves only when
//           some score exceeds it by more than 8 (log2 units): one vote a page instead of a maximum a head; sums of weights
//           stay per lane until the end.
#include "tcgen05_common.cuh"

#define LD_THREADS 192
#define LD_PAGE_BLOCK (RF_PAGE * 128)                // bytes of 64 columns of a page
#define LD_MAX_SPLITS 16

struct LatentDecode {
    __nv_bfloat16* out;                              // [T][heads][rank]
    const int *tok_seq, *tok_pos, *seq_slot, *seq_start, *block_table;
    int max_pages;
    int heads, rank;
    int nb, n_steps;                                 // 64-column blocks of a row; 16-column MMA steps of a score
    int m_blocks;                                    // 128-row blocks of O^T
    int stages, tmem_cols;
    float scale;
    int span, splits;
    int* status;
};

__device__ __forceinline__ uint32_t ld_rank() { uint32_t r; asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ void ld_cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ uint32_t ld_peer(uint32_t addr, int rank) {
    uint32_t r;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
    return r;
}
__device__ __forceinline__ float2 ld_pull2(uint32_t addr) {
    float2 v;
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(addr) : "memory");
    return v;
}
__device__ __forceinline__ float4 ld_pull4(uint32_t addr) {
    float4 v;
    asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
    return v;
}
__device__ __forceinline__ void ld_group_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ bool ld_group_any(bool mine) {        // whether any of the 128 softmax threads says so
    uint32_t any;
    asm volatile("{\n\t.reg .pred p, q;\n\t"
                 "setp.ne.u32 q, %1, 0;\n\t"
                 "barrier.cta.red.or.pred p, 1, 128, q;\n\t"
                 "selp.u32 %0, 1, 0, p;\n\t}" : "=r"(any) : "r"((uint32_t)mine) : "memory");
    return any != 0;
}
// Whether the phase of parity `parity` is over; never suspends the thread.
__device__ __forceinline__ bool ld_test(uint32_t bar, uint32_t parity) {
    uint32_t ok;
    asm volatile("{\n\t.reg .pred p;\n\t"
                 "mbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
                 "selp.u32 %0, 1, 0, p;\n\t}" : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
    return ok != 0;
}
// Over the 16 lanes of each half warp: lane l ends with op(v[l % 16] of all of them); 15 exchanges instead of 16 x 4.
template <bool MAX>
__device__ __forceinline__ float ld_scatter16(float* v, int lane) {
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int j = 0; j < o; ++j) {
            const float send = up ? v[j] : v[j + o], keep = up ? v[j + o] : v[j];
            const float got = __shfl_xor_sync(0xffffffffu, send, o);
            v[j] = MAX ? fmaxf(keep, got) : keep + got;
        }
    }
    return v[0];
}
// bf16 x bf16 -> f32; a_mn: A is MN-major
__device__ __forceinline__ uint32_t ld_idesc(int m, int n, int a_mn) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)a_mn << 15) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(m >> 4) << 24);
}

template <int NH>
__global__ void __launch_bounds__(LD_THREADS, 1)
attention_latent_decode_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_c, LatentDecode a) {
    extern __shared__ __align__(1024) uint8_t smem[];              // no static shared memory: the window starts aligned
    const uint32_t tile_bytes = a.nb * LD_PAGE_BLOCK;
    uint8_t* c_s = smem;                                           // [stages][nb][64][128 B]; at the end the partial O
    uint8_t* q_s = c_s + (size_t)a.stages * tile_bytes;            // [nb][NH][128 B]
    uint8_t* p_s = q_s + (size_t)a.nb * NH * 128;                  // [2][NH][128 B]
    float* m_s = reinterpret_cast<float*>(p_s + 2 * NH * 128);     // [NH] the heads' references (log2 units)
    float* l_s = m_s + NH;                                         // [NH][2] the heads' references and sums, for the merge
    float* corr_s = l_s + 2 * NH;                                      // [NH]
    float* part_s = corr_s + NH;                                   // [4][NH] per-warp maxima, then sums
    float* wts_s = part_s + 4 * NH;                                // [LD_MAX_SPLITS][NH][2] the merge: references (then weights) and sums
    uint64_t* bars = reinterpret_cast<uint64_t*>(wts_s + 2 * LD_MAX_SPLITS * NH);
    // q_full, s_full[2], p_ready[2], pv_done[2] (two each: no barrier completes two phases between two looks of a waiter),
    // c_full[4], c_free[4]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
    int& abort_flag = *reinterpret_cast<int*>(tmem_slot + 1);
    const uint32_t b_q = smem_u32(&bars[0]), b_sfull = smem_u32(&bars[1]), b_pready = smem_u32(&bars[3]);
    const uint32_t b_pvdone = smem_u32(&bars[5]), b_cfull = smem_u32(&bars[7]), b_cfree = smem_u32(&bars[11]);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int split = a.splits > 1 ? (int)ld_rank() : 0;
    const int t = blockIdx.z, h0 = blockIdx.y * NH;
    const int seq = a.tok_seq[t], pos = a.tok_pos[t];
    const int* bt = a.block_table + (size_t)a.seq_slot[seq] * a.max_pages;
    const int lo = rf_first_key(pos, a.span);
    const int p_lo = lo / RF_PAGE + split, p_hi = pos / RF_PAGE;
    const int n_t = p_hi >= p_lo ? (p_hi - p_lo) / a.splits + 1 : 0;

    if (threadIdx.x == 0) {
        abort_flag = 0;
        mbar_init(b_q, 1);
        for (int s = 0; s < 2; ++s) { mbar_init(b_sfull + 8 * s, 1); mbar_init(b_pready + 8 * s, 128); mbar_init(b_pvdone + 8 * s, 1); }
        for (int s = 0; s < 4; ++s) { mbar_init(b_cfull + 8 * s, 1); mbar_init(b_cfree + 8 * s, 1); }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_q) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_c) : "memory");
    }
    if (warp == 1) {
        tcgen05_alloc(smem_u32(tmem_slot), a.tmem_cols);
        tcgen05_relinquish();
    }
    if (threadIdx.x >= 64 && threadIdx.x - 64 < NH) { m_s[threadIdx.x - 64] = -INFINITY; }
    tcgen05_fence_before();
    __syncthreads();
    tcgen05_fence_after();
    // only now may the kernels behind this one start: they take tensor memory too, and they give it back only after this
    // kernel has finished
    pdl_trigger();
    const uint32_t tmem_base = *tmem_slot;
    const uint32_t tmem_s = tmem_base, tmem_o = tmem_base + 2 * NH;

    if (warp == 0) {
        if (lane == 0) {
            auto load = [&](int i) -> bool {
                const int st = i % a.stages;
                if (!mbar_wait(b_cfree + 8 * st, ((i / a.stages) & 1) ^ 1, &abort_flag)) return false;
                mbar_expect_tx(b_cfull + 8 * st, tile_bytes);
                const int row = bt[p_lo + i * a.splits] * RF_PAGE;
                const uint32_t dst = smem_u32(c_s) + st * tile_bytes;
                for (int b = 0; b < a.nb; ++b) tma_load_2d(dst + b * LD_PAGE_BLOCK, &map_c, b * 64, row, b_cfull + 8 * st);
                return true;
            };
            const int old_pages = a.seq_start[seq] / RF_PAGE;      // pages below this were complete before the step
            int i = 0;
            bool ok = true;
            for (; ok && i < n_t && i < a.stages && p_lo + i * a.splits < old_pages; ++i) ok = load(i);
            pdl_wait();
            mbar_expect_tx(b_q, a.nb * NH * 128);
            for (int b = 0; b < a.nb; ++b) tma_load_2d(smem_u32(q_s) + b * NH * 128, &map_q, b * 64, t * a.heads + h0, b_q);
            for (; ok && i < n_t; ++i) ok = load(i);
        }
    } else if (warp == 1) {
        if (elect_one()) {
            const uint32_t idesc_s = ld_idesc(64, NH, 0), idesc_o = ld_idesc(128, NH, 1);
            bool ok = mbar_wait(b_q, 0, &abort_flag);              // (also with no page of its own: the copy must have landed)
            // Two kinds of work, each in page order: the scores of page si (its copy has landed, the softmax has read the scores of
            // page si - 2) and the values of page vi (its weights are written).  Values first: they free a place in the ring.
            // Neither waits behind the other: waiting for page si's copy with page vi's weights at hand would hold up the very copy.
            int si = 0, vi = 0;
            unsigned long long t0 = 0;
            for (int spin = 0; ok && vi < n_t; ++spin) {
                if (vi < si && ld_test(b_pready + 8 * (vi & 1), (vi >> 1) & 1)) {
                    tcgen05_fence_after();
                    const int cnt = min(RF_PAGE, pos + 1 - (p_lo + vi * a.splits) * RF_PAGE), st = vi % a.stages;
                    const int k_steps = (cnt + 15) >> 4;           // 16 keys each; rows behind the last key are zeroed up to there
                    uint64_t cd = make_smem_desc_mn(smem_u32(c_s) + st * tile_bytes, LD_PAGE_BLOCK);
                    const uint64_t pd = make_smem_desc(smem_u32(p_s) + (vi & 1) * NH * 128);
                    // a step of 16 keys is 16 rows of 128 bytes further in C and 32 bytes in P
                    if (k_steps == 4) {
                        for (int mb = 0; mb < a.m_blocks; ++mb, cd += (2 * LD_PAGE_BLOCK) >> 4) {
                            tcgen05_mma_bf16(tmem_o + mb * NH, cd, pd, idesc_o, vi ? 1u : 0u);
                            tcgen05_mma_bf16(tmem_o + mb * NH, cd + 128, pd + 2, idesc_o, 1u);
                            tcgen05_mma_bf16(tmem_o + mb * NH, cd + 256, pd + 4, idesc_o, 1u);
                            tcgen05_mma_bf16(tmem_o + mb * NH, cd + 384, pd + 6, idesc_o, 1u);
                        }
                    } else {
                        for (int mb = 0; mb < a.m_blocks; ++mb, cd += (2 * LD_PAGE_BLOCK) >> 4)
                            for (int ks = 0; ks < k_steps; ++ks)
                                tcgen05_mma_bf16(tmem_o + mb * NH, cd + 128 * ks, pd + 2 * ks, idesc_o, (vi | ks) ? 1u : 0u);
                    }
                    tcgen05_commit(b_cfree + 8 * st);
                    tcgen05_commit(b_pvdone + 8 * (vi & 1));
                    ++vi;
                    spin = 0; t0 = 0;
                } else if (si < n_t && si < vi + 2 && ld_test(b_cfull + 8 * (si % a.stages), (si / a.stages) & 1)) {
                    tcgen05_fence_after();
                    uint64_t cd = make_smem_desc(smem_u32(c_s) + (si % a.stages) * tile_bytes), qd = make_smem_desc(smem_u32(q_s));
                    const uint32_t d = tmem_s + (si & 1) * NH;
                    const int whole = a.n_steps >> 2;               // blocks of four steps, then the rest of the row
                    for (int b = 0; b < whole; ++b, cd += LD_PAGE_BLOCK >> 4, qd += (NH * 128) >> 4) {
                        tcgen05_mma_bf16(d, cd, qd, idesc_s, b ? 1u : 0u);
                        tcgen05_mma_bf16(d, cd + 2, qd + 2, idesc_s, 1u);
                        tcgen05_mma_bf16(d, cd + 4, qd + 4, idesc_s, 1u);
                        tcgen05_mma_bf16(d, cd + 6, qd + 6, idesc_s, 1u);
                    }
                    for (int k = 0; k < (a.n_steps & 3); ++k) tcgen05_mma_bf16(d, cd + 2 * k, qd + 2 * k, idesc_s, (whole | k) ? 1u : 0u);
                    tcgen05_commit(b_sfull + 8 * (si & 1));
                    ++si;
                    spin = 0; t0 = 0;
                } else if ((spin & 63) == 63) {                    // bounded, like every wait here
                    if (*(volatile int*)&abort_flag) ok = false;
                    const unsigned long long now = global_ns();
                    if (t0 == 0) t0 = now;
                    if (now - t0 > TC_WAIT_LIMIT_NS) { abort_flag = 1; ok = false; }
                }
            }
        }
    } else {
        const int quarter = warp & 3, tid = threadIdx.x - 64;
        const uint32_t lane_base = (uint32_t)(quarter * 32) << 16;
        const int my_row = quarter * 16 + lane;                    // of the page, for lanes below 16
        const float sl2 = a.scale * 1.4426950408889634f;
        const uint32_t p_chunk = (uint32_t)(my_row >> 3), p_byte = (uint32_t)(my_row & 7) * 2;
        constexpr bool REG = NH <= 32;                             // the heads' references also in registers
        float l[NH], m_reg[REG ? NH : 1];
#pragma unroll
        for (int h = 0; h < NH; ++h) { l[h] = 0.f; if (REG) m_reg[h] = -INFINITY; }
        auto ref = [&](int h) { return REG ? m_reg[REG ? h : 0] : m_s[h]; };
        pdl_wait();                                                // the output may still be read by a kernel before us
        bool ok = true;
        for (int i = 0; i < n_t; ++i) {
            const int key0 = (p_lo + i * a.splits) * RF_PAGE;
            ok = mbar_wait(b_sfull + 8 * (i & 1), (i >> 1) & 1, &abort_flag);
            // a CTA whose threads part ways must not meet in a barrier: the vote below also tells of a wait that ran out
            if (ok) tcgen05_fence_after();
            const int cnt = pos + 1 - key0;
            if (ok && cnt < RF_PAGE) {
                // rows behind the newest key were never written, or hold an earlier sequence's bits: their weights are zero, but
                // 0 * (whatever lies there) must be 0 as far as the last MMA step reaches
                const int st = i % a.stages, upto = (cnt + 15) & ~15;
                ok = mbar_wait(b_cfull + 8 * st, (i / a.stages) & 1, &abort_flag);
                if (ok) {
                    const uint32_t c_t = smem_u32(c_s) + st * tile_bytes;
                    for (int e = tid; e < (upto - cnt) * a.nb * 8; e += 128) {
                        const int c = e % (a.nb * 8), r = cnt + e / (a.nb * 8);
                        asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};"
                                     ::"r"(c_t + (c >> 3) * LD_PAGE_BLOCK + r * 128 + (c & 7) * 16), "r"(0u) : "memory");
                    }
                }
            }
            ok = __all_sync(0xffffffffu, ok);                      // (tensor memory is read by whole warps)
            float s[NH];
            if (ok) {
#pragma unroll
                for (int c0 = 0; c0 < NH; c0 += 16) tcgen05_ld16(tmem_s + (i & 1) * NH + lane_base + c0, reinterpret_cast<uint32_t*>(s) + c0);
                tcgen05_wait_ld();
            }
            const bool visible = lane < 16 && key0 + my_row <= pos && key0 + my_row >= lo;
            bool moves = !ok;
#pragma unroll
            for (int h = 0; h < NH; ++h) {
                s[h] = visible ? s[h] * sl2 : -INFINITY;
                moves |= s[h] > ref(h) + 8.f;
            }
            bool seen = i == 0;                                    // whether this step has looked at the previous P V's barrier
            if (ld_group_any(moves)) {
                if (ld_group_any(!ok)) { ok = false; break; }      // somebody gave up: all leave together
#pragma unroll
                for (int c0 = 0; c0 < NH; c0 += 16) {
                    float v[16];
#pragma unroll
                    for (int j = 0; j < 16; ++j) v[j] = s[c0 + j];
                    const float w = ld_scatter16<true>(v, lane);   // (the upper half warp holds no keys)
                    if (lane < 16) part_s[quarter * NH + c0 + lane] = w;
                }
                ld_group_sync();
                if (tid < NH) {
                    const float m_old = m_s[tid];
                    const float m_new = fmaxf(m_old, fmaxf(fmaxf(part_s[tid], part_s[NH + tid]), fmaxf(part_s[2 * NH + tid], part_s[3 * NH + tid])));
                    corr_s[tid] = m_old == -INFINITY ? 0.f : at_exp2(m_old - m_new);
                    m_s[tid] = m_new;
                }
                ld_group_sync();
#pragma unroll
                for (int h = 0; h < NH; ++h) { l[h] *= corr_s[h]; if (REG) m_reg[h] = m_s[h]; }
                if (i > 0) {
                    ok = mbar_wait(b_pvdone + 8 * ((i - 1) & 1), ((i - 1) >> 1) & 1, &abort_flag);
                    seen = true;
                    if (ok) {
                        tcgen05_fence_after();
#pragma unroll 1
                        for (int c0 = 0; c0 < a.m_blocks * NH; c0 += 16) {
                            uint32_t r[16];
                            tcgen05_ld16(tmem_o + lane_base + c0, r);
                            tcgen05_wait_ld();
#pragma unroll
                            for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * corr_s[(c0 + j) % NH]);
                            tcgen05_st16(tmem_o + lane_base + c0, r);
                        }
                        asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
                    }
                }
            }
            // the weights, transposed: row = head, 64 keys = 128 bytes, 16-byte pieces swizzled by the row
            if (lane < 16) {
                const uint32_t p_t = smem_u32(p_s) + (i & 1) * NH * 128 + p_byte;
#pragma unroll
                for (int h = 0; h < NH; ++h) {
                    const float p = at_exp2(s[h] - ref(h));
                    l[h] += p;
                    const unsigned short b = __bfloat16_as_ushort(__float2bfloat16_rn(p));
                    asm volatile("st.shared.u16 [%0], %1;" ::"r"(p_t + h * 128 + ((p_chunk ^ (h & 7)) << 4)), "h"(b) : "memory");
                }
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");      // weights and cleared rows are for the MMA to read
            tcgen05_fence_before();
            at_arrive(b_pready + 8 * (i & 1));
            if (!seen) {
                const bool got = mbar_wait(b_pvdone + 8 * ((i - 1) & 1), ((i - 1) >> 1) & 1, &abort_flag);
                (void)got;                                         // a wait that ran out shows in the next vote (abort_flag is set)
            }
        }
        if (ok && n_t > 0) ok = mbar_wait(b_pvdone + 8 * ((n_t - 1) & 1), ((n_t - 1) >> 1) & 1, &abort_flag);
        // sums over the keys
#pragma unroll
        for (int c0 = 0; c0 < NH; c0 += 16) {
            const float w = ld_scatter16<false>(l + c0, lane);
            if (lane < 16) part_s[quarter * NH + c0 + lane] = w;
        }
        ld_group_sync();
        if (tid < NH) {
            const float sum = (part_s[tid] + part_s[NH + tid]) + (part_s[2 * NH + tid] + part_s[3 * NH + tid]);
            *reinterpret_cast<float2*>(l_s + 2 * tid) = make_float2(m_s[tid], sum);
            corr_s[tid] = sum > 0.f ? 1.f / sum : 0.f;
        }
        ld_group_sync();
        if (n_t > 0) {
            tcgen05_fence_after();
            const int row = (a.rank + 3) / 4 * 4;
            float* o_s = reinterpret_cast<float*>(c_s);            // [NH][row]: every page of the ring has been used
            const int hn = a.splits > 1 ? NH : min(NH, a.heads - h0);
            for (int mb = 0; mb < a.m_blocks; mb += 2) {           // two blocks' reads in flight
                const int d = mb * 128 + quarter * 32 + lane;
                const bool on0 = d < a.rank, on1 = mb + 1 < a.m_blocks && d + 128 < a.rank;
#pragma unroll
                for (int c0 = 0; c0 < NH; c0 += 16) {
                    uint32_t r[2][16];
                    tcgen05_ld16(tmem_o + mb * NH + lane_base + c0, r[0]);
                    if (mb + 1 < a.m_blocks) tcgen05_ld16(tmem_o + (mb + 1) * NH + lane_base + c0, r[1]);
                    tcgen05_wait_ld();
                    if (a.splits > 1) {
                        float* o = o_s + c0 * row + d;
#pragma unroll
                        for (int j = 0; j < 16; ++j, o += row) {
                            if (on0) o[0] = __uint_as_float(r[0][j]);
                            if (on1) o[128] = __uint_as_float(r[1][j]);
                        }
                        continue;
                    }
                    __nv_bfloat16* o = a.out + ((size_t)t * a.heads + h0 + c0) * a.rank + d;
                    if (c0 + 16 <= hn) {
#pragma unroll
                        for (int j = 0; j < 16; ++j, o += a.rank) {
                            if (on0) o[0] = __float2bfloat16_rn(__uint_as_float(r[0][j]) * corr_s[c0 + j]);
                            if (on1) o[128] = __float2bfloat16_rn(__uint_as_float(r[1][j]) * corr_s[c0 + j]);
                        }
                    } else {
#pragma unroll
                        for (int j = 0; j < 16; ++j, o += a.rank) {
                            if (c0 + j < hn && on0) o[0] = __float2bfloat16_rn(__uint_as_float(r[0][j]) * corr_s[c0 + j]);
                            if (c0 + j < hn && on1) o[128] = __float2bfloat16_rn(__uint_as_float(r[1][j]) * corr_s[c0 + j]);
                        }
                    }
                }
            }
        }
    }
    if (a.splits > 1) {
        // ---- the CTAs of a token merge: CTA r finishes the dimensions r * per .. of all heads, from every CTA's O (in its ring's
        // memory by now), reference and sum; 16 bytes a load, the loads of eight CTAs in flight.
        __syncthreads();
        ld_cluster_sync();
        const int tid = threadIdx.x, hn = min(NH, a.heads - h0);
        const int row = (a.rank + 3) / 4 * 4, per = ((a.rank + a.splits - 1) / a.splits + 3) / 4 * 4;
        const int dn4 = (max(0, min(per, a.rank - split * per)) + 3) / 4;
        auto pull = [&](int e, int r0, float4* x) {
            const int h = e / dn4, d4 = e - h * dn4;
            const uint32_t at = smem_u32(c_s) + (uint32_t)(h * row + split * per + 4 * d4) * 4;
#pragma unroll
            for (int u = 0; u < 8; ++u)
                if (r0 + u < a.splits) x[u] = ld_pull4(ld_peer(at, r0 + u));
        };
        for (int e = tid; e < a.splits * NH; e += LD_THREADS)
            *reinterpret_cast<float2*>(wts_s + 2 * e) = ld_pull2(ld_peer(smem_u32(l_s + 2 * (e % NH)), e / NH));
        float4 x[8];
        if (tid < hn * dn4) pull(tid, 0, x);                       // under way while the weights are made
        __syncthreads();
        if (tid < NH) {
            float top = -INFINITY, sum = 0.f;
#pragma unroll 4
            for (int r = 0; r < a.splits; ++r) top = fmaxf(top, wts_s[(r * NH + tid) * 2]);
#pragma unroll 4
            for (int r = 0; r < a.splits; ++r) {
                const float m = wts_s[(r * NH + tid) * 2];
                const float w = m == -INFINITY ? 0.f : at_exp2(m - top);
                sum = fmaf(w, wts_s[(r * NH + tid) * 2 + 1], sum);
                wts_s[(r * NH + tid) * 2] = w;
            }
            const float inv = sum > 0.f ? 1.f / sum : 0.f;
#pragma unroll 4
            for (int r = 0; r < a.splits; ++r) wts_s[(r * NH + tid) * 2] *= inv;
        }
        __syncthreads();
        for (int e = tid; e < hn * dn4; e += LD_THREADS) {
            const int h = e / dn4, d = split * per + 4 * (e - h * dn4);
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int r0 = 0; r0 < a.splits; r0 += 8) {             // ranks in order
                if (e != tid || r0 > 0) pull(e, r0, x);
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    const float w = r0 + u < a.splits ? wts_s[((r0 + u) * NH + h) * 2] : 0.f;
                    if (w != 0.f) {                                // (a CTA without a page has nothing in its memory)
                        o.x = fmaf(w, x[u].x, o.x); o.y = fmaf(w, x[u].y, o.y); o.z = fmaf(w, x[u].z, o.z); o.w = fmaf(w, x[u].w, o.w);
                    }
                }
            }
            __nv_bfloat16* dst = a.out + ((size_t)t * a.heads + h0 + h) * a.rank + d;
            if (a.rank % 4 == 0) {
                *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(o.x, o.y), pack_bf16x2(o.z, o.w));
            } else {
                const float v[4] = {o.x, o.y, o.z, o.w};
                for (int i = 0; i < 4; ++i)
                    if (d + i < a.rank) dst[i] = __float2bfloat16_rn(v[i]);
            }
        }
        ld_cluster_sync();                                         // nobody leaves while its memory is read
    }
    tcgen05_fence_before();
    __syncthreads();
    if (warp == 1) {
        tcgen05_fence_after();
        tcgen05_dealloc(tmem_base, a.tmem_cols);
    }
    if (threadIdx.x == 0 && abort_flag && a.status) atomicExch(a.status, 9);
}

// ---------------------------------------------------------------- host side
struct LatentDecodePlan { int nh, nb, m_blocks, stages, cols; size_t smem; };

static bool ld_plan(int heads, int rank, int ld, LatentDecodePlan* p) {
    if (heads < 1 || rank < 1 || ld < rank || ld % 8) return false;
    const int nb = (ld + 63) / 64, mb = (rank + 127) / 128;
    for (int nh = heads <= 16 ? 16 : (heads <= 32 ? 32 : 64); nh >= 16; nh /= 2) {
        int cols = 32;
        while (cols < (2 + mb) * nh) cols *= 2;
        if (cols > 512) continue;
        const size_t fixed = (size_t)nb * nh * 128 + 2 * nh * 128 + (size_t)(8 + 2 * LD_MAX_SPLITS) * nh * 4 + 15 * 8 + 16;
        const size_t tile = (size_t)nb * LD_PAGE_BLOCK, limit = 227 * 1024;
        if (fixed + tile > limit) continue;
        int stages = (int)((limit - fixed) / tile);
        if (stages > 4) stages = 4;
        // the merge keeps [nh][rank in whole fours] floats where the ring was
        if ((size_t)nh * (rank + 4) * 4 > stages * tile) continue;
        *p = LatentDecodePlan{nh, nb, mb, stages, cols, fixed + stages * tile};
        // as many CTAs on a multiprocessor as its tensor memory serves, no more: a CTA that waits for tensor memory while its
        // cluster's other CTAs hold theirs could wait for good
        const size_t least = 228 * 1024 / (512 / cols + 1) + 1;
        if (p->smem < least) p->smem = least;
        // O^T's last block may read a column block behind the row (dimensions that nobody stores)
        const size_t reach = stages * tile + (2 * mb > nb ? (size_t)(2 * mb - nb) * LD_PAGE_BLOCK : 0);
        if (reach > limit) continue;
        if (p->smem < reach) p->smem = reach;
        return true;
    }
    return false;
}

template <int NH>
static int ld_launch(const CUtensorMap& mq, const CUtensorMap& mc, const LatentDecode& a, int T, int groups, size_t smem, cudaStream_t st) {
    static size_t configured = 0;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(attention_latent_decode_kernel<NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        if ((e = cudaFuncSetAttribute(attention_latent_decode_kernel<NH>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1)) != cudaSuccess) return (int)e;
        configured = smem;
    }
    const dim3 grid(a.splits, groups, T);
    cudaError_t e = a.splits > 1 ? rf_launch_cluster(attention_latent_decode_kernel<NH>, grid, dim3(LD_THREADS), smem, st, a.splits, mq, mc, a)
                                 : rf_launch(attention_latent_decode_kernel<NH>, grid, dim3(LD_THREADS), smem, st, mq, mc, a);
    if (e != cudaSuccess) return (int)e;
    RF_LAUNCH_CHECK();
    return 0;
}

extern "C" {

int rf_attention_latent_decode_supported(int heads, int rank, int ld) {
    LatentDecodePlan p;
    return ld_plan(heads, rank, ld, &p) && encode_fn() != nullptr;
}
// Groups of heads that a token is worked on by (each a CTA or a cluster of CTAs).
int rf_attention_latent_decode_groups(int heads, int rank, int ld) {
    LatentDecodePlan p;
    return ld_plan(heads, rank, ld, &p) ? (heads + p.nh - 1) / p.nh : 0;
}

// q [T][heads][ld], pages [n_pages][RF_PAGE][ld] (rows [latent rank | rotated part | zeros]), out [T][heads][rank].
int rf_attention_latent_decode(const void* q, const void* pages, long long n_pages, void* out, const int* tok_seq, const int* tok_pos,
                               const int* seq_slot, const int* seq_start, const int* block_table, int max_pages, int heads, int rank,
                               int ld, float scale, int span, int splits, int T, int* status, cudaStream_t st) {
    if (T <= 0) return 0;
    LatentDecodePlan p;
    if (!ld_plan(heads, rank, ld, &p) || T > 65535) return RF_ERR_UNSUPPORTED;
    if (splits < 1 || splits > LD_MAX_SPLITS || (reinterpret_cast<uintptr_t>(out) & 15)) return RF_ERR_BAD_ARG;
    CUtensorMap mq, mc;
    int e;
    if ((e = make_map(&mq, q, (long long)T * heads, ld, ld, p.nh)) || (e = make_map(&mc, pages, n_pages * RF_PAGE, ld, ld, RF_PAGE))) return e;
    LatentDecode a{};
    a.out = reinterpret_cast<__nv_bfloat16*>(out);
    a.tok_seq = tok_seq; a.tok_pos = tok_pos; a.seq_slot = seq_slot; a.seq_start = seq_start; a.block_table = block_table;
    a.max_pages = max_pages; a.heads = heads; a.rank = rank; a.nb = p.nb; a.n_steps = (ld + 15) / 16; a.m_blocks = p.m_blocks;
    a.stages = p.stages; a.tmem_cols = p.cols; a.scale = scale; a.span = span; a.splits = splits; a.status = status;
    const int groups = (heads + p.nh - 1) / p.nh;
    if (p.nh == 16) return ld_launch<16>(mq, mc, a, T, groups, p.smem, st);
    if (p.nh == 32) return ld_launch<32>(mq, mc, a, T, groups, p.smem, st);
    return ld_launch<64>(mq, mc, a, T, groups, p.smem, st);
}

}
