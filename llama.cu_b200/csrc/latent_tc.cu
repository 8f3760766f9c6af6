// Absorbed latent attention of decode rounds on the 5th-generation tensor cores.
//
// All heads of a token attend the SAME cached rows, so both products are computed with the cache on the 128-row side of
// the MMA and the heads on N (16, 32 or 64), over one shared-memory copy of a tile of 128 positions:
//   scores   S^T[128 positions x heads]  = C[positions x latent]   Q^T     C as stored (K-major operand)
//   output   O^T[latent x heads]        += C^T[latent x positions] P       the same bytes as an MN-major operand
// S^T and O^T live in TMEM.  Per CTA (one row block of one token, one split of its context):
//   - warp 0 (one lane): TMA producer; a ring of pieces [128 positions x 128 latents], loaded page by page (two boxes of
//     64 latents, 128-byte swizzle); pieces return to the ring as the second product finishes with them;
//   - warp 1: MMA issuer (the whole warp runs the loop, so operand descriptors stay in uniform registers; one elected lane
//     issues);
//   - warps 2..5: softmax, one position per thread.  Weights are taken relative to a reference maximum per head that moves
//     only when some score exceeds it by more than a factor of 2^8 (which changes nothing but the weights' common scale): the
//     usual tile needs one vote, no reduction and no rescale.  When the reference moves, column maxima come from a
//     transposing butterfly over the warp and across the four warps, and O^T is rescaled in TMEM.  Probabilities go to
//     shared memory as bf16 rows of heads (an MN-major operand); the row sums are those of the rounded values.
// Rows of a tile past the context are zeroed in shared memory before the products.  Every wait is bounded: when one runs
// out the CTA records a status bit, waits for its own copies, frees its TMEM and returns.
#include "stack.cuh"
#include "tc.cuh"

namespace lcu {

typedef __nv_bfloat16 bf16;

constexpr int LT_THREADS = 192;
constexpr int LT_POS = 128;                // positions per tile
constexpr int LT_BOX = LT_POS * 128;       // bytes of [128 positions x 64 latents]
constexpr int LT_PIECE = 2 * LT_BOX;
constexpr int LT_MAX_SLOTS = 8;
constexpr float LT_GROW = 8.f;             // growth of a running maximum (in powers of two) that triggers a rescale

template <int N>
struct LtShared {
    unsigned long long full[LT_MAX_SLOTS], empty[LT_MAX_SLOTS], q_full, s_full, z_ready, p_ready, o_done;
    uint32_t tmem_base;
    int abort_flag;
    alignas(16) float mx[4][N];    // column maxima of each softmax warp
    alignas(16) float ref[4][N], corr[4][N];   // every warp's own copy of the reference maxima and the rescale factors
};

__device__ __forceinline__ void lt_tma_3d(uint32_t dst, const CUtensorMap *map, int x, int y, int z, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];"
                 ::"r"(dst), "l"(map), "r"(x), "r"(y), "r"(z), "r"(bar) : "memory");
}
// MN-major operand, 128-byte swizzle: 64 elements per 128-byte row, 64-element pieces LT_BOX bytes apart, groups of 8 rows
// (the K direction) 1024 bytes apart
__device__ __forceinline__ uint64_t lt_desc_mn(uint32_t saddr) {
    return (uint64_t)((saddr >> 4) & 0x3FFFu) | ((uint64_t)(LT_BOX >> 4) << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}
// probabilities [position][N heads], MN-major with the swizzle of their row size; groups of 8 positions 16 N bytes apart
template <int N>
__device__ __forceinline__ uint64_t lt_desc_p(uint32_t saddr) {
    constexpr uint64_t layout = N == 64 ? 2 : (N == 32 ? 4 : 6);  // 128-, 64-, 32-byte swizzle
    return (uint64_t)((saddr >> 4) & 0x3FFFu) | (1ull << 16) | ((uint64_t)N << 32) | (1ull << 46) | (layout << 61);
}
// byte offset of 16-byte chunk j (8 heads) of position p
template <int N>
__device__ __forceinline__ int lt_p_off(int p, int j) {
    const int x = N == 64 ? (p & 7) : (N == 32 ? ((p >> 1) & 3) : ((p >> 2) & 1));
    return p * (2 * N) + ((j ^ x) << 4);
}
__device__ __forceinline__ bool lt_elect() {
    uint32_t r;
    asm volatile("{\n .reg .pred p;\n elect.sync _|p, 0xffffffff;\n selp.u32 %0, 1, 0, p;\n}" : "=r"(r));
    return r != 0;
}
__device__ __forceinline__ float lt_exp2(float v) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
}
// barrier of the four softmax warps that also ORs a flag
__device__ __forceinline__ bool lt_sync_or(bool v) {
    uint32_t r;
    asm volatile("{\n .reg .pred p, q;\n setp.ne.u32 p, %1, 0;\n bar.red.or.pred q, 4, 128, p;\n selp.u32 %0, 1, 0, q;\n}"
                 : "=r"(r) : "r"((uint32_t)v) : "memory");
    return r != 0;
}
__device__ __forceinline__ void lt_st16(uint32_t taddr, const uint32_t r[16]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
                 ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
                 "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
}
__device__ __forceinline__ void lt_arrive(uint32_t bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory");
}
// barrier of the four softmax warps that also ANDs a flag, so that they leave a loop together
__device__ __forceinline__ bool lt_sync_and(bool ok) {
    uint32_t r;
    asm volatile("{\n .reg .pred p, q;\n setp.ne.u32 p, %1, 0;\n bar.red.and.pred q, 3, 128, p;\n selp.u32 %0, 1, 0, q;\n}"
                 : "=r"(r) : "r"((uint32_t)ok) : "memory");
    return r != 0;
}
// Reduction over the 32 lanes of CNT (16 or 32) values per lane: lane l ends with the result of value l % CNT.
template <int CNT, bool MAX>
__device__ __forceinline__ float lt_columns(float *v) {
    const int lane = threadIdx.x & 31;
    int n = CNT;
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) {
        if (n > o) {
#pragma unroll
            for (int i = 0; i < CNT / 2; ++i)
                if (i < n / 2) {
                    const float keep = (lane & o) ? v[i + n / 2] : v[i], send = (lane & o) ? v[i] : v[i + n / 2];
                    const float got = __shfl_xor_sync(0xffffffffu, send, o);
                    v[i] = MAX ? fmaxf(keep, got) : keep + got;
                }
            n /= 2;
        } else {
#pragma unroll
            for (int i = 0; i < CNT; ++i)
                if (i < n) {
                    const float got = __shfl_xor_sync(0xffffffffu, v[i], o);
                    v[i] = MAX ? fmaxf(v[i], got) : v[i] + got;
                }
        }
    }
    return v[0];
}

template <int N>
__global__ void __launch_bounds__(LT_THREADS, 1)
latent_tc_kernel(const LatentAttnArgs a, const __grid_constant__ CUtensorMap map_c, const __grid_constant__ CUtensorMap map_q, int n_slots, int tm_cols) {
    constexpr int GC = N < 32 ? N : 32, NG = N / GC;  // columns per butterfly, butterflies
    extern __shared__ unsigned char smem_raw[];
    unsigned char *smem = smem_raw + ((1024u - (tc_smem(smem_raw) & 1023u)) & 1023u);
    const int R = a.r_p, nbox = R / 64, npiece = (nbox + 1) / 2;
    unsigned char *ring = smem;                                    // [n_slots][LT_PIECE]
    unsigned char *Qs = ring + (size_t)n_slots * LT_PIECE;         // [nbox][N][128 bytes]
    unsigned char *Ps = Qs + (size_t)nbox * N * 128;               // [128 positions][N], swizzled
    LtShared<N> *sh = reinterpret_cast<LtShared<N> *>(Ps + (size_t)2 * N * 128);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    grid_dep_launch();
    if (tid == 0) {
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_c) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_q) : "memory");
    }

    // row block: one token, up to N of its heads
    const int bpt = (a.heads + N - 1) / N, req = (int)blockIdx.x / bpt, h0 = ((int)blockIdx.x - req * bpt) * N;
    const int row0 = req * a.heads + h0, rows = min(N, a.heads - h0);
    const int rr = req;  // a decode round: every request of it, in order
    const int ctx = a.req_pos[rr] + 1;
    const int sp = blockIdx.y;
    const int n_tiles = (ctx + LT_POS - 1) / LT_POS;
    const int tps = (n_tiles + a.splits - 1) / a.splits;
    const int my_splits = (n_tiles + tps - 1) / tps;
    if (sp >= my_splits) return;
    const int tile0 = sp * tps, tile1 = min(n_tiles, tile0 + tps);
    const int32_t *pages = a.page_table + (size_t)rr * a.pt_stride;

    if (tid == 0) {
        for (int i = 0; i < n_slots; ++i) {
            tc_mbar_init(tc_smem(&sh->full[i]), 1);
            tc_mbar_init(tc_smem(&sh->empty[i]), 1);
        }
        tc_mbar_init(tc_smem(&sh->q_full), 1);
        tc_mbar_init(tc_smem(&sh->s_full), 1);
        tc_mbar_init(tc_smem(&sh->z_ready), 128);
        tc_mbar_init(tc_smem(&sh->p_ready), 128);
        tc_mbar_init(tc_smem(&sh->o_done), 1);
        sh->abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tc_smem(&sh->tmem_base)), "r"(tm_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = sh->tmem_base, tmem_o = tmem + N;  // S^T in columns [0, N), O^T piece p in [N + p N, ...)
    const bool tail = tile1 * LT_POS > ctx;                  // the last tile has rows past the context
    auto stop = [&]() {
        atomicOr(a.status, 4u);
        sh->abort_flag = 1;
    };

    if (warp == 0 && lane == 0) {
        // ---------------- TMA producer
        grid_dep_wait();
        const uint32_t qb = tc_smem(&sh->q_full);
        tc_mbar_expect_tx(qb, (uint32_t)(nbox * N * 128));
        for (int k = 0; k < nbox; ++k) tc_tma_2d(tc_smem(Qs + (size_t)k * N * 128), &map_q, k * 64, row0, qb);
        int it = 0;
        const int pmask = (1 << a.page_shift) - 1;
        for (int tile = tile0; tile < tile1 && !sh->abort_flag; ++tile) {
            const int p0 = tile * LT_POS;
            const int halves = ctx - p0 > 64 ? 2 : 1;
            const int pg0 = pages[p0 >> a.page_shift], pg1 = halves > 1 ? pages[(p0 + 64) >> a.page_shift] : 0;
            for (int p = 0; p < npiece; ++p, ++it) {
                const int slot = it % n_slots;
                if (it >= n_slots && !tc_mbar_wait(tc_smem(&sh->empty[slot]), ((uint32_t)(it / n_slots) & 1u) ^ 1u, &sh->abort_flag)) {
                    stop();
                    break;
                }
                const uint32_t bar = tc_smem(&sh->full[slot]), dst = tc_smem(ring + (size_t)slot * LT_PIECE);
                const int boxes = min(2, nbox - 2 * p);
                tc_mbar_expect_tx(bar, (uint32_t)(boxes * halves * (LT_BOX / 2)));
                for (int b = 0; b < boxes; ++b) {
                    lt_tma_3d(dst + b * LT_BOX, &map_c, (2 * p + b) * 64, p0 & pmask, pg0, bar);
                    if (halves > 1) lt_tma_3d(dst + b * LT_BOX + LT_BOX / 2, &map_c, (2 * p + b) * 64, (p0 + 64) & pmask, pg1, bar);
                }
            }
        }
        if (sh->abort_flag) {  // copies in flight must land before the CTA gives its memory up
            int never = 0;
            tc_mbar_wait(qb, 0u, &never);
            for (int j = it > n_slots ? it - n_slots : 0; j < it; ++j)
                tc_mbar_wait(tc_smem(&sh->full[j % n_slots]), (uint32_t)(j / n_slots) & 1u, &never);
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer
        const uint32_t id_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
        const uint32_t id_o = id_s | (1u << 15) | (1u << 16);  // both operands MN-major
        const uint64_t ring_k = tc_desc(tc_smem(ring)), ring_mn = lt_desc_mn(tc_smem(ring)), q_k = tc_desc(tc_smem(Qs)), p_mn = lt_desc_p<N>(tc_smem(Ps));
        bool ok = __all_sync(0xffffffffu, tc_mbar_wait(tc_smem(&sh->q_full), 0u, &sh->abort_flag));
        int slot = 0;        // ring position of the tile's first piece
        uint32_t phase = 0;  // its parity
        for (int tile = tile0; tile < tile1 && ok; ++tile) {
            if (tail && tile == tile1 - 1) ok = __all_sync(0xffffffffu, tc_mbar_wait(tc_smem(&sh->z_ready), 0u, &sh->abort_flag));
            int sl = slot;
            uint32_t ph = phase;
            for (int p = 0; p < npiece && ok; ++p) {
                ok = __all_sync(0xffffffffu, tc_mbar_wait(tc_smem(&sh->full[sl]), ph, &sh->abort_flag));
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint64_t da = ring_k + (uint64_t)(sl * (LT_PIECE >> 4)), db = q_k + (uint64_t)(p * (2 * N * 128 >> 4));
                if (lt_elect()) {
#pragma unroll
                    for (int k = 0; k < 4; ++k) tc_mma_f16(tmem, da + 2 * k, db + 2 * k, id_s, (p > 0 || k > 0) ? 1u : 0u);
                    if (2 * p + 1 < nbox) {
#pragma unroll
                        for (int k = 0; k < 4; ++k) tc_mma_f16(tmem, da + (LT_BOX >> 4) + 2 * k, db + (N * 128 >> 4) + 2 * k, id_s, 1u);
                    }
                }
                __syncwarp();
                if (++sl == n_slots) { sl = 0; ph ^= 1u; }
            }
            if (!ok) break;
            if (lt_elect()) tc_commit(tc_smem(&sh->s_full));
            __syncwarp();
            ok = __all_sync(0xffffffffu, tc_mbar_wait(tc_smem(&sh->p_ready), (uint32_t)(tile - tile0) & 1u, &sh->abort_flag));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            for (int p = 0; p < npiece; ++p) {
                const uint64_t da = ring_mn + (uint64_t)(slot * (LT_PIECE >> 4));
                if (lt_elect()) {
#pragma unroll
                    for (int k = 0; k < 8; ++k)  // 16 positions: 2 KB of the tile, 16 rows of probabilities
                        tc_mma_f16(tmem_o + p * N, da + k * (2048 >> 4), p_mn + k * (32 * N >> 4), id_o, (tile > tile0 || k > 0) ? 1u : 0u);
                    tc_commit(tc_smem(&sh->empty[slot]));
                }
                __syncwarp();
                if (++slot == n_slots) { slot = 0; phase ^= 1u; }
            }
        }
        if (!ok) {
            if (lane == 0) stop();
        } else if (lt_elect()) {
            tc_commit(tc_smem(&sh->o_done));
        }
        __syncwarp();
    } else if (warp >= 2) {
        // ---------------- softmax and epilogue
        const int q = warp & 3, pt = q * 32 + lane;  // a warp may only touch TMEM lanes [32 q, 32 q + 32)
        const uint32_t lanes = (uint32_t)(q * 32) << 16;
        const float scale2 = a.scale * 1.4426950408889634f;  // scores in powers of two
        float l[N], ref_c[NG];  // row sums of this position, reference maxima of this lane's columns
#pragma unroll
        for (int c = 0; c < N; ++c) l[c] = 0.f;
#pragma unroll
        for (int g = 0; g < NG; ++g) ref_c[g] = -INFINITY;
        for (int c = lane; c < N; c += 32) sh->ref[q][c] = 0.f;
        __syncwarp();
        bool ok = true;
        for (int tile = tile0; tile < tile1; ++tile) {
            const int p0 = tile * LT_POS;
            if (tail && tile == tile1 - 1) {
                // rows past the context: whatever the page holds there becomes zero
                const int it = (tile - tile0) * npiece, nv = ctx - p0;
                for (int p = 0; p < npiece && ok; ++p)
                    ok = tc_mbar_wait(tc_smem(&sh->full[(it + p) % n_slots]), (uint32_t)((it + p) / n_slots) & 1u, &sh->abort_flag);
                for (int p = 0; p < npiece && ok; ++p) {
                    uint4 *base = reinterpret_cast<uint4 *>(ring + (size_t)((it + p) % n_slots) * LT_PIECE);
                    for (int i = nv * 8 + (tid - 64); i < LT_POS * 8; i += 128)
                        base[i] = base[i + LT_BOX / 16] = make_uint4(0, 0, 0, 0);
                }
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
                lt_arrive(tc_smem(&sh->z_ready));
            }
            ok = ok && tc_mbar_wait(tc_smem(&sh->s_full), (uint32_t)(tile - tile0) & 1u, &sh->abort_flag);
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            uint32_t raw[N];
            if (ok) {
#pragma unroll
                for (int c = 0; c < N; c += 16) tc_ld16(tmem + lanes + c, raw + c);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
            }
            if (!lt_sync_and(ok)) { ok = false; break; }
            const bool visible = p0 + pt < ctx;
            // scores relative to the references; the first tile always sets them
            float v[N], top = -INFINITY;
#pragma unroll
            for (int c = 0; c < N; c += 4) {
                const float4 f = *reinterpret_cast<const float4 *>(&sh->ref[q][c]);
                v[c] = fmaf(__uint_as_float(raw[c]), scale2, -f.x);
                v[c + 1] = fmaf(__uint_as_float(raw[c + 1]), scale2, -f.y);
                v[c + 2] = fmaf(__uint_as_float(raw[c + 2]), scale2, -f.z);
                v[c + 3] = fmaf(__uint_as_float(raw[c + 3]), scale2, -f.w);
                top = fmaxf(top, fmaxf(fmaxf(v[c], v[c + 1]), fmaxf(v[c + 2], v[c + 3])));
            }
            if (lt_sync_or(tile == tile0 || (visible && top > LT_GROW))) {
#pragma unroll
                for (int g = 0; g < NG; ++g) {
                    float w[GC];
#pragma unroll
                    for (int c = 0; c < GC; ++c) w[c] = visible ? __uint_as_float(raw[g * GC + c]) * scale2 : -INFINITY;
                    const float m = lt_columns<GC, true>(w);
                    if (lane < GC) sh->mx[q][g * GC + lane] = m;
                }
                lt_sync_and(true);
#pragma unroll
                for (int g = 0; g < NG; ++g) {
                    const int c = g * GC + lane % GC;
                    const float m = fmaxf(fmaxf(fmaxf(sh->mx[0][c], sh->mx[1][c]), fmaxf(sh->mx[2][c], sh->mx[3][c])), ref_c[g]);
                    if (lane < GC) {
                        sh->ref[q][c] = m;
                        sh->corr[q][c] = ref_c[g] == -INFINITY ? 0.f : exp2f(ref_c[g] - m);
                    }
                    ref_c[g] = m;
                }
                __syncwarp();
#pragma unroll
                for (int c = 0; c < N; ++c) {
                    l[c] *= sh->corr[q][c];
                    v[c] = fmaf(__uint_as_float(raw[c]), scale2, -sh->ref[q][c]);
                }
                if (tile > tile0) {  // the scores' commit covers the earlier products: O^T is at rest
                    for (int p = 0; p < npiece; ++p)
#pragma unroll
                        for (int c = 0; c < N; c += 16) {
                            uint32_t o[16];
                            tc_ld16(tmem_o + lanes + p * N + c, o);
                            asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                            for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * sh->corr[q][c + i]);
                            lt_st16(tmem_o + lanes + p * N + c, o);
                        }
                    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
                }
            }
#pragma unroll
            for (int j = 0; j < N / 8; ++j) {
                uint32_t w[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int c = 8 * j + 2 * i;
                    w[i] = visible ? Act<bf16>::pack(lt_exp2(v[c]), lt_exp2(v[c + 1])) : 0u;
                    const float2 f = Act<bf16>::to_f2(w[i]);
                    l[c] += f.x;
                    l[c + 1] += f.y;
                }
                *reinterpret_cast<uint4 *>(Ps + lt_p_off<N>(pt, j)) = make_uint4(w[0], w[1], w[2], w[3]);
            }
            __syncwarp();  // every lane has read this tile's references before the next tile may replace them
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            lt_arrive(tc_smem(&sh->p_ready));
        }
        if (ok) ok = tc_mbar_wait(tc_smem(&sh->o_done), 0u, &sh->abort_flag);
        if (!ok) stop();
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        // row sums over the 128 positions, then the unnormalised rows
#pragma unroll
        for (int g = 0; g < NG; ++g) {
            float w[GC];
#pragma unroll
            for (int c = 0; c < GC; ++c) w[c] = l[g * GC + c];
            const float s = lt_columns<GC, false>(w);
            if (lane < GC) sh->mx[q][g * GC + lane] = s;
        }
        if (lt_sync_and(ok)) {
            const int c0 = tid - 64;
            if (c0 < rows) {
                const float s = sh->mx[0][c0] + sh->mx[1][c0] + sh->mx[2][c0] + sh->mx[3][c0];
                reinterpret_cast<float2 *>(a.part_ml)[(size_t)(row0 + c0) * a.splits + sp] = make_float2(sh->ref[q][c0], s);
                if (sp == 0) a.part_n[row0 + c0] = my_splits;
            }
            for (int p = 0; p < npiece; ++p) {
                uint32_t o[N];
#pragma unroll
                for (int c = 0; c < N; c += 16) tc_ld16(tmem_o + lanes + p * N + c, o + c);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                if (p * 128 + pt < R) {
                    float *dst = a.part_o + ((size_t)row0 * a.splits + sp) * R + p * 128 + pt;
#pragma unroll
                    for (int c = 0; c < N; ++c)
                        if (c < rows) __stcg(dst + (size_t)c * a.splits * R, __uint_as_float(o[c]));
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
        }
    }
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(tm_cols) : "memory");
    }
}

// ------------------------------------------------------------------ host side

// cache pool of one layer as [pages][page_tokens][r_p]; absorbed queries as [rows][r_p]; boxes of 64 columns, 128-byte swizzle
static int lt_map(CUtensorMap *m, const void *base, int rank, const cuuint64_t *dims, const cuuint64_t *strides, const cuuint32_t *box) {
    TcEncodeFn fn = tc_encode_fn();
    if (!fn) {
        set_error("latent attention: cuTensorMapEncodeTiled is not available");
        return LCU_ERR_CUDA;
    }
    const cuuint32_t es[3] = {1, 1, 1};
    CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (cuuint32_t)rank, const_cast<void *>(base), dims, strides, box, es,
                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) {
        set_error("latent attention: cuTensorMapEncodeTiled failed with %d", (int)r);
        return LCU_ERR_CUDA;
    }
    return LCU_OK;
}

template <int N>
static int lt_launch(const LatentAttnArgs &a, cudaStream_t s, bool pdl, bool dry) {
    if (dry) {
        LCU_CHECK_CUDA(cudaFuncSetAttribute(latent_tc_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        return LCU_OK;
    }
    const int R = a.r_p, nbox = R / 64, npiece = (nbox + 1) / 2;
    const size_t fixed = 1024 + (size_t)nbox * N * 128 + (size_t)2 * N * 128 + sizeof(LtShared<N>) + 64;
    int slots = (int)(((size_t)227 * 1024 - fixed) / LT_PIECE);
    if (slots > LT_MAX_SLOTS) slots = LT_MAX_SLOTS;
    LCU_REQUIRE(slots >= npiece, "latent attention: %d pieces of a tile do not fit", npiece);
    int tm_cols = 32;
    while (tm_cols < N * (1 + npiece)) tm_cols *= 2;
    CUtensorMap mc, mq;
    const cuuint64_t cd[3] = {(cuuint64_t)R, (cuuint64_t)1 << a.page_shift, (cuuint64_t)a.n_pages};
    const cuuint64_t cs[2] = {(cuuint64_t)R * 2, (cuuint64_t)a.page_elems * 2};
    const cuuint32_t cb[3] = {64, 64, 1};
    int rc = lt_map(&mc, reinterpret_cast<const bf16 *>(a.pool) + a.c_off, 3, cd, cs, cb);
    if (rc) return rc;
    const cuuint64_t qd[2] = {(cuuint64_t)R, (cuuint64_t)a.n_tok * a.heads}, qs[1] = {(cuuint64_t)R * 2};
    const cuuint32_t qb[2] = {64, N};
    rc = lt_map(&mq, a.q, 2, qd, qs, qb);
    if (rc) return rc;
    const dim3 grid((unsigned)(a.n_tok * ((a.heads + N - 1) / N)), (unsigned)a.splits);
    LCU_CHECK_CUDA(launch_kernel(latent_tc_kernel<N>, grid, dim3(LT_THREADS), fixed + (size_t)slots * LT_PIECE, s, pdl, a, mc, mq, slots, tm_cols));
    return LCU_OK;
}

bool latent_tc_supported(int page_tokens) { return tuning().latent_tc && page_tokens >= 64 && tc_encode_fn() != nullptr; }
int latent_tc_rows(int heads) { return heads > 32 ? 64 : (heads > 16 ? 32 : 16); }

int latent_tc_launch(const LatentAttnArgs &a, cudaStream_t s, bool pdl, bool dry) {
    if (dry) {
        int rc = lt_launch<16>(a, s, pdl, true);
        if (!rc) rc = lt_launch<32>(a, s, pdl, true);
        return rc ? rc : lt_launch<64>(a, s, pdl, true);
    }
    if (a.n_tok <= 0) return LCU_OK;
    switch (latent_tc_rows(a.heads)) {
    case 16: return lt_launch<16>(a, s, pdl, false);
    case 32: return lt_launch<32>(a, s, pdl, false);
    default: return lt_launch<64>(a, s, pdl, false);
    }
}

}  // namespace lcu
