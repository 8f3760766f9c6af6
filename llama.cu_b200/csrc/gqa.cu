// Softmax attention over cached keys and values: grouped heads of any ratio, query/key and value sizes that may differ, any
// multiple of 16 up to 256, pages of any size.
//
//   short form  decoded tokens and portions of a few tokens: the (token, head) rows that share a key/value head are the 16 rows
//               of a tensor-core tile; every warp walks its own blocks of 16 cached rows with a copy ring and running softmax of
//               its own (no barrier in the loop); contexts are cut into splits, the last CTA of a row tile to arrive merges;
//   long form   64 (token, head) rows per CTA share tiles of 64 cached rows.
// Options: a sliding window, with or without the first tokens of a sequence (tiles that no row sees are skipped), a sink in the
// softmax's denominator, a gate per head, outputs rotated back where the cached values are rotated.
//
// Arithmetic: scores, softmax and its running state in f32; probabilities are rounded to bf16 only as operands of the second
// product, the row sum is taken over the rounded values; all sums accumulate in f32.  All-32-bit contexts use f32 FMA throughout.
#include "gqa_prep.cuh"

namespace lcu {

typedef __nv_bfloat16 bf16;

namespace {

__device__ __forceinline__ void ga_cp16(void *smem_dst, const void *gsrc, bool valid) {
    unsigned dst = (unsigned)__cvta_generic_to_shared(smem_dst);
    int sz = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(gsrc), "r"(sz) : "memory");
}
__device__ __forceinline__ void ga_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void ga_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ga_ldsm4(uint32_t r[4], const void *row) {
    unsigned a = (unsigned)__cvta_generic_to_shared(row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ga_ldsm4t(uint32_t r[4], const void *row) {
    unsigned a = (unsigned)__cvta_generic_to_shared(row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ float quad_max(float v) {
    v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
    return fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
}
__device__ __forceinline__ float quad_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    return v + __shfl_xor_sync(0xffffffffu, v, 2);
}

template <class T, int FORM>
__global__ void __launch_bounds__(256, FORM == GQA_PREP ? 6 : (FORM == GQA_PREP_CONV ? 4 : 5)) gqa_prep_kernel(const GqaArgs a) {
    grid_dep_launch();
    const int per = FORM >= GQA_PREP_WIDE ? (gqa_prep_items(a) + (int)gridDim.x - 1) / (int)gridDim.x : 8;
    grid_dep_wait();
    gqa_prep_block<T, FORM>(a, blockIdx.y, blockIdx.x * per, blockIdx.x * per + per);
}

template <class T, int TAPS, int RUN>
__global__ void __launch_bounds__(256, RUN == 1 ? 4 : (TAPS > 2 ? 2 : (TAPS ? 3 : 4))) gqa_prep_run_kernel(const GqaArgs a) {
    grid_dep_launch();
    const int item = blockIdx.x * 8 + (threadIdx.x >> 5);
    grid_dep_wait();
    if (item < gqa_prep_items(a)) gqa_prep_run<T, TAPS, RUN>(a, blockIdx.y * RUN, item, threadIdx.x & 31);
}

// Denominator and factor that end a row of softmax (scores in powers of two): maximum M, sum L over it.  A key without
// value may count in the denominator; the head's gate multiplies the output.
__device__ __forceinline__ float softmax_end(const GqaArgs &a, float M, float L, int tok, int head) {
    float f = 1.f;
    if (a.sink) {
        const float z = a.sink_score ? a.sink_score[head] * 1.4426950408889634f : 0.f, top = fmaxf(M, z);
        f = exp2f(M - top);
        L = fmaf(L, f, exp2f(z - top));
    }
    if (a.gate) f /= 1.f + expf(-a.gate[(size_t)tok * a.stride + head]);
    return f / L;
}
// first position that position p sees
__device__ __forceinline__ int first_seen(const GqaArgs &a, int p) { return a.window > 0 && p >= a.window ? p - a.window + 1 : 0; }
// Tiles of `size` positions, from the one at position `lo` up to `ctx`, those of the kept first tokens ahead of them: number of
// both, and a tile's number in the sequence.
struct SeenTiles {
    int kept, jump, n;
    __device__ __forceinline__ SeenTiles(const GqaArgs &a, int lo, int ctx, int size) {
        const int tile0 = lo / size;
        kept = min((a.keep + size - 1) / size, tile0);
        jump = tile0 - kept;
        n = (ctx + size - 1) / size - jump;
    }
    __device__ __forceinline__ int at(int i) const { return i < kept ? i : i + jump; }
};
// Positions [keep, keep + gap) are those up to p's first seen one that p does not see.
__device__ __forceinline__ int gap_of(const GqaArgs &a, int p) { return max(first_seen(a, p) - a.keep, 0); }
__device__ __forceinline__ bool seen(int pos, int lim, int keep, int gap) { return pos <= lim && (unsigned)(pos - keep) >= (unsigned)gap; }
// Columns d and d + 1 of an output, rotated back by position p.
__device__ __forceinline__ float2 turn_back(const GqaArgs &a, int p, int d, float x, float y) {
    if (d >= a.v_dim) return make_float2(x, y);
    const float2 c = a.vrot[(size_t)p * (a.v_dim >> 1) + (d >> 1)];
    return make_float2(x * c.x + y * c.y, y * c.x - x * c.y);
}
// Eight columns from d on of a row's output, rounded; p: position of its token.
__device__ __forceinline__ uint4 end_of_row(const GqaArgs &a, const float x[8], float f, int p, int d) {
    float2 v[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        v[i] = make_float2(x[2 * i] * f, x[2 * i + 1] * f);
        if (a.vrot) v[i] = turn_back(a, p, d + 2 * i, v[i].x, v[i].y);
    }
    return make_uint4(Act<bf16>::pack(v[0].x, v[0].y), Act<bf16>::pack(v[1].x, v[1].y), Act<bf16>::pack(v[2].x, v[2].y), Act<bf16>::pack(v[3].x, v[3].y));
}

// ------------------------------------------------------------------ short form
constexpr int GS_WARPS = 4, GS_KEYS = 16, GS_STAGES = 3;
constexpr int GS_UNIT = GS_WARPS * GS_KEYS;  // cached rows all warps of a CTA take per step

template <int DQ, int DV> constexpr size_t gs_smem() {
    const size_t ring = (size_t)GS_WARPS * GS_STAGES * GS_KEYS * (DQ + DV + 16) * sizeof(bf16);
    const size_t merge = (size_t)GS_WARPS * 16 * (DV + 4) * 4;
    return ring > merge ? ring : merge;
}

template <int DQ, int DV>
__global__ void __launch_bounds__(GS_WARPS * 32) gqa_short_kernel(const GqaArgs a) {
    constexpr int KROW = DQ + 8, VROW = DV + 8, KS = DQ / 16, NTO = DV / 8;
    constexpr int STAGE = GS_KEYS * (KROW + VROW);
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float s_ml[GS_WARPS][16][2];
    __shared__ int s_last;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, t4 = lane & 3;
    const int g = a.group();
    const int kvh = blockIdx.x % a.kv_heads, row0 = blockIdx.x / a.kv_heads * 16;
    const int4 rq = a.reqs[blockIdx.y];  // request, first token, tokens, position
    const int rows = rq.z * g, sp = blockIdx.z;
    const int ctx = rq.w + rq.z;
    const SeenTiles tiles(a, first_seen(a, rq.w), ctx, GS_UNIT);
    const int ups = (tiles.n + a.splits - 1) / a.splits, n_split = (tiles.n + ups - 1) / ups;
    grid_dep_launch();
    if (row0 >= rows || sp >= n_split) return;
    const int u0 = sp * ups, u1 = min(tiles.n, u0 + ups);
    const bf16 *pool = reinterpret_cast<const bf16 *>(a.pool);
    const size_t koff = a.c_off + ((size_t)kvh << a.page_shift) * a.dim_p, voff = a.v_off() + ((size_t)kvh << a.page_shift) * a.vdim_p;
    const int32_t *pages = a.page_table + (size_t)rq.x * a.pt_stride;
    const int kch = a.dim_p / 8, vch = a.vdim_p / 8;
    bf16 *ring = reinterpret_cast<bf16 *>(smem) + (size_t)warp * GS_STAGES * STAGE;

    auto load = [&](int u, int stage) {
        bf16 *kd = ring + stage * STAGE, *vd = kd + GS_KEYS * KROW;
        const int key0 = tiles.at(u) * GS_UNIT + warp * GS_KEYS;
        constexpr int KL = DQ / 8, VL = DV / 8;  // lanes per row (columns past the head's size stay idle)
#pragma unroll
        for (int i = 0; i < GS_KEYS * KL / 32; ++i) {
            const int j = (i * 32 + lane) / KL, c = lane % KL, key = key0 + j;
            if (c >= kch) continue;
            const bool ok = key < ctx;
            const size_t src = ok ? (size_t)pages[key >> a.page_shift] * a.page_elems + koff + (size_t)(key & ((1 << a.page_shift) - 1)) * a.dim_p + c * 8 : 0;
            ga_cp16(kd + j * KROW + c * 8, pool + src, ok);
        }
#pragma unroll
        for (int i = 0; i < GS_KEYS * VL / 32; ++i) {
            const int j = (i * 32 + lane) / VL, c = lane % VL, key = key0 + j;
            if (c >= vch) continue;
            const bool ok = key < ctx;
            const size_t src = ok ? (size_t)pages[key >> a.page_shift] * a.page_elems + voff + (size_t)(key & ((1 << a.page_shift) - 1)) * a.vdim_p + c * 8 : 0;
            ga_cp16(vd + j * VROW + c * 8, pool + src, ok);
        }
    };
    grid_dep_wait();
    for (int i = 0; i < GS_STAGES - 1; ++i) {
        if (u0 + i < u1) load(u0 + i, i);
        ga_commit();
    }
    // this lane's two rows of the tile
    const int r0 = row0 + gid, r1 = r0 + 8;
    const bool v0 = r0 < rows, v1 = r1 < rows;
    const int tk0 = v0 ? r0 / g : 0, tk1 = v1 ? r1 / g : 0;
    const int lim0 = v0 ? rq.w + tk0 : -1, lim1 = v1 ? rq.w + tk1 : -1;
    const int gap0 = gap_of(a, lim0), gap1 = gap_of(a, lim1);
    uint32_t qa[KS][4];
    {
        const bf16 *q = reinterpret_cast<const bf16 *>(a.q);
        const bf16 *q0 = q + ((size_t)(rq.y + tk0) * a.heads + kvh * g + (v0 ? r0 % g : 0)) * a.dim_p + 2 * t4;
        const bf16 *q1 = q + ((size_t)(rq.y + tk1) * a.heads + kvh * g + (v1 ? r1 % g : 0)) * a.dim_p + 2 * t4;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            const bool in = ks * 16 < a.dim_p;
            qa[ks][0] = in && v0 ? *reinterpret_cast<const uint32_t *>(q0 + ks * 16) : 0u;
            qa[ks][1] = in && v1 ? *reinterpret_cast<const uint32_t *>(q1 + ks * 16) : 0u;
            qa[ks][2] = in && v0 ? *reinterpret_cast<const uint32_t *>(q0 + ks * 16 + 8) : 0u;
            qa[ks][3] = in && v1 ? *reinterpret_cast<const uint32_t *>(q1 + ks * 16 + 8) : 0u;
        }
    }
    const float scale2 = a.scale * 1.4426950408889634f;  // scores in powers of two
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    float o[NTO][4];
#pragma unroll
    for (int i = 0; i < NTO; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    for (int u = u0; u < u1; ++u) {
        const int stage = (u - u0) % GS_STAGES;
        ga_wait<GS_STAGES - 2>();
        __syncwarp();
        if (u + GS_STAGES - 1 < u1) load(u + GS_STAGES - 1, (u - u0 + GS_STAGES - 1) % GS_STAGES);
        ga_commit();
        const bf16 *Kt = ring + stage * STAGE, *Vt = Kt + GS_KEYS * KROW;
        float sc[2][4] = {};
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            if (ks * 16 >= a.dim_p) continue;
            uint32_t kb[4];
            ga_ldsm4(kb, Kt + ((lane & 7) + ((lane >> 4) & 1) * 8) * KROW + ks * 16 + ((lane >> 3) & 1) * 8);
            mma16816<bf16>(sc[0], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], kb[0], kb[1]);
            mma16816<bf16>(sc[1], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], kb[2], kb[3]);
        }
        float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
            const int p = tiles.at(u) * GS_UNIT + warp * GS_KEYS + nt * 8 + 2 * t4;
            sc[nt][0] = seen(p, lim0, a.keep, gap0) ? sc[nt][0] * scale2 : -INFINITY;
            sc[nt][1] = seen(p + 1, lim0, a.keep, gap0) ? sc[nt][1] * scale2 : -INFINITY;
            sc[nt][2] = seen(p, lim1, a.keep, gap1) ? sc[nt][2] * scale2 : -INFINITY;
            sc[nt][3] = seen(p + 1, lim1, a.keep, gap1) ? sc[nt][3] * scale2 : -INFINITY;
            t0 = fmaxf(t0, fmaxf(sc[nt][0], sc[nt][1]));
            t1 = fmaxf(t1, fmaxf(sc[nt][2], sc[nt][3]));
        }
        const float n0 = fmaxf(m0, quad_max(t0)), n1 = fmaxf(m1, quad_max(t1));
        if (__any_sync(0xffffffffu, n0 > m0 || n1 > m1)) {
            const float c0 = m0 == -INFINITY ? 0.f : exp2f(m0 - n0), c1 = m1 == -INFINITY ? 0.f : exp2f(m1 - n1);
            m0 = n0;
            m1 = n1;
            l0 *= c0;
            l1 *= c1;
#pragma unroll
            for (int i = 0; i < NTO; ++i) {
                o[i][0] *= c0; o[i][1] *= c0;
                o[i][2] *= c1; o[i][3] *= c1;
            }
        }
        const float mu0 = m0 == -INFINITY ? 0.f : m0, mu1 = m1 == -INFINITY ? 0.f : m1;
        uint32_t pa[2][2];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
            pa[nt][0] = Act<bf16>::pack(exp2f(sc[nt][0] - mu0), exp2f(sc[nt][1] - mu0));
            pa[nt][1] = Act<bf16>::pack(exp2f(sc[nt][2] - mu1), exp2f(sc[nt][3] - mu1));
            const float2 f0 = Act<bf16>::to_f2(pa[nt][0]), f1 = Act<bf16>::to_f2(pa[nt][1]);
            l0 += f0.x + f0.y;
            l1 += f1.x + f1.y;
        }
#pragma unroll
        for (int dp = 0; dp < NTO / 2; ++dp) {
            if (dp * 16 >= a.vdim_p) continue;
            uint32_t vb[4];
            ga_ldsm4t(vb, Vt + (lane & 15) * VROW + dp * 16 + (lane >> 4) * 8);
            mma16816<bf16>(o[2 * dp], pa[0][0], pa[0][1], pa[1][0], pa[1][1], vb[0], vb[1]);
            mma16816<bf16>(o[2 * dp + 1], pa[0][0], pa[0][1], pa[1][0], pa[1][1], vb[2], vb[3]);
        }
        __syncwarp();
    }
    ga_wait<0>();
    l0 = quad_sum(l0);
    l1 = quad_sum(l1);
    __syncthreads();  // the rings become the merge buffer
    float *mo = reinterpret_cast<float *>(smem);  // [warp][16][DV + 4]
    constexpr int MLD = DV + 4;
#pragma unroll
    for (int i = 0; i < NTO; ++i) {
        if (i * 8 >= a.vdim_p) continue;
        float *d0 = mo + ((size_t)warp * 16 + gid) * MLD + i * 8 + 2 * t4;
        *reinterpret_cast<float2 *>(d0) = make_float2(o[i][0], o[i][1]);
        *reinterpret_cast<float2 *>(d0 + 8 * MLD) = make_float2(o[i][2], o[i][3]);
    }
    if (t4 == 0) {
        s_ml[warp][gid][0] = m0; s_ml[warp][gid][1] = l0;
        s_ml[warp][gid + 8][0] = m1; s_ml[warp][gid + 8][1] = l1;
    }
    __syncthreads();
    const int n_rows = min(16, rows - row0);
    const size_t cell = (size_t)blockIdx.y * gridDim.x + blockIdx.x;
    bf16 *out = reinterpret_cast<bf16 *>(a.o);
    for (int i = tid; i < n_rows * vch; i += GS_WARPS * 32) {
        const int r = i / vch, c = (i - r * vch) * 8;
        float M = -INFINITY, L = 0.f, x[8] = {};
#pragma unroll
        for (int w = 0; w < GS_WARPS; ++w) M = fmaxf(M, s_ml[w][r][0]);
#pragma unroll
        for (int w = 0; w < GS_WARPS; ++w) {
            const float f = s_ml[w][r][0] == -INFINITY ? 0.f : exp2f(s_ml[w][r][0] - M);
            L += s_ml[w][r][1] * f;
            const float *src = mo + ((size_t)w * 16 + r) * MLD + c;
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] += src[e] * f;
        }
        if (n_split == 1) {
            const int row = row0 + r;
            const float inv = softmax_end(a, M, L, rq.y + row / g, kvh * g + row % g);
            *reinterpret_cast<uint4 *>(out + (size_t)(rq.y + row / g) * a.stride_o + (size_t)(kvh * g + row % g) * a.vdim_p + c) =
                end_of_row(a, x, inv, rq.w + row / g, c);
        } else {
            float *dst = a.part_o + ((cell * a.splits + sp) * 16 + r) * a.vdim_p + c;
            *reinterpret_cast<float4 *>(dst) = make_float4(x[0], x[1], x[2], x[3]);
            *reinterpret_cast<float4 *>(dst + 4) = make_float4(x[4], x[5], x[6], x[7]);
            if (c == 0) *reinterpret_cast<float2 *>(a.part_ml + ((cell * a.splits + sp) * 16 + r) * 2) = make_float2(M, L);
        }
    }
    if (n_split == 1) return;
    __threadfence();
    __syncthreads();
    if (tid == 0) s_last = atomicAdd(&a.tickets[cell], 1u) == (unsigned)n_split - 1;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    for (int i = tid; i < n_rows * vch; i += GS_WARPS * 32) {
        const int r = i / vch, c = (i - r * vch) * 8;
        float M = -INFINITY, L = 0.f, x[8] = {};
        for (int k = 0; k < n_split; ++k) M = fmaxf(M, __ldcg(a.part_ml + ((cell * a.splits + k) * 16 + r) * 2));
        for (int k = 0; k < n_split; ++k) {
            const float2 ml = __ldcg(reinterpret_cast<const float2 *>(a.part_ml + ((cell * a.splits + k) * 16 + r) * 2));
            const float f = ml.x == -INFINITY ? 0.f : exp2f(ml.x - M);
            const float4 *src = reinterpret_cast<const float4 *>(a.part_o + ((cell * a.splits + k) * 16 + r) * a.vdim_p + c);
            const float4 lo = __ldcg(src), hi = __ldcg(src + 1);
            L += ml.y * f;
            x[0] += lo.x * f; x[1] += lo.y * f; x[2] += lo.z * f; x[3] += lo.w * f;
            x[4] += hi.x * f; x[5] += hi.y * f; x[6] += hi.z * f; x[7] += hi.w * f;
        }
        const int row = row0 + r;
        const float inv = softmax_end(a, M, L, rq.y + row / g, kvh * g + row % g);
        *reinterpret_cast<uint4 *>(out + (size_t)(rq.y + row / g) * a.stride_o + (size_t)(kvh * g + row % g) * a.vdim_p + c) =
            end_of_row(a, x, inv, rq.w + row / g, c);
    }
    if (tid == 0) a.tickets[cell] = 0;  // ready for the next launch
}

// ------------------------------------------------------------------ long form
constexpr int GL_TILE = 64;

template <int DQ, int DV>
__global__ void __launch_bounds__(128) gqa_long_kernel(const GqaArgs a) {
    constexpr int KROW = DQ + 8, VROW = DV + 8, KS = DQ / 16, NTS = GL_TILE / 8, NTO = DV / 8;
    extern __shared__ __align__(16) unsigned char smem[];
    bf16 *Ks = reinterpret_cast<bf16 *>(smem);      // [2][TILE][KROW]
    bf16 *Vs = Ks + (size_t)2 * GL_TILE * KROW;     // [2][TILE][VROW]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, t4 = lane & 3;
    const int g = a.group(), kvh = blockIdx.x;
    // request of this block of 64 (token, head) rows; the longest contexts of the last request come first
    int blk = (int)gridDim.y - 1 - (int)blockIdx.y, ri = 0;
    for (int base = 0; base < a.n_reqs; base += 32) {
        const int i = base + lane;
        const int nb = i < a.n_reqs ? (a.reqs[i].z * g + 63) / 64 : 0;
        int incl = nb;
#pragma unroll
        for (int s = 1; s < 32; s <<= 1) {
            const int up = __shfl_up_sync(0xffffffffu, incl, s);
            if (lane >= s) incl += up;
        }
        const unsigned hit = __ballot_sync(0xffffffffu, blk < incl);
        if (hit) {
            const int src = __ffs(hit) - 1;
            ri = base + src;
            blk -= __shfl_sync(0xffffffffu, incl - nb, src);
            break;
        }
        blk -= __shfl_sync(0xffffffffu, incl, 31);
    }
    const int4 rq = a.reqs[ri];
    const int rows = rq.z * g, row0 = blk * 64;
    const int last_tok = min(rq.z - 1, (row0 + 63) / g);
    const int ctx = rq.w + last_tok + 1;
    const SeenTiles tiles(a, first_seen(a, rq.w + row0 / g), ctx, GL_TILE);
    const bf16 *pool = reinterpret_cast<const bf16 *>(a.pool);
    const size_t koff = a.c_off + ((size_t)kvh << a.page_shift) * a.dim_p, voff = a.v_off() + ((size_t)kvh << a.page_shift) * a.vdim_p;
    const int32_t *pages = a.page_table + (size_t)rq.x * a.pt_stride;
    const int kch = a.dim_p / 8, vch = a.vdim_p / 8;

    auto load_tile = [&](int tile, int buf) {
        bf16 *kd = Ks + (size_t)buf * GL_TILE * KROW, *vd = Vs + (size_t)buf * GL_TILE * VROW;
        constexpr int KL = DQ / 8, VL = DV / 8;
#pragma unroll 4
        for (int i = 0; i < GL_TILE * KL / 128; ++i) {
            const int j = (i * 128 + tid) / KL, c = tid % KL, key = tile * GL_TILE + j;
            if (c >= kch) continue;
            const bool ok = key < ctx;
            const size_t src = ok ? (size_t)pages[key >> a.page_shift] * a.page_elems + koff + (size_t)(key & ((1 << a.page_shift) - 1)) * a.dim_p + c * 8 : 0;
            ga_cp16(kd + j * KROW + c * 8, pool + src, ok);
        }
#pragma unroll 4
        for (int i = 0; i < GL_TILE * VL / 128; ++i) {
            const int j = (i * 128 + tid) / VL, c = tid % VL, key = tile * GL_TILE + j;
            if (c >= vch) continue;
            const bool ok = key < ctx;
            const size_t src = ok ? (size_t)pages[key >> a.page_shift] * a.page_elems + voff + (size_t)(key & ((1 << a.page_shift) - 1)) * a.vdim_p + c * 8 : 0;
            ga_cp16(vd + j * VROW + c * 8, pool + src, ok);
        }
    };
    const int r0 = row0 + warp * 16 + gid, r1 = r0 + 8;
    const bool v0 = r0 < rows, v1 = r1 < rows;
    const int tk0 = v0 ? r0 / g : 0, tk1 = v1 ? r1 / g : 0;
    const int lim0 = v0 ? rq.w + tk0 : -1, lim1 = v1 ? rq.w + tk1 : -1;
    const int gap0 = gap_of(a, lim0), gap1 = gap_of(a, lim1);
    const int h0 = kvh * g + (v0 ? r0 % g : 0), h1 = kvh * g + (v1 ? r1 % g : 0);
    uint32_t qa[KS][4];
    {
        const bf16 *q0 = reinterpret_cast<const bf16 *>(a.q) + ((size_t)(rq.y + tk0) * a.heads + h0) * a.dim_p + 2 * t4;
        const bf16 *q1 = reinterpret_cast<const bf16 *>(a.q) + ((size_t)(rq.y + tk1) * a.heads + h1) * a.dim_p + 2 * t4;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            const bool in = ks * 16 < a.dim_p;
            qa[ks][0] = in && v0 ? *reinterpret_cast<const uint32_t *>(q0 + ks * 16) : 0u;
            qa[ks][1] = in && v1 ? *reinterpret_cast<const uint32_t *>(q1 + ks * 16) : 0u;
            qa[ks][2] = in && v0 ? *reinterpret_cast<const uint32_t *>(q0 + ks * 16 + 8) : 0u;
            qa[ks][3] = in && v1 ? *reinterpret_cast<const uint32_t *>(q1 + ks * 16 + 8) : 0u;
        }
    }
    load_tile(tiles.at(0), 0);
    ga_commit();
    const float scale2 = a.scale * 1.4426950408889634f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    float o[NTO][4];
#pragma unroll
    for (int i = 0; i < NTO; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;

    for (int i = 0; i < tiles.n; ++i) {
        const int buf = i & 1, tile = tiles.at(i);
        if (i + 1 < tiles.n) load_tile(tiles.at(i + 1), buf ^ 1);
        ga_commit();
        ga_wait<1>();
        __syncthreads();
        const bf16 *Kt = Ks + (size_t)buf * GL_TILE * KROW, *Vt = Vs + (size_t)buf * GL_TILE * VROW;
        float sc[NTS][4];
#pragma unroll
        for (int nt = 0; nt < NTS; ++nt) sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            if (ks * 16 < a.dim_p) {
#pragma unroll
                for (int np = 0; np < NTS / 2; ++np) {
                    uint32_t kb[4];
                    ga_ldsm4(kb, Kt + (size_t)(np * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * KROW + ks * 16 + ((lane >> 3) & 1) * 8);
                    mma16816<bf16>(sc[2 * np], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], kb[0], kb[1]);
                    mma16816<bf16>(sc[2 * np + 1], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], kb[2], kb[3]);
                }
            }
        }
        float t0 = -INFINITY, t1 = -INFINITY;
        if (tile * GL_TILE + GL_TILE - 1 <= min(lim0, lim1) && (tile * GL_TILE >= a.keep + max(gap0, gap1) || tile * GL_TILE + GL_TILE <= a.keep)) {  // every position visible
#pragma unroll
            for (int nt = 0; nt < NTS; ++nt) {
#pragma unroll
                for (int e = 0; e < 4; ++e) sc[nt][e] *= scale2;
                t0 = fmaxf(t0, fmaxf(sc[nt][0], sc[nt][1]));
                t1 = fmaxf(t1, fmaxf(sc[nt][2], sc[nt][3]));
            }
        } else {
#pragma unroll
            for (int nt = 0; nt < NTS; ++nt) {
                const int p = tile * GL_TILE + nt * 8 + 2 * t4;
                sc[nt][0] = seen(p, lim0, a.keep, gap0) ? sc[nt][0] * scale2 : -INFINITY;
                sc[nt][1] = seen(p + 1, lim0, a.keep, gap0) ? sc[nt][1] * scale2 : -INFINITY;
                sc[nt][2] = seen(p, lim1, a.keep, gap1) ? sc[nt][2] * scale2 : -INFINITY;
                sc[nt][3] = seen(p + 1, lim1, a.keep, gap1) ? sc[nt][3] * scale2 : -INFINITY;
                t0 = fmaxf(t0, fmaxf(sc[nt][0], sc[nt][1]));
                t1 = fmaxf(t1, fmaxf(sc[nt][2], sc[nt][3]));
            }
        }
        const float n0 = fmaxf(m0, quad_max(t0)), n1 = fmaxf(m1, quad_max(t1));
        if (__any_sync(0xffffffffu, n0 > m0 || n1 > m1)) {
            const float c0 = m0 == -INFINITY ? 0.f : exp2f(m0 - n0), c1 = m1 == -INFINITY ? 0.f : exp2f(m1 - n1);
            m0 = n0;
            m1 = n1;
            l0 *= c0;
            l1 *= c1;
#pragma unroll
            for (int i = 0; i < NTO; ++i) {
                o[i][0] *= c0; o[i][1] *= c0;
                o[i][2] *= c1; o[i][3] *= c1;
            }
        }
        const float mu0 = m0 == -INFINITY ? 0.f : m0, mu1 = m1 == -INFINITY ? 0.f : m1;  // a fully masked row stays at zero
        uint32_t pa[NTS][2];
#pragma unroll
        for (int nt = 0; nt < NTS; ++nt) {
            pa[nt][0] = Act<bf16>::pack(exp2f(sc[nt][0] - mu0), exp2f(sc[nt][1] - mu0));
            pa[nt][1] = Act<bf16>::pack(exp2f(sc[nt][2] - mu1), exp2f(sc[nt][3] - mu1));
            const float2 f0 = Act<bf16>::to_f2(pa[nt][0]), f1 = Act<bf16>::to_f2(pa[nt][1]);
            l0 += f0.x + f0.y;
            l1 += f1.x + f1.y;
        }
#pragma unroll
        for (int kk = 0; kk < GL_TILE / 16; ++kk) {
#pragma unroll
            for (int dp = 0; dp < NTO / 2; ++dp) {
                if (dp * 16 < a.vdim_p) {
                    uint32_t vb[4];
                    ga_ldsm4t(vb, Vt + (size_t)(kk * 16 + (lane & 15)) * VROW + dp * 16 + (lane >> 4) * 8);
                    mma16816<bf16>(o[2 * dp], pa[2 * kk][0], pa[2 * kk][1], pa[2 * kk + 1][0], pa[2 * kk + 1][1], vb[0], vb[1]);
                    mma16816<bf16>(o[2 * dp + 1], pa[2 * kk][0], pa[2 * kk][1], pa[2 * kk + 1][0], pa[2 * kk + 1][1], vb[2], vb[3]);
                }
            }
        }
        __syncthreads();
    }
    ga_wait<0>();
    l0 = quad_sum(l0);
    l1 = quad_sum(l1);
    bf16 *out = reinterpret_cast<bf16 *>(a.o);
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
        if (!(hf ? v1 : v0)) continue;
        const float inv = softmax_end(a, hf ? m1 : m0, hf ? l1 : l0, rq.y + (hf ? tk1 : tk0), hf ? h1 : h0);
        bf16 *dst = out + (size_t)(rq.y + (hf ? tk1 : tk0)) * a.stride_o + (size_t)(hf ? h1 : h0) * a.vdim_p + 2 * t4;
#pragma unroll
        for (int i = 0; i < NTO; ++i) {
            if (i * 8 >= a.vdim_p) continue;
            float2 v = make_float2(o[i][2 * hf] * inv, o[i][2 * hf + 1] * inv);
            if (a.vrot) v = turn_back(a, hf ? lim1 : lim0, 8 * i + 2 * t4, v.x, v.y);
            *reinterpret_cast<uint32_t *>(dst + 8 * i) = Act<bf16>::pack(v.x, v.y);
        }
    }
}

// ------------------------------------------------------------------ all-32-bit form: a warp per (token, head) row
__global__ void __launch_bounds__(256) gqa_f32_kernel(const GqaArgs a) {
    __shared__ __align__(16) float qs[8][MIX_MAX_HEAD];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const long row = (long)blockIdx.x * 8 + warp;
    if (row >= (long)a.n_tok * a.heads) return;
    const int t = (int)(row / a.heads), h = (int)(row - (long)t * a.heads), kvh = h / a.group();
    const float *q = reinterpret_cast<const float *>(a.q) + row * a.dim_p;
    for (int d = lane; d < a.dim_p; d += 32) qs[warp][d] = q[d];
    __syncwarp();
    const int ctx = (int)a.pos[t] + 1;
    const float *pool = reinterpret_cast<const float *>(a.pool);
    const size_t koff = a.c_off + ((size_t)kvh << a.page_shift) * a.dim_p, voff = a.v_off() + ((size_t)kvh << a.page_shift) * a.vdim_p;
    const int32_t *pages = a.page_table + (size_t)a.tok_req[t] * a.pt_stride;
    float m = -INFINITY, l = 0.f, acc[MIX_MAX_HEAD / 32] = {};
    const int lo = first_seen(a, ctx - 1), kept = min(a.keep, lo);
    for (int k0 = kept > 0 ? 0 : lo; k0 < ctx; k0 = k0 < lo && k0 + 32 >= kept ? lo : k0 + 32) {
        const int key = k0 + lane, end = k0 < lo ? kept : ctx;
        const bool ok = key < end;
        const int slot = key & ((1 << a.page_shift) - 1);
        const size_t base = ok ? (size_t)pages[key >> a.page_shift] * a.page_elems : 0;
        float s = -INFINITY;
        if (ok) {
            const float4 *kr = reinterpret_cast<const float4 *>(pool + base + koff + (size_t)slot * a.dim_p);
            const float4 *qr = reinterpret_cast<const float4 *>(qs[warp]);
            float x = 0.f;
            for (int i = 0; i < a.dim_p / 4; ++i) {
                const float4 u = kr[i], w = qr[i];
                x = fmaf(u.x, w.x, x); x = fmaf(u.y, w.y, x); x = fmaf(u.z, w.z, x); x = fmaf(u.w, w.w, x);
            }
            s = x * a.scale;
        }
        const float mn = fmaxf(m, warp_max(s)), c = m == -INFINITY ? 0.f : expf(m - mn);
        const float p = ok ? expf(s - mn) : 0.f;
        m = mn;
        l = l * c + warp_sum(p);
#pragma unroll
        for (int j = 0; j < MIX_MAX_HEAD / 32; ++j) acc[j] *= c;
        const size_t vrow = base + voff + (size_t)slot * a.vdim_p;
        for (int i = 0; i < 32 && k0 + i < end; ++i) {
            const float pi = __shfl_sync(0xffffffffu, p, i);
            const float *vr = pool + __shfl_sync(0xffffffffu, (unsigned long long)vrow, i);
#pragma unroll
            for (int j = 0; j < MIX_MAX_HEAD / 32; ++j)
                if (lane + 32 * j < a.vdim_p) acc[j] = fmaf(pi, vr[lane + 32 * j], acc[j]);
        }
    }
    const float inv = softmax_end(a, m * 1.4426950408889634f, l, t, h);
    float *out = reinterpret_cast<float *>(a.o) + (size_t)t * a.stride_o + (size_t)h * a.vdim_p;
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 32; ++j) {
        float v = acc[j] * inv;
        if (a.vrot) {  // the other one of a pair is in the neighbouring lane
            const float w = __shfl_xor_sync(0xffffffffu, v, 1);
            const float2 x = turn_back(a, ctx - 1, (lane & ~1) + 32 * j, lane & 1 ? w : v, lane & 1 ? v : w);
            v = lane & 1 ? x.y : x.x;
        }
        if (lane + 32 * j < a.vdim_p) out[lane + 32 * j] = v;
    }
}

template <class K>
int raise_smem(K kernel, size_t smem) {
    if (smem > 48 * 1024) LCU_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return LCU_OK;
}

// (query/key, value) size variant of a shape: calls f.template run<DQ, DV>()
template <class F>
int by_size(int dim_p, int vdim_p, const F &f) {
    if (vdim_p <= 64) return dim_p <= 64 ? f.template run<64, 64>() : (dim_p <= 128 ? f.template run<128, 64>() : f.template run<256, 64>());
    if (vdim_p <= 128) return dim_p <= 64 ? f.template run<64, 128>() : (dim_p <= 128 ? f.template run<128, 128>() : f.template run<256, 128>());
    return dim_p <= 64 ? f.template run<64, 256>() : (dim_p <= 128 ? f.template run<128, 256>() : f.template run<256, 256>());
}

struct ShortLaunch {
    const GqaArgs &a;
    cudaStream_t s;
    bool pdl, dry;
    template <int DQ, int DV> int run() const {
        if (dry) return raise_smem(gqa_short_kernel<DQ, DV>, gs_smem<DQ, DV>());
        const dim3 grid(a.kv_heads * gqa_row_tiles(a.heads, a.kv_heads, a.max_len), a.n_reqs, a.splits);
        LCU_CHECK_CUDA(launch_kernel(gqa_short_kernel<DQ, DV>, grid, dim3(GS_WARPS * 32), gs_smem<DQ, DV>(), s, pdl, a));
        return LCU_OK;
    }
};
struct LongLaunch {
    const GqaArgs &a;
    cudaStream_t s;
    bool dry;
    template <int DQ, int DV> int run() const {
        const size_t smem = (size_t)2 * GL_TILE * (DQ + DV + 16) * sizeof(bf16);
        if (dry) return raise_smem(gqa_long_kernel<DQ, DV>, smem);
        LCU_CHECK_CUDA(launch_kernel(gqa_long_kernel<DQ, DV>, dim3(a.kv_heads, a.n_blocks), dim3(128), smem, s, false, a));
        return LCU_OK;
    }
};
struct ShortCtas {
    template <int DQ, int DV> int run() const {
        const int n = (int)((size_t)220 * 1024 / gs_smem<DQ, DV>());
        return n < 1 ? 1 : (n > 4 ? 4 : n);
    }
};

}  // namespace

int gqa_prep_launch(const GqaArgs &a, int dt, cudaStream_t s, bool pdl) {
    if (a.n_tok <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_tok <= 65535, "attention: %d tokens in a round", a.n_tok);
    // a norm over all heads is summed once per block: one block per token where there are many
    const dim3 grid(a.qk_norm == 3 && a.n_tok > 64 ? 1 : (gqa_prep_items(a) + 7) / 8, a.n_tok);
    auto go = [&](auto kernel) -> int {
        LCU_CHECK_CUDA(launch_kernel(kernel, grid, dim3(256), 0, s, pdl, a));
        return LCU_OK;
    };
    const bool f32 = dt == LCU_F32;
    if (gqa_prep_more(a) && gqa_prep_runs(a)) {
        const bool runs = a.n_tok >= 64;
        auto run = [&](auto one, auto four) -> int {
            const int n = runs ? 4 : 1;
            LCU_CHECK_CUDA(launch_kernel(runs ? four : one, dim3((gqa_prep_items(a) + 7) / 8, (a.n_tok + n - 1) / n), dim3(256), 0, s, pdl, a));
            return LCU_OK;
        };
        auto by_taps = [&](auto t) -> int {
            using T = decltype(t);
            switch (a.conv ? a.taps : 0) {
            case 0: return run(gqa_prep_run_kernel<T, 0, 1>, gqa_prep_run_kernel<T, 0, 4>);
            case 1: return run(gqa_prep_run_kernel<T, 1, 1>, gqa_prep_run_kernel<T, 1, 4>);
            case 2: return run(gqa_prep_run_kernel<T, 2, 1>, gqa_prep_run_kernel<T, 2, 4>);
            case 3: return run(gqa_prep_run_kernel<T, 3, 1>, gqa_prep_run_kernel<T, 3, 4>);
            default: return run(gqa_prep_run_kernel<T, 4, 1>, gqa_prep_run_kernel<T, 4, 4>);
            }
        };
        return f32 ? by_taps(float{}) : by_taps(bf16{});
    }
    if (a.conv) return f32 ? go(gqa_prep_kernel<float, GQA_PREP_CONV>) : go(gqa_prep_kernel<bf16, GQA_PREP_CONV>);
    if (gqa_prep_more(a)) return f32 ? go(gqa_prep_kernel<float, GQA_PREP_TURN>) : go(gqa_prep_kernel<bf16, GQA_PREP_TURN>);
    if (gqa_prep_wide(a)) return f32 ? go(gqa_prep_kernel<float, GQA_PREP_WIDE>) : go(gqa_prep_kernel<bf16, GQA_PREP_WIDE>);
    return f32 ? go(gqa_prep_kernel<float, GQA_PREP>) : go(gqa_prep_kernel<bf16, GQA_PREP>);
}

int gqa_short_tokens(int heads, int kv_heads) {
    const int n = 32 / (heads / kv_heads);
    return n < 1 ? 1 : n;
}
int gqa_row_tiles(int heads, int kv_heads, int len) { return (len * (heads / kv_heads) + 15) / 16; }
size_t gqa_part_floats(int ctas, int vdim_p) { return (size_t)ctas * 16 * (vdim_p + 2); }
int gqa_short_ctas_per_sm(int dim_p, int vdim_p) { return by_size(dim_p, vdim_p, ShortCtas{}); }

int gqa_short_launch(const GqaArgs &a, cudaStream_t s, bool pdl, bool dry) {
    LCU_REQUIRE(a.dim_p <= MIX_MAX_HEAD && a.vdim_p <= MIX_MAX_HEAD, "attention: head sizes %d / %d (at most %d)", a.dim_p, a.vdim_p, MIX_MAX_HEAD);
    if (!dry && a.n_reqs <= 0) return LCU_OK;
    LCU_REQUIRE(dry || (a.n_reqs <= 65535 && a.splits >= 1 && a.splits <= 65535), "attention: grid out of range");
    return by_size(a.dim_p, a.vdim_p, ShortLaunch{a, s, pdl, dry});
}
int gqa_long_launch(const GqaArgs &a, cudaStream_t s, bool dry) {
    LCU_REQUIRE(a.dim_p <= MIX_MAX_HEAD && a.vdim_p <= MIX_MAX_HEAD, "attention: head sizes %d / %d (at most %d)", a.dim_p, a.vdim_p, MIX_MAX_HEAD);
    if (!dry && a.n_reqs <= 0) return LCU_OK;
    LCU_REQUIRE(dry || a.n_blocks <= 65535, "attention: %d row blocks", a.n_blocks);
    return by_size(a.dim_p, a.vdim_p, LongLaunch{a, s, dry});
}
int gqa_f32_launch(const GqaArgs &a, cudaStream_t s) {
    if (a.n_tok <= 0) return LCU_OK;
    LCU_REQUIRE(a.dim_p <= MIX_MAX_HEAD && a.vdim_p <= MIX_MAX_HEAD, "attention: head sizes %d / %d (at most %d)", a.dim_p, a.vdim_p, MIX_MAX_HEAD);
    const long rows = (long)a.n_tok * a.heads;
    LCU_CHECK_CUDA(launch_kernel(gqa_f32_kernel, dim3((unsigned)((rows + 7) / 8)), dim3(256), 0, s, false, a));
    return LCU_OK;
}

}  // namespace lcu
