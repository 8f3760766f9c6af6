// Gated delta rule.  Per head a matrix S (f32, one per sequence) is decayed, corrected towards the new value along the new key
// and read along the query: at token i
//     u_i = beta_i (v_i - g_i S_{i-1}^T k_i),   S_i = g_i S_{i-1} + k_i u_i^T,   o_i = S_i^T q_i
// with q, k, v behind short causal convolutions, q and k unit vectors, and o normed and gated per head.
//
// Portions run in blocks of eight tokens.  With S the matrix ahead of a block, D_ij the decay between tokens j and i, and
// G_i the decay up to token i, the recurrence unrolls to
//     w_i = v_i - G_i (S^T k_i)
//     u_i = beta_i (w_i - sum_{j < i} D_ij (k_i . k_j) u_j)       u = T w, T a lower triangle that depends on k, g, beta alone
//     o_i = G_i (S^T q_i) + sum_{j <= i} D_ij (q_i . k_j) u_j     the sum is (B T) w with B_ij = D_ij (q_i . k_j)
//     S   <- G_8 S + sum_j k_j (D_8j u_j)^T
// The preparation solves for T and B T of every block in parallel; the scan then needs one pass of dot products with S, one
// eight-term sum per token and one pass of updates, with a single reduction across lanes per block.  All decays are products of
// numbers up to one: nothing is divided by a decay.  S is f32 and stays in registers throughout a portion.  Everything is
// 32-bit arithmetic whatever the activation dtype; the scan's products run on the f32 pipes in all-32-bit contexts, and on
// tensor cores with factors of three bf16 numbers (24 bits, f32 sums) otherwise.
//
// Rounds with several tokens per request take three launches (convolutions, gates and triangles / the scan / norm and output
// gate), rounds of one token per request a single one.  The inputs of the convolutions that a later round needs are
// double-buffered by generation (a request's first token reads one half, its last token writes the other); the matrices are
// updated in place, every column by the one warp that read it.
#include "rec_common.cuh"

namespace lcu {

namespace {

// two f32 values per instruction
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pk2(float x, float y) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
    return r;
}
__device__ __forceinline__ float2 up2(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// ------------------------------------------------------------------ portions: convolutions, gates, triangles
// One warp per (block of tokens, query/key head) or (block, value head).  Coefficients of a block and head: rows of T [8][8],
// rows of B T [8][8], G [8], decay from token j to the block's end [8].
constexpr int DB = DELTA_BLOCK;
static_assert(DB == 8 && DB == CONV_BLOCK, "the lane layouts below are those of blocks of eight tokens");

constexpr int DP_WARPS = 4;
template <int TAPS>
__global__ void __launch_bounds__(DP_WARPS * 32, 4) delta_prep_kernel(const DeltaArgs a) {
    extern __shared__ __align__(16) float sm[];
    grid_dep_launch();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    int item = blockIdx.x * DP_WARPS + warp;
    if (item >= a.kv_heads + a.heads) return;
    const int4 blk = a.blocks[blockIdx.y];  // request, first token, tokens, slot of the coefficients
    const int t0 = blk.y, count = blk.z;
    const bool last = t0 + count == a.req_first[blk.x + 1];
    grid_dep_wait();
    const ConvIn in = conv_in(a, t0, blk.x);
    float *out = last ? conv_out(a, blk.x) : nullptr;
    if (item >= a.kv_heads) {
        item -= a.kv_heads;
        const int c0 = 2 * a.kv_heads * a.dk_p + item * a.dv_p;
        float *v = a.v + (size_t)t0 * a.heads * a.dv_p + (size_t)item * a.dv_p;
        for (int d = 4 * lane; d < a.dv_p; d += 128)
            conv_block<TAPS>(a, in, c0 + d, count, out, [&](int i, const float4 &y) { if (i < count) *reinterpret_cast<float4 *>(v + (size_t)i * a.heads * a.dv_p + d) = y; });
        return;
    }
    const int ld = a.dk_p + 4;
    float *ks = sm + (size_t)warp * (2 * DB * ld + 2 * DB * DB), *qs = ks + DB * ld, *kk = qs + DB * ld, *qk = kk + DB * DB;
    for (int d = 4 * lane; d < a.dk_p; d += 128) {
        conv_block<TAPS>(a, in, item * a.dk_p + d, count, out, [&](int i, const float4 &y) { *reinterpret_cast<float4 *>(qs + i * ld + d) = y; });
        conv_block<TAPS>(a, in, (a.kv_heads + item) * a.dk_p + d, count, out, [&](int i, const float4 &y) { *reinterpret_cast<float4 *>(ks + i * ld + d) = y; });
    }
    __syncwarp();
    {  // unit vectors: four lanes sum the squares of a token
        float sq = 0.f, sk = 0.f;
        for (int d = 4 * (lane & 3); d < a.dk_p; d += 16) {
            sq += dot4(*reinterpret_cast<const float4 *>(qs + (lane >> 2) * ld + d));
            sk += dot4(*reinterpret_cast<const float4 *>(ks + (lane >> 2) * ld + d));
        }
        sq += __shfl_xor_sync(0xffffffffu, sq, 1); sk += __shfl_xor_sync(0xffffffffu, sk, 1);
        sq += __shfl_xor_sync(0xffffffffu, sq, 2); sk += __shfl_xor_sync(0xffffffffu, sk, 2);
        const float my_rq = 1.f / sqrtf(sq + 1e-6f) * (1.f / sqrtf((float)a.dk)), my_rk = 1.f / sqrtf(sk + 1e-6f);
#pragma unroll
        for (int i = 0; i < DB; ++i) {
            const float rq = __shfl_sync(0xffffffffu, my_rq, 4 * i), rk = __shfl_sync(0xffffffffu, my_rk, 4 * i);
            for (int d = 4 * lane; d < a.dk_p; d += 128) {
                float4 x = *reinterpret_cast<float4 *>(qs + i * ld + d), y = *reinterpret_cast<float4 *>(ks + i * ld + d);
                x.x *= rq; x.y *= rq; x.z *= rq; x.w *= rq;
                y.x *= rk; y.y *= rk; y.z *= rk; y.w *= rk;
                *reinterpret_cast<float4 *>(qs + i * ld + d) = x;
                *reinterpret_cast<float4 *>(ks + i * ld + d) = y;
                if (i < count) {
                    const size_t at = ((size_t)(t0 + i) * a.kv_heads + item) * a.dk_p;
                    if (a.split) {
                        store_split4(reinterpret_cast<bf16 *>(a.q) + 3 * at, a.dk_p, d, x);
                        store_split4(reinterpret_cast<bf16 *>(a.k) + 3 * at, a.dk_p, d, y);
                    } else {
                        *reinterpret_cast<float4 *>(a.q + at + d) = x;
                        *reinterpret_cast<float4 *>(a.k + at + d) = y;
                    }
                }
            }
        }
    }
    __syncwarp();
    {  // products of all pairs of tokens: this lane's row i against columns j and j + 1
        const int i = lane >> 2, j = 2 * (lane & 3);
        float k0 = 0.f, k1 = 0.f, q0 = 0.f, q1 = 0.f;
        for (int d = 0; d < a.dk_p; d += 4) {
            const float4 ki = *reinterpret_cast<const float4 *>(ks + i * ld + d), qi = *reinterpret_cast<const float4 *>(qs + i * ld + d);
            const float4 x = *reinterpret_cast<const float4 *>(ks + j * ld + d), y = *reinterpret_cast<const float4 *>(ks + (j + 1) * ld + d);
            k0 = fmaf(ki.x, x.x, k0); k0 = fmaf(ki.y, x.y, k0); k0 = fmaf(ki.z, x.z, k0); k0 = fmaf(ki.w, x.w, k0);
            k1 = fmaf(ki.x, y.x, k1); k1 = fmaf(ki.y, y.y, k1); k1 = fmaf(ki.z, y.z, k1); k1 = fmaf(ki.w, y.w, k1);
            q0 = fmaf(qi.x, x.x, q0); q0 = fmaf(qi.y, x.y, q0); q0 = fmaf(qi.z, x.z, q0); q0 = fmaf(qi.w, x.w, q0);
            q1 = fmaf(qi.x, y.x, q1); q1 = fmaf(qi.y, y.y, q1); q1 = fmaf(qi.z, y.z, q1); q1 = fmaf(qi.w, y.w, q1);
        }
        kk[i * DB + j] = k0; kk[i * DB + j + 1] = k1;
        qk[i * DB + j] = q0; qk[i * DB + j + 1] = q1;
    }
    __syncwarp();
    // four heads at a time, eight lanes each: lane c solves column c of the head's triangles
    const int reps = a.heads / a.kv_heads, c = lane & 7;
    for (int r0 = 0; r0 < reps; r0 += 4) {
        const int rep = r0 + (lane >> 3);
        const bool ok = rep < reps;
        const int h = item * reps + (ok ? rep : 0);
        float my_g = 1.f, my_b = 0.f;  // a token past the end changes nothing
        if (c < count) {
            const float *row = in.row + (size_t)c * in.stride;
            my_g = expf(-expf(a.decay[h]) * softplus_of(row[a.a_off() + h] + a.decay[a.heads_p + h]));
            my_b = 1.f / (1.f + expf(-row[a.b_off() + h]));
        }
        float g[DB], x[DB], m[DB], total = 1.f, upto = 1.f, rest = 1.f;
#pragma unroll
        for (int i = 0; i < DB; ++i) {
            g[i] = __shfl_sync(0xffffffffu, my_g, i, 8);
            total *= g[i];
            if (i <= c) upto = total;
        }
#pragma unroll
        for (int i = DB - 1; i > 0; --i)
            if (i > c) rest *= g[i];
#pragma unroll
        for (int i = 0; i < DB; ++i) {
            const float bi = __shfl_sync(0xffffffffu, my_b, i, 8);
            float sum = 0.f, p = 1.f, mm = 0.f;
#pragma unroll
            for (int j = i - 1; j >= 0; --j) {
                p *= g[j + 1];
                sum = fmaf(p * kk[i * DB + j], x[j], sum);
                mm = fmaf(p * qk[i * DB + j], x[j], mm);
            }
            x[i] = (i == c ? my_b : 0.f) - bi * sum;
            m[i] = fmaf(qk[i * DB + i], x[i], mm);
        }
        if (ok) {
            float *dst = a.coef + ((size_t)blk.w * a.heads + h) * DELTA_COEF;
#pragma unroll
            for (int i = 0; i < DB; ++i) {
                dst[i * DB + c] = x[i];
                dst[(DB + i) * DB + c] = m[i];
            }
            dst[2 * DB * DB + c] = upto;
            dst[2 * DB * DB + DB + c] = rest;
        }
    }
}

// ------------------------------------------------------------------ portions: the scan
__device__ __forceinline__ void ds_cp16(float *smem_dst, const float *src, bool valid) {
    unsigned d = (unsigned)__cvta_generic_to_shared(smem_dst);
    int sz = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(sz) : "memory");
}
constexpr int DS_STAGES = 3;

// grid (column slices, heads, requests).  A half warp holds NC columns; lane p of it the key dimensions 2 p, 2 p + 1 of every 32
// (R in all).  After the reduction lane p holds the products of token p & 7, with its key (p < 8) or its query.
template <int R, int NC>
__global__ void __launch_bounds__(128) delta_scan_kernel(const DeltaArgs a) {
    constexpr int DK = 16 * R;
    extern __shared__ __align__(16) float sm[];
    __shared__ __align__(16) float s_w[4][2][DB][NC], s_u[4][2][DB][NC];
    grid_dep_launch();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, grp = lane >> 4, p = lane & 15, tok = p & 7;
    const bool is_q = p >= 8;
    const int h = blockIdx.y, r = blockIdx.z, kvh = h / (a.heads / a.kv_heads);
    const int cols = (blockDim.x >> 5) * 2 * NC, col0 = blockIdx.x * cols, lc = (warp * 2 + grp) * NC, col = col0 + lc;
    const bool valid = col < a.dv_p;  // columns come in whole groups of 16
    const int stage = 2 * DB * DK + DB * cols + DELTA_COEF;
    const int first = a.req_first[r], end = a.req_first[r + 1], n_blk = (end - first + DB - 1) / DB;
    const size_t slot0 = first / DB + r;
    float *st = a.state + (((size_t)(a.req_slot[r] >> 1) * a.heads + h) * a.dv_p + (valid ? col : 0)) * DK + 2 * p;
    const bool fresh = a.req_pos[r] == 0;
    f32x2 s[R / 2][NC];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int i = 0; i < R / 2; ++i) {
            const float2 v = valid && !fresh ? *reinterpret_cast<const float2 *>(st + (size_t)c * DK + 32 * i) : make_float2(0.f, 0.f);
            s[i][c] = pk2(v.x, v.y);
        }
    grid_dep_wait();
    const int vch = min(cols, a.dv_p - col0) / 4;  // 16-byte pieces of a value row
    auto load = [&](int b) {
        float *dst = sm + (size_t)(b % DS_STAGES) * stage;
        const int t0 = first + b * DB;
        for (int i = tid; i < DB * (DK / 4); i += blockDim.x) {
            const int j = i / (DK / 4), c = 4 * (i % (DK / 4));
            const bool ok = t0 + j < end;
            const size_t off = ((size_t)(ok ? t0 + j : first) * a.kv_heads + kvh) * DK + c;
            ds_cp16(dst + j * DK + c, a.k + off, ok);
            ds_cp16(dst + (DB + j) * DK + c, a.q + off, ok);
        }
        for (int i = tid; i < DB * (cols / 4); i += blockDim.x) {
            const int j = i / (cols / 4), c = i % (cols / 4);
            const bool ok = t0 + j < end && c < vch;
            ds_cp16(dst + 2 * DB * DK + j * cols + 4 * c, a.v + ((size_t)(ok ? t0 + j : first) * a.heads + h) * a.dv_p + (ok ? col0 + 4 * c : 0), ok);
        }
        for (int i = tid; i < DELTA_COEF / 4; i += blockDim.x)
            ds_cp16(dst + 2 * DB * DK + DB * cols + 4 * i, a.coef + ((slot0 + b) * a.heads + h) * DELTA_COEF + 4 * i, true);
    };
#pragma unroll
    for (int b = 0; b < DS_STAGES - 1; ++b) {
        if (b < n_blk) load(b);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    for (int b = 0; b < n_blk; ++b) {
        asm volatile("cp.async.wait_group %0;" ::"n"(DS_STAGES - 2) : "memory");
        __syncthreads();  // block b has landed, block b - 1 has been read
        if (b + DS_STAGES - 1 < n_blk) load(b + DS_STAGES - 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        const float *tile = sm + (size_t)(b % DS_STAGES) * stage, *coef = tile + 2 * DB * DK + DB * cols;

        float acc[8][NC];  // after the first exchange: products with the eight keys (p < 8) or queries
        {
            f32x2 d[2 * DB][NC];
#pragma unroll
            for (int i = 0; i < 2 * DB; ++i)
#pragma unroll
                for (int c = 0; c < NC; ++c) d[i][c] = 0ull;
#pragma unroll
            for (int i = 0; i < R / 2; ++i)
#pragma unroll
                for (int j = 0; j < 2 * DB; ++j) {
                    const f32x2 x = *reinterpret_cast<const f32x2 *>(tile + j * DK + 32 * i + 2 * p);
#pragma unroll
                    for (int c = 0; c < NC; ++c) d[j][c] = fma2(s[i][c], x, d[j][c]);
                }
#pragma unroll
            for (int j = 0; j < DB; ++j)
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const float2 x = up2(d[j][c]), y = up2(d[DB + j][c]);
                    const float kd = x.x + x.y, qd = y.x + y.y;
                    acc[j][c] = (is_q ? qd : kd) + __shfl_xor_sync(0xffffffffu, is_q ? kd : qd, 8);
                }
        }
#pragma unroll
        for (int m = 4; m > 0; m >>= 1)
#pragma unroll
            for (int j = 0; j < m; ++j)
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const float lo = acc[j][c], hi = acc[j + m][c];
                    acc[j][c] = ((p & m) ? hi : lo) + __shfl_xor_sync(0xffffffffu, (p & m) ? lo : hi, m);
                }
        const float upto = coef[2 * DB * DB + tok], rest = coef[2 * DB * DB + DB + tok], total = coef[2 * DB * DB + DB - 1];
        if (!is_q)
#pragma unroll
            for (int c = 0; c < NC; ++c) s_w[warp][grp][tok][c] = (valid ? tile[2 * DB * DK + tok * cols + lc + c] : 0.f) - upto * acc[0][c];
        __syncwarp();
        float row[DB], y[NC];
#pragma unroll
        for (int j = 0; j < DB; j += 4) {
            const float4 x = *reinterpret_cast<const float4 *>(coef + p * DB + j);
            row[j] = x.x; row[j + 1] = x.y; row[j + 2] = x.z; row[j + 3] = x.w;
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) y[c] = is_q ? upto * acc[0][c] : 0.f;
#pragma unroll
        for (int j = 0; j < DB; ++j)
#pragma unroll
            for (int c = 0; c < NC; ++c) y[c] = fmaf(row[j], s_w[warp][grp][j][c], y[c]);
        const int t = first + b * DB + tok;
        if (!is_q) {
#pragma unroll
            for (int c = 0; c < NC; ++c) s_u[warp][grp][tok][c] = rest * y[c];
        } else if (valid && t < end) {
            float *dst = a.v + ((size_t)t * a.heads + h) * a.dv_p + col;
            if constexpr (NC == 4) *reinterpret_cast<float4 *>(dst) = make_float4(y[0], y[1], y[2], y[3]);
            else *reinterpret_cast<float2 *>(dst) = make_float2(y[0], y[1]);
        }
        __syncwarp();
        const f32x2 total2 = pk2(total, total);
#pragma unroll
        for (int i = 0; i < R / 2; ++i)
#pragma unroll
            for (int c = 0; c < NC; ++c) s[i][c] = mul2(s[i][c], total2);
#pragma unroll
        for (int j = 0; j < DB; ++j) {
            f32x2 u[NC];
#pragma unroll
            for (int c = 0; c < NC; ++c) { const float x = s_u[warp][grp][j][c]; u[c] = pk2(x, x); }
#pragma unroll
            for (int i = 0; i < R / 2; ++i) {
                const f32x2 x = *reinterpret_cast<const f32x2 *>(tile + j * DK + 32 * i + 2 * p);
#pragma unroll
                for (int c = 0; c < NC; ++c) s[i][c] = fma2(x, u[c], s[i][c]);
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (!valid) return;
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int i = 0; i < R / 2; ++i) *reinterpret_cast<float2 *>(st + (size_t)c * DK + 32 * i) = up2(s[i][c]);
}

// ---- the same on tensor cores, for contexts whose activations are bf16
// Every f32 factor is the sum of three bf16 numbers (24 bits); a product is the six largest of their nine products, summed in
// f32.  A group of 16 value columns belongs to DT_PARTS warps, each with its part of the key dimension: KW tiles of eight.  All
// matrices are kept transposed (value columns are the rows), so that the accumulator of one product IS, pair by pair, the first
// operand of the next.  Keys and queries come split from the preparation.  Dot products of the parts are summed through shared
// memory, once per block.
constexpr int DT_PARTS = 4;

template <int KW>
__global__ void __launch_bounds__(256) delta_scan_tc_kernel(const DeltaArgs a) {
    constexpr int DK = 8 * KW * DT_PARTS, RB = 6 * DK + 16;  // bytes of a token's row of planes, padded against bank conflicts
    extern __shared__ __align__(16) unsigned char smb[];
    __shared__ __align__(16) float s_part[2][DT_PARTS][32][8];
    grid_dep_launch();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int part = warp % DT_PARTS, cg = warp / DT_PARTS;  // part of the key dimension, group of columns
    const int h = blockIdx.y, r = blockIdx.z, kvh = h / (a.heads / a.kv_heads);
    const int cols = (blockDim.x >> 5) / DT_PARTS * 16, ldv = cols + 4, col0 = blockIdx.x * cols, col = col0 + 16 * cg;
    const bool valid = col < a.dv_p;
    const int stage = 2 * DB * RB + (DB * ldv + DELTA_COEF) * 4;
    const int first = a.req_first[r], end = a.req_first[r + 1], n_blk = (end - first + DB - 1) / DB;
    const size_t slot0 = first / DB + r;
    const int d0 = part * KW * 8;  // first key dimension of this warp
    float *st = a.state + (((size_t)(a.req_slot[r] >> 1) * a.heads + h) * a.dv_p + (valid ? col + g : 0)) * DK + d0 + 2 * t;
    const bool fresh = a.req_pos[r] == 0;
    float s[KW][4];
#pragma unroll
    for (int k = 0; k < KW; ++k) {
        const float2 x = valid && !fresh ? *reinterpret_cast<const float2 *>(st + 8 * k) : make_float2(0.f, 0.f);
        const float2 y = valid && !fresh ? *reinterpret_cast<const float2 *>(st + (size_t)8 * DK + 8 * k) : make_float2(0.f, 0.f);
        s[k][0] = x.x; s[k][1] = x.y; s[k][2] = y.x; s[k][3] = y.y;
    }
    grid_dep_wait();
    const int vch = min(cols, a.dv_p - col0) / 4;  // 16-byte pieces of a value row
    const bf16 *kg = reinterpret_cast<const bf16 *>(a.k), *qg = reinterpret_cast<const bf16 *>(a.q);
    auto load = [&](int b) {
        unsigned char *dst = smb + (size_t)(b % DS_STAGES) * stage;
        const int t0 = first + b * DB;
        constexpr int CH = 3 * DK / 8;  // 16-byte pieces of a row of planes
        for (int i = tid; i < DB * CH; i += blockDim.x) {
            const int j = i / CH, c = i - j * CH;
            const bool ok = t0 + j < end;
            const size_t off = ((size_t)(ok ? t0 + j : first) * a.kv_heads + kvh) * 3 * DK + 8 * c;
            dt_cp16(dst + j * RB + 16 * c, kg + off, ok);
            dt_cp16(dst + (DB + j) * RB + 16 * c, qg + off, ok);
        }
        unsigned char *dv = dst + 2 * DB * RB;
        if (tid < DB * 8) {
            const int j = tid >> 3, c = tid & 7;
            const bool ok = t0 + j < end && c < vch;
            if (4 * c < cols) dt_cp16(dv + (j * ldv + 4 * c) * 4, a.v + ((size_t)(ok ? t0 + j : first) * a.heads + h) * a.dv_p + (ok ? col0 + 4 * c : 0), ok);
        } else if (tid - DB * 8 < DELTA_COEF / 4) {
            const int i = tid - DB * 8;
            dt_cp16(dv + (DB * ldv + 4 * i) * 4, a.coef + ((slot0 + b) * a.heads + h) * DELTA_COEF + 4 * i, true);
        }
    };
#pragma unroll
    for (int b = 0; b < DS_STAGES - 1; ++b) {
        if (b < n_blk) load(b);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    for (int b = 0; b < n_blk; ++b) {
        asm volatile("cp.async.wait_group %0;" ::"n"(DS_STAGES - 2) : "memory");
        __syncthreads();  // block b has landed, block b - 1 has been read
        if (b + DS_STAGES - 1 < n_blk) load(b + DS_STAGES - 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        const unsigned char *tile = smb + (size_t)(b % DS_STAGES) * stage;
        const float *tv = reinterpret_cast<const float *>(tile + 2 * DB * RB), *coef = tv + DB * ldv;

        // products of the 16 columns with the eight keys (0) and the eight queries (1), this warp's key dimensions
        uint32_t x[2][3][KW];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int i = 0; i < 3; ++i) dt_tiles<KW, false>(x[n][i], tile + (n * DB + (lane & 7)) * RB + (i * DK + d0) * 2, lane);
        float dot[2][4] = {}, low[2][4] = {}, mid[2][4] = {};
#pragma unroll
        for (int k = 0; k < KW; k += 2) {
            uint32_t s0[3][2], s1[3][2];
            dt_operand(s[k], s0);
            if (k + 1 < KW) dt_operand(s[k + 1 < KW ? k + 1 : k], s1);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                auto mul = [&](float c[4], int i, int j) {
                    if (k + 1 < KW) dt_mma16(c, s0[i], s1[i], x[n][j][k], x[n][j][k + 1 < KW ? k + 1 : k]);
                    else dt_mma8(c, s0[i], x[n][j][k]);
                };
                mul(low[n], 1, 1);
                mul(mid[n], 0, 1);
                mul(dot[n], 0, 0);
                mul(low[n], 0, 2);
                mul(mid[n], 1, 0);
                mul(low[n], 2, 0);
            }
        }
        float4 *mine = reinterpret_cast<float4 *>(s_part[cg][part][lane]);
#pragma unroll
        for (int n = 0; n < 2; ++n)
            mine[n] = make_float4(dot[n][0] + (mid[n][0] + low[n][0]), dot[n][1] + (mid[n][1] + low[n][1]), dot[n][2] + (mid[n][2] + low[n][2]),
                                  dot[n][3] + (mid[n][3] + low[n][3]));
        const float2 upto = *reinterpret_cast<const float2 *>(coef + 2 * DB * DB + 2 * t), rest = *reinterpret_cast<const float2 *>(coef + 2 * DB * DB + DB + 2 * t);
        const float total = coef[2 * DB * DB + DB - 1];
        const float *vp = tv + 2 * t * ldv + 16 * cg + g;
        float w[4] = {vp[0], vp[ldv], vp[8], vp[ldv + 8]};  // values of columns g, g + 8 at tokens 2 t, 2 t + 1
        uint32_t tri[2][3];                                 // rows g of T and of B T at tokens 2 t, 2 t + 1
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const float2 z = *reinterpret_cast<const float2 *>(coef + (n * DB + g) * DB + 2 * t);
            split3(z.x, z.y, tri[n]);
        }
        asm volatile("bar.sync %0, %1;" ::"r"(1 + cg), "n"(32 * DT_PARTS) : "memory");
        float dk[4] = {}, y[4] = {};
#pragma unroll
        for (int i = 0; i < DT_PARTS; ++i) {
            const float4 *src = reinterpret_cast<const float4 *>(s_part[cg][i][lane]);
            const float4 e = src[0], f = src[1];
            dk[0] += e.x; dk[1] += e.y; dk[2] += e.z; dk[3] += e.w;
            y[0] += f.x; y[1] += f.y; y[2] += f.z; y[3] += f.w;
        }
        w[0] -= upto.x * dk[0]; w[1] -= upto.y * dk[1]; w[2] -= upto.x * dk[2]; w[3] -= upto.y * dk[3];
        y[0] *= upto.x; y[1] *= upto.y; y[2] *= upto.x; y[3] *= upto.y;
        float u[4] = {};
        uint32_t op[3][2];
        dt_operand(w, op);
        dt_mma8x6(u, op, tri[0]);
        dt_mma8x6(y, op, tri[1]);
        {  // every warp of the group has all outputs: each stores a quarter, (column g or g + 8, token 2 t or 2 t + 1)
            const int tok = first + b * DB + 2 * t + (part & 1), c = col + g + (part >> 1) * 8;
            const float out = part == 0 ? y[0] : (part == 1 ? y[1] : (part == 2 ? y[2] : y[3]));
            if (valid && tok < end) a.v[((size_t)tok * a.heads + h) * a.dv_p + c] = out;
        }
        u[0] *= rest.x; u[1] *= rest.y; u[2] *= rest.x; u[3] *= rest.y;
        dt_operand(u, op);
        uint32_t kt[3][KW];
#pragma unroll
        for (int i = 0; i < 3; ++i) dt_tiles<KW, true>(kt[i], tile + (lane & 7) * RB + (i * DK + d0) * 2, lane);
#pragma unroll
        for (int k = 0; k < KW; ++k) {
#pragma unroll
            for (int e = 0; e < 4; ++e) s[k][e] *= total;
            const uint32_t kb[3] = {kt[0][k], kt[1][k], kt[2][k]};
            dt_mma8x6(s[k], op, kb);
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (!valid) return;
#pragma unroll
    for (int k = 0; k < KW; ++k) {
        *reinterpret_cast<float2 *>(st + 8 * k) = make_float2(s[k][0], s[k][1]);
        *reinterpret_cast<float2 *>(st + (size_t)8 * DK + 8 * k) = make_float2(s[k][2], s[k][3]);
    }
}

// ------------------------------------------------------------------ portions: norm and output gate, a warp per (token, head)
template <class T>
__global__ void __launch_bounds__(256) delta_out_kernel(const DeltaArgs a) {
    grid_dep_launch();
    const int lane = threadIdx.x & 31;
    const long i = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (i >= (long)a.n_tok * a.heads) return;
    const int t = (int)(i / a.heads), h = (int)(i - (long)t * a.heads);
    grid_dep_wait();
    const float *o = a.v + (size_t)i * a.dv_p, *g = a.lat + (size_t)t * a.stride + a.g_off() + h * a.dv_p;
    float4 v[MIX_MAX_HEAD / 128], z[MIX_MAX_HEAD / 128];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 128; ++j) {
        const int d = 4 * lane + 128 * j;
        v[j] = z[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (d < a.dv_p) {
            v[j] = *reinterpret_cast<const float4 *>(o + d);
            z[j] = *reinterpret_cast<const float4 *>(g + d);
        }
        ss += dot4(v[j]);
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)a.dv + a.eps);
    T *dst = reinterpret_cast<T *>(a.o) + (size_t)t * a.stride_o + (size_t)h * a.dv_p;
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 128; ++j) {
        const int d = 4 * lane + 128 * j;
        if (d >= a.dv_p) continue;
        const float4 w = *reinterpret_cast<const float4 *>(a.norm + d);
        st4<T>(dst + d, make_float4(v[j].x * r * w.x * silu_f(z[j].x), v[j].y * r * w.y * silu_f(z[j].y), v[j].z * r * w.z * silu_f(z[j].z),
                                    v[j].w * r * w.w * silu_f(z[j].w)));
    }
}

// ------------------------------------------------------------------ one token per request: everything in one launch
// CTAs [0, heads) of a request: one head each; the CTAs behind them prepare the attention's queries, keys and values.
template <class T, int R>
__global__ void __launch_bounds__(256) delta_decode_kernel(const DeltaArgs a, const GqaArgs attn, int has_attn) {
    constexpr int DK = 8 * R;
    __shared__ __align__(16) float qs[DK], ks[DK], vs[MIX_MAX_HEAD], os[MIX_MAX_HEAD];
    grid_dep_launch();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = lane & 7;
    const int t = blockIdx.y;  // token t is request t
    if (blockIdx.x >= a.heads) {
        grid_dep_wait();
        const int item0 = ((int)blockIdx.x - a.heads) * 8;
        if (has_attn) gqa_prep_any<T>(attn, t, item0, item0 + 8);
        return;
    }
    const int h = blockIdx.x, reps = a.heads / a.kv_heads, kvh = h / reps;
    const bool fresh = a.req_pos[t] == 0;
    float *st = a.state + ((size_t)(a.req_slot[t] >> 1) * a.heads + h) * a.dv_p * DK + part * 4;
    float4 cur[R / 4], nxt[R / 4];
    auto fetch = [&](int c, float4 *d) {
#pragma unroll
        for (int j = 0; j < R / 4; ++j)
            d[j] = !fresh && c < a.dv_p ? *reinterpret_cast<const float4 *>(st + (size_t)c * DK + 32 * j) : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    const int c0 = warp * 4 + (lane >> 3);
    fetch(c0, cur);  // the state is that of an earlier round
    fetch(c0 + 32, nxt);
    grid_dep_wait();
    const ConvIn in = conv_in(a, t, t);
    float *out = conv_out(a, t);
    float *qk_out = h == kvh * reps ? out : nullptr;  // one of the heads that share q and k leaves their inputs behind
    for (int i = tid; i < 2 * DK + a.dv_p; i += 256) {
        if (i < DK) qs[i] = conv_silu(a, in, kvh * DK + i, qk_out);
        else if (i < 2 * DK) ks[i - DK] = conv_silu(a, in, (a.kv_heads + kvh) * DK + i - DK, qk_out);
        else vs[i - 2 * DK] = conv_silu(a, in, 2 * a.kv_heads * DK + h * a.dv_p + i - 2 * DK, out);
    }
    const float g = expf(-expf(a.decay[h]) * softplus_of(in.row[a.a_off() + h] + a.decay[a.heads_p + h]));
    const float beta = 1.f / (1.f + expf(-in.row[a.b_off() + h]));
    __syncthreads();
    float sq = 0.f, sk = 0.f, qk = 0.f;
#pragma unroll
    for (int i = 0; i < DK / 32; ++i) {
        const float x = qs[lane + 32 * i], y = ks[lane + 32 * i];
        sq += x * x;
        sk += y * y;
        qk += x * y;
    }
    const float rq = 1.f / sqrtf(warp_sum(sq) + 1e-6f) * (1.f / sqrtf((float)a.dk)), rk = 1.f / sqrtf(warp_sum(sk) + 1e-6f);
    qk = warp_sum(qk) * rq * rk;
    for (int cb = 0; cb < a.dv_p; cb += 32) {
        const int c = cb + c0;
        float dk = 0.f, dq = 0.f;
        float4 kv[R / 4];
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
            kv[j] = *reinterpret_cast<const float4 *>(ks + 32 * j + part * 4);
            const float4 q = *reinterpret_cast<const float4 *>(qs + 32 * j + part * 4), s = cur[j];
            dk = fmaf(s.x, kv[j].x, dk); dk = fmaf(s.y, kv[j].y, dk); dk = fmaf(s.z, kv[j].z, dk); dk = fmaf(s.w, kv[j].w, dk);
            dq = fmaf(s.x, q.x, dq); dq = fmaf(s.y, q.y, dq); dq = fmaf(s.z, q.z, dq); dq = fmaf(s.w, q.w, dq);
        }
        dk = octet_sum(dk) * rk;
        dq = octet_sum(dq) * rq;
        if (c < a.dv_p) {
            const float u = beta * (vs[c] - g * dk), ur = u * rk;
#pragma unroll
            for (int j = 0; j < R / 4; ++j) {
                const float4 s = cur[j];
                *reinterpret_cast<float4 *>(st + (size_t)c * DK + 32 * j) =
                    make_float4(fmaf(kv[j].x, ur, s.x * g), fmaf(kv[j].y, ur, s.y * g), fmaf(kv[j].z, ur, s.z * g), fmaf(kv[j].w, ur, s.w * g));
            }
            if (part == 0) os[c] = g * dq + qk * u;
        }
#pragma unroll
        for (int j = 0; j < R / 4; ++j) cur[j] = nxt[j];
        fetch(c + 64, nxt);
    }
    __syncthreads();
    float ss = 0.f;
    for (int i = lane; i < a.dv_p; i += 32) ss += os[i] * os[i];
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)a.dv + a.eps);
    T *dst = reinterpret_cast<T *>(a.o) + (size_t)t * a.stride_o + (size_t)h * a.dv_p;
    for (int i = tid; i < a.dv_p; i += 256) {
        const float x = os[i] * r * a.norm[i] * silu_f(in.row[a.g_off() + h * a.dv_p + i]);
        if constexpr (sizeof(T) == 4) dst[i] = x;
        else dst[i] = Act<T>::from_f(x);
    }
}

// calls f.template run<R>() with the key dimensions per lane
template <class F>
int by_dk(int dk_p, const F &f) {
    switch (dk_p) {
    case 32: return f.template run<4>();
    case 64: return f.template run<8>();
    case 96: return f.template run<12>();
    case 128: return f.template run<16>();
    case 160: return f.template run<20>();
    case 192: return f.template run<24>();
    case 224: return f.template run<28>();
    case 256: return f.template run<32>();
    default: set_error("delta rule: key size %d (a multiple of 32, at most 256)", dk_p); return LCU_ERR_INVALID;
    }
}

struct ScanLaunch {
    const DeltaArgs &a;
    cudaStream_t s;
    bool pdl;
    template <class K> int launch(K kernel, int cols, int threads, size_t row_bytes, int ldv) const {
        const size_t smem = (size_t)DS_STAGES * (2 * DB * row_bytes + (DB * ldv + DELTA_COEF) * 4);
        const dim3 grid((a.dv_p + cols - 1) / cols, a.heads, a.n_req);
        if (smem > 32 * 1024) LCU_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));  // beside up to 8 KB of static memory
        LCU_CHECK_CUDA(launch_kernel(kernel, grid, dim3(threads), smem, s, pdl, a));
        return LCU_OK;
    }
    template <int R8> int run() const {
        constexpr int DK = 8 * R8;
        if (a.split) {
            // two groups of columns share a CTA's tiles where one group each would not fit the SMs at once
            const int groups = a.dv_p > 16 && (long)a.n_req * a.heads * (a.dv_p / 16) > sm_count() ? 2 : 1;
            return launch(delta_scan_tc_kernel<DK / 8 / DT_PARTS>, 16 * groups, 32 * DT_PARTS * groups, 6 * DK + 16, 16 * groups + 4);
        }
        constexpr int NC = DK <= 128 ? 4 : 2;  // columns per half warp
        int warps = (a.dv_p + 2 * NC - 1) / (2 * NC);
        if (warps > 4) warps = 4;
        return launch(delta_scan_kernel<DK / 16, NC>, warps * 2 * NC, warps * 32, 4 * DK, warps * 2 * NC);
    }
};
struct DecodeLaunch {
    const DeltaArgs &a;
    const GqaArgs *attn;
    int dt;
    cudaStream_t s;
    bool pdl;
    template <int R> int run() const {
        const dim3 grid(a.heads + (attn ? (gqa_prep_items(*attn) + 7) / 8 : 0), a.n_req);
        const GqaArgs none{};
        if (dt == LCU_F32) LCU_CHECK_CUDA(launch_kernel(delta_decode_kernel<float, R>, grid, dim3(256), 0, s, pdl, a, attn ? *attn : none, attn ? 1 : 0));
        else LCU_CHECK_CUDA(launch_kernel(delta_decode_kernel<bf16, R>, grid, dim3(256), 0, s, pdl, a, attn ? *attn : none, attn ? 1 : 0));
        return LCU_OK;
    }
};

}  // namespace

int delta_prep_launch(const DeltaArgs &a, cudaStream_t s, bool pdl) {
    if (a.n_blocks <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_blocks <= 65535 && a.dk_p <= MIX_MAX_HEAD && a.dv_p <= MIX_MAX_HEAD, "delta rule: %d blocks, head sizes %d / %d", a.n_blocks, a.dk_p, a.dv_p);
    const dim3 grid((a.kv_heads + a.heads + DP_WARPS - 1) / DP_WARPS, a.n_blocks);
    const size_t smem = (size_t)DP_WARPS * (2 * DB * (a.dk_p + 4) + 2 * DB * DB) * 4;
    auto go = [&](auto kernel) -> int {
        if (smem > 48 * 1024) LCU_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        LCU_CHECK_CUDA(launch_kernel(kernel, grid, dim3(DP_WARPS * 32), smem, s, pdl, a));
        return LCU_OK;
    };
    switch (a.taps) {
    case 2: return go(delta_prep_kernel<2>);
    case 3: return go(delta_prep_kernel<3>);
    case 4: return go(delta_prep_kernel<4>);
    default: return go(delta_prep_kernel<0>);
    }
}
int delta_scan_launch(const DeltaArgs &a, cudaStream_t s, bool pdl) {
    if (a.n_req <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_req <= 65535 && a.heads <= 65535, "delta rule: grid out of range");
    return by_dk(a.dk_p, ScanLaunch{a, s, pdl});
}
int delta_out_launch(const DeltaArgs &a, int dt, cudaStream_t s, bool pdl) {
    if (a.n_tok <= 0) return LCU_OK;
    const unsigned grid = (unsigned)(((long)a.n_tok * a.heads + 7) / 8);
    if (dt == LCU_F32) LCU_CHECK_CUDA(launch_kernel(delta_out_kernel<float>, dim3(grid), dim3(256), 0, s, pdl, a));
    else LCU_CHECK_CUDA(launch_kernel(delta_out_kernel<bf16>, dim3(grid), dim3(256), 0, s, pdl, a));
    return LCU_OK;
}
int delta_decode_launch(const DeltaArgs &a, const GqaArgs *attn, int dt, cudaStream_t s, bool pdl) {
    if (a.n_req <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_req <= 65535 && a.dv_p <= MIX_MAX_HEAD, "delta rule: %d requests, value size %d", a.n_req, a.dv_p);
    return by_dk(a.dk_p, DecodeLaunch{a, attn, dt, s, pdl});
}

}  // namespace lcu
