// Linear recurrences: per head a matrix S (f32, one per sequence) decays, takes k v^T up and is read along the query,
//     S_i = D_i S_{i-1} + k_i v_i^T,   o_i = S_i^T q_i.
// State space duality (SSD): D_i one number per head, exp(-rate dt_i); keys and queries belong to a group of heads; v_i = dt_i x_i.
// Gated linear attention (GLA): D_i diagonal, one number per key channel.
//
// Portions run in blocks of 16 tokens.  With S the matrix ahead of a block, G_i the decay up to and with token i, R_j that of the
// tokens behind j, and D_ij that of the tokens behind j up to i,
//     o_i = (G_i q_i)^T S + sum_{j <= i} A_ij v_j,   A_ij = q_i^T D_ij k_j
//     S  <- G_16 S + sum_j (R_j k_j) v_j^T.
// The preparation computes A and the decayed operands of all blocks in parallel (for SSD the decays are numbers per token and
// head, so keys and queries stay shared by a group, and A is one triangle of products per group times decays per head).  All
// decays are products of numbers up to one: nothing is divided by a decay.  The scan keeps S in registers throughout a portion;
// the sums over its parts of the key dimension are not on the path from one block's S to the next's.
//
// Everything that enters the recurrence is 32-bit: on tensor cores f32 factors are sums of three bf16 numbers (24 bits, f32
// sums).  Values, SSD's keys and queries -- projections, or short convolutions of them -- enter products as bf16.
//
// Rounds of one token per request, and all portions of all-32-bit contexts, go token by token on the f32 pipes.
#include "rec_common.cuh"

namespace lcu {

namespace {

constexpr int SB = SCAN_BLOCK;
static_assert(SB == 2 * CONV_BLOCK, "blocks are two blocks of the convolutions");

// decay and step size of an SSD head at a token
__device__ __forceinline__ float2 ssd_gates(const ScanArgs &a, const float *row, int h) {
    const float dt = softplus_of(row[a.b_off() + h] + a.decay[a.heads_p + h]);
    return make_float2(expf(-expf(a.decay[h]) * dt), dt);
}

// ------------------------------------------------------------------ portions: operands and coefficients of blocks
// SSD.  Blocks [0, kv_heads) of grid.x: keys, queries and coefficients of a group; behind them: values, 128 pieces of 4 channels.
constexpr int SP_PIECES = 128;
template <int TAPS>
__global__ void __launch_bounds__(256) ssd_prep_kernel(const ScanArgs a) {
    extern __shared__ __align__(16) float sm[];
    grid_dep_launch();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int4 blk = a.blocks[blockIdx.y];  // request, first token, tokens, slot of the coefficients
    const int t0 = blk.y, count = blk.z;
    const bool last = t0 + count == a.req_first[blk.x + 1];
    grid_dep_wait();
    const ConvIn in0 = conv_in(a, t0, blk.x);
    float *out = last ? conv_out(a, blk.x) : nullptr;
    // convolution of four channels for half a block
    auto half_block = [&](int half, int c, auto put) {
        ConvIn in = in0;
        const int n = min(max(count - half * CONV_BLOCK, 0), CONV_BLOCK);
        in.row += (size_t)(half * CONV_BLOCK) * in.stride;
        in.in_portion += half * CONV_BLOCK;
        in.seen += half * CONV_BLOCK;
        conv_block<TAPS>(a, in, c, n, count > half * CONV_BLOCK && count <= (half + 1) * CONV_BLOCK ? out : nullptr, put);
    };
    if ((int)blockIdx.x >= a.kv_heads) {
        const int piece = ((int)blockIdx.x - a.kv_heads) * SP_PIECES + (tid & (SP_PIECES - 1)), half = tid / SP_PIECES, width = a.heads * a.dv_p;
        if (4 * piece >= width || half * CONV_BLOCK >= count) return;
        float *v = a.v + (size_t)(t0 + half * CONV_BLOCK) * width + 4 * piece;
        half_block(half, 2 * a.kv_heads * a.dk_p + 4 * piece, [&](int i, const float4 &y) {
            if (half * CONV_BLOCK + i < count) *reinterpret_cast<float4 *>(v + (size_t)i * width) = y;
        });
        return;
    }
    const int kvh = blockIdx.x, ld = a.dk_p + 4;
    float *qs = sm, *ks = sm + SB * ld, *qk = ks + SB * ld;  // [16][ld], [16][ld], [16][16]
    for (int i = tid; i < a.dk_p; i += 256) {  // (query or key, half, piece)
        const int pieces = a.dk_p / 4, piece = i % pieces, half = i / pieces & 1;
        const bool key = i / pieces >= 2;
        bf16 *dst = reinterpret_cast<bf16 *>(key ? a.k : a.q) + ((size_t)(t0 + half * CONV_BLOCK) * a.kv_heads + kvh) * a.dk_p + 4 * piece;
        float *row = (key ? ks : qs) + half * CONV_BLOCK * ld + 4 * piece;
        half_block(half, (key ? a.kv_heads + kvh : kvh) * a.dk_p + 4 * piece, [&](int j, const float4 &y) {
            const uint2 u = make_uint2(Act<bf16>::pack(y.x, y.y), Act<bf16>::pack(y.z, y.w));
            const float2 lo = Act<bf16>::to_f2(u.x), hi = Act<bf16>::to_f2(u.y);
            *reinterpret_cast<float4 *>(row + j * ld) = make_float4(lo.x, lo.y, hi.x, hi.y);
            if (half * CONV_BLOCK + j < count) *reinterpret_cast<uint2 *>(dst + (size_t)j * a.kv_heads * a.dk_p) = u;
        });
    }
    __syncthreads();
    {
        const int i = tid >> 4, j = tid & 15;
        float x = 0.f;
        if (j <= i)
            for (int d = 0; d < a.dk_p; d += 4) {
                const float4 u = *reinterpret_cast<const float4 *>(qs + i * ld + d), w = *reinterpret_cast<const float4 *>(ks + j * ld + d);
                x = fmaf(u.x, w.x, x); x = fmaf(u.y, w.y, x); x = fmaf(u.z, w.z, x); x = fmaf(u.w, w.w, x);
            }
        qk[tid] = x;
    }
    __syncthreads();
    // two heads per warp at a time, 16 lanes each: lane j has column j of the head's triangle
    const int reps = a.heads / a.kv_heads, j = lane & 15;
    for (int r0 = 2 * warp; r0 < reps; r0 += 16) {
        const int rep = r0 + (lane >> 4);
        const bool ok = rep < reps;
        const int h = kvh * reps + (ok ? rep : 0);
        float2 gd = make_float2(1.f, 0.f);  // a token past the end changes nothing
        if (j < count) gd = ssd_gates(a, in0.row + (size_t)j * in0.stride, h);
        const float skip = a.decay[2 * a.heads_p + h];
        float *dst = a.coef + ((size_t)blk.w * a.heads + h) * SCAN_COEF;
        float p = 0.f, upto = 1.f, rest = 1.f;
#pragma unroll
        for (int i = 0; i < SB; ++i) {
            const float g = __shfl_sync(0xffffffffu, gd.x, i, 16);
            p = i == j ? 1.f : p * g;
            if (i <= j) upto *= g;
            else rest *= g;
            if (ok) dst[i * SB + j] = (i >= j ? p * qk[i * SB + j] * gd.y : 0.f) + (i == j ? skip : 0.f);
        }
        if (ok) {
            dst[SB * SB + j] = upto;
            dst[SB * SB + SB + j] = gd.y * rest;
        }
    }
}

// GLA: one block per head.
__global__ void __launch_bounds__(128) gla_prep_kernel(const ScanArgs a) {
    extern __shared__ __align__(16) float sm[];
    grid_dep_launch();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, ld = a.dk_p + 2, pairs = a.dk_p / 2;
    float *us = sm, *red = us + SB * a.rank_p, *al = red + 4 * SB * SB, *qs = al + SB * ld, *ks = qs + SB * ld;  // [16][rank_p], [4][16][16], [16][ld] x 3
    const int4 blk = a.blocks[blockIdx.y];
    const int t0 = blk.y, count = blk.z;
    grid_dep_wait();
    const float *row0 = a.lat + (size_t)t0 * a.stride;
    for (int i = tid; i < SB * a.rank_p; i += 128) {
        const int t = i / a.rank_p, r = i - t * a.rank_p;
        us[i] = t < count ? row0[(size_t)t * a.stride + a.b_off() + r] : 0.f;
    }
    __syncthreads();
    // decays, queries and keys of four tokens and two channels at a time
    const int width = a.heads * a.dk_p;
    for (int item = tid; item < 4 * pairs; item += 128) {
        const int d = 2 * (item % pairs), tb = item / pairs * 4;
        const float *map = a.gate_map + h * a.dk_p + d;
        const float2 bias = *reinterpret_cast<const float2 *>(map + (size_t)a.rank * width), zero = make_float2(0.f, 0.f);
        float2 z[4] = {bias, bias, bias, bias}, q[4], k[4];
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const float *src = row0 + (size_t)(tb + t) * a.stride + h * a.dk_p + d;
            q[t] = tb + t < count ? *reinterpret_cast<const float2 *>(src) : zero;
            k[t] = tb + t < count ? *reinterpret_cast<const float2 *>(src + width) : zero;
        }
        for (int r = 0; r < a.rank; r += 4) {
            float2 w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) w[e] = r + e < a.rank ? *reinterpret_cast<const float2 *>(map + (size_t)(r + e) * width) : zero;
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const float4 u = *reinterpret_cast<const float4 *>(us + (tb + t) * a.rank_p + r);
                z[t].x = fmaf(w[0].x, u.x, z[t].x); z[t].x = fmaf(w[1].x, u.y, z[t].x); z[t].x = fmaf(w[2].x, u.z, z[t].x); z[t].x = fmaf(w[3].x, u.w, z[t].x);
                z[t].y = fmaf(w[0].y, u.x, z[t].y); z[t].y = fmaf(w[1].y, u.y, z[t].y); z[t].y = fmaf(w[2].y, u.z, z[t].y); z[t].y = fmaf(w[3].y, u.w, z[t].y);
            }
        }
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const bool ok = tb + t < count;  // a token past the end changes nothing
            const int at = (tb + t) * ld + d;
            *reinterpret_cast<float2 *>(al + at) = ok ? make_float2(expf(-softplus_of(-z[t].x) * a.inv_tau), expf(-softplus_of(-z[t].y) * a.inv_tau)) : make_float2(1.f, 1.f);
            *reinterpret_cast<float2 *>(qs + at) = make_float2(q[t].x * a.q_scale, q[t].y * a.q_scale);
            *reinterpret_cast<float2 *>(ks + at) = k[t];
        }
    }
    __syncthreads();
    // operands of the scan: queries with the decays up to them, keys with those behind them
    for (int item = tid; item < 2 * pairs; item += 128) {
        const int d = 2 * (item % pairs);
        const bool key = item >= pairs;
        bf16 *dst = reinterpret_cast<bf16 *>(key ? a.k : a.q) + ((size_t)t0 * a.heads + h) * 3 * a.dk_p + d;
        const float *src = key ? ks : qs;
        float2 g = make_float2(1.f, 1.f);
#pragma unroll
        for (int i = 0; i < SB; ++i) {
            const int t = key ? SB - 1 - i : i;
            const float2 x = *reinterpret_cast<const float2 *>(src + t * ld + d), f = *reinterpret_cast<const float2 *>(al + t * ld + d);
            if (!key) { g.x *= f.x; g.y *= f.y; }
            uint32_t pl[3];
            split3(x.x * g.x, x.y * g.y, pl);
            if (t < count)
#pragma unroll
                for (int p = 0; p < 3; ++p) *reinterpret_cast<uint32_t *>(dst + ((size_t)t * a.heads * 3 + p) * a.dk_p) = pl[p];
            if (key) { g.x *= f.x; g.y *= f.y; }
        }
        if (!key) *reinterpret_cast<float2 *>(a.tail + ((size_t)blk.w * a.heads + h) * a.dk_p + d) = g;
    }
    // rows i and i + 8 of the triangle by four lanes, two channels at a time
    const int i0 = lane >> 2, i1 = i0 + 8;
    float acc0[8], acc1[SB];
#pragma unroll
    for (int j = 0; j < SB; ++j) {
        acc1[j] = 0.f;
        if (j < 8) acc0[j] = 0.f;
    }
    for (int d = 8 * warp + 2 * (lane & 3); d < a.dk_p; d += 32) {
        const float2 q0 = *reinterpret_cast<const float2 *>(qs + i0 * ld + d), q1 = *reinterpret_cast<const float2 *>(qs + i1 * ld + d);
        float2 p0 = q0, p1 = q1;
#pragma unroll
        for (int j = SB - 1; j >= 0; --j) {
            const float2 k = *reinterpret_cast<const float2 *>(ks + j * ld + d);
            if (j < SB - 1) {
                const float2 f = *reinterpret_cast<const float2 *>(al + (j + 1) * ld + d);
                p1.x *= j < i1 ? f.x : 1.f; p1.y *= j < i1 ? f.y : 1.f;
                if (j < 7) { p0.x *= j < i0 ? f.x : 1.f; p0.y *= j < i0 ? f.y : 1.f; }
            }
            acc1[j] = fmaf(p1.y, k.y, fmaf(p1.x, k.x, acc1[j]));
            if (j < 8) acc0[j] = fmaf(p0.y, k.y, fmaf(p0.x, k.x, acc0[j]));
        }
    }
#pragma unroll
    for (int j = 0; j < SB; ++j) {
        float x = acc1[j], y = j < 8 ? acc0[j < 8 ? j : 0] : 0.f;
        x += __shfl_xor_sync(0xffffffffu, x, 1); y += __shfl_xor_sync(0xffffffffu, y, 1);
        x += __shfl_xor_sync(0xffffffffu, x, 2); y += __shfl_xor_sync(0xffffffffu, y, 2);
        if ((lane & 3) == 0) {
            red[(warp * SB + i1) * SB + j] = j <= i1 ? x : 0.f;
            red[(warp * SB + i0) * SB + j] = j <= i0 ? y : 0.f;
        }
    }
    __syncthreads();
    float *dst = a.coef + ((size_t)blk.w * a.heads + h) * SCAN_COEF;
    for (int e = tid; e < SB * SB; e += 128) dst[e] = (red[e] + red[SB * SB + e]) + (red[2 * SB * SB + e] + red[3 * SB * SB + e]);
}

// ------------------------------------------------------------------ portions: the scan on tensor cores
// grid (column slices, heads, requests).  A group of 16 value columns belongs to ST_PARTS warps, each with its part of the key
// dimension: KW tiles of eight.  All matrices are kept transposed (value columns are the rows), so that S, the accumulator of the
// update, is pair by pair the first operand of the products with the queries.
constexpr int ST_PARTS = 4, ST_STAGES = 3;
static_assert(32 * ST_PARTS == 128, "group_sync");

template <int KW, bool VEC> constexpr int st_row_bytes() { return (VEC ? 3 : 1) * 8 * KW * ST_PARTS * 2 + 16; }  // a token's row of planes, padded against bank conflicts
template <int KW, bool VEC> constexpr int st_coef() { return SCAN_COEF + (VEC ? 8 * KW * ST_PARTS : 0); }
template <int KW, bool VEC> constexpr int st_stage(int cols) { return 2 * SB * st_row_bytes<KW, VEC>() + (SB * (cols + 4) + st_coef<KW, VEC>()) * 4; }

template <int KW, bool VEC, int GROUPS>
__global__ void __launch_bounds__(128 * GROUPS) scan_tc_kernel(const ScanArgs a) {
    constexpr int DK = 8 * KW * ST_PARTS, PL = VEC ? 3 : 1, RB = st_row_bytes<KW, VEC>(), THREADS = 128 * GROUPS;
    constexpr int cols = 16 * GROUPS, ldv = cols + 4, stage = st_stage<KW, VEC>(cols);
    extern __shared__ __align__(16) unsigned char smb[];
    __shared__ __align__(16) float s_part[2][GROUPS][ST_PARTS][32][8];
    grid_dep_launch();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int part = warp % ST_PARTS, cg = warp / ST_PARTS;  // part of the key dimension, group of columns
    const int h = blockIdx.y, r = blockIdx.z, kvh = h / (a.heads / a.kv_heads);
    const int col0 = blockIdx.x * cols, col = col0 + 16 * cg;
    const bool valid = col < a.dv_p;
    const int first = a.req_first[r], end = a.req_first[r + 1], n_blk = (end - first + SB - 1) / SB;
    const size_t slot0 = first / SB + r;
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
    // sources of the next block to fetch, and where its piece of the ring is
    const int vch = min(cols, a.dv_p - col0) / 4;  // 16-byte pieces of a value row
    const size_t key_row = (size_t)a.kv_heads * PL * DK;
    const bf16 *kg = reinterpret_cast<const bf16 *>(a.k) + first * key_row + (size_t)kvh * PL * DK, *qg = reinterpret_cast<const bf16 *>(a.q) + (kg - reinterpret_cast<const bf16 *>(a.k));
    const float *vg = a.vin + (size_t)first * a.vin_stride + h * a.dv_p + col0, *cf = a.coef + (slot0 * a.heads + h) * SCAN_COEF;
    const float *tg = VEC ? a.tail + (slot0 * a.heads + h) * DK : nullptr;
    unsigned char *fetch = smb;
    int rows = end - first;  // tokens from the next block on
    auto load = [&]() {
        constexpr int CH = PL * DK / 8, VC = cols / 4;  // 16-byte pieces of a row of planes, of values
#pragma unroll
        for (int i = 0; i < (SB * CH + THREADS - 1) / THREADS; ++i) {
            const int at = i * THREADS + tid, j = at / CH, c = at % CH;
            if (SB * CH % THREADS && at >= SB * CH) break;
            const bool ok = j < rows;
            const size_t off = ok ? j * key_row + 8 * c : 0;
            dt_cp16(fetch + j * RB + 16 * c, kg + off, ok);
            dt_cp16(fetch + (SB + j) * RB + 16 * c, qg + off, ok);
        }
        unsigned char *dv = fetch + 2 * SB * RB, *dc = dv + SB * ldv * 4;
        if (tid < SB * VC) {
            const int j = tid / VC, c = tid % VC;
            const bool ok = j < rows && c < vch;
            dt_cp16(dv + (j * ldv + 4 * c) * 4, vg + (ok ? (size_t)j * a.vin_stride + 4 * c : 0), ok);
        }
        if (THREADS - 1 - tid < SCAN_COEF / 4) {
            const int i = THREADS - 1 - tid;
            dt_cp16(dc + 16 * i, cf + 4 * i, true);
        }
        if constexpr (VEC)
            if (tid < DK / 4) dt_cp16(dc + (SCAN_COEF + 4 * tid) * 4, tg + 4 * tid, true);
        kg += SB * key_row; qg += SB * key_row; vg += (size_t)SB * a.vin_stride; cf += (size_t)a.heads * SCAN_COEF; rows -= SB;
        if constexpr (VEC) tg += (size_t)a.heads * DK;
        fetch = fetch + stage == smb + ST_STAGES * stage ? smb : fetch + stage;
    };
    static_assert(SB * (cols / 4) <= THREADS && SCAN_COEF / 4 <= THREADS && DK / 4 <= THREADS, "one piece per thread");
    const size_t out_row = (size_t)a.heads * a.dv_p;
    float *o = a.v + (size_t)(first + (part >> 1) * 8 + 2 * t) * out_row + (size_t)h * a.dv_p + col + g + (part & 1) * 8;  // this lane's two outputs of a block
    int left = end - first - (part >> 1) * 8 - 2 * t;  // tokens from the first of them on
    const unsigned char *tile = smb;
#pragma unroll
    for (int b = 0; b < ST_STAGES - 1; ++b) {
        if (b < n_blk) load();
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    for (int b = 0; b < n_blk; ++b, tile = tile + stage == smb + ST_STAGES * stage ? smb : tile + stage) {
        asm volatile("cp.async.wait_group %0;" ::"n"(ST_STAGES - 2) : "memory");
        __syncthreads();  // block b has landed, block b - 1 has been read
        if (b + ST_STAGES - 1 < n_blk) load();
        asm volatile("cp.async.commit_group;" ::: "memory");
        const float *tv = reinterpret_cast<const float *>(tile + 2 * SB * RB), *coef = tv + SB * ldv;

        // products of the 16 columns with the queries of tokens 0..7 and 8..15, this warp's key dimensions
        float dot[2][4] = {};
        {
            uint32_t x[2][PL][KW];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int i = 0; i < PL; ++i) dt_tiles<KW, false>(x[n][i], tile + (SB + n * 8 + (lane & 7)) * RB + (i * DK + d0) * 2, lane);
            float low[2][4] = {};
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
                    if constexpr (VEC) {
                        mul(low[n], 1, 1);
                        mul(low[n], 0, PL - 1);
                        mul(low[n], 2, 0);
                        mul(low[n], 0, 1);
                        mul(low[n], 1, 0);
                    } else {
                        mul(low[n], 2, 0);
                        mul(low[n], 1, 0);
                    }
                    mul(dot[n], 0, 0);
                }
            }
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) dot[n][e] += low[n][e];
        }
        // values as first operand: columns g and g + 8, tokens 2 t, 2 t + 1 and 8 behind them
        const float *vp = tv + 2 * t * ldv + 16 * cg + g;
        const float v[2][4] = {{vp[0], vp[ldv], vp[8], vp[ldv + 8]}, {vp[8 * ldv], vp[9 * ldv], vp[8 * ldv + 8], vp[9 * ldv + 8]}};
        const uint32_t v0[2] = {Act<bf16>::pack(v[0][0], v[0][1]), Act<bf16>::pack(v[0][2], v[0][3])},
                       v1[2] = {Act<bf16>::pack(v[1][0], v[1][1]), Act<bf16>::pack(v[1][2], v[1][3])};
        if constexpr (!VEC) {
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const float2 u = *reinterpret_cast<const float2 *>(coef + SB * SB + 8 * n + 2 * t);
                dot[n][0] *= u.x; dot[n][1] *= u.y; dot[n][2] *= u.x; dot[n][3] *= u.y;
            }
        }
        if (part < 2) {  // the block's own tokens: part 0 adds them to tokens 0..7, part 1 to tokens 8..15
            const float2 lo = *reinterpret_cast<const float2 *>(coef + (8 * part + g) * SB + 2 * t), hi = *reinterpret_cast<const float2 *>(coef + (8 * part + g) * SB + 8 + 2 * t);
            uint32_t b0[3], b1[3];
            split3(lo.x, lo.y, b0);
            split3(hi.x, hi.y, b1);
            float c[4] = {};
#pragma unroll
            for (int i = 2; i >= 0; --i) dt_mma16(c, v0, v1, b0[i], b1[i]);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                dot[0][e] += part == 0 ? c[e] : 0.f;
                dot[1][e] += part == 1 ? c[e] : 0.f;
            }
        }
        float4 *mine = reinterpret_cast<float4 *>(s_part[b & 1][cg][part][lane]);
        mine[0] = make_float4(dot[0][0], dot[0][1], dot[0][2], dot[0][3]);
        mine[1] = make_float4(dot[1][0], dot[1][1], dot[1][2], dot[1][3]);

        // the update
        {
            uint32_t kt[PL][2][KW];
#pragma unroll
            for (int i = 0; i < PL; ++i)
#pragma unroll
                for (int n = 0; n < 2; ++n) dt_tiles<KW, true>(kt[i][n], tile + (n * 8 + (lane & 7)) * RB + (i * DK + d0) * 2, lane);
            if constexpr (VEC) {
#pragma unroll
                for (int k = 0; k < KW; ++k) {
                    const float2 u = *reinterpret_cast<const float2 *>(coef + SCAN_COEF + d0 + 8 * k + 2 * t);
                    s[k][0] *= u.x; s[k][1] *= u.y; s[k][2] *= u.x; s[k][3] *= u.y;
#pragma unroll
                    for (int i = PL - 1; i >= 0; --i) dt_mma16(s[k], v0, v1, kt[i][0][k], kt[i][1][k]);
                }
            } else {
                const float total = coef[SB * SB + SB - 1];
                const float2 w0 = *reinterpret_cast<const float2 *>(coef + SB * SB + SB + 2 * t), w1 = *reinterpret_cast<const float2 *>(coef + SB * SB + SB + 8 + 2 * t);
                uint32_t p0[3][2], p1[3][2];
                const float a0[4] = {v[0][0] * w0.x, v[0][1] * w0.y, v[0][2] * w0.x, v[0][3] * w0.y};
                const float a1[4] = {v[1][0] * w1.x, v[1][1] * w1.y, v[1][2] * w1.x, v[1][3] * w1.y};
                dt_operand(a0, p0);
                dt_operand(a1, p1);
#pragma unroll
                for (int k = 0; k < KW; ++k) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) s[k][e] *= total;
#pragma unroll
                    for (int i = 2; i >= 0; --i) dt_mma16(s[k], p0[i], p1[i], kt[0][0][k], kt[0][1][k]);
                }
            }
        }
        group_sync(cg);
        {  // a quarter of the outputs: (column g or g + 8, tokens 2 t and 2 t + 1 of one half)
            float2 y = make_float2(0.f, 0.f);
#pragma unroll
            for (int i = 0; i < ST_PARTS; ++i) {
                const float2 e = *reinterpret_cast<const float2 *>(s_part[b & 1][cg][i][lane] + 2 * part);
                y.x += e.x;
                y.y += e.y;
            }
            if (valid && left > 0) o[0] = y.x;
            if (valid && left > 1) o[out_row] = y.y;
            o += SB * out_row;
            left -= SB;
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

// ------------------------------------------------------------------ token by token
// CTAs [0, heads) of a request: one head each; the CTAs behind them (rounds of one token per request) prepare the attention's
// queries, keys and values.
template <class T, int R, bool VEC>
__global__ void __launch_bounds__(256) scan_step_kernel(const ScanArgs a, const GqaArgs attn, int has_attn) {
    constexpr int DK = 8 * R;
    __shared__ __align__(16) float qs[DK], ks[DK], gs[VEC ? DK : 4], vs[MIX_MAX_HEAD], os[MIX_MAX_HEAD];
    grid_dep_launch();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = lane & 7, r = blockIdx.y;
    if ((int)blockIdx.x >= a.heads) {
        grid_dep_wait();
        const int item0 = ((int)blockIdx.x - a.heads) * 8;
        if (has_attn) gqa_prep_any<T>(attn, r, item0, item0 + 8);  // token r is request r
        return;
    }
    const int h = blockIdx.x, reps = a.heads / a.kv_heads, kvh = h / reps;
    float *st = a.state + ((size_t)(a.req_slot[r] >> 1) * a.heads + h) * a.dv_p * DK + part * 4;
    const int first = a.req_first[r], end = a.req_first[r + 1];
    bool fresh = a.req_pos[r] == 0;
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
    for (int t = first; t < end; ++t) {
        if (t > first) {
            fresh = false;
            fetch(c0, cur);
            fetch(c0 + 32, nxt);
        }
        const ConvIn in = conv_in(a, t, r);
        float decay = 1.f, step = 1.f, skip = 0.f;
        if constexpr (VEC) {
            for (int i = tid; i < DK; i += 256) {
                const float *map = a.gate_map + h * DK + i;
                float z = map[(size_t)a.rank * a.heads * DK];
                for (int e = 0; e < a.rank; ++e) z = fmaf(map[(size_t)e * a.heads * DK], in.row[a.b_off() + e], z);
                gs[i] = expf(-softplus_of(-z) * a.inv_tau);
                qs[i] = in.row[h * DK + i] * a.q_scale;
                ks[i] = in.row[(a.heads + h) * DK + i];
            }
            for (int i = tid; i < a.dv_p; i += 256) vs[i] = in.row[2 * a.heads * DK + h * a.dv_p + i];
        } else {
            float *out = t + 1 == end ? conv_out(a, r) : nullptr;
            float *qk_out = h == kvh * reps ? out : nullptr;  // one of the heads that share q and k leaves their inputs behind
            for (int i = tid; i < 2 * DK + a.dv_p; i += 256) {
                if (i < DK) qs[i] = conv_silu(a, in, kvh * DK + i, qk_out);
                else if (i < 2 * DK) ks[i - DK] = conv_silu(a, in, (a.kv_heads + kvh) * DK + i - DK, qk_out);
                else vs[i - 2 * DK] = conv_silu(a, in, 2 * a.kv_heads * DK + h * a.dv_p + i - 2 * DK, out);
            }
            const float2 g = ssd_gates(a, in.row, h);
            decay = g.x;
            step = g.y;
            skip = a.decay[2 * a.heads_p + h];
        }
        __syncthreads();
        for (int cb = 0; cb < a.dv_p; cb += 32) {
            const int c = cb + c0;
            const float v = c < a.dv_p ? vs[c] : 0.f, u = v * step;
            float o = 0.f;
#pragma unroll
            for (int j = 0; j < R / 4; ++j) {
                const float4 k = *reinterpret_cast<const float4 *>(ks + 32 * j + part * 4), q = *reinterpret_cast<const float4 *>(qs + 32 * j + part * 4);
                float4 g = make_float4(decay, decay, decay, decay);
                if constexpr (VEC) g = *reinterpret_cast<const float4 *>(gs + 32 * j + part * 4);
                float4 &x = cur[j];
                x = make_float4(fmaf(k.x, u, x.x * g.x), fmaf(k.y, u, x.y * g.y), fmaf(k.z, u, x.z * g.z), fmaf(k.w, u, x.w * g.w));
                o = fmaf(x.x, q.x, o); o = fmaf(x.y, q.y, o); o = fmaf(x.z, q.z, o); o = fmaf(x.w, q.w, o);
                if (c < a.dv_p) *reinterpret_cast<float4 *>(st + (size_t)c * DK + 32 * j) = x;
            }
            o = octet_sum(o);
            if (part == 0 && c < a.dv_p) os[c] = fmaf(skip, v, o);
#pragma unroll
            for (int j = 0; j < R / 4; ++j) cur[j] = nxt[j];
            fetch(c + 64, nxt);
        }
        __syncthreads();
        if constexpr (VEC) {
            float ss = 0.f;
            for (int i = lane; i < a.dv_p; i += 32) ss += os[i] * os[i];
            const float n = 1.f / sqrtf(warp_sum(ss) / (float)a.dv + a.eps);
            T *dst = reinterpret_cast<T *>(a.o) + (size_t)t * a.stride_o + (size_t)h * a.dv_p;
            for (int i = tid; i < a.dv_p; i += 256) {
                const float x = os[i] * n * a.norm[i] * silu_f(in.row[a.g_off() + h * a.dv_p + i]);
                if constexpr (sizeof(T) == 4) dst[i] = x;
                else dst[i] = Act<T>::from_f(x);
            }
        } else {
            for (int i = tid; i < a.dv_p; i += 256) a.v[((size_t)t * a.heads + h) * a.dv_p + i] = os[i];
        }
        if (t + 1 < end) __syncthreads();  // the next token's q, k and v
    }
}

// ------------------------------------------------------------------ SSD: gate, then norm in equal parts of all heads' outputs
// grid (parts, tokens).  V numbers at a time: 4 where neither a head nor a part ends inside four.
constexpr int SO_STASH = 8192;  // gated numbers of a part kept in shared memory (longer parts are computed twice)
template <class T, int V>
__global__ void __launch_bounds__(1024) ssd_out_kernel(const ScanArgs a) {
    extern __shared__ __align__(16) float stash[];
    __shared__ float2 sums[32];
    grid_dep_launch();
    const int t = blockIdx.y, len = a.heads * a.dv / a.parts, first = blockIdx.x * len;
    const bool keep = len <= SO_STASH;
    grid_dep_wait();
    const float *y = a.v + (size_t)t * a.heads * a.dv_p, *z = a.lat + (size_t)t * a.stride + a.g_off();
    T *dst = reinterpret_cast<T *>(a.o) + (size_t)t * a.stride_o;
    auto place = [&](int i) { const int h = (first + i) / a.dv; return h * a.dv_p + (first + i) - h * a.dv; };  // of number i of the part
    auto gated4 = [&](int at) {
        const float4 u = *reinterpret_cast<const float4 *>(y + at), w = *reinterpret_cast<const float4 *>(z + at);
        return make_float4(u.x * silu_f(w.x), u.y * silu_f(w.y), u.z * silu_f(w.z), u.w * silu_f(w.w));
    };
    float ss = 0.f;
    for (int i = V * threadIdx.x; i < len; i += V * blockDim.x) {
        const int at = place(i);
        if constexpr (V == 4) {
            const float4 x = gated4(at);
            if (keep) *reinterpret_cast<float4 *>(stash + i) = x;
            ss += dot4(x);
        } else {
            const float x = y[at] * silu_f(z[at]);
            if (keep) stash[i] = x;
            ss += x * x;
        }
    }
    const float n = 1.f / sqrtf(block_sum2(ss, 0.f, sums).x / (float)len + a.eps);
    for (int i = V * threadIdx.x; i < len; i += V * blockDim.x) {
        const int at = place(i);
        if constexpr (V == 4) {
            const float4 x = keep ? *reinterpret_cast<const float4 *>(stash + i) : gated4(at), w = *reinterpret_cast<const float4 *>(a.norm + at);
            st4<T>(dst + at, make_float4(x.x * n * w.x, x.y * n * w.y, x.z * n * w.z, x.w * n * w.w));
        } else {
            const float x = (keep ? stash[i] : y[at] * silu_f(z[at])) * n * a.norm[at];
            if constexpr (sizeof(T) == 4) dst[at] = x;
            else dst[at] = Act<T>::from_f(x);
        }
    }
}

// calls f.template run<K>() with the tiles of eight key dimensions per warp of the scan
template <class F>
int by_key(int dk_p, const F &f) {
    switch (dk_p) {
    case 32: return f.template run<1>();
    case 64: return f.template run<2>();
    case 96: return f.template run<3>();
    case 128: return f.template run<4>();
    case 160: return f.template run<5>();
    case 192: return f.template run<6>();
    case 224: return f.template run<7>();
    case 256: return f.template run<8>();
    default: set_error("linear recurrence: key size %d (a multiple of 32, at most 256)", dk_p); return LCU_ERR_INVALID;
    }
}

template <class K>
int raise_smem(K kernel, size_t smem) {
    if (smem > 32 * 1024) LCU_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));  // beside up to 16 KB of static memory
    return LCU_OK;
}

struct ScanTcLaunch {
    const ScanArgs &a;
    cudaStream_t s;
    bool pdl;
    template <int KW, bool VEC, int GROUPS> int go() const {
        constexpr int cols = 16 * GROUPS;
        const size_t smem = (size_t)ST_STAGES * st_stage<KW, VEC>(cols);
        int rc = raise_smem(scan_tc_kernel<KW, VEC, GROUPS>, smem);
        if (rc) return rc;
        LCU_CHECK_CUDA(launch_kernel(scan_tc_kernel<KW, VEC, GROUPS>, dim3((a.dv_p + cols - 1) / cols, a.heads, a.n_req), dim3(32 * ST_PARTS * GROUPS), smem, s, pdl, a));
        return LCU_OK;
    }
    template <int KW> int run() const {
        // two groups of columns share a CTA's tiles where one group each would not fit the SMs at once
        const bool two = a.dv_p > 16 && (long)a.n_req * a.heads * (a.dv_p / 16) > sm_count();
        if (two) return a.per_channel ? go<KW, true, 2>() : go<KW, false, 2>();
        return a.per_channel ? go<KW, true, 1>() : go<KW, false, 1>();
    }
};
struct ScanStepLaunch {
    const ScanArgs &a;
    const GqaArgs *attn;
    int dt;
    cudaStream_t s;
    bool pdl;
    template <class T, int R, bool VEC> int go() const {
        const dim3 grid(a.heads + (attn ? (gqa_prep_items(*attn) + 7) / 8 : 0), a.n_req);
        LCU_CHECK_CUDA(launch_kernel(scan_step_kernel<T, R, VEC>, grid, dim3(256), 0, s, pdl, a, attn ? *attn : GqaArgs{}, attn ? 1 : 0));
        return LCU_OK;
    }
    template <int KW> int run() const {
        constexpr int R = 4 * KW;
        if (dt == LCU_F32) return a.per_channel ? go<float, R, true>() : go<float, R, false>();
        return a.per_channel ? go<bf16, R, true>() : go<bf16, R, false>();
    }
};

}  // namespace

int scan_prep_launch(const ScanArgs &a, cudaStream_t s, bool pdl) {
    if (a.n_blocks <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_blocks <= 65535 && a.dk_p <= MIX_MAX_HEAD && a.dv_p <= MIX_MAX_HEAD, "linear recurrence: %d blocks, head sizes %d / %d", a.n_blocks, a.dk_p, a.dv_p);
    if (a.per_channel) {
        const size_t smem = (size_t)(3 * SB * (a.dk_p + 2) + SB * a.rank_p + 4 * SB * SB) * 4;
        LCU_REQUIRE(smem <= (size_t)200 * 1024, "linear recurrence: inner size %d of the decays' map", a.rank);
        int rc = raise_smem(gla_prep_kernel, smem);
        if (rc) return rc;
        LCU_CHECK_CUDA(launch_kernel(gla_prep_kernel, dim3(a.heads, a.n_blocks), dim3(128), smem, s, pdl, a));
        return LCU_OK;
    }
    const size_t smem = (size_t)(2 * SB * (a.dk_p + 4) + SB * SB) * 4;
    const dim3 grid(a.kv_heads + (a.heads * a.dv_p / 4 + SP_PIECES - 1) / SP_PIECES, a.n_blocks);
    auto go = [&](auto kernel) -> int {
        int rc = raise_smem(kernel, smem);
        if (rc) return rc;
        LCU_CHECK_CUDA(launch_kernel(kernel, grid, dim3(256), smem, s, pdl, a));
        return LCU_OK;
    };
    switch (a.taps) {
    case 2: return go(ssd_prep_kernel<2>);
    case 3: return go(ssd_prep_kernel<3>);
    case 4: return go(ssd_prep_kernel<4>);
    default: return go(ssd_prep_kernel<0>);
    }
}
int scan_launch(const ScanArgs &a, cudaStream_t s, bool pdl) {
    if (a.n_req <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_req <= 65535 && a.heads <= 65535, "linear recurrence: grid out of range");
    return by_key(a.dk_p, ScanTcLaunch{a, s, pdl});
}
int scan_step_launch(const ScanArgs &a, const GqaArgs *attn, int dt, cudaStream_t s, bool pdl) {
    if (a.n_req <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_req <= 65535 && a.dv_p <= MIX_MAX_HEAD, "linear recurrence: %d requests, value size %d", a.n_req, a.dv_p);
    return by_key(a.dk_p, ScanStepLaunch{a, attn, dt, s, pdl});
}
int scan_out_launch(const ScanArgs &a, int dt, cudaStream_t s, bool pdl) {
    if (a.n_tok <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_tok <= 65535, "linear recurrence: %d tokens in a round", a.n_tok);
    const int len = a.heads * a.dv / a.parts;
    const bool four = a.dv % 4 == 0 && len % 4 == 0;
    const size_t smem = len <= SO_STASH ? (size_t)len * 4 : 0;
    // eight numbers per thread where that takes little time, small blocks where there are many
    const int want = (len / 8 + 31) / 32 * 32, most = (long)a.parts * a.n_tok > 8 * sm_count() ? (len > 2048 ? 256 : 128) : 1024;
    const int threads = want < 128 ? 128 : want > most ? most : want;
    const dim3 grid(a.parts, a.n_tok), block(threads);
    if (dt == LCU_F32) LCU_CHECK_CUDA(launch_kernel(four ? ssd_out_kernel<float, 4> : ssd_out_kernel<float, 1>, grid, block, smem, s, pdl, a));
    else LCU_CHECK_CUDA(launch_kernel(four ? ssd_out_kernel<bf16, 4> : ssd_out_kernel<bf16, 1>, grid, block, smem, s, pdl, a));
    return LCU_OK;
}

}  // namespace lcu
