// Latent attention: per-head keys and values are linear maps of one short cached vector per token (the latent), so only the
// latent is cached.  Two forms of the same attention:
//
//   absorbed  the key map is applied to the QUERY instead (q'_h = W_uk_h^T q_h) and the value map to the weighted sum of
//             latents (W_uv_h sum_j p_j c_j): every head then attends the same cached rows, which are read once for all
//             heads -- the form for decoded tokens and short portions (memory-bound);
//   expanded  keys and values of the whole context are materialised once per layer and round and attended per head: fewer
//             operations per (query, key) pair -- the form for long portions (compute-bound).
//
// Arithmetic: scores, softmax and its running state in f32; probabilities are rounded to bf16 only as operands of the
// tensor-core product, the row sum is taken over the rounded values; all sums accumulate in f32.  All-32-bit contexts use
// the absorbed form with f32 FMA throughout.
#include "gemv.cuh"
#include "stack.cuh"

namespace lcu {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ void la_cp_async_16(void *smem_dst, const void *gsrc, bool valid) {
    unsigned dst = (unsigned)__cvta_generic_to_shared(smem_dst);
    int sz = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(gsrc), "r"(sz) : "memory");
}
__device__ __forceinline__ void la_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void la_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void la_ldsm4(uint32_t r[4], const void *row) {
    unsigned a = (unsigned)__cvta_generic_to_shared(row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void la_ldsm2(uint32_t r[2], const void *row) {
    unsigned a = (unsigned)__cvta_generic_to_shared(row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(a));
}
__device__ __forceinline__ void la_ldsm4t(uint32_t r[4], const void *row) {
    unsigned a = (unsigned)__cvta_generic_to_shared(row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}

// ------------------------------------------------------------------ norms of the two latents, append to the cache
template <class T>
__global__ void __launch_bounds__(256) latent_norm_kernel(const LatentNormArgs a) {
    grid_dep_launch();
    __shared__ float2 part[32];
    const int t = blockIdx.x;
    const uint32_t p = a.pos[t];
    const int page = a.page_table[(size_t)a.tok_req[t] * a.pt_stride + (p >> a.page_shift)];
    const int slot = p & ((1 << a.page_shift) - 1);
    grid_dep_wait();
    const float *q = a.lat + (size_t)t * a.stride, *c = q + a.qr_p;
    float sq = 0.f, sc = 0.f;
    for (int i = threadIdx.x; i < a.qr_p / 4; i += blockDim.x) sq += dot4(reinterpret_cast<const float4 *>(q)[i]);
    for (int i = threadIdx.x; i < a.r_p / 4; i += blockDim.x) sc += dot4(reinterpret_cast<const float4 *>(c)[i]);
    const float2 s = block_sum2(sq, sc, part);
    const float rq = 1.f / sqrtf(s.x / (float)a.q_rank + a.eps), rc = 1.f / sqrtf(s.y / (float)a.kv_rank + a.eps);
    T *cq = reinterpret_cast<T *>(a.cq) + (size_t)t * a.qr_p;
    for (int i = threadIdx.x; i < a.qr_p / 4; i += blockDim.x) {
        const float4 v = reinterpret_cast<const float4 *>(q)[i], g = ld4_bf16(a.q_norm, 4 * i);
        st4<T>(cq + 4 * i, make_float4(v.x * rq * g.x, v.y * rq * g.y, v.z * rq * g.z, v.w * rq * g.w));
    }
    T *dst = reinterpret_cast<T *>(a.pool) + (size_t)page * a.page_elems + a.c_off + (size_t)slot * a.r_p;
    for (int i = threadIdx.x; i < a.r_p / 4; i += blockDim.x) {
        const float4 v = reinterpret_cast<const float4 *>(c)[i], g = ld4_bf16(a.kv_norm, 4 * i);
        st4<T>(dst + 4 * i, make_float4(v.x * rc * g.x, v.y * rc * g.y, v.z * rc * g.z, v.w * rc * g.w));
    }
}

int latent_norm_launch(const LatentNormArgs &a, int dt, cudaStream_t s, bool pdl) {
    if (a.n_tok <= 0) return LCU_OK;
    const int block = a.qr_p + a.r_p > 512 ? 256 : 128;
    if (dt == LCU_F32) LCU_CHECK_CUDA(launch_kernel(latent_norm_kernel<float>, dim3(a.n_tok), dim3(block), 0, s, pdl, a));
    else LCU_CHECK_CUDA(launch_kernel(latent_norm_kernel<bf16>, dim3(a.n_tok), dim3(block), 0, s, pdl, a));
    return LCU_OK;
}

// ------------------------------------------------------------------ per-head linear layers
// Weight rows on M (16 per warp), tokens on N.  The whole K range of both operands is requested up front, the weights ahead of the
// dependency wait.  Without `x` the activations are the merged attention partials:
// sum over splits of 2^(m_s - M) o_s (running maxima are kept in powers of two), divided by the merged sum.
constexpr int HL_THREADS = 256, HL_WARPS = 8;
constexpr int HL_MAX_SPLITS = 64;

template <int NT>
__global__ void __launch_bounds__(HL_THREADS) head_linear_kernel(const HeadLinearArgs a) {
    constexpr int NF = NT / 8, YLD = 64 + 8;
    constexpr int NFW = NF == 1 ? 1 : NF / 2;  // 8-token tiles per warp: four warps over the rows, twice over the tokens
    extern __shared__ __align__(16) unsigned char smem[];
    const int ld = a.in + 8;
    bf16 *Ws = reinterpret_cast<bf16 *>(smem);   // [64][in + 8]
    bf16 *Xs = Ws + (size_t)64 * ld;             // [NT][in + 8]
    __shared__ __align__(16) bf16 Ys[NT * YLD];  // output tile, token-major
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, t4 = lane & 3;
    const int o0 = blockIdx.x * 64, h = blockIdx.y, n0 = blockIdx.z * NT;
    const int nt = min(NT, a.n - n0), no = min(64, a.out - o0);
    const bf16 *w = reinterpret_cast<const bf16 *>(a.w) + ((size_t)h * a.out + o0) * a.in;
    grid_dep_launch();
    const int ch = a.in / 8;
    // rows are dealt to lane groups of the chunk count's next power of two, so no lane computes a division per chunk
    const int lpr = ch >= 32 ? 32 : (ch > 16 ? 32 : (ch > 8 ? 16 : (ch > 4 ? 8 : (ch > 2 ? 4 : 2)))), rpw = 32 / lpr;
    const int lr = warp * rpw + lane / lpr, lc = lane % lpr, rstep = HL_WARPS * rpw;
    for (int r = lr; r < 64; r += rstep)  // weights do not depend on the previous kernel
        for (int c = lc; c < ch; c += lpr) la_cp_async_16(Ws + (size_t)r * ld + c * 8, w + (r < no ? (size_t)r * a.in + c * 8 : 0), r < no);
    la_commit();
    grid_dep_wait();
    if (a.x) {
        const bf16 *x = reinterpret_cast<const bf16 *>(a.x) + (size_t)h * a.head_x;
        for (int r = lr; r < NT; r += rstep) {
            const size_t row = r < nt ? (size_t)(a.x_rows ? a.x_rows[n0 + r] : n0 + r) * a.stride_x : 0;
            for (int c = lc; c < ch; c += lpr) la_cp_async_16(Xs + (size_t)r * ld + c * 8, x + row + (r < nt ? c * 8 : 0), r < nt);
        }
        la_commit();
    } else {
        // a warp per row: lane s holds split s's weight 2^(m_s - M) / sum (two splits per lane)
        for (int r = warp; r < NT; r += HL_WARPS) {
            const size_t row = (size_t)(n0 + (r < nt ? r : 0)) * a.heads + h;
            const float2 *ml = reinterpret_cast<const float2 *>(a.part_ml) + row * a.splits;
            // (max, sum) of every split the grid has, requested together with the number in use
            float2 e0 = lane < a.splits ? ml[lane] : make_float2(-INFINITY, 0.f);
            float2 e1 = lane + 32 < a.splits ? ml[lane + 32] : make_float2(-INFINITY, 0.f);
            const int ns = r < nt ? a.part_n[row] : 0;
            if (lane >= ns) e0 = make_float2(-INFINITY, 0.f);
            if (lane + 32 >= ns) e1 = make_float2(-INFINITY, 0.f);
            const float M = warp_max(fmaxf(e0.x, e1.x));
            float w0 = e0.x == -INFINITY ? 0.f : exp2f(e0.x - M), w1 = e1.x == -INFINITY ? 0.f : exp2f(e1.x - M);
            const float inv = ns ? 1.f / warp_sum(w0 * e0.y + w1 * e1.y) : 0.f;
            w0 *= inv;
            w1 *= inv;
            const int c = lane * 4;  // up to four 4-column pieces of the row per lane (a row holds at most 512)
            float4 v[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
            const float *src = a.part_o + row * a.splits * a.in + c;
#pragma unroll 4
            for (int s2 = 0; s2 < ns; ++s2, src += a.in) {
                const float f = __shfl_sync(0xffffffffu, s2 < 32 ? w0 : w1, s2 & 31);
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    if (c + 128 * k < a.in) {
                        const float4 o = *reinterpret_cast<const float4 *>(src + 128 * k);
                        v[k].x = fmaf(f, o.x, v[k].x); v[k].y = fmaf(f, o.y, v[k].y);
                        v[k].z = fmaf(f, o.z, v[k].z); v[k].w = fmaf(f, o.w, v[k].w);
                    }
            }
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (c + 128 * k < a.in) st4<bf16>(Xs + (size_t)r * ld + c + 128 * k, v[k]);
        }
    }
    la_wait<0>();
    __syncthreads();
    const int wm = warp & 3, wn = NF == 1 ? 0 : warp >> 2;
    if (NF > 1 || warp < 4) {
        float acc[NFW][4];
#pragma unroll
        for (int i = 0; i < NFW; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
        const bf16 *wrow = Ws + (size_t)(wm * 16 + (lane & 15)) * ld + (lane >> 4) * 8;
        const bf16 *xrow = Xs + (size_t)(wn * NFW * 8) * ld;
#pragma unroll 4
        for (int k = 0; k < a.in; k += 16) {
            uint32_t af[4];
            la_ldsm4(af, wrow + k);
            if constexpr (NFW == 1) {
                uint32_t b[2];
                la_ldsm2(b, xrow + (size_t)(lane & 7) * ld + k + ((lane >> 3) & 1) * 8);
                mma16816<bf16>(acc[0], af[0], af[1], af[2], af[3], b[0], b[1]);
            } else {
#pragma unroll
                for (int np = 0; np < NFW / 2; ++np) {
                    uint32_t b[4];
                    la_ldsm4(b, xrow + (size_t)(np * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * ld + k + ((lane >> 3) & 1) * 8);
                    mma16816<bf16>(acc[2 * np], af[0], af[1], af[2], af[3], b[0], b[1]);
                    mma16816<bf16>(acc[2 * np + 1], af[0], af[1], af[2], af[3], b[2], b[3]);
                }
            }
        }
#pragma unroll
        for (int f = 0; f < NFW; ++f)
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                const int nl = (wn * NFW + f) * 8 + 2 * t4 + c;
                bf16 *d = Ys + nl * YLD + wm * 16 + gid;
                float g = 1.f;
                if (a.gate && nl < nt) {
                    const int n = n0 + nl;
                    g = 1.f / (1.f + expf(-a.gate[(size_t)(a.y_rows ? a.y_rows[n] : n) * a.stride_gate + h]));
                }
                d[0] = __float2bfloat16_rn(acc[f][c] * g);
                d[8] = __float2bfloat16_rn(acc[f][c + 2] * g);
            }
    }
    __syncthreads();
    bf16 *y = reinterpret_cast<bf16 *>(a.y) + (size_t)h * a.head_y + o0;
    for (int i = tid; i < nt * 8; i += HL_THREADS) {
        const int r = i >> 3, c = (i & 7) * 8;
        if (c < no)
            *reinterpret_cast<uint4 *>(y + (size_t)(a.y_rows ? a.y_rows[n0 + r] : n0 + r) * a.stride_y + c) =
                *reinterpret_cast<const uint4 *>(Ys + r * YLD + c);
    }
}

// Shared-memory attribute of a kernel (set when a context is created: nothing but launches may happen inside a capture).
template <class K>
static int raise_smem(K kernel, size_t smem) {
    if (smem > 48 * 1024) LCU_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return LCU_OK;
}

template <int NT>
static int head_linear_t(const HeadLinearArgs &a, cudaStream_t s, bool pdl, bool dry) {
    const size_t smem = (size_t)(64 + NT) * (a.in + 8) * sizeof(bf16);
    if (dry) return raise_smem(head_linear_kernel<NT>, (size_t)(64 + NT) * (512 + 8) * sizeof(bf16));
    dim3 grid((a.out + 63) / 64, a.heads, (a.n + NT - 1) / NT);
    LCU_REQUIRE(grid.z <= 65535, "head_linear: %d rows", a.n);
    LCU_CHECK_CUDA(launch_kernel(head_linear_kernel<NT>, grid, dim3(HL_THREADS), smem, s, pdl, a));
    return LCU_OK;
}

int head_linear_launch(const HeadLinearArgs &a, cudaStream_t s, bool pdl, bool dry) {
    LCU_REQUIRE(dry || (a.in % 16 == 0 && a.in <= 512), "head_linear: in = %d (a multiple of 16, at most 512)", a.in);
    LCU_REQUIRE(a.x || a.splits <= HL_MAX_SPLITS, "head_linear: %d splits", a.splits);
    if (dry) {
        int rc = head_linear_t<8>(a, s, pdl, true);
        if (!rc) rc = head_linear_t<16>(a, s, pdl, true);
        if (!rc) rc = head_linear_t<32>(a, s, pdl, true);
        return rc ? rc : head_linear_t<64>(a, s, pdl, true);
    }
    if (a.n <= 0) return LCU_OK;
    LCU_REQUIRE(a.out % 8 == 0 && a.stride_y % 8 == 0 && a.head_y % 8 == 0, "head_linear: outputs must be multiples of 8");
    // the widest token tile that still gives every SM a CTA (weights are read once per token tile)
    const long tiles = (long)((a.out + 63) / 64) * a.heads;
    int nt = 64;
    while (nt > 8 && (nt >= 2 * a.n || tiles * ((a.n + nt - 1) / nt) < sm_count())) nt /= 2;
    if (nt == 8) return head_linear_t<8>(a, s, pdl, false);
    if (nt == 16) return head_linear_t<16>(a, s, pdl, false);
    return nt == 32 ? head_linear_t<32>(a, s, pdl, false) : head_linear_t<64>(a, s, pdl, false);
}

// ------------------------------------------------------------------ absorbed attention
constexpr int LA_THREADS = 256;
constexpr int LA_TILE = 64;
constexpr int LA_ROWS_F32 = 8;
constexpr int LD_WARPS = 8, LD_THREADS = 32 * LD_WARPS, LD_SLICES = LD_WARPS / 2;

// Row block b of this launch: its request, first row (token, head pairs of absorbed tokens, token-major), row count.
// Called by every thread; the search runs in warp 0.
struct LaBlock { int req, row0, rows, tok0; };
__device__ __forceinline__ LaBlock la_find_block(const LatentAttnArgs &a, int b, int rows_per_block) {
    LaBlock r;
    if (a.decode) {
        const int bpt = (a.heads + rows_per_block - 1) / rows_per_block;
        r.req = b / bpt;
        r.tok0 = r.req;
        const int j = (b - r.req * bpt) * rows_per_block;
        r.row0 = r.req * a.heads + j;
        r.rows = min(rows_per_block, a.heads - j);
        return r;
    }
    __shared__ LaBlock found;
    if (threadIdx.x < 32) {
        int base = 0;
        for (int i0 = 0; i0 < a.n_req; i0 += 32) {
            const int i = i0 + (int)threadIdx.x;
            int first = 0, rows = 0;
            if (i < a.n_req) {
                first = a.req_first[i];
                rows = (a.req_first[i + 1] - first) * a.heads;
            }
            const int nb = (rows + rows_per_block - 1) / rows_per_block;
            int incl = nb;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, incl, o);
                if ((int)threadIdx.x >= o) incl += v;
            }
            const int lo = base + incl - nb;
            if (b >= lo && b < lo + nb) {
                found.req = i;
                found.tok0 = first;
                found.row0 = first * a.heads + (b - lo) * rows_per_block;
                found.rows = min(rows_per_block, rows - (b - lo) * rows_per_block);
            }
            base += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (threadIdx.x == 0 && b >= base) found.req = -1;
    }
    __syncthreads();
    r = found;
    return r;
}

// Portion form: up to 64 rows of one request against the tiles of one split.  Both products run on tensor cores over the SAME
// shared-memory tile of latents (keys as stored, values through a transposing ldmatrix); tiles are double-buffered.
//   scores  [64 rows x 64 positions]: warps tile rows x positions;   output [64 rows x R]: a warp owns R / 8 columns
template <int RB>
__global__ void __launch_bounds__(LA_THREADS, 1) latent_attn_kernel(const LatentAttnArgs a) {
    constexpr int MT = 4, ROWS = 16 * MT;
    constexpr int NTW = RB / 64;          // most 8-column output tiles per warp
    constexpr int PG = 8 / MT;            // position groups of the score product
    constexpr int SN = LA_TILE / PG / 8;  // 8-position score tiles per warp
    constexpr int PROW = LA_TILE + 8, SROW = LA_TILE + 4;
    extern __shared__ __align__(16) unsigned char smem[];
    const int R = a.r_p, ld = R + 8;
    bf16 *Qs = reinterpret_cast<bf16 *>(smem);                  // [ROWS][ld]
    bf16 *Cs = Qs + (size_t)ROWS * ld;                          // [2][TILE][ld]
    bf16 *Ps = Cs + (size_t)2 * LA_TILE * ld;                   // [ROWS][PROW]
    float *S = reinterpret_cast<float *>(Ps + ROWS * PROW);     // [ROWS][SROW]
    float *corr = S + ROWS * SROW, *m_run = corr + ROWS, *l_run = m_run + ROWS;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, t4 = lane & 3;
    const int sp = blockIdx.y;
    grid_dep_launch();

    const LaBlock blk = la_find_block(a, blockIdx.x, ROWS);
    if (blk.req < 0) return;
    const int rr = a.req_id[blk.req];
    const int pos0 = a.req_pos[rr] - blk.tok0;  // a row's position: pos0 + row / heads
    const int ctx = pos0 + (blk.row0 + blk.rows - 1) / a.heads + 1;
    const int n_tiles = (ctx + LA_TILE - 1) / LA_TILE;
    const int tps = (n_tiles + a.splits - 1) / a.splits;
    const int my_splits = (n_tiles + tps - 1) / tps;
    if (sp >= my_splits) return;
    const int tile0 = sp * tps, tile1 = min(n_tiles, tile0 + tps);
    const int32_t *pages = a.page_table + (size_t)rr * a.pt_stride;
    const bf16 *pool = reinterpret_cast<const bf16 *>(a.pool);
    const int CH = R / 8, dj = LA_THREADS / CH, dc = LA_THREADS - dj * CH;
    const int pmask = (1 << a.page_shift) - 1;

    auto load_tile = [&](int tile, int buf) {
        bf16 *dst = Cs + (size_t)buf * LA_TILE * ld;
        int j = tid / CH, c = tid - j * CH;
        while (j < LA_TILE) {
            const int pos = tile * LA_TILE + j;
            const bool ok = pos < ctx;
            const size_t off = ok ? (size_t)pages[pos >> a.page_shift] * a.page_elems + a.c_off + (size_t)(pos & pmask) * R + c * 8 : 0;
            la_cp_async_16(dst + (size_t)j * ld + c * 8, pool + off, ok);
            j += dj;
            c += dc;
            if (c >= CH) { c -= CH; ++j; }
        }
    };
    for (int i = tid; i < ROWS; i += LA_THREADS) {
        m_run[i] = -INFINITY;
        l_run[i] = 0.f;
    }
    grid_dep_wait();
    {
        const bf16 *q = reinterpret_cast<const bf16 *>(a.q) + (size_t)blk.row0 * R;
        int j = tid / CH, c = tid - j * CH;
        while (j < ROWS) {
            const bool ok = j < blk.rows;
            la_cp_async_16(Qs + (size_t)j * ld + c * 8, q + (ok ? (size_t)j * R + c * 8 : 0), ok);
            j += dj;
            c += dc;
            if (c >= CH) { c -= CH; ++j; }
        }
    }
    load_tile(tile0, 0);
    la_commit();

    float acc[MT][NTW][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < NTW; ++i) acc[m][i][0] = acc[m][i][1] = acc[m][i][2] = acc[m][i][3] = 0.f;
    const int ntw = R / 64;
    const float scale2 = a.scale * 1.4426950408889634f;  // scores in powers of two
    const int wm = warp % MT, wp = warp / MT;  // score product: row tile, position group

    for (int tile = tile0; tile < tile1; ++tile) {
        const int buf = (tile - tile0) & 1;
        if (tile + 1 < tile1) load_tile(tile + 1, buf ^ 1);
        la_commit();
        la_wait<1>();
        __syncthreads();
        const bf16 *C = Cs + (size_t)buf * LA_TILE * ld;
        {
            float sc[SN][4];
#pragma unroll
            for (int i = 0; i < SN; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
            const bf16 *qrow = Qs + (size_t)(wm * 16 + (lane & 15)) * ld + (lane >> 4) * 8;
            const bf16 *crow = C + (size_t)(wp * SN * 8 + (lane & 7) + ((lane >> 4) & 1) * 8) * ld + ((lane >> 3) & 1) * 8;
#pragma unroll 4
            for (int k = 0; k < R; k += 16) {
                uint32_t af[4];
                la_ldsm4(af, qrow + k);
#pragma unroll
                for (int np = 0; np < SN / 2; ++np) {
                    uint32_t b[4];
                    la_ldsm4(b, crow + (size_t)np * 16 * ld + k);
                    mma16816<bf16>(sc[2 * np], af[0], af[1], af[2], af[3], b[0], b[1]);
                    mma16816<bf16>(sc[2 * np + 1], af[0], af[1], af[2], af[3], b[2], b[3]);
                }
            }
#pragma unroll
            for (int i = 0; i < SN; ++i) {
                float *d = S + (size_t)(wm * 16 + gid) * SROW + wp * SN * 8 + i * 8 + 2 * t4;
                *reinterpret_cast<float2 *>(d) = make_float2(sc[i][0], sc[i][1]);
                *reinterpret_cast<float2 *>(d + 8 * SROW) = make_float2(sc[i][2], sc[i][3]);
            }
        }
        __syncthreads();
        // online softmax, a warp per row; a row without a visible position in this tile keeps its state
#pragma unroll
        for (int i = 0; i < 2 * MT; ++i) {
            const int r = warp + 8 * i;
            const int lim = r < blk.rows ? pos0 + (blk.row0 + r) / a.heads : -1;
            const int p0 = tile * LA_TILE + lane, p1 = p0 + 32;
            const float s0 = p0 <= lim ? S[r * SROW + lane] * scale2 : -INFINITY;
            const float s1 = p1 <= lim ? S[r * SROW + lane + 32] * scale2 : -INFINITY;
            const float mo = m_run[r], mn = fmaxf(mo, warp_max(fmaxf(s0, s1)));
            const bf16 pa = __float2bfloat16_rn(s0 == -INFINITY ? 0.f : exp2f(s0 - mn));
            const bf16 pb = __float2bfloat16_rn(s1 == -INFINITY ? 0.f : exp2f(s1 - mn));
            const float sum = warp_sum(__bfloat162float(pa) + __bfloat162float(pb));
            Ps[r * PROW + lane] = pa;
            Ps[r * PROW + lane + 32] = pb;
            if (lane == 0) {
                const float c = mo == -INFINITY ? 0.f : exp2f(mo - mn);
                corr[r] = c;
                l_run[r] = l_run[r] * c + sum;
                m_run[r] = mn;
            }
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float c0 = corr[m * 16 + gid], c1 = corr[m * 16 + gid + 8];
#pragma unroll
            for (int i = 0; i < NTW; ++i) {
                acc[m][i][0] *= c0; acc[m][i][1] *= c0;
                acc[m][i][2] *= c1; acc[m][i][3] *= c1;
            }
        }
#pragma unroll
        for (int k = 0; k < LA_TILE; k += 16) {
            uint32_t pf[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) la_ldsm4(pf[m], Ps + (m * 16 + (lane & 15)) * PROW + k + (lane >> 4) * 8);
            const bf16 *vrow = C + (size_t)(k + (lane & 15)) * ld + warp * (R / 8) + (lane >> 4) * 8;
#pragma unroll
            for (int i = 0; i < NTW; i += 2) {
                if (i < ntw) {  // an odd count reads 8 columns past the warp's own: inside the padded row, not used
                    uint32_t b[4];
                    la_ldsm4t(b, vrow + i * 8);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma16816<bf16>(acc[m][i], pf[m][0], pf[m][1], pf[m][2], pf[m][3], b[0], b[1]);
                        if (NTW > 1 && i + 1 < ntw)
                            mma16816<bf16>(acc[m][i + 1 < NTW ? i + 1 : i], pf[m][0], pf[m][1], pf[m][2], pf[m][3], b[2], b[3]);
                    }
                }
            }
        }
        __syncthreads();
    }
    la_wait<0>();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
            const int r = m * 16 + gid + 8 * hf;
            if (r >= blk.rows) continue;
            float *o = a.part_o + ((size_t)(blk.row0 + r) * a.splits + sp) * R + warp * (R / 8) + 2 * t4;
#pragma unroll
            for (int i = 0; i < NTW; ++i)
                if (i < ntw) *reinterpret_cast<float2 *>(o + i * 8) = make_float2(acc[m][i][2 * hf], acc[m][i][2 * hf + 1]);
        }
    if (tid < blk.rows) {
        const size_t row = blk.row0 + tid;
        reinterpret_cast<float2 *>(a.part_ml)[row * a.splits + sp] = make_float2(m_run[tid], l_run[tid]);
        if (sp == 0) a.part_n[row] = my_splits;
    }
}

// Decode form for pages of fewer than 64 tokens (see latent_tc.cu for the others), up to 32 rows per CTA.  The latent dimension is cut into slices, one per pair of warps; a warp keeps
// its slice of the query fragments in registers for the whole kernel and computes partial scores of 32 positions, which the
// softmax sums over the slices: every byte of a tile crosses the shared-memory port once per product.  Slices and output
// columns are dealt in whole MMA steps, so any latent size that is a multiple of 16 works.  The gather of tile
// t + 1 is in flight during all of tile t.
template <int MT, int RB>
__global__ void __launch_bounds__(LD_THREADS, 1) latent_decode_kernel(const LatentAttnArgs a) {
    constexpr int ROWS = 16 * MT, RPW = ROWS / LD_WARPS;  // rows of the CTA, softmax rows per warp
    constexpr int NTW = RB > 8 * LD_WARPS ? RB / (8 * LD_WARPS) : 1;  // most 8-column output tiles per warp == most k-steps of a slice
    constexpr int PROW = LA_TILE + 8, SROW = LA_TILE + 4;
    extern __shared__ __align__(16) unsigned char smem[];
    const int R = a.r_p, ld = R + 8;
    bf16 *Cs = reinterpret_cast<bf16 *>(smem);                  // [2][TILE][ld]
    bf16 *Ps = Cs + (size_t)2 * LA_TILE * ld;                   // [ROWS][PROW]
    float *S = reinterpret_cast<float *>(Ps + ROWS * PROW);     // [slices][ROWS][SROW]
    float *corr = S + LD_SLICES * ROWS * SROW, *m_run = corr + ROWS, *l_run = m_run + ROWS;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, t4 = lane & 3;
    const int sp = blockIdx.y;
    grid_dep_launch();

    const LaBlock blk = la_find_block(a, blockIdx.x, ROWS);
    if (blk.req < 0) return;
    const int rr = a.req_id[blk.req];
    const int pos0 = a.req_pos[rr] - blk.tok0;
    const int ctx = pos0 + (blk.row0 + blk.rows - 1) / a.heads + 1;
    const int n_tiles = (ctx + LA_TILE - 1) / LA_TILE;
    const int tps = (n_tiles + a.splits - 1) / a.splits;
    const int my_splits = (n_tiles + tps - 1) / tps;
    if (sp >= my_splits) return;
    const int tile0 = sp * tps, tile1 = min(n_tiles, tile0 + tps);
    const int32_t *pages = a.page_table + (size_t)rr * a.pt_stride;
    const bf16 *pool = reinterpret_cast<const bf16 *>(a.pool) + a.c_off;
    const int pmask = (1 << a.page_shift) - 1;
    const int CH = R / 8, dj = LD_THREADS / CH, dc = LD_THREADS - dj * CH, lj = tid / CH, lc = tid - lj * CH;
    const bool whole_page = a.page_shift >= 6 && dc == 0;  // a tile lies in one page and a thread keeps its column
    auto load_tile = [&](int tile, int buf) {
        bf16 *dst = Cs + (size_t)buf * LA_TILE * ld;
        const int p0 = tile * LA_TILE;
        if (whole_page) {
            const bf16 *src = pool + (size_t)pages[p0 >> a.page_shift] * a.page_elems + (size_t)(p0 & pmask) * R + lc * 8;
            bf16 *d = dst + lc * 8;
            const int last = ctx - p0;
#pragma unroll 4
            for (int j = lj; j < LA_TILE; j += dj) la_cp_async_16(d + (size_t)j * ld, src + (j < last ? (size_t)j * R : 0), j < last);
            return;
        }
        int j = lj, c = lc;
        while (j < LA_TILE) {
            const int pos = p0 + j;
            const bool ok = pos < ctx;
            const size_t off = ok ? (size_t)pages[pos >> a.page_shift] * a.page_elems + (size_t)(pos & pmask) * R + c * 8 : 0;
            la_cp_async_16(dst + (size_t)j * ld + c * 8, pool + off, ok);
            j += dj;
            c += dc;
            if (c >= CH) { c -= CH; ++j; }
        }
    };
    for (int i = tid; i < ROWS; i += LD_THREADS) {
        m_run[i] = -INFINITY;
        l_run[i] = 0.f;
    }
    const int ksl = warp >> 1, ph = warp & 1;  // latent slice, half of the tile's positions
    const int k_first = ksl * (R / 16) / LD_SLICES, nk = (ksl + 1) * (R / 16) / LD_SLICES - k_first;      // 16-wide steps of the slice
    const int c_first = warp * (R / 8) / LD_WARPS, ntw = (warp + 1) * (R / 8) / LD_WARPS - c_first;       // 8-wide output tiles
    const float scale2 = a.scale * 1.4426950408889634f;  // scores in powers of two
    grid_dep_wait();
    load_tile(tile0, 0);
    la_commit();
    uint32_t qf[MT][NTW][4];
    {
        const bf16 *q = reinterpret_cast<const bf16 *>(a.q) + (size_t)blk.row0 * R + k_first * 16 + 2 * t4;
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const int ra = m * 16 + gid, rb = ra + 8;
#pragma unroll
            for (int k = 0; k < NTW; ++k) {
                const bool in = k < nk;
                qf[m][k][0] = in && ra < blk.rows ? *reinterpret_cast<const uint32_t *>(q + (size_t)ra * R + k * 16) : 0u;
                qf[m][k][1] = in && rb < blk.rows ? *reinterpret_cast<const uint32_t *>(q + (size_t)rb * R + k * 16) : 0u;
                qf[m][k][2] = in && ra < blk.rows ? *reinterpret_cast<const uint32_t *>(q + (size_t)ra * R + k * 16 + 8) : 0u;
                qf[m][k][3] = in && rb < blk.rows ? *reinterpret_cast<const uint32_t *>(q + (size_t)rb * R + k * 16 + 8) : 0u;
            }
        }
    }
    float acc[MT][NTW][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < NTW; ++i) acc[m][i][0] = acc[m][i][1] = acc[m][i][2] = acc[m][i][3] = 0.f;
    int lim[RPW];  // last visible position of the rows whose softmax this warp computes
#pragma unroll
    for (int i = 0; i < RPW; ++i) lim[i] = warp + LD_WARPS * i < blk.rows ? pos0 + (blk.row0 + warp + LD_WARPS * i) / a.heads : -1;

    for (int tile = tile0; tile < tile1; ++tile) {
        const int buf = (tile - tile0) & 1;
        la_wait<0>();
        __syncthreads();  // the tile has landed for everyone, and everyone is done with the other buffer
        if (tile + 1 < tile1) load_tile(tile + 1, buf ^ 1);
        la_commit();
        const bf16 *C = Cs + (size_t)buf * LA_TILE * ld;
        {
            float sc[MT][4][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int i = 0; i < 4; ++i) sc[m][i][0] = sc[m][i][1] = sc[m][i][2] = sc[m][i][3] = 0.f;
            const bf16 *crow = C + (size_t)(ph * 32 + (lane & 7) + ((lane >> 4) & 1) * 8) * ld + k_first * 16 + ((lane >> 3) & 1) * 8;
#pragma unroll
            for (int k = 0; k < NTW; ++k) {
                if (k < nk) {
#pragma unroll
                    for (int np = 0; np < 2; ++np) {
                        uint32_t b[4];
                        la_ldsm4(b, crow + (size_t)np * 16 * ld + k * 16);
#pragma unroll
                        for (int m = 0; m < MT; ++m) {
                            mma16816<bf16>(sc[m][2 * np], qf[m][k][0], qf[m][k][1], qf[m][k][2], qf[m][k][3], b[0], b[1]);
                            mma16816<bf16>(sc[m][2 * np + 1], qf[m][k][0], qf[m][k][1], qf[m][k][2], qf[m][k][3], b[2], b[3]);
                        }
                    }
                }
            }
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    float *d = S + ((size_t)ksl * ROWS + m * 16 + gid) * SROW + ph * 32 + i * 8 + 2 * t4;
                    *reinterpret_cast<float2 *>(d) = make_float2(sc[m][i][0], sc[m][i][1]);
                    *reinterpret_cast<float2 *>(d + 8 * SROW) = make_float2(sc[m][i][2], sc[m][i][3]);
                }
        }
        __syncthreads();
        {
            float s0[RPW], s1[RPW], mx[RPW], sum[RPW];
            const int p0 = tile * LA_TILE + lane, p1 = p0 + 32;
#pragma unroll
            for (int i = 0; i < RPW; ++i) {
                const float *sr = S + (warp + LD_WARPS * i) * SROW + lane;
                s0[i] = s1[i] = 0.f;
#pragma unroll
                for (int k = 0; k < LD_SLICES; ++k) {
                    s0[i] += sr[k * ROWS * SROW];
                    s1[i] += sr[k * ROWS * SROW + 32];
                }
                s0[i] = p0 <= lim[i] ? s0[i] * scale2 : -INFINITY;
                s1[i] = p1 <= lim[i] ? s1[i] * scale2 : -INFINITY;
                mx[i] = fmaxf(s0[i], s1[i]);
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int i = 0; i < RPW; ++i) mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], o));
#pragma unroll
            for (int i = 0; i < RPW; ++i) {
                const int r = warp + LD_WARPS * i;
                mx[i] = fmaxf(m_run[r], mx[i]);
                const bf16 pa = __float2bfloat16_rn(s0[i] == -INFINITY ? 0.f : exp2f(s0[i] - mx[i]));
                const bf16 pb = __float2bfloat16_rn(s1[i] == -INFINITY ? 0.f : exp2f(s1[i] - mx[i]));
                Ps[r * PROW + lane] = pa;
                Ps[r * PROW + lane + 32] = pb;
                sum[i] = __bfloat162float(pa) + __bfloat162float(pb);
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int i = 0; i < RPW; ++i) sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], o);
            __syncwarp();
            if (lane == 0) {
#pragma unroll
                for (int i = 0; i < RPW; ++i) {
                    const int r = warp + LD_WARPS * i;
                    const float c = m_run[r] == -INFINITY ? 0.f : exp2f(m_run[r] - mx[i]);
                    corr[r] = c;
                    l_run[r] = l_run[r] * c + sum[i];
                    m_run[r] = mx[i];
                }
            }
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float c0 = corr[m * 16 + gid], c1 = corr[m * 16 + gid + 8];
            if (!__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) continue;  // no running maximum moved
#pragma unroll
            for (int i = 0; i < NTW; ++i) {
                acc[m][i][0] *= c0; acc[m][i][1] *= c0;
                acc[m][i][2] *= c1; acc[m][i][3] *= c1;
            }
        }
#pragma unroll
        for (int k = 0; k < LA_TILE; k += 16) {
            uint32_t pf[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) la_ldsm4(pf[m], Ps + (m * 16 + (lane & 15)) * PROW + k + (lane >> 4) * 8);
            const bf16 *vrow = C + (size_t)(k + (lane & 15)) * ld + c_first * 8 + (lane >> 4) * 8;
#pragma unroll
            for (int i = 0; i < NTW; i += 2) {
                if (i < ntw) {  // an odd count reads 8 columns past the warp's own: inside the padded row, not used
                    uint32_t b[4];
                    la_ldsm4t(b, vrow + i * 8);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma16816<bf16>(acc[m][i], pf[m][0], pf[m][1], pf[m][2], pf[m][3], b[0], b[1]);
                        if (NTW > 1 && i + 1 < ntw)
                            mma16816<bf16>(acc[m][i + 1 < NTW ? i + 1 : i], pf[m][0], pf[m][1], pf[m][2], pf[m][3], b[2], b[3]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
            const int r = m * 16 + gid + 8 * hf;
            if (r >= blk.rows) continue;
            float *o = a.part_o + ((size_t)(blk.row0 + r) * a.splits + sp) * R + c_first * 8 + 2 * t4;
#pragma unroll
            for (int i = 0; i < NTW; ++i)
                if (i < ntw) *reinterpret_cast<float2 *>(o + i * 8) = make_float2(acc[m][i][2 * hf], acc[m][i][2 * hf + 1]);
        }
    if (tid < blk.rows) {
        const size_t row = blk.row0 + tid;
        reinterpret_cast<float2 *>(a.part_ml)[row * a.splits + sp] = make_float2(m_run[tid], l_run[tid]);
        if (sp == 0) a.part_n[row] = my_splits;
    }
}

// 32-bit form: one row per warp, a lane per position for the scores, R / 32 output columns per lane; writes normalised rows.
__global__ void __launch_bounds__(LA_ROWS_F32 * 32) latent_attn_f32_kernel(const LatentAttnArgs a) {
    extern __shared__ __align__(16) unsigned char smem[];
    const int R = a.r_p, ld = R + 1;
    float *Qs = reinterpret_cast<float *>(smem);       // [8][R]
    float *Cs = Qs + LA_ROWS_F32 * R;                  // [32][R + 1]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const LaBlock blk = la_find_block(a, blockIdx.x, LA_ROWS_F32);
    if (blk.req < 0) return;
    const int rr = a.req_id[blk.req];
    const int pos0 = a.req_pos[rr] - blk.tok0;
    const int ctx = pos0 + (blk.row0 + blk.rows - 1) / a.heads + 1;
    const int lim = warp < blk.rows ? pos0 + (blk.row0 + warp) / a.heads : -1;
    const int32_t *pages = a.page_table + (size_t)rr * a.pt_stride;
    const float *pool = reinterpret_cast<const float *>(a.pool);
    const float *q = reinterpret_cast<const float *>(a.q) + (size_t)blk.row0 * R;
    for (int i = tid; i < blk.rows * R; i += blockDim.x) Qs[i] = q[i];
    float m = -INFINITY, l = 0.f, acc[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) acc[i] = 0.f;
    for (int p0 = 0; p0 < ctx; p0 += 32) {
        __syncthreads();
        for (int i = tid; i < 32 * R; i += blockDim.x) {
            const int j = i / R, c = i - j * R, pos = p0 + j;
            Cs[j * ld + c] = pos < ctx ? pool[(size_t)pages[pos >> a.page_shift] * a.page_elems + a.c_off +
                                              (size_t)(pos & ((1 << a.page_shift) - 1)) * R + c]
                                       : 0.f;
        }
        __syncthreads();
        if (p0 > lim) continue;  // nothing visible to this warp's row
        float s = 0.f;
        for (int c = 0; c < R; ++c) s = fmaf(Qs[warp * R + c], Cs[lane * ld + c], s);
        s = p0 + lane <= lim ? s * a.scale : -INFINITY;
        const float mn = fmaxf(m, warp_max(s));
        const float p = s == -INFINITY ? 0.f : expf(s - mn), cr = m == -INFINITY ? 0.f : expf(m - mn);
        l = l * cr + warp_sum(p);
        m = mn;
#pragma unroll
        for (int i = 0; i < 16; ++i) acc[i] *= cr;
        for (int j = 0; j < 32; ++j) {
            const float pj = __shfl_sync(0xffffffffu, p, j);
#pragma unroll
            for (int i = 0; i < 16; ++i)
                if (i * 32 < R) acc[i] = fmaf(pj, Cs[j * ld + i * 32 + lane], acc[i]);
        }
    }
    if (warp < blk.rows) {
        const float inv = 1.f / l;
        float *o = a.part_o + (size_t)(blk.row0 + warp) * R;
#pragma unroll
        for (int i = 0; i < 16; ++i)
            if (i * 32 < R) o[i * 32 + lane] = acc[i] * inv;
    }
}

// rows per CTA: as many 16-row tiles as the heads of one token need (decode), or 64 to share every tile among many queries
int latent_attn_rows_per_block(int heads, bool decode, int dt, int page_tokens) {
    if (dt == LCU_F32) return LA_ROWS_F32;
    if (decode && latent_tc_supported(page_tokens)) return latent_tc_rows(heads);
    return !decode ? 64 : (heads > 16 ? 32 : 16);
}

static size_t ld_smem(int mt, int r_p) {
    return (size_t)2 * LA_TILE * (r_p + 8) * 2 + (size_t)16 * mt * (LA_TILE + 8) * 2 + (size_t)16 * mt * (LD_SLICES * (LA_TILE + 4) + 3) * 4;
}
static size_t lp_smem(int mt, int r_p) {
    return (size_t)(16 * mt + 2 * LA_TILE) * (r_p + 8) * 2 + (size_t)16 * mt * (LA_TILE + 8) * 2 + (size_t)16 * mt * (LA_TILE + 4 + 3) * 4;
}

template <int MT, int RB>
static int la_inst(const LatentAttnArgs &a, dim3 grid, cudaStream_t s, bool pdl, bool dry) {
    if constexpr (MT == 4) {
        if (dry) return raise_smem(latent_attn_kernel<RB>, lp_smem(MT, RB));
        LCU_CHECK_CUDA(launch_kernel(latent_attn_kernel<RB>, grid, dim3(LA_THREADS), lp_smem(MT, a.r_p), s, pdl, a));
    } else {
        if (dry) return raise_smem(latent_decode_kernel<MT, RB>, ld_smem(MT, RB));
        LCU_CHECK_CUDA(launch_kernel(latent_decode_kernel<MT, RB>, grid, dim3(LD_THREADS), ld_smem(MT, a.r_p), s, pdl, a));
    }
    return LCU_OK;
}

template <int MT>
static int la_rb(const LatentAttnArgs &a, dim3 grid, cudaStream_t s, bool pdl, bool dry) {
    if (dry) {
        int rc = la_inst<MT, 64>(a, grid, s, pdl, true);
        if (!rc) rc = la_inst<MT, 128>(a, grid, s, pdl, true);
        if (!rc) rc = la_inst<MT, 256>(a, grid, s, pdl, true);
        return rc ? rc : la_inst<MT, 512>(a, grid, s, pdl, true);
    }
    if (a.r_p <= 64) return la_inst<MT, 64>(a, grid, s, pdl, dry);
    if (a.r_p <= 128) return la_inst<MT, 128>(a, grid, s, pdl, dry);
    if (a.r_p <= 256) return la_inst<MT, 256>(a, grid, s, pdl, dry);
    return la_inst<MT, 512>(a, grid, s, pdl, dry);
}

int latent_attn_launch(const LatentAttnArgs &a, int dt, cudaStream_t s, bool pdl, bool dry) {
    LCU_REQUIRE(dry || (a.r_p % 64 == 0 && a.r_p <= 512), "latent attention: latent of %d (a multiple of 64, at most 512)", a.r_p);
    const size_t smem_f32 = (size_t)(LA_ROWS_F32 * a.r_p + 32 * (a.r_p + 1)) * 4;
    if (dry) {
        if (dt == LCU_F32) return raise_smem(latent_attn_f32_kernel, (size_t)(LA_ROWS_F32 * 512 + 32 * 513) * 4);
        int rc = latent_tc_launch(a, s, false, true);
        if (!rc) rc = la_rb<1>(a, dim3(1), s, false, true);
        if (!rc) rc = la_rb<2>(a, dim3(1), s, false, true);
        return rc ? rc : la_rb<4>(a, dim3(1), s, false, true);
    }
    if (a.n_tok <= 0) return LCU_OK;
    const int rpb = latent_attn_rows_per_block(a.heads, a.decode != 0, dt, 1 << a.page_shift);
    // upper bound of row blocks: the exact count of a decode round, one partial block per request otherwise
    const long blocks = a.decode ? (long)a.n_tok * ((a.heads + rpb - 1) / rpb) : (long)a.n_tok * a.heads / rpb + a.n_req;
    LCU_REQUIRE(blocks < (1l << 31) && a.splits >= 1 && a.splits <= HL_MAX_SPLITS, "latent attention: grid out of range");
    const dim3 grid((unsigned)blocks, (unsigned)a.splits);
    if (dt == LCU_F32) {
        LCU_REQUIRE(a.splits == 1, "latent attention: the 32-bit form takes no splits");
        LCU_CHECK_CUDA(launch_kernel(latent_attn_f32_kernel, grid, dim3(LA_ROWS_F32 * 32), smem_f32, s, false, a));
        return LCU_OK;
    }
    if (a.decode && latent_tc_supported(1 << a.page_shift)) return latent_tc_launch(a, s, pdl);
    return rpb == 16 ? la_rb<1>(a, grid, s, pdl, false) : (rpb == 32 ? la_rb<2>(a, grid, s, pdl, false) : la_rb<4>(a, grid, s, pdl, false));
}

// ------------------------------------------------------------------ expanded form
// reqs[i] = (request of the round, cached tokens, first destination row, -)
__global__ void __launch_bounds__(256) latent_gather_kernel(bf16 *dst, const bf16 *pool, size_t page_elems, size_t c_off, int page_shift,
                                                            const int32_t *page_table, int pt_stride, const int4 *reqs, int r_p) {
    const int4 q = reqs[blockIdx.y];
    const int ch = r_p / 8, per = blockDim.x / ch > 0 ? blockDim.x / ch : 1;  // rows per pass
    const int j = threadIdx.x / ch, c = threadIdx.x - j * ch;
    if (j >= per) return;
    for (int row = blockIdx.x * per + j; row < q.y; row += gridDim.x * per) {
        const int page = page_table[(size_t)q.x * pt_stride + (row >> page_shift)];
        const uint4 *src = reinterpret_cast<const uint4 *>(pool + (size_t)page * page_elems + c_off + (size_t)(row & ((1 << page_shift) - 1)) * r_p);
        reinterpret_cast<uint4 *>(dst + (size_t)(q.z + row) * r_p)[c] = src[c];
    }
}

int latent_gather_launch(void *dst, const void *pool, size_t page_elems, size_t c_off, int page_shift, const int32_t *page_table,
                         int pt_stride, const int4 *reqs, int n_req, int max_rows, int r_p, cudaStream_t s) {
    if (n_req <= 0) return LCU_OK;
    LCU_REQUIRE(r_p % 8 == 0 && r_p <= 2048 && n_req <= 65535, "latent gather: latent of %d, %d requests", r_p, n_req);
    const int per = 256 / (r_p / 8) > 0 ? 256 / (r_p / 8) : 1;
    int gx = (max_rows + per - 1) / per;
    if (gx > 1024) gx = 1024;
    latent_gather_kernel<<<dim3(gx, n_req), 256, 0, s>>>((bf16 *)dst, (const bf16 *)pool, page_elems, c_off, page_shift, page_table, pt_stride,
                                                         reqs, r_p);
    LCU_CHECK_CUDA(cudaGetLastError());
    return LCU_OK;
}

// One CTA: 64 query tokens of one request, one head (4 warps x 16 rows).  Query fragments and the output stay in registers,
// key and value tiles of 64 positions are double-buffered, probabilities feed the second product from registers.  Sizes up
// to (DQ, DV); dim_p and vdim_p are multiples of 16.
template <int DQ, int DV>
__global__ void __launch_bounds__(128) expanded_attn_kernel(const ExpandedAttnArgs a) {
    constexpr int KROW = DQ + 8, VROW = DV + 8;
    constexpr int KSTEPS = DQ / 16, NTS = LA_TILE / 8, NTO = DV / 8;
    extern __shared__ __align__(16) unsigned char smem[];
    bf16 *Ks = reinterpret_cast<bf16 *>(smem);        // [2][TILE][KROW]
    bf16 *Vs = Ks + (size_t)2 * LA_TILE * KROW;       // [2][TILE][VROW]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, t4 = lane & 3;
    const int h = blockIdx.x;
    const int4 grp = a.groups[gridDim.y - 1 - blockIdx.y];  // the longest contexts of a prompt first
    const int first = grp.x, count = grp.y, pos0 = grp.z;
    const int ctx = pos0 + count, n_tiles = (ctx + LA_TILE - 1) / LA_TILE;
    const bf16 *kbase = reinterpret_cast<const bf16 *>(a.kv) + (size_t)grp.w * a.stride_kv + (size_t)h * a.dim_p;
    const bf16 *vbase = reinterpret_cast<const bf16 *>(a.kv) + (size_t)grp.w * a.stride_kv + (size_t)a.heads * a.dim_p + (size_t)h * a.vdim_p;
    const int kch = a.dim_p / 8, vch = a.vdim_p / 8;

    auto load_tile = [&](int tile, int buf) {
        bf16 *kd = Ks + (size_t)buf * LA_TILE * KROW, *vd = Vs + (size_t)buf * LA_TILE * VROW;
        for (int i = tid; i < LA_TILE * kch; i += 128) {
            const int j = i / kch, c = (i - j * kch) * 8, pos = tile * LA_TILE + j;
            la_cp_async_16(kd + j * KROW + c, kbase + (pos < ctx ? (size_t)pos * a.stride_kv + c : 0), pos < ctx);
        }
        for (int i = tid; i < LA_TILE * vch; i += 128) {
            const int j = i / vch, c = (i - j * vch) * 8, pos = tile * LA_TILE + j;
            la_cp_async_16(vd + j * VROW + c, vbase + (pos < ctx ? (size_t)pos * a.stride_kv + c : 0), pos < ctx);
        }
    };
    const int r0 = warp * 16 + gid, r1 = r0 + 8;
    const bool v0 = r0 < count, v1 = r1 < count;
    const int lim0 = v0 ? pos0 + r0 : -1, lim1 = v1 ? pos0 + r1 : -1;
    uint32_t qa[KSTEPS][4];
    {
        const bf16 *q0 = reinterpret_cast<const bf16 *>(a.q) + (size_t)(first + (v0 ? r0 : 0)) * a.stride_q + (size_t)h * a.dim_p;
        const bf16 *q1 = reinterpret_cast<const bf16 *>(a.q) + (size_t)(first + (v1 ? r1 : 0)) * a.stride_q + (size_t)h * a.dim_p;
#pragma unroll
        for (int ks = 0; ks < KSTEPS; ++ks) {
            const bool in = ks * 16 < a.dim_p;
            qa[ks][0] = in && v0 ? *reinterpret_cast<const uint32_t *>(q0 + ks * 16 + 2 * t4) : 0u;
            qa[ks][1] = in && v1 ? *reinterpret_cast<const uint32_t *>(q1 + ks * 16 + 2 * t4) : 0u;
            qa[ks][2] = in && v0 ? *reinterpret_cast<const uint32_t *>(q0 + ks * 16 + 8 + 2 * t4) : 0u;
            qa[ks][3] = in && v1 ? *reinterpret_cast<const uint32_t *>(q1 + ks * 16 + 8 + 2 * t4) : 0u;
        }
    }
    load_tile(0, 0);
    la_commit();
    const float scale2 = a.scale * 1.4426950408889634f;  // scores in powers of two
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    float o[NTO][4];
#pragma unroll
    for (int i = 0; i < NTO; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;

    for (int tile = 0; tile < n_tiles; ++tile) {
        const int buf = tile & 1;
        if (tile + 1 < n_tiles) load_tile(tile + 1, buf ^ 1);
        la_commit();
        la_wait<1>();
        __syncthreads();
        const bf16 *Kt = Ks + (size_t)buf * LA_TILE * KROW, *Vt = Vs + (size_t)buf * LA_TILE * VROW;
        float sc[NTS][4];
#pragma unroll
        for (int nt = 0; nt < NTS; ++nt) sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < KSTEPS; ++ks) {
            if (ks * 16 < a.dim_p) {
#pragma unroll
                for (int np = 0; np < NTS / 2; ++np) {
                    uint32_t kb[4];
                    la_ldsm4(kb, Kt + (size_t)(np * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * KROW + ks * 16 + ((lane >> 3) & 1) * 8);
                    mma16816<bf16>(sc[2 * np], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], kb[0], kb[1]);
                    mma16816<bf16>(sc[2 * np + 1], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], kb[2], kb[3]);
                }
            }
        }
        float mt0 = -INFINITY, mt1 = -INFINITY;
#pragma unroll
        for (int nt = 0; nt < NTS; ++nt) {
            const int p = tile * LA_TILE + nt * 8 + 2 * t4;
            sc[nt][0] = p <= lim0 ? sc[nt][0] * scale2 : -INFINITY;
            sc[nt][1] = p + 1 <= lim0 ? sc[nt][1] * scale2 : -INFINITY;
            sc[nt][2] = p <= lim1 ? sc[nt][2] * scale2 : -INFINITY;
            sc[nt][3] = p + 1 <= lim1 ? sc[nt][3] * scale2 : -INFINITY;
            mt0 = fmaxf(mt0, fmaxf(sc[nt][0], sc[nt][1]));
            mt1 = fmaxf(mt1, fmaxf(sc[nt][2], sc[nt][3]));
        }
        mt0 = fmaxf(mt0, __shfl_xor_sync(0xffffffffu, mt0, 1));
        mt0 = fmaxf(mt0, __shfl_xor_sync(0xffffffffu, mt0, 2));
        mt1 = fmaxf(mt1, __shfl_xor_sync(0xffffffffu, mt1, 1));
        mt1 = fmaxf(mt1, __shfl_xor_sync(0xffffffffu, mt1, 2));
        const float mn0 = fmaxf(m0, mt0), mn1 = fmaxf(m1, mt1);
        const float c0 = m0 == -INFINITY ? 0.f : exp2f(m0 - mn0), c1 = m1 == -INFINITY ? 0.f : exp2f(m1 - mn1);
        const float mu0 = mn0 == -INFINITY ? 0.f : mn0, mu1 = mn1 == -INFINITY ? 0.f : mn1;
        m0 = mn0;
        m1 = mn1;
        uint32_t pa[NTS][2];
        float s0 = 0.f, s1 = 0.f;
#pragma unroll
        for (int nt = 0; nt < NTS; ++nt) {
            pa[nt][0] = Act<bf16>::pack(exp2f(sc[nt][0] - mu0), exp2f(sc[nt][1] - mu0));
            pa[nt][1] = Act<bf16>::pack(exp2f(sc[nt][2] - mu1), exp2f(sc[nt][3] - mu1));
            const float2 f0 = Act<bf16>::to_f2(pa[nt][0]), f1 = Act<bf16>::to_f2(pa[nt][1]);
            s0 += f0.x + f0.y;
            s1 += f1.x + f1.y;
        }
        l0 = l0 * c0 + s0;
        l1 = l1 * c1 + s1;
#pragma unroll
        for (int i = 0; i < NTO; ++i) {
            o[i][0] *= c0; o[i][1] *= c0;
            o[i][2] *= c1; o[i][3] *= c1;
        }
#pragma unroll
        for (int kk = 0; kk < LA_TILE / 16; ++kk) {
#pragma unroll
            for (int dp = 0; dp < NTO / 2; ++dp) {
                if (dp * 16 < a.vdim_p) {
                    uint32_t vb[4];
                    la_ldsm4t(vb, Vt + (size_t)(kk * 16 + (lane & 15)) * VROW + dp * 16 + (lane >> 4) * 8);
                    mma16816<bf16>(o[2 * dp], pa[2 * kk][0], pa[2 * kk][1], pa[2 * kk + 1][0], pa[2 * kk + 1][1], vb[0], vb[1]);
                    mma16816<bf16>(o[2 * dp + 1], pa[2 * kk][0], pa[2 * kk][1], pa[2 * kk + 1][0], pa[2 * kk + 1][1], vb[2], vb[3]);
                }
            }
        }
        __syncthreads();
    }
    la_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
        const int r = hf ? r1 : r0;
        if (r >= count) continue;
        float inv = 1.f / (hf ? l1 : l0);
        if (a.gate) inv *= 1.f / (1.f + expf(-a.gate[(size_t)(first + r) * a.stride_gate + h]));
        bf16 *dst = reinterpret_cast<bf16 *>(a.o) + (size_t)(first + r) * a.stride_o + (size_t)h * a.vdim_p + 2 * t4;
#pragma unroll
        for (int i = 0; i < NTO; ++i)
            if (i * 8 < a.vdim_p) *reinterpret_cast<uint32_t *>(dst + 8 * i) = Act<bf16>::pack(o[i][2 * hf] * inv, o[i][2 * hf + 1] * inv);
    }
}

bool expanded_attn_supported(int dim_p, int vdim_p) { return dim_p <= 192 && vdim_p <= 128; }

template <int DQ, int DV>
static int ea_inst(const ExpandedAttnArgs &a, cudaStream_t s, bool dry) {
    const size_t smem = (size_t)2 * LA_TILE * (DQ + DV + 16) * sizeof(bf16);
    if (dry) return raise_smem(expanded_attn_kernel<DQ, DV>, smem);
    LCU_CHECK_CUDA(launch_kernel(expanded_attn_kernel<DQ, DV>, dim3(a.heads, a.n_groups), dim3(128), smem, s, false, a));
    return LCU_OK;
}

int expanded_attn_launch(const ExpandedAttnArgs &a, cudaStream_t s, bool dry) {
    LCU_REQUIRE(expanded_attn_supported(a.dim_p, a.vdim_p) && a.dim_p % 16 == 0 && a.vdim_p % 16 == 0,
                "expanded attention: head sizes %d / %d", a.dim_p, a.vdim_p);
    LCU_REQUIRE(dry || a.n_groups <= 65535, "expanded attention: %d query groups", a.n_groups);
    if (!dry && a.n_groups <= 0) return LCU_OK;
    if (a.vdim_p <= 64) {
        if (a.dim_p <= 64) return ea_inst<64, 64>(a, s, dry);
        if (a.dim_p <= 128) return ea_inst<128, 64>(a, s, dry);
        return ea_inst<192, 64>(a, s, dry);
    }
    if (a.dim_p <= 64) return ea_inst<64, 128>(a, s, dry);
    if (a.dim_p <= 128) return ea_inst<128, 128>(a, s, dry);
    return ea_inst<192, 128>(a, s, dry);
}

}  // namespace lcu
