// Feed-forwards of experts.  A token's router logits choose `top` experts.  Weights on the inputs: the products' linearity lets the
// epilogue apply them, W (s x) = s (W x).  Weights on the outputs, and experts that return their input: the step that adds them up.
#include "moe.cuh"
#include "stack.cuh"

namespace lcu {

namespace {

typedef __nv_bfloat16 bf16;

// The k-th largest scores z(expert) of a token, one warp: calls put(k, expert, score) on every lane.  Equal ones: the lower index
// first.  Scores of up to 32 PER experts are asked for once.
template <int PER, class Z, class F>
__device__ __forceinline__ void top_experts(const Z &z, int n, int top, int lane, const F &put) {
    float last = INFINITY, own[PER ? PER : 1];
    int last_e = -1;
#pragma unroll
    for (int j = 0; j < PER; ++j) own[j] = lane + 32 * j < n ? z(lane + 32 * j) : 0.f;
    for (int k = 0; k < top; ++k) {
        float v = -INFINITY;
        int e = n;
        auto look = [&](int i, float x) {
            if ((x < last || (x == last && i > last_e)) && (x > v || e == n)) { v = x; e = i; }
        };
        if constexpr (PER > 0) {
#pragma unroll
            for (int j = 0; j < PER; ++j)
                if (lane + 32 * j < n) look(lane + 32 * j, own[j]);
        } else {
            for (int i = lane; i < n; i += 32) look(i, z(i));
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float x = __shfl_xor_sync(0xffffffffu, v, o);
            const int i = __shfl_xor_sync(0xffffffffu, e, o);
            if (i < n && (e == n || x > v || (x == v && i < e))) { v = x; e = i; }
        }
        if (e >= n) { e = min(k, n - 1); v = z(e); }  // scores that are not numbers
        put(k, e, v);
        last = v;
        last_e = e;
    }
}
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

// Experts and weights of token t, one warp; put(k, expert) on lane 0.  PER: as above, 0: any number of experts.
template <int PER, class F>
__device__ __forceinline__ void route_token_n(const MoeRoute &a, int t, int lane, const F &put) {
    const float *z = a.logits + (size_t)t * a.experts_p;
    float *weight = a.weight + (size_t)t * a.top;
    const int n = a.experts + a.identity;
    if (!a.softmax) {
        top_experts<PER>([&](int e) { return z[e]; }, n, a.top, lane, [&](int k, int e, float v) {
            if (lane == 0) {
                put(k, e);
                weight[k] = sigmoid_f(v);
            }
        });
        return;
    }
    float m = -INFINITY, sum = 0.f, chosen = 0.f, own[PER ? PER : 1];
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        own[j] = lane + 32 * j < n ? z[lane + 32 * j] : -INFINITY;
        m = fmaxf(m, own[j]);
    }
    if constexpr (PER == 0)
        for (int e = lane; e < n; e += 32) m = fmaxf(m, z[e]);
    m = warp_max(m);
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        own[j] = expf(own[j] - m);
        sum += own[j];
    }
    if constexpr (PER == 0)
        for (int e = lane; e < n; e += 32) sum += expf(z[e] - m);
    sum = warp_sum(sum);
    auto score = [&](int e) {  // of this lane's expert e
        if constexpr (PER > 0) {
            float s = own[0];
#pragma unroll
            for (int j = 1; j < PER; ++j) s = e >= 32 * j ? own[j] : s;
            return s / sum;
        }
        return expf(z[e] - m) / sum;
    };
    top_experts<PER>([&](int e) { return score(e) + a.correction[e]; }, n, a.top, lane, [&](int k, int e, float) {
        const float s = PER > 0 ? __shfl_sync(0xffffffffu, score((e & ~31) + lane), e & 31) : score(e);
        chosen += s;
        if (lane == 0) {
            put(k, e);
            weight[k] = s;
        }
    });
    __syncwarp();
    for (int k = lane; k < a.top; k += 32) weight[k] /= chosen + 1e-20f;
}
template <class F>
__device__ __forceinline__ void route_token(const MoeRoute &a, int t, int lane, const F &put) {
    const int n = a.experts + a.identity;
    if (n <= 32) route_token_n<1>(a, t, lane, put);
    else if (n <= 128) route_token_n<4>(a, t, lane, put);
    else route_token_n<0>(a, t, lane, put);
}

// Exclusive sums of count[0..n) into first, and of (count + per - 1) / per into tile0; one warp; returns the sums of all.
__device__ __forceinline__ int2 warp_offsets(const unsigned *count, int n, int per, int lane, int *first, int *tile0) {
    int2 total = make_int2(0, 0);
    for (int b = 0; b < n; b += 32) {
        const int i = b + lane, c = i < n ? (int)count[i] : 0, t = (c + per - 1) / per;
        int x = c, y = t;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int u = __shfl_up_sync(0xffffffffu, x, o), w = __shfl_up_sync(0xffffffffu, y, o);
            if (lane >= o) { x += u; y += w; }
        }
        if (i < n) { first[i] = total.x + x - c; tile0[i] = total.y + y - t; }
        total.x += __shfl_sync(0xffffffffu, x, 31);
        total.y += __shfl_sync(0xffffffffu, y, 31);
    }
    return total;
}

// ------------------------------------------------------------------ small rounds: one block does it all
__global__ void __launch_bounds__(1024) moe_plan_kernel(const MoeRoute a) {
    extern __shared__ int sm[];
    unsigned *count = reinterpret_cast<unsigned *>(sm);
    int *first = sm + a.experts, *tile0 = first + a.experts, *expert = tile0 + a.experts, *place = expert + a.n_tok * a.top;
    __shared__ int n_tiles;
    grid_dep_launch();
    const int tid = threadIdx.x, lane = tid & 31, rows = a.n_tok * a.top;
    for (int e = tid; e < a.experts; e += blockDim.x) count[e] = 0;
    __syncthreads();
    grid_dep_wait();
    for (int t = tid >> 5; t < a.n_tok; t += blockDim.x >> 5)
        route_token(a, t, lane, [&](int k, int e) {
            expert[t * a.top + k] = e;
            if (e < a.experts) place[t * a.top + k] = (int)atomicAdd(&count[e], 1u);
        });
    __syncthreads();
    if (tid < 32) {
        const int2 n = warp_offsets(count, a.experts, a.n_tok, lane, first, tile0);
        if (lane == 0) n_tiles = n.y;
    }
    __syncthreads();
    for (int i = tid; i < rows; i += blockDim.x) {
        const int slot = expert[i] < a.experts ? first[expert[i]] + place[i] : -1;
        a.slot_of[i] = slot;
        if (slot < 0) continue;
        a.slot_tok[slot] = i / a.top;
        a.slot_w[slot] = a.weight[i];
    }
    for (int e = tid; e < a.experts; e += blockDim.x)
        if (count[e]) a.tiles[tile0[e]] = make_int4(e, first[e], (int)count[e], 0);
    for (int j = n_tiles + tid; j < a.max_tiles; j += blockDim.x) a.tiles[j] = make_int4(0, 0, 0, 0);
}

// ------------------------------------------------------------------ large rounds
__global__ void __launch_bounds__(256) moe_route_kernel(const MoeRoute a) {
    grid_dep_launch();
    const int t = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= a.n_tok) return;
    grid_dep_wait();
    route_token(a, t, lane, [&](int k, int e) {
        a.expert[t * a.top + k] = e;
        if (e < a.experts) a.place[t * a.top + k] = (int)atomicAdd(&a.count[e], 1u);
    });
}

// one block per token; the first one also writes the tiles
template <class T>
__global__ void __launch_bounds__(256) moe_gather_kernel(const MoeRoute a) {
    extern __shared__ int sm[];
    int *first = sm, *tile0 = first + a.experts;
    __shared__ int n_tiles;
    grid_dep_launch();
    const int tid = threadIdx.x, t = blockIdx.x;
    grid_dep_wait();
    if (tid < 32) {
        const int2 n = warp_offsets(a.count, a.experts, a.tile_rows, tid, first, tile0);
        if (tid == 0) n_tiles = n.y;
    }
    __syncthreads();
    const uint4 *src = reinterpret_cast<const uint4 *>(reinterpret_cast<const T *>(a.h) + (size_t)t * a.d_p);
    constexpr int V = 16 / sizeof(T);
    for (int k = 0; k < a.top; ++k) {
        const int i = t * a.top + k, slot = a.expert[i] < a.experts ? first[a.expert[i]] + a.place[i] : -1;
        if (tid == 0) a.slot_of[i] = slot;
        if (slot < 0) continue;
        uint4 *dst = reinterpret_cast<uint4 *>(reinterpret_cast<T *>(a.xg) + (size_t)slot * a.d_p);
        for (int c = tid; c < a.d_p / V; c += 256) dst[c] = src[c];
        if (tid == 0) {
            a.slot_tok[slot] = t;
            a.slot_w[slot] = a.weight[i];
        }
    }
    if (t) return;
    for (int e = tid; e < a.experts; e += 256) {
        const int n = (int)a.count[e];
        for (int j = 0; j < n; j += a.tile_rows) a.tiles[tile0[e] + j / a.tile_rows] = make_int4(e, first[e] + j, min(a.tile_rows, n - j), 0);
    }
    for (int j = n_tiles + tid; j < a.max_tiles; j += 256) a.tiles[j] = make_int4(0, 0, 0, 0);
}

// ------------------------------------------------------------------ products of small rounds
// grid (blocks of 16 output rows, shared expert and tiles).  The four warps of a block take the 64-wide pieces of the summed
// dimension in turn; lane (g, t) holds 16 consecutive numbers of weight rows g and g + 8 and of activation row g, whatever order
// of the summed dimension that makes is the same for both operands.
constexpr int MP_WARPS = 4;
constexpr int MP_LD = 33;
template <int NT, bool UP>  // 8 NT rows at a time
__device__ __forceinline__ void moe_rows(const MoeProduct &a, const int4 &tile, bool sh, int out, int in, int row0, float (*red)[16][MP_LD]) {
    constexpr int DEPTH = NT == 1 ? 4 : (NT == 2 ? 3 : 2);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const unsigned char *w0 = reinterpret_cast<const unsigned char *>(sh ? a.ws : a.w) + (((size_t)tile.x * out + row0 + g) * in + 16 * t) * 2;
    const unsigned char *w1 = w0 + (size_t)16 * in;  // eight rows further
    const bf16 *x = reinterpret_cast<const bf16 *>(sh ? a.xs : a.x);
    const int pieces = in / 64;
    for (int tb = 0; tb < tile.z; tb += 8 * NT) {
        const uint4 *xr[NT];
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            const int j = tb + 8 * n + g;
            const int row = tile.y + j;
            xr[n] = j < tile.z ? reinterpret_cast<const uint4 *>(x + (size_t)(UP && !sh ? a.slot_tok[row] : row) * in + 16 * t) : nullptr;
        }
        float acc[NT][4] = {};
        u32x8 wa[DEPTH], wb[DEPTH];
        uint4 xa[DEPTH][NT], xb[DEPTH][NT];
        auto load = [&](int i, int p) {
            if (p < pieces) {
                wa[i] = ld_stream_256(w0 + (size_t)p * 128);
                wb[i] = ld_stream_256(w1 + (size_t)p * 128);
#pragma unroll
                for (int n = 0; n < NT; ++n) {
                    xa[i][n] = xr[n] ? xr[n][p * 8] : make_uint4(0, 0, 0, 0);
                    xb[i][n] = xr[n] ? xr[n][p * 8 + 1] : make_uint4(0, 0, 0, 0);
                }
            }
        };
#pragma unroll
        for (int i = 0; i < DEPTH; ++i) load(i, warp + MP_WARPS * i);
        for (int p = warp; p < pieces; p += MP_WARPS * DEPTH) {
#pragma unroll
            for (int i = 0; i < DEPTH; ++i) {
                if (p + MP_WARPS * i < pieces) {
#pragma unroll
                    for (int n = 0; n < NT; ++n) {
                        mma16816<bf16>(acc[n], wa[i].lo.x, wb[i].lo.x, wa[i].lo.y, wb[i].lo.y, xa[i][n].x, xa[i][n].y);
                        mma16816<bf16>(acc[n], wa[i].lo.z, wb[i].lo.z, wa[i].lo.w, wb[i].lo.w, xa[i][n].z, xa[i][n].w);
                        mma16816<bf16>(acc[n], wa[i].hi.x, wb[i].hi.x, wa[i].hi.y, wb[i].hi.y, xb[i][n].x, xb[i][n].y);
                        mma16816<bf16>(acc[n], wa[i].hi.z, wb[i].hi.z, wa[i].hi.w, wb[i].hi.w, xb[i][n].z, xb[i][n].w);
                    }
                }
                load(i, p + MP_WARPS * (i + DEPTH));
            }
        }
        if (tb) __syncthreads();  // the last pass has been read
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            red[warp][g][8 * n + 2 * t] = acc[n][0];
            red[warp][g][8 * n + 2 * t + 1] = acc[n][1];
            red[warp][g + 8][8 * n + 2 * t] = acc[n][2];
            red[warp][g + 8][8 * n + 2 * t + 1] = acc[n][3];
        }
        __syncthreads();
        auto sum = [&](int r, int c) {
            float v = 0.f;
#pragma unroll
            for (int i = 0; i < MP_WARPS; ++i) v += red[i][r][c];
            return v;
        };
        for (int i = tid; i < (UP ? 8 : 16) * 8 * NT; i += MP_WARPS * 32) {
            const int r = i % (UP ? 8 : 16), c = i / (UP ? 8 : 16);
            if (tb + c >= tile.z) continue;
            const int row = tile.y + tb + c;
            if constexpr (UP) {
                const float s = sh || !a.slot_w ? 1.f : a.slot_w[row];
                const float v = glu_act(s * sum(2 * r, c), s * sum(2 * r + 1, c), sh ? a.glus : a.glu);
                reinterpret_cast<bf16 *>(sh ? a.ys : a.y)[(size_t)row * (out / 2) + row0 / 2 + r] = Act<bf16>::from_f(v);
            } else {
                reinterpret_cast<float *>(sh ? a.ys : a.y)[(size_t)row * out + row0 + r] = sum(r, c);
            }
        }
    }
}
template <bool UP>
__global__ void __launch_bounds__(MP_WARPS * 32, 4) moe_product_kernel(const MoeProduct a) {
    __shared__ float red[MP_WARPS][16][MP_LD];
    grid_dep_launch();
    const bool sh = a.shared && blockIdx.y == 0;
    const int out = sh ? a.outs : a.out, in = sh ? a.ins : a.in, row0 = blockIdx.x * 16;
    if (row0 >= out) return;
    grid_dep_wait();
    const int4 tile = sh ? make_int4(0, 0, a.n_tok, 0) : a.tiles[(int)blockIdx.y - a.shared];
    if (tile.z == 0) return;
    if (tile.z <= 8) moe_rows<1, UP>(a, tile, sh, out, in, row0, red);
    else if (tile.z <= 16) moe_rows<2, UP>(a, tile, sh, out, in, row0, red);
    else moe_rows<4, UP>(a, tile, sh, out, in, row0, red);
}

}  // namespace

int moe_plan_launch(const MoeRoute &a, cudaStream_t s, bool pdl) {
    const size_t smem = (size_t)(3 * a.experts + 2 * a.n_tok * a.top) * 4;
    LCU_REQUIRE(a.n_tok <= MOE_SMALL_ROUND && smem <= 48 * 1024, "experts: %d tokens, %d experts, %d per token", a.n_tok, a.experts, a.top);
    LCU_CHECK_CUDA(launch_kernel(moe_plan_kernel, dim3(1), dim3(1024), smem, s, pdl, a));
    return LCU_OK;
}
int moe_route_launch(const MoeRoute &a, cudaStream_t s, bool pdl) {
    LCU_CHECK_CUDA(launch_kernel(moe_route_kernel, dim3((a.n_tok + 7) / 8), dim3(256), 0, s, pdl, a));
    return LCU_OK;
}
int moe_gather_launch(const MoeRoute &a, int dt, cudaStream_t s, bool pdl) {
    const size_t smem = (size_t)2 * a.experts * 4;
    if (dt == LCU_F32) LCU_CHECK_CUDA(launch_kernel(moe_gather_kernel<float>, dim3(a.n_tok), dim3(256), smem, s, pdl, a));
    else LCU_CHECK_CUDA(launch_kernel(moe_gather_kernel<bf16>, dim3(a.n_tok), dim3(256), smem, s, pdl, a));
    return LCU_OK;
}
int moe_product_launch(const MoeProduct &a, cudaStream_t s, bool pdl) {
    LCU_REQUIRE(a.in % 64 == 0 && a.out % 16 == 0 && (!a.shared || (a.ins % 64 == 0 && a.outs % 16 == 0)), "experts: product of %d x %d", a.out, a.in);
    const int rows = a.shared && a.outs > a.out ? a.outs : a.out;
    const dim3 grid(rows / 16, a.max_tiles + a.shared);
    auto go = [&](auto kernel) -> int {
        LCU_CHECK_CUDA(launch_kernel(kernel, grid, dim3(MP_WARPS * 32), 0, s, pdl, a));
        return LCU_OK;
    };
    return a.up ? go(moe_product_kernel<true>) : go(moe_product_kernel<false>);
}

}  // namespace lcu
