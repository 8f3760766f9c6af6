// Residual, norm and token-shift steps of layered models, and small row operations.
#include "stack.cuh"

namespace lcu {

// One block per token.  A token's shifted input needs the PREVIOUS token's new residual: the block computes that row as
// well (it may belong to another block of this launch, so it cannot be read), except at the start of a request, where it
// comes from the sequence's state.  The state is double-buffered by generation: the block of a request's first token reads
// one half, the block of its last token writes the other, so their order does not matter.  MAXV float4 values of each row
// per thread stay in registers between the two passes.
template <class T, int MAXV>
__global__ void mix_input_kernel(const MixInputArgs a) {
    grid_dep_launch();
    const int t = blockIdx.x;
    __shared__ float2 part[32];
    const int r = a.tok_req[t];
    const int first = a.req_first[r];
    const bool shifted = a.shift != nullptr;
    const bool at_start = t == first;
    const bool prev_row = shifted && !at_start;
    const int n4 = a.d_p / 4;
    grid_dep_wait();
    float4 x0[MAXV], x1[MAXV], y0[MAXV], y1[MAXV];
    float s0 = 0.f, s1 = 0.f;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const size_t row0 = (size_t)t * a.d_p, row1 = prev_row ? row0 - a.d_p : row0;
    const size_t e0 = a.embd ? (size_t)a.tokens[t] * a.d_p : 0, e1 = a.embd && prev_row ? (size_t)a.tokens[t - 1] * a.d_p : e0;
#pragma unroll
    for (int j = 0; j < MAXV; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        x0[j] = x1[j] = y0[j] = y1[j] = zero;
        if (i < n4) {
            if (a.embd) {
                x0[j] = ld4_bf16(a.embd, e0 + 4 * i);
                if (prev_row) x1[j] = ld4_bf16(a.embd, e1 + 4 * i);
            } else {
                x0[j] = *reinterpret_cast<const float4 *>(a.x_in + row0 + 4 * i);
                y0[j] = *reinterpret_cast<const float4 *>(a.y + row0 + 4 * i);
                s0 += dot4(y0[j]);
                if (prev_row) {
                    x1[j] = *reinterpret_cast<const float4 *>(a.x_in + row1 + 4 * i);
                    y1[j] = *reinterpret_cast<const float4 *>(a.y + row1 + 4 * i);
                    s1 += dot4(y1[j]);
                }
            }
        }
    }
    float r0 = 0.f, r1 = 0.f;
    if (!a.embd) {
        const float2 s = block_sum2(s0, s1, part);
        r0 = 1.f / sqrtf(s.x / (float)a.d + a.eps);
        r1 = 1.f / sqrtf(s.y / (float)a.d + a.eps);
    }
    const float *st_in = nullptr;
    float *st_out = nullptr;
    if (shifted) {
        const int sg = a.req_slot[r];
        const size_t off = (size_t)(sg >> 1) * a.d_p;
        if (at_start && a.req_pos[r] > 0) st_in = a.state + (size_t)(sg & 1) * a.state_gen_stride + off;
        if (t + 1 == a.req_first[r + 1]) st_out = a.state + (size_t)((sg & 1) ^ 1) * a.state_gen_stride + off;
    }
#pragma unroll
    for (int j = 0; j < MAXV; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i >= n4) continue;
        float4 v = x0[j], p = x1[j];
        if (!a.embd) {
            const float4 g = a.gain_stride ? *reinterpret_cast<const float4 *>(a.gain + 4 * i)
                                           : make_float4(a.gain[0], a.gain[0], a.gain[0], a.gain[0]);
            v.x += y0[j].x * r0 * g.x; v.y += y0[j].y * r0 * g.y; v.z += y0[j].z * r0 * g.z; v.w += y0[j].w * r0 * g.w;
            p.x += y1[j].x * r1 * g.x; p.y += y1[j].y * r1 * g.y; p.z += y1[j].z * r1 * g.z; p.w += y1[j].w * r1 * g.w;
        }
        if (a.x_out) *reinterpret_cast<float4 *>(a.x_out + row0 + 4 * i) = v;
        if (st_out) *reinterpret_cast<float4 *>(st_out + 4 * i) = v;
        if (!a.h) continue;
        if (shifted) {
            if (at_start) p = st_in ? *reinterpret_cast<const float4 *>(st_in + 4 * i) : zero;
            const float4 m = ld4_bf16(a.shift, 4 * i);
            v.x += (p.x - v.x) * m.x; v.y += (p.y - v.y) * m.y; v.z += (p.z - v.z) * m.z; v.w += (p.w - v.w) * m.w;
        }
        st4<T>(reinterpret_cast<T *>(a.h) + row0 + 4 * i, v);
    }
}

template <class T>
static int mix_input_t(const MixInputArgs &a, cudaStream_t s, bool pdl) {
    const int n4 = a.d_p / 4;
    if (n4 <= 128) LCU_CHECK_CUDA(launch_kernel(mix_input_kernel<T, 1>, dim3(a.n_tok), dim3(128), 0, s, pdl, a));
    else if (n4 <= 1024) LCU_CHECK_CUDA(launch_kernel(mix_input_kernel<T, 2>, dim3(a.n_tok), dim3(512), 0, s, pdl, a));
    else LCU_CHECK_CUDA(launch_kernel(mix_input_kernel<T, 4>, dim3(a.n_tok), dim3(1024), 0, s, pdl, a));
    return LCU_OK;
}

int op_mix_input(const MixInputArgs &a, int dt, cudaStream_t s, bool pdl) {
    if (a.n_tok <= 0) return LCU_OK;
    LCU_REQUIRE(a.d_p % 4 == 0 && a.d_p <= 16384, "mix_input: width %d (a multiple of 4, at most 16384)", a.d_p);
    return dt == LCU_F32 ? mix_input_t<float>(a, s, pdl) : mix_input_t<__nv_bfloat16>(a, s, pdl);
}

// Row of the pair table for token t: the previous token is in this round, or the last one of the sequence's state.
__device__ __forceinline__ size_t pair_row(const PreNormArgs &a, int t) {
    const int r = a.tok_req[t], sg = a.req_slot[r];
    const bool at_start = t == a.req_first[r];
    if (threadIdx.x == 0 && t + 1 == a.req_first[r + 1]) a.last_token[(size_t)((sg & 1) ^ 1) * a.last_gen_stride + (sg >> 1)] = a.tokens[t];
    if (at_start && a.req_pos[r] == 0) return (size_t)a.pair_buckets;
    const unsigned long long prev = at_start ? a.last_token[(size_t)(sg & 1) * a.last_gen_stride + (sg >> 1)] : a.tokens[t - 1];
    return (size_t)((prev * (unsigned)a.pair_prev + (unsigned long long)a.tokens[t] * (unsigned)a.pair_cur) % (unsigned)a.pair_buckets);
}

// One block per token: the residual step of pre-norm layers.  FORM 1 and 2: the outputs are one sum, of experts' rows too.  1: the
// sum may be normed; token pairs.  2: weights on experts' rows, experts that return their input, a bias, a second norm.
constexpr int pre_norm_threads(int maxv) { return maxv == 1 ? 128 : 256 * maxv; }
template <class T, int MAXV, int FORM>
__global__ void __launch_bounds__(pre_norm_threads(MAXV), FORM && MAXV == 2 ? 3 : 1) pre_norm_kernel(const PreNormArgs a) {
    constexpr bool POST = FORM > 0, PAIR = FORM == 2;
    grid_dep_launch();
    const int t = blockIdx.x, n4 = a.d_p / 4;
    __shared__ float2 part[32], part2[32];
    const size_t row = (size_t)t * a.d_p;
    grid_dep_wait();
    const size_t e0 = a.embd ? (size_t)a.tokens[t] * a.d_p : 0;  // fed-back tokens are written by the kernel before the round's first one
    const size_t e1 = FORM == 1 && a.pair_embd ? pair_row(a, t) * a.d_p : 0;
    if (POST && t == 0)
        for (int i = threadIdx.x; i < a.n_zero; i += blockDim.x) a.zero[i] = 0;
    float4 x[MAXV], y0[MAXV], y1[POST ? 1 : MAXV];
    float s0 = 0.f, s1 = 0.f;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < MAXV; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        float4 &u = y0[j], &v = y1[POST ? 0 : j];
        x[j] = u = v = zero;
        if (i >= n4) continue;
        if (a.x_in) x[j] = *reinterpret_cast<const float4 *>(a.x_in + row + 4 * i);
        if (a.y[0]) u = *reinterpret_cast<const float4 *>(a.y[0] + row + 4 * i);
        if (a.y[1]) v = *reinterpret_cast<const float4 *>(a.y[1] + row + 4 * i);
        if constexpr (POST) {
            u = make_float4(u.x * a.y_scale[0] + v.x * a.y_scale[1], u.y * a.y_scale[0] + v.y * a.y_scale[1], u.z * a.y_scale[0] + v.z * a.y_scale[1],
                            u.w * a.y_scale[0] + v.w * a.y_scale[1]);
#pragma unroll 2
            for (int k = 0; k < a.top; ++k) {
                const int slot = a.slot_of[t * a.top + k];
                const float4 e = !PAIR || slot >= 0 ? *reinterpret_cast<const float4 *>(a.ye + (size_t)slot * a.d_p + 4 * i)
                                                    : ld4<T>(reinterpret_cast<const T *>(a.ff_in) + row + 4 * i);
                const float w = PAIR && a.ye_w ? a.ye_w[t * a.top + k] : 1.f;
                u.x += e.x * w; u.y += e.y * w; u.z += e.z * w; u.w += e.w * w;
            }
            if (PAIR && a.y_bias) {
                const float4 e = *reinterpret_cast<const float4 *>(a.y_bias + 4 * i);
                u.x += e.x; u.y += e.y; u.z += e.z; u.w += e.w;
            }
        }
        s0 += dot4(u);
        if constexpr (!POST) s1 += dot4(v);
    }
    if (FORM == 2 ? false : FORM == 1 ? a.post_gain != nullptr : a.y_gain != nullptr) {
        const float2 s = block_sum2(s0, s1, part);
        s0 = 1.f / sqrtf(s.x / (float)a.d + a.eps);
        s1 = 1.f / sqrtf(s.y / (float)a.d + a.eps);
    }
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < MAXV; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i >= n4) continue;
        float4 v = x[j];
        const float4 one = make_float4(1.f, 1.f, 1.f, 1.f);
        if constexpr (PAIR) {
            v.x += y0[j].x; v.y += y0[j].y; v.z += y0[j].z; v.w += y0[j].w;
        } else if constexpr (POST) {
            const float4 g = a.post_gain ? *reinterpret_cast<const float4 *>(a.post_gain + 4 * i) : one;
            const float r = a.post_gain ? s0 : 1.f;
            v.x += y0[j].x * r * g.x; v.y += y0[j].y * r * g.y; v.z += y0[j].z * r * g.z; v.w += y0[j].w * r * g.w;
        } else {
            float4 g0 = one, g1 = one;
            if (a.y_gain) {
                g0 = *reinterpret_cast<const float4 *>(a.y_gain + 4 * i);
                g1 = *reinterpret_cast<const float4 *>(a.y_gain + a.d_p + 4 * i);
                g0.x *= s0; g0.y *= s0; g0.z *= s0; g0.w *= s0;
                g1.x *= s1; g1.y *= s1; g1.z *= s1; g1.w *= s1;
            }
            v.x += y0[j].x * g0.x + y1[j].x * g1.x; v.y += y0[j].y * g0.y + y1[j].y * g1.y;
            v.z += y0[j].z * g0.z + y1[j].z * g1.z; v.w += y0[j].w * g0.w + y1[j].w * g1.w;
        }
        if (a.embd) {
            const float4 e = ld4_bf16(a.embd, e0 + 4 * i);
            v.x += e.x * a.embd_scale; v.y += e.y * a.embd_scale; v.z += e.z * a.embd_scale; v.w += e.w * a.embd_scale;
        }
        if (FORM == 1 && a.pair_embd) {
            const float4 e = ld4_bf16(a.pair_embd, e1 + 4 * i);
            v.x += e.x; v.y += e.y; v.z += e.z; v.w += e.w;
        }
        if (a.step) {
            const float4 e = *reinterpret_cast<const float4 *>(a.step + 4 * i);
            v.x += e.x; v.y += e.y; v.z += e.z; v.w += e.w;
        }
        *reinterpret_cast<float4 *>(a.x_out + row + 4 * i) = v;
        x[j] = v;
        ss += dot4(v);
    }
    if (!a.h) return;
    const float r = 1.f / sqrtf(block_sum2(ss, 0.f, part2).x / (float)a.d + a.eps);
#pragma unroll
    for (int j = 0; j < MAXV; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i >= n4) continue;
        const float4 g = *reinterpret_cast<const float4 *>(a.gain + 4 * i), v = x[j];
        st4<T>(reinterpret_cast<T *>(a.h) + row + 4 * i, make_float4(v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w));
        if (PAIR && a.h2) {
            const float4 q = *reinterpret_cast<const float4 *>(a.gain2 + 4 * i);
            st4<T>(reinterpret_cast<T *>(a.h2) + row + 4 * i, make_float4(v.x * r * q.x, v.y * r * q.y, v.z * r * q.z, v.w * r * q.w));
        }
    }
}

template <class T, int FORM>
static int pre_norm_t(const PreNormArgs &a, cudaStream_t s, bool pdl) {
    const int n4 = a.d_p / 4;
    if (n4 <= 128) LCU_CHECK_CUDA(launch_kernel(pre_norm_kernel<T, 1, FORM>, dim3(a.n_tok), dim3(pre_norm_threads(1)), 0, s, pdl, a));
    else if (n4 <= 1024) LCU_CHECK_CUDA(launch_kernel(pre_norm_kernel<T, 2, FORM>, dim3(a.n_tok), dim3(pre_norm_threads(2)), 0, s, pdl, a));
    else LCU_CHECK_CUDA(launch_kernel(pre_norm_kernel<T, 4, FORM>, dim3(a.n_tok), dim3(pre_norm_threads(4)), 0, s, pdl, a));
    return LCU_OK;
}

int op_pre_norm(const PreNormArgs &a, int dt, cudaStream_t s, bool pdl) {
    if (a.n_tok <= 0) return LCU_OK;
    LCU_REQUIRE(a.d_p % 4 == 0 && a.d_p <= 16384, "pre_norm: width %d (a multiple of 4, at most 16384)", a.d_p);
    const bool post = a.post_gain || a.pair_embd || a.n_zero || a.top;
    LCU_REQUIRE(!post || !a.y_gain, "pre_norm: outputs normed one by one and as a sum");
    if (a.h2 || a.ye_w || a.y_bias) {
        LCU_REQUIRE(!a.post_gain && !a.pair_embd && !a.y_gain && (!a.h2 || a.h), "pre_norm: two norms ahead of sublayers, and norms on outputs or token pairs");
        return dt == LCU_F32 ? pre_norm_t<float, 2>(a, s, pdl) : pre_norm_t<__nv_bfloat16, 2>(a, s, pdl);
    }
    if (post) return dt == LCU_F32 ? pre_norm_t<float, 1>(a, s, pdl) : pre_norm_t<__nv_bfloat16, 1>(a, s, pdl);
    return dt == LCU_F32 ? pre_norm_t<float, 0>(a, s, pdl) : pre_norm_t<__nv_bfloat16, 0>(a, s, pdl);
}

// One block per token: a z / rms(z) + b z^2 / rms(z^2) + c z^3 / rms(z^3) + e, z = row + bias.  MAXV float4 values of the row per
// thread stay in registers between the passes; 0: any width, the row is read twice.
template <class T, int MAXV>
__global__ void __launch_bounds__(MAXV == 1 ? 128 : 512, MAXV == 1 ? 8 : (MAXV == 8 ? 2 : 3)) poly_norm_kernel(const PolyNormArgs a) {
    grid_dep_launch();
    __shared__ float2 part[32], part2[32];
    const int t = blockIdx.x, n4 = a.ff_p / 4;
    const float *z = a.z + (size_t)t * a.ff_p;
    const float k1 = a.act[0], k2 = a.act[1], k3 = a.act[2], k0 = a.act[3];
    grid_dep_wait();
    auto load = [&](int i) {
        float4 v = *reinterpret_cast<const float4 *>(z + 4 * i);
        if (a.bias) {
            const float4 b = *reinterpret_cast<const float4 *>(a.bias + 4 * i);
            v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
        }
        return v;
    };
    float s1 = 0.f, s2 = 0.f, s3 = 0.f;
    auto count = [&](const float4 &v) {  // padding is zero
        const float4 q = make_float4(v.x * v.x, v.y * v.y, v.z * v.z, v.w * v.w);
        s1 += q.x + q.y + q.z + q.w;
        s2 += dot4(q);
        s3 += q.x * q.x * q.x + q.y * q.y * q.y + q.z * q.z * q.z + q.w * q.w * q.w;
    };
    float4 x[MAXV ? MAXV : 1];
    if constexpr (MAXV > 0) {
#pragma unroll
        for (int j = 0; j < MAXV; ++j) {
            const int i = threadIdx.x + j * blockDim.x;
            x[j] = i < n4 ? load(i) : make_float4(0.f, 0.f, 0.f, 0.f);
            count(x[j]);
        }
    } else {
        for (int i = threadIdx.x; i < n4; i += blockDim.x) count(load(i));
    }
    const float2 s = block_sum2(s1, s2, part);
    s3 = block_sum2(s3, 0.f, part2).x;
    const float n = (float)a.ff, r1 = k1 / sqrtf(s.x / n + a.eps), r2 = k2 / sqrtf(s.y / n + a.eps), r3 = k3 / sqrtf(s3 / n + a.eps);
    auto act = [&](float v, int i) { return i < a.ff ? fmaf(v, fmaf(v, fmaf(v, r3, r2), r1), k0) : 0.f; };
    auto put = [&](const float4 &v, int i) {
        st4<T>(reinterpret_cast<T *>(a.y) + (size_t)t * a.ff_p + 4 * i, make_float4(act(v.x, 4 * i), act(v.y, 4 * i + 1), act(v.z, 4 * i + 2), act(v.w, 4 * i + 3)));
    };
    if constexpr (MAXV > 0) {
#pragma unroll
        for (int j = 0; j < MAXV; ++j) {
            const int i = threadIdx.x + j * blockDim.x;
            if (i < n4) put(x[j], i);
        }
    } else {
        for (int i = threadIdx.x; i < n4; i += blockDim.x) put(load(i), i);
    }
}

int op_poly_norm(const PolyNormArgs &a, int dt, cudaStream_t s, bool pdl) {
    if (a.n_tok <= 0) return LCU_OK;
    LCU_REQUIRE(a.ff_p % 4 == 0 && a.ff > 0 && a.ff <= a.ff_p, "poly_norm: width %d padded to %d", a.ff, a.ff_p);
    const int n4 = a.ff_p / 4;
    auto go = [&](auto kernel, int threads) -> int {
        LCU_CHECK_CUDA(launch_kernel(kernel, dim3(a.n_tok), dim3(threads), 0, s, pdl, a));
        return LCU_OK;
    };
    auto by_width = [&](auto t) -> int {
        using T = decltype(t);
        if (n4 <= 128) return go(poly_norm_kernel<T, 1>, 128);
        if (n4 <= 1024) return go(poly_norm_kernel<T, 2>, 512);
        if (n4 <= 2048) return go(poly_norm_kernel<T, 4>, 512);
        if (n4 <= 4096) return go(poly_norm_kernel<T, 8>, 512);
        return go(poly_norm_kernel<T, 0>, 512);
    };
    return dt == LCU_F32 ? by_width(float{}) : by_width(__nv_bfloat16{});
}

template <class T>
__global__ void __launch_bounds__(256) scalar_norm_rows_kernel(T *__restrict__ y, const float *__restrict__ x, const uint32_t *__restrict__ rows,
                                                               int d, int d_p, const float *__restrict__ gain, int gain_stride, float eps) {
    grid_dep_launch();
    __shared__ float2 part[32];
    grid_dep_wait();
    const float *xr = x + (size_t)rows[blockIdx.x] * d_p;
    float ss = 0.f;
    for (int i = threadIdx.x; i < d_p / 4; i += blockDim.x) ss += dot4(reinterpret_cast<const float4 *>(xr)[i]);
    const float r = 1.f / sqrtf(block_sum2(ss, 0.f, part).x / (float)d + eps);
    for (int i = threadIdx.x; i < d_p / 4; i += blockDim.x) {
        float4 v = reinterpret_cast<const float4 *>(xr)[i];
        const float4 g = gain_stride ? reinterpret_cast<const float4 *>(gain)[i] : make_float4(gain[0], gain[0], gain[0], gain[0]);
        v.x *= r * g.x; v.y *= r * g.y; v.z *= r * g.z; v.w *= r * g.w;
        st4<T>(y + (size_t)blockIdx.x * d_p + 4 * i, v);
    }
}

int op_scalar_norm_rows(void *y, const float *x, const uint32_t *rows, int n, int d, int d_p, const float *gain, int gain_stride, float eps,
                        int dt, cudaStream_t s, bool pdl) {
    if (n <= 0) return LCU_OK;
    if (dt == LCU_F32)
        LCU_CHECK_CUDA(launch_kernel(scalar_norm_rows_kernel<float>, dim3(n), dim3(256), 0, s, pdl, (float *)y, x, rows, d, d_p, gain, gain_stride, eps));
    else
        LCU_CHECK_CUDA(launch_kernel(scalar_norm_rows_kernel<__nv_bfloat16>, dim3(n), dim3(256), 0, s, pdl, (__nv_bfloat16 *)y, x, rows, d, d_p,
                                     gain, gain_stride, eps));
    return LCU_OK;
}

template <class T>
__global__ void rows_to_f32_kernel(float *__restrict__ dst, const T *__restrict__ src, size_t n) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) dst[i] = Act<T>::to_f(src[i]);
}

int op_rows_to_f32(float *dst, const void *src, size_t n, int dt, cudaStream_t s) {
    if (!n) return LCU_OK;
    const unsigned grid = (unsigned)((n + 255) / 256);
    if (dt == LCU_F16) rows_to_f32_kernel<__half><<<grid, 256, 0, s>>>(dst, (const __half *)src, n);
    else rows_to_f32_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(dst, (const __nv_bfloat16 *)src, n);
    LCU_CHECK_CUDA(cudaGetLastError());
    return LCU_OK;
}

}  // namespace lcu
