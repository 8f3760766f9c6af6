// The step between the fused input projection and softmax attention, one warp per (token, head): bias or convolution over time,
// norm, rotation; the query to its buffer, key and value to the cache.  Shared by the kernels of gqa.cu and the decode kernels of the recurrent mixers.
#pragma once
#include "conv.cuh"
#include "stack.cuh"

namespace lcu {

__host__ __device__ __forceinline__ int gqa_prep_items(const GqaArgs &a) { return a.heads + (a.own_kv ? 2 * a.kv_heads : 0); }

// Steps that only some designs have, kept out of the kernels of the others: norms with weights ahead of the rotation, neighbouring pairs.
__host__ __device__ __forceinline__ bool gqa_prep_wide(const GqaArgs &a) { return a.qk_norm > 1 || a.rot_adjacent; }
// ... and only layers without a recurrent mixer: rotated values, factors per head; convolutions.
enum GqaPrepForm { GQA_PREP = 0, GQA_PREP_WIDE = 1, GQA_PREP_TURN = 2, GQA_PREP_CONV = 3 };
__host__ __device__ __forceinline__ bool gqa_prep_more(const GqaArgs &a) { return a.vrot || a.head_temp || a.conv; }

// row_norm: what qk_norm 3 divides all of q and all of k by (as factors)
template <class T, int FORM>
__device__ __forceinline__ void gqa_prep_item(const GqaArgs &a, int t, int item, int lane, const float2 &row_norm) {
    constexpr bool WIDE = FORM >= GQA_PREP_WIDE, TURN = FORM >= GQA_PREP_TURN, CONV = FORM == GQA_PREP_CONV;
    const bool is_v = item >= a.heads + a.kv_heads, is_q = item < a.heads;
    const int size_p = is_v ? a.vdim_p : a.dim_p;
    const int head = is_q ? item : (is_v ? item - a.heads - a.kv_heads : item - a.heads);
    const int off = is_q ? head * a.dim_p : (is_v ? (a.heads + a.kv_heads) * a.dim_p + head * a.vdim_p : (a.heads + head) * a.dim_p);
    const float *src = a.lat + (size_t)t * a.stride + off, *bias = a.bias ? a.bias + off : nullptr;
    const uint32_t p = a.pos[t];
    T *dst;
    if (is_q) dst = reinterpret_cast<T *>(a.q) + ((size_t)t * a.heads + head) * a.dim_p;
    else {
        const int page = a.page_table[(size_t)a.tok_req[t] * a.pt_stride + (p >> a.page_shift)];
        const size_t row = ((size_t)head << a.page_shift) + (p & ((1u << a.page_shift) - 1));
        dst = reinterpret_cast<T *>(a.pool) + (size_t)page * a.page_elems + (is_v ? a.v_off() : a.c_off) + row * size_p;
    }
    const int half = a.rot_dims >> 1;
    const float2 *rot = a.rot + (size_t)p * half;
    // A norm ahead of the rotation: its weights go in here, its one factor at the end (the rotation is linear).
    const float *gain = WIDE && !is_v && a.qk_norm > 1 ? a.qk_gain + (a.qk_norm == 3 ? off : (is_q ? 0 : a.dim_p)) : nullptr;
    [[maybe_unused]] ConvIn in_time;
    [[maybe_unused]] float *state_out = nullptr;
    if constexpr (CONV) {
        const int r = a.tok_req[t], sg = a.req_slot[r];
        const size_t row = (size_t)(sg >> 1) * (a.taps - 1) * a.channels();
        in_time.row = a.lat + (size_t)t * a.stride;
        in_time.stride = a.stride; in_time.channels = a.channels(); in_time.taps = a.taps;
        in_time.in_portion = t - a.req_first[r];
        in_time.seen = (int)p;
        in_time.state = a.conv_state + (size_t)(sg & 1) * a.conv_gen_stride + row;
        if (t + 1 == a.req_first[r + 1]) state_out = a.conv_state + (size_t)((sg & 1) ^ 1) * a.conv_gen_stride + row;
    }
    auto raw4 = [&](int d) {
        if constexpr (CONV) {
            float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
            for (int j = 0; j < a.taps; ++j) {
                const float4 x = in_time.at4(a.taps - 1 - j, off + d), w = *reinterpret_cast<const float4 *>(a.conv + (size_t)j * in_time.channels + off + d);
                y.x = fmaf(x.x, w.x, y.x); y.y = fmaf(x.y, w.y, y.y); y.z = fmaf(x.z, w.z, y.z); y.w = fmaf(x.w, w.w, y.w);
            }
            return y;
        }
        float4 x = *reinterpret_cast<const float4 *>(src + d);
        if (bias) {
            const float4 y = *reinterpret_cast<const float4 *>(bias + d);
            x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
        }
        return x;
    };
    auto raw1 = [&](int d) {
        if constexpr (CONV) {
            float y = 0.f;
            for (int j = 0; j < a.taps; ++j) y = fmaf(in_time.at(a.taps - 1 - j, off + d), a.conv[(size_t)j * in_time.channels + off + d], y);
            return y;
        }
        return src[d] + (bias ? bias[d] : 0.f);
    };
    auto weigh4 = [&](float4 x, int d) {
        if (WIDE && gain) {
            const float4 g = *reinterpret_cast<const float4 *>(gain + d);
            x.x *= g.x; x.y *= g.y; x.z *= g.z; x.w *= g.w;
        }
        return x;
    };
    float4 v[MIX_MAX_HEAD / 128];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 128; ++j) {
        const int d = 4 * lane + 128 * j;
        v[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (d >= size_p) continue;
        const float4 in = raw4(d);
        float4 x = weigh4(in, d);
        if (!is_v && d < a.rot_dims) {
            if (WIDE && a.rot_adjacent) {  // two pairs
                const float2 c0 = rot[d >> 1], c1 = d + 2 < a.rot_dims ? rot[(d >> 1) + 1] : make_float2(1.f, 0.f);
                x = make_float4(x.x * c0.x - x.y * c0.y, x.y * c0.x + x.x * c0.y, x.z * c1.x - x.w * c1.y, x.w * c1.x + x.z * c1.y);
            } else if (half % 4 == 0) {  // four pairs: the partners are four consecutive dimensions too
                const bool lower = d < half;
                const int e = lower ? d + half : d - half;
                const float4 y = weigh4(raw4(e), e), c0 = *reinterpret_cast<const float4 *>(rot + (lower ? d : e)), c1 = *reinterpret_cast<const float4 *>(rot + (lower ? d : e) + 2);
                const float sgn = lower ? -1.f : 1.f;
                x.x = x.x * c0.x + sgn * y.x * c0.y; x.y = x.y * c0.z + sgn * y.y * c0.w;
                x.z = x.z * c1.x + sgn * y.z * c1.y; x.w = x.w * c1.z + sgn * y.w * c1.w;
            } else {
                float *xs = reinterpret_cast<float *>(&x);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const int i = d + k;
                    if (i >= a.rot_dims) continue;
                    const int e = i < half ? i + half : i - half;
                    const float y = raw1(e) * (WIDE && gain ? gain[e] : 1.f);
                    const float2 cs = rot[i < half ? i : e];
                    xs[k] = i < half ? xs[k] * cs.x - y * cs.y : xs[k] * cs.x + y * cs.y;
                }
            }
        }
        if (TURN && is_v && a.vrot && d < a.v_dim) {  // two pairs
            const float2 *vr = a.vrot + (size_t)p * (a.v_dim >> 1) + (d >> 1);
            const float2 c0 = vr[0], c1 = d + 2 < a.v_dim ? vr[1] : make_float2(1.f, 0.f);
            x = make_float4(x.x * c0.x - x.y * c0.y, x.y * c0.x + x.x * c0.y, x.z * c1.x - x.w * c1.y, x.w * c1.x + x.z * c1.y);
        }
        v[j] = x;
        ss += dot4(WIDE && a.qk_norm == 2 ? in : x);
    }
    float r = 1.f;
    if (!is_v && (a.qk_norm == 1 || (WIDE && a.qk_norm == 2))) r = 1.f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
    if (WIDE && !is_v && a.qk_norm == 3) r = is_q ? row_norm.x : row_norm.y;
    if (TURN && is_q && a.head_temp) r *= a.head_temp[head];
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 128; ++j) {
        const int d = 4 * lane + 128 * j;
        if (d < size_p) st4<T>(dst + d, make_float4(v[j].x * r, v[j].y * r, v[j].z * r, v[j].w * r));
        if constexpr (CONV) {
            if (state_out && d < size_p)
                for (int i = 1; i < a.taps; ++i) *reinterpret_cast<float4 *>(state_out + (size_t)(i - 1) * in_time.channels + off + d) = in_time.at4(a.taps - 1 - i, off + d);
        }
    }
}

// Items [item0, item1) of token t by one block (at most one per warp unless WIDE); every thread of the block calls it.
template <class T, int FORM>
__device__ __forceinline__ void gqa_prep_block(const GqaArgs &a, int t, int item0, int item1) {
    constexpr bool WIDE = FORM >= GQA_PREP_WIDE;
    float2 norm = make_float2(1.f, 1.f);
    if (WIDE && a.qk_norm == 3) {
        __shared__ float2 part[32];
        const int nq = a.heads * a.dim_p, n = nq + (a.own_kv ? a.kv_heads * a.dim_p : 0);
        const float *src = a.lat + (size_t)t * a.stride;
        float2 ss = make_float2(0.f, 0.f);
#pragma unroll 2
        for (int d = 4 * threadIdx.x; d < n; d += 4 * blockDim.x) {
            float4 x = *reinterpret_cast<const float4 *>(src + d);
            if (a.bias) {
                const float4 y = *reinterpret_cast<const float4 *>(a.bias + d);
                x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
            }
            (d < nq ? ss.x : ss.y) += dot4(x);
        }
        ss = block_sum2(ss.x, ss.y, part);
        norm.x = 1.f / sqrtf(ss.x / (float)(a.heads * a.dim) + a.eps);
        norm.y = 1.f / sqrtf(ss.y / (float)(a.kv_heads * a.dim) + a.eps);
    }
    item1 = min(item1, gqa_prep_items(a));
    int item = item0 + (int)(threadIdx.x >> 5);
    if constexpr (WIDE) {
#pragma unroll 1
        for (; item < item1; item += (int)(blockDim.x >> 5)) gqa_prep_item<T, FORM>(a, t, item, threadIdx.x & 31, norm);
    } else {
        if (item < item1) gqa_prep_item<T, FORM>(a, t, item, threadIdx.x & 31, norm);
    }
}

// Layers with these steps alone: rotation of neighbouring pairs, rotated values, factors per head, convolutions of
// at most four taps.  A warp takes one head of RUN tokens in a row and holds the rows its convolution needs; every row is requested
// before the first is used.  TAPS 0: no convolution.
__host__ __device__ __forceinline__ bool gqa_prep_runs(const GqaArgs &a) {
    return !a.bias && !a.qk_norm && (a.rot_dims == 0 || a.rot_adjacent) && (!a.conv || a.taps <= 4);
}
template <class T, int TAPS, int RUN>
__device__ __forceinline__ void gqa_prep_run(const GqaArgs &a, int t0, int item, int lane) {
    constexpr int BACK = TAPS > 1 ? TAPS - 1 : 0;
    const bool is_v = item >= a.heads + a.kv_heads, is_q = item < a.heads;
    const int size_p = is_v ? a.vdim_p : a.dim_p;
    const int head = is_q ? item : (is_v ? item - a.heads - a.kv_heads : item - a.heads);
    const int off = is_q ? head * a.dim_p : (is_v ? (a.heads + a.kv_heads) * a.dim_p + head * a.vdim_p : (a.heads + head) * a.dim_p);
    const float2 *rot = is_v ? a.vrot : a.rot;
    const int turned = is_v ? (a.vrot ? a.v_dim : 0) : a.rot_dims;
    const float temp = is_q && a.head_temp ? a.head_temp[head] : 1.f;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int d = 4 * lane; d < size_p; d += 128) {
        float4 x[BACK + RUN], w[TAPS ? TAPS : 1];
#pragma unroll
        for (int i = 0; i < BACK + RUN; ++i) {
            const int t = t0 + i - BACK;
            x[i] = t >= 0 && t < a.n_tok ? *reinterpret_cast<const float4 *>(a.lat + (size_t)t * a.stride + off + d) : zero;
        }
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = *reinterpret_cast<const float4 *>(a.conv + (size_t)j * a.channels() + off + d);
#pragma unroll
        for (int i = 0; i < RUN; ++i) {
            const int t = t0 + i;
            if (t >= a.n_tok) break;
            const int p = (int)a.pos[t], r = a.tok_req[t];
            float4 y = x[BACK + i];
            if constexpr (TAPS > 0) {
                const int before = t - a.req_first[r];  // tokens of the portion before this one
                float4 u[TAPS];                         // inputs of the taps
#pragma unroll
                for (int j = 0; j < TAPS; ++j) u[j] = x[i + j];
                const bool last = TAPS > 1 && t + 1 == a.req_first[r + 1];
                if (TAPS > 1 && (before < BACK || last)) {
                    const int sg = a.req_slot[r];
                    const size_t row = (size_t)(sg >> 1) * BACK * a.channels() + off + d;
                    const float *in = a.conv_state + (size_t)(sg & 1) * a.conv_gen_stride + row;
                    float *out = a.conv_state + (size_t)((sg & 1) ^ 1) * a.conv_gen_stride + row;
#pragma unroll
                    for (int j = 0; j < BACK; ++j) {
                        const int back = BACK - j;
                        if (back > before) u[j] = back > p ? zero : *reinterpret_cast<const float4 *>(in + (size_t)(before + j) * a.channels());
                    }
                    if (last)
#pragma unroll
                        for (int j = 0; j < BACK; ++j) *reinterpret_cast<float4 *>(out + (size_t)j * a.channels()) = u[j + 1];
                }
                y = zero;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) {
                    y.x = fmaf(u[j].x, w[j].x, y.x); y.y = fmaf(u[j].y, w[j].y, y.y);
                    y.z = fmaf(u[j].z, w[j].z, y.z); y.w = fmaf(u[j].w, w[j].w, y.w);
                }
            }
            if (d < turned) {  // two pairs
                const float2 *cs = rot + (size_t)p * (turned >> 1) + (d >> 1);
                const float2 c0 = cs[0], c1 = d + 2 < turned ? cs[1] : make_float2(1.f, 0.f);
                y = make_float4(y.x * c0.x - y.y * c0.y, y.y * c0.x + y.x * c0.y, y.z * c1.x - y.w * c1.y, y.w * c1.x + y.z * c1.y);
            }
            T *dst;
            if (is_q) dst = reinterpret_cast<T *>(a.q) + ((size_t)t * a.heads + head) * a.dim_p;
            else {
                const int page = a.page_table[(size_t)r * a.pt_stride + (p >> a.page_shift)];
                const size_t row = ((size_t)head << a.page_shift) + (p & ((1 << a.page_shift) - 1));
                dst = reinterpret_cast<T *>(a.pool) + (size_t)page * a.page_elems + (is_v ? a.v_off() : a.c_off) + row * size_p;
            }
            st4<T>(dst + d, make_float4(y.x * temp, y.y * temp, y.z * temp, y.w * temp));
        }
    }
}

template <class T>
__device__ __forceinline__ void gqa_prep_any(const GqaArgs &a, int t, int item0, int item1) {
    if (gqa_prep_wide(a)) gqa_prep_block<T, GQA_PREP_WIDE>(a, t, item0, item1);
    else gqa_prep_block<T, GQA_PREP>(a, t, item0, item1);
}

}  // namespace lcu
