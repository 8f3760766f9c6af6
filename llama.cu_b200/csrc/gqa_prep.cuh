// The step between the fused input projection and softmax attention, one warp per (token, head): bias, norm, rotation; the
// query to its buffer, key and value to the cache.  Shared by the kernels of gqa.cu and the decode kernels of the recurrent mixers.
#pragma once
#include "stack.cuh"

namespace lcu {

__host__ __device__ __forceinline__ int gqa_prep_items(const GqaArgs &a) { return a.heads + (a.own_kv ? 2 * a.kv_heads : 0); }

// Steps that only some designs have, kept out of the kernels of the others: norms with weights ahead of the rotation, neighbouring pairs.
__host__ __device__ __forceinline__ bool gqa_prep_wide(const GqaArgs &a) { return a.qk_norm > 1 || a.rot_adjacent; }

// row_norm: what qk_norm 3 divides all of q and all of k by (as factors)
template <class T, bool WIDE>
__device__ __forceinline__ void gqa_prep_item(const GqaArgs &a, int t, int item, int lane, const float2 &row_norm) {
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
    auto raw4 = [&](int d) {
        float4 x = *reinterpret_cast<const float4 *>(src + d);
        if (bias) {
            const float4 y = *reinterpret_cast<const float4 *>(bias + d);
            x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
        }
        return x;
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
                    const float y = (src[e] + (bias ? bias[e] : 0.f)) * (WIDE && gain ? gain[e] : 1.f);
                    const float2 cs = rot[i < half ? i : e];
                    xs[k] = i < half ? xs[k] * cs.x - y * cs.y : xs[k] * cs.x + y * cs.y;
                }
            }
        }
        v[j] = x;
        ss += dot4(WIDE && a.qk_norm == 2 ? in : x);
    }
    float r = 1.f;
    if (!is_v && (a.qk_norm == 1 || (WIDE && a.qk_norm == 2))) r = 1.f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
    if (WIDE && !is_v && a.qk_norm == 3) r = is_q ? row_norm.x : row_norm.y;
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 128; ++j) {
        const int d = 4 * lane + 128 * j;
        if (d < size_p) st4<T>(dst + d, make_float4(v[j].x * r, v[j].y * r, v[j].z * r, v[j].w * r));
    }
}

// Items [item0, item1) of token t by one block (at most one per warp unless WIDE); every thread of the block calls it.
template <class T, bool WIDE>
__device__ __forceinline__ void gqa_prep_block(const GqaArgs &a, int t, int item0, int item1) {
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
        for (; item < item1; item += (int)(blockDim.x >> 5)) gqa_prep_item<T, true>(a, t, item, threadIdx.x & 31, norm);
    } else {
        if (item < item1) gqa_prep_item<T, false>(a, t, item, threadIdx.x & 31, norm);
    }
}

template <class T>
__device__ __forceinline__ void gqa_prep_any(const GqaArgs &a, int t, int item0, int item1) {
    if (gqa_prep_wide(a)) gqa_prep_block<T, true>(a, t, item0, item1);
    else gqa_prep_block<T, false>(a, t, item0, item1);
}

}  // namespace lcu
