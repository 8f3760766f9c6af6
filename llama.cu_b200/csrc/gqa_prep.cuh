// The step between the fused input projection and softmax attention, one warp per (token, head): bias, rotation, norm; the
// query to its buffer, key and value to the cache.  Shared by the kernels of gqa.cu and the decode kernel of delta.cu.
#pragma once
#include "mixers.cuh"

namespace lcu {

__device__ __forceinline__ int gqa_prep_items(const GqaArgs &a) { return a.heads + 2 * a.kv_heads; }

template <class T>
__device__ __forceinline__ void gqa_prep_item(const GqaArgs &a, int t, int item, int lane) {
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
    float v[MIX_MAX_HEAD / 32];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 32; ++j) {
        const int d = lane + 32 * j;
        v[j] = 0.f;
        if (d >= size_p) continue;
        float x = src[d] + (bias ? bias[d] : 0.f);
        if (!is_v && d < a.rot_dims) {
            const int e = d < half ? d + half : d - half;
            const float y = src[e] + (bias ? bias[e] : 0.f);
            const float2 cs = rot[d < half ? d : e];
            x = d < half ? x * cs.x - y * cs.y : x * cs.x + y * cs.y;
        }
        v[j] = x;
        ss += x * x;
    }
    float r = 1.f;
    if (!is_v && a.qk_norm) r = 1.f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 32; ++j) {
        const int d = lane + 32 * j;
        if (d < size_p) {
            if constexpr (sizeof(T) == 4) dst[d] = v[j] * r;
            else dst[d] = Act<T>::from_f(v[j] * r);
        }
    }
}

}  // namespace lcu
