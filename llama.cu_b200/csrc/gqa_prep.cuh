// The step between the fused input projection and softmax attention, one warp per (token, head): bias, rotation, norm; the
// query to its buffer, key and value to the cache.  Shared by the kernels of gqa.cu and the decode kernel of delta.cu.
#pragma once
#include "stack.cuh"

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
    auto load4 = [&](int d) {
        float4 x = *reinterpret_cast<const float4 *>(src + d);
        if (bias) {
            const float4 y = *reinterpret_cast<const float4 *>(bias + d);
            x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
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
        float4 x = load4(d);
        if (!is_v && d < a.rot_dims) {
            if (half % 4 == 0) {  // four pairs: the partners are four consecutive dimensions too
                const bool lower = d < half;
                const int e = lower ? d + half : d - half;
                const float4 y = load4(e), c0 = *reinterpret_cast<const float4 *>(rot + (lower ? d : e)), c1 = *reinterpret_cast<const float4 *>(rot + (lower ? d : e) + 2);
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
                    const float y = src[e] + (bias ? bias[e] : 0.f);
                    const float2 cs = rot[i < half ? i : e];
                    xs[k] = i < half ? xs[k] * cs.x - y * cs.y : xs[k] * cs.x + y * cs.y;
                }
            }
        }
        v[j] = x;
        ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    }
    float r = 1.f;
    if (!is_v && a.qk_norm) r = 1.f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 128; ++j) {
        const int d = 4 * lane + 128 * j;
        if (d < size_p) st4<T>(dst + d, make_float4(v[j].x * r, v[j].y * r, v[j].z * r, v[j].w * r));
    }
}

}  // namespace lcu
