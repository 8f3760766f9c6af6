// What the kernels of the recurrent mixers share: short convolutions with their state, f32 numbers as sums of bf16 ones, and the
// legacy tensor-core products of 8 x 8 tiles.
#pragma once
#include "conv.cuh"
#include "gqa_prep.cuh"
#include "stack.cuh"

namespace lcu {

typedef __nv_bfloat16 bf16;

// Two f32 numbers as sums of three bf16 ones (24 bits): planes[0] + planes[1] + planes[2], two numbers per word.
__device__ __forceinline__ void split3(float x, float y, uint32_t planes[3]) {
#pragma unroll
    for (int i = 0; i < 3; ++i) {
        planes[i] = Act<bf16>::pack(x, y);
        const float2 v = Act<bf16>::to_f2(planes[i]);
        x -= v.x;
        y -= v.y;
    }
}
__device__ __forceinline__ void store_split4(void *row, int dk, int d, const float4 &v) {  // row: [3][dk] bf16
    uint32_t a[3], b[3];
    split3(v.x, v.y, a);
    split3(v.z, v.w, b);
#pragma unroll
    for (int i = 0; i < 3; ++i) *reinterpret_cast<uint2 *>(reinterpret_cast<bf16 *>(row) + (size_t)i * dk + d) = make_uint2(a[i], b[i]);
}

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_of(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float octet_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    return v + __shfl_xor_sync(0xffffffffu, v, 4);
}

__device__ __forceinline__ ConvIn conv_in(const DeltaArgs &a, int t, int r) {
    ConvIn c;
    const int sg = a.req_slot[r];
    c.row = a.lat + (size_t)t * a.stride;
    c.stride = a.stride; c.channels = a.channels(); c.taps = a.taps;
    c.in_portion = t - a.req_first[r];
    c.seen = a.req_pos[r] + c.in_portion;
    c.state = a.conv_state + (size_t)(sg & 1) * a.conv_gen_stride + (size_t)(sg >> 1) * (a.taps - 1) * c.channels;
    return c;
}
__device__ __forceinline__ float *conv_out(const DeltaArgs &a, int r) {
    const int sg = a.req_slot[r];
    return a.conv_state + (size_t)((sg & 1) ^ 1) * a.conv_gen_stride + (size_t)(sg >> 1) * (a.taps - 1) * a.channels();
}
// convolution and activation of one channel; `out`: state to leave behind (the request's last token), or nullptr
__device__ __forceinline__ float conv_silu(const DeltaArgs &a, const ConvIn &in, int c, float *out) {
    float y = a.conv_bias ? a.conv_bias[c] : 0.f;
#pragma unroll 4
    for (int j = 0; j < a.taps; ++j) y = fmaf(in.at(a.taps - 1 - j, c), a.conv[(size_t)j * in.channels + c], y);
    if (out)  // after all loads: stores in between would hold them up
#pragma unroll 4
        for (int j = 1; j < a.taps; ++j) out[(size_t)(j - 1) * in.channels + c] = in.at(a.taps - 1 - j, c);
    return silu_f(y);
}

constexpr int CONV_BLOCK = 8;  // tokens conv_block takes
// Convolution and activation of four channels for the tokens of a block, put(token, values); tokens past `count` give zero.
// Every input is requested before the first is used.
__device__ __forceinline__ float4 fma4(const float4 &x, const float4 &w, const float4 &y) {
    return make_float4(fmaf(x.x, w.x, y.x), fmaf(x.y, w.y, y.y), fmaf(x.z, w.z, y.z), fmaf(x.w, w.w, y.w));
}
template <int TAPS, class F>
__device__ __forceinline__ void conv_block(const DeltaArgs &a, const ConvIn &in, int c, int count, float *out, const F &put) {
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), bias = a.conv_bias ? *reinterpret_cast<const float4 *>(a.conv_bias + c) : zero;
    if constexpr (TAPS > 0) {
        float4 w[TAPS], x[TAPS - 1 + CONV_BLOCK];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = __ldg(reinterpret_cast<const float4 *>(a.conv + (size_t)j * in.channels + c));
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) x[j] = in.at4(TAPS - 1 - j, c);
#pragma unroll
        for (int i = 0; i < CONV_BLOCK; ++i) x[TAPS - 1 + i] = i < count ? *reinterpret_cast<const float4 *>(in.row + c + (size_t)i * in.stride) : zero;
#pragma unroll
        for (int i = 0; i < CONV_BLOCK; ++i) {
            float4 y = bias;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) y = fma4(x[i + j], w[j], y);
            put(i, i < count ? make_float4(silu_f(y.x), silu_f(y.y), silu_f(y.z), silu_f(y.w)) : zero);
            if (out && i + 1 == count)
#pragma unroll
                for (int j = 1; j < TAPS; ++j) *reinterpret_cast<float4 *>(out + (size_t)(j - 1) * in.channels + c) = x[i + j];
        }
    } else {
        ConvIn t = in;
        for (int i = 0; i < CONV_BLOCK; ++i) {
            float4 y = bias;
            for (int j = 0; j < a.taps && i < count; ++j) {
                const float4 x = t.at4(a.taps - 1 - j, c);
                y = fma4(x, *reinterpret_cast<const float4 *>(a.conv + (size_t)j * in.channels + c), y);
                if (out && i + 1 == count && j > 0) *reinterpret_cast<float4 *>(out + (size_t)(j - 1) * in.channels + c) = x;
            }
            put(i, i < count ? make_float4(silu_f(y.x), silu_f(y.y), silu_f(y.z), silu_f(y.w)) : zero);
            t.row += t.stride; ++t.in_portion; ++t.seen;
        }
    }
}

__device__ __forceinline__ void dt_mma16(float c[4], const uint32_t a[2], const uint32_t a2[2], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a2[0]), "r"(a2[1]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void dt_mma8(float c[4], const uint32_t a[2], uint32_t b) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5}, {%6}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(b));
}
// accumulator -> first operand (rows g and g + 8, columns 2 t and 2 t + 1), split: [plane][row half]
__device__ __forceinline__ void dt_operand(const float c[4], uint32_t a[3][2]) {
    uint32_t x[3], y[3];
    split3(c[0], c[1], x);
    split3(c[2], c[3], y);
#pragma unroll
    for (int i = 0; i < 3; ++i) { a[i][0] = x[i]; a[i][1] = y[i]; }
}
__device__ __forceinline__ void dt_mma8x6(float c[4], const uint32_t a[3][2], const uint32_t b[3]) {  // smallest products first
    dt_mma8(c, a[1], b[1]);
    dt_mma8(c, a[0], b[2]);
    dt_mma8(c, a[2], b[0]);
    dt_mma8(c, a[0], b[1]);
    dt_mma8(c, a[1], b[0]);
    dt_mma8(c, a[0], b[0]);
}
// tiles [0, KW) of 8 x 8 at `row` (this lane's row of a tile), 16 bytes apart
template <int KW, bool TRANS>
__device__ __forceinline__ void dt_tiles(uint32_t *dst, const unsigned char *row, int lane) {
#pragma unroll
    for (int k = 0; k < KW; k += 4) {
        const int tile = min(k + (lane >> 3), KW - 1);
        const unsigned at = (unsigned)__cvta_generic_to_shared(row + tile * 16);
        uint32_t r[4];
        if constexpr (TRANS) asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at));
        else asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at));
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (k + i < KW) dst[k + i] = r[i];
    }
}
__device__ __forceinline__ void dt_cp16(unsigned char *smem_dst, const void *src, bool valid) {
    unsigned d = (unsigned)__cvta_generic_to_shared(smem_dst);
    int sz = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(sz) : "memory");
}

// Barrier of one of two groups of four warps.
__device__ __forceinline__ void group_sync(int group) {
    if (group == 0) asm volatile("bar.sync 1, 128;" ::: "memory");
    else asm volatile("bar.sync 2, 128;" ::: "memory");
}

}  // namespace lcu
