// Inputs of causal convolutions over time, for portions of a sequence.
#pragma once
#include "common.cuh"

namespace lcu {

// A request's view of the convolutions' inputs: rows of this round, before them the state, before the sequence zeros.
struct ConvIn {
    const float *row;        // this token's row of the projection
    const float *state;      // [taps - 1][channels] of the generation to read, newest last
    int stride, channels, taps, in_portion, seen;  // tokens of the portion before this one, of the sequence before this one
    __device__ __forceinline__ float at(int back, int c) const {
        if (back <= in_portion) return row[c - (ptrdiff_t)back * stride];
        if (back > seen) return 0.f;
        return state[(size_t)(taps - 1 - (back - in_portion)) * channels + c];
    }
    __device__ __forceinline__ float4 at4(int back, int c) const {  // four channels
        if (back <= in_portion) return *reinterpret_cast<const float4 *>(row + (c - (ptrdiff_t)back * stride));
        if (back > seen) return make_float4(0.f, 0.f, 0.f, 0.f);
        return *reinterpret_cast<const float4 *>(state + (size_t)(taps - 1 - (back - in_portion)) * channels + c);
    }
};

}  // namespace lcu
