// Gated delta rule.  Per head a matrix S (f32, one per sequence) is decayed, corrected towards the new value along the new key
// and read along the query:
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// with q, k, v behind short causal convolutions, q and k unit vectors, and o normed and gated per head.
//
// Both products with the state run over the matrix as it was BEFORE the token, so that their reductions share one pass:
//     u = beta (v - g (S^T k)),  S <- g S + k u^T,  o = g (S^T q) + (q . k) u
// A column of S (one value dimension) lies in the registers of eight lanes, four columns in a warp; S never leaves the
// registers inside a portion.  All of it is f32 arithmetic (two values per instruction), whatever the activation dtype.
//
// Rounds with several tokens per request take three launches (convolutions and gates / the scan / norm and output gate), rounds
// of one token per request a single one.  The inputs of the convolutions that a later round needs are double-buffered by
// generation (a request's first token reads one half, its last token writes the other); the matrices are updated in place, every
// column by the one warp that read it.
#include "gqa_prep.cuh"
#include "stack.cuh"

namespace lcu {

typedef __nv_bfloat16 bf16;

namespace {

// two f32 values per instruction
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pk2(float x, float y) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
    return r;
}
__device__ __forceinline__ float2 up2(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_of(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float octet_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    return v + __shfl_xor_sync(0xffffffffu, v, 4);
}

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
};
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
    float y = 0.f;
    for (int j = 0; j < a.taps; ++j) {
        const int back = a.taps - 1 - j;
        const float x = in.at(back, c);
        y = fmaf(a.conv[(size_t)j * in.channels + c], x, y);
        if (out && j > 0) out[(size_t)(j - 1) * in.channels + c] = x;
    }
    return silu_f(y);
}

// ------------------------------------------------------------------ portions: convolutions and gates
// One warp per (token, query/key head) or (token, value head).
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaArgs a) {
    grid_dep_launch();
    const int t = blockIdx.y, lane = threadIdx.x & 31;
    int item = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (item >= a.kv_heads + a.heads) return;
    const int r = a.tok_req[t];
    const bool last = t + 1 == a.req_first[r + 1];
    grid_dep_wait();
    const ConvIn in = conv_in(a, t, r);
    float *out = last ? conv_out(a, r) : nullptr;
    if (item >= a.kv_heads) {
        item -= a.kv_heads;
        const int c0 = 2 * a.kv_heads * a.dk_p + item * a.dv_p;
        float *v = a.v + (size_t)t * a.heads * a.dv_p + (size_t)item * a.dv_p;
        for (int d = lane; d < a.dv_p; d += 32) v[d] = conv_silu(a, in, c0 + d, out);
        return;
    }
    float q[MIX_MAX_HEAD / 32], k[MIX_MAX_HEAD / 32], sq = 0.f, sk = 0.f, qk = 0.f;
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 32; ++j) {
        const int d = lane + 32 * j;
        q[j] = k[j] = 0.f;
        if (d < a.dk_p) {
            q[j] = conv_silu(a, in, item * a.dk_p + d, out);
            k[j] = conv_silu(a, in, (a.kv_heads + item) * a.dk_p + d, out);
        }
        sq += q[j] * q[j];
        sk += k[j] * k[j];
        qk += q[j] * k[j];
    }
    const float rq = 1.f / sqrtf(warp_sum(sq) + 1e-6f) * (1.f / sqrtf((float)a.dk)), rk = 1.f / sqrtf(warp_sum(sk) + 1e-6f);
    qk = warp_sum(qk) * rq * rk;
    const size_t base = ((size_t)t * a.kv_heads + item) * a.dk_p;
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 32; ++j) {
        const int d = lane + 32 * j;
        if (d < a.dk_p) {
            a.q[base + d] = q[j] * rq;
            a.k[base + d] = k[j] * rk;
        }
    }
    const int reps = a.heads / a.kv_heads;
    for (int i = lane; i < reps; i += 32) {
        const int h = item * reps + i;
        const float g = expf(-expf(a.decay[h]) * softplus_of(in.row[a.a_off() + h] + a.decay[a.heads_p + h]));
        const float beta = 1.f / (1.f + expf(-in.row[a.b_off() + h]));
        a.gate[(size_t)t * a.heads + h] = make_float4(g, beta, qk, 0.f);
    }
}

// ------------------------------------------------------------------ portions: the scan
constexpr int DS_TOK = 16;  // tokens per shared-memory tile

__device__ __forceinline__ void ds_cp16(float *smem_dst, const float *src) {
    unsigned d = (unsigned)__cvta_generic_to_shared(smem_dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}

// grid (column slices, heads, requests); a warp holds four columns, lane = 8 (column of the warp) + part of the key dimension.
// R key dimensions per lane: 4 consecutive ones of every 32.
template <int R>
__global__ void __launch_bounds__(256) delta_scan_kernel(const DeltaArgs a) {
    constexpr int DK = 8 * R;
    extern __shared__ __align__(16) float sm[];
    grid_dep_launch();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = lane & 7;
    const int h = blockIdx.y, r = blockIdx.z, kvh = h / (a.heads / a.kv_heads);
    const int cols = blockDim.x / 8, col0 = blockIdx.x * cols, lc = warp * 4 + (lane >> 3), col = col0 + lc;
    const bool valid = col < a.dv_p;
    const int row = 2 * DK + cols + 4;  // q | k | v | gate of a token
    const int first = a.req_first[r], end = a.req_first[r + 1];
    float *st = a.state + (((size_t)(a.req_slot[r] >> 1) * a.heads + h) * a.dv_p + (valid ? col : 0)) * DK + part * 4;
    const bool fresh = a.req_pos[r] == 0;
    f32x2 s[R / 2];
#pragma unroll
    for (int j = 0; j < R / 4; ++j) {
        const float4 v = valid && !fresh ? *reinterpret_cast<const float4 *>(st + 32 * j) : make_float4(0.f, 0.f, 0.f, 0.f);
        s[2 * j] = pk2(v.x, v.y);
        s[2 * j + 1] = pk2(v.z, v.w);
    }
    grid_dep_wait();
    const int vcols = min(cols, a.dv_p - col0);
    auto load = [&](int t0, int buf) {
        float *dst = sm + (size_t)buf * DS_TOK * row;
        const int n = min(DS_TOK, end - t0), per = 2 * (DK / 4) + vcols / 4 + 1;
        for (int i = tid; i < n * per; i += blockDim.x) {
            const int j = i / per, c = i - j * per;
            const size_t t = t0 + j;
            const float *src;
            int at;
            if (c < DK / 4) src = a.q + (t * a.kv_heads + kvh) * DK + 4 * c, at = 4 * c;
            else if (c < 2 * (DK / 4)) src = a.k + (t * a.kv_heads + kvh) * DK + 4 * c - DK, at = 4 * c;
            else if (c < 2 * (DK / 4) + vcols / 4) src = a.v + (t * a.heads + h) * a.dv_p + col0 + 4 * c - 2 * DK, at = 4 * c;
            else src = reinterpret_cast<const float *>(a.gate + t * a.heads + h), at = 2 * DK + cols;
            ds_cp16(dst + j * row + at, src);
        }
    };
    load(first, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    int buf = 0;
    for (int t0 = first; t0 < end; t0 += DS_TOK, buf ^= 1) {
        if (t0 + DS_TOK < end) load(t0 + DS_TOK, buf ^ 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const float *tile = sm + (size_t)buf * DS_TOK * row;
        const int n = min(DS_TOK, end - t0);
        for (int j = 0; j < n; ++j) {
            const float *p = tile + j * row;
            const float4 gate = *reinterpret_cast<const float4 *>(p + 2 * DK + cols);
            const float v = p[2 * DK + (valid ? lc : 0)];
            f32x2 k[R / 2], k2[2] = {0ull, 0ull}, q2[2] = {0ull, 0ull};
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const ulonglong2 kv = *reinterpret_cast<const ulonglong2 *>(p + DK + 32 * i + part * 4);
                const ulonglong2 qv = *reinterpret_cast<const ulonglong2 *>(p + 32 * i + part * 4);
                k[2 * i] = kv.x;
                k[2 * i + 1] = kv.y;
                k2[0] = fma2(s[2 * i], kv.x, k2[0]);
                k2[1] = fma2(s[2 * i + 1], kv.y, k2[1]);
                q2[0] = fma2(s[2 * i], qv.x, q2[0]);
                q2[1] = fma2(s[2 * i + 1], qv.y, q2[1]);
            }
            const float2 ka = up2(k2[0]), kb = up2(k2[1]), qa = up2(q2[0]), qb = up2(q2[1]);
            const float sk = octet_sum((ka.x + ka.y) + (kb.x + kb.y));
            const float u = gate.y * (v - gate.x * sk);
            const f32x2 g2 = pk2(gate.x, gate.x), u2 = pk2(u, u);
#pragma unroll
            for (int i = 0; i < R / 2; ++i) s[i] = fma2(k[i], u2, mul2(s[i], g2));
            const float sq = octet_sum((qa.x + qa.y) + (qb.x + qb.y));
            if (part == 0 && valid) a.v[((size_t)(t0 + j) * a.heads + h) * a.dv_p + col] = gate.x * sq + gate.z * u;
        }
        __syncthreads();
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (!valid) return;
#pragma unroll
    for (int j = 0; j < R / 4; ++j) {
        const float2 x = up2(s[2 * j]), y = up2(s[2 * j + 1]);
        *reinterpret_cast<float4 *>(st + 32 * j) = make_float4(x.x, x.y, y.x, y.y);
    }
}

// ------------------------------------------------------------------ portions: norm and output gate, a warp per (token, head)
template <class T>
__global__ void __launch_bounds__(256) delta_out_kernel(const DeltaArgs a) {
    grid_dep_launch();
    const int lane = threadIdx.x & 31;
    const long i = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (i >= (long)a.n_tok * a.heads) return;
    const int t = (int)(i / a.heads), h = (int)(i - (long)t * a.heads);
    grid_dep_wait();
    const float *o = a.v + (size_t)i * a.dv_p, *g = a.lat + (size_t)t * a.stride + a.g_off() + h * a.dv_p;
    float v[MIX_MAX_HEAD / 32], ss = 0.f;
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 32; ++j) {
        const int d = lane + 32 * j;
        v[j] = d < a.dv_p ? o[d] : 0.f;
        ss += v[j] * v[j];
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)a.dv + a.eps);
    T *dst = reinterpret_cast<T *>(a.o) + (size_t)t * a.stride_o + (size_t)h * a.dv_p;
#pragma unroll
    for (int j = 0; j < MIX_MAX_HEAD / 32; ++j) {
        const int d = lane + 32 * j;
        if (d >= a.dv_p) continue;
        const float x = v[j] * r * a.norm[d] * silu_f(g[d]);
        if constexpr (sizeof(T) == 4) dst[d] = x;
        else dst[d] = Act<T>::from_f(x);
    }
}

// ------------------------------------------------------------------ one token per request: everything in one launch
// CTAs [0, heads) of a request: one head each; the CTAs behind them prepare the attention's queries, keys and values.
template <class T, int R>
__global__ void __launch_bounds__(256) delta_decode_kernel(const DeltaArgs a, const GqaArgs attn, int has_attn) {
    constexpr int DK = 8 * R;
    __shared__ __align__(16) float qs[DK], ks[DK], vs[MIX_MAX_HEAD], os[MIX_MAX_HEAD];
    grid_dep_launch();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = lane & 7;
    const int t = blockIdx.y;  // token t is request t
    if (blockIdx.x >= a.heads) {
        grid_dep_wait();
        const int item = ((int)blockIdx.x - a.heads) * 8 + warp;
        if (has_attn && item < gqa_prep_items(attn)) gqa_prep_item<T>(attn, t, item, lane);
        return;
    }
    const int h = blockIdx.x, reps = a.heads / a.kv_heads, kvh = h / reps;
    const bool fresh = a.req_pos[t] == 0;
    float *st = a.state + ((size_t)(a.req_slot[t] >> 1) * a.heads + h) * a.dv_p * DK + part * 4;
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
    const ConvIn in = conv_in(a, t, t);
    float *out = conv_out(a, t);
    float *qk_out = h == kvh * reps ? out : nullptr;  // one of the heads that share q and k leaves their inputs behind
    for (int i = tid; i < 2 * DK + a.dv_p; i += 256) {
        if (i < DK) qs[i] = conv_silu(a, in, kvh * DK + i, qk_out);
        else if (i < 2 * DK) ks[i - DK] = conv_silu(a, in, (a.kv_heads + kvh) * DK + i - DK, qk_out);
        else vs[i - 2 * DK] = conv_silu(a, in, 2 * a.kv_heads * DK + h * a.dv_p + i - 2 * DK, out);
    }
    const float g = expf(-expf(a.decay[h]) * softplus_of(in.row[a.a_off() + h] + a.decay[a.heads_p + h]));
    const float beta = 1.f / (1.f + expf(-in.row[a.b_off() + h]));
    __syncthreads();
    float sq = 0.f, sk = 0.f, qk = 0.f;
#pragma unroll
    for (int i = 0; i < DK / 32; ++i) {
        const float x = qs[lane + 32 * i], y = ks[lane + 32 * i];
        sq += x * x;
        sk += y * y;
        qk += x * y;
    }
    const float rq = 1.f / sqrtf(warp_sum(sq) + 1e-6f) * (1.f / sqrtf((float)a.dk)), rk = 1.f / sqrtf(warp_sum(sk) + 1e-6f);
    qk = warp_sum(qk) * rq * rk;
    for (int cb = 0; cb < a.dv_p; cb += 32) {
        const int c = cb + c0;
        float dk = 0.f, dq = 0.f;
        float4 kv[R / 4];
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
            kv[j] = *reinterpret_cast<const float4 *>(ks + 32 * j + part * 4);
            const float4 q = *reinterpret_cast<const float4 *>(qs + 32 * j + part * 4), s = cur[j];
            dk = fmaf(s.x, kv[j].x, dk); dk = fmaf(s.y, kv[j].y, dk); dk = fmaf(s.z, kv[j].z, dk); dk = fmaf(s.w, kv[j].w, dk);
            dq = fmaf(s.x, q.x, dq); dq = fmaf(s.y, q.y, dq); dq = fmaf(s.z, q.z, dq); dq = fmaf(s.w, q.w, dq);
        }
        dk = octet_sum(dk) * rk;
        dq = octet_sum(dq) * rq;
        if (c < a.dv_p) {
            const float u = beta * (vs[c] - g * dk), ur = u * rk;
#pragma unroll
            for (int j = 0; j < R / 4; ++j) {
                const float4 s = cur[j];
                *reinterpret_cast<float4 *>(st + (size_t)c * DK + 32 * j) =
                    make_float4(fmaf(kv[j].x, ur, s.x * g), fmaf(kv[j].y, ur, s.y * g), fmaf(kv[j].z, ur, s.z * g), fmaf(kv[j].w, ur, s.w * g));
            }
            if (part == 0) os[c] = g * dq + qk * u;
        }
#pragma unroll
        for (int j = 0; j < R / 4; ++j) cur[j] = nxt[j];
        fetch(c + 64, nxt);
    }
    __syncthreads();
    float ss = 0.f;
    for (int i = lane; i < a.dv_p; i += 32) ss += os[i] * os[i];
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)a.dv + a.eps);
    T *dst = reinterpret_cast<T *>(a.o) + (size_t)t * a.stride_o + (size_t)h * a.dv_p;
    for (int i = tid; i < a.dv_p; i += 256) {
        const float x = os[i] * r * a.norm[i] * silu_f(in.row[a.g_off() + h * a.dv_p + i]);
        if constexpr (sizeof(T) == 4) dst[i] = x;
        else dst[i] = Act<T>::from_f(x);
    }
}

// calls f.template run<R>() with the key dimensions per lane
template <class F>
int by_dk(int dk_p, const F &f) {
    switch (dk_p) {
    case 32: return f.template run<4>();
    case 64: return f.template run<8>();
    case 96: return f.template run<12>();
    case 128: return f.template run<16>();
    case 160: return f.template run<20>();
    case 192: return f.template run<24>();
    case 224: return f.template run<28>();
    case 256: return f.template run<32>();
    default: set_error("delta rule: key size %d (a multiple of 32, at most 256)", dk_p); return LCU_ERR_INVALID;
    }
}

struct ScanLaunch {
    const DeltaArgs &a;
    cudaStream_t s;
    bool pdl;
    template <int R> int run() const {
        // 32 columns per CTA where that still fills the SMs, 16 otherwise
        const int cols = a.dv_p > 16 && (long)a.n_req * a.heads * ((a.dv_p + 31) / 32) * 4 >= 3 * sm_count() ? 32 : 16;
        const size_t smem = (size_t)2 * DS_TOK * (16 * R + cols + 4) * 4;
        const dim3 grid((a.dv_p + cols - 1) / cols, a.heads, a.n_req);
        if (smem > 48 * 1024) LCU_CHECK_CUDA(cudaFuncSetAttribute(delta_scan_kernel<R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        LCU_CHECK_CUDA(launch_kernel(delta_scan_kernel<R>, grid, dim3(cols * 8), smem, s, pdl, a));
        return LCU_OK;
    }
};
struct DecodeLaunch {
    const DeltaArgs &a;
    const GqaArgs *attn;
    int dt;
    cudaStream_t s;
    bool pdl;
    template <int R> int run() const {
        const dim3 grid(a.heads + (attn ? (attn->heads + 2 * attn->kv_heads + 7) / 8 : 0), a.n_req);
        const GqaArgs none{};
        if (dt == LCU_F32) LCU_CHECK_CUDA(launch_kernel(delta_decode_kernel<float, R>, grid, dim3(256), 0, s, pdl, a, attn ? *attn : none, attn ? 1 : 0));
        else LCU_CHECK_CUDA(launch_kernel(delta_decode_kernel<bf16, R>, grid, dim3(256), 0, s, pdl, a, attn ? *attn : none, attn ? 1 : 0));
        return LCU_OK;
    }
};

}  // namespace

int delta_prep_launch(const DeltaArgs &a, cudaStream_t s, bool pdl) {
    if (a.n_tok <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_tok <= 65535 && a.dk_p <= MIX_MAX_HEAD && a.dv_p <= MIX_MAX_HEAD, "delta rule: %d tokens, head sizes %d / %d", a.n_tok, a.dk_p, a.dv_p);
    LCU_CHECK_CUDA(launch_kernel(delta_prep_kernel, dim3((a.kv_heads + a.heads + 7) / 8, a.n_tok), dim3(256), 0, s, pdl, a));
    return LCU_OK;
}
int delta_scan_launch(const DeltaArgs &a, cudaStream_t s, bool pdl) {
    if (a.n_req <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_req <= 65535 && a.heads <= 65535, "delta rule: grid out of range");
    return by_dk(a.dk_p, ScanLaunch{a, s, pdl});
}
int delta_out_launch(const DeltaArgs &a, int dt, cudaStream_t s, bool pdl) {
    if (a.n_tok <= 0) return LCU_OK;
    const unsigned grid = (unsigned)(((long)a.n_tok * a.heads + 7) / 8);
    if (dt == LCU_F32) LCU_CHECK_CUDA(launch_kernel(delta_out_kernel<float>, dim3(grid), dim3(256), 0, s, pdl, a));
    else LCU_CHECK_CUDA(launch_kernel(delta_out_kernel<bf16>, dim3(grid), dim3(256), 0, s, pdl, a));
    return LCU_OK;
}
int delta_decode_launch(const DeltaArgs &a, const GqaArgs *attn, int dt, cudaStream_t s, bool pdl) {
    if (a.n_req <= 0) return LCU_OK;
    LCU_REQUIRE(a.n_req <= 65535 && a.dv_p <= MIX_MAX_HEAD, "delta rule: %d requests, value size %d", a.n_req, a.dv_p);
    return by_dk(a.dk_p, DecodeLaunch{a, attn, dt, s, pdl});
}

}  // namespace lcu
