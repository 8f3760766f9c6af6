// Linear layer in true 32-bit arithmetic: f32 activations, bf16 weights widened exactly, f32 FMA.  It serves all-32-bit
// contexts (checking and debugging), not the benchmarked path: a 64 x 64 output tile per CTA, 4 x 4 outputs per thread.
#include "gemv.cuh"
#include "stack.cuh"

namespace lcu {

__global__ void __launch_bounds__(256) linear_f32_kernel(const LinearF32Args a) {
    __shared__ float xs[16][68], ws[16][68];
    const int o0 = blockIdx.x * 64;
    int t0 = blockIdx.y * 64, head = blockIdx.z, n = a.n;
    if (a.tiles) {  // rows t.y .. t.y + t.z meet matrix t.x
        const int4 t = a.tiles[blockIdx.y];
        if (t.z == 0) return;
        t0 = t.y; n = t.y + t.z; head = t.x;
    }
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const __nv_bfloat16 *w = reinterpret_cast<const __nv_bfloat16 *>(a.w) + (size_t)head * a.out * a.in;
    const float *x = a.x + (a.tiles ? 0 : (size_t)head * a.head_x);
    float acc[4][4] = {};
    const int lr = tid >> 2, lk = (tid & 3) * 4;  // loader: row of the tile, first of 4 columns
    const int xt = t0 + lr;
    const size_t xrow = xt < n ? (size_t)(a.x_rows ? a.x_rows[xt] : xt) * a.stride_x : 0;
    for (int k0 = 0; k0 < a.in; k0 += 16) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int k = k0 + lk + i;
            xs[lk + i][lr] = (xt < n && k < a.in) ? x[xrow + k] : 0.f;
            ws[lk + i][lr] = (o0 + lr < a.out && k < a.in) ? __bfloat162float(w[(size_t)(o0 + lr) * a.in + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            float xv[4], wv[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { xv[i] = xs[k][ty * 4 + i]; wv[i] = ws[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = t0 + ty * 4 + i;
        if (t >= n) continue;
        const size_t yr = (size_t)(a.y_rows ? a.y_rows[t] : t);
        float g = 1.f;
        if (a.gate) g = 1.f / (1.f + expf(-a.gate[yr * a.stride_gate + head]));
        if (a.epilogue == EPI_GLU) {
            const float sc = a.row_scale ? a.row_scale[yr] : 1.f;
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int o = o0 + tx * 4 + j;
                if (o + 1 < a.out) a.y[yr * a.stride_y + o / 2] = glu_act(sc * acc[i][j], sc * acc[i][j + 1], a.glu);
            }
            continue;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int o = o0 + tx * 4 + j;
            if (o >= a.out) continue;
            float v = acc[i][j];
            if (a.epilogue == EPI_XIELU) v = xielu_act(v, softplus_f(a.act_pq[0]), softplus_f(a.act_pq[1]));
            else if (a.epilogue == EPI_RELU2) v = relu2_act(v);
            else if (a.epilogue == EPI_CAP_F32) v = cap_logit(v, a.cap);
            a.y[yr * a.stride_y + (a.tiles ? 0 : (size_t)head * a.head_y) + o] = a.gate ? v * g : v;
        }
    }
}

int linear_f32_launch(const LinearF32Args &a, cudaStream_t s) {
    if (a.n <= 0) return LCU_OK;
    LCU_REQUIRE(a.epilogue == EPI_STORE_F32 || a.epilogue == EPI_RELU2 || a.epilogue == EPI_GLU || a.epilogue == EPI_CAP_F32 || (a.epilogue == EPI_XIELU && a.act_pq), "linear_f32: epilogue %d", a.epilogue);
    dim3 grid((a.out + 63) / 64, a.tiles ? a.n_tiles : (a.n + 63) / 64, a.heads);
    LCU_REQUIRE(grid.y <= 65535 && grid.z <= 65535, "linear_f32: grid out of range");
    LCU_CHECK_CUDA(launch_kernel(linear_f32_kernel, grid, dim3(256), 0, s, false, a));
    return LCU_OK;
}

}  // namespace lcu
