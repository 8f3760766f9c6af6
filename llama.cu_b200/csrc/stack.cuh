// Models described layer by layer (lcu_ctx_create_layers): per-layer shapes and weights, the part of a round that is
// theirs, and the kernels their layers are made of.  Interface only; rounds are built in stack.cu, the mixer kernels
// are in latent.cu, gqa.cu and delta.cu, norms / residual / token shift in stack_ops.cu, the 32-bit linear layer in
// linear_f32.cu.
//
// Storage conventions: every dimension a matrix product sums over is padded with zeros to a multiple of 64 (per-head
// query/key and value sizes to a multiple of 16), so each shape takes the tensor-core kernels; the pads stay zero through
// every layer.  The residual stream, the norms' inputs and outputs before rounding, scores and softmax are f32 whatever
// the activation dtype; the activation dtype (bf16, or f32 for an all-32-bit context) is that of matrix-product operands.
#pragma once
#include <vector>

#include "common.cuh"
#include "gemv.cuh"
#include "mixers.cuh"

struct lcu_ctx;

namespace lcu {

constexpr int stack_pad(int v, int m) { return (v + m - 1) / m * m; }

struct StackLayer {
    lcu_layer_desc d;
    int src;        // the layer whose tensors this one uses (itself unless weights are shared)
    size_t c_off;   // element offset of this layer's cached rows inside a page: [page_tokens][r_p]
    // padded sizes
    int dim_p, vdim_p, qr_p, r_p, g_p, ff_p, hv_p;
    // softmax attention and recurrent mixers
    int att_rows = 0;                     // rows of the fused input projection that are the attention's q, k, v (the first ones; g_p head gates behind them)
    int kv_src = 0;                       // layer whose cache this one reads
    int dk_p = 0, dv_p = 0, dh_p = 0, dhv_p = 0, rank_p = 0;
    int e_p = 0, sff_p = 0;               // experts, width of the shared one
    size_t conv_off = 0, mat_off = 0;     // f32 offsets of this layer's recurrent state in its arena section (inputs of the mixer's convolutions, matrices)
    const float2 *rot = nullptr, *vrot = nullptr;  // [nctx][rot_dims / 2] (cos, sin); of values [nctx][v_dim / 2]
    bool latent() const { return d.mixer == LCU_MIX_LATENT; }
    bool attention() const { return (d.mixer & LCU_MIX_ATTENTION) != 0; }
    bool delta() const { return (d.mixer & LCU_MIX_DELTA) != 0; }
    bool ssd() const { return (d.mixer & LCU_MIX_SSD) != 0; }
    bool gla() const { return (d.mixer & LCU_MIX_GLA) != 0; }
    bool recurrent() const { return delta() || ssd() || gla(); }
    bool own_kv() const { return d.kv_from == 0; }
    bool glu() const { return d.ff_act == LCU_ACT_GLU; }
    bool poly() const { return d.ff_act == LCU_ACT_POLYNORM; }
    bool parallel() const { return d.parallel_ff && has_ff(); }
    bool has_ff() const { return d.ff > 0 || d.shared_ff > 0; }
    int qkv_rows() const { return 2 * d.delta_kv_heads * dk_p + d.delta_heads * dv_p; }  // of a recurrent mixer
    int rec_rows() const { return recurrent() ? qkv_rows() + d.delta_heads * dv_p + (gla() ? rank_p : ssd() ? dh_p : 2 * dh_p) : 0; }
    int conv_channels() const { return gla() ? 0 : qkv_rows(); }
    int in_rows() const { return latent() ? qr_p + r_p + g_p : att_rows + g_p + rec_rows(); }  // rows of the fused input projection: query latent | latent | gate, or attention | recurrent mixer
    int kv_cols() const { return d.heads * (dim_p + vdim_p); }  // columns of the expanded keys and values
};

struct StackWeights {
    const void *in = nullptr, *q_norm = nullptr, *kv_norm = nullptr, *uq = nullptr, *ukt = nullptr, *ukv = nullptr,
               *out = nullptr, *up = nullptr, *down = nullptr, *shift = nullptr;
    const float *scalars = nullptr;  // mixer norm gain, feed-forward norm gain, activation p, q
    // pre-norm layers
    const void *att_out = nullptr, *delta_out = nullptr;
    const float *bias = nullptr, *conv = nullptr, *decay = nullptr, *delta_norm = nullptr, *branch_norm = nullptr, *norm1 = nullptr,
                *norm2 = nullptr, *step = nullptr, *post1 = nullptr, *post2 = nullptr, *qk_gain = nullptr, *conv_bias = nullptr, *gate_map = nullptr;
    const void *router = nullptr, *shared_up = nullptr, *shared_down = nullptr;
    const float *att_conv = nullptr, *sink = nullptr, *head_temp = nullptr, *up_bias = nullptr, *down_bias = nullptr, *act = nullptr, *correction = nullptr;
};

// What the host decides about a round: which requests run their attention in latent space ("absorbed") and which expand
// keys and values first, in batches that fit the expansion buffer.
struct StackRound {
    int n_abs_tok = 0, n_abs_req = 0;
    bool abs_decode = false;  // every absorbed request brings one token
    struct Batch { int n_rows, req0, n_req, group0, n_groups; };
    std::vector<Batch> batches;
    // softmax attention: requests whose portion takes the short form, and those that take the long one
    int n_short = 0, max_short = 0, n_long = 0;
    std::vector<int> long_len;
    int n_delta_blocks = 0, n_scan_blocks = 0;  // recurrent mixers: blocks of tokens
};

struct Stack {
    std::vector<StackLayer> layers;
    std::vector<StackWeights> w;
    int d_p = 0, vocab_p = 0;
    int n_slots = 0;
    // arena sections (see stack_create)
    float *x[2] = {nullptr, nullptr}, *y = nullptr, *lat = nullptr, *state = nullptr;
    void *h = nullptr, *cq = nullptr, *q = nullptr, *qa = nullptr, *att = nullptr, *act = nullptr, *xc = nullptr, *xkv = nullptr,
         *hout = nullptr;
    float *part_o = nullptr, *part_ml = nullptr;
    int *part_n = nullptr;
    void *arena = nullptr;
    size_t part_rows = 0;   // rows of absorbed attention (tokens x heads) times splits the partial buffers hold
    int abs_cap = 0;        // absorbed tokens a round may hold
    int expand_cap = 0;     // rows of the expansion buffer (0: never expand)
    int max_heads = 0, max_r = 0;
    // pre-norm models
    bool pre_norm = false;
    float *y2 = nullptr, *dq = nullptr, *dk = nullptr, *dv = nullptr, *dcoef = nullptr, *conv_state = nullptr, *mat_state = nullptr, *gqa_part = nullptr;
    void *att2 = nullptr;
    unsigned *gqa_tickets = nullptr;
    size_t conv_gen = 0;    // f32 values of one generation of the convolutions' state
    int gqa_ctas = 0;       // CTAs of split short-form attention the partial buffer holds
    struct RotTable { int dims; double base, factor, original, fast, slow; float2 *dev; };
    std::vector<RotTable> rot_tables;  // layers with the same rotation share one
    void *h2 = nullptr;                // input of a feed-forward beside a mixer
    float *z = nullptr;                // f32 rows of the up projection (LCU_ACT_POLYNORM)
    // mixers beside a feed-forward: a stream of their own between two events, with scratch for its linear layers
    cudaStream_t side = nullptr;
    cudaEvent_t fork = nullptr, join = nullptr;
    void *side_ws = nullptr;
    unsigned *side_tickets = nullptr;
    const void *pair_embd = nullptr;
    uint32_t *last_token = nullptr;  // [generation 2][slots]
    float *dtail = nullptr;          // linear recurrences: decays over blocks
    // experts: routing, lists, activations in slot order, products
    float *router = nullptr, *ye = nullptr, *moe_w = nullptr, *moe_slot_w = nullptr;
    int *moe_ints = nullptr;         // expert, place, slot_of, slot_tok: [max_tokens * top] each
    unsigned *moe_count = nullptr;
    int4 *moe_tiles = nullptr;
    void *xg = nullptr, *act_e = nullptr;
    int max_rows = 0, max_experts = 0, n_tiles = 0;  // capacities
    bool caps() const { return layers[0].d.logit_cap > 0.f || (layers[0].d.logit_scale != 0.f && layers[0].d.logit_scale != 1.f); }
};

// ---- stack.cu
int stack_create(lcu_ctx *c, const lcu_layer_desc *layers);
void stack_destroy(lcu_ctx *c);
size_t stack_page_elems(const Stack &s, int page_tokens);
bool stack_weight_shape(const lcu_ctx *c, int layer, int kind, int *rows, int *cols, int *elem_bytes);
int stack_set_weight(lcu_ctx *c, int layer, int kind, const void *ptr);  // layer < 0: a weight of the model
bool stack_ready(const lcu_ctx *c);
size_t stack_desc_bytes(int max_tok, int max_req);
struct Round;
// plans the round's attention and fills its section of the descriptor (host copy H)
int stack_stage(lcu_ctx *c, Round &r, const lcu_req *reqs, unsigned char *H);
// every layer of one round; leaves the residual stream in lcu_ctx::x
int stack_layers(lcu_ctx *c, const Round &r, cudaStream_t s, int *count);
// final norm of the asked rows and the LM head; logits in the activation dtype, or f32 at `out_f32`
int stack_head(lcu_ctx *c, const Round &r, const uint32_t *rows, int n_rows, float *out_f32, cudaStream_t s, int *count);
// rounds short enough for every launch to be a programmatic dependent of its predecessor
bool stack_pdl(const lcu_ctx *c, int n_tok);
double stack_step_bytes(const lcu_ctx *c, const lcu_req *reqs, int n_req, int n_out);

// ---- stack_ops.cu
// x_out = x_in + g * y / rms(y) (or an embedding row when `embd` is given), then
// h = x_out + (previous token's x_out - x_out) * shift, rounded to the activation dtype; either output may be missing
struct MixInputArgs {
    const float *x_in, *y;
    float *x_out;
    void *h;
    int n_tok, d, d_p;
    const float *gain;   // g: gain[0] for every coordinate, or a vector when gain_stride is 1
    int gain_stride;
    float eps;
    const void *embd;    // bf16 [vocab, d_p]
    const uint32_t *tokens;
    const void *shift;   // bf16 [d_p]; nullptr: no token shift
    // recurrent state of the shift: f32 [2][slots][d_p] of this layer, rows (generation, slot)
    float *state;
    size_t state_gen_stride;
    const int32_t *tok_req, *req_first, *req_pos, *req_slot;  // request of a token; first token, position, slot * 2 + generation of a request
};
int op_mix_input(const MixInputArgs &a, int dt, cudaStream_t s, bool pdl);
// Pre-norm layers: x_out = x_in + the sublayer's output + embedding + step, then h = gain * x_out / rms(x_out), rounded to the
// activation dtype; every input and h may be missing.  The sublayer's output is one of
//     sum of y (each y * y_gain / rms(y) when gains are given)
//     post_gain * s / rms(s), s = sum of y_scale * y and of the token's rows of ye
//     sum of y, y_bias and ye_w * the token's rows of ye (slot -1: of ff_in)
// h2 = gain2 * x_out / rms(x_out) for a feed-forward beside the mixer.
struct PreNormArgs {
    const float *x_in;
    const float *y[2];
    const float *y_gain;  // [2][d_p]
    const float *post_gain;
    float y_scale[2];
    const float *ye;      // outputs of experts [slot][d_p], `top` slots per token
    const float *ye_w;    // [n_tok][top] or nullptr
    const void *ff_in;    // [n_tok][d_p], activation dtype
    const float *y_bias;  // [d_p] or nullptr
    const int *slot_of;
    int top;
    const void *embd;     // bf16 [vocab, d_p], times embd_scale
    float embd_scale;
    const uint32_t *tokens;
    // embedding of token pairs: bf16 [buckets + 1, d_p]; a sequence's last token is kept per (generation, slot)
    const void *pair_embd;
    int pair_buckets, pair_prev, pair_cur;
    uint32_t *last_token;
    size_t last_gen_stride;
    const int32_t *tok_req, *req_first, *req_pos, *req_slot;
    const float *step;
    float *x_out;
    void *h, *h2;
    const float *gain, *gain2;
    float eps;
    int n_tok, d, d_p;
    unsigned *zero;       // counters that the kernels behind expect to be zero
    int n_zero;
};
int op_pre_norm(const PreNormArgs &a, int dt, cudaStream_t s, bool pdl);
// Activation of LCU_ACT_POLYNORM on z + bias, rounded; columns past ff are zero.
struct PolyNormArgs {
    const float *z;       // [n_tok][ff_p]
    const float *bias;    // [ff_p] or nullptr
    const float *act;     // a, b, c, e
    void *y;              // [n_tok][ff_p]
    int n_tok, ff, ff_p;
    float eps;
};
int op_poly_norm(const PolyNormArgs &a, int dt, cudaStream_t s, bool pdl);
// y = x[rows[i]] * gain / rms(x), rounded
int op_scalar_norm_rows(void *y, const float *x, const uint32_t *rows, int n, int d, int d_p, const float *gain, int gain_stride, float eps,
                        int dt, cudaStream_t s, bool pdl);
// 16-bit rows to f32
int op_rows_to_f32(float *dst, const void *src, size_t n, int dt, cudaStream_t s);

// ---- linear_f32.cu: y = x W^T per head with f32 activations and bf16 weights, true 32-bit products and sums
struct LinearF32Args {
    const float *x;
    int stride_x, head_x;       // row and head strides
    const int32_t *x_rows;      // optional row gather
    const void *w;              // bf16 [heads][out][in]
    float *y;
    int stride_y, head_y;
    const int32_t *y_rows;      // optional row scatter
    int n, in, out, heads;
    int epilogue;               // EPI_STORE_F32, EPI_XIELU, EPI_RELU2, EPI_GLU, EPI_CAP_F32
    const float *act_pq;
    const float *gate;          // optional: multiplied by sigmoid(gate[y row * stride_gate + head])
    int stride_gate;
    GluArgs glu;                // EPI_GLU
    CapArgs cap;                // EPI_CAP_F32
    const int4 *tiles;          // grouped: (matrix, first row, rows up to 64), `heads` 1, no gather; see GemvArgs
    int n_tiles;
    const float *row_scale;
};
int linear_f32_launch(const LinearF32Args &a, cudaStream_t s);

// ---- latent.cu
struct LatentNormArgs {
    const float *lat;           // [n_tok, stride]: query latent | latent | gate logits
    int stride, n_tok, q_rank, qr_p, kv_rank, r_p;
    const void *q_norm, *kv_norm;  // bf16, padded with zeros
    float eps;
    void *cq;                   // [n_tok, qr_p]
    void *pool;
    size_t page_elems, c_off;
    int page_shift;
    const int32_t *tok_req;
    const uint32_t *pos;
    const int32_t *page_table;
    int pt_stride;
};
int latent_norm_launch(const LatentNormArgs &a, int dt, cudaStream_t s, bool pdl);

// per-head linear layer on tensor cores: y[row][h][:] = W[h] x[row][h][:]
struct HeadLinearArgs {
    const void *x;              // activation dtype, row stride_x, head stride head_x; nullptr: merge attention partials instead
    int stride_x, head_x;
    const int32_t *x_rows, *y_rows;
    const void *w;              // [heads][out][in]
    void *y;
    int stride_y, head_y;
    int n, in, out, heads;
    const float *part_o, *part_ml;  // [row * heads + h][splits][in], (max, sum)
    const int *part_n;
    int splits;
    const float *gate;
    int stride_gate;
};
int head_linear_launch(const HeadLinearArgs &a, cudaStream_t s, bool pdl, bool dry = false);

// attention of absorbed queries over the cached latents; rows are (absorbed token, head) pairs
struct LatentAttnArgs {
    const void *q;              // [rows, r_p]
    const void *pool;
    size_t page_elems, c_off;
    int page_shift, n_pages;
    const int32_t *page_table;
    int pt_stride;
    const int32_t *req_first;   // [n_req + 1] first absorbed token of each absorbed request
    const int32_t *req_id;      // its index in the round
    const int32_t *req_pos;     // position of the first token of request req_id (indexed by round request)
    int n_req, n_tok, decode;   // decode: one token per request
    int heads, r_p;
    float scale;
    float *part_o, *part_ml;    // [row][splits][r_p] unnormalised, [row][splits][2]
    int *part_n;                // [row] splits used
    int splits;                 // grid depth
    uint32_t *status;           // bit 4: a bounded wait ran out
};
int latent_attn_rows_per_block(int heads, bool decode, int dt, int page_tokens);
int latent_attn_launch(const LatentAttnArgs &a, int dt, cudaStream_t s, bool pdl, bool dry = false);
// ---- latent_tc.cu: the decode form on tcgen05 (pages of at least 64 tokens)
bool latent_tc_supported(int page_tokens);
int latent_tc_rows(int heads);
int latent_tc_launch(const LatentAttnArgs &a, cudaStream_t s, bool pdl, bool dry = false);
// copies the cached latents of the batch's requests into consecutive rows
int latent_gather_launch(void *dst, const void *pool, size_t page_elems, size_t c_off, int page_shift, const int32_t *page_table,
                         int pt_stride, const int4 *reqs, int n_req, int max_rows, int r_p, cudaStream_t s);
// causal attention over expanded keys and values, one query group of 64 tokens and one head per CTA
struct ExpandedAttnArgs {
    const void *q;              // [n_tok, heads, dim_p]
    int stride_q;
    const void *kv;             // [rows, heads * dim_p | heads * vdim_p]
    int stride_kv;
    void *o;                    // [n_tok, heads, vdim_p]
    int stride_o;
    const int4 *groups;         // first token, tokens, position of the first token, first row of the sequence's keys
    int n_groups, heads, dim_p, vdim_p;
    float scale;
    const float *gate;
    int stride_gate;
};
bool expanded_attn_supported(int dim_p, int vdim_p);
int expanded_attn_launch(const ExpandedAttnArgs &a, cudaStream_t s, bool dry = false);

#ifdef __CUDACC__
template <class T> __device__ __forceinline__ void st4(T *p, const float4 &v);
template <> __device__ __forceinline__ void st4<float>(float *p, const float4 &v) { *reinterpret_cast<float4 *>(p) = v; }
template <> __device__ __forceinline__ void st4<__nv_bfloat16>(__nv_bfloat16 *p, const float4 &v) {
    *reinterpret_cast<uint2 *>(p) = make_uint2(Act<__nv_bfloat16>::pack(v.x, v.y), Act<__nv_bfloat16>::pack(v.z, v.w));
}
__device__ __forceinline__ float4 ld4_bf16(const void *base, size_t i) {
    const uint2 u = __ldg(reinterpret_cast<const uint2 *>(reinterpret_cast<const __nv_bfloat16 *>(base) + i));
    const float2 a = Act<__nv_bfloat16>::to_f2(u.x), b = Act<__nv_bfloat16>::to_f2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
template <class T> __device__ __forceinline__ float4 ld4(const T *p);
template <> __device__ __forceinline__ float4 ld4<float>(const float *p) { return *reinterpret_cast<const float4 *>(p); }
template <> __device__ __forceinline__ float4 ld4<__nv_bfloat16>(const __nv_bfloat16 *p) {
    const uint2 u = *reinterpret_cast<const uint2 *>(p);
    const float2 a = Act<__nv_bfloat16>::to_f2(u.x), b = Act<__nv_bfloat16>::to_f2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float dot4(const float4 &a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }

// Sum of two values over the block (at most 32 warps); every thread gets both.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2 *part) {
    a = warp_sum(a);
    b = warp_sum(b);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    if (lane == 0) part[warp] = make_float2(a, b);
    __syncthreads();
    float2 v = lane < nw ? part[lane] : make_float2(0.f, 0.f);
    v.x = warp_sum(v.x);
    v.y = warp_sum(v.y);
    return v;
}
#endif  // __CUDACC__

}  // namespace lcu
