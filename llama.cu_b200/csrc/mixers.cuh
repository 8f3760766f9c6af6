// Mixers of pre-norm layers: softmax attention over cached keys and values (gqa.cu), the gated delta rule (delta.cu), state space
// duality and gated linear attention (scan.cu).  All read f32 rows of one fused input projection and write operands of their output projections.  Interface only.
#pragma once
#include "common.cuh"

namespace lcu {

constexpr int MIX_MAX_HEAD = 256;  // largest head size of either mixer

// ---- softmax attention, grouped heads, rotary positions
struct GqaArgs {
    // rows of the fused projection: q heads | k heads | v heads, every head padded to dim_p / vdim_p (q heads alone when the layer
    // reads another one's cache)
    const float *lat;
    int stride, n_tok;
    int heads, kv_heads, dim, dim_p, v_dim, vdim_p;
    const float *bias;          // [q | k | v] or nullptr
    int own_kv;                 // 0: the cache at c_off is another layer's
    int qk_norm;                // RMS norm of q and k: 1 per head after the rotation, 2 / 3 ahead of it, per head / over all heads
    const float *qk_gain;       // qk_norm 2: [q dim_p | k dim_p], 3: [q heads | k heads]
    float eps;
    int rot_dims, rot_adjacent; // pairs (i, i + rot_dims / 2), or (2 i, 2 i + 1)
    const float2 *rot;          // [positions][rot_dims / 2] (cos, sin), the frequency scaling's factor included
    const float2 *vrot;         // [positions][v_dim / 2]: values are rotated by their positions, outputs back by theirs; or nullptr
    const float *head_temp;     // [heads] factors on the queries, or nullptr
    // convolutions over time on the rows of the projection: [taps][channels]; inputs before the portion in the state
    // [generation][slot][taps - 1][channels]
    const float *conv;
    int taps;
    float *conv_state;
    size_t conv_gen_stride;
    const int32_t *req_first, *req_pos, *req_slot;
    void *q;                    // [n_tok][heads * dim_p]
    // pages: this layer's keys [kv head][slot][dim_p] at c_off, its values [kv head][slot][vdim_p] behind them
    void *pool;
    size_t page_elems, c_off;
    int page_shift;
    const int32_t *tok_req, *page_table;
    const uint32_t *pos;
    int pt_stride;
    // attention
    void *o;                    // [n_tok][stride_o], heads x vdim_p
    int stride_o;
    float scale;
    int window;                 // > 0: a position sees the `window` last ones up to itself
    int keep;                   // with a window: the first tokens of the sequence stay visible
    int sink;                   // one more key without value, of score 0 or sink_score[head]
    const float *sink_score;
    const float *gate;          // output gates before the sigmoid: gate[token * stride + head], or nullptr
    const int4 *reqs;           // (request of the round, first token, tokens, position of the first token)
    int n_reqs, max_len;        // longest of them in tokens
    int n_blocks;               // long form: blocks of 64 (token, head) rows of all requests
    // short form: contexts cut into splits, merged by the last CTA to arrive
    int splits;
    float *part_o, *part_ml;    // [request][kv head x row tile][split][16][vdim_p], [...][16][2]
    unsigned *tickets;          // [request][kv head x row tile], zero between launches
    __host__ __device__ size_t v_off() const { return c_off + ((size_t)kv_heads * dim_p << page_shift); }
    __host__ __device__ int group() const { return heads / kv_heads; }
    __host__ __device__ int channels() const { return heads * dim_p + (own_kv ? kv_heads * (dim_p + vdim_p) : 0); }
};
// Biases, rotation, norms; queries to q, keys and values to the cache.
int gqa_prep_launch(const GqaArgs &a, int dt, cudaStream_t s, bool pdl);
// A portion takes the short form up to this many tokens.
int gqa_short_tokens(int heads, int kv_heads);
int gqa_row_tiles(int heads, int kv_heads, int len);   // 16-row tiles of a request's short form, per key/value head
size_t gqa_part_floats(int ctas, int vdim_p);          // scratch of `ctas` CTAs of the short form (part_o and part_ml)
int gqa_short_ctas_per_sm(int dim_p, int vdim_p);
int gqa_short_launch(const GqaArgs &a, cudaStream_t s, bool pdl, bool dry = false);
int gqa_long_launch(const GqaArgs &a, cudaStream_t s, bool dry = false);
int gqa_f32_launch(const GqaArgs &a, cudaStream_t s);

// ---- gated delta rule
constexpr int DELTA_BLOCK = 8;                                                   // tokens of a block of the scan
constexpr int DELTA_COEF = 2 * DELTA_BLOCK * DELTA_BLOCK + 2 * DELTA_BLOCK;      // coefficients of a block and head
struct DeltaArgs {
    // rows of the fused projection: q heads | k heads (dk_p) | v heads | output gate (dv_p) | step size | decay (heads_p)
    const float *lat;
    int stride, n_tok, n_req;
    int heads, kv_heads, dk, dk_p, dv, dv_p, heads_p, taps;
    float eps;
    const float *conv;          // [taps][channels]
    const float *conv_bias;     // [channels] or nullptr
    const float *decay;         // [2][heads_p]: logarithm of the rate, bias
    const float *norm;          // [dv_p]
    // state: inputs of the convolutions [generation][slot][taps - 1][channels], matrices [slot][head][dv_p][dk_p]
    float *conv_state;
    size_t conv_gen_stride;
    float *state;
    const int32_t *tok_req, *req_first, *req_pos, *req_slot;
    // between the kernels of a round with several tokens per request
    int split;                  // the scan runs on tensor cores: q and k as three bf16 planes [n_tok][kv_heads][3][dk_p]
    float *q, *k;               // [n_tok][kv_heads * dk_p], unit vectors, q scaled
    float *v;                   // [n_tok][heads * dv_p]; the scan overwrites it with its outputs
    const int4 *blocks;         // (request, first token, tokens, slot first / 8 + request + number of the block in its request)
    int n_blocks;
    float *coef;                // [slot][heads][DELTA_COEF]
    void *o;                    // [n_tok][stride_o], heads x dv_p
    int stride_o;
    __host__ __device__ int channels() const { return 2 * kv_heads * dk_p + heads * dv_p; }
    __host__ __device__ int g_off() const { return channels(); }
    __host__ __device__ int b_off() const { return channels() + heads * dv_p; }
    __host__ __device__ int a_off() const { return b_off() + heads_p; }
    __host__ __device__ int rows() const { return a_off() + heads_p; }
};
// Rounds with several tokens per request: convolutions, gates and triangles; the scan; norm and output gate.
int delta_prep_launch(const DeltaArgs &a, cudaStream_t s, bool pdl);
int delta_scan_launch(const DeltaArgs &a, cudaStream_t s, bool pdl);
int delta_out_launch(const DeltaArgs &a, int dt, cudaStream_t s, bool pdl);
// Rounds of one token per request: all of it in one launch, beside the attention's preparation (nullptr: none).
int delta_decode_launch(const DeltaArgs &a, const GqaArgs *attn, int dt, cudaStream_t s, bool pdl);

// ---- linear recurrences: S <- decay S + k v^T, o = S^T q
// SSD: one decay per head, keys and queries of a group of heads behind short convolutions, values scaled by a step size; the
// output takes D v up, is gated, then normed in parts of the whole width.  GLA: one decay per head and key channel, no
// convolutions, output normed per head, then gated.  The rows of the fused projection are those of DeltaArgs with, behind the
// output gate, SSD: step size (heads_p), GLA: the first map of the decays (rank_p).
constexpr int SCAN_BLOCK = 16;                                      // tokens of a block of the scan
constexpr int SCAN_COEF = SCAN_BLOCK * SCAN_BLOCK + 2 * SCAN_BLOCK; // coefficients of a block and head
struct ScanArgs : DeltaArgs {   // decay: SSD [3][heads_p], weight of v behind the bias; norm: SSD [heads][dv_p]
    int per_channel;            // GLA
    const float *gate_map;      // GLA: [rank + 1][heads * dk_p]
    int rank, rank_p;
    float inv_tau, q_scale;
    int parts;                  // SSD: parts of the output norm
    const float *vin;           // values the scan reads: [n_tok][vin_stride], heads x dv_p
    int vin_stride;
    float *tail;                // GLA: decay over a block [slot][heads][dk_p]
    __host__ __device__ int rec_rows() const { return b_off() + (per_channel ? rank_p : heads_p); }
};
// Portions in bf16 contexts: operands and coefficients of blocks; the scan.  Then scan_out.
int scan_prep_launch(const ScanArgs &a, cudaStream_t s, bool pdl);
int scan_launch(const ScanArgs &a, cudaStream_t s, bool pdl);
// Token by token, everything up to the output's norm (GLA: with it): rounds of one token per request, beside the attention's
// preparation, and portions of all-32-bit contexts (attn nullptr).
int scan_step_launch(const ScanArgs &a, const GqaArgs *attn, int dt, cudaStream_t s, bool pdl);
// SSD: gate and norm
int scan_out_launch(const ScanArgs &a, int dt, cudaStream_t s, bool pdl);

}  // namespace lcu
