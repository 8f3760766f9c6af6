// What the layer loops of stack.cu and stack_pre.cu share: the stack section of the round descriptor and the linear layer.
#pragma once
#include "ctx.cuh"
#include "gemv.cuh"
#include "stack.cuh"

namespace lcu {

inline size_t act_bytes(const lcu_ctx *c) { return c->dt == LCU_F32 ? 4 : 2; }

// offsets inside the stack section of the round descriptor
struct StackDesc {
    size_t req_first, req_pos, req_slot, abs_first, abs_id, abs_tok, xreq, xgroups, sreq, lreq, dblk, sblk, total;
};
constexpr int EXPAND_GROUP = 64;  // query tokens per group of the expanded attention
inline StackDesc stack_desc(int n_tok, int n_req) {
    StackDesc d;
    size_t o = 0;
    auto take = [&](size_t bytes) { size_t r = o; o += (bytes + 15) & ~(size_t)15; return r; };
    d.req_first = take((size_t)(n_req + 1) * 4);
    d.req_pos = take((size_t)n_req * 4);
    d.req_slot = take((size_t)n_req * 4);
    d.abs_first = take((size_t)(n_req + 1) * 4);
    d.abs_id = take((size_t)n_req * 4);
    d.abs_tok = take((size_t)n_tok * 4);
    d.xreq = take((size_t)n_req * 16);
    d.xgroups = take((size_t)(n_tok / EXPAND_GROUP + n_req) * 16);
    d.sreq = take((size_t)n_req * 16);
    d.lreq = take((size_t)n_req * 16);
    d.dblk = take((size_t)(n_tok / DELTA_BLOCK + n_req) * 16);
    d.sblk = take((size_t)(n_tok / SCAN_BLOCK + n_req) * 16);
    d.total = o;
    return d;
}

struct Launcher {
    lcu_ctx *c;
    cudaStream_t s;
    int *count;
    bool pdl;
    bool weights_first = false;  // one-token GEMVs of this round request weights before activations
    CapArgs cap{};               // of EPI_CAP and EPI_CAP_F32
    bool joined = false;         // the next launch follows an event of another stream: no programmatic dependent

    bool dependent() {
        const bool r = pdl && !joined;
        joined = false;
        return r;
    }

    // y[n, out] = x[n, in] W^T; x and bf16 y in the activation dtype, EPI_STORE_F32 into f32 rows
    int linear(const void *w, int in, int out, const void *x, int n, void *y, int stride_y, int epilogue, const float *act_pq = nullptr,
               int prologue = PRO_NONE, const GemvArgs *pro = nullptr, const GluArgs &glu = GluArgs{}) {
        if (c->dt == LCU_F32) {
            LinearF32Args a{};
            a.x = reinterpret_cast<const float *>(x); a.stride_x = in; a.w = w;
            a.y = reinterpret_cast<float *>(y); a.stride_y = stride_y;
            a.n = n; a.in = in; a.out = out; a.heads = 1;
            a.epilogue = epilogue == EPI_STORE ? EPI_STORE_F32 : epilogue == EPI_CAP ? EPI_CAP_F32 : epilogue;
            a.act_pq = act_pq; a.glu = glu; a.cap = cap;
            ++*count;
            return linear_f32_launch(a, s);
        }
        const size_t yb = epilogue == EPI_STORE_F32 || epilogue == EPI_CAP_F32 ? 4 : 2;
        // three and four tokens: the GEMV streams small matrices faster, the tcgen05 kernels large ones (4 sequences at 8192, per
        // 8-layer step: width 4096 1.88 -> 1.55 ms, width 2048 0.88 -> 1.04 ms)
        const bool tc = n > 4 || (n > 2 && (tuning().stack_tc == 2 || (tuning().stack_tc == 1 && (long)in * out >= (32l << 20))));
        for (int t0 = 0; t0 < n;) {
            const int most = tc ? (tuning().tc_block < 256 ? tuning().tc_block : GEMM_TC_MAX_TOKENS) : gemv_max_tokens(in);
            const int nt = n - t0 < most ? n - t0 : most;
            const bool pdl = dependent();
            GemvArgs a{};
            a.w = w;
            a.x = reinterpret_cast<const unsigned char *>(x) + (size_t)t0 * in * 2;
            a.stride_x = in; a.n_tok = nt; a.in = in; a.out = out;
            a.prologue = PRO_NONE; a.epilogue = epilogue; a.act_pq = act_pq; a.glu = glu; a.cap = cap;
            a.y = reinterpret_cast<unsigned char *>(y) + (size_t)t0 * stride_y * yb;
            a.stride_y = stride_y;
            if (pro) {  // one launch (at most two tokens): the prologue's rows, and the tokens' places in the cache
                a.pro = pro->pro; a.pos = pro->pos; a.tok_seq = pro->tok_seq; a.page_table = pro->page_table; a.pt_stride = pro->pt_stride;
                a.eps = pro->eps; a.prologue = prologue;
            }
            // Dependent launches.  The GEMV's CTAs fill every register file, so it releases its own dependents at its exit only
            // (releasing them at entry: 0.79 -> 0.91 ms per 8-layer step of width 4096 at batch 1), and asks for weights ahead of
            // the wait only where that measured faster (one token, no norm prologue: 0.79 -> 0.77 ms; two tokens 0.92 -> 0.94).
            a.pdl_trigger = pdl && tc ? 0 : 2;
            a.early_prefetch = pdl && weights_first && n == 1 ? 3 : 1;
            int rc = tc ? gemm_tc_launch(a, c->dt, s, pdl) : gemv_launch(a, c->dt, s, pdl);
            if (rc) return rc;
            ++*count;
            t0 += nt;
        }
        return LCU_OK;
    }
};

// every layer of one round of a pre-norm model
int pre_norm_layers(lcu_ctx *c, const Round &r, cudaStream_t s, int *count);
// CTAs and splits of the short-form attention of `reqs` requests of at most `len` tokens
int gqa_splits_for(const lcu_ctx *c, const StackLayer &L, int reqs, int len);

}  // namespace lcu
