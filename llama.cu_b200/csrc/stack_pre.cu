// Layers of pre-norm models: x += mixer(norm(x)), x += ff(norm(x)).  A mixer is softmax attention, a gated delta rule, or both
// side by side on the same input, their outputs normed and added.  One projection serves both; rounds, pages, state slots, head
// and sampling are those of every layered model.
#include "stack_round.cuh"

namespace lcu {

namespace {

struct PreNormRound {
    lcu_ctx *c;
    const Round &r;
    cudaStream_t s;
    int *count;
    Launcher L;
    const unsigned char *D, *B;
    StackDesc o;
    int cur = 0;  // which of the two residual buffers holds x

    PreNormRound(lcu_ctx *c_, const Round &r_, cudaStream_t s_, int *count_)
        : c(c_), r(r_), s(s_), count(count_), L{c_, s_, count_, stack_pdl(c_, r_.n_tok)}, D(c_->desc_dev), B(c_->desc_dev + r_.L.stack),
          o(stack_desc(r_.n_tok, r_.n_req)) {
        L.weights_first = true;
    }
    Stack &S() const { return *c->stack; }
    const int32_t *i32(size_t off) const { return reinterpret_cast<const int32_t *>(B + off); }
    int done(int rc) {
        if (!rc) ++*count;
        return rc;
    }

    // x after a sublayer's outputs (none: the embedding), what comes ahead of layer `next`, and h, normed with `gain`
    int residual(const float *y0, const float *y1, const float *y_gain, bool embed, const float *step, const float *gain) {
        PreNormArgs a{};
        const lcu_model_desc &d = c->desc;
        a.n_tok = r.n_tok; a.d = d.d; a.d_p = S().d_p; a.eps = d.eps;
        if (y0) {
            a.x_in = S().x[cur];
            cur ^= 1;
        }
        a.y[0] = y0; a.y[1] = y1; a.y_gain = y_gain;
        if (embed) { a.embd = c->embd; a.tokens = reinterpret_cast<const uint32_t *>(D + r.L.tokens); }
        a.step = step; a.x_out = S().x[cur]; a.gain = gain; a.h = gain ? S().h : nullptr;
        return done(op_pre_norm(a, c->dt, s, L.pdl));
    }
    // ... ahead of layer `next` (past the last one: the head reads x itself)
    int residual_into(int next, const float *y0, const float *y1, const float *y_gain) {
        if (next >= c->desc.n_layers) return residual(y0, y1, y_gain, false, nullptr, nullptr);
        const StackLayer &Y = S().layers[next];
        return residual(y0, y1, y_gain, !y0 || Y.d.add_embed, Y.d.add_step ? S().w[next].step : nullptr, S().w[Y.src].norm1);
    }

    GqaArgs gqa(const StackLayer &Y, const StackWeights &W) const {
        GqaArgs a{};
        a.lat = S().lat; a.stride = Y.in_rows(); a.n_tok = r.n_tok;
        a.heads = Y.d.heads; a.kv_heads = Y.d.kv_heads; a.dim = Y.d.dim; a.dim_p = Y.dim_p; a.v_dim = Y.d.v_dim; a.vdim_p = Y.vdim_p;
        a.bias = W.bias; a.qk_norm = Y.d.qk_norm; a.eps = c->desc.eps; a.rot_dims = Y.d.rot_dims; a.rot = Y.rot; a.q = S().q;
        a.pool = c->pool; a.page_elems = c->geom.page_elems; a.c_off = Y.c_off; a.page_shift = c->geom.page_shift;
        a.tok_req = reinterpret_cast<const int32_t *>(D + r.L.tok_req); a.page_table = reinterpret_cast<const int32_t *>(D + r.L.page_table);
        a.pos = reinterpret_cast<const uint32_t *>(D + r.L.pos); a.pt_stride = c->pt_stride;
        a.o = S().att; a.stride_o = Y.hv_p; a.scale = Y.d.scale;
        return a;
    }
    int attention(GqaArgs a, const StackLayer &Y) {
        if (c->dt == LCU_F32) return done(gqa_f32_launch(a, s));
        const StackRound &q = r.sr;
        int rc = LCU_OK;
        if (q.n_short) {
            a.reqs = reinterpret_cast<const int4 *>(B + o.sreq); a.n_reqs = q.n_short; a.max_len = q.max_short;
            a.splits = gqa_splits_for(c, Y, q.n_short, q.max_short);
            const int cells = q.n_short * a.kv_heads * gqa_row_tiles(a.heads, a.kv_heads, q.max_short);
            LCU_REQUIRE(a.splits == 1 || cells * a.splits <= S().gqa_ctas, "step: %d attention partials do not fit", cells * a.splits);
            a.tickets = S().gqa_tickets;
            a.part_ml = S().gqa_part; a.part_o = S().gqa_part + (size_t)cells * a.splits * 32;
            rc = done(gqa_short_launch(a, s, L.pdl));
        }
        if (!rc && q.n_long) {
            a.reqs = reinterpret_cast<const int4 *>(B + o.lreq); a.n_reqs = q.n_long; a.n_blocks = 0;
            for (int len : q.long_len) a.n_blocks += (len * a.group() + 63) / 64;
            rc = done(gqa_long_launch(a, s));
        }
        return rc;
    }

    DeltaArgs delta(const StackLayer &Y, const StackWeights &W) const {
        DeltaArgs a{};
        a.lat = S().lat + Y.att_rows; a.stride = Y.in_rows(); a.n_tok = r.n_tok; a.n_req = r.n_req;
        a.heads = Y.d.delta_heads; a.kv_heads = Y.d.delta_kv_heads; a.dk = Y.d.delta_dim; a.dk_p = Y.dk_p; a.dv = Y.d.delta_v_dim; a.dv_p = Y.dv_p;
        a.heads_p = Y.dh_p; a.taps = Y.d.delta_conv; a.eps = c->desc.eps; a.conv = W.conv; a.decay = W.decay; a.norm = W.delta_norm;
        a.conv_state = S().conv_state + Y.conv_off * S().n_slots; a.conv_gen_stride = S().conv_gen; a.state = S().mat_state + Y.mat_off * S().n_slots;
        a.tok_req = reinterpret_cast<const int32_t *>(D + r.L.tok_req);
        a.req_first = i32(o.req_first); a.req_pos = i32(o.req_pos); a.req_slot = i32(o.req_slot);
        a.split = c->dt != LCU_F32 && tuning().delta_tc;
        a.q = S().dq; a.k = S().dk; a.v = S().dv; a.coef = S().dcoef;
        a.blocks = reinterpret_cast<const int4 *>(B + o.dblk); a.n_blocks = r.sr.n_delta_blocks; a.o = S().att2; a.stride_o = Y.dhv_p;
        return a;
    }

    // h -> outputs of the layer's mixers in y and y2
    int mixers(const StackLayer &Y, const StackWeights &W) {
        const int n = r.n_tok, dt = c->dt;
        int rc = L.linear(W.in, S().d_p, Y.in_rows(), S().h, n, S().lat, Y.in_rows(), EPI_STORE_F32);
        const GqaArgs g = gqa(Y, W);
        const DeltaArgs e = delta(Y, W);
        if (Y.delta() && r.decode_only) {
            if (!rc) rc = done(delta_decode_launch(e, Y.attention() ? &g : nullptr, dt, s, L.pdl));
        } else {
            if (!rc && Y.attention()) rc = done(gqa_prep_launch(g, dt, s, L.pdl));
            if (!rc && Y.delta()) rc = done(delta_prep_launch(e, s, L.pdl));
            if (!rc && Y.delta()) rc = done(delta_scan_launch(e, s, L.pdl));
            if (!rc && Y.delta()) rc = done(delta_out_launch(e, dt, s, L.pdl));
        }
        if (!rc && Y.attention()) rc = attention(g, Y);
        if (!rc && Y.attention()) rc = L.linear(W.att_out, Y.hv_p, S().d_p, S().att, n, S().y, S().d_p, EPI_STORE_F32);
        if (!rc && Y.delta()) rc = L.linear(W.delta_out, Y.dhv_p, S().d_p, S().att2, n, Y.attention() ? S().y2 : S().y, S().d_p, EPI_STORE_F32);
        return rc;
    }

    int run() {
        gemm_tc_set_scratch(c->sk_ws, c->sk_ws_bytes, c->sk_tickets, 4096, c->dev_status);
        int rc = residual_into(0, nullptr, nullptr, nullptr);
        for (int l = 0; l < c->desc.n_layers && !rc; ++l) {
            const StackLayer &Y = S().layers[l];
            const StackWeights &W = S().w[Y.src];
            const bool both = Y.attention() && Y.delta();
            rc = mixers(Y, W);
            if (rc) break;
            if (!Y.d.ff) {
                rc = residual_into(l + 1, S().y, both ? S().y2 : nullptr, both ? W.branch_norm : nullptr);
                continue;
            }
            rc = residual(S().y, both ? S().y2 : nullptr, both ? W.branch_norm : nullptr, false, nullptr, W.norm2);
            if (!rc) rc = L.linear(W.up, S().d_p, Y.ff_p, S().h, r.n_tok, S().act, Y.ff_p, EPI_RELU2);
            if (!rc) rc = L.linear(W.down, Y.ff_p, S().d_p, S().act, r.n_tok, S().y, S().d_p, EPI_STORE_F32);
            if (!rc) rc = residual_into(l + 1, S().y, nullptr, nullptr);
        }
        c->x = S().x[cur];
        return rc;
    }
};

}  // namespace

int pre_norm_layers(lcu_ctx *c, const Round &r, cudaStream_t s, int *count) { return PreNormRound(c, r, s, count).run(); }

}  // namespace lcu
