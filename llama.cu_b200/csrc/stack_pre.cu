// Layers of pre-norm models: x += mixer(norm(x)), x += ff(norm(x)), or with norms on the outputs too, or both at once on one x with
// a norm each.  A mixer is softmax
// attention, a recurrent mixer (delta rule, state space duality, gated linear attention), or one of each side by side on the same
// input, their outputs added.  One projection serves both; the feed-forward is one for all tokens or one of experts.  Rounds,
// pages, state slots, head and sampling are those of every layered model.
#include "moe.cuh"
#include "stack_round.cuh"

#include <cmath>

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

    // what a sublayer left behind (see PreNormArgs); no output at all: the embedding
    struct Outputs {
        const float *y0 = nullptr, *y1 = nullptr, *y_gain = nullptr, *post_gain = nullptr;
        float scale0 = 1.f, scale1 = 1.f;
        int top = 0;  // rows of experts per token
        const float *weights = nullptr, *bias = nullptr;  // on experts' rows; of the feed-forward's last matrix
        const void *ff_in = nullptr;                      // what experts without matrices return
    };
    // x after a sublayer's outputs, what comes ahead of the next one, and h, normed with `gain` (and h2 with `gain2`)
    int residual(const Outputs &u, bool embed, const float *step, const float *gain, int n_zero = 0, const float *gain2 = nullptr) {
        PreNormArgs a{};
        const lcu_model_desc &d = c->desc;
        const bool start = !u.y0 && !u.top;
        a.n_tok = r.n_tok; a.d = d.d; a.d_p = S().d_p; a.eps = d.eps;
        if (!start) {
            a.x_in = S().x[cur];
            cur ^= 1;
        }
        a.y[0] = u.y0; a.y[1] = u.y1; a.y_gain = u.y_gain; a.post_gain = u.post_gain; a.y_scale[0] = u.scale0; a.y_scale[1] = u.scale1;
        if (u.top) { a.top = u.top; a.ye = S().ye; a.slot_of = moe_int(2); a.ye_w = u.weights; a.ff_in = u.ff_in; }
        a.y_bias = u.bias; a.gain2 = gain2; a.h2 = gain2 ? S().h2 : nullptr;
        if (embed || start) {
            const lcu_layer_desc &l = S().layers[0].d;
            a.embd = c->embd; a.tokens = reinterpret_cast<const uint32_t *>(D + r.L.tokens);
            a.embd_scale = l.embed_scale ? l.embed_scale : 1.f;
            if (l.pair_buckets) {
                a.pair_embd = S().pair_embd; a.pair_buckets = l.pair_buckets; a.pair_prev = l.pair_prev; a.pair_cur = l.pair_cur;
                a.last_token = S().last_token; a.last_gen_stride = S().n_slots;
                a.tok_req = reinterpret_cast<const int32_t *>(D + r.L.tok_req);
                a.req_first = i32(o.req_first); a.req_pos = i32(o.req_pos); a.req_slot = i32(o.req_slot);
            }
        }
        a.step = step; a.x_out = S().x[cur]; a.gain = gain; a.h = gain ? S().h : nullptr;
        a.zero = S().moe_count; a.n_zero = n_zero;
        return done(op_pre_norm(a, c->dt, s, L.dependent()));
    }
    // ... ahead of layer `next` (past the last one: the head reads x itself)
    int residual_into(int next, const Outputs &u) {
        if (next >= c->desc.n_layers) return residual(u, false, nullptr, nullptr);
        const StackLayer &Y = S().layers[next];
        const StackWeights &W = S().w[Y.src];
        return residual(u, Y.d.add_embed, Y.d.add_step ? S().w[next].step : nullptr, W.norm1, Y.parallel() ? counters(Y) : 0, Y.parallel() ? W.norm2 : nullptr);
    }

    GqaArgs gqa(const StackLayer &Y, const StackWeights &W) const {
        GqaArgs a{};
        a.lat = S().lat; a.stride = Y.in_rows(); a.n_tok = r.n_tok;
        a.heads = Y.d.heads; a.kv_heads = Y.d.kv_heads; a.dim = Y.d.dim; a.dim_p = Y.dim_p; a.v_dim = Y.d.v_dim; a.vdim_p = Y.vdim_p;
        a.bias = W.bias; a.own_kv = Y.own_kv(); a.qk_norm = Y.d.qk_norm; a.qk_gain = W.qk_gain; a.eps = c->desc.eps;
        a.rot_dims = Y.d.rot_dims; a.rot_adjacent = Y.d.rot_adjacent; a.rot = Y.rot; a.q = S().q;
        a.vrot = Y.vrot; a.head_temp = W.head_temp; a.keep = Y.d.window ? Y.d.keep_first : 0; a.sink_score = W.sink;
        if (Y.d.conv) {
            a.conv = W.att_conv; a.taps = Y.d.conv; a.conv_state = S().conv_state + Y.conv_off * S().n_slots; a.conv_gen_stride = S().conv_gen;
            a.req_first = i32(o.req_first); a.req_pos = i32(o.req_pos); a.req_slot = i32(o.req_slot);
        }
        a.window = Y.d.window; a.sink = Y.d.sink; a.gate = Y.d.out_gate ? S().lat + Y.att_rows : nullptr;
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
            rc = done(gqa_short_launch(a, s, L.dependent()));
        }
        if (!rc && q.n_long) {
            a.reqs = reinterpret_cast<const int4 *>(B + o.lreq); a.n_reqs = q.n_long; a.n_blocks = 0;
            for (int len : q.long_len) a.n_blocks += (len * a.group() + 63) / 64;
            rc = done(gqa_long_launch(a, s));
        }
        return rc;
    }

    void recurrent(DeltaArgs &a, const StackLayer &Y, const StackWeights &W) const {
        a.lat = S().lat + Y.att_rows + Y.g_p; a.stride = Y.in_rows(); a.n_tok = r.n_tok; a.n_req = r.n_req;
        a.heads = Y.d.delta_heads; a.kv_heads = Y.d.delta_kv_heads; a.dk = Y.d.delta_dim; a.dk_p = Y.dk_p; a.dv = Y.d.delta_v_dim; a.dv_p = Y.dv_p;
        a.heads_p = Y.dh_p; a.taps = Y.d.delta_conv; a.eps = c->desc.eps; a.conv = W.conv; a.conv_bias = W.conv_bias; a.decay = W.decay; a.norm = W.delta_norm;
        a.conv_state = S().conv_state + Y.conv_off * S().n_slots; a.conv_gen_stride = S().conv_gen; a.state = S().mat_state + Y.mat_off * S().n_slots;
        a.tok_req = reinterpret_cast<const int32_t *>(D + r.L.tok_req);
        a.req_first = i32(o.req_first); a.req_pos = i32(o.req_pos); a.req_slot = i32(o.req_slot);
        a.split = c->dt != LCU_F32 && tuning().delta_tc;
        a.q = S().dq; a.k = S().dk; a.v = S().dv; a.coef = S().dcoef;
        a.blocks = reinterpret_cast<const int4 *>(B + o.dblk); a.n_blocks = r.sr.n_delta_blocks; a.o = S().att2; a.stride_o = Y.dhv_p;
    }
    ScanArgs scan(const StackLayer &Y, const StackWeights &W) const {
        ScanArgs a{};
        recurrent(a, Y, W);
        a.blocks = reinterpret_cast<const int4 *>(B + o.sblk); a.n_blocks = r.sr.n_scan_blocks;
        a.per_channel = Y.gla(); a.gate_map = W.gate_map; a.rank = Y.d.gate_rank; a.rank_p = Y.rank_p;
        if (Y.gla()) {
            a.inv_tau = 1.f / Y.d.gate_tau;
            a.q_scale = 1.f / sqrtf((float)Y.d.delta_dim);
            a.vin = a.lat + 2 * a.heads * a.dk_p; a.vin_stride = a.stride;
        } else {
            a.vin = a.v; a.vin_stride = a.heads * a.dv_p;
        }
        a.parts = Y.d.norm_parts; a.tail = S().dtail;
        return a;
    }

    // the recurrent mixer and, ahead of the attention itself, its preparation
    int recurrent_and_prep(const StackLayer &Y, const StackWeights &W, const GqaArgs &g) {
        const int dt = c->dt;
        const GqaArgs *attn = Y.attention() ? &g : nullptr;
        int rc = LCU_OK;
        if (Y.delta()) {
            DeltaArgs e{};
            recurrent(e, Y, W);
            if (r.decode_only) return done(delta_decode_launch(e, attn, dt, s, L.dependent()));
            if (attn) rc = done(gqa_prep_launch(g, dt, s, L.dependent()));
            if (!rc) rc = done(delta_prep_launch(e, s, L.dependent()));
            if (!rc) rc = done(delta_scan_launch(e, s, L.dependent()));
            return rc ? rc : done(delta_out_launch(e, dt, s, L.dependent()));
        }
        if (!Y.recurrent() || !r.decode_only) rc = attn ? done(gqa_prep_launch(g, dt, s, L.dependent())) : LCU_OK;
        if (rc || !Y.recurrent()) return rc;
        const ScanArgs e = scan(Y, W);
        if (r.decode_only) rc = done(scan_step_launch(e, attn, dt, s, L.dependent()));
        else if (dt == LCU_F32) rc = done(scan_step_launch(e, nullptr, dt, s, L.dependent()));
        else {
            rc = done(scan_prep_launch(e, s, L.dependent()));
            if (!rc) rc = done(scan_launch(e, s, L.dependent()));
            if (!rc && Y.gla()) rc = done(delta_out_launch(e, dt, s, L.dependent()));
        }
        return rc || !Y.ssd() ? rc : done(scan_out_launch(e, dt, s, L.dependent()));
    }

    // h -> outputs of the layer's mixers in y and y2
    int mixers(const StackLayer &Y, const StackWeights &W) {
        const int n = r.n_tok;
        int rc = L.linear(W.in, S().d_p, Y.in_rows(), S().h, n, S().lat, Y.in_rows(), EPI_STORE_F32);
        const GqaArgs g = gqa(Y, W);
        if (!rc) rc = recurrent_and_prep(Y, W, g);
        if (!rc && Y.attention()) rc = attention(g, Y);
        if (!rc && Y.attention()) rc = L.linear(W.att_out, Y.hv_p, S().d_p, S().att, n, S().y, S().d_p, EPI_STORE_F32);
        if (!rc && Y.recurrent()) rc = L.linear(W.delta_out, Y.dhv_p, S().d_p, S().att2, n, Y.attention() ? S().y2 : S().y, S().d_p, EPI_STORE_F32);
        return rc;
    }

    // ---- feed-forward: h -> y (or rows of experts in ye)
    int *moe_int(int i) const { return S().moe_ints + (size_t)i * S().max_rows; }
    GluArgs glu(const StackLayer &Y, float limit) const { return GluArgs{limit, Y.d.glu_alpha, Y.d.glu_shift}; }
    int dense_glu(const void *up, const void *down, int ff_p, const GluArgs &u, const void *h, float *y) {
        int rc = L.linear(up, S().d_p, 2 * ff_p, h, r.n_tok, S().act, ff_p, EPI_GLU, nullptr, PRO_NONE, nullptr, u);
        return rc ? rc : L.linear(down, ff_p, S().d_p, S().act, r.n_tok, y, S().d_p, EPI_STORE_F32);
    }
    bool small_experts() const { return c->dt != LCU_F32 && r.n_tok <= MOE_SMALL_ROUND; }
    // counters that a round's routing expects to be zero
    int counters(const StackLayer &Y) const { return Y.d.experts && !small_experts() ? Y.d.experts : 0; }
    int experts(const StackLayer &Y, const StackWeights &W, const void *h, float *y) {
        const int n = r.n_tok, d_p = S().d_p, rows = n * Y.d.top;
        const GluArgs u = glu(Y, Y.d.glu_limit), us = glu(Y, Y.d.shared_limit);
        int rc = L.linear(W.router, d_p, Y.e_p, h, n, S().router, Y.e_p, EPI_STORE_F32);
        MoeRoute m{};
        m.logits = S().router; m.n_tok = n; m.experts = Y.d.experts; m.experts_p = Y.e_p; m.top = Y.d.top;
        m.softmax = Y.d.route_softmax; m.correction = W.correction; m.identity = Y.d.identity;
        m.expert = moe_int(0); m.place = moe_int(1); m.slot_of = moe_int(2); m.slot_tok = moe_int(3);
        m.weight = S().moe_w; m.slot_w = S().moe_slot_w; m.count = S().moe_count; m.tiles = S().moe_tiles;
        m.h = h; m.xg = S().xg; m.d_p = d_p;
        const float *in_scale = Y.d.route_softmax ? nullptr : m.slot_w;  // weights on the inputs
        if (small_experts()) {
            m.max_tiles = rows < Y.d.experts ? rows : Y.d.experts; m.tile_rows = n;
            if (!rc) rc = done(moe_plan_launch(m, s, L.dependent()));
            MoeProduct p{};
            p.tiles = m.tiles; p.max_tiles = m.max_tiles; p.n_tok = n; p.shared = Y.d.shared_ff > 0; p.slot_w = in_scale; p.slot_tok = m.slot_tok;
            p.up = 1; p.w = W.up; p.ws = W.shared_up; p.out = 2 * Y.ff_p; p.in = d_p; p.outs = 2 * Y.sff_p; p.ins = d_p;
            p.x = p.xs = h; p.y = S().act_e; p.ys = S().act; p.glu = u; p.glus = us;
            if (!rc) rc = done(moe_product_launch(p, s, L.dependent()));
            p.up = 0; p.w = W.down; p.ws = W.shared_down; p.out = p.outs = d_p; p.in = Y.ff_p; p.ins = Y.sff_p;
            p.x = S().act_e; p.xs = S().act; p.y = S().ye; p.ys = y;
            return rc ? rc : done(moe_product_launch(p, s, L.dependent()));
        }
        // tiles as wide as an expert's share of the round
        const int share = rows / (Y.d.experts + Y.d.identity);
        m.tile_rows = c->dt == LCU_F32 || share <= 64 ? 64 : (share <= 128 ? 128 : 256);
        m.max_tiles = moe_max_tiles(rows, Y.d.experts, m.tile_rows);
        if (!rc) rc = done(moe_route_launch(m, s, L.dependent()));
        if (!rc) rc = done(moe_gather_launch(m, c->dt, s, L.dependent()));
        auto grouped = [&](const void *w, int in, int out, const void *x, void *y, int stride_y, int epilogue) -> int {
            if (c->dt == LCU_F32) {
                LinearF32Args a{};
                a.x = reinterpret_cast<const float *>(x); a.stride_x = in; a.w = w; a.y = reinterpret_cast<float *>(y); a.stride_y = stride_y;
                a.n = rows; a.in = in; a.out = out; a.heads = 1; a.epilogue = epilogue; a.glu = u;
                a.tiles = m.tiles; a.n_tiles = m.max_tiles; a.row_scale = in_scale;
                return done(linear_f32_launch(a, s));
            }
            GemvArgs a{};
            a.w = w; a.x = x; a.stride_x = in; a.n_tok = rows; a.in = in; a.out = out; a.epilogue = epilogue; a.y = y; a.stride_y = stride_y; a.glu = u;
            a.tiles = m.tiles; a.n_tiles = m.max_tiles; a.tile_rows = m.tile_rows; a.groups = Y.d.experts; a.row_scale = in_scale;
            return done(gemm_tc_launch(a, c->dt, s, L.dependent()));
        };
        if (!rc) rc = grouped(W.up, d_p, 2 * Y.ff_p, S().xg, S().act_e, Y.ff_p, EPI_GLU);
        if (!rc) rc = grouped(W.down, Y.ff_p, d_p, S().act_e, S().ye, d_p, EPI_STORE_F32);
        if (!rc && Y.d.shared_ff) rc = dense_glu(W.shared_up, W.shared_down, Y.sff_p, us, h, y);
        return rc;
    }
    int feed_forward(const StackLayer &Y, const StackWeights &W, const void *h, float *y) {
        if (Y.d.experts) return experts(Y, W, h, y);
        if (Y.glu()) return dense_glu(W.up, W.down, Y.ff_p, glu(Y, Y.d.glu_limit), h, y);
        int rc;
        if (Y.poly()) {
            rc = L.linear(W.up, S().d_p, Y.ff_p, h, r.n_tok, S().z, Y.ff_p, EPI_STORE_F32);
            const PolyNormArgs a{S().z, W.up_bias, W.act, S().act, r.n_tok, Y.d.ff, Y.ff_p, c->desc.eps};
            if (!rc) rc = done(op_poly_norm(a, c->dt, s, L.dependent()));
        } else {
            rc = L.linear(W.up, S().d_p, Y.ff_p, h, r.n_tok, S().act, Y.ff_p, EPI_RELU2);
        }
        return rc ? rc : L.linear(W.down, Y.ff_p, S().d_p, S().act, r.n_tok, y, S().d_p, EPI_STORE_F32);
    }
    // outputs of a feed-forward, dense ones in y
    void add_ff(Outputs &u, const StackLayer &Y, const StackWeights &W, const void *h) const {
        u.bias = W.down_bias;
        if (!Y.d.experts) return;
        u.top = Y.d.top;
        if (Y.d.route_softmax) { u.weights = S().moe_w; u.ff_in = h; }
    }

    void stream_scratch(bool side) const {
        gemm_tc_set_scratch(side ? S().side_ws : c->sk_ws, c->sk_ws_bytes, side ? S().side_tickets : c->sk_tickets, 4096, c->dev_status);
    }
    // Mixer and feed-forward of one x: one after the other, or the mixer on a stream of its own, of higher priority, so that its short
    // steps run while the feed-forward's weights stream.
    int both(const StackLayer &Y, const StackWeights &W) {
        if (!forks()) {
            const int rc = feed_forward(Y, W, S().h2, S().y2);
            return rc ? rc : mixers(Y, W);
        }
        const cudaStream_t main = s;
        LCU_CHECK_CUDA(cudaEventRecord(S().fork, main));
        LCU_CHECK_CUDA(cudaStreamWaitEvent(S().side, S().fork, 0));
        s = L.s = S().side;
        L.joined = true;
        stream_scratch(true);
        int rc = mixers(Y, W);
        s = L.s = main;
        L.joined = false;
        stream_scratch(false);
        LCU_CHECK_CUDA(cudaEventRecord(S().join, S().side));
        if (!rc) rc = feed_forward(Y, W, S().h2, S().y2);
        LCU_CHECK_CUDA(cudaStreamWaitEvent(main, S().join, 0));
        L.joined = true;
        return rc;
    }
    bool forks() const { return S().side && tuning().stack_fork; }

    int run() {
        stream_scratch(false);
        int rc = residual_into(0, Outputs{});
        for (int l = 0; l < c->desc.n_layers && !rc; ++l) {
            const StackLayer &Y = S().layers[l];
            const StackWeights &W = S().w[Y.src];
            const bool pair = Y.attention() && Y.recurrent();
            rc = Y.parallel() ? both(Y, W) : mixers(Y, W);
            if (rc) break;
            Outputs u;
            u.y0 = S().y; u.y1 = pair ? S().y2 : nullptr; u.y_gain = pair ? W.branch_norm : nullptr; u.post_gain = W.post1;
            if (pair && Y.d.post_norm) { u.scale0 = Y.d.out_scale; u.scale1 = Y.d.out_scale2; }
            if (Y.parallel()) {
                if (!Y.d.experts) u.y1 = S().y2;
                add_ff(u, Y, W, S().h2);
            }
            if (!Y.has_ff() || Y.parallel()) {
                rc = residual_into(l + 1, u);
                continue;
            }
            rc = residual(u, false, nullptr, W.norm2, counters(Y));
            if (!rc) rc = feed_forward(Y, W, S().h, S().y);
            u = Outputs{};
            u.y0 = Y.d.experts && !Y.d.shared_ff ? nullptr : S().y; u.post_gain = W.post2;
            add_ff(u, Y, W, S().h);
            if (!rc) rc = residual_into(l + 1, u);
        }
        c->x = S().x[cur];
        return rc;
    }
};

}  // namespace

int pre_norm_layers(lcu_ctx *c, const Round &r, cudaStream_t s, int *count) { return PreNormRound(c, r, s, count).run(); }

}  // namespace lcu
