// Rounds of models described layer by layer: shapes and storage, the plan of a round's attention, and the launches of every
// layer.  Context, pages, descriptor staging, graphs and sampling are those of ctx.cu.
#include "moe.cuh"
#include "stack_round.cuh"

#include <cmath>

namespace lcu {

static size_t align256(size_t v) { return (v + 255) & ~(size_t)255; }

size_t stack_desc_bytes(int max_tok, int max_req) { return stack_desc(max_tok, max_req).total; }

// Fewest tokens of a portion for which expanding pays: per cached token and head the absorbed form multiplies 2 r_p
// numbers per query, the expanded one dim + v_dim per query plus r_p (dim + v_dim) for the expansion itself.
static int layer_expand_min(const StackLayer &L) {
    const int t = tuning().expand_min;
    if (t < 0 || !expanded_attn_supported(L.dim_p, L.vdim_p)) return 1 << 30;
    if (t > 0) return t < 2 ? 2 : t;
    const long kv = L.dim_p + L.vdim_p, gain = 2l * L.r_p - kv;
    if (gain <= 0) return 1 << 30;
    const long n = L.r_p * kv / gain + 1;
    return n < 16 ? 16 : (int)n;
}
static int round_expand_min(const Stack &S) {
    int m = 2;  // one decision per request and round: the most demanding layer decides
    for (const StackLayer &L : S.layers) { const int v = layer_expand_min(L); if (v > m) m = v; }
    return m;
}

// Split-KV depth of the absorbed attention for a round: enough CTAs to fill the SMs once (a CTA takes most of an SM's shared
// memory) when every context is full, fixed per round shape so that captured rounds stay valid.
static int attn_splits_for(const lcu_ctx *c, int blocks) {
    if (c->dt == LCU_F32) return 1;
    const int tiles = (c->desc.nctx + 63) / 64;
    int z = sm_count() / (blocks > 0 ? blocks : 1);
    if (z > 32) z = 32;
    if (z > tiles) z = tiles;
    return z < 1 ? 1 : z;
}

static int check_layer(const lcu_model_desc &d, const lcu_layer_desc *layers, int i) {
    const lcu_layer_desc &l = layers[i];
    LCU_REQUIRE((l.pre_norm != 0) == (layers[0].pre_norm != 0), "layer %d: pre-norm and post-norm layers in one model", i);
    if (!l.pre_norm) {
        LCU_REQUIRE(l.mixer == LCU_MIX_LATENT, "layer %d: unknown mixer %d", i, l.mixer);
        LCU_REQUIRE(l.heads > 0 && l.dim > 0 && l.v_dim > 0 && l.q_rank > 0 && l.kv_rank > 0 && l.ff >= 0, "layer %d: non-positive size", i);
        LCU_REQUIRE(l.kv_rank <= 512 && l.dim <= 512, "layer %d: latent of %d, head size %d (at most 512)", i, l.kv_rank, l.dim);
        LCU_REQUIRE(l.ff == 0 || l.ff_act == LCU_ACT_XIELU, "layer %d: unknown activation %d", i, l.ff_act);
        LCU_REQUIRE(!l.add_embed && !l.add_step, "layer %d: additions to the residual stream need pre-norm layers", i);
    } else {
        const int most = MIX_MAX_HEAD, rec = l.mixer & (LCU_MIX_DELTA | LCU_MIX_SSD | LCU_MIX_GLA);
        LCU_REQUIRE(l.mixer > 0 && (l.mixer & ~(LCU_MIX_ATTENTION | LCU_MIX_DELTA | LCU_MIX_SSD | LCU_MIX_GLA)) == 0 && (rec & (rec - 1)) == 0,
                    "layer %d: unknown mixer %d", i, l.mixer);
        LCU_REQUIRE(l.ff >= 0 && l.shared_ff >= 0 && l.experts >= 0 && !l.token_shift, "layer %d: negative size, or a token shift", i);
        if (l.mixer & LCU_MIX_ATTENTION) {
            LCU_REQUIRE(l.heads > 0 && l.kv_heads > 0 && l.heads % l.kv_heads == 0, "layer %d: %d query heads, %d key heads", i, l.heads, l.kv_heads);
            LCU_REQUIRE(l.dim > 0 && l.dim <= most && l.v_dim > 0 && l.v_dim <= most, "layer %d: head sizes %d / %d (1..%d)", i, l.dim, l.v_dim, most);
            LCU_REQUIRE(l.rot_dims >= 0 && l.rot_dims % 2 == 0 && l.rot_dims <= l.dim && (l.rot_dims == 0 || l.rot_base > 0),
                        "layer %d: %d rotated dimensions of %d, base %g", i, l.rot_dims, l.dim, l.rot_base);
            LCU_REQUIRE(l.rot_dims == 0 || l.rot_factor <= 0 || (l.rot_original > 0 && l.rot_fast > 0 && l.rot_slow > 0 && l.rot_base != 1),
                        "layer %d: frequency scaling by %g needs positive constants", i, l.rot_factor);
            LCU_REQUIRE(l.qk_norm >= 0 && l.qk_norm <= 3 && l.window >= 0, "layer %d: norm %d of queries and keys, window of %d", i, l.qk_norm, l.window);
            LCU_REQUIRE(l.kv_from >= 0 && l.kv_from <= i, "layer %d: keys and values of layer %d", i, l.kv_from - 1);
            if (l.kv_from) {
                const lcu_layer_desc &o = layers[l.kv_from - 1];
                LCU_REQUIRE((o.mixer & LCU_MIX_ATTENTION) && !o.kv_from && o.kv_heads == l.kv_heads && o.dim == l.dim && o.v_dim == l.v_dim &&
                                o.rot_values == l.rot_values && (!l.rot_values || o.rot_base == l.rot_base),
                            "layer %d: the keys and values of layer %d do not fit", i, l.kv_from - 1);
            }
            LCU_REQUIRE(l.sink >= 0 && l.sink <= 2 && l.keep_first >= 0 && (l.keep_first == 0 || l.window > 0), "layer %d: sink %d, %d first tokens behind a window of %d",
                        i, l.sink, l.keep_first, l.window);
            LCU_REQUIRE(l.conv >= 0 && l.conv <= 64 && (l.conv == 0 || (!l.bias && l.qk_norm != 3)),
                        "layer %d: convolution of %d taps (0..64), beside biases or a norm over all heads", i, l.conv);
            LCU_REQUIRE(!l.rot_values || (l.v_dim % 2 == 0 && l.rot_base > 0 && l.rot_factor <= 0 && (l.rot_dims == 0 || l.rot_adjacent)),
                        "layer %d: rotated values of size %d take neighbouring pairs", i, l.v_dim);
            LCU_REQUIRE(!rec || !(l.conv || l.rot_values || l.head_temp), "layer %d: convolutions, rotated values or factors per head beside a recurrent mixer", i);
        }
        if (rec) {
            LCU_REQUIRE(l.delta_heads > 0 && l.delta_kv_heads > 0 && l.delta_heads % l.delta_kv_heads == 0, "layer %d: %d value heads, %d key heads", i,
                        l.delta_heads, l.delta_kv_heads);
            LCU_REQUIRE(l.delta_dim > 0 && l.delta_dim <= most && l.delta_v_dim > 0 && l.delta_v_dim <= most, "layer %d: head sizes %d / %d (1..%d)", i,
                        l.delta_dim, l.delta_v_dim, most);
            LCU_REQUIRE(rec == LCU_MIX_GLA || (l.delta_conv >= 1 && l.delta_conv <= 64), "layer %d: convolution of %d taps (1..64)", i, l.delta_conv);
            LCU_REQUIRE(rec != LCU_MIX_SSD || (l.norm_parts > 0 && l.delta_heads * l.delta_v_dim % l.norm_parts == 0), "layer %d: norm of %d values in %d parts", i,
                        l.delta_heads * l.delta_v_dim, l.norm_parts);
            LCU_REQUIRE(rec != LCU_MIX_GLA || (l.gate_rank > 0 && l.gate_rank <= 1024 && l.gate_tau > 0 && l.delta_kv_heads == l.delta_heads),
                        "layer %d: decays of rank %d, tau %g, %d key heads for %d", i, l.gate_rank, l.gate_tau, l.delta_kv_heads, l.delta_heads);
        }
        LCU_REQUIRE((l.mixer & LCU_MIX_ATTENTION) == 0 || rec == 0 || (rec == LCU_MIX_DELTA) == (l.post_norm == 0),
                    "layer %d: side by side, outputs of a delta rule are normed one by one, those of other mixers added ahead of a norm", i);
        const bool ff = l.ff > 0 || l.shared_ff > 0;
        LCU_REQUIRE(!ff || l.ff_act == LCU_ACT_RELU2 || l.ff_act == LCU_ACT_GLU || l.ff_act == LCU_ACT_POLYNORM, "layer %d: unknown activation %d", i, l.ff_act);
        LCU_REQUIRE(!l.ff_bias || (l.ff > 0 && l.ff_act == LCU_ACT_POLYNORM), "layer %d: biases of activation %d", i, l.ff_act);
        LCU_REQUIRE(l.experts == 0 ? l.shared_ff == 0 && l.identity == 0 : (l.ff_act == LCU_ACT_GLU && l.ff > 0 && l.identity >= 0 && l.top > 0 && l.top <= l.experts + l.identity),
                    "layer %d: %d experts, %d per token, widths %d and %d", i, l.experts, l.top, l.ff, l.shared_ff);
        LCU_REQUIRE(l.experts <= 4096 && l.identity <= 4096 && l.experts * 12 + MOE_SMALL_ROUND * l.top * 8 <= 48 * 1024, "layer %d: %d experts, %d per token", i, l.experts, l.top);
        LCU_REQUIRE((l.route_softmax && l.experts && !l.post_norm) || (!l.route_softmax && !l.identity), "layer %d: weights on the outputs of experts take a softmax and no norm on them", i);
        LCU_REQUIRE(!l.parallel_ff || (!l.post_norm && !((l.mixer & LCU_MIX_ATTENTION) && rec) && !l.shared_ff && layers[0].pair_buckets == 0),
                    "layer %d: a feed-forward beside two mixers, a shared expert, norms on outputs or an embedding of pairs", i);
        LCU_REQUIRE(!ff || l.ff_act != LCU_ACT_GLU || (l.glu_limit > 0 && (l.shared_ff == 0 || l.shared_limit > 0)), "layer %d: limit %g of a gated activation", i, l.glu_limit);
        LCU_REQUIRE((l.post_norm != 0) == (layers[0].post_norm != 0), "layer %d: norms on outputs in some layers only", i);
    }
    if (i == 0)
        LCU_REQUIRE(l.pair_buckets >= 0 && l.pair_prev >= 0 && l.pair_cur >= 0 && (l.pair_buckets == 0 || (l.pre_norm && l.pair_prev < l.pair_buckets && l.pair_cur < l.pair_buckets)),
                    "embedding of token pairs: %d buckets, factors %d and %d", l.pair_buckets, l.pair_prev, l.pair_cur);
    if (i == 0) LCU_REQUIRE(l.logit_cap >= 0, "logits capped at %g", l.logit_cap);
    LCU_REQUIRE(l.weights_of >= -1 && l.weights_of < d.n_layers && l.weights_of != i, "layer %d uses the weights of layer %d", i, l.weights_of);
    return LCU_OK;
}

// Fewest split CTAs per SM that keep a decode round's copies in flight: two waves of what fits.
static int gqa_target_ctas(const StackLayer &L) { return 2 * sm_count() * gqa_short_ctas_per_sm(L.dim_p, L.vdim_p); }
int gqa_splits_for(const lcu_ctx *c, const StackLayer &L, int reqs, int len) {
    const int ctas = reqs * L.d.kv_heads * gqa_row_tiles(L.d.heads, L.d.kv_heads, len);
    const int some = L.d.window + L.d.keep_first + len, seen = L.d.window > 0 && some < c->desc.nctx ? some + 63 : c->desc.nctx, units = (seen + 63) / 64;
    int z = ctas > 0 ? gqa_target_ctas(L) / ctas : 1;
    if (z > 64) z = 64;
    if (z > units) z = units;
    return z < 1 ? 1 : z;
}

// (cos, sin) of every position and rotated pair, angles in f64; YaRN: frequencies of fewer than `slow` turns in `original`
// positions are divided by the factor, those of more than `fast` stay, a linear ramp over the pair's index lies between, and
// both functions are scaled by 0.1 ln(factor) + 1.
static int make_rot_table(Stack *S, Stack::RotTable t, int nctx, const float2 **out) {
    for (const Stack::RotTable &o : S->rot_tables)
        if (o.dims == t.dims && o.base == t.base && o.factor == t.factor && o.original == t.original && o.fast == t.fast && o.slow == t.slow) {
            *out = o.dev;
            return LCU_OK;
        }
    const int half = t.dims / 2;
    std::vector<double> freq(half);
    double gain = 1.0;
    for (int i = 0; i < half; ++i) freq[i] = pow(t.base, -2.0 * i / t.dims);
    if (t.factor > 0) {
        auto index_of = [&](double turns) { return t.dims * log(t.original / (2.0 * M_PI * turns)) / (2.0 * log(t.base)); };
        const double lo = fmax(floor(index_of(t.fast)), 0.0), hi = fmin(ceil(index_of(t.slow)), t.dims - 1.0);
        for (int i = 0; i < half; ++i) {
            const double ramp = fmin(fmax((i - lo) / fmax(hi - lo, 0.001), 0.0), 1.0);
            freq[i] = freq[i] / t.factor * ramp + freq[i] * (1.0 - ramp);
        }
        gain = 0.1 * log(t.factor) + 1.0;
    }
    std::vector<float2> host((size_t)nctx * half);
    for (int p = 0; p < nctx; ++p)
        for (int i = 0; i < half; ++i) host[(size_t)p * half + i] = make_float2((float)(cos(p * freq[i]) * gain), (float)(sin(p * freq[i]) * gain));
    float2 *dev = nullptr;
    LCU_CHECK_CUDA(cudaMalloc(reinterpret_cast<void **>(&dev), host.size() * sizeof(float2)));
    t.dev = dev;
    S->rot_tables.push_back(t);
    LCU_CHECK_CUDA(cudaMemcpy(dev, host.data(), host.size() * sizeof(float2), cudaMemcpyHostToDevice));
    *out = dev;
    return LCU_OK;
}

int stack_create(lcu_ctx *c, const lcu_layer_desc *layers) {
    const lcu_model_desc &d = c->desc;
    for (int i = 0; i < d.n_layers; ++i) {
        int rc = check_layer(d, layers, i);
        if (rc) return rc;
    }
    Stack *S = new Stack();
    c->stack = S;
    S->d_p = stack_pad(d.d, 64);
    S->vocab_p = stack_pad(d.vocab, 8);
    S->layers.resize(d.n_layers);
    S->w.resize(d.n_layers);
    size_t off = 0;
    int max_lat = 0, max_qr = 0, max_q = 0, max_hr = 0, max_hv = 64, max_ff = 64, max_kv = 0;
    int max_dk = 0, max_dv = 0, max_coef = 0, max_tail = 0, max_dhv = 0, max_vp = 0, max_top = 0, max_ep = 0, max_eff = 0, max_z = 0;
    size_t conv_total = 0, mat_total = 0;  // f32 values of recurrent state per slot
    S->pre_norm = layers[0].pre_norm != 0;
    bool any_shift = false, any_parallel = false, any_rec = layers[0].pair_buckets > 0, can_expand = c->dt != LCU_F32 && !S->pre_norm;
    for (int i = 0; i < d.n_layers; ++i) {
        StackLayer &L = S->layers[i];
        L.d = layers[i];
        L.src = i;
        for (int hops = 0; layers[L.src].weights_of >= 0; ++hops) {
            LCU_REQUIRE(hops < d.n_layers, "layer %d: the shared weights form a circle", i);
            L.src = layers[L.src].weights_of;
        }
        const lcu_layer_desc &o = layers[L.src];
        LCU_REQUIRE(o.heads == L.d.heads && o.dim == L.d.dim && o.v_dim == L.d.v_dim && o.q_rank == L.d.q_rank && o.kv_rank == L.d.kv_rank &&
                        o.out_gate == L.d.out_gate && o.ff == L.d.ff && o.token_shift == L.d.token_shift && o.mixer == L.d.mixer &&
                        o.kv_heads == L.d.kv_heads && o.bias == L.d.bias && o.delta_heads == L.d.delta_heads &&
                        o.delta_kv_heads == L.d.delta_kv_heads && o.delta_dim == L.d.delta_dim && o.delta_v_dim == L.d.delta_v_dim &&
                        o.delta_conv == L.d.delta_conv && o.qk_norm == L.d.qk_norm && o.kv_from == L.d.kv_from && o.norm_parts == L.d.norm_parts &&
                        o.gate_rank == L.d.gate_rank && o.experts == L.d.experts && o.shared_ff == L.d.shared_ff && o.ff_act == L.d.ff_act &&
                        o.conv == L.d.conv && o.sink == L.d.sink && o.head_temp == L.d.head_temp && o.ff_bias == L.d.ff_bias &&
                        o.route_softmax == L.d.route_softmax && o.identity == L.d.identity,
                    "layer %d differs from layer %d whose weights it uses", i, L.src);
        auto up = [](int &m, int v) { if (v > m) m = v; };
        L.ff_p = stack_pad(L.d.ff, 64);
        L.c_off = off;
        up(max_ff, L.ff_p);
        if (L.latent()) {
            L.dim_p = stack_pad(L.d.dim, 16);
            L.vdim_p = stack_pad(L.d.v_dim, 16);
            L.qr_p = stack_pad(L.d.q_rank, 64);
            L.r_p = stack_pad(L.d.kv_rank, 64);
            L.g_p = L.d.out_gate ? stack_pad(L.d.heads, 8) : 0;
            L.hv_p = stack_pad(L.d.heads * L.vdim_p, 64);
            off += (size_t)L.r_p * c->geom.page_tokens;
            any_shift = any_shift || L.d.token_shift;
            can_expand = can_expand && expanded_attn_supported(L.dim_p, L.vdim_p);
            up(max_hr, L.d.heads * L.r_p); up(max_kv, L.kv_cols()); up(S->max_heads, L.d.heads); up(S->max_r, L.r_p);
            up(max_q, L.d.heads * L.dim_p);
        }
        if (L.attention()) {
            L.dim_p = stack_pad(L.d.dim, 16);
            L.vdim_p = stack_pad(L.d.v_dim, 16);
            L.hv_p = stack_pad(L.d.heads * L.vdim_p, 64);
            L.att_rows = L.d.heads * L.dim_p + (L.own_kv() ? L.d.kv_heads * (L.dim_p + L.vdim_p) : 0);
            L.g_p = L.d.out_gate ? stack_pad(L.d.heads, 8) : 0;
            L.kv_src = L.own_kv() ? i : L.d.kv_from - 1;
            if (L.own_kv()) off += (size_t)L.d.kv_heads * (L.dim_p + L.vdim_p) * c->geom.page_tokens;
            else L.c_off = S->layers[L.kv_src].c_off;
            up(max_q, L.d.heads * L.dim_p); up(max_vp, L.vdim_p);
            if (gqa_target_ctas(L) > S->gqa_ctas) S->gqa_ctas = gqa_target_ctas(L);
            int rc = LCU_OK;
            if (L.d.rot_dims)
                rc = make_rot_table(S, {L.d.rot_dims, L.d.rot_base, L.d.rot_factor, L.d.rot_original, L.d.rot_fast, L.d.rot_slow, nullptr}, d.nctx, &L.rot);
            if (!rc && L.d.rot_values) rc = make_rot_table(S, {L.d.v_dim, L.d.rot_base, 0.0, 0.0, 0.0, 0.0, nullptr}, d.nctx, &L.vrot);
            if (rc) return rc;
            if (L.d.conv > 1) {
                L.conv_off = conv_total;
                conv_total += (size_t)(L.d.conv - 1) * L.att_rows;
                any_rec = true;
            }
        }
        any_parallel = any_parallel || L.parallel();
        if (L.poly()) up(max_z, L.ff_p);
        if (L.recurrent()) {
            L.dk_p = stack_pad(L.d.delta_dim, 32);
            L.dv_p = stack_pad(L.d.delta_v_dim, 16);
            L.dh_p = stack_pad(L.d.delta_heads, 8);
            L.dhv_p = stack_pad(L.d.delta_heads * L.dv_p, 64);
            L.conv_off = conv_total;
            if (L.conv_channels()) conv_total += (size_t)(L.d.delta_conv - 1) * L.conv_channels();
            if (L.gla()) L.rank_p = stack_pad(L.d.gate_rank, 8);
            L.mat_off = mat_total;
            mat_total += (size_t)L.d.delta_heads * L.dv_p * L.dk_p;
            any_rec = true;
            const int coef = L.delta() ? DELTA_COEF * SCAN_BLOCK / DELTA_BLOCK : SCAN_COEF;
            up(max_coef, L.d.delta_heads * coef);
            if (L.gla()) up(max_tail, L.d.delta_heads * L.dk_p);
            up(max_dk, L.d.delta_kv_heads * L.dk_p); up(max_dv, L.d.delta_heads * L.dv_p); up(max_dhv, L.dhv_p);
        }
        if (L.d.shared_ff) { L.sff_p = stack_pad(L.d.shared_ff, 64); up(max_ff, L.sff_p); }
        if (L.d.experts) {
            L.e_p = stack_pad(L.d.experts + L.d.identity, 8);
            up(max_ep, L.e_p); up(max_top, L.d.top); up(max_eff, L.ff_p); up(S->max_experts, L.d.experts);
        }
        up(max_lat, L.in_rows()); up(max_qr, L.qr_p); up(max_hv, L.hv_p);
    }
    c->geom.page_elems = off;
    if (off == 0) c->geom.page_elems = 8;  // nothing is cached per token: pages still count tokens
    S->n_slots = any_shift || any_rec ? c->max_seqs : 0;
    c->free_slots.clear();
    for (int i = S->n_slots - 1; i >= 0; --i) c->free_slots.push_back(i);

    const size_t T = (size_t)c->max_tokens, eb = act_bytes(c);
    S->max_rows = c->max_tokens * max_top;
    S->n_tiles = max_top ? moe_max_tiles(S->max_rows, S->max_experts, 64) : 0;
    S->abs_cap = c->max_tokens;
    S->conv_gen = conv_total * S->n_slots;
    S->expand_cap = can_expand ? stack_pad(d.nctx > c->max_tokens ? d.nctx : c->max_tokens, 64) : 0;
    // partial rows: a small round is split so that about one CTA per SM runs, a large one is not split
    size_t rows = 0;
    for (const StackLayer &L : S->layers)
        for (int dec = 0; dec < 2 && L.latent(); ++dec)
            for (int n = 1; n <= c->max_tokens; n = n < 64 ? n + 1 : (n == c->max_tokens ? n + 1 : (2 * n < c->max_tokens ? 2 * n : c->max_tokens))) {
                const int rpb = latent_attn_rows_per_block(L.d.heads, dec != 0, c->dt, c->geom.page_tokens);
                const int blocks = dec ? n * ((L.d.heads + rpb - 1) / rpb) : n * L.d.heads / rpb + 1;
                // between two sampled sizes the split depth does not grow while the rows at most double
                const size_t r = (size_t)(n < 64 || n == c->max_tokens ? n : 2 * n) * L.d.heads * attn_splits_for(c, blocks);
                if (r > rows) rows = r;
            }
    S->part_rows = rows;
    size_t total = 0;
    auto reserve = [&](size_t bytes) { size_t r = total; total += align256(bytes); return r; };
    const size_t o_x0 = reserve(T * S->d_p * 4), o_x1 = reserve(T * S->d_p * 4), o_y = reserve(T * S->d_p * 4), o_lat = reserve(T * max_lat * 4),
                 o_state = reserve(any_shift ? (size_t)2 * d.n_layers * S->n_slots * S->d_p * 4 : 0), o_h = reserve(T * S->d_p * eb), o_cq = reserve(T * max_qr * eb),
                 o_q = reserve(T * max_q * eb), o_qa = reserve(T * max_hr * eb), o_att = reserve(T * max_hv * eb), o_act = reserve(T * max_ff * eb),
                 o_xc = reserve((size_t)S->expand_cap * S->max_r * eb), o_xkv = reserve((size_t)S->expand_cap * max_kv * eb),
                 o_hout = reserve((T > (size_t)c->max_seqs ? T : c->max_seqs) * S->d_p * eb), o_po = reserve(rows * S->max_r * 4),
                 o_pml = reserve(rows * 2 * 4), o_pn = reserve(T * S->max_heads * 4), o_y2 = reserve(S->pre_norm ? T * S->d_p * 4 : 0),
                 o_dq = reserve(T * max_dk * 6), o_dk = reserve(T * max_dk * 6), o_dv = reserve(T * max_dv * 4), o_dg = reserve((T / SCAN_BLOCK + c->max_seqs + 1) * (size_t)max_coef * 4), o_dt = reserve((T / SCAN_BLOCK + c->max_seqs + 1) * (size_t)max_tail * 4),
                 o_att2 = reserve(T * max_dhv * eb), o_conv = reserve(2 * S->conv_gen * 4), o_mat = reserve(mat_total * S->n_slots * 4),
                 o_gp = reserve(gqa_part_floats(S->gqa_ctas, max_vp) * 4), o_gt = reserve((size_t)S->gqa_ctas * 4);
    const size_t R = S->max_rows, o_lt = reserve((size_t)2 * S->n_slots * 4), o_ro = reserve(T * max_ep * 4), o_ye = reserve(R * S->d_p * 4), o_mi = reserve(R * 16), o_mw = reserve(R * 8),
                 o_mc = reserve((size_t)S->max_experts * 4), o_mt = reserve((size_t)S->n_tiles * 16), o_xg = reserve(R * S->d_p * eb), o_ae = reserve(R * max_eff * eb);
    const size_t o_h2 = reserve(any_parallel ? T * S->d_p * eb : 0), o_z = reserve(T * max_z * 4);
    const size_t o_sw = reserve(any_parallel ? c->sk_ws_bytes : 0), o_st = reserve(any_parallel ? 4096 * sizeof(unsigned) : 0);
    LCU_CHECK_CUDA(cudaMalloc(&S->arena, total));
    LCU_CHECK_CUDA(cudaMemset(S->arena, 0, total));  // pads of att (columns past the heads) stay zero from here on
    unsigned char *p = reinterpret_cast<unsigned char *>(S->arena);
    S->x[0] = reinterpret_cast<float *>(p + o_x0); S->x[1] = reinterpret_cast<float *>(p + o_x1);
    S->y = reinterpret_cast<float *>(p + o_y); S->lat = reinterpret_cast<float *>(p + o_lat); S->state = reinterpret_cast<float *>(p + o_state);
    S->h = p + o_h; S->cq = p + o_cq; S->q = p + o_q; S->qa = p + o_qa; S->att = p + o_att; S->act = p + o_act;
    S->xc = p + o_xc; S->xkv = p + o_xkv; S->hout = p + o_hout;
    S->part_o = reinterpret_cast<float *>(p + o_po); S->part_ml = reinterpret_cast<float *>(p + o_pml); S->part_n = reinterpret_cast<int *>(p + o_pn);

    S->y2 = reinterpret_cast<float *>(p + o_y2); S->dq = reinterpret_cast<float *>(p + o_dq); S->dk = reinterpret_cast<float *>(p + o_dk);
    S->dv = reinterpret_cast<float *>(p + o_dv); S->dcoef = reinterpret_cast<float *>(p + o_dg); S->att2 = p + o_att2;
    S->conv_state = reinterpret_cast<float *>(p + o_conv); S->mat_state = reinterpret_cast<float *>(p + o_mat);
    S->gqa_part = reinterpret_cast<float *>(p + o_gp); S->gqa_tickets = reinterpret_cast<unsigned *>(p + o_gt);

    S->dtail = reinterpret_cast<float *>(p + o_dt); S->last_token = reinterpret_cast<uint32_t *>(p + o_lt);
    S->router = reinterpret_cast<float *>(p + o_ro); S->ye = reinterpret_cast<float *>(p + o_ye); S->moe_ints = reinterpret_cast<int *>(p + o_mi);
    S->moe_w = reinterpret_cast<float *>(p + o_mw); S->moe_slot_w = S->moe_w + R; S->moe_count = reinterpret_cast<unsigned *>(p + o_mc);
    S->moe_tiles = reinterpret_cast<int4 *>(p + o_mt); S->xg = p + o_xg; S->act_e = p + o_ae;

    S->h2 = p + o_h2; S->z = reinterpret_cast<float *>(p + o_z);
    S->side_ws = p + o_sw; S->side_tickets = reinterpret_cast<unsigned *>(p + o_st);
    if (any_parallel) {
        int least = 0, greatest = 0;
        LCU_CHECK_CUDA(cudaDeviceGetStreamPriorityRange(&least, &greatest));
        LCU_CHECK_CUDA(cudaStreamCreateWithPriority(&S->side, cudaStreamNonBlocking, greatest));
        LCU_CHECK_CUDA(cudaEventCreateWithFlags(&S->fork, cudaEventDisableTiming));
        LCU_CHECK_CUDA(cudaEventCreateWithFlags(&S->join, cudaEventDisableTiming));
    }

    // every kernel variant a round can launch
    if (S->pre_norm) {
        if (c->dt == LCU_F32) return LCU_OK;
        int rc = gemm_tc_warm(c->dt);
        for (const StackLayer &L : S->layers) {
            GqaArgs g{};
            g.dim_p = L.dim_p; g.vdim_p = L.vdim_p;
            if (!rc && L.attention()) rc = gqa_short_launch(g, nullptr, false, true);
            if (!rc && L.attention()) rc = gqa_long_launch(g, nullptr, true);
            if (!rc) rc = gemv_warm(S->d_p, L.in_rows(), false, c->dt, EPI_STORE_F32);
            if (!rc && L.attention()) rc = gemv_warm(L.hv_p, S->d_p, false, c->dt, EPI_STORE_F32);
            if (!rc && L.recurrent()) rc = gemv_warm(L.dhv_p, S->d_p, false, c->dt, EPI_STORE_F32);
            if (!rc && L.d.experts) rc = gemv_warm(S->d_p, L.e_p, false, c->dt, EPI_STORE_F32);
            else if (!rc && L.d.ff) rc = L.glu() ? gemv_warm(S->d_p, 2 * L.ff_p, false, c->dt, EPI_GLU) : gemv_warm(S->d_p, L.ff_p, false, c->dt, L.poly() ? EPI_STORE_F32 : EPI_RELU2);
            if (!rc && L.d.ff && !L.d.experts) rc = gemv_warm(L.ff_p, S->d_p, false, c->dt, EPI_STORE_F32);
        }
        if (!rc) rc = gemv_warm(S->d_p, S->vocab_p, false, c->dt, S->caps() ? EPI_CAP : EPI_STORE);
        if (!rc) rc = gemv_warm(S->d_p, S->vocab_p, false, c->dt, S->caps() ? EPI_CAP_F32 : EPI_STORE_F32);
        return rc;
    }
    int rc = latent_attn_launch(LatentAttnArgs{}, c->dt, nullptr, false, true);
    if (rc || c->dt == LCU_F32) return rc;
    rc = head_linear_launch(HeadLinearArgs{}, nullptr, false, true);
    if (!rc) rc = gemm_tc_warm(c->dt);
    for (const StackLayer &L : S->layers) {
        if (rc) break;
        if (S->expand_cap) {
            ExpandedAttnArgs e{};
            e.dim_p = L.dim_p; e.vdim_p = L.vdim_p;
            rc = expanded_attn_launch(e, nullptr, true);
        }
        if (!rc) rc = gemv_warm(S->d_p, L.in_rows(), false, c->dt, EPI_STORE_F32);
        if (!rc) rc = gemv_warm(L.qr_p, L.d.heads * L.dim_p, false, c->dt);
        if (!rc) rc = gemv_warm_stack(S->d_p, L.in_rows(), 0, EPI_STORE_F32, PRO_RESIDUAL);
        if (!rc) rc = gemv_warm_stack(L.qr_p, L.d.heads * L.dim_p, L.r_p, EPI_STORE, PRO_LATENT);
        if (!rc && L.d.ff) rc = gemv_warm_stack(S->d_p, L.ff_p, 0, EPI_XIELU, PRO_RESIDUAL);
        if (!rc) rc = gemv_warm(L.hv_p, S->d_p, false, c->dt, EPI_STORE_F32);
        if (!rc && L.d.ff) rc = gemv_warm(S->d_p, L.ff_p, false, c->dt, EPI_XIELU);
        if (!rc && L.d.ff) rc = gemv_warm(L.ff_p, S->d_p, false, c->dt, EPI_STORE_F32);
    }
    if (!rc) rc = gemv_warm(S->d_p, S->vocab_p, false, c->dt);
    if (!rc) rc = gemv_warm(S->d_p, S->vocab_p, false, c->dt, EPI_STORE_F32);
    return rc;
}

void stack_destroy(lcu_ctx *c) {
    if (!c->stack) return;
    if (c->stack->arena) cudaFree(c->stack->arena);
    if (c->stack->side) cudaStreamDestroy(c->stack->side);
    if (c->stack->fork) cudaEventDestroy(c->stack->fork);
    if (c->stack->join) cudaEventDestroy(c->stack->join);
    for (const Stack::RotTable &t : c->stack->rot_tables) cudaFree(t.dev);
    delete c->stack;
    c->stack = nullptr;
}

// ------------------------------------------------------------------ weights

bool stack_weight_shape(const lcu_ctx *c, int layer, int kind, int *rows, int *cols, int *elem_bytes) {
    const Stack &S = *c->stack;
    *elem_bytes = 2;
    switch (kind) {
    case LCU_W_EMBD: *rows = c->desc.vocab; *cols = S.d_p; return true;
    case LCU_W_LM_HEAD: *rows = S.vocab_p; *cols = S.d_p; return true;
    case LCU_W_OUT_NORM: *rows = 1; *cols = S.pre_norm ? S.d_p : 1; *elem_bytes = 4; return true;
    case LCU_W_PAIR_EMBD: *rows = S.layers[0].d.pair_buckets + 1; *cols = S.d_p; return S.layers[0].d.pair_buckets > 0;
    default: break;
    }
    if (layer < 0 || layer >= c->desc.n_layers) return false;
    const StackLayer &L = S.layers[layer];
    auto f32 = [&](int r, int n, bool has) { *rows = r; *cols = n; *elem_bytes = 4; return has; };
    if (kind == LCU_W_STEP) return f32(1, S.d_p, L.d.add_step != 0);
    if (L.src != layer) return false;
    switch (kind) {
    case LCU_W_UP: *rows = (L.d.experts ? L.d.experts : 1) * (L.glu() ? 2 : 1) * L.ff_p; *cols = S.d_p; return L.d.ff > 0;
    case LCU_W_FF_DOWN: *rows = (L.d.experts ? L.d.experts : 1) * S.d_p; *cols = L.ff_p; return L.d.ff > 0;
    default: break;
    }
    if (S.pre_norm) switch (kind) {
    case LCU_W_MIX_IN: *rows = L.in_rows(); *cols = S.d_p; return true;
    case LCU_W_MIX_BIAS: return f32(1, L.att_rows, L.attention() && L.d.bias);
    case LCU_W_ATT_OUT: *rows = S.d_p; *cols = L.hv_p; return L.attention();
    case LCU_W_DELTA_OUT: *rows = S.d_p; *cols = L.dhv_p; return L.recurrent();
    case LCU_W_QK_GAIN: return L.d.qk_norm == 2 ? f32(1, 2 * L.dim_p, L.attention()) : f32(1, (L.d.heads + (L.own_kv() ? L.d.kv_heads : 0)) * L.dim_p, L.attention() && L.d.qk_norm == 3);
    case LCU_W_CONV: return f32(L.d.delta_conv, L.conv_channels(), L.conv_channels() > 0);
    case LCU_W_CONV_BIAS: return f32(1, L.conv_channels(), L.ssd());
    case LCU_W_DELTA_DECAY: return f32(L.ssd() ? 3 : 2, L.dh_p, L.delta() || L.ssd());
    case LCU_W_GATE_MAP: return f32(L.d.gate_rank + 1, L.d.delta_heads * L.dk_p, L.gla());
    case LCU_W_DELTA_NORM: return f32(1, L.ssd() ? L.d.delta_heads * L.dv_p : L.dv_p, L.recurrent());
    case LCU_W_BRANCH_NORM: return f32(2, S.d_p, L.attention() && L.delta());
    case LCU_W_NORM1: return f32(1, S.d_p, true);
    case LCU_W_NORM2: return f32(1, S.d_p, L.has_ff());
    case LCU_W_POST1: return f32(1, S.d_p, L.d.post_norm != 0);
    case LCU_W_POST2: return f32(1, S.d_p, L.d.post_norm && L.has_ff());
    case LCU_W_ROUTER: *rows = L.e_p; *cols = S.d_p; return L.d.experts > 0;
    case LCU_W_CORRECTION: return f32(1, L.e_p, L.d.route_softmax != 0);
    case LCU_W_ATT_CONV: return f32(L.d.conv, L.att_rows, L.attention() && L.d.conv > 0);
    case LCU_W_SINK: return f32(1, L.d.heads, L.attention() && L.d.sink == 2);
    case LCU_W_HEAD_TEMP: return f32(1, L.d.heads, L.attention() && L.d.head_temp);
    case LCU_W_UP_BIAS: return f32(1, L.ff_p, L.d.ff_bias != 0);
    case LCU_W_DOWN_BIAS: return f32(1, S.d_p, L.d.ff_bias != 0);
    case LCU_W_ACT: return f32(1, 4, L.d.ff > 0 && L.poly());
    case LCU_W_SHARED_UP: *rows = 2 * L.sff_p; *cols = S.d_p; return L.d.shared_ff > 0;
    case LCU_W_SHARED_DOWN: *rows = S.d_p; *cols = L.sff_p; return L.d.shared_ff > 0;
    default: return false;
    }
    switch (kind) {
    case LCU_W_LAT_IN: *rows = L.in_rows(); *cols = S.d_p; return true;
    case LCU_W_Q_NORM: *rows = 1; *cols = L.qr_p; return true;
    case LCU_W_KV_NORM: *rows = 1; *cols = L.r_p; return true;
    case LCU_W_UQ: *rows = L.d.heads * L.dim_p; *cols = L.qr_p; return true;
    case LCU_W_UKT: *rows = L.d.heads * L.r_p; *cols = L.dim_p; return true;
    case LCU_W_UKV: *rows = L.kv_cols(); *cols = L.r_p; return true;
    case LCU_W_LAT_OUT: *rows = S.d_p; *cols = L.hv_p; return true;
    case LCU_W_SHIFT: *rows = 1; *cols = S.d_p; return L.d.token_shift != 0;
    case LCU_W_SCALARS: *rows = 1; *cols = 4; *elem_bytes = 4; return true;
    default: return false;
    }
}

int stack_set_weight(lcu_ctx *c, int layer, int kind, const void *ptr) {
    if (kind == LCU_W_PAIR_EMBD) {
        c->stack->pair_embd = ptr;
        return LCU_OK;
    }
    StackWeights &w = c->stack->w[layer];
    const float *f = reinterpret_cast<const float *>(ptr);
    switch (kind) {
    case LCU_W_MIX_IN: w.in = ptr; break;
    case LCU_W_MIX_BIAS: w.bias = f; break;
    case LCU_W_ATT_OUT: w.att_out = ptr; break;
    case LCU_W_DELTA_OUT: w.delta_out = ptr; break;
    case LCU_W_CONV: w.conv = f; break;
    case LCU_W_DELTA_DECAY: w.decay = f; break;
    case LCU_W_DELTA_NORM: w.delta_norm = f; break;
    case LCU_W_BRANCH_NORM: w.branch_norm = f; break;
    case LCU_W_NORM1: w.norm1 = f; break;
    case LCU_W_NORM2: w.norm2 = f; break;
    case LCU_W_STEP: w.step = f; break;
    case LCU_W_POST1: w.post1 = f; break;
    case LCU_W_POST2: w.post2 = f; break;
    case LCU_W_QK_GAIN: w.qk_gain = f; break;
    case LCU_W_CONV_BIAS: w.conv_bias = f; break;
    case LCU_W_GATE_MAP: w.gate_map = f; break;
    case LCU_W_ROUTER: w.router = ptr; break;
    case LCU_W_CORRECTION: w.correction = f; break;
    case LCU_W_ATT_CONV: w.att_conv = f; break;
    case LCU_W_SINK: w.sink = f; break;
    case LCU_W_HEAD_TEMP: w.head_temp = f; break;
    case LCU_W_UP_BIAS: w.up_bias = f; break;
    case LCU_W_DOWN_BIAS: w.down_bias = f; break;
    case LCU_W_ACT: w.act = f; break;
    case LCU_W_SHARED_UP: w.shared_up = ptr; break;
    case LCU_W_SHARED_DOWN: w.shared_down = ptr; break;
    case LCU_W_LAT_IN: w.in = ptr; break;
    case LCU_W_Q_NORM: w.q_norm = ptr; break;
    case LCU_W_KV_NORM: w.kv_norm = ptr; break;
    case LCU_W_UQ: w.uq = ptr; break;
    case LCU_W_UKT: w.ukt = ptr; break;
    case LCU_W_UKV: w.ukv = ptr; break;
    case LCU_W_LAT_OUT: w.out = ptr; break;
    case LCU_W_UP: w.up = ptr; break;
    case LCU_W_FF_DOWN: w.down = ptr; break;
    case LCU_W_SHIFT: w.shift = ptr; break;
    case LCU_W_SCALARS: w.scalars = reinterpret_cast<const float *>(ptr); break;
    default: set_error("set_weight: unknown kind %d", kind); return LCU_ERR_INVALID;
    }
    return LCU_OK;
}

bool stack_ready(const lcu_ctx *c) {
    const Stack &S = *c->stack;
    if (S.layers[0].d.pair_buckets && !S.pair_embd) {
        set_error("step: the embedding of token pairs is missing");
        return false;
    }
    for (size_t i = 0; i < S.layers.size(); ++i) {
        const StackWeights &w = S.w[i];
        const StackLayer &L = S.layers[i];
        const lcu_layer_desc &d = L.d;
        bool ok = !d.add_step || w.step;
        if (L.src == (int)i) {
            ok = ok && w.in && (!d.ff || (w.up && w.down)) && (!d.token_shift || w.shift);
            if (L.latent()) ok = ok && w.q_norm && w.kv_norm && w.uq && w.ukt && w.ukv && w.out && w.scalars;
            if (L.attention()) ok = ok && w.att_out && (!d.bias || w.bias) && (d.qk_norm < 2 || w.qk_gain) && (!d.conv || w.att_conv) && (d.sink != 2 || w.sink) && (!d.head_temp || w.head_temp);
            ok = ok && (!d.ff_bias || (w.up_bias && w.down_bias)) && (!d.ff || !L.poly() || w.act) && (!d.route_softmax || w.correction);
            if (L.recurrent()) ok = ok && w.delta_out && w.delta_norm && (L.gla() ? w.gate_map != nullptr : w.conv && w.decay) && (!L.ssd() || w.conv_bias);
            if (S.pre_norm) ok = ok && w.norm1 && (!L.has_ff() || w.norm2) && (!(L.attention() && L.delta()) || w.branch_norm);
            if (d.post_norm) ok = ok && w.post1 && (!L.has_ff() || w.post2);
            ok = ok && (!d.experts || w.router) && (!d.shared_ff || (w.shared_up && w.shared_down));
        }
        if (!ok) {
            set_error("step: weights of layer %zu missing", i);
            return false;
        }
    }
    return true;
}

// ------------------------------------------------------------------ the round

int stack_stage(lcu_ctx *c, Round &r, const lcu_req *reqs, unsigned char *H) {
    const Stack &S = *c->stack;
    StackRound &q = r.sr;
    q = StackRound();
    const StackDesc D = stack_desc(r.n_tok, r.n_req);
    unsigned char *B = H + r.L.stack;
    int32_t *first = reinterpret_cast<int32_t *>(B + D.req_first), *pos = reinterpret_cast<int32_t *>(B + D.req_pos),
            *slot = reinterpret_cast<int32_t *>(B + D.req_slot), *afirst = reinterpret_cast<int32_t *>(B + D.abs_first),
            *aid = reinterpret_cast<int32_t *>(B + D.abs_id), *atok = reinterpret_cast<int32_t *>(B + D.abs_tok);
    int4 *xreq = reinterpret_cast<int4 *>(B + D.xreq), *xg = reinterpret_cast<int4 *>(B + D.xgroups);
    int4 *sreq = reinterpret_cast<int4 *>(B + D.sreq), *lreq = reinterpret_cast<int4 *>(B + D.lreq), *dblk = reinterpret_cast<int4 *>(B + D.dblk), *sblk = reinterpret_cast<int4 *>(B + D.sblk);
    int short_max = 1 << 30;  // one decision per request and round: the layer with the largest head groups decides
    for (const StackLayer &L : S.layers)
        if (L.attention()) { const int v = gqa_short_tokens(L.d.heads, L.d.kv_heads); if (v < short_max) short_max = v; }
    const int expand_min = S.expand_cap ? round_expand_min(S) : 1 << 30;
    int t = 0, nx = 0, ng = 0;
    StackRound::Batch cur{0, 0, 0, 0, 0};
    for (int i = 0; i < r.n_req; ++i) {
        const SeqState &sq = c->seqs[reqs[i].seq];
        const int len = (int)reqs[i].len, ctx = (int)reqs[i].pos + len;
        first[i] = t;
        pos[i] = (int)reqs[i].pos;
        slot[i] = sq.slot * 2 + sq.gen;
        if (S.pre_norm) {
            if (len <= short_max) {
                sreq[q.n_short++] = make_int4(i, t, len, pos[i]);
                if (len > q.max_short) q.max_short = len;
            } else {
                lreq[q.n_long++] = make_int4(i, t, len, pos[i]);
                q.long_len.push_back(len);
            }
            for (int j = 0; j < len; j += DELTA_BLOCK)
                dblk[q.n_delta_blocks++] = make_int4(i, t + j, len - j < DELTA_BLOCK ? len - j : DELTA_BLOCK, t / DELTA_BLOCK + i + j / DELTA_BLOCK);
            for (int j = 0; j < len; j += SCAN_BLOCK)
                sblk[q.n_scan_blocks++] = make_int4(i, t + j, len - j < SCAN_BLOCK ? len - j : SCAN_BLOCK, t / SCAN_BLOCK + i + j / SCAN_BLOCK);
        } else if (len < expand_min) {
            aid[q.n_abs_req] = i;
            afirst[q.n_abs_req++] = q.n_abs_tok;
            for (int j = 0; j < len; ++j) atok[q.n_abs_tok++] = t + j;
        } else {
            if (cur.n_req && cur.n_rows + ctx > S.expand_cap) {  // the batch is full (one request always fits)
                q.batches.push_back(cur);
                cur = StackRound::Batch{0, nx, 0, ng, 0};
            }
            xreq[nx++] = make_int4(i, ctx, cur.n_rows, 0);
            for (int j = 0; j < len; j += EXPAND_GROUP) {
                xg[ng++] = make_int4(t + j, len - j < EXPAND_GROUP ? len - j : EXPAND_GROUP, pos[i] + j, cur.n_rows);
                ++cur.n_groups;
            }
            cur.n_rows += ctx;
            ++cur.n_req;
        }
        t += len;
    }
    first[r.n_req] = t;
    afirst[q.n_abs_req] = q.n_abs_tok;
    if (cur.n_req) q.batches.push_back(cur);
    q.abs_decode = r.decode_only;
    return LCU_OK;
}

bool stack_pdl(const lcu_ctx *c, int n_tok) { return tuning().stack_pdl && c->dt != LCU_F32 && n_tok <= 256; }

int stack_layers(lcu_ctx *c, const Round &r, cudaStream_t s, int *count) {
    Stack &S = *c->stack;
    if (S.pre_norm) return pre_norm_layers(c, r, s, count);
    const lcu_model_desc &d = c->desc;
    const int dt = c->dt, n = r.n_tok;
    const size_t eb = act_bytes(c);
    const bool pdl = stack_pdl(c, n);
    Launcher L{c, s, count, pdl};
    unsigned char *D = c->desc_dev, *B = D + r.L.stack;
    const StackDesc o = stack_desc(r.n_tok, r.n_req);
    const uint32_t *tokens = reinterpret_cast<const uint32_t *>(D + r.L.tokens), *pos = reinterpret_cast<const uint32_t *>(D + r.L.pos);
    const int32_t *tok_req = reinterpret_cast<const int32_t *>(D + r.L.tok_req), *page_table = reinterpret_cast<const int32_t *>(D + r.L.page_table);
    auto i32 = [&](size_t off) { return reinterpret_cast<const int32_t *>(B + off); };
    const StackRound &q = r.sr;
    gemm_tc_set_scratch(c->sk_ws, c->sk_ws_bytes, c->sk_tickets, 4096, c->dev_status);
    int rc, cur = 0;

    MixInputArgs mi{};
    mi.n_tok = n; mi.d = d.d; mi.d_p = S.d_p; mi.eps = d.eps;
    mi.state_gen_stride = (size_t)d.n_layers * S.n_slots * S.d_p;
    mi.tok_req = tok_req; mi.req_first = i32(o.req_first); mi.req_pos = i32(o.req_pos); mi.req_slot = i32(o.req_slot);
    mi.h = S.h;
    // rounds of one or two decoded tokens: norms, residual and token shift run as prologues of the projections that read them,
    // up to the width where the rows every CTA then re-reads cost more than the launches saved (batch 1, 8 layers: width 2048
    // 0.410 -> 0.409 ms per step with 23 launches less, width 4096 0.773 -> 0.793 ms)
    bool fused = (tuning().stack_fuse == 2 || (tuning().stack_fuse == 1 && S.d_p <= 2048)) && dt == LCU_BF16 && r.decode_only && gemv_stack_fits(S.d_p, n, PRO_RESIDUAL);
    for (const StackLayer &Y : S.layers) fused = fused && gemv_stack_fits(Y.qr_p, n, PRO_LATENT);
    L.weights_first = !fused;
    GemvArgs pend{};  // the prologue the next projection of x takes (fused rounds)
    bool pending = false;
    pend.pos = pos; pend.tok_seq = tok_req; pend.page_table = page_table; pend.pt_stride = c->pt_stride; pend.eps = d.eps;
    // x (and the shifted input of layer `next`, if there is one) after a sublayer's output y; layer -1: the embedding
    auto residual = [&](const float *gain, int next, bool mixer_input) -> int {
        MixInputArgs a = mi;
        if (gain) {
            a.x_in = S.x[cur]; a.y = S.y; a.gain = gain;
            cur ^= 1;
        } else {
            a.embd = c->embd; a.tokens = tokens;
        }
        a.x_out = S.x[cur];
        if (mixer_input) {
            if (next >= d.n_layers) a.h = nullptr;  // the head reads x itself
            else if (S.layers[next].d.token_shift) {
                a.shift = S.w[S.layers[next].src].shift;
                a.state = S.state + (size_t)next * S.n_slots * S.d_p;
            }
        }
        if (fused && gain && a.h) {
            StackPrologue &p = pend.pro;
            p = StackPrologue{};
            p.x_in = a.x_in; p.y_in = a.y; p.x_out = a.x_out; p.gain = gain; p.n_true = d.d; p.shift = a.shift; p.state = a.state;
            p.state_gen_stride = a.state_gen_stride; p.req_pos = a.req_pos; p.req_slot = a.req_slot;
            pending = true;
            return LCU_OK;
        }
        ++*count;
        return op_mix_input(a, dt, s, pdl);
    };
    // projection of the residual stream (or its shifted form), through the pending prologue if there is one
    auto project = [&](const void *w, int out, void *y, int epilogue, const float *act_pq) -> int {
        const bool p = pending;
        pending = false;
        return L.linear(w, S.d_p, out, S.h, n, y, out, epilogue, act_pq, p ? PRO_RESIDUAL : PRO_NONE, p ? &pend : nullptr);
    };
    rc = residual(nullptr, 0, true);
    if (rc) return rc;
    for (int l = 0; l < d.n_layers; ++l) {
        const StackLayer &Y = S.layers[l];
        const StackWeights &W = S.w[Y.src];
        const int heads = Y.d.heads, lat_stride = Y.in_rows(), q_stride = heads * Y.dim_p;
        // --- both latents and the head gates in one projection; norms; append to the cache; queries
        rc = project(W.in, lat_stride, S.lat, EPI_STORE_F32, nullptr);
        if (rc) return rc;
        LatentNormArgs ln{};
        ln.lat = S.lat; ln.stride = lat_stride; ln.n_tok = n; ln.q_rank = Y.d.q_rank; ln.qr_p = Y.qr_p; ln.kv_rank = Y.d.kv_rank; ln.r_p = Y.r_p;
        ln.q_norm = W.q_norm; ln.kv_norm = W.kv_norm; ln.eps = d.eps; ln.cq = S.cq;
        ln.pool = c->pool; ln.page_elems = c->geom.page_elems; ln.c_off = Y.c_off; ln.page_shift = c->geom.page_shift;
        ln.tok_req = tok_req; ln.pos = pos; ln.page_table = page_table; ln.pt_stride = c->pt_stride;
        if (fused) {
            GemvArgs g = pend;
            g.pro = StackPrologue{};
            g.pro.lat = S.lat; g.pro.lat_stride = lat_stride; g.pro.n_true = Y.d.q_rank; g.pro.kv_rank = Y.d.kv_rank; g.pro.r_p = Y.r_p;
            g.pro.q_norm = W.q_norm; g.pro.kv_norm = W.kv_norm; g.pro.pool = c->pool; g.pro.page_elems = c->geom.page_elems;
            g.pro.c_off = Y.c_off; g.pro.page_shift = c->geom.page_shift;
            rc = L.linear(W.uq, Y.qr_p, q_stride, S.cq, n, S.q, q_stride, EPI_STORE, nullptr, PRO_LATENT, &g);
        } else {
            rc = latent_norm_launch(ln, dt, s, pdl);
            if (rc) return rc;
            ++*count;
            rc = L.linear(W.uq, Y.qr_p, q_stride, S.cq, n, S.q, q_stride, EPI_STORE);
        }
        if (rc) return rc;
        const float *gate = Y.d.out_gate ? S.lat + Y.qr_p + Y.r_p : nullptr;
        const unsigned char *uv = reinterpret_cast<const unsigned char *>(W.ukv) + (size_t)heads * Y.dim_p * Y.r_p * 2;

        // --- absorbed form: queries into latent space, attention over the cached latents, value map of the merged rows
        if (q.n_abs_tok) {
            const int rpb = latent_attn_rows_per_block(heads, q.abs_decode, dt, c->geom.page_tokens);
            const int blocks = q.abs_decode ? q.n_abs_tok * ((heads + rpb - 1) / rpb) : q.n_abs_tok * heads / rpb + 1;
            const int splits = attn_splits_for(c, blocks);
            LCU_REQUIRE((size_t)q.n_abs_tok * heads * splits <= S.part_rows, "step: attention partials of %d tokens do not fit", q.n_abs_tok);
            LatentAttnArgs a{};
            a.q = S.qa; a.pool = c->pool; a.page_elems = c->geom.page_elems; a.c_off = Y.c_off; a.page_shift = c->geom.page_shift; a.n_pages = c->n_pages;
            a.page_table = page_table; a.pt_stride = c->pt_stride; a.req_first = i32(o.abs_first); a.req_id = i32(o.abs_id); a.req_pos = i32(o.req_pos);
            a.n_req = q.n_abs_req; a.n_tok = q.n_abs_tok; a.decode = q.abs_decode; a.heads = heads; a.r_p = Y.r_p; a.scale = Y.d.scale;
            a.part_o = S.part_o; a.part_ml = S.part_ml; a.part_n = S.part_n; a.splits = splits; a.status = c->dev_status;
            if (dt == LCU_F32) {
                LinearF32Args f{};
                f.x = reinterpret_cast<const float *>(S.q); f.stride_x = q_stride; f.head_x = Y.dim_p; f.x_rows = i32(o.abs_tok);
                f.w = W.ukt; f.y = reinterpret_cast<float *>(S.qa); f.stride_y = heads * Y.r_p; f.head_y = Y.r_p;
                f.n = q.n_abs_tok; f.in = Y.dim_p; f.out = Y.r_p; f.heads = heads; f.epilogue = EPI_STORE_F32;
                rc = linear_f32_launch(f, s);
                if (!rc) rc = latent_attn_launch(a, dt, s, pdl);
                f = LinearF32Args{};
                f.x = S.part_o; f.stride_x = heads * Y.r_p; f.head_x = Y.r_p; f.w = uv;
                f.y = reinterpret_cast<float *>(S.att); f.stride_y = Y.hv_p; f.head_y = Y.vdim_p; f.y_rows = i32(o.abs_tok);
                f.n = q.n_abs_tok; f.in = Y.r_p; f.out = Y.vdim_p; f.heads = heads; f.epilogue = EPI_STORE_F32;
                f.gate = gate; f.stride_gate = lat_stride;
                if (!rc) rc = linear_f32_launch(f, s);
            } else {
                HeadLinearArgs f{};
                f.x = S.q; f.stride_x = q_stride; f.head_x = Y.dim_p; f.x_rows = i32(o.abs_tok); f.w = W.ukt;
                f.y = S.qa; f.stride_y = heads * Y.r_p; f.head_y = Y.r_p; f.n = q.n_abs_tok; f.in = Y.dim_p; f.out = Y.r_p; f.heads = heads;
                rc = head_linear_launch(f, s, pdl);
                if (!rc) rc = latent_attn_launch(a, dt, s, pdl);
                f = HeadLinearArgs{};
                f.w = uv; f.y = S.att; f.stride_y = Y.hv_p; f.head_y = Y.vdim_p; f.y_rows = i32(o.abs_tok);
                f.n = q.n_abs_tok; f.in = Y.r_p; f.out = Y.vdim_p; f.heads = heads;
                f.part_o = S.part_o; f.part_ml = S.part_ml; f.part_n = S.part_n; f.splits = splits;
                f.gate = gate; f.stride_gate = lat_stride;
                if (!rc) rc = head_linear_launch(f, s, pdl);
            }
            if (rc) return rc;
            *count += 3;
        }
        // --- expanded form, a batch of requests at a time
        for (const StackRound::Batch &b : q.batches) {
            const int4 *xreq = reinterpret_cast<const int4 *>(B + o.xreq) + b.req0, *xg = reinterpret_cast<const int4 *>(B + o.xgroups) + b.group0;
            rc = latent_gather_launch(S.xc, c->pool, c->geom.page_elems, Y.c_off, c->geom.page_shift, page_table, c->pt_stride, xreq, b.n_req,
                                      b.n_rows, Y.r_p, s);
            if (!rc) rc = L.linear(W.ukv, Y.r_p, Y.kv_cols(), S.xc, b.n_rows, S.xkv, Y.kv_cols(), EPI_STORE);
            if (rc) return rc;
            ExpandedAttnArgs a{};
            a.q = S.q; a.stride_q = q_stride; a.kv = S.xkv; a.stride_kv = Y.kv_cols(); a.o = S.att; a.stride_o = Y.hv_p;
            a.groups = xg; a.n_groups = b.n_groups; a.heads = heads; a.dim_p = Y.dim_p; a.vdim_p = Y.vdim_p; a.scale = Y.d.scale;
            a.gate = gate; a.stride_gate = lat_stride;
            rc = expanded_attn_launch(a, s);
            if (rc) return rc;
            *count += 2;
        }
        // --- output projection, norm of its result, residual
        rc = L.linear(W.out, Y.hv_p, S.d_p, S.att, n, S.y, S.d_p, EPI_STORE_F32);
        if (!rc) rc = residual(W.scalars, l + 1, Y.d.ff == 0);
        if (rc || !Y.d.ff) {
            if (rc) return rc;
            continue;
        }
        // --- feed-forward
        rc = project(W.up, Y.ff_p, S.act, EPI_XIELU, W.scalars + 2);
        if (!rc) rc = L.linear(W.down, Y.ff_p, S.d_p, S.act, n, S.y, S.d_p, EPI_STORE_F32);
        if (!rc) rc = residual(W.scalars + 1, l + 1, true);
        if (rc) return rc;
    }
    (void)eb;
    c->x = S.x[cur];
    return LCU_OK;
}

int stack_head(lcu_ctx *c, const Round &r, const uint32_t *rows, int n_rows, float *out_f32, cudaStream_t s, int *count) {
    if (n_rows <= 0) return LCU_OK;
    Stack &S = *c->stack;
    const bool pdl = stack_pdl(c, r.n_tok);
    int rc = op_scalar_norm_rows(S.hout, reinterpret_cast<const float *>(c->x), rows, n_rows, c->desc.d, S.d_p,
                                 reinterpret_cast<const float *>(c->out_norm), S.pre_norm, c->desc.eps, c->dt, s, pdl);
    if (rc) return rc;
    ++*count;
    Launcher L{c, s, count, pdl};
    void *y = out_f32 ? reinterpret_cast<void *>(out_f32) : c->logits;
    const lcu_layer_desc &d = S.layers[0].d;
    L.cap = CapArgs{d.logit_scale ? d.logit_scale : 1.f, d.logit_cap};
    const int f32 = S.caps() ? EPI_CAP_F32 : EPI_STORE_F32, act = S.caps() ? EPI_CAP : EPI_STORE;
    return L.linear(c->lm_head, S.d_p, S.vocab_p, S.hout, n_rows, y, S.vocab_p, out_f32 ? f32 : act);
}

// Algorithmic bytes of a round: the weights the round's forms of attention touch, the head, cached rows and state.
double stack_step_bytes(const lcu_ctx *c, const lcu_req *reqs, int n_req, int n_out) {
    const Stack &S = *c->stack;
    const double wb = 2.0, eb = (double)act_bytes(c);
    double bytes = n_out ? (double)S.vocab_p * S.d_p * wb : 0.0;
    for (const StackLayer &L : S.layers) {
        const lcu_layer_desc &d = L.d;
        double ff = (L.glu() ? 3.0 : 2.0) * L.ff_p * S.d_p;
        if (d.experts) {  // the experts that this many tokens use when they choose evenly
            double tokens = 0.0;
            for (int i = 0; i < n_req; ++i) tokens += reqs[i].len;
            ff *= d.experts * (1.0 - pow(1.0 - (double)d.top / (d.experts + d.identity), tokens));
        }
        bytes += wb * ((double)L.in_rows() * S.d_p + ff + 3.0 * L.sff_p * S.d_p + (double)L.e_p * S.d_p + (double)S.d_p * (L.hv_p + L.dhv_p));
        if (L.latent()) bytes += wb * ((double)d.heads * L.dim_p * L.qr_p + (double)L.kv_cols() * L.r_p);
        const double row = L.latent() ? L.r_p : (L.attention() ? (double)d.kv_heads * (L.dim_p + L.vdim_p) : 0.0);
        for (int i = 0; i < n_req; ++i) {
            for (uint32_t j = 0; j < reqs[i].len; ++j) {
                const uint32_t seen = reqs[i].pos + j + 1;
                const uint32_t most = (uint32_t)(d.window + d.keep_first);
                bytes += (double)(d.window > 0 && seen > most ? most : seen) * row * eb;
            }
            if (L.recurrent()) bytes += 8.0 * d.delta_heads * L.dv_p * L.dk_p;  // matrices read and written
        }
    }
    return bytes;
}

}  // namespace lcu
