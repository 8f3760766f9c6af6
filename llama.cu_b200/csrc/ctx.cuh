// The context (one GPU's share of a model) and the descriptor of a round, shared by the translation units that build
// and run rounds: ctx.cu (context, pages, LLaMA layers, head) and stack.cu (models described layer by layer).
#pragma once
#include <map>
#include <vector>

#include "attention.cuh"
#include "common.cuh"
#include "p2p.cuh"
#include "stack.cuh"

struct LayerWeights {
    const void *attn_norm = nullptr, *qkv = nullptr, *o = nullptr, *ffn_norm = nullptr, *gate_up = nullptr,
               *down = nullptr;
};

struct SeqState {
    bool used = false;
    uint32_t len = 0;  // tokens backed by pages
    std::vector<int> pages;
    // recurrent state of a layered model: slot (-1: none), half of the double buffer that holds it, tokens it covers
    int slot = -1;
    int gen = 0;
    uint32_t state_len = 0;
};

struct StepGraph {
    cudaGraphExec_t exec = nullptr;
    int launches = 0;
};

struct lcu_ctx {
    lcu_model_desc desc;
    int device = 0, tp_rank = 0, tp_size = 1;
    void *comm = nullptr;
    int dt = LCU_F16;
    // per-rank shapes
    int nh_l = 0, nkvh_l = 0, di_l = 0, qd = 0, kvd = 0;
    int max_tokens = 0, max_seqs = 0;

    std::vector<LayerWeights> layers;
    const void *embd = nullptr, *out_norm = nullptr, *lm_head = nullptr;
    const float *sin_t = nullptr, *cos_t = nullptr;
    float *own_tables = nullptr;

    // KV pages
    void *pool = nullptr;
    bool own_pool = false;
    lcu::KvGeom geom{};
    int n_pages = 0, pt_stride = 0;
    std::vector<int> free_pages;
    std::vector<SeqState> seqs;

    // arena (one allocation)
    void *arena = nullptr;
    void *x = nullptr, *q = nullptr, *att = nullptr, *act = nullptr, *logits = nullptr, *hbuf = nullptr;
    void *sk_ws = nullptr;
    unsigned *sk_tickets = nullptr;
    size_t sk_ws_bytes = 0;
    bool batched_ok = false;  // tensor-core path for rounds of more than 4 tokens
    void *attn_scratch = nullptr, *sample_ws = nullptr;
    size_t sample_ws_bytes = 0;
    lcu_kv_pair *pre_pairs = nullptr;  // copy of the last round's output pairs (token feedback)
    uint32_t *dev_status = nullptr;
    unsigned char *desc_dev = nullptr;  // per-round descriptor
    size_t desc_cap = 0;
    // pinned staging ring for the descriptor
    static constexpr int RING = 4;
    unsigned char *desc_host[RING] = {nullptr, nullptr, nullptr, nullptr};
    cudaEvent_t desc_event[RING] = {nullptr, nullptr, nullptr, nullptr};
    bool desc_used[RING] = {false, false, false, false};
    int ring_idx = 0;

    // tensor parallelism over peer memory (set up by lcu_p2p_create / lcu_p2p_attach)
    lcu::P2pState p2p;

    // LM head sharded by vocabulary rows under tensor parallelism (peer-memory transport, arg-max rounds)
    bool head_shard = true;           // lcu_set_head_sharding
    lcu_kv_pair *head_local = nullptr;  // this rank's candidates
    uint32_t sticky_status = 0;       // last value lcu_device_status read

    // model described layer by layer (lcu_ctx_create_layers); nullptr for the LLaMA family
    lcu::Stack *stack = nullptr;
    std::vector<int> free_slots;      // recurrent-state slots

    bool use_graph = true;
    std::map<std::vector<int>, StepGraph> graphs;
    int last_launches = 0;
    double last_bytes = 0;
    int last_n_tok = 0, last_n_req = 0;
};

// offsets of the sections of a round descriptor (all 16-byte aligned)
struct DescLayout {
    size_t tokens, pos, tok_req, out_idx, fast_map, args, randoms, page_table, groups, stack, total;
};

namespace lcu {

struct Round {
    int n_tok, n_req, n_fast;
    int n_out;     // rows of logits: one per request, or what lcu_step_logits asks for
    int n_groups;  // token groups for the prefill form of attention (0: decode form)
    bool any_sampling;
    bool decode_only;  // one new token per sequence
    float *logits_f32;  // lcu_step_logits: f32 logits of the asked rows go here, nothing is sampled
    StackRound sr;      // layered models
    DescLayout L;
};

}  // namespace lcu
