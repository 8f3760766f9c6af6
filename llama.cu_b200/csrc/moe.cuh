// Feed-forwards of experts: routing, the lists that group tokens by expert, and the grouped products of small rounds.  Interface
// only; kernels in moe.cu, the grouped products of large rounds are those of gemm_tc.cu and linear_f32.cu with a table of tiles.
#pragma once
#include "common.cuh"
#include "gemv.cuh"

namespace lcu {

constexpr int MOE_SMALL_ROUND = 64;  // tokens up to which a round takes the small form

// A token's (token, rank) pairs become slots: rows sorted by expert.
struct MoeRoute {
    const float *logits;  // [n_tok][experts_p]
    int n_tok, experts, experts_p, top;
    // softmax: scores are the softmax of all logits, those + correction choose, the chosen ones divided by their sum are the weights;
    // otherwise the largest logits choose and their sigmoids are the weights
    int softmax;
    const float *correction;
    int identity;         // experts behind the others that have no matrices: slot_of is -1
    // per (token, rank): expert, its place among the expert's rows, slot; per slot: token, weight
    int *expert, *place, *slot_of, *slot_tok;
    float *weight, *slot_w;  // per (token, rank) and per slot
    unsigned *count;         // [experts] rows of each; large rounds: zero ahead of the routing
    int4 *tiles;             // (expert, first slot, rows, 0); rows == 0 past the last one
    int max_tiles, tile_rows;
    const void *h;           // [n_tok][d_p] activations, and their copies in slot order (large rounds)
    void *xg;
    int d_p;
};
// one launch: routing and lists, a tile per expert in use (small rounds)
int moe_plan_launch(const MoeRoute &a, cudaStream_t s, bool pdl);
// large rounds: routing; then lists, tiles of at most tile_rows rows, activations in slot order
int moe_route_launch(const MoeRoute &a, cudaStream_t s, bool pdl);
int moe_gather_launch(const MoeRoute &a, int dt, cudaStream_t s, bool pdl);
inline int moe_max_tiles(int rows, int experts, int tile_rows) { return rows / tile_rows + (rows < experts ? rows : experts); }

// Products of the experts in use, and of the shared expert (all tokens), for small rounds on mma.sync: weights stream straight into
// fragments, once per 32 rows of a tile.  up: activated products of gate and up rows; down: f32 rows.
struct MoeProduct {
    const int4 *tiles;
    int max_tiles, n_tok;
    int up, shared;          // shared: the first grid row is the shared expert
    const void *w, *ws;      // [expert][out][in], [outs][ins]
    int out, in, outs, ins;
    const void *x, *xs;      // rows in slot order (slot_tok: of the slots' tokens), rows of tokens
    const int *slot_tok;
    const float *slot_w;     // up: factor on a row
    void *y, *ys;
    GluArgs glu, glus;
};
int moe_product_launch(const MoeProduct &a, cudaStream_t s, bool pdl);

}  // namespace lcu
