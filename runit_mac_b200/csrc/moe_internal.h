// Launchers of the mixture-of-experts building blocks (moe_route.cu, moe_permute.cu).
#pragma once

#include "runit_internal.h"

namespace runit {

int32_t moe_router(runit_ctx* ctx, const float* router_w, const float* x, float* logits, uint32_t E, uint32_t h, uint32_t T);
int32_t moe_topk(runit_ctx* ctx, const float* logits, uint32_t E, uint32_t k, int32_t renorm, uint32_t T, int32_t* idx, float* w);
// rows of ld logits, the first E of a row are the experts'; score: RUNIT_SCORE_*
int32_t moe_topk_rows(runit_ctx* ctx, const void* logits, int32_t logits_f16, uint32_t ld, uint32_t E, uint32_t k, int32_t score,
                      int32_t renorm, uint32_t T, int32_t* idx, float* w);
// one token: [RMSNorm,] router, softmax and top-k in one launch (h = 1024 / 2048 / 4096)
int32_t moe_route_fused(runit_ctx* ctx, const float* w, const float* x, float* logits, uint32_t E, uint32_t h, uint32_t k, int32_t renorm,
                        int32_t* idx, float* wts, uint32_t* counter, const float* gamma, float eps, float* xn_out);
// one token, any width: norm with one gain, router of E experts and R - E gates, scores, top-k and the gates' sigmoids
int32_t moe_route_gated(runit_ctx* ctx, const float* w, const float* x, float* logits, uint32_t R, uint32_t E, uint32_t K, uint32_t k,
                        int32_t score, int32_t renorm, int32_t* idx, float* wts, float* gates, uint32_t* counter, const float* gain,
                        float eps, float* xn_out);

constexpr int kMoeRowAlign = 128;   // every expert's rows start at a multiple of this in the permuted order
struct MoePermutation {
    int32_t *counts;                                    // [256]
    int32_t *n_tok_tiles, *tile_expert, *tile_nvalid, *tile_row0;
    int32_t *pos_of_slot;                               // [S], -1: unused slot
};
int32_t moe_permute(runit_ctx* ctx, const int32_t* idx, uint32_t S, uint32_t E, uint32_t tile_tok, const MoePermutation& p);
int32_t moe_dense_tiles(runit_ctx* ctx, uint32_t T, uint32_t tile_tok, int32_t* tile_expert, int32_t* tile_nvalid, int32_t* tile_row0,
                        int32_t* n_tok_tiles);
// xperm[pos(s)][:] = x[s / k][:], rows of row_bytes (a multiple of 16)
int32_t moe_gather_rows(runit_ctx* ctx, const void* x, const int32_t* pos_of_slot, void* xperm, uint32_t S, size_t row_bytes, uint32_t k);
int32_t moe_gather_values(runit_ctx* ctx, const float* v, const int32_t* pos_of_slot, float* out, uint32_t S);
// out[t] = residual[t] + sum_i w[t][i] * y[pos_of_slot[t*k+i]]  (w == nullptr: all ones)
int32_t moe_grouped_combine(runit_ctx* ctx, const float* y, const int32_t* pos_of_slot, const float* w, const float* residual, float* out,
                            uint32_t T, uint32_t h, uint32_t k);

}  // namespace runit
