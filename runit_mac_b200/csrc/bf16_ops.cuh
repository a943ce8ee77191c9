// Launchers of the operators over bf16 weight matrices (row-major, rows of ldw elements, ldw a multiple of 8, padding zero):
// GEMV for one token (gemv_bf16.cu), GEMM for many (gemm_bf16.cu), latent attention (latent_attention.cu).
#pragma once

#include <cuda_bf16.h>

#include "runit_internal.h"

namespace runit {

static inline uint32_t pad8(uint32_t n) { return (n + 7) & ~7u; }
static inline uint32_t pad16(uint32_t n) { return (n + 15) & ~15u; }

// What is done to a product before it is stored.
//   ADD    out += v (f32)
//   SILU_GLU  rows 2i and 2i+1 are gate and up of output i: silu(g) * u          (f32 or bf16 out, rows / 2 wide)
//   RELU2  max(v, 0)^2                                                          (f32 or bf16 out)
// SILU_GLU and RELU2 take two optional factors per token: `pre` multiplies the product (a weight on the input of the
// feed-forward block), `post` the activated value (a weight on its output).
enum GemmEpi { EPI_F32 = 0, EPI_ADD = 1, EPI_CAST = 2, EPI_SILU_GLU = 3, EPI_RELU2 = 4 };

// ── one token ──
struct GemvDesc {
    const void* w = nullptr;
    uint32_t rows = 0, K = 0, ldw = 0;
    const float* x = nullptr;
    const float* gain = nullptr;    // not null: x is first divided by its root mean square (eps) and multiplied by *gain
    float eps = 0.f;
    float* out = nullptr;
    const float* res = nullptr;     // EPI_F32: added (may be out)
    int epi = EPI_F32;              // EPI_F32, EPI_SILU_GLU, EPI_RELU2
    int32_t* argmax = nullptr;      // EPI_F32: index of the largest output, lowest index among equal ones
    unsigned long long* argmax_ctl = nullptr;   // two zeroed words (zero again when the launch ends)
    // Several feed-forward blocks over the same x: slot s < n_routed takes block slot_expert[s] of the stacked matrices w
    // ([..][rows][ldw]) with pre[s]; one more slot takes w_extra (rows_extra rows) with post = *post_extra.  Slot s writes
    // out + s * slot_stride.
    uint32_t n_routed = 0, slot_stride = 0;
    const int32_t* slot_expert = nullptr;
    const float* pre = nullptr;
    const void* w_extra = nullptr;
    uint32_t rows_extra = 0;
    const float* post_extra = nullptr;
};
int32_t gemv_bf16(runit_ctx* ctx, const char* name, const GemvDesc& d);

// out[r] = res[r] + sum over slots of W_slot[r] . x[slot * x_stride ..]: slot s < n_routed multiplies block slot_expert[s] of w
// ([..][rows][ldw], K columns), the last one w_extra ([rows][ldw_extra], K_extra columns) when it is not null.
struct GemvSumDesc {
    const void* w = nullptr;
    uint32_t rows = 0, K = 0, ldw = 0, n_routed = 0, x_stride = 0;
    const int32_t* slot_expert = nullptr;
    const void* w_extra = nullptr;
    uint32_t K_extra = 0, ldw_extra = 0;
    const float* x = nullptr;
    const float* res = nullptr;
    float* out = nullptr;
};
int32_t gemv_bf16_sum(runit_ctx* ctx, const char* name, const GemvSumDesc& d);

// ── many tokens ──
struct GemmDesc {
    const void* w = nullptr;        // [n_experts][rows][ldw]
    uint32_t rows = 0, K = 0, ldw = 0, n_experts = 1;
    const void* x = nullptr;        // [x_rows][ldx], bf16 or f32
    uint32_t ldx = 0, x_rows = 0;
    uint32_t T = 0;                 // tokens (dense); slots when grouped
    int epi = EPI_F32;
    void* out = nullptr;            // [..][ldo]; EPI_CAST / SILU_GLU / RELU2 store the activation type
    uint32_t ldo = 0;
    const float *pre = nullptr, *post = nullptr;    // per row of x
    // grouped: token tiles of tile_tok rows, each of one expert (moe_permute); null: dense
    const int32_t *tile_expert = nullptr, *tile_nvalid = nullptr, *tile_row0 = nullptr, *n_tok_tiles = nullptr;
    uint32_t tile_tok = 0, max_tiles = 0;
};
// exact = false: bf16 activations on the tensor cores (f32 accumulators); true: f32 activations, f32 multiply-adds.
int32_t gemm_bf16(runit_ctx* ctx, const char* name, const GemmDesc& d, bool exact);
uint32_t gemm_bf16_tile_tok(uint32_t tokens_per_expert, bool exact);

// ── rows: embedding and norms with one gain for all coordinates ──
// x[t] = RMSNorm(embed[token[t]]) * gain; tokens == nullptr: one row, the step's token (state, forced; see model_core.h)
int32_t embed_norm_rows(runit_ctx* ctx, const void* embed, uint32_t ld, const int32_t* tokens, const int32_t* state, const int32_t* forced,
                        uint32_t n_forced, uint32_t vocab, const float* gain, float eps, float* x, uint32_t T, uint32_t width);
// y = RMSNorm(x[rows]) * gain as bf16 or f32 rows of ldy elements (padding zero), and f32 rows of `width` in y2 when it is not
// null; gate_row not null: gate_out[t] = sigmoid(gate_row . y[t])
int32_t norm_rows(runit_ctx* ctx, const float* x, const int32_t* row_index, const float* gain, float eps, void* y, bool y_f32, uint32_t ldy,
                  float* y2, uint32_t T, uint32_t width, const float* gate_row = nullptr, float* gate_out = nullptr);

// ── latent attention ──
// Keys and values of all heads come from one cached row per position: the normed latent c (kv_rank values, padded to a
// multiple of 16) and the rotated key part all heads share (rot_dim, padded likewise).  Score of head h:
// (q_un . W_uk,h c + q_rot . k_rot) * scale; value W_uv,h c.
struct LatentDims {
    uint32_t heads, dim, rot_dim, vdim, kv_rank;
    float scale, eps;
    uint32_t cp() const { return pad16(kv_rank); }
    uint32_t pitch() const { return pad16(kv_rank) + pad16(rot_dim); }       // elements of a cache row
    uint32_t q_width() const { return heads * (dim + rot_dim); }
};
// Position of token t: *pos_ptr + t when pos_ptr is not null, else start + t.
struct LatentPos {
    const int32_t* pos_ptr;
    uint32_t start;
};
// Query side folded with W_uk: q_eff[t*heads+h] = [W_uk,h^T q_un | rotated q_rot], rows of pitch() values: f32, or with a bf16
// cache the high bf16 parts of all and then their low parts (4 bytes a value either way).  One more CTA per token
// writes the cache row of its position from qkv[t][q_width() ..] when kv_norm is not null (the layer owns its latent).
int32_t latent_query(runit_ctx* ctx, const LatentDims& d, bool cache_f32, const float* qkv, uint32_t ldq, const void* w_uk, uint32_t ldk,
                     const float* kv_norm, const float* freq, void* cache, void* q_eff, uint32_t T, LatentPos pos);
// The same without W_uk: cache rows, and the rotated parts of q in place (f32).
int32_t latent_rows(runit_ctx* ctx, const LatentDims& d, bool cache_f32, float* qkv, uint32_t ldq, const float* kv_norm, const float* freq,
                    void* cache, uint32_t T, LatentPos pos);
// Attention over cached rows: query row r = t*heads+h sees positions 0 .. pos(t); keys split nsplit ways.  part_o f32
// [row][nsplit][cp()], part_ml f32 [row][nsplit][2] (maximum, sum).
int32_t latent_attention(runit_ctx* ctx, const LatentDims& d, bool cache_f32, const void* q_eff, const void* cache, float* part_o,
                         float* part_ml, uint32_t nsplit, uint32_t T, LatentPos pos);
uint32_t latent_splits(const runit_ctx* ctx, const LatentDims& d, bool cache_f32, uint32_t T);
// out[t][h*vdim + j] = W_uv,h (merged latent output), f32 or bf16 rows of ldo
int32_t latent_value(runit_ctx* ctx, const LatentDims& d, const float* part_o, const float* part_ml, uint32_t nsplit, const void* w_uv,
                     uint32_t ldk, void* out, bool out_f32, uint32_t ldo, uint32_t T);
// Causal attention over keys and values of every head expanded beforehand: kv bf16 [S][ldkv] = [k_un of all heads | v of all
// heads]; q f32 (rotated) [T][ldq]; out bf16 [T][ldo].  Sizes: see latent_prefill_supported.
bool latent_prefill_supported(const LatentDims& d);
int32_t latent_prefill(runit_ctx* ctx, const LatentDims& d, const float* q, uint32_t ldq, const void* kv, uint32_t ldkv, const void* cache,
                       void* out_bf16, uint32_t ldo, uint32_t T, uint32_t start);

}  // namespace runit
