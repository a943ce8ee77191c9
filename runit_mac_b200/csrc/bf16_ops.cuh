// Launchers of the operators over bf16 weight matrices (row-major, rows of ldw elements, ldw a multiple of 8, padding zero):
// GEMV for one token (gemv_bf16.cu), GEMM for many (gemm_bf16.cu), latent attention (latent_attention.cu), attention over keys
// and values per head (head_attention.cu), layers with a decaying linear state (linear_state.cu).
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
// What the vector of a GEMV is made from, when it is not x itself (or x times one norm factor and gain):
//   RESIDUAL  v = x + y / rms(y) * y_gain: a sublayer's output is normed and added to the residual stream on its way into the
//             next matrix; v is also stored in x_out (not x: other CTAs still read it).  gain (may be null): v is then divided
//             by its own root mean square and multiplied by it, coordinate by coordinate.  y null: v = x, nothing stored.
//   GROUPS    the first `plain` values are x itself; the rest is cut into groups of `group` values, each divided by the group's
//             root mean square and multiplied by factor[i - plain].
enum { GEMV_PRO_NONE = 0, GEMV_PRO_RESIDUAL = 1, GEMV_PRO_GROUPS = 2 };
struct GemvPrologue {
    int kind = GEMV_PRO_NONE;
    const float *y = nullptr, *y_gain = nullptr, *gain = nullptr;
    float* x_out = nullptr;
    // the caller vouches that x and y_gain (RESIDUAL) are final before the launch in front of this one starts: they are read
    // before the dependency wait
    bool early = false;
    const float* factor = nullptr;
    bool factor_early = false;          // the same for factor
    uint32_t plain = 0, group = 0;
    const float* squares = nullptr;     // GROUPS, not null: [groups][squares_n] partial sums of squares of the groups
    uint32_t squares_n = 0;
};
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
    GemvPrologue pro;               // eps is that of its norms
    float cap = 0.f;                // EPI_F32, not 0: out = cap * tanh(product / cap)
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
    float* tail = nullptr;          // EPI_CAST: outputs from tail_from on are stored here as f32, rows of ldt
    uint32_t tail_from = 0, ldt = 0;
    float cap = 0.f;                // EPI_F32, not 0: cap * tanh(product / cap)
    // grouped: token tiles of tile_tok rows, each of one expert (moe_permute); null: dense
    const int32_t *tile_expert = nullptr, *tile_nvalid = nullptr, *tile_row0 = nullptr, *n_tok_tiles = nullptr;
    uint32_t tile_tok = 0, max_tiles = 0;
};
// exact = false: bf16 activations on the tensor cores (f32 accumulators); true: f32 activations, f32 multiply-adds.
int32_t gemm_bf16(runit_ctx* ctx, const char* name, const GemmDesc& d, bool exact);
uint32_t gemm_bf16_tile_tok(uint32_t tokens_per_expert, bool exact);

// ── rows: embedding and norms ──
// x[t] = RMSNorm(embed[token[t]]) * gain, or embed[token[t]] * scale when gain is null; tokens == nullptr: one row, the step's
// token (state, forced; see model_core.h)
int32_t embed_norm_rows(runit_ctx* ctx, const void* embed, uint32_t ld, const int32_t* tokens, const int32_t* state, const int32_t* forced,
                        uint32_t n_forced, uint32_t vocab, const float* gain, float eps, float* x, uint32_t T, uint32_t width, float scale = 1.f);
// x[t] += y[t] / rms(y[t]) * gain[i] (y null: nothing is added); out (may be null): x in the operand type, rows of ldo elements
// (padding zero).  out_gain not null: out is x / rms(x) * out_gain[i].  row_index: rows of x (with y null).
int32_t add_norm_rows(runit_ctx* ctx, float* x, const float* y, const float* gain, float eps, const int32_t* row_index, const float* out_gain,
                      void* out, bool out_f32, uint32_t ldo, uint32_t T, uint32_t width);
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

// ── attention over keys and values per head ──
// Query head h uses key / value head h / (heads / kv_heads).  A projected row holds [q: heads x dim | k: kv_heads x dim |
// v: kv_heads x vdim].  Score (q . k) * scale - slopes[h] * (i - j), scores and softmax in f32.
struct HeadAttn {
    uint32_t heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    uint32_t window = 0;               // 0: every earlier position is visible; else itself and the window - 1 before it
    uint32_t cap = 0;                  // rows of the cache: position p lives in row p % cap
    uint32_t unit_qk = 0;              // q and k are divided by their root mean square over dim
    float scale = 1.f, out_scale = 1.f, eps = 0.f;
    const float* slopes = nullptr;     // [heads]; null: none
    void *kc = nullptr, *vc = nullptr; // [kv_heads][cap][kd], [kv_heads][cap][vd], bf16 or f32, padding zero
    __host__ __device__ uint32_t kd() const { return (dim + 7) & ~7u; }
    __host__ __device__ uint32_t vd() const { return (vdim + 7) & ~7u; }
    __host__ __device__ uint32_t in_rows() const { return heads * dim + kv_heads * (dim + vdim); }
    __host__ __device__ uint32_t out_rows() const { return heads * vdim; }
};
// ── layers with a decaying linear state: S <- decay S + k v^T, o = S^T q per head, S [dk][dv] f32 ──
// Retention: decay fixed per head, rotated q and k (pairs (i, i + rot_dims/2)), k also times dim^(-1/2); o is divided by its
// root mean square per head and multiplied by silu(g).  A projected row holds [q | k: heads x dim | v | g: heads x vdim].
struct Retention {
    uint32_t heads = 0, dim = 0, vdim = 0, rot_dims = 0;
    float out_scale = 1.f, eps = 0.f, k_scale = 1.f;
    const float* freq = nullptr;       // [2][rot_dims / 2]: the frequencies, then what their rounding to f32 has left
    const float* decay = nullptr;      // [2][heads]: the decays, then their logarithms
    float* state = nullptr;            // [heads][dim][vdim]
    __host__ __device__ uint32_t in_rows() const { return 2 * heads * (dim + vdim); }
    __host__ __device__ uint32_t out_rows() const { return heads * vdim; }
};
// State-space layer (scalar decay per head and token).  A projected row holds [z: inner | x: inner | B: groups x state |
// C: groups x state | dt: heads]; x, B, C pass a causal convolution per channel and silu.
struct Ssm {
    uint32_t heads = 0, vdim = 0, state = 0, groups = 0, taps = 0, norm_groups = 0;
    float eps = 0.f;
    const float *conv_w = nullptr;     // [channels][taps], last column: the current token
    const float *conv_b = nullptr, *dt_bias = nullptr, *a = nullptr /* log decay per unit of dt */, *skip = nullptr, *norm = nullptr;
    float* s = nullptr;                // [heads][state][vdim]
    float* ring = nullptr;             // [taps][channels]: the projected inputs of position p in row p % taps
    __host__ __device__ uint32_t inner() const { return heads * vdim; }
    __host__ __device__ uint32_t channels() const { return heads * vdim + 2 * groups * state; }
    __host__ __device__ uint32_t in_rows() const { return 2 * heads * vdim + 2 * groups * state + heads; }
};
// One token.  Attention and / or retention on one projected row (a null one is left out): ao = [attention output * out_scale |
// retention o as it is], factor = silu(g) * out_scale of the retention, squares = sums of o^2 over the 32-column slices of every
// head ([heads][ceil(vdim / 32)]).  Writes this position's cache row, updates the state.  *pos_ptr, the cache and the state are
// read before the dependency wait: they must be final before the launch in front of this one starts.
// part / tickets: heads_step_scratch() floats and kv_heads * ceil(rep / 8) zeroed words (zero again afterwards).
uint32_t heads_step_splits(const runit_ctx* ctx, const HeadAttn& a, uint32_t T);
size_t heads_part_floats(const HeadAttn& a, uint32_t nsplit, uint32_t T);
int32_t heads_step(runit_ctx* ctx, const HeadAttn* a, const Retention* r, bool exact, const float* proj, float* ao, float* factor, float* squares,
                   float* part, uint32_t* tickets, uint32_t nsplit, const int32_t* pos_ptr);
// Many tokens: cache rows of their positions; rotated q and k of the retention in place.
int32_t heads_rows(runit_ctx* ctx, const HeadAttn* a, const Retention* r, bool exact, void* proj, uint32_t ld, uint32_t T, uint32_t start);
// Attention of T tokens whose cache rows are written: out rows of ldo.  part / tickets (see heads_step) serve few tokens; the
// number of splits is lowered until part_cap floats and 4096 tickets suffice.
int32_t head_attention_rows(runit_ctx* ctx, const HeadAttn& a, bool exact, const void* proj, uint32_t ld, void* out, uint32_t ldo, uint32_t T,
                            uint32_t start, float* part, size_t part_cap, uint32_t* tickets);
// One token of a state-space layer: y = (S^T C + skip x) * silu(z), squares as above; state and ring updated.  The state is
// read before the dependency wait.
int32_t ssm_step(runit_ctx* ctx, const Ssm& m, const float* proj, float* y, float* squares, const int32_t* pos_ptr);
// Many tokens: convolution, silu and softplus.  xbc rows of ld_out in the operand type, dt f32 [T][heads] in place.
int32_t ssm_conv_rows(runit_ctx* ctx, const Ssm& m, bool exact, const void* proj, uint32_t ld, void* xbc, uint32_t ld_out, float* dt, uint32_t T,
                      uint32_t start);
// The recurrence over T tokens.  q, k: [groups][dk] per token, v: [heads][dv]; log decay of a token log_decay[h] * dt, k times
// dt (dt null: 1); skip (may be null): o += skip[h] * v.  out: operand type.
struct LinearRows {
    uint32_t heads = 0, groups = 0, dk = 0, dv = 0;
    const void *q = nullptr, *k = nullptr, *v = nullptr;
    uint32_t ldq = 0, ldk = 0, ldv = 0;
    const float *dt = nullptr, *log_decay = nullptr, *decay = nullptr, *skip = nullptr;
    float* state = nullptr;
    void* out = nullptr;
    uint32_t ldo = 0;
};
size_t linear_chunk_bytes(uint32_t heads, uint32_t dk, uint32_t dv, uint32_t T);      // 0: sizes the chunked form does not take
int32_t linear_rows(runit_ctx* ctx, const LinearRows& d, bool exact, void* chunk_states, uint32_t T, uint32_t start);
// Norm of groups of a[t] in place (operand type).  before: a * silu(gate), normed, times weight; else a normed, times
// silu(gate) * out_scale.
int32_t gated_norm_rows(runit_ctx* ctx, bool exact, void* a, uint32_t lda, uint32_t n, uint32_t group, const void* gate, uint32_t ldg, bool before,
                        const float* weight, float out_scale, float eps, uint32_t T);

}  // namespace runit
