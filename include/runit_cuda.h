/*
 * runit_cuda.h — C ABI of the B200 (sm_100a) implementation of RunIT's quantized decode path.
 *
 * Every "twin" entry point replaces one free function of the reference's dispatch layer
 * (crates/kernels/src/dispatch.rs, cited per function as dispatch.rs:LINE; paths are relative
 * to the reference project root).  Names are the reference's, prefixed `runit_`; the argument
 * order is the reference's with `&MetalContext` -> `runit_ctx_t*`, `&metal::Buffer` -> device
 * pointer, `u32` -> uint32_t, `Result<()>` -> int32_t status.
 *
 * Execution model (replaces MetalContext::encode / flush, crates/kernels/src/context.rs:248-296):
 * every op is an in-order launch on the context's CUDA stream and returns at once;
 * runit_flush() waits for the stream and returns the first error since the last flush.
 * Ops never allocate, never synchronise and never retain pointers; the caller keeps buffers
 * alive until the next flush.  `output == residual` aliasing is allowed (the engine relies on
 * it, crates/engine/src/forward.rs:1619).  Arguments are validated on the host: a bad call
 * returns a status and launches nothing.
 *
 * There is no CPU fallback: without a CUDA device runit_ctx_create fails with
 * RUNIT_ERR_NO_DEVICE.  A context is used by one host thread at a time (the reference's
 * MetalContext is !Sync, context.rs:158).
 *
 * Weight layouts (row-major rows of blocks, as the reference lays them out):
 *   Q8_0: 34-byte blocks {f16 d; i8 qs[32]}, value = d*qs            gemv_q8_0.metal:11-14
 *   Q4_0: 18-byte blocks {f16 d; u8 qs[16]}, low nibble = element 2i, high = 2i+1,
 *         value = d*(nibble-8)                                        gemv_q4_0.metal:10-15
 *   Q4_K: 144-byte superblocks {f16 d; f16 dmin; u8 scales[12]; u8 qs[128]} of 256 elements;
 *         pair j: low nibbles of qs[32j..] -> elements 64j.., scale index j; high nibbles ->
 *         elements 64j+32.., scale index j+4                          dequant.metal:74-82
 * Alignment contract: weight base pointers 16-byte aligned (cudaMalloc gives 256); vectors
 * 16-byte aligned; k a multiple of 32 (Q8_0, Q4_0) or 256 (Q4_K).
 */
#ifndef RUNIT_CUDA_H
#define RUNIT_CUDA_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef struct runit_ctx runit_ctx_t;

/* Status codes; the Rust shim maps them onto KernelError (crates/kernels/src/error.rs:4-22). */
enum {
    RUNIT_OK = 0,
    RUNIT_ERR_NO_DEVICE = 1,   /* KernelError::NoDevice */
    RUNIT_ERR_BAD_ARG = 2,     /* null pointer, k not a block multiple, zero rows, ... */
    RUNIT_ERR_BUFFER_SIZE = 3, /* KernelError::BufferSize */
    RUNIT_ERR_LAUNCH = 4,      /* a CUDA call failed; text in runit_last_error_string */
    RUNIT_ERR_NCCL = 5,
    RUNIT_ERR_TIMEOUT = 6,     /* a bounded device- or host-side wait ran out */
    RUNIT_ERR_UNSUPPORTED = 7,
    RUNIT_ERR_ALLOC = 8
};

enum { RUNIT_BUF_DEVICE = 0, RUNIT_BUF_HOST_VISIBLE = 1 };
enum { RUNIT_FMT_Q8_0 = 0, RUNIT_FMT_Q4_0 = 1, RUNIT_FMT_Q4K = 2, RUNIT_FMT_Q5_0 = 3, RUNIT_FMT_Q5K = 4, RUNIT_FMT_Q6K = 5 };

/* ── context, buffers, flush: MetalContext::{new,new_buffer,flush}, context.rs:163-296 ── */
int32_t runit_ctx_create(int32_t device, runit_ctx_t** out);
/* Adopt a stream the caller owns (e.g. the stream a collective library runs on). */
int32_t runit_ctx_create_on_stream(int32_t device, void* cuda_stream, runit_ctx_t** out);
int32_t runit_ctx_destroy(runit_ctx_t* ctx);
void*   runit_ctx_stream(runit_ctx_t* ctx);
int32_t runit_flush(runit_ctx_t* ctx);
const char* runit_last_error_string(runit_ctx_t* ctx);
const char* runit_status_string(int32_t status);
/* Device buffers are 1024-byte aligned. */
int32_t runit_buf_alloc(runit_ctx_t* ctx, size_t bytes, int32_t flags, void** dptr);
int32_t runit_buf_free(runit_ctx_t* ctx, void* dptr);
int32_t runit_memcpy_h2d(runit_ctx_t* ctx, void* dst_dev, const void* src_host, size_t bytes);
int32_t runit_memcpy_d2h(runit_ctx_t* ctx, void* dst_host, const void* src_dev, size_t bytes);
int32_t runit_memset(runit_ctx_t* ctx, void* dst_dev, int32_t byte, size_t bytes);
/* Per-op launch counter (kernels launched by this context since creation). */
uint64_t runit_launch_count(runit_ctx_t* ctx);
/* Test-only: selects kernel variants so that the parity tests can exercise every code path of the GEMV family
 * (0 = the default choice for every key).  Not part of the reference's interface; an engine never calls it. */
int32_t runit_set_tuning(runit_ctx_t* ctx, const char* key, int32_t value);

/* ── recorded command lists (no twin as a function; the role of the reference's command buffer,
 *    context.rs:248-296: ops are encoded once and committed together) ──
 * Between begin and end every op call on the context is recorded instead of executed; the
 * recorded list replays with one launch.  Pointers and sizes are baked in at record time.  */
typedef struct runit_graph runit_graph_t;
int32_t runit_graph_begin(runit_ctx_t* ctx);
int32_t runit_graph_end(runit_ctx_t* ctx, runit_graph_t** out);
int32_t runit_graph_launch(runit_ctx_t* ctx, runit_graph_t* graph);
int32_t runit_graph_destroy(runit_ctx_t* ctx, runit_graph_t* graph);
/* Opt-in (runit_set_tuning(ctx, "stream_fuse", 1) before runit_graph_begin): runs of consecutive batch-1 fused-dequant
 * GEMVs (4-bit formats, f32 activations) of a recording are executed by ONE persistent launch whose warps stream the
 * weights of the whole run without stopping at the boundaries between the GEMVs; the ops keep their recorded order
 * wherever one reads or overwrites what another wrote or read, and the results equal those of the separate launches up
 * to the summation order over K-slices.  Off by default: on B200 the separate launches (with dependent launch) are still
 * faster for decode-size matrices.  Returns how many of the recorded GEMV launches the list folded this way. */
uint32_t runit_graph_fused_launches(runit_graph_t* graph);
/* Kernel launches one replay of the list performs (after that folding). */
uint32_t runit_graph_kernel_launches(runit_graph_t* graph);

/* ── Q8_0 fused-dequant GEMV family ── */
/* dispatch.rs:1280  y_f32[m] = W_q8_0[m,k] . x_f32[k] */
int32_t runit_gemv_q8_0_f32in_f32out(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
/* dispatch.rs:1298  y_f32 = W.x_f32 + residual_f32 (output may alias residual) */
int32_t runit_gemv_q8_0_add_f32_f32in(runit_ctx_t*, const void* weight, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
/* dispatch.rs:1317  y_f16 = W.x_f32 */
int32_t runit_gemv_q8_0_f32in(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
/* dispatch.rs:1335  y_f16 = W.x_f16 */
int32_t runit_gemv_q8_0_f16(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
/* dispatch.rs:1353  y_f16 = W.x_f16 + residual_f16 */
int32_t runit_gemv_q8_0_add_f16(runit_ctx_t*, const void* weight, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
/* dispatch.rs:1372  y_f32 = W.x_f16 + residual_f32 */
int32_t runit_gemv_q8_0_add_f32res_f16(runit_ctx_t*, const void* weight, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
/* dispatch.rs:1083,1101 (4 rows per threadgroup) and dispatch.rs:1397,1414,1432 (256-wide):
 * launch-shape variants of the same operators; here they are the same kernel. */
int32_t runit_gemv_q8_0_f32in_f32out_mr(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
int32_t runit_gemv_q8_0_add_f32_f32in_mr(runit_ctx_t*, const void* weight, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
int32_t runit_gemv_q8_0_f32in_f32out_wide(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
int32_t runit_gemv_q8_0_add_f32_f32in_wide(runit_ctx_t*, const void* weight, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
int32_t runit_gemv_q8_0_f32in_wide(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
/* dispatch.rs:813  Q|K|V rows in one launch, f32 in/out */
int32_t runit_fused_qkv_q8_0_f32(runit_ctx_t*, const void* w_q, const void* w_k, const void* w_v, const void* x_vec,
                                 void* out_q, void* out_k, void* out_v, uint32_t q_dim, uint32_t kv_dim, uint32_t k);
/* dispatch.rs:842  same + f16 bias per row (the reference uploads biases as f16) */
int32_t runit_fused_qkv_bias_q8_0_f32(runit_ctx_t*, const void* w_q, const void* w_k, const void* w_v, const void* x_vec,
                                      void* out_q, void* out_k, void* out_v, const void* bias_q, const void* bias_k,
                                      const void* bias_v, uint32_t q_dim, uint32_t kv_dim, uint32_t k);
/* dispatch.rs:903  act_f32[ff] = silu(Wg.x) * (Wu.x) */
int32_t runit_fused_ffn_q8_0_f32(runit_ctx_t*, const void* w_gate, const void* w_up, const void* x_vec, void* act_out, uint32_t ff_dim, uint32_t k);

/* ── Q4_0 ── */
/* dispatch.rs:1456 */
int32_t runit_gemv_q4_0_f32in_f32out(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
/* dispatch.rs:1471 */
int32_t runit_gemv_q4_0_add_f32_f32in(runit_ctx_t*, const void* weight, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
/* dispatch.rs:1486  f32 in, f16 out */
int32_t runit_gemv_q4_0_f32in(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
/* dispatch.rs:1501  f16 in, f16 out */
int32_t runit_gemv_q4_0_f16(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
/* dispatch.rs:1516  f16 in, f16 out + f16 residual */
int32_t runit_gemv_q4_0_add_f16(runit_ctx_t*, const void* weight, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
/* dispatch.rs:1531 */
int32_t runit_fused_ffn_q4_0_f32(runit_ctx_t*, const void* w_gate, const void* w_up, const void* x_vec, void* act_out, uint32_t ff_dim, uint32_t k);

/* ── Q4_K ── */
/* dispatch.rs:1229 */
int32_t runit_gemv_q4k_f32in_f32out(runit_ctx_t*, const void* weight_q4k, const void* input, void* output, uint32_t m, uint32_t k);
/* dispatch.rs:1251 */
int32_t runit_gemv_q4k_add_f32_f32in(runit_ctx_t*, const void* weight_q4k, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
/* dispatch.rs:621  f16 in, f16 out */
int32_t runit_gemv_q4k_f16(runit_ctx_t*, const void* weight_q4k, const void* input, void* output, uint32_t m, uint32_t k);
/* dispatch.rs:585  f16 in, f16 out + f16 residual */
int32_t runit_gemv_q4k_add_f16(runit_ctx_t*, const void* weight_q4k, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
/* dispatch.rs:358  f16 in, f32 out + f32 residual */
int32_t runit_gemv_q4k_add_f32res_f16(runit_ctx_t*, const void* weight_q4k, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
/* dispatch.rs:756  Q4_K blocks -> f16 elements */
int32_t runit_dequant_q4k_f16(runit_ctx_t*, const void* input, void* output, uint32_t n_blocks);

/* ── Q5_0, Q5_K, Q6_K: fused-dequant GEMVs for formats the reference only expands on the CPU at load time
 *    (crates/engine/src/forward.rs:900-919 Q5_0, 920-949 Q6_K, 979-1012 Q5_K) and then multiplies as f16.  No twin in
 *    dispatch.rs; names follow the Q4_K twins.  Layouts as the reference decodes them:
 *      Q5_0: 22-byte blocks {f16 d; u8 qh[4]; u8 qs[16]}, byte j = elements j (low nibble) and j+16 (high), fifth bits in
 *            bit j of qh (little-endian u32) and bit j+16, value = d*(q-16); k a multiple of 32
 *      Q5_K: 176-byte superblocks {f16 d; f16 dmin; u8 scales[12]; u8 qh[32]; u8 qs[128]}: Q4_K plus the fifth bit of
 *            element e in bit e%8 of qh[e/8]; k a multiple of 256
 *      Q6_K: 210-byte superblocks {u8 ql[128]; u8 qh[64]; i8 scales[16]; f16 d}, value = d*scale*(q-32), scale index
 *            8*(e/128) + 2*((e%128)/32); k a multiple of 256
 *    y_f32[m] = W[m,k] . x_f32[k] (+ residual_f32; output may alias residual). ── */
int32_t runit_gemv_q5_0_f32in_f32out(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
int32_t runit_gemv_q5_0_add_f32_f32in(runit_ctx_t*, const void* weight, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
int32_t runit_gemv_q5k_f32in_f32out(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
int32_t runit_gemv_q5k_add_f32_f32in(runit_ctx_t*, const void* weight, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);
int32_t runit_gemv_q6k_f32in_f32out(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
int32_t runit_gemv_q6k_add_f32_f32in(runit_ctx_t*, const void* weight, const void* input, void* output, const void* residual, uint32_t m, uint32_t k);

/* ── MoE glue and router ── */
/* dispatch.rs:270  y_f16[m] = W_f16[m,k] . x_f32[k]  (router logits) */
int32_t runit_gemv_f16w_f32in(runit_ctx_t*, const void* weight, const void* input, void* output, uint32_t m, uint32_t k);
/* dispatch.rs:15 / dispatch.rs:35 */
int32_t runit_silu_mul_f16(runit_ctx_t*, const void* gate, const void* up, void* out, uint32_t n);
int32_t runit_silu_mul_f32(runit_ctx_t*, const void* gate, const void* up, void* out, uint32_t n);
/* dispatch.rs:1639  acc_f16 += half(float(src_f16) * weight) */
int32_t runit_scale_accumulate_f16(runit_ctx_t*, const void* src, void* acc, float weight, uint32_t n);
/* dispatch.rs:316  acc_f32 += float(src_f16) */
int32_t runit_add_f16_into_f32(runit_ctx_t*, const void* src, void* acc, uint32_t n);

/* ── entry points with no twin in the reference ── */
/* Q|K|V in one launch for the 4-bit formats and gate/up+SiLU for Q4_K (the reference has these fusions only
 * for Q8_0 / Q4_0: dispatch.rs:813, 903, 1531). */
int32_t runit_fused_qkv_q4_0_f32(runit_ctx_t*, const void* w_q, const void* w_k, const void* w_v, const void* x_vec,
                                 void* out_q, void* out_k, void* out_v, uint32_t q_dim, uint32_t kv_dim, uint32_t k);
int32_t runit_fused_qkv_q4k_f32(runit_ctx_t*, const void* w_q, const void* w_k, const void* w_v, const void* x_vec,
                                void* out_q, void* out_k, void* out_v, uint32_t q_dim, uint32_t kv_dim, uint32_t k);
int32_t runit_fused_ffn_q4k_f32(runit_ctx_t*, const void* w_gate, const void* w_up, const void* x_vec, void* act_out,
                                uint32_t ff_dim, uint32_t k);
/* Batched fused-dequant GEMV: x [batch][k] f32, y [batch][m] f32 (+ residual [batch][m], may be
 * NULL); weights streamed once for the whole batch; batch in 1..8. */
int32_t runit_gemv_batched_f32(runit_ctx_t*, int32_t fmt, const void* weight, const void* input, void* output,
                               const void* residual, uint32_t m, uint32_t k, uint32_t batch);
/* The same for up to three matrices that share the input (q | k | v, gate | up): one launch, the activations are
 * prepared once; outputs[i] f32 [batch][rows[i]].  (Host pointer tables of n_mats device pointers.) */
int32_t runit_gemv_batched_multi_f32(runit_ctx_t*, int32_t fmt, uint32_t n_mats, const void* const* weights, const void* input,
                                     void* const* outputs, const uint32_t* rows, uint32_t k, uint32_t batch);
/* RMSNorm fused into the GEMV that consumes it: x is the un-normalised f32 vector [k], gamma f32 [k]; the matrices multiply
 * x * rsqrt(mean(x^2) + eps) * gamma (the reference runs rms_norm_f32_f32_f32g, forward.rs:1528-1569 / dispatch.rs:177, then the
 * GEMV, as two encoders).  Every CTA computes the scale itself, so the scale agrees with the stand-alone operator to
 * rounding, not to the bit.  fmt: RUNIT_FMT_Q8_0 / Q4_0 / Q4K.  residual f32 [m], may be NULL. */
int32_t runit_rms_norm_gemv_f32(runit_ctx_t*, int32_t fmt, const void* weight, const void* x, const void* gamma, float eps,
                                void* output, const void* residual, uint32_t m, uint32_t k);
int32_t runit_rms_norm_fused_qkv_f32(runit_ctx_t*, int32_t fmt, const void* w_q, const void* w_k, const void* w_v, const void* x,
                                     const void* gamma, float eps, void* out_q, void* out_k, void* out_v, uint32_t q_dim,
                                     uint32_t kv_dim, uint32_t k);
/* Greedy lm_head: the GEMV of runit_rms_norm_gemv_f32 (gamma may be NULL: then x is used as it is) whose epilogue also
 * finds the index of the largest logit, lowest index among equal values (argmax after lm_head, forward.rs:1967-1973):
 * logits f32 [m] and result int32 [1] come out of one launch.  Needs 16-byte aligned weight rows and m <= 2,097,152. */
int32_t runit_gemv_argmax_f32(runit_ctx_t*, int32_t fmt, const void* weight, const void* x, const void* gamma, float eps,
                              void* logits, void* result, uint32_t m, uint32_t k);
/* Row-sharded greedy lm_head: rank `rank` multiplies its rows_total / world rows (logits_local f32, this rank's slice) and
 * stores its (largest logit, global row index) pair, 8 bytes, into slot `rank` of every rank's pair table pairs_all[p]
 * (uint2 [world], peer-mapped memory, plain stores).  After runit_peer_barrier, runit_argmax_pairs over the own table gives
 * the same token on every rank: an 8-byte all-gather instead of the logits. */
int32_t runit_gemv_argmax_allgather(runit_ctx_t*, int32_t fmt, const void* w_local, const void* x, void* logits_local,
                                    void* const* pairs_all, uint32_t world, uint32_t rank, uint32_t rows_total, uint32_t k);
int32_t runit_argmax_pairs(runit_ctx_t*, const void* pairs, uint32_t n, void* result);
/* runit_peer_barrier followed by runit_argmax_pairs over this rank's own table (uint2 [world]) in one launch */
int32_t runit_peer_barrier_argmax(runit_ctx_t*, void* const* signal_pads, uint32_t world, uint32_t rank, uint32_t epoch,
                                  const void* pairs, void* result);
/* Fused Q|K|V with an f32 bias (the benchmark configuration states an f32 bias); bias may be NULL. */
int32_t runit_fused_qkv_f32bias_q8_0_f32(runit_ctx_t*, const void* w_q, const void* w_k, const void* w_v, const void* x_vec,
                                         void* out_q, void* out_k, void* out_v, const void* bias_q, const void* bias_k,
                                         const void* bias_v, uint32_t q_dim, uint32_t kv_dim, uint32_t k);
/* ── row-sharded GEMV with the all-gather fused into the epilogue (no twin: the reference is single-device,
 *    crates/engine/src/server/mod.rs:20-30).  Rank `rank` of `world` (<= 8) owns rows [rank*n, (rank+1)*n), n =
 *    rows_total/world, of the weight matrix (w_local: those n rows).  y_all: HOST array of `world` DEVICE pointers, entry p
 *    = rank p's full-length f32 output vector as mapped into this process (peer memory for p != rank, e.g. from CUDA
 *    virtual-memory or IPC mappings / torch symmetric memory).  Every result is stored into all of them by plain peer
 *    stores.  The vectors are complete on every rank once all ranks have passed runit_peer_barrier.
 *    Reuse: passing the barrier of call n means every rank has ANNOUNCED epoch n, not that it has finished reading
 *    the result of call n.  A rank that runs ahead would overwrite a vector a slower rank still reads, so alternate
 *    between two sets of output vectors from call to call (call n+2 can only start after barrier n+1, which each rank
 *    announces in stream order after its own reads of result n), or put a second barrier after the consumer. ── */
int32_t runit_gemv_allgather_f32(runit_ctx_t*, int32_t fmt, const void* w_local, const void* x, void* const* y_all,
                                 uint32_t world, uint32_t rank, uint32_t rows_total, uint32_t k);
/* ── expert-parallel MoE block for prefill-sized batches (no twin: the reference is single-device) ──
 * Tokens are data-parallel (the same T on every rank), experts are split over the ranks (E / world each; placement 0:
 * expert e on rank e / (E/world), 1: on rank e % world); token rows are stored into the owners' receive buffers and the
 * expert outputs back into the senders' return buffers with plain peer stores, two bounded barriers per call, no host
 * read and no collective library on the data path.  The result equals runit_moe_layer_q4k_bf16 on one GPU bit for bit.
 * Peer-mapped buffers, one per rank, given as pointer tables of `world` entries (this rank's own included):
 *   recv_rows   bf16  [world * T * k][h]     recv_meta  int32 [world * T * k][2]     recv_counts  int32 [world]
 *   return_rows f32   [T * k][h]             signal_pads uint32 [>= world], zeroed before the first call
 * epoch counts the calls on these buffers from 1 (it uses barrier epochs 2*epoch-1 and 2*epoch).  scratch: local memory,
 * runit_moe_ep_prefill_scratch_bytes, 1024-byte aligned.  x / residual / out: f32 [T][h]; idx_out / w_out may be NULL. */
size_t  runit_moe_ep_prefill_scratch_bytes(uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, uint32_t world);
int32_t runit_moe_layer_q4k_bf16_ep(runit_ctx_t*, const void* router_w, const void* gate_local, const void* up_local,
                                    const void* down_local, const void* x, const void* residual, void* out, void* idx_out, void* w_out,
                                    void* scratch, size_t scratch_bytes, void* const* recv_rows_all, void* const* recv_meta_all,
                                    void* const* recv_counts_all, void* const* return_rows_all, void* const* signal_pads, uint32_t T,
                                    uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm, uint32_t world, uint32_t rank,
                                    uint32_t epoch, int32_t placement);
/* One-kernel barrier over peer memory.  signal_pads: HOST array of `world` DEVICE pointers, entry p = rank p's pad of at
 * least `world` uint32 words (zero before the first use), as mapped into this process.  Announces `epoch` (> 0,
 * strictly increasing from call to call) to every rank and waits until every rank has announced it; a rank that does
 * not show up within about half a second makes the next runit_flush return RUNIT_ERR_TIMEOUT (the context stays
 * usable). */
int32_t runit_peer_barrier(runit_ctx_t*, void* const* signal_pads, uint32_t world, uint32_t rank, uint32_t epoch);

/* ── MoE block (no twin as one function; replaces the sequence crates/engine/src/forward.rs:1644-1679
 *    and the CPU routing forward.rs:2420-2448, without the per-layer host synchronisation) ── */
/* logits_f32[T][E] = router_f32[E][h] . x_f32[T][h] */
int32_t runit_moe_router_f32(runit_ctx_t*, const void* router_w, const void* x, void* logits, uint32_t E, uint32_t h, uint32_t T);
/* softmax over all E experts, top-k by probability (descending; ties: lowest index), weights optionally
 * renormalised to sum 1.  logits: [T][E] f32, or f16 when logits_f16 != 0 (the reference's router dtype);
 * out_idx: int32 [T][k]; out_w: f32 [T][k].  E <= 256, k <= 32. */
int32_t runit_moe_route_topk(runit_ctx_t*, const void* logits, int32_t logits_f16, uint32_t E, uint32_t k, int32_t renorm,
                             uint32_t T, void* out_idx, void* out_w);
/* The same with the scoring function as a parameter: rows of ld logits (the first E are the experts'), softmax over the
 * experts or the sigmoid of each logit.  f32 logits. */
enum { RUNIT_SCORE_SOFTMAX = 0, RUNIT_SCORE_SIGMOID = 1 };
int32_t runit_moe_route_scored(runit_ctx_t*, const void* logits, uint32_t ld, uint32_t E, uint32_t k, int32_t score, int32_t renorm,
                               uint32_t T, void* out_idx, void* out_w);
/* Scratch bytes runit_moe_layer_q4k needs for these shapes. */
size_t runit_moe_scratch_bytes(uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k);
/* One MoE block over T tokens, all on the device:
 *   out[t] = (residual ? residual[t] : 0) + sum_i w_i * Wdown[e_i] . (silu(Wgate[e_i].x[t]) * (Wup[e_i].x[t]))
 * router_w: f32 [E][h]; gate, up: Q4_K [E][ff][h]; down: Q4_K [E][h][ff] (experts stacked contiguously, as
 * the reference slices merged expert tensors, forward.rs:1339-1408); x, residual, out: f32 [T][h] (out may
 * alias residual); idx_out (int32 [T][k]) and w_out (f32 [T][k]) may be NULL; scratch: caller-owned device
 * memory of at least runit_moe_scratch_bytes(), 256-byte aligned.  h, ff multiples of 256. */
int32_t runit_moe_layer_q4k(runit_ctx_t*, const void* router_w, const void* gate, const void* up, const void* down,
                            const void* x, const void* residual, void* out, void* idx_out, void* w_out, void* scratch,
                            size_t scratch_bytes, uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm);

/* The expert part alone, for expert-parallel execution: slot s holds one token row x_slots[s] (f32 [h]) routed to
 * local expert slot_expert[s] (int32; a negative id marks an unused slot: nothing is computed or written for it);
 * y_slots[s] = Wdown[e] . (silu(Wgate[e].x) * (Wup[e].x)).  gate/up: Q4_K [n_experts][ff][h]; down: Q4_K
 * [n_experts][h][ff]; act_scratch: f32 [n_slots][ff], caller-owned. */
int32_t runit_moe_experts_q4k(runit_ctx_t*, const void* gate, const void* up, const void* down, const void* x_slots,
                              const void* slot_expert, void* y_slots, void* act_scratch, uint32_t n_slots, uint32_t h,
                              uint32_t ff, uint32_t n_experts);

/* Expert-parallel form of runit_moe_layer_q4k for decode sizes, tokens replicated on every rank (no counterpart in
 * the reference, which runs on one device).  Rank r holds the replicated router and the experts
 * [r * E/world, (r+1) * E/world) (gate_local, up_local: Q4_K [E/world][ff][h]; down_local: Q4_K [E/world][h][ff]).  Every
 * rank routes all T tokens itself, computes only the (token, expert) slots it owns, and stores its weighted partial sum
 * into slot r of the partial buffer of EVERY rank with plain peer stores (the combine exchange fused into the kernel: no
 * collective library call, no TMA, no multicast); after the one-kernel barrier each rank adds the `world` partial sums in
 * rank order plus the residual, so all ranks end with identical bits in `out`.
 * partial_all: HOST array of `world` DEVICE pointers, entry p = rank p's partial buffer, f32 [2][world][T][h], as mapped
 * into this process (the two halves alternate by epoch parity, so a fast rank's next call never overwrites what a slow
 * rank is still adding); signal_pads / epoch: as for runit_peer_barrier (a missing rank makes the next runit_flush return
 * RUNIT_ERR_TIMEOUT).  scratch: runit_moe_scratch_bytes(T, h, ff, E, k). */
int32_t runit_moe_layer_q4k_ep(runit_ctx_t*, const void* router_w, const void* gate_local, const void* up_local,
                               const void* down_local, const void* x, const void* residual, void* out, void* idx_out, void* w_out,
                               void* scratch, size_t scratch_bytes, void* const* partial_all, void* const* signal_pads,
                               uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm, uint32_t world,
                               uint32_t rank, uint32_t epoch);

/* No counterpart in the reference.  The same MoE block as runit_moe_layer_q4k for callers that cannot hand
 * over scratch memory: a host engine that gives every free byte of device memory to its own weight and
 * KV-cache pools at start-up, or a serving loop that must not call cudaMalloc because that call stalls the
 * whole device.  This entry point allocates nothing (no cudaMalloc/cudaFree, no allocating library call);
 * its intermediates live in a fixed 4 MiB region (runit_moe_static_scratch_capacity()) built into the
 * library image, which every GPU that loads the library holds until the process exits.
 *   - Shapes whose intermediates do not fit (runit_moe_scratch_bytes(T,h,ff,E,k) > capacity; e.g. OLMoE
 *     shapes beyond 32 tokens) are rejected with RUNIT_ERR_BUFFER_SIZE and nothing is launched.
 *   - The first call on a device looks up the region's device address (once per device, with that device
 *     made current for the lookup) and keeps it for the life of the process; make that first call before any
 *     stream capture is started.  The kept address does not survive cudaDeviceReset: a process that resets a
 *     device must not use this entry point on it afterwards.
 *   - All calls share the one region and it keeps the previous call's contents; every part the block reads
 *     is rewritten first, so nothing needs clearing, but two calls that overlap on the GPU (different
 *     streams or contexts of one process on the same device) race on it: keep them ordered. */
size_t  runit_moe_static_scratch_capacity(void);
int32_t runit_moe_layer_q4k_static(runit_ctx_t*, const void* router_w, const void* gate, const void* up, const void* down,
                                   const void* x, const void* residual, void* out, void* idx_out, void* w_out,
                                   uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm);

/* ── batched (prefill-sized) MoE block on the tensor cores.  No twin: the reference's prefill runs the decode
 *    block once per token (crates/engine/src/prefill.rs:156-215).  Same block as runit_moe_layer_q4k with bf16
 *    operands: slots are sorted by expert on the device, every Q4_K weight d*sc*q - dmin*m
 *    (crates/engine/src/forward.rs:1026-1057) is rounded to bf16 in shared-memory tiles, activations are rounded to
 *    bf16, products accumulate in f32 (tcgen05.mma, accumulators in tensor memory):
 *      act[s] = bf16(silu(Wg[e].bf16(x[t])) * (Wu[e].bf16(x[t]))), y[s] = Wd[e].act[s],
 *      out[t] = (residual ? residual[t] : 0) + sum_i w_i * y[s_i]        (routing order)
 *    Shapes: h, ff multiples of 256; E <= 256; k <= min(E, 32).  scratch: caller-owned, 1024-byte aligned,
 *    at least runit_moe_grouped_scratch_bytes(); tensors 16-byte aligned; out may alias residual. ── */
size_t  runit_moe_grouped_scratch_bytes(uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k);
/* router (f32 [E][h]) -> softmax/top-k -> experts; idx_out (int32 [T][k]) and w_out (f32 [T][k]) may be NULL. */
int32_t runit_moe_layer_q4k_bf16(runit_ctx_t*, const void* router_w, const void* gate, const void* up, const void* down,
                                 const void* x, const void* residual, void* out, void* idx_out, void* w_out, void* scratch,
                                 size_t scratch_bytes, uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm);
/* The expert part for given routing: idx int32 [T][k] (ids outside [0, E) are skipped), w f32 [T][k]. */
int32_t runit_moe_experts_grouped_q4k_bf16(runit_ctx_t*, const void* gate, const void* up, const void* down, const void* x,
                                           const void* idx, const void* w, const void* residual, void* out, void* scratch,
                                           size_t scratch_bytes, uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k);

/* ── decode-step operators besides the GEMVs ── */
/* dispatch.rs:152  y = x * rsqrt(mean(x^2)+eps) * gamma_f16, num_rows rows of `hidden` (x may equal y) */
int32_t runit_rms_norm_f32_f32(runit_ctx_t*, const void* x, void* y, const void* gamma, float eps, uint32_t hidden, uint32_t num_rows);
/* dispatch.rs:177  same with f32 gamma */
int32_t runit_rms_norm_f32_f32_f32g(runit_ctx_t*, const void* x, void* y, const void* gamma, float eps, uint32_t hidden, uint32_t num_rows);
/* dispatch.rs:945  rotary embedding of Q [q_heads][hd] and K [kv_heads][hd] in place, pairs (d, d+hd/2) */
int32_t runit_fused_rope_qk_f32(runit_ctx_t*, void* q, void* k, uint32_t head_dim, uint32_t q_heads, uint32_t kv_heads, uint32_t pos, float theta);
/* dispatch.rs:1159 / 1183  scatter [kv_heads][hd] into the cache [kv_heads][max_seq][hd] at pos */
int32_t runit_kv_copy_to_cache_f16(runit_ctx_t*, const void* src, void* dst, uint32_t pos, uint32_t max_seq, uint32_t head_dim, uint32_t num_kv_heads);
int32_t runit_kv_copy_to_cache_f32(runit_ctx_t*, const void* src, void* dst, uint32_t pos, uint32_t max_seq, uint32_t head_dim, uint32_t num_kv_heads);
/* no twin: f32 source rounded into an f16 cache */
int32_t runit_kv_copy_to_cache_f32_f16(runit_ctx_t*, const void* src, void* dst, uint32_t pos, uint32_t max_seq, uint32_t head_dim, uint32_t num_kv_heads);
/* dispatch.rs:1575 (f32) / dispatch.rs:697 (f16)  q_len = 1 attention over kv_len cached positions,
 * scale 1/sqrt(head_dim), GQA kv_head = q_head / (heads/kv_heads); head_dim in {32,64,96,128} */
int32_t runit_decode_attention_f32(runit_ctx_t*, const void* q, const void* k, const void* v, void* out, uint32_t batch, uint32_t kv_len,
                                   uint32_t num_heads, uint32_t num_kv_heads, uint32_t head_dim, uint32_t kv_head_stride);
int32_t runit_decode_attention_f16(runit_ctx_t*, const void* q, const void* k, const void* v, void* out, uint32_t batch, uint32_t kv_len,
                                   uint32_t num_heads, uint32_t num_kv_heads, uint32_t head_dim, uint32_t kv_head_stride);
/* no twin: f32 query and output over an f16 cache */
int32_t runit_decode_attention_f32q_f16kv(runit_ctx_t*, const void* q, const void* k, const void* v, void* out, uint32_t batch, uint32_t kv_len,
                                          uint32_t num_heads, uint32_t num_kv_heads, uint32_t head_dim, uint32_t kv_head_stride);
/* dispatch.rs:1615  index of the maximum of n f16 values -> result[0] (int32); ties: lowest index */
int32_t runit_argmax_f16(runit_ctx_t*, const void* input, void* result, uint32_t n);
/* no twin: f32 input (sampler.rs:111-116 on the device) */
int32_t runit_argmax_f32(runit_ctx_t*, const void* input, void* result, uint32_t n);

/* ── token sampling on the device: the reference's host sampler (crates/engine/src/sampler.rs:61-111) as one launch ──
 * Steps, in the reference's order: end-of-sequence ids suppressed while the context is shorter than min_tokens;
 * repetition penalty once per occurrence of a token in the context; temperature 0 -> argmax (last index among equal
 * maxima, as Iterator::max_by); else scores / temperature, softmax, top-k (the first k entries in index order with
 * p >= the k-th largest), top-p (descending order until the running sum has reached p), and the draw r = rng * total over
 * the survivors in index order.  The generator is the reference's xorshift64 (sampler.rs:12-27); its state lives in
 * device memory and advances by one draw.  top_k in 0..1024 (0 = off); with top-k off and top_p < 1 the nucleus must lie
 * within the 1024 most probable tokens (else status: RUNIT_ERR_UNSUPPORTED at the next flush, most probable token returned). */
typedef struct {
    float   temperature;          /* 0 = greedy */
    int32_t top_k;                /* 0 = off */
    float   top_p;                /* >= 1 = off */
    float   repetition_penalty;   /* 1 = off */
    int32_t min_tokens;
} runit_sampler_cfg;
/* logits f32 [n]; scores_scratch f32 [n] (holds the final distribution afterwards, unless greedy); context int32 tokens,
 * the range [ctx_begin, ctx_end) of it is the context, or, when ctx_range is not NULL, the two device words it points to
 * give that range; eos_ids int32 [n_eos]; rng_state uint64 [1]; result int32 [1].  All pointers are device pointers. */
int32_t runit_sample_f32(runit_ctx_t*, const void* logits, void* scores_scratch, uint32_t n, const runit_sampler_cfg* cfg,
                         const void* context, const void* ctx_range, uint32_t ctx_begin, uint32_t ctx_end, const void* eos_ids,
                         uint32_t n_eos, void* rng_state, void* result);
/* SimpleRng::new (sampler.rs:15-17): the state to store in rng_state for a seed */
uint64_t runit_sampler_seed_state(uint64_t seed);

/* ── greedy decoder for an OLMoE-shaped model with Q4_K matrices: the role of Executor::forward_greedy,
 *    crates/engine/src/forward.rs:1795-1975, with token id, position and arg-max kept on the device ── */
typedef struct {
    int32_t n_layers, hidden, n_heads, n_kv_heads, head_dim, vocab;
    int32_t n_experts, top_k, ff, max_seq, renorm;
    float   eps, theta;
} runit_model_cfg;
typedef struct {          /* device pointers; the model keeps them, the caller keeps the memory alive */
    const void* tok_emb;   /* f32 [vocab][hidden] */
    const void* attn_norm; /* f32 [L][hidden] */
    const void* ffn_norm;  /* f32 [L][hidden] */
    const void* out_norm;  /* f32 [hidden] */
    const void* wq;        /* Q4_K [L][n_heads*head_dim][hidden] */
    const void* wk;        /* Q4_K [L][n_kv_heads*head_dim][hidden] */
    const void* wv;        /* Q4_K [L][n_kv_heads*head_dim][hidden] */
    const void* wo;        /* Q4_K [L][hidden][n_heads*head_dim] */
    const void* router;    /* f32 [L][E][hidden] */
    const void* gate;      /* Q4_K [L][E][ff][hidden] */
    const void* up;        /* Q4_K [L][E][ff][hidden] */
    const void* down;      /* Q4_K [L][E][hidden][ff] */
    const void* lm_head;   /* Q4_K [vocab][hidden] */
} runit_model_weights;
typedef struct runit_model runit_model_t;
/* Allocates the f16 KV cache and all scratch, runs one warm-up step and records the per-token command lists. */
int32_t runit_model_create(runit_ctx_t* ctx, const runit_model_cfg* cfg, const runit_model_weights* weights, runit_model_t** out);
/* The same decoder with the experts split over `world` ranks (one process and context per GPU): weights->gate / up / down
 * hold this rank's experts [rank * E/world, (rank+1) * E/world) only ([L][E/world][...]), everything else is replicated and
 * every rank decodes the same token stream (runit_moe_layer_q4k_ep per layer, barrier epochs kept on the device so the
 * recorded command list can be replayed).  partial_all / signal_pads: as for runit_moe_layer_q4k_ep with T = 1.  All ranks
 * must call this (and every generate call) together: the warm-up step already runs the barriers. */
int32_t runit_model_create_ep(runit_ctx_t* ctx, const runit_model_cfg* cfg, const runit_model_weights* weights, uint32_t world,
                              uint32_t rank, void* const* partial_all, void* const* signal_pads, runit_model_t** out);
int32_t runit_model_destroy(runit_model_t* model);
int32_t runit_model_reset(runit_model_t* model, int32_t token, int32_t pos);
/* forward.rs:1795  one token at position pos -> arg-max next token (synchronous, like the reference) */
int32_t runit_model_forward_greedy(runit_model_t* model, int32_t token_id, int32_t pos, int32_t* next_token);
/* prompt (forced tokens) + n_gen greedy steps without host round trips; out_tokens: n_prompt+n_gen int32 on the host */
int32_t runit_model_generate_greedy(runit_model_t* model, const int32_t* prompt, uint32_t n_prompt, uint32_t n_gen,
                                    int32_t start_pos, int32_t skip_prompt_logits, int32_t* out_tokens);
/* The same loop with the sampler in place of the argmax (generate.rs:299, 346: the context of a draw is what has been
 * generated so far, empty for the first one).  eos_ids: host array, at most 16.  The command list of the sampled step is
 * recorded on first use and again whenever cfg changes. */
int32_t runit_model_generate_sampled(runit_model_t* model, const int32_t* prompt, uint32_t n_prompt, uint32_t n_gen,
                                     int32_t start_pos, const runit_sampler_cfg* cfg, uint64_t seed, const int32_t* eos_ids,
                                     uint32_t n_eos, int32_t* out_tokens);
/* Executor::prefill (crates/engine/src/prefill.rs:29-255): the whole prompt in one batched pass from an empty cache
 * (tensor-core GEMMs with bf16 operands over the Q4_K matrices, causal attention over the f16 cache, the batched MoE
 * block).  Afterwards the cache holds positions 0 .. n-1, *next_token is the argmax of the last position's logits, and
 * runit_model_generate_greedy(&next, 1, n_gen, n, ...) continues.  head_dim 64 or 128; tokens: host array. */
int32_t runit_model_prefill(runit_model_t* model, const int32_t* tokens, uint32_t n, int32_t* next_token);
/* The causal attention kernel of the prefill by itself: q f32 [T][heads*head_dim] (already rotated), caches f16
 * [kv_heads][max_seq][head_dim] holding positions 0 .. start_pos+T-1, out bf16 [T][heads*head_dim]; query t sees keys
 * 0 .. start_pos+t (attention.metal:36-158). */
int32_t runit_prefill_attention_f16kv(runit_ctx_t*, const void* q, const void* kcache, const void* vcache, void* out_bf16, uint32_t T,
                                      uint32_t heads, uint32_t kv_heads, uint32_t head_dim, uint32_t max_seq, uint32_t start_pos);
/* Dense feed-forward block of a prefill pass (prefill.rs:217-227: gemm_f16 gate, gemm_f16 up, silu_mul_f16, gemm_f16 down,
 * add_f16) on the tensor cores with bf16 operands: out[t] = residual[t] + Wd . bf16(silu(Wg . xb[t]) * (Wu . xb[t])), where
 * xb = bf16(x) or, when gamma is not NULL, bf16(RMSNorm(x) * gamma) (the rms_norm_f16 of prefill.rs:150-151).  x / residual /
 * out f32 [T][h] (residual may be NULL or equal to out); Q4_K matrices; scratch 1024-byte aligned. */
size_t  runit_ffn_q4k_bf16_scratch_bytes(uint32_t T, uint32_t h, uint32_t ff);
int32_t runit_ffn_q4k_bf16(runit_ctx_t*, const void* w_gate, const void* w_up, const void* w_down, const void* x, const void* gamma,
                           float eps, const void* residual, void* out, void* scratch, size_t scratch_bytes, uint32_t T, uint32_t h,
                           uint32_t ff);
/* A portion of a sequence through the batched pass: tokens at positions start_pos .. start_pos + n - 1 on top of the
 * start_pos cached ones (one token runs as a recorded decode step).  want: places inside the portion whose logits are
 * returned, logits: host, f32 [n_want][vocab] in the order of want.  Layered decoders only (RUNIT_ERR_UNSUPPORTED else);
 * start_pos must not exceed what the cache holds, a smaller one drops what comes after it. */
int32_t runit_model_forward(runit_model_t* model, const int32_t* tokens, uint32_t n, uint32_t start_pos, const uint32_t* want,
                            uint32_t n_want, float* logits);

/* ── operators over bf16 weight matrices (no twin): rows of pad8(k) elements, zero padding ── */
/* y[m] = W . x (+ residual, may be y); gain f32 [1] not NULL: x is first divided by its root mean square and multiplied by it */
int32_t runit_gemv_bf16_f32(runit_ctx_t*, const void* weight, const void* x, const void* gain, float eps, void* y, const void* residual,
                            uint32_t m, uint32_t k);
/* What becomes of a product: stored as f32; added to the f32 output; stored in the activation type; pairs of rows (2i, 2i+1)
 * as silu(g) * u, or max(v, 0)^2, in the activation type.  pre / post (f32 per token, may be NULL) multiply the product / the
 * activated value of the last two. */
enum { RUNIT_EPI_F32 = 0, RUNIT_EPI_ADD = 1, RUNIT_EPI_CAST = 2, RUNIT_EPI_SILU_GLU = 3, RUNIT_EPI_RELU2 = 4 };
/* y[T][outputs] = epilogue(W[m][k] . x[t]); x rows of pad8(k) elements: bf16 on the tensor cores (exact = 0; the activation
 * type is bf16), or f32 with f32 multiply-adds (exact = 1; f32).  y rows of ldy elements. */
int32_t runit_gemm_bf16_rows(runit_ctx_t*, const void* weight, const void* x, void* y, uint32_t ldy, uint32_t T, uint32_t m, uint32_t k,
                             int32_t exact, int32_t epi, const void* pre, const void* post);
/* y[t] = x[t] / sqrt(mean(x[t]^2) + eps) * gain[0], x f32 [T][width], y f32 or bf16 rows of pad8(width) */
int32_t runit_norm_gain_rows(runit_ctx_t*, const void* x, const void* gain, float eps, void* y, int32_t y_f32, uint32_t T, uint32_t width);
/* Latent attention.  One cache row per position: the normed latent (kv_rank values padded to a multiple of 16), then the
 * rotated shared key part (rot_dim padded likewise), bf16 or f32 (cache_f32).  qkv: f32 rows of ldq values, the queries of all
 * heads [dim | rot_dim] and then, when kv_norm is not NULL, the raw latent and key part of the token, which become the cache
 * row of its position.  freq f32 [rot_dim / 2]: angle = position * freq[i] for the pair (2i, 2i+1). */
typedef struct {
    uint32_t heads, dim, rot_dim, vdim, kv_rank;
    float    scale, eps;
} runit_latent_cfg;
/* folded queries q_eff [T * heads][row] (row = elements of a cache row): [W_uk^T q_un | rotated q_rot], f32 with an f32 cache,
 * else the high bf16 parts of a row followed by its low parts; w_uk [heads*dim][pad8(kv_rank)] */
int32_t runit_latent_query(runit_ctx_t*, const runit_latent_cfg* cfg, int32_t cache_f32, const void* qkv, uint32_t ldq, const void* w_uk,
                           const void* kv_norm, const void* freq, void* cache, void* q_eff, uint32_t T, uint32_t start);
/* softmax over positions 0 .. start+t per (token, head), keys split nsplit ways: part_o f32 [T*heads][nsplit][pad16(kv_rank)]
 * (weighted latent sums), part_ml f32 [T*heads][nsplit][2] (maximum, sum of weights) */
int32_t runit_latent_attention(runit_ctx_t*, const runit_latent_cfg* cfg, int32_t cache_f32, const void* q_eff, const void* cache,
                               void* part_o, void* part_ml, uint32_t nsplit, uint32_t T, uint32_t start);
/* merges the splits and applies W_uv [heads*vdim][pad8(kv_rank)]: out f32 [T][heads*vdim] */
int32_t runit_latent_value(runit_ctx_t*, const runit_latent_cfg* cfg, const void* part_o, const void* part_ml, uint32_t nsplit,
                           const void* w_uv, void* out, uint32_t T);
/* cache rows (bf16 or f32) of T tokens, and the rotated parts of their queries in place */
int32_t runit_latent_rows(runit_ctx_t*, const runit_latent_cfg* cfg, int32_t cache_f32, void* qkv, uint32_t ldq, const void* kv_norm,
                          const void* freq, void* cache, uint32_t T, uint32_t start);
/* the same attention over expanded keys and values, kv bf16 [start + T][ldkv] = [keys of all heads (dim each) | values (vdim)];
 * q f32 with rotated parts; bf16 cache (for the shared key part); out bf16 [T][ldo].  dim, rot_dim, vdim multiples of 8,
 * dim + rot_dim <= 192, vdim <= 128, ldq even, ldkv a multiple of 8, ldo even. */
int32_t runit_latent_prefill_attention(runit_ctx_t*, const runit_latent_cfg* cfg, const void* q, uint32_t ldq, const void* kv, uint32_t ldkv,
                                       const void* cache, void* out, uint32_t ldo, uint32_t T, uint32_t start);

/* Attention over cached keys and values per head.  A projected row holds [q: heads x dim | k: kv_heads x dim | v: kv_heads x
 * vdim]; query head h uses key head h / (heads / kv_heads).  Score (q . k) * scale - slopes[h] * (i - j) (slopes f32 [heads] or
 * NULL); window 0: all earlier positions, else a position sees itself and the window - 1 before it; unit_qk: q and k are divided by
 * their root mean square.  Caches: bf16 or f32 (cache_f32), [kv_heads][cap][dim, vdim padded to 8], position p in row p % cap. */
typedef struct {
    uint32_t heads, kv_heads, dim, vdim, window, cap, unit_qk;
    float    scale, out_scale, eps;
    const void* slopes;
    void*    k_cache;
    void*    v_cache;
} runit_heads_cfg;
/* Retention, S <- decay_h S + k v^T, o = S^T q.  A projected row holds [q, k: heads x dim | v, gate: heads x vdim]; the first
 * rot_dims coordinates of q and k rotate (pairs (i, i + rot_dims/2), angle position * (freq[0][i] + freq[1][i]), freq f32
 * [2][rot_dims/2]: the frequencies and what their rounding to f32 has left), k is multiplied by dim^(-1/2).  decay f32 [2][heads]: the decays, then their logarithms; state f32 [heads][dim][vdim]. */
typedef struct {
    uint32_t heads, dim, vdim, rot_dims;
    float    out_scale;
    const void* freq;
    const void* decay;
    void*    state;
} runit_retention_cfg;
/* State-space layer.  A projected row holds [z: heads x vdim | x: heads x vdim | B, C: groups x state_dim | dt: heads]; the other
 * fields are those of runit_layer_desc; state f32 [heads][state_dim][vdim]; ring f32 [taps][channels]: the inputs of the
 * convolution at position p in row p % taps. */
typedef struct {
    uint32_t heads, vdim, state_dim, groups, taps;
    const void* conv;
    const void* conv_b;
    const void* dt_bias;
    const void* a;
    const void* skip;
    void*    state;
    void*    ring;
} runit_ssm_cfg;
/* One token at position *pos (device int32): attention and / or retention (either NULL) on one f32 projected row; writes the
 * position's cache row and the state.  ao f32 = [attention * out_scale | retention o], factor f32 = silu(gate) * out_scale of the
 * retention, squares f32 [heads][ceil(vdim / 32)] = sums of o^2 over slices of 32 columns.  part f32 [heads * nsplit * (vdim + 2)],
 * tickets uint32 [4096], zero (zero again afterwards); nsplit <= 64.  Cache, state and pos must not be outputs of the launch in
 * front of this one (they are read before it has ended). */
int32_t runit_heads_step(runit_ctx_t*, const runit_heads_cfg* attn, const runit_retention_cfg* ret, int32_t cache_f32, const void* proj, void* ao,
                         void* factor, void* squares, void* part, void* tickets, uint32_t nsplit, const void* pos);
/* T tokens, projected rows of ld elements (bf16, or f32 with an f32 cache): cache rows of their positions, rotated q and k of the
 * retention in place (k scaled); then attention over them: out rows of ldo, the same type.  part: part_floats f32 (any number). */
int32_t runit_heads_rows(runit_ctx_t*, const runit_heads_cfg* attn, const runit_retention_cfg* ret, int32_t cache_f32, void* proj, uint32_t ld,
                         uint32_t T, uint32_t start);
int32_t runit_head_attention_rows(runit_ctx_t*, const runit_heads_cfg* attn, int32_t cache_f32, const void* proj, uint32_t ld, void* out,
                                  uint32_t ldo, uint32_t T, uint32_t start, void* part, size_t part_floats, void* tickets);
/* One token of a state-space layer: y f32 [heads * vdim] = (S^T C + skip x) * silu(z), squares f32 [heads][ceil(vdim / 32)] its sums
 * of squares over slices of 32 columns.  The state must not be an output of the launch in front of this one. */
int32_t runit_ssm_step(runit_ctx_t*, const runit_ssm_cfg* cfg, const void* proj, void* y, void* squares, const void* pos);
/* T tokens: x, B, C convolved and activated into rows of ldx (bf16 or f32); dt f32 [T][heads] becomes softplus(dt + dt_bias). */
int32_t runit_ssm_conv_rows(runit_ctx_t*, const runit_ssm_cfg* cfg, int32_t f32, const void* proj, uint32_t ld, void* xbc, uint32_t ldx, void* dt,
                            uint32_t T, uint32_t start);
/* The recurrence over T tokens: q, k [groups][dk] and v [heads][dv] per token (rows of ldq, ldk, ldv, bf16 or f32), head h uses group
 * h / (heads / groups).  dt f32 [T][heads]: decay exp(log_decay[h] * dt), k times dt; dt NULL: decay[h] (and its logarithm).  skip
 * f32 [heads] or NULL: o += skip[h] v.  start 0: from a zero state.  scratch: runit_linear_scratch_bytes (NULL: token by token). */
typedef struct {
    uint32_t heads, groups, dk, dv, ldq, ldk, ldv, ldo;
    const void* q;
    const void* k;
    const void* v;
    const void* dt;
    const void* log_decay;
    const void* decay;
    const void* skip;
    void*    state;
    void*    out;
} runit_linear_cfg;
size_t  runit_linear_scratch_bytes(uint32_t heads, uint32_t dk, uint32_t dv, uint32_t T);
int32_t runit_linear_rows(runit_ctx_t*, const runit_linear_cfg* cfg, int32_t f32, void* scratch, uint32_t T, uint32_t start);
/* Groups of `group` values of the n in every row of a (in place): before: a * silu(gate), normed, times weight (f32 [n]); else a
 * normed, times silu(gate) * out_scale. */
int32_t runit_gated_norm_rows(runit_ctx_t*, int32_t f32, void* a, uint32_t lda, uint32_t n, uint32_t group, const void* gate, uint32_t ldg,
                              int32_t before, const void* weight, float out_scale, float eps, uint32_t T);
/* x[t] += norm(y[t]) (y NULL: x stays), a gain per coordinate; out (may be NULL) = x in rows of pad8(width), or norm(x) with
 * out_gain when that is not NULL */
int32_t runit_add_norm_rows(runit_ctx_t*, void* x, const void* y, const void* gain, float eps, const void* out_gain, void* out, int32_t out_f32,
                            uint32_t T, uint32_t width);
/* out[m] = W . v (cap != 0: cap * tanh(. / cap)) with v = x + norm(y) (gain y_gain per coordinate; y NULL: v = x), stored in x_out,
 * and then norm(v) with `gain` when that is not NULL.  relu2: max(., 0)^2 instead of cap. */
int32_t runit_gemv_bf16_residual_f32(runit_ctx_t*, const void* weight, const void* x, const void* y, const void* y_gain, const void* gain, void* x_out,
                                     void* out, float eps, float cap, int32_t relu2, uint32_t m, uint32_t k);
/* out[m] = W . v: the first `plain` values of v are x, the others groups of `group` values of x, normed, times factor [k - plain];
 * squares (may be NULL): f32 [groups][squares_n], sums of squares that add up to those of the groups */
int32_t runit_gemv_bf16_groups_f32(runit_ctx_t*, const void* weight, const void* x, const void* factor, const void* squares, uint32_t squares_n,
                                   void* out, float eps, uint32_t plain, uint32_t group, uint32_t m, uint32_t k);

/* ── decoders described layer by layer (no twin), weights in bf16 ──
 * Every matrix is row-major [rows][pad8(columns)] bf16 with zero padding; norms and router are f32.  Linear maps W x.
 * Residual stream, norms, scores, softmax, router, angles and recurrent state are f32.  norm(x) = x / sqrt(mean(x^2) + eps) * gain.
 *   post_norm = 0: x += mixer(norm1(x));  x += ff(norm2(x));  one gain for all coordinates.
 *   post_norm = 1: x += norm1(mixer(x));  x += norm2(ff(x));  a gain per coordinate (dense feed-forward only).
 * A decoder with retention or state-space layers carries state from token to token: a pass starts at position 0 (from a zero
 * state) or where the last one ended.
 * exact = 0: activations and cache bf16 with f32 accumulation (batched passes on the tensor cores); exact = 1: activations
 * and cache f32 throughout.  The step, the generate and sampling loops, prefill and forward are those of any runit_model_t. */
enum { RUNIT_FF_NONE = 0, RUNIT_FF_DENSE = 1, RUNIT_FF_MOE = 2 };
enum { RUNIT_MIX_LATENT = 0,      /* latent attention */
       RUNIT_MIX_HEADS = 1,       /* attention over keys and values per head and / or retention, side by side */
       RUNIT_MIX_SSM = 2 };       /* state-space layer with a scalar decay per head and token */
enum { RUNIT_ACT_SILU_GLU = 0,    /* rows 2i and 2i+1 of the up matrix are gate and up of unit i: silu(g) * u */
       RUNIT_ACT_RELU2 = 1 };     /* max(u, 0)^2 */
typedef struct {
    /* latent attention: q rows [heads][dim | rot_dim]; latent of kv_rank values and a rotated key part of rot_dim values per
     * position, in the cache of this layer (kv_from < 0) or of the earlier layer kv_from.  Rotation: pairs (2i, 2i+1), angle
     * position * rot_base^(-2i/rot_dim). */
    int32_t heads, dim, rot_dim, vdim, kv_rank, kv_from;
    float   scale, rot_base;
    /* feed-forward: ff units (per expert for RUNIT_FF_MOE); routing weights are the scores of the top_k largest of n_experts,
     * and multiply an expert's input; a shared block of shared_ff units (0 = none) runs for every token, its output times the
     * sigmoid of its own gate row */
    int32_t ff_kind, ff_act, ff, n_experts, top_k, score, renorm, shared_ff;
    const void* norm1;        /* f32 [1] ([width] with post_norm) */
    const void* norm2;        /* the same; NULL without feed-forward */
    /* projections of the mixer's input, one under the other.  Latent attention: [heads*(dim+rot_dim) (+ kv_rank+rot_dim when the
     * layer owns its latent)][width]; RUNIT_MIX_HEADS: q, k, v of the attention, then q, k, v, gate of the retention;
     * RUNIT_MIX_SSM: gate, x, B, C, step sizes */
    const void* w_q;
    const void* kv_norm;      /* f32 [kv_rank]; NULL when kv_from >= 0 */
    const void* w_ukv;        /* [heads*dim + heads*vdim][kv_rank]: keys of all heads, then values */
    const void* w_o;          /* [width][outputs of the mixer]; RUNIT_MIX_HEADS: attention heads, then retention heads */
    const void* ff_up;        /* [ff (2 ff for a gated block)][width], experts stacked */
    const void* ff_down;      /* [width][ff], experts stacked */
    const void* router;       /* f32 [n_experts (+ 1 gate row of the shared block)][width], no padding */
    const void* shared_up;    /* [shared_ff (2 shared_ff)][width] */
    const void* shared_down;  /* [width][shared_ff] */
    int32_t mixer;
    /* RUNIT_MIX_HEADS, attention (at_heads = 0: none): query head h uses key / value head h / (at_heads / at_kv_heads); score
     * (q . k) * at_scale - at_slopes[h] * (i - j); position i sees the at_window positions up to its own (0: all of them);
     * at_unit_qk: q and k are divided by their root mean square per head; the output is multiplied by at_out_scale */
    int32_t at_heads, at_kv_heads, at_dim, at_vdim, at_window, at_unit_qk;
    /* retention (rt_heads = 0: none): S <- decay_h S + k v^T, o = S^T q; the first rt_rot_dims coordinates of q and k are rotated
     * (pairs (i, i + rt_rot_dims / 2), angle position * rt_rot_base^(-2i / rt_rot_dims)), k is multiplied by rt_dim^(-1/2); o is
     * divided by its root mean square per head and multiplied by silu(gate) and rt_out_scale */
    int32_t rt_heads, rt_dim, rt_vdim, rt_rot_dims;
    /* RUNIT_MIX_SSM: x, B, C pass a causal convolution over ss_taps tokens and silu; dt = softplus(. + ss_dt_bias);
     * S <- exp(ss_a dt) S + dt B x^T, y = (S^T C + ss_skip x) * silu(gate), normed in ss_norm_groups parts */
    int32_t ss_heads, ss_vdim, ss_state, ss_groups, ss_taps, ss_norm_groups;
    float   at_scale, at_out_scale, rt_rot_base, rt_out_scale;
    const void* at_slopes;    /* f32 [at_heads]; NULL: no bias */
    const void* rt_decay;     /* f32 [2][rt_heads]: the decays, then their logarithms */
    const void* ss_conv;      /* f32 [channels][ss_taps], last column: the current token; channels = ss_heads*ss_vdim + 2*ss_groups*ss_state */
    const void* ss_conv_b;    /* f32 [channels] */
    const void* ss_dt_bias;   /* f32 [ss_heads] */
    const void* ss_a;         /* f32 [ss_heads], negative: logarithm of the decay per unit of dt */
    const void* ss_skip;      /* f32 [ss_heads] */
    const void* ss_norm;      /* f32 [ss_heads*ss_vdim] */
} runit_layer_desc;
typedef struct {
    int32_t n_layers, width, vocab, max_seq, exact, post_norm;
    float   eps, embed_scale;   /* embed_scale: factor of the embedding when embed_norm is NULL */
    float   logit_cap;          /* 0: none; else logits = cap * tanh(logits / cap) */
} runit_layered_cfg;
typedef struct {
    const void* embed;        /* [vocab][width] */
    const void* embed_norm;   /* f32 [1]; NULL: no norm */
    const void* final_norm;   /* f32 [1] ([width] with post_norm) */
    const void* head;         /* [vocab][width] */
} runit_layered_weights;
/* Device pointers; the model keeps them, the caller keeps the memory alive. */
int32_t runit_model_create_layered(runit_ctx_t* ctx, const runit_layered_cfg* cfg, const runit_layer_desc* layers,
                                   const runit_layered_weights* weights, runit_model_t** out);
/* Device pointer, f32 [n][width]: the residual stream of the last portion's tokens after its last layer; and the number of
 * layers a portion runs (tests bring a model up layer by layer): n_layers < 0 restores all of them. */
void*   runit_model_residual(runit_model_t* model);
int32_t runit_model_set_depth(runit_model_t* model, int32_t n_layers);
void*   runit_model_logits(runit_model_t* model);           /* device pointer, f32 [vocab], of the last step */
uint64_t runit_model_launches_per_token(runit_model_t* model);

/* Synthetic weights written on the device (benchmark / test data, distributions of the
 * benchmark configurations): n_blocks blocks of the format from a counter-based generator. */
int32_t runit_fill_weights(runit_ctx_t*, int32_t fmt, void* dst, uint64_t n_blocks, uint64_t seed, float sigma);
/* Q4_K blocks whose weights have zero mean: dmin = f16(7.5 d) and min index = scale index in every sub-block, so that
 * d*sc*q - dmin*m = d*sc*(q - 7.5).  With the benchmark's distributions every weight has a positive mean and a
 * random-init decoder repeats one token; the parity tests of the full decoder use this variant so that the greedy
 * token stream depends on its input. */
int32_t runit_fill_weights_q4k_zero_mean(runit_ctx_t*, void* dst, uint64_t n_blocks, uint64_t seed, float sigma);
/* N(0, sigma) f32 values from the same generator. */
int32_t runit_fill_normal_f32(runit_ctx_t*, void* dst, uint64_t n, uint64_t seed, float sigma);

#ifdef __cplusplus
}
#endif
#endif
