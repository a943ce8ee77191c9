// OLMoE-style mixture-of-experts block on the device, without the reference's per-layer host sync.
//
// Reference sequence (crates/engine/src/forward.rs:1644-1679): router GEMV -> flush -> CPU
// softmax/top-k (forward.rs:2420-2448) -> per selected expert: gate GEMV, up GEMV, silu*up, down
// GEMV, scale-accumulate -> residual add.  Here: router GEMV, device softmax/top-k, ONE grouped
// launch for gate+up+SiLU of all (token, expert) slots, ONE grouped launch for down, and a combine
// kernel that adds the weighted expert outputs in routing order (deterministic) plus the residual.
// All intermediates are f32.
#include "decode_ops.cuh"
#include "gemv_common.cuh"
#include "moe_internal.h"
#include "runit_internal.h"
#include "tma.cuh"

namespace runit {

// out[t][r] = (res ? res[t][r] : 0) + sum_i w[t][i] * y[t*k+i][r], i ascending (routing order).
__global__ void __launch_bounds__(256) moe_combine_kernel(const float* __restrict__ y, const float* __restrict__ w,
                                                           const float* res, float* out, uint32_t T, uint32_t h, uint32_t k) {
    grid_dependency_wait();      // inputs come from the previous kernel of the chain
    grid_launch_dependents();
    const uint32_t r = blockIdx.x * blockDim.x + threadIdx.x, t = blockIdx.y;
    if (r >= h) return;
    float acc = 0.f;
    for (uint32_t i = 0; i < k; i++) acc = fmaf(w[(size_t)t * k + i], y[((size_t)t * k + i) * h + r], acc);
    const size_t o = (size_t)t * h + r;
    out[o] = (res ? res[o] : 0.f) + acc;
}

struct MoeScratch {
    float* logits;   // [T][E]
    int32_t* idx;    // [T][k]
    float* w;        // [T][k]
    float* act;      // [T*k][ff]
    float* y;        // [T*k][h]
    size_t bytes;
};

// Expert-parallel decode block, replicated tokens.  This rank's weighted sum over the slots whose expert it owns
// (routing order), stored into slot `rank` of the partial buffer of every rank: plain stores into peer memory.
struct EpPeers {
    float* p[8];   // rank r's partial buffer [world][T][h], as mapped into this process
};
// The partial buffers have two halves that alternate by epoch parity.  The epoch is either given (call-by-call use)
// or read from a device word that the barrier kernel advances (recorded command lists: the same launch runs every token).
// (One launch that pushes the partial sums, lets its last CTA run the barrier and add everything was measured slower
// than these three: 37.6 vs 33.2 us per layer at one token, 172 vs 102 us at 16, two ranks.)
__global__ void __launch_bounds__(256) ep_partial_kernel(const float* __restrict__ y, const float* __restrict__ w,
                                                          const int32_t* __restrict__ idx, const EpPeers peers, uint32_t world,
                                                          uint32_t rank, int32_t lo, uint32_t cnt, uint32_t T, uint32_t h, uint32_t k,
                                                          uint32_t epoch, const uint32_t* __restrict__ epoch_ptr) {
    grid_dependency_wait();
    grid_launch_dependents();
    const uint32_t c = blockIdx.x * 256 + threadIdx.x, t = blockIdx.y;
    if (c >= h) return;
    const size_t half = (size_t)((epoch_ptr ? *epoch_ptr + 1u : epoch) & 1u) * world * T * h;
    float acc = 0.f;
    for (uint32_t i = 0; i < k; i++) {
        const int32_t e = idx[t * k + i] - lo;
        if (e >= 0 && (uint32_t)e < cnt) acc = fmaf(w[t * k + i], y[(size_t)(t * k + i) * h + c], acc);
    }
    const size_t o = half + ((size_t)rank * T + t) * h + c;
    for (uint32_t p = 0; p < world; p++) peers.p[p][o] = acc;
}
// out[t] = residual[t] + sum over ranks (rank order) of the partial sums that arrived in this rank's buffer.
// `out` may be the same buffer as `residual` (the decoder adds into its hidden state in place): neither is restrict.
__global__ void __launch_bounds__(256) ep_reduce_kernel(const float* __restrict__ partial, const float* residual,
                                                         float* out, uint32_t world, uint32_t T, uint32_t h,
                                                         uint32_t epoch, const uint32_t* __restrict__ epoch_ptr) {
    const uint32_t c = blockIdx.x * 256 + threadIdx.x, t = blockIdx.y;
    if (c >= h) return;
    partial += (size_t)((epoch_ptr ? *epoch_ptr : epoch) & 1u) * world * T * h;   // the barrier has advanced the word already
    float acc = residual ? residual[(size_t)t * h + c] : 0.f;
    for (uint32_t r = 0; r < world; r++) acc += partial[((size_t)r * T + t) * h + c];
    out[(size_t)t * h + c] = acc;
}

static MoeScratch moe_carve(void* base, uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k) {
    auto up = [](size_t v) { return (v + 255) / 256 * 256; };
    uint8_t* p = reinterpret_cast<uint8_t*>(base);
    MoeScratch s;
    size_t o = 0;
    s.logits = reinterpret_cast<float*>(p + o); o += up((size_t)T * E * 4);
    s.idx = reinterpret_cast<int32_t*>(p + o); o += up((size_t)T * k * 4);
    s.w = reinterpret_cast<float*>(p + o); o += up((size_t)T * k * 4);
    s.act = reinterpret_cast<float*>(p + o); o += up((size_t)T * k * ff * 4);
    s.y = reinterpret_cast<float*>(p + o); o += up((size_t)T * k * h * 4);
    s.bytes = o;
    return s;
}

size_t moe_scratch_bytes_impl(uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k) {
    return moe_carve(nullptr, T, h, ff, E, k).bytes;
}

// The whole block; scratch carved from `scratch`.
int32_t moe_layer_q4k_impl(runit_ctx* ctx, const void* router_w, const void* gate, const void* up, const void* down,
                           const void* x, const void* residual, void* out, int32_t* idx_out, float* w_out, void* scratch,
                           size_t scratch_bytes, uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm,
                           const float* next_gamma, float* next_xn, float next_eps, uint32_t* route_counter,
                           const float* pre_x, const float* pre_gamma, float pre_eps) {
    RUNIT_REQUIRE(ctx, router_w && gate && up && down && x && out && scratch, "moe_layer_q4k: null pointer");
    RUNIT_REQUIRE(ctx, T > 0 && T <= 65536, "moe_layer_q4k: T=%u out of range", T);
    RUNIT_REQUIRE(ctx, h % 256 == 0 && ff % 256 == 0 && h > 0 && ff > 0, "moe_layer_q4k: h=%u, ff=%u must be multiples of 256", h, ff);
    RUNIT_REQUIRE(ctx, E > 0 && E <= 256 && k > 0 && k <= E && k <= 32, "moe_layer_q4k: E=%u, k=%u unsupported", E, k);
    RUNIT_REQUIRE(ctx, runit_aligned(scratch, 256), "moe_layer_q4k: scratch must be 256-byte aligned");
    const MoeScratch s = moe_carve(scratch, T, h, ff, E, k);
    if (s.bytes > scratch_bytes)
        return runit_fail(ctx, RUNIT_ERR_BUFFER_SIZE, "moe_layer_q4k: scratch has %zu bytes, needs %zu", scratch_bytes, s.bytes);
    int32_t* idx = idx_out ? idx_out : s.idx;
    float* wts = w_out ? w_out : s.w;
    int32_t st;
    // pre_gamma != nullptr: the block starts with the RMSNorm of pre_x (the un-normalised hidden state, another buffer than
    // x) into x, which the router and the experts then consume; one token takes it inside the routing launch, else it is a
    // launch of its own
    const bool fused_route = route_counter && T == 1 && (h == 1024 || h == 2048 || h == 4096) && runit_aligned(router_w, 16) && runit_aligned(x, 16) &&
                             (!pre_gamma || (pre_x && pre_x != x && runit_aligned(pre_x, 16)));
    float* pre_out = pre_gamma ? (float*)const_cast<void*>(x) : nullptr;
    const float* x_route = pre_gamma ? pre_x : (const float*)x;
    if (pre_gamma && !fused_route) {
        RUNIT_REQUIRE(ctx, pre_x, "moe_layer_q4k: null pre-norm input");
        if ((st = launch_rms_norm(ctx, pre_x, pre_out, pre_gamma, false, pre_eps, h, T)) != RUNIT_OK) return st;
        pre_gamma = nullptr;
        x_route = (const float*)x;
    }
    if (fused_route) {
        // one token: router GEMV and routing in one launch (same bits as the two launches below)
        const dim3 grid((E + 7) / 8);
        st = moe_route_fused(ctx, (const float*)router_w, x_route, s.logits, E, h, k, renorm, idx, wts, route_counter, pre_gamma, pre_eps, pre_out);
        if ((st = runit_after_launch(ctx, "moe_route_fused")) != RUNIT_OK) return st;
    } else {
        st = moe_router(ctx, (const float*)router_w, (const float*)x, s.logits, E, h, T);
        if (st != RUNIT_OK) return st;
        st = moe_topk(ctx, s.logits, E, k, renorm, T, idx, wts);
        st = runit_after_launch(ctx, "moe_route_topk");
        if (st != RUNIT_OK) return st;
    }
    const uint32_t slots = T * k;
    // gate+up+SiLU for every (token, expert) slot: act[s][ff]
    const bool fused_sum = fused_route && h <= 32 * 960;
    st = gemv_grouped(ctx, "moe_gate_up", RUNIT_FMT_Q4K, gate, up, E, ff, h, x, k, s.act, idx, slots, 0, nullptr, nullptr, nullptr,
                      nullptr, fused_sum ? 1 : 0);
    if (st != RUNIT_OK) return st;
    // down: y[s][h] = Wd[e_s] . act[s]
    if (fused_sum) {
        // one token: the last down-projection tile of every 32 rows adds the experts' rows (same order as moe_combine_kernel)
        st = gemv_grouped(ctx, "moe_down", RUNIT_FMT_Q4K, down, nullptr, E, h, ff, s.act, 1, s.y, idx, slots, 0, wts,
                          (const float*)residual, (float*)out, route_counter + 32, 2);
        if (st != RUNIT_OK || !next_gamma) return st;
        return launch_rms_norm(ctx, (const float*)out, next_xn, next_gamma, false, next_eps, h, T);
    }
    st = gemv_grouped(ctx, "moe_down", RUNIT_FMT_Q4K, down, nullptr, E, h, ff, s.act, 1, s.y, idx, slots);
    if (st != RUNIT_OK) return st;
    runit_launch_chain(ctx, moe_combine_kernel, dim3((h + 255) / 256, T), dim3(256), (const float*)s.y, (const float*)wts, (const float*)residual, (float*)out, T, h, k);
    st = runit_after_launch(ctx, "moe_combine");
    if (st != RUNIT_OK || !next_gamma) return st;
    return launch_rms_norm(ctx, (const float*)out, next_xn, next_gamma, false, next_eps, h, T);
}

// ───────────────────────── built-in scratch (entry point that allocates nothing) ─────────────────────────
// A fixed region inside the library's own device image.  Every GPU that loads the library carries it
// until the process exits.  In host code `g_moe_static_scratch` is only a stand-in for the symbol, never a
// device address: the address a kernel may use comes from cudaGetSymbolAddress, asked once per device
// with that device current.
constexpr size_t kMoeStaticScratchBytes = 4u << 20;   // 4 MiB
static __device__ __align__(256) unsigned char g_moe_static_scratch[kMoeStaticScratchBytes];

static int32_t moe_static_scratch(runit_ctx* ctx, void** out) {
    static void* per_device[64] = {nullptr};
    *out = nullptr;
    if (ctx->device < 0 || ctx->device >= 64) return runit_fail(ctx, RUNIT_ERR_UNSUPPORTED, "device index %d out of range", ctx->device);
    if (!per_device[ctx->device]) {
        int cur = -1;
        RUNIT_CUDA_TRY(ctx, cudaGetDevice(&cur));
        if (cur != ctx->device) RUNIT_CUDA_TRY(ctx, cudaSetDevice(ctx->device));
        void* p = nullptr;
        cudaError_t e = cudaGetSymbolAddress(&p, g_moe_static_scratch);
        if (cur != ctx->device) cudaSetDevice(cur);
        if (e != cudaSuccess || !p)
            return runit_fail(ctx, RUNIT_ERR_LAUNCH, "cudaGetSymbolAddress(built-in MoE scratch): %s", cudaGetErrorString(e));
        per_device[ctx->device] = p;
    }
    *out = per_device[ctx->device];
    return RUNIT_OK;
}

// The expert-parallel block behind runit_moe_layer_q4k_ep; epoch_ptr != nullptr: the epoch lives in that device word.
int32_t moe_layer_q4k_ep_impl(runit_ctx* ctx, const void* router_w, const void* gate_local, const void* up_local,
                              const void* down_local, const void* x, const void* residual, void* out, void* idx_out, void* w_out,
                              void* scratch, size_t scratch_bytes, void* const* partial_all, void* const* signal_pads,
                              uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm, uint32_t world,
                              uint32_t rank, uint32_t epoch, uint32_t* epoch_ptr, uint32_t* route_counter, const float* pre_x,
                              const float* pre_gamma, float pre_eps) {
    RUNIT_REQUIRE(ctx, router_w && gate_local && up_local && down_local && x && out && scratch && partial_all && signal_pads,
                  "moe_layer_q4k_ep: null pointer");
    RUNIT_REQUIRE(ctx, world >= 1 && world <= 8 && rank < world && E % world == 0 && (epoch > 0 || epoch_ptr),
                  "moe_layer_q4k_ep: world=%u rank=%u E=%u unsupported (1..8 ranks, experts divisible)", world, rank, E);
    RUNIT_REQUIRE(ctx, T > 0 && T <= 4096, "moe_layer_q4k_ep: T=%u out of range (replicated tokens, decode sizes)", T);
    RUNIT_REQUIRE(ctx, h % 256 == 0 && ff % 256 == 0 && h > 0 && ff > 0, "moe_layer_q4k_ep: h=%u, ff=%u must be multiples of 256", h, ff);
    RUNIT_REQUIRE(ctx, E > 0 && E <= 256 && k > 0 && k <= E && k <= 32, "moe_layer_q4k_ep: E=%u, k=%u unsupported", E, k);
    RUNIT_REQUIRE(ctx, runit_aligned(scratch, 256), "moe_layer_q4k_ep: scratch must be 256-byte aligned");
    const MoeScratch s = moe_carve(scratch, T, h, ff, E, k);
    if (s.bytes > scratch_bytes)
        return runit_fail(ctx, RUNIT_ERR_BUFFER_SIZE, "moe_layer_q4k_ep: scratch has %zu bytes, needs %zu", scratch_bytes, s.bytes);
    EpPeers peers{};
    for (uint32_t p = 0; p < world; p++) {
        RUNIT_REQUIRE(ctx, partial_all[p] && runit_aligned(partial_all[p], 4), "moe_layer_q4k_ep: null or misaligned partial buffer %u", p);
        // the two halves of a partial buffer alternate by epoch parity (in the kernels): a fast rank's next call cannot
        // overwrite what a slow rank is still adding (it would first have to pass the next barrier, which the slow rank
        // announces after its sum)
        peers.p[p] = (float*)partial_all[p];
    }
    int32_t* idx = idx_out ? (int32_t*)idx_out : s.idx;
    float* wts = w_out ? (float*)w_out : s.w;
    // every rank routes every token itself (the router is replicated): no dispatch exchange
    int32_t st;
    const bool fused_route = route_counter && T == 1 && (h == 1024 || h == 2048 || h == 4096) && runit_aligned(router_w, 16) && runit_aligned(x, 16) &&
                             (!pre_gamma || (pre_x && pre_x != x && runit_aligned(pre_x, 16)));
    float* pre_out = pre_gamma ? (float*)const_cast<void*>(x) : nullptr;
    const float* x_route = pre_gamma ? pre_x : (const float*)x;
    if (pre_gamma && !fused_route) {
        RUNIT_REQUIRE(ctx, pre_x, "moe_layer_q4k_ep: null pre-norm input");
        if ((st = launch_rms_norm(ctx, pre_x, pre_out, pre_gamma, false, pre_eps, h, T)) != RUNIT_OK) return st;
        pre_gamma = nullptr;
        x_route = (const float*)x;
    }
    if (fused_route) {
        // one token: (RMSNorm,) router GEMV and routing in one launch (same bits as the separate launches)
        const dim3 grid((E + 7) / 8);
        st = moe_route_fused(ctx, (const float*)router_w, x_route, s.logits, E, h, k, renorm, idx, wts, route_counter, pre_gamma, pre_eps, pre_out);
        if ((st = runit_after_launch(ctx, "moe_route_fused")) != RUNIT_OK) return st;
    } else {
        if ((st = moe_router(ctx, (const float*)router_w, (const float*)x, s.logits, E, h, T)) != RUNIT_OK) return st;
        st = moe_topk(ctx, s.logits, E, k, renorm, T, idx, wts);
        if ((st = runit_after_launch(ctx, "moe_route_topk")) != RUNIT_OK) return st;
    }
    const uint32_t n_local = E / world, slots = T * k;
    const int32_t lo = (int32_t)(rank * n_local);
    // only the slots of this rank's experts are computed (the others are unused slots of the grouped launches)
    st = gemv_grouped(ctx, "moe_gate_up_ep", RUNIT_FMT_Q4K, gate_local, up_local, n_local, ff, h, x, k, s.act, idx, slots, lo);
    if (st != RUNIT_OK) return st;
    st = gemv_grouped(ctx, "moe_down_ep", RUNIT_FMT_Q4K, down_local, nullptr, n_local, h, ff, s.act, 1, s.y, idx, slots, lo);
    if (st != RUNIT_OK) return st;
    runit_launch_chain(ctx, ep_partial_kernel, dim3((h + 255) / 256, T), dim3(256), (const float*)s.y, (const float*)wts, (const int32_t*)idx,
                       peers, world, rank, lo, n_local, T, h, k, epoch, (const uint32_t*)epoch_ptr);
    if ((st = runit_after_launch(ctx, "moe_ep_partial")) != RUNIT_OK) return st;
    if ((st = peer_barrier_launch(ctx, signal_pads, world, rank, epoch, epoch_ptr)) != RUNIT_OK) return st;
    ep_reduce_kernel<<<dim3((h + 255) / 256, T), 256, 0, ctx->stream>>>(peers.p[rank], (const float*)residual, (float*)out, world, T, h,
                                                                         epoch, (const uint32_t*)epoch_ptr);
    return runit_after_launch(ctx, "moe_ep_reduce");
}

// Expert-parallel decode block of one token without launches of its own for the exchange: routing, grouped gate/up, and a
// grouped down projection whose epilogue pushes this rank's weighted partial sum to every rank and raises the flags
// (EpPush); the residual add and the sum over the ranks happen in the prologue of the next GEMV that reads the hidden
// state (EpWait).  Three launches, as on one GPU.
int32_t moe_layer_q4k_ep_push_impl(runit_ctx* ctx, const void* router_w, const void* gate_local, const void* up_local,
                                   const void* down_local, float* xn, const float* pre_x, const float* pre_gamma, float pre_eps,
                                   void* scratch, size_t scratch_bytes, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm,
                                   uint32_t* counters, const EpPush* push) {
    RUNIT_REQUIRE(ctx, router_w && gate_local && up_local && down_local && xn && pre_x && pre_gamma && scratch && counters && push,
                  "moe_layer_q4k_ep_push: null pointer");
    RUNIT_REQUIRE(ctx, (h == 1024 || h == 2048 || h == 4096) && ff % 256 == 0 && E % push->world == 0 && k <= 32 && k <= E,
                  "moe_layer_q4k_ep_push: hidden 1024 / 2048 / 4096, experts divisible by the ranks");
    const MoeScratch s = moe_carve(scratch, 1, h, ff, E, k);
    if (s.bytes > scratch_bytes)
        return runit_fail(ctx, RUNIT_ERR_BUFFER_SIZE, "moe_layer_q4k_ep_push: scratch has %zu bytes, needs %zu", scratch_bytes, s.bytes);
    int32_t st;
    const dim3 grid((E + 7) / 8);
    st = moe_route_fused(ctx, (const float*)router_w, pre_x, s.logits, E, h, k, renorm, s.idx, s.w, counters, pre_gamma, pre_eps, xn);
    if ((st = runit_after_launch(ctx, "moe_route_fused")) != RUNIT_OK) return st;
    const uint32_t n_local = E / push->world;
    const int32_t lo = (int32_t)(push->rank * n_local);
    st = gemv_grouped(ctx, "moe_gate_up_ep", RUNIT_FMT_Q4K, gate_local, up_local, n_local, ff, h, xn, k, s.act, s.idx, k, lo, nullptr, nullptr,
                      nullptr, nullptr, 1);
    if (st != RUNIT_OK) return st;
    return gemv_grouped(ctx, "moe_down_ep_push", RUNIT_FMT_Q4K, down_local, nullptr, n_local, h, ff, s.act, 1, s.y, s.idx, k, lo, s.w, nullptr,
                        nullptr, counters + 32, 2, push);
}

}  // namespace runit

using namespace runit;

extern "C" {

size_t runit_moe_static_scratch_capacity(void) { return kMoeStaticScratchBytes; }

int32_t runit_moe_layer_q4k_static(runit_ctx_t* ctx, const void* router_w, const void* gate, const void* up,
                                   const void* down, const void* x, const void* residual, void* out, void* idx_out,
                                   void* w_out, uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, T > 0 && h > 0 && ff > 0 && E > 0 && k > 0, "moe_layer_q4k_static: empty shape");
    const size_t need = moe_carve(nullptr, T, h, ff, E, k).bytes;
    if (need > kMoeStaticScratchBytes)
        return runit_fail(ctx, RUNIT_ERR_BUFFER_SIZE,
                          "moe_layer_q4k_static: T=%u k=%u h=%u ff=%u E=%u needs %zu bytes of scratch, the built-in region "
                          "holds %zu; use runit_moe_layer_q4k with caller-owned scratch",
                          T, k, h, ff, E, need, (size_t)kMoeStaticScratchBytes);
    void* scratch = nullptr;
    int32_t st = moe_static_scratch(ctx, &scratch);
    if (st != RUNIT_OK) return st;
    return moe_layer_q4k_impl(ctx, router_w, gate, up, down, x, residual, out, (int32_t*)idx_out, (float*)w_out, scratch,
                              kMoeStaticScratchBytes, T, h, ff, E, k, renorm, nullptr, nullptr, 0.f, nullptr, nullptr, nullptr, 0.f);
}

size_t runit_moe_scratch_bytes(uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k) {
    return moe_carve(nullptr, T, h, ff, E, k).bytes;
}

int32_t runit_moe_router_f32(runit_ctx_t* ctx, const void* router_w, const void* x, void* logits, uint32_t E, uint32_t h,
                             uint32_t T) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, router_w && x && logits && E > 0 && T > 0 && h > 0 && h % 4 == 0, "moe_router_f32: bad argument");
    return moe_router(ctx, (const float*)router_w, (const float*)x, (float*)logits, E, h, T);
}

int32_t runit_moe_route_topk(runit_ctx_t* ctx, const void* logits, int32_t logits_f16, uint32_t E, uint32_t k, int32_t renorm,
                             uint32_t T, void* out_idx, void* out_w) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, logits && out_idx && out_w, "moe_route_topk: null pointer");
    RUNIT_REQUIRE(ctx, E > 0 && E <= 256 && k > 0 && k <= E && k <= 32 && T > 0, "moe_route_topk: E=%u k=%u T=%u unsupported", E, k, T);
    return moe_topk_rows(ctx, logits, logits_f16, E, E, k, RUNIT_SCORE_SOFTMAX, renorm, T, (int32_t*)out_idx, (float*)out_w);
}

int32_t runit_moe_route_scored(runit_ctx_t* ctx, const void* logits, uint32_t ld, uint32_t E, uint32_t k, int32_t score, int32_t renorm,
                               uint32_t T, void* out_idx, void* out_w) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, logits && out_idx && out_w && T > 0 && E > 0 && E <= 256 && k > 0 && k <= E && k <= 32 && ld >= E,
                  "moe_route_scored: bad argument");
    RUNIT_REQUIRE(ctx, score == RUNIT_SCORE_SOFTMAX || score == RUNIT_SCORE_SIGMOID, "moe_route_scored: unknown scoring function %d", score);
    return moe_topk_rows(ctx, logits, 0, ld, E, k, score, renorm, T, (int32_t*)out_idx, (float*)out_w);
}

int32_t runit_moe_experts_q4k(runit_ctx_t* ctx, const void* gate, const void* up, const void* down, const void* x_slots,
                              const void* slot_expert, void* y_slots, void* act_scratch, uint32_t n_slots, uint32_t h,
                              uint32_t ff, uint32_t n_experts) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, gate && up && down && x_slots && slot_expert && y_slots && act_scratch, "moe_experts_q4k: null pointer");
    RUNIT_REQUIRE(ctx, n_slots > 0 && n_experts > 0 && h % 256 == 0 && ff % 256 == 0 && h > 0 && ff > 0, "moe_experts_q4k: bad shape");
    int32_t st = gemv_grouped(ctx, "moe_gate_up", RUNIT_FMT_Q4K, gate, up, n_experts, ff, h, x_slots, 1, act_scratch,
                              (const int32_t*)slot_expert, n_slots);
    if (st != RUNIT_OK) return st;
    return gemv_grouped(ctx, "moe_down", RUNIT_FMT_Q4K, down, nullptr, n_experts, h, ff, act_scratch, 1, y_slots,
                        (const int32_t*)slot_expert, n_slots);
}

int32_t runit_moe_layer_q4k_ep(runit_ctx_t* ctx, const void* router_w, const void* gate_local, const void* up_local,
                               const void* down_local, const void* x, const void* residual, void* out, void* idx_out, void* w_out,
                               void* scratch, size_t scratch_bytes, void* const* partial_all, void* const* signal_pads,
                               uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm, uint32_t world,
                               uint32_t rank, uint32_t epoch) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, epoch > 0, "moe_layer_q4k_ep: epoch must be positive");
    return moe_layer_q4k_ep_impl(ctx, router_w, gate_local, up_local, down_local, x, residual, out, idx_out, w_out, scratch,
                                 scratch_bytes, partial_all, signal_pads, T, h, ff, E, k, renorm, world, rank, epoch, nullptr, nullptr, nullptr, nullptr, 0.f);
}

int32_t runit_moe_layer_q4k(runit_ctx_t* ctx, const void* router_w, const void* gate, const void* up, const void* down,
                            const void* x, const void* residual, void* out, void* idx_out, void* w_out, void* scratch,
                            size_t scratch_bytes, uint32_t T, uint32_t h, uint32_t ff, uint32_t E, uint32_t k, int32_t renorm) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    return moe_layer_q4k_impl(ctx, router_w, gate, up, down, x, residual, out, (int32_t*)idx_out, (float*)w_out, scratch,
                              scratch_bytes, T, h, ff, E, k, renorm, nullptr, nullptr, 0.f, nullptr, nullptr, nullptr, 0.f);
}

}  // extern "C"
