// Routing of the mixture-of-experts blocks: router products for one token and for many, scores, top-k, and the decode-size
// launches that do all of it at once.  Used by the Q4_K blocks (moe.cu, moe_grouped.cu, ep_prefill.cu) and by the layered
// decoders (layered_model.cu).
#include "gemv_common.cuh"
#include "moe_internal.h"
#include "runit_internal.h"
#include "tma.cuh"

namespace runit {

// logits[t][e] = W[e][:] . x[t][:]   (f32 router weights).  One warp per expert; the weight row
// stays in registers while the warp walks the tokens.
template <int KPL>   // floats of the row per lane (K = 32*KPL)
__global__ void __launch_bounds__(256) router_f32_kernel(const float* __restrict__ w, const float* __restrict__ x,
                                                          float* __restrict__ logits, uint32_t E, uint32_t K, uint32_t T) {
    grid_dependency_wait();      // inputs come from the previous kernel of the chain
    grid_launch_dependents();
    const uint32_t e = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (e >= E) return;
    float wr[KPL];
    const float4* wrow = reinterpret_cast<const float4*>(w + (size_t)e * K);
#pragma unroll
    for (int i = 0; i < KPL / 4; i++) {
        const float4 v = wrow[lane + 32 * i];
        wr[4 * i] = v.x; wr[4 * i + 1] = v.y; wr[4 * i + 2] = v.z; wr[4 * i + 3] = v.w;
    }
    for (uint32_t t = blockIdx.y; t < T; t += gridDim.y) {
        const float4* xr = reinterpret_cast<const float4*>(x + (size_t)t * K);
        float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
        for (int i = 0; i < KPL / 4; i++) {
            const float4 v = xr[lane + 32 * i];
            a0 = fmaf(wr[4 * i], v.x, a0); a1 = fmaf(wr[4 * i + 1], v.y, a1);
            a2 = fmaf(wr[4 * i + 2], v.z, a2); a3 = fmaf(wr[4 * i + 3], v.w, a3);
        }
        float acc = (a0 + a1) + (a2 + a3);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (lane == 0) logits[(size_t)t * E + e] = acc;
    }
}

// The same product for many tokens: a tiled f32 GEMM (CTA: TM tokens x 64 experts, thread: TM/16 x 4, K in chunks of 32
// through shared memory; TM = 32 or 16 when larger token tiles would leave SMs idle).  Every logit is one fused multiply-add chain
// over k in ascending order, whatever the tile.
template <int TM>
__global__ void __launch_bounds__(256) router_f32_tiled_kernel(const float* __restrict__ w, const float* __restrict__ x,
                                                                float* __restrict__ logits, uint32_t E, uint32_t K, uint32_t T) {
    grid_dependency_wait();      // inputs come from the previous kernel of the chain
    grid_launch_dependents();
    constexpr int RT = TM / 16;                  // token rows per thread
    __shared__ __align__(16) float xs[32][TM + 4];   // [k][token]
    __shared__ __align__(16) float ws[32][68];       // [k][expert]
    const uint32_t tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const uint32_t e0 = blockIdx.x * 64, t0 = blockIdx.y * TM;
    float acc[RT][4];
#pragma unroll
    for (int i = 0; i < RT; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    for (uint32_t kc = 0; kc < K; kc += 32) {
#pragma unroll
        for (int j = 0; j < 2; j++) {
            const uint32_t i = tid + 256 * j, row = i >> 3, kq = i & 7;
            float4 wv = make_float4(0.f, 0.f, 0.f, 0.f);
            if (e0 + row < E) wv = *reinterpret_cast<const float4*>(w + (size_t)(e0 + row) * K + kc + kq * 4);
            ws[kq * 4][row] = wv.x; ws[kq * 4 + 1][row] = wv.y; ws[kq * 4 + 2][row] = wv.z; ws[kq * 4 + 3][row] = wv.w;
            if (row < TM) {
                float4 xv = make_float4(0.f, 0.f, 0.f, 0.f);
                if (t0 + row < T) xv = *reinterpret_cast<const float4*>(x + (size_t)(t0 + row) * K + kc + kq * 4);
                xs[kq * 4][row] = xv.x; xs[kq * 4 + 1][row] = xv.y; xs[kq * 4 + 2][row] = xv.z; xs[kq * 4 + 3][row] = xv.w;
            }
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < 32; kk++) {
            float av[RT];
            if constexpr (RT == 4) {
                const float4 a = *reinterpret_cast<const float4*>(&xs[kk][ty * 4]);
                av[0] = a.x; av[1] = a.y; av[2] = a.z; av[3] = a.w;
            } else if constexpr (RT == 2) {
                const float2 a = *reinterpret_cast<const float2*>(&xs[kk][ty * 2]);
                av[0] = a.x; av[1] = a.y;
            } else {
                av[0] = xs[kk][ty];
            }
            const float4 b = *reinterpret_cast<const float4*>(&ws[kk][tx * 4]);
            const float bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < RT; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(bv[j], av[i], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < RT; i++) {
        const uint32_t t = t0 + ty * RT + i;
        if (t >= T) continue;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const uint32_t e = e0 + tx * 4 + j;
            if (e < E) logits[(size_t)t * E + e] = acc[i][j];
        }
    }
}

// Many tokens, few experts: the same product with K split over the eight warps of a CTA.  CTA = 16 tokens x 64 experts;
// warp w multiplies the whole tile over its eighth of K (chunks of 32 staged by cp.async in its own two shared-memory
// buffers, rows as in memory), a lane keeps 4 tokens x 8 experts (tokens ty + 4 i, experts tx + 8 j: consecutive rows per load, no bank
// conflicts) and reads 12 x 128 bits per 128 multiply-adds; the eight partial tiles are added in warp order.  Every logit is
// eight fused multiply-add chains over ascending k, added in order: the same bits whatever T is.  K must be a multiple of 256.
constexpr int kRsPitch = 36;                                    // floats per staged row (32 + 4)
constexpr int kRsWarpFloats = (16 + 64) * kRsPitch;             // one warp's slice
__global__ void __launch_bounds__(256) router_f32_splitk_kernel(const float* __restrict__ w, const float* __restrict__ x,
                                                                 float* __restrict__ logits, uint32_t E, uint32_t K, uint32_t T) {
    grid_dependency_wait();      // inputs come from the previous kernel of the chain
    grid_launch_dependents();
    extern __shared__ __align__(16) float rs_smem[];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, ty = lane >> 3, tx = lane & 7;
    const uint32_t e0 = blockIdx.x * 64, t0 = blockIdx.y * 16;
    float* xs = rs_smem + warp * (2 * kRsWarpFloats);            // two buffers of [16][36] + [64][36]
    float* ws = xs + 16 * kRsPitch;
    float acc[4][8];
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 8; j++) acc[i][j] = 0.f;
    const uint32_t kw = K / 8, k_begin = warp * kw, n_chunks = kw / 32;
    const uint32_t lrow = lane >> 3, lkq = lane & 7;             // a copy instruction covers 4 rows x 32 k
    // two buffers per warp: chunk c + 1 is copied (cp.async, 16 bytes per lane and row group) while chunk c is multiplied;
    // rows past T or E are copied from row 0 of the same matrix (never stored)
    auto stage = [&](uint32_t c) {
        if (c < n_chunks) {
            const uint32_t kc = k_begin + 32 * c;
            const uint32_t xb = smem_u32(xs + (c & 1) * kRsWarpFloats), wb = smem_u32(ws + (c & 1) * kRsWarpFloats);
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const uint32_t row = lrow + 4 * j, tr = t0 + row < T ? t0 + row : 0u;
                cp_async16(xb + (row * kRsPitch + 4 * lkq) * 4, x + (size_t)tr * K + kc + 4 * lkq);
            }
#pragma unroll
            for (int j = 0; j < 16; j++) {
                const uint32_t row = lrow + 4 * j, er = e0 + row < E ? e0 + row : 0u;
                cp_async16(wb + (row * kRsPitch + 4 * lkq) * 4, w + (size_t)er * K + kc + 4 * lkq);
            }
        }
        cp_async_commit();
    };
    stage(0);
    for (uint32_t c = 0; c < n_chunks; c++) {
        stage(c + 1);
        cp_async_wait<1>();
        __syncwarp();
        const float* xs_c = xs + (c & 1) * kRsWarpFloats;
        const float* ws_c = ws + (c & 1) * kRsWarpFloats;
#pragma unroll
        for (int k4 = 0; k4 < 8; k4++) {
            float4 xa[4], wb[8];
#pragma unroll
            for (int i = 0; i < 4; i++) xa[i] = *reinterpret_cast<const float4*>(xs_c + (ty + 4 * i) * kRsPitch + 4 * k4);
#pragma unroll
            for (int j = 0; j < 8; j++) wb[j] = *reinterpret_cast<const float4*>(ws_c + (tx + 8 * j) * kRsPitch + 4 * k4);
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 8; j++) {
                    float a = acc[i][j];
                    a = fmaf(wb[j].x, xa[i].x, a);
                    a = fmaf(wb[j].y, xa[i].y, a);
                    a = fmaf(wb[j].z, xa[i].z, a);
                    a = fmaf(wb[j].w, xa[i].w, a);
                    acc[i][j] = a;
                }
        }
        __syncwarp();
    }
    // the eight partial tiles meet in shared memory ([warp][token][expert]) and are added in warp order
    __syncthreads();
    float* red = rs_smem;
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 8; j++) red[(warp * 16 + ty + 4 * i) * 64 + tx + 8 * j] = acc[i][j];
    __syncthreads();
#pragma unroll
    for (int q = 0; q < 4; q++) {
        const uint32_t o = tid + 256 * q, tok = o >> 6, e = o & 63;
        float v = red[tok * 64 + e];
#pragma unroll
        for (int p = 1; p < 8; p++) v += red[(p * 16 + tok) * 64 + e];
        if (t0 + tok < T && e0 + e < E) logits[(size_t)(t0 + tok) * E + e0 + e] = v;
    }
}

// Generic fallback for any K (multiple of 4).
__global__ void __launch_bounds__(256) router_f32_generic_kernel(const float* __restrict__ w, const float* __restrict__ x,
                                                                  float* __restrict__ logits, uint32_t E, uint32_t K, uint32_t T) {
    grid_dependency_wait();      // inputs come from the previous kernel of the chain
    grid_launch_dependents();
    const uint32_t e = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (e >= E) return;
    for (uint32_t t = blockIdx.y; t < T; t += gridDim.y) {
        float acc = 0.f;
        for (uint32_t c = lane; c < K; c += 32) acc = fmaf(w[(size_t)e * K + c], x[(size_t)t * K + c], acc);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (lane == 0) logits[(size_t)t * E + e] = acc;
    }
}

// Scores of all experts (softmax over them, or the sigmoid of each logit), then the top-k in descending order (ties: lowest
// index), optionally renormalised to sum 1 (softmax: crates/engine/src/forward.rs:2420-2448).  One warp per token,
// E <= 256.  in_f16 != 0: the logits are f16 (the reference's router output dtype).
// Routing of one token by one warp; `logits` points at the token's E logits (global or shared memory),
// out_idx / out_w at its k outputs.
template <int NG>   // groups of 32 experts that can be non-empty (E <= 32 * NG); skipping the empty ones adds exact zeros less
__device__ __forceinline__ void route_topk_groups(const void* logits, int in_f16, uint32_t E, uint32_t k, int score, int renorm, uint32_t lane,
                                                int32_t* out_idx, float* out_w) {
    float v[NG];
    float mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < NG; i++) {
        const uint32_t e = lane + 32 * i;
        float lv = -INFINITY;
        if (e < E) lv = in_f16 ? __half2float(reinterpret_cast<const __half*>(logits)[e])
                               : reinterpret_cast<const float*>(logits)[e];
        v[i] = lv;
        mx = fmaxf(mx, lv);
    }
    if (score == RUNIT_SCORE_SOFTMAX) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        // exp values; the sum runs over experts in index order so that it is reproducible
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < NG; i++) v[i] = (lane + 32 * i < E) ? expf(v[i] - mx) : 0.f;
#pragma unroll
        for (int i = 0; i < NG; i++) {
            float part = v[i];   // 0 beyond E; a fixed shuffle tree per group of 32 experts: deterministic
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) part += __shfl_xor_sync(0xffffffffu, part, o);
            sum += part;
        }
#pragma unroll
        for (int i = 0; i < NG; i++) v[i] = v[i] / sum;   // probabilities (0 beyond E)
    }
    // (sigmoid keeps the order of the logits: the largest logits are taken and their scores formed below, so that scores
    // which round to the same value do not decide)
    uint32_t taken = 0;
    float wsum = 0.f;
    float my_w = 0.f;   // lane s keeps the s-th selected weight (k <= 32)
    int my_i = 0;
    for (uint32_t s = 0; s < k; s++) {
        float bv = -INFINITY;
        uint32_t bi = 0xFFFFFFFFu;
#pragma unroll
        for (int i = 0; i < NG; i++) {
            const uint32_t e = lane + 32 * i;
            if (e < E && !((taken >> i) & 1u) && (v[i] > bv)) { bv = v[i]; bi = e; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const uint32_t oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
        }
        if ((bi & 31u) == lane && bi != 0xFFFFFFFFu) taken |= 1u << (bi >> 5);
        if (score == RUNIT_SCORE_SIGMOID) bv = 1.0f / (1.0f + expf(-bv));
        if (lane == s) { my_w = bv; my_i = (int)bi; }
        wsum += bv;
    }
    if (lane < k) {
        float wv = my_w;
        if (renorm && wsum > 0.f) wv = wv / wsum;
        out_idx[lane] = my_i;
        out_w[lane] = wv;
    }
}

__device__ __forceinline__ void route_topk_warp(const void* logits, int in_f16, uint32_t E, uint32_t k, int score, int renorm, uint32_t lane,
                                                int32_t* out_idx, float* out_w) {
    if (E <= 32) route_topk_groups<1>(logits, in_f16, E, k, score, renorm, lane, out_idx, out_w);
    else if (E <= 64) route_topk_groups<2>(logits, in_f16, E, k, score, renorm, lane, out_idx, out_w);
    else if (E <= 128) route_topk_groups<4>(logits, in_f16, E, k, score, renorm, lane, out_idx, out_w);
    else route_topk_groups<8>(logits, in_f16, E, k, score, renorm, lane, out_idx, out_w);
}

// Rows of ld logits; a row's first E are the experts'.
__global__ void __launch_bounds__(128) route_topk_kernel(const void* __restrict__ logits, int in_f16, uint32_t ld, uint32_t E, uint32_t k,
                                                          int score, int renorm, uint32_t T, int32_t* __restrict__ out_idx,
                                                          float* __restrict__ out_w) {
    grid_dependency_wait();      // inputs come from the previous kernel of the chain
    grid_launch_dependents();
    const uint32_t t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= T) return;
    const void* row = in_f16 ? (const void*)(reinterpret_cast<const __half*>(logits) + (size_t)t * ld)
                             : (const void*)(reinterpret_cast<const float*>(logits) + (size_t)t * ld);
    route_topk_warp(row, in_f16, E, k, score, renorm, lane, out_idx + (size_t)t * k, out_w + (size_t)t * k);
}

// Router and routing of ONE token in one launch (decode): CTAs of 8 warps compute 8 logits each with exactly the
// arithmetic of router_f32_kernel (same bits), publish them and take a ticket; the CTA that draws the last ticket
// routes from the complete logits and puts the ticket counter back to zero.  *counter must be zero before the
// first launch.
// gamma != nullptr: x is the un-normalised hidden state; every CTA first computes its RMSNorm (thread order, shuffle tree
// and rounding of rms_norm_kernel: the same bits in every CTA and as the separate launch), CTA 0 stores the normalised
// vector to xn_out for the expert GEMVs, and the router reads it from shared memory.
template <int KPL>
__global__ void __launch_bounds__(256) route_fused_kernel(const float* __restrict__ w, const float* __restrict__ x,
                                                           float* logits, uint32_t E, uint32_t K, uint32_t k, int renorm,
                                                           int32_t* __restrict__ out_idx, float* __restrict__ out_w, uint32_t* counter,
                                                           const float* __restrict__ gamma, float eps, float* __restrict__ xn_out) {
    __shared__ uint32_t s_last;
    __shared__ __align__(16) float xs[KPL * 32];
    __shared__ float part[8];
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t e = blockIdx.x * 8 + warp;
    // the router row and gamma do not depend on the previous kernel of the chain: they are requested before the wait
    float4 wv[KPL / 4];
    float gv[KPL / 8];
    if (e < E) {
        const float4* wrow = reinterpret_cast<const float4*>(w + (size_t)e * K);
#pragma unroll
        for (int i = 0; i < KPL / 4; i++) wv[i] = wrow[lane + 32 * i];
    }
    if (gamma) {
#pragma unroll
        for (int j = 0; j < KPL / 8; j++) gv[j] = gamma[threadIdx.x + 256 * j];
    }
    grid_dependency_wait();
    grid_launch_dependents();
    if (gamma) {
        float xv[KPL / 8];
#pragma unroll
        for (int j = 0; j < KPL / 8; j++) xv[j] = x[threadIdx.x + 256 * j];
        float sq = 0.f;
#pragma unroll
        for (int j = 0; j < KPL / 8; j++) sq = fmaf(xv[j], xv[j], sq);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
        if (lane == 0) part[warp] = sq;
        __syncthreads();
        float tot = 0.f;
#pragma unroll
        for (int i = 0; i < 8; i++) tot += part[i];
        const float r = rsqrtf(tot / (float)K + eps);
#pragma unroll
        for (int j = 0; j < KPL / 8; j++) {
            const float v = xv[j] * r * gv[j];
            xs[threadIdx.x + 256 * j] = v;
            if (blockIdx.x == 0) xn_out[threadIdx.x + 256 * j] = v;
        }
        __syncthreads();
    }
    if (e < E) {
        const float4* xr = gamma ? reinterpret_cast<const float4*>(xs) : reinterpret_cast<const float4*>(x);
        float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
        for (int i = 0; i < KPL / 4; i++) {
            const float4 v = xr[lane + 32 * i];
            a0 = fmaf(wv[i].x, v.x, a0); a1 = fmaf(wv[i].y, v.y, a1);
            a2 = fmaf(wv[i].z, v.z, a2); a3 = fmaf(wv[i].w, v.w, a3);
        }
        float acc = (a0 + a1) + (a2 + a3);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (lane == 0) logits[e] = acc;
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        __threadfence();                                   // this CTA's logits are visible before its ticket
        s_last = atomicAdd(counter, 1u) == gridDim.x - 1;
    }
    __syncthreads();
    if (s_last && warp == 0) {
        __threadfence();
        route_topk_warp(logits, 0, E, k, RUNIT_SCORE_SOFTMAX, renorm, lane, out_idx, out_w);
        if (lane == 0) *counter = 0;
    }
}

// The same for any width and for routers with more to say than a softmax: w has R >= E rows, the first E are the experts' and
// the others belong to gates whose sigmoid is wanted (a shared expert's, for instance).  The norm has one gain for all
// coordinates (*gain).  xn (shared memory) is filled by every CTA; CTA 0 stores it for the expert GEMVs.
__global__ void __launch_bounds__(256) route_gated_kernel(const float* __restrict__ w, const float* __restrict__ x, float* logits, uint32_t R,
                                                           uint32_t E, uint32_t K, uint32_t k, int score, int renorm,
                                                           int32_t* __restrict__ out_idx, float* __restrict__ out_w,
                                                           float* __restrict__ out_gate, uint32_t* counter, const float* __restrict__ gain,
                                                           float eps, float* __restrict__ xn_out) {
    extern __shared__ __align__(16) float xs[];
    __shared__ float part[8];
    __shared__ uint32_t s_last;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = blockIdx.x * 8 + warp;
    const float g = *gain;
    const float* wrow = w + (size_t)r * K;
    const bool vec = (K & 3u) == 0;
    const float4* w4 = reinterpret_cast<const float4*>(wrow);
    // the first part of the row does not depend on the previous kernel of the chain: requested before the wait
    constexpr int P = 16;
    float4 wv[P];
#pragma unroll
    for (int i = 0; i < P; i++) {
        const uint32_t c = lane + 32 * i;
        wv[i] = (vec && r < R && c < K / 4) ? __ldg(w4 + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    grid_dependency_wait();
    grid_launch_dependents();
    float sq = 0.f;
    for (uint32_t i = threadIdx.x; i < K; i += 256) {
        const float v = x[i];
        xs[i] = v;
        sq = fmaf(v, v, sq);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    if (lane == 0) part[warp] = sq;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) tot += part[i];
    const float sc = rsqrtf(tot / (float)K + eps) * g;
    if (blockIdx.x == 0)
        for (uint32_t i = threadIdx.x; i < K; i += 256) xn_out[i] = xs[i] * sc;
    if (r < R) {
        float acc = 0.f;
        if (vec) {
            const float4* x4 = reinterpret_cast<const float4*>(xs);
            auto step = [&](const float4& a, const float4& v) {
                acc = fmaf(a.x, v.x, acc); acc = fmaf(a.y, v.y, acc); acc = fmaf(a.z, v.z, acc); acc = fmaf(a.w, v.w, acc);
            };
#pragma unroll
            for (int i = 0; i < P; i++)
                if (lane + 32 * i < K / 4) step(wv[i], x4[lane + 32 * i]);
#pragma unroll 8
            for (uint32_t c = lane + 32 * P; c < K / 4; c += 32) step(__ldg(w4 + c), x4[c]);
        } else {
            for (uint32_t c = lane; c < K; c += 32) acc = fmaf(wrow[c], xs[c], acc);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (lane == 0) {
            acc *= sc;
            logits[r] = acc;
            if (r >= E) out_gate[r - E] = 1.0f / (1.0f + expf(-acc));
        }
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        __threadfence();
        s_last = atomicAdd(counter, 1u) == gridDim.x - 1;
    }
    __syncthreads();
    if (s_last && warp == 0) {
        __threadfence();
        route_topk_warp(logits, 0, E, k, score, renorm, lane, out_idx, out_w);
        if (lane == 0) *counter = 0;
    }
}

int32_t moe_router(runit_ctx* ctx, const float* w, const float* x, float* logits, uint32_t E, uint32_t K, uint32_t T) {
    // (the tiled kernel, one CTA per 64 tokens walking all of K, has a floor of about 85 us: it serves K that is not a
    // multiple of 256 at large sizes and stays selectable, router_variant = 2)
    // measured (h = 2048, warm, us): one warp per expert / tiled / split over the warps of a CTA: 64 experts x 256 tokens
    // 10 / 87 / 22, x 1024: 32 / 87 / 22, x 2048: 60 / 87 / 22, x 4096: 117 / 122 / 42; 128 experts x 256: 19 / 86 / 22,
    // x 1024: 62 / 87 / 23, x 4096: 230 / 134 / 82 (the split kernel re-reads the router for every 16 tokens: about 4 TB/s from L2)
    if ((((uint64_t)T * E >= 49152ull && ctx->tune.router_variant == 0) || ctx->tune.router_variant == 3) && K % 256 == 0 && runit_aligned(w, 16) &&
        runit_aligned(x, 16)) {
        constexpr int smem = 8 * 2 * kRsWarpFloats * 4;
        static bool configured[64] = {false};
        if (ctx->device >= 0 && ctx->device < 64 && !configured[ctx->device]) {
            RUNIT_CUDA_TRY(ctx, cudaFuncSetAttribute(router_f32_splitk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
            configured[ctx->device] = true;
        }
        runit_launch_chain_smem(ctx, router_f32_splitk_kernel, dim3((E + 63) / 64, (T + 15) / 16), dim3(256), smem, w, x, logits, E, K, T);
        return runit_after_launch(ctx, "moe_router_f32_splitk");
    }
    const bool big = (uint64_t)T * E >= 400000ull;
    if (ctx->tune.router_variant != 1 && (big || ctx->tune.router_variant == 2) && K % 32 == 0 && runit_aligned(w, 16) && runit_aligned(x, 16)) {
        const uint32_t ge = (E + 63) / 64;
        if (ge * ((T + 63) / 64) >= (uint32_t)ctx->sm_count)
            runit_launch_chain(ctx, router_f32_tiled_kernel<64>, dim3(ge, (T + 63) / 64), dim3(256), w, x, logits, E, K, T);
        else if (ge * ((T + 31) / 32) >= (uint32_t)ctx->sm_count)
            runit_launch_chain(ctx, router_f32_tiled_kernel<32>, dim3(ge, (T + 31) / 32), dim3(256), w, x, logits, E, K, T);
        else
            runit_launch_chain(ctx, router_f32_tiled_kernel<16>, dim3(ge, (T + 15) / 16), dim3(256), w, x, logits, E, K, T);
        return runit_after_launch(ctx, "moe_router_f32_tiled");
    }
    dim3 grid((E + 7) / 8, T < 64 ? T : 64);
    if (K == 2048) runit_launch_chain(ctx, router_f32_kernel<64>, dim3(grid), dim3(256), w, x, logits, E, K, T);
    else if (K == 1024) runit_launch_chain(ctx, router_f32_kernel<32>, dim3(grid), dim3(256), w, x, logits, E, K, T);
    else if (K == 4096) runit_launch_chain(ctx, router_f32_kernel<128>, dim3(grid), dim3(256), w, x, logits, E, K, T);
    else runit_launch_chain(ctx, router_f32_generic_kernel, dim3(grid), dim3(256), w, x, logits, E, K, T);
    return runit_after_launch(ctx, "moe_router_f32");
}

int32_t moe_topk_rows(runit_ctx* ctx, const void* logits, int32_t logits_f16, uint32_t ld, uint32_t E, uint32_t k, int32_t score,
                      int32_t renorm, uint32_t T, int32_t* idx, float* w) {
    runit_launch_chain(ctx, route_topk_kernel, dim3((T + 3) / 4), dim3(128), logits, logits_f16, ld, E, k, score, renorm, T, idx, w);
    return runit_after_launch(ctx, "moe_route_topk");
}
int32_t moe_topk(runit_ctx* ctx, const float* logits, uint32_t E, uint32_t k, int32_t renorm, uint32_t T, int32_t* idx, float* w) {
    return moe_topk_rows(ctx, logits, 0, E, E, k, RUNIT_SCORE_SOFTMAX, renorm, T, idx, w);
}

int32_t moe_route_fused(runit_ctx* ctx, const float* w, const float* x, float* logits, uint32_t E, uint32_t h, uint32_t k, int32_t renorm,
                        int32_t* idx, float* wts, uint32_t* counter, const float* gamma, float eps, float* xn_out) {
    const dim3 grid((E + 7) / 8);
    if (h == 2048) runit_launch_chain(ctx, route_fused_kernel<64>, grid, dim3(256), w, x, logits, E, h, k, (int)renorm, idx, wts, counter, gamma, eps, xn_out);
    else if (h == 1024) runit_launch_chain(ctx, route_fused_kernel<32>, grid, dim3(256), w, x, logits, E, h, k, (int)renorm, idx, wts, counter, gamma, eps, xn_out);
    else runit_launch_chain(ctx, route_fused_kernel<128>, grid, dim3(256), w, x, logits, E, h, k, (int)renorm, idx, wts, counter, gamma, eps, xn_out);
    return runit_after_launch(ctx, "moe_route_fused");
}

int32_t moe_route_gated(runit_ctx* ctx, const float* w, const float* x, float* logits, uint32_t R, uint32_t E, uint32_t K, uint32_t k,
                        int32_t score, int32_t renorm, int32_t* idx, float* wts, float* gates, uint32_t* counter, const float* gain,
                        float eps, float* xn_out) {
    if ((size_t)K * 4 > 40 * 1024)
        RUNIT_CUDA_TRY(ctx, cudaFuncSetAttribute(route_gated_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(K * 4)));
    runit_launch_chain_smem(ctx, route_gated_kernel, dim3((R + 7) / 8), dim3(256), (size_t)K * 4, w, x, logits, R, E, K, k, (int)score,
                            (int)renorm, idx, wts, gates, counter, gain, eps, xn_out);
    return runit_after_launch(ctx, "moe_route_gated");
}

}  // namespace runit
