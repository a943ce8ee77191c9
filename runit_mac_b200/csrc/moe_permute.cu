// Token permutation of the batched mixture-of-experts blocks: slots (token, expert) sorted by expert and cut into token
// tiles, rows gathered into that order, and the sum of the experts' outputs per token.  Shared by the Q4_K block
// (moe_grouped.cu) and the bf16 grouped GEMM (gemm_bf16.cu).
#include "moe_internal.h"
#include "runit_internal.h"

namespace runit {

// counts[e] = slots routed to expert e; slots with an id outside [0, E) get position -1.
__global__ void __launch_bounds__(256) count_kernel(const int32_t* __restrict__ idx, uint32_t S, uint32_t E,
                                                     int32_t* __restrict__ counts, int32_t* __restrict__ pos_of_slot) {
    __shared__ int hist[256];
    hist[threadIdx.x] = 0;
    __syncthreads();
    for (uint32_t s = blockIdx.x * 4096 + threadIdx.x, i = 0; i < 16 && s < S; i++, s += 256) {
        const int32_t e = idx[s];
        if (e >= 0 && (uint32_t)e < E) atomicAdd(&hist[e], 1);
        else pos_of_slot[s] = -1;
    }
    __syncthreads();
    if (threadIdx.x < E && hist[threadIdx.x]) atomicAdd(&counts[threadIdx.x], hist[threadIdx.x]);
}

// One CTA per expert: first row of the expert in the permuted order (experts in index order, each padded to a
// multiple of 128 rows), the token-tile table (tiles of `tile_tok` slots, 128 or 256, never across experts), and the
// position of each of its slots (slot order kept).
__global__ void __launch_bounds__(1024) place_kernel(const int32_t* __restrict__ idx, uint32_t S, uint32_t E,
                                                      const int32_t* __restrict__ counts, int tile_tok,
                                                      int32_t* __restrict__ pos_of_slot, int32_t* __restrict__ tile_expert,
                                                      int32_t* __restrict__ tile_nvalid, int32_t* __restrict__ tile_row0,
                                                      int32_t* __restrict__ n_tok_tiles) {
    __shared__ int s_cnt[256];
    __shared__ int s_warp[32];
    __shared__ int s_off, s_tile0, s_chunk;
    const uint32_t e = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid < 256) s_cnt[tid] = tid < E ? counts[tid] : 0;
    __syncthreads();
    if (tid == 0) {
        int off = 0, tiles = 0;
        for (uint32_t i = 0; i < E; i++) {
            if (i == e) { s_off = off; s_tile0 = tiles; }
            off += ((s_cnt[i] + kMoeRowAlign - 1) / kMoeRowAlign) * kMoeRowAlign;
            tiles += (s_cnt[i] + tile_tok - 1) / tile_tok;
        }
        if (e == 0) n_tok_tiles[0] = tiles;
    }
    __syncthreads();
    const int cnt = s_cnt[e], off = s_off, tile0 = s_tile0;
    for (int i = tid; i * tile_tok < cnt; i += 1024) {
        tile_expert[tile0 + i] = (int32_t)e;
        tile_nvalid[tile0 + i] = min(tile_tok, cnt - i * tile_tok);
        tile_row0[tile0 + i] = off + i * tile_tok;
    }
    // every thread takes 4 consecutive slots per round, so a round covers 4096 slots in slot order
    int running = 0;
    for (uint32_t s0 = 0; s0 < S; s0 += 4096) {
        const uint32_t s = s0 + 4 * tid;
        bool hit[4];
        int mine = 0;
#pragma unroll
        for (int i = 0; i < 4; i++) {
            hit[i] = s + i < S && idx[s + i] == (int32_t)e;
            mine += hit[i];
        }
        int incl = mine;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int t = __shfl_up_sync(0xffffffffu, incl, o);
            if ((int)lane >= o) incl += t;
        }
        if (lane == 31) s_warp[warp] = incl;
        __syncthreads();
        if (warp == 0) {
            int v = s_warp[lane], wi = v;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int t = __shfl_up_sync(0xffffffffu, wi, o);
                if ((int)lane >= o) wi += t;
            }
            s_warp[lane] = wi - v;   // exclusive prefix over the warps
            if (lane == 31) s_chunk = wi;
        }
        __syncthreads();
        int p = off + running + s_warp[warp] + incl - mine;
#pragma unroll
        for (int i = 0; i < 4; i++)
            if (hit[i]) pos_of_slot[s + i] = p++;
        running += s_chunk;
        __syncthreads();
    }
}

// Token rows into the permuted order: dst[pos(s)][:] = src[s / k][:], rows of row16 16-byte pieces; one warp per slot, 8 slots
// per CTA.
__global__ void __launch_bounds__(256) gather_rows_kernel(const uint4* __restrict__ x, const int32_t* __restrict__ pos_of_slot,
                                                           uint4* __restrict__ xperm, uint32_t S, uint32_t row16, uint32_t k) {
    const uint32_t s = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (s >= S) return;
    const int32_t pos = pos_of_slot[s];
    if (pos < 0) return;
    const uint4* src = x + (size_t)(s / k) * row16;
    uint4* dst = xperm + (size_t)pos * row16;
    for (uint32_t c = lane; c < row16; c += 32) dst[c] = src[c];
}

// One value per slot into the permuted order.
__global__ void __launch_bounds__(256) gather_values_kernel(const float* __restrict__ v, const int32_t* __restrict__ pos_of_slot,
                                                             float* __restrict__ out, uint32_t S) {
    const uint32_t s = blockIdx.x * 256 + threadIdx.x;
    if (s < S && pos_of_slot[s] >= 0) out[pos_of_slot[s]] = v[s];
}

// out[t] = (residual ? residual[t] : 0) + sum_i w[t][i] * y[pos(t, i)]   (routing order; product and sum rounded
// separately, like the reference's scale-accumulate followed by the residual add).
__global__ void __launch_bounds__(256) combine_kernel(const float* __restrict__ y, const int32_t* __restrict__ pos_of_slot,
                                                       const float* __restrict__ w, const float* residual,
                                                       float* out, uint32_t h, uint32_t k) {
    const uint32_t t = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
    if (c >= h / 4) return;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (uint32_t i = 0; i < k; i++) {
        const int32_t pos = pos_of_slot[t * k + i];
        if (pos < 0) continue;
        const float wi = w ? w[t * k + i] : 1.0f;
        const float4 v = __ldg(reinterpret_cast<const float4*>(y + (size_t)pos * h) + c);
        acc.x = __fadd_rn(acc.x, __fmul_rn(wi, v.x)); acc.y = __fadd_rn(acc.y, __fmul_rn(wi, v.y));
        acc.z = __fadd_rn(acc.z, __fmul_rn(wi, v.z)); acc.w = __fadd_rn(acc.w, __fmul_rn(wi, v.w));
    }
    float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
    if (residual) b = reinterpret_cast<const float4*>(residual + (size_t)t * h)[c];
    reinterpret_cast<float4*>(out + (size_t)t * h)[c] = make_float4(b.x + acc.x, b.y + acc.y, b.z + acc.z, b.w + acc.w);
}

// Any width (rows that are not a multiple of four floats).
__global__ void __launch_bounds__(256) combine_any_kernel(const float* __restrict__ y, const int32_t* __restrict__ pos_of_slot,
                                                           const float* __restrict__ w, const float* residual, float* out, uint32_t h,
                                                           uint32_t k) {
    const uint32_t t = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
    if (c >= h) return;
    float acc = 0.f;
    for (uint32_t i = 0; i < k; i++) {
        const int32_t pos = pos_of_slot[t * k + i];
        if (pos >= 0) acc = __fadd_rn(acc, __fmul_rn(w ? w[t * k + i] : 1.0f, y[(size_t)pos * h + c]));
    }
    out[(size_t)t * h + c] = (residual ? residual[(size_t)t * h + c] : 0.f) + acc;
}

// One "expert" that owns everything, tokens in their own order.
__global__ void dense_tiles_kernel(uint32_t T, uint32_t tile_tok, int32_t* tile_expert, int32_t* tile_nvalid, int32_t* tile_row0, int32_t* n_tok_tiles) {
    const uint32_t n = (T + tile_tok - 1) / tile_tok;
    for (uint32_t i = threadIdx.x; i < n; i += blockDim.x) {
        tile_expert[i] = 0;
        tile_nvalid[i] = (int32_t)min(tile_tok, T - i * tile_tok);
        tile_row0[i] = (int32_t)(i * tile_tok);
    }
    if (threadIdx.x == 0) n_tok_tiles[0] = (int32_t)n;
}

int32_t moe_permute(runit_ctx* ctx, const int32_t* idx, uint32_t S, uint32_t E, uint32_t tile_tok, const MoePermutation& p) {
    RUNIT_CUDA_TRY(ctx, cudaMemsetAsync(p.counts, 0, 4 * 256, ctx->stream));
    count_kernel<<<(S + 4095) / 4096, 256, 0, ctx->stream>>>(idx, S, E, p.counts, p.pos_of_slot);
    int32_t st = runit_after_launch(ctx, "moe_grouped_count");
    if (st != RUNIT_OK) return st;
    place_kernel<<<E, 1024, 0, ctx->stream>>>(idx, S, E, p.counts, (int)tile_tok, p.pos_of_slot, p.tile_expert, p.tile_nvalid, p.tile_row0,
                                              p.n_tok_tiles);
    return runit_after_launch(ctx, "moe_grouped_place");
}

int32_t moe_dense_tiles(runit_ctx* ctx, uint32_t T, uint32_t tile_tok, int32_t* tile_expert, int32_t* tile_nvalid, int32_t* tile_row0,
                        int32_t* n_tok_tiles) {
    dense_tiles_kernel<<<1, 256, 0, ctx->stream>>>(T, tile_tok, tile_expert, tile_nvalid, tile_row0, n_tok_tiles);
    return runit_after_launch(ctx, "dense_tiles");
}

int32_t moe_gather_rows(runit_ctx* ctx, const void* x, const int32_t* pos_of_slot, void* xperm, uint32_t S, size_t row_bytes, uint32_t k) {
    gather_rows_kernel<<<(S + 7) / 8, 256, 0, ctx->stream>>>((const uint4*)x, pos_of_slot, (uint4*)xperm, S, (uint32_t)(row_bytes / 16), k);
    return runit_after_launch(ctx, "moe_grouped_gather");
}

int32_t moe_gather_values(runit_ctx* ctx, const float* v, const int32_t* pos_of_slot, float* out, uint32_t S) {
    gather_values_kernel<<<(S + 255) / 256, 256, 0, ctx->stream>>>(v, pos_of_slot, out, S);
    return runit_after_launch(ctx, "moe_gather_values");
}

int32_t moe_grouped_combine(runit_ctx* ctx, const float* y, const int32_t* pos_of_slot, const float* w, const float* residual, float* out,
                            uint32_t T, uint32_t h, uint32_t k) {
    if (h % 4 == 0) combine_kernel<<<dim3((h / 4 + 255) / 256, T), 256, 0, ctx->stream>>>(y, pos_of_slot, w, residual, out, h, k);
    else combine_any_kernel<<<dim3((h + 255) / 256, T), 256, 0, ctx->stream>>>(y, pos_of_slot, w, residual, out, h, k);
    return runit_after_launch(ctx, "moe_grouped_combine");
}

}  // namespace runit
