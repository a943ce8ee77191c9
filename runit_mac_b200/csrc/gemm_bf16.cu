// GEMM of many tokens with a bf16 weight matrix, dense or grouped by expert, with the consumer's arithmetic in the epilogue.
//
// Two kernels behind one descriptor (GemmDesc in bf16_ops.cuh):
//   * gemm_tc_kernel: bf16 activations, tcgen05.mma into f32 accumulators.  Weight rows ride the M of the MMA (128 per tile),
//     token rows ride N (tiles of 64, 128 or 256).  Persistent CTAs; warp 0 loads both operand tiles by TMA (64 K elements per
//     stage, 128-byte swizzle), one lane of warp 1 issues the MMAs, warps 2-5 drain one of two accumulators while the other
//     is filled.  A lane of the epilogue holds one output row, so the stores of a token are contiguous over a warp.
//   * gemm_f32_kernel: f32 activations and f32 multiply-adds (the weights are bf16 values, exact in f32), for passes that
//     run in 32-bit throughout.
// A tile never mixes experts: token tiles come from a table (moe_permute), or are cut from the token index when dense.
// Every wait is bounded; a wait that gives up raises the CTA's abort flag, all roles leave their loops, the loads in flight
// are waited for, tensor memory is freed and the host sees RUNIT_ERR_TIMEOUT at the next flush.
#include "bf16_ops.cuh"
#include "gemv_common.cuh"
#include "tcgen05.cuh"
#include "tma.cuh"

namespace runit {
namespace gm {

static_assert(EPI_F32 == RUNIT_EPI_F32 && EPI_ADD == RUNIT_EPI_ADD && EPI_CAST == RUNIT_EPI_CAST && EPI_SILU_GLU == RUNIT_EPI_SILU_GLU &&
                  EPI_RELU2 == RUNIT_EPI_RELU2,
              "the epilogues of the C interface");

struct Args {
    const __nv_bfloat16* w;
    const float* x32;
    uint32_t rows, K, ldw, ldx, nb, T, tile_tok;
    const int32_t *tile_expert, *tile_nvalid, *tile_row0, *n_tok_tiles;
    void* out;
    uint32_t ldo;
    const float *pre, *post;
    float* tail;
    uint32_t tail_from, ldt;
    float cap;
    int32_t* status;
};

struct Tile {
    uint32_t rb, expert, row0, nvalid;
};
// Dense: the token tiles of a row block are neighbours (the weight block is read from HBM once); grouped: the row blocks of a
// token tile are neighbours.
__device__ __forceinline__ Tile tile_of(const Args& a, uint32_t item, uint32_t ntt) {
    Tile t;
    if (a.tile_expert) {
        const uint32_t tt = item / a.nb;
        t.rb = item % a.nb;
        t.expert = (uint32_t)a.tile_expert[tt];
        t.row0 = (uint32_t)a.tile_row0[tt];
        t.nvalid = (uint32_t)a.tile_nvalid[tt];
    } else {
        const uint32_t tt = item % ntt;
        t.rb = item / ntt;
        t.expert = 0;
        t.row0 = tt * a.tile_tok;
        t.nvalid = min(a.tile_tok, a.T - t.row0);
    }
    return t;
}
__device__ __forceinline__ uint32_t tok_tiles(const Args& a) {
    return a.tile_expert ? (uint32_t)*a.n_tok_tiles : (a.T + a.tile_tok - 1) / a.tile_tok;
}

template <typename TO>
__device__ __forceinline__ void store(TO* p, float v) {
    if constexpr (sizeof(TO) == 2) *p = __float2bfloat16_rn(v);
    else *p = v;
}
__device__ __forceinline__ float relu2(float v) {
    v = fmaxf(v, 0.f);
    return v * v;
}

// Lane l of a quad holds v[0..3] = its row's values of tokens 0..3; afterwards y[0..3] = the quad's four rows of token l & 3.
__device__ __forceinline__ void quad_transpose(const uint32_t* v, float (&y)[4], bool odd, bool high) {
    const uint32_t a = __shfl_xor_sync(0xffffffffu, odd ? v[0] : v[1], 1), b = __shfl_xor_sync(0xffffffffu, odd ? v[2] : v[3], 1);
    // even lanes: rows (0, 1) of tokens 0 and 2; odd lanes: of tokens 1 and 3
    const uint32_t p0 = odd ? a : v[0], p1 = odd ? v[1] : a, q0 = odd ? b : v[2], q1 = odd ? v[3] : b;
    const uint32_t c = __shfl_xor_sync(0xffffffffu, high ? p0 : q0, 2), d = __shfl_xor_sync(0xffffffffu, high ? p1 : q1, 2);
    y[0] = __uint_as_float(high ? c : p0);
    y[1] = __uint_as_float(high ? d : p1);
    y[2] = __uint_as_float(high ? q0 : c);
    y[3] = __uint_as_float(high ? q1 : d);
}
// N neighbouring outputs of one token, `left` of them inside the matrix
template <int N>
__device__ __forceinline__ void store_rows(__nv_bfloat16* o, const float (&y)[4], uint32_t left, uint32_t ldo) {
    if (left >= N && ldo % N == 0) {
        __nv_bfloat162 p[N / 2];
#pragma unroll
        for (int i = 0; i < N / 2; i++) p[i] = __floats2bfloat162_rn(y[2 * i], y[2 * i + 1]);
        if constexpr (N == 4) *reinterpret_cast<uint2*>(o) = *reinterpret_cast<const uint2*>(p);
        else *reinterpret_cast<uint32_t*>(o) = *reinterpret_cast<const uint32_t*>(p);
    } else {
        for (uint32_t i = 0; i < N && i < left; i++) o[i] = __float2bfloat16_rn(y[i]);
    }
}

constexpr int kThreads = 192, kRowsTile = 128, kABytes = kRowsTile * 128;
template <int NT>
struct Cfg {
    static constexpr int stage = kABytes + NT * 128;
    static constexpr int ns = 200 * 1024 / stage;
    static constexpr int smem = ns * stage + 1024 + 512;
    static constexpr int tmem_cols = 2 * NT;
};

template <int EPI, int NT>
__global__ void __launch_bounds__(kThreads, 1)
gemm_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, const Args a) {
    constexpr int NS = Cfg<NT>::ns;
    extern __shared__ uint8_t smem_raw[];
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t* base_p = smem_raw + (base - smem_u32(smem_raw));
    const uint32_t ctrl = base + NS * Cfg<NT>::stage;
    const uint32_t bar_full = ctrl, bar_empty = bar_full + 8 * NS, bar_accf = bar_empty + 8 * NS, bar_acce = bar_accf + 16, holder = bar_acce + 16;
    volatile uint32_t* holder_p = reinterpret_cast<volatile uint32_t*>(base_p + (holder - base));
    volatile int* abort_flag = reinterpret_cast<volatile int*>(base_p + (holder - base) + 4);
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (int s = 0; s < NS; s++) {
            mbar_init(bar_full + 8 * s, 1);
            mbar_init(bar_empty + 8 * s, 1);
        }
        for (int s = 0; s < 2; s++) {
            mbar_init(bar_accf + 8 * s, 1);
            mbar_init(bar_acce + 8 * s, 4);
        }
        *abort_flag = 0;
        fence_mbar_init();
    }
    if (warp == 1) {
        tmem_alloc(holder, Cfg<NT>::tmem_cols);
        tmem_relinquish();
    }
    __syncwarp();
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = *holder_p;
    const uint32_t ntt = tok_tiles(a), n_items = ntt * a.nb, ksteps = (a.K + 63) / 64;

    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;
            bool ok = true;
            for (uint32_t item = blockIdx.x; item < n_items && ok && !*abort_flag; item += gridDim.x) {
                const Tile t = tile_of(a, item, ntt);
                const int32_t wrow = (int32_t)(t.expert * a.rows + t.rb * kRowsTile);
                for (uint32_t k = 0; k < ksteps; k++, it++) {
                    const uint32_t s = it % NS, ph = (it / NS) & 1;
                    if (!mbar_wait_timed(bar_empty + 8 * s, ph ^ 1, abort_flag)) { ok = false; break; }
                    const uint32_t dst = base + s * Cfg<NT>::stage;
                    mbar_expect_tx(bar_full + 8 * s, Cfg<NT>::stage);
                    tma_load_2d(dst, &map_w, (int32_t)(k * 128), wrow, bar_full + 8 * s);
                    tma_load_2d(dst + kABytes, &map_x, (int32_t)(k * 128), (int32_t)t.row0, bar_full + 8 * s);
                }
            }
            if (!ok || *abort_flag) {       // nobody consumes them any more: wait (bounded) for the loads in flight
                const uint32_t n = it < (uint32_t)NS ? it : (uint32_t)NS;
                for (uint32_t i = it - n; i < it; i++) mbar_wait(bar_full + 8 * (i % NS), (i / NS) & 1);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            uint32_t it = 0, n = 0;
            bool ok = true;
            for (uint32_t item = blockIdx.x; item < n_items && ok && !*abort_flag; item += gridDim.x, n++) {
                const Tile t = tile_of(a, item, ntt);
                const uint32_t idesc = umma_idesc_bf16(kRowsTile, (t.nvalid + 15) & ~15u);
                const uint32_t acc = n & 1, d = tmem + acc * NT;
                if (!mbar_wait_timed(bar_acce + 8 * acc, ((n >> 1) & 1) ^ 1, abort_flag)) break;
                tc_fence_after_sync();
                for (uint32_t k = 0; k < ksteps; k++, it++) {
                    const uint32_t s = it % NS, ph = (it / NS) & 1;
                    if (!mbar_wait_timed(bar_full + 8 * s, ph, abort_flag)) { ok = false; break; }
                    tc_fence_after_sync();
                    const uint64_t da = umma_desc_sw128(base + s * Cfg<NT>::stage), db = umma_desc_sw128(base + s * Cfg<NT>::stage + kABytes);
#pragma unroll
                    for (uint32_t k4 = 0; k4 < 4; k4++) umma_bf16(d, da + 2 * k4, db + 2 * k4, idesc, (k | k4) != 0);
                    umma_commit(bar_empty + 8 * s);
                }
                if (ok) umma_commit(bar_accf + 8 * acc);
            }
        }
    } else {
        const uint32_t quarter = warp & 3;
        uint32_t n = 0;
        for (uint32_t item = blockIdx.x; item < n_items; item += gridDim.x, n++) {
            const Tile t = tile_of(a, item, ntt);
            const uint32_t acc = n & 1;
            uint32_t ready = 1;
            if (lane == 0) ready = mbar_wait_timed(bar_accf + 8 * acc, (n >> 1) & 1, abort_flag);
            ready = __shfl_sync(0xffffffffu, ready, 0);
            if (!ready) break;
            tc_fence_after_sync();
            const uint32_t taddr = tmem + ((quarter * 32) << 16) + acc * NT;
            const uint32_t r = t.rb * kRowsTile + quarter * 32 + lane;     // row of the weight matrix
            const bool live = r < a.rows;
#pragma unroll 1
            for (uint32_t cg = 0; cg * 32 < t.nvalid; cg++) {
                uint32_t v[32];
                tmem_ld32(taddr + cg * 32, v);
                tmem_ld_wait();
                const uint32_t tok0 = t.row0 + cg * 32, cnt = min(32u, t.nvalid - cg * 32);
                if constexpr (EPI == EPI_SILU_GLU || EPI == EPI_RELU2 || EPI == EPI_CAST) {
                    // Four lanes exchange their values of four tokens, so that each holds four neighbouring rows of one token: one
                    // wide store and one pair of factors instead of four.
                    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out);
                    const bool odd = lane & 1, high = lane & 2;
                    const uint32_t r4 = r & ~3u;
#pragma unroll
                    for (int j = 0; j < 32; j += 4) {
                        float y[4];
                        quad_transpose(v + j, y, odd, high);
                        const uint32_t jj = j + (lane & 3);
                        if (jj >= cnt || r4 >= a.rows) continue;
                        const uint32_t tok = tok0 + jj;
                        __nv_bfloat16* o = out + (size_t)tok * a.ldo;
                        if constexpr (EPI == EPI_CAST) {
                            if (r4 + 4 <= a.tail_from) {
                                store_rows<4>(o + r4, y, a.rows - r4, a.ldo);
                            } else {
                                for (uint32_t i = 0; i < 4 && r4 + i < a.rows; i++) {
                                    if (r4 + i < a.tail_from) o[r4 + i] = __float2bfloat16_rn(y[i]);
                                    else a.tail[(size_t)tok * a.ldt + r4 + i - a.tail_from] = y[i];
                                }
                            }
                        } else {
                            const float pre = a.pre ? a.pre[tok] : 1.f, post = a.post ? a.post[tok] : 1.f;
                            if constexpr (EPI == EPI_SILU_GLU) {      // rows 2i, 2i+1: gate and up of output i
#pragma unroll
                                for (int i = 0; i < 2; i++) {
                                    const float g = y[2 * i] * pre, u = y[2 * i + 1] * pre;
                                    y[i] = __fdividef(g, 1.0f + __expf(-g)) * u * post;
                                }
                                store_rows<2>(o + r4 / 2, y, (a.rows - r4) / 2, a.ldo);
                            } else {
#pragma unroll
                                for (int i = 0; i < 4; i++) y[i] = relu2(y[i] * pre) * post;
                                store_rows<4>(o + r4, y, a.rows - r4, a.ldo);
                            }
                        }
                    }
                } else if constexpr (EPI == EPI_ADD) {
                    // all loads of the group before its first store (the compiler may not reorder them across one)
                    float* out = reinterpret_cast<float*>(a.out) + (size_t)tok0 * a.ldo + r;
                    float old[32];
#pragma unroll
                    for (int j = 0; j < 32; j++) old[j] = (live && (uint32_t)j < cnt) ? out[(size_t)j * a.ldo] : 0.f;
#pragma unroll
                    for (int j = 0; j < 32; j++)
                        if (live && (uint32_t)j < cnt) out[(size_t)j * a.ldo] = old[j] + __uint_as_float(v[j]);
                } else {
#pragma unroll
                    for (int j = 0; j < 32; j++) {
                        if (!live || (uint32_t)j >= cnt) continue;
                        float f = __uint_as_float(v[j]);
                        if (a.cap != 0.f) f = a.cap * tanhf(f / a.cap);
                        const size_t o = (size_t)(tok0 + j) * a.ldo + r;
                        reinterpret_cast<float*>(a.out)[o] = f;
                    }
                }
            }
            tc_fence_before_sync();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_acce + 8 * acc);
        }
    }
    __syncwarp();
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after_sync();
        tmem_dealloc(tmem, Cfg<NT>::tmem_cols);
    }
    if (tid == 0 && *abort_flag && a.status) atomicExch(a.status, 2);
}

// 64 weight rows x 64 tokens per CTA, K in chunks of 16 through shared memory; a thread keeps 4 consecutive rows x 4 tokens.
// Every product is one chain of multiply-adds over ascending k.
template <int EPI>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const Args a) {
    __shared__ __align__(16) float ws[16][68], xs[16][68];      // [k][row], [k][token]
    const uint32_t tid = threadIdx.x, tr = tid & 15, tt = tid >> 4;
    const uint32_t ntt = tok_tiles(a), n_items = ntt * a.nb;
    for (uint32_t item = blockIdx.x; item < n_items; item += gridDim.x) {
        const Tile t = tile_of(a, item, ntt);
        float acc[4][4];
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
        const uint32_t lr = tid >> 2, lk = (tid & 3) * 4;         // a thread stages 4 k of one row and of one token
        for (uint32_t k0 = 0; k0 < a.K; k0 += 16) {
            const uint32_t row = t.rb * 64 + lr;
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const uint32_t k = k0 + lk + i;
                ws[lk + i][lr] = (row < a.rows && k < a.K) ? __bfloat162float(a.w[((size_t)t.expert * a.rows + row) * a.ldw + k]) : 0.f;
                xs[lk + i][lr] = (lr < t.nvalid && k < a.K) ? a.x32[(size_t)(t.row0 + lr) * a.ldx + k] : 0.f;
            }
            __syncthreads();
#pragma unroll
            for (int k = 0; k < 16; k++) {
                const float4 w4 = *reinterpret_cast<const float4*>(&ws[k][tr * 4]), x4 = *reinterpret_cast<const float4*>(&xs[k][tt * 4]);
                const float wv[4] = {w4.x, w4.y, w4.z, w4.w}, xv[4] = {x4.x, x4.y, x4.z, x4.w};
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++) acc[i][j] = fmaf(wv[i], xv[j], acc[i][j]);
            }
            __syncthreads();
        }
        float* out = reinterpret_cast<float*>(a.out);
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const uint32_t tok = tt * 4 + j;
            if (tok >= t.nvalid) continue;
            const float pre = a.pre ? a.pre[t.row0 + tok] : 1.f, post = a.post ? a.post[t.row0 + tok] : 1.f;
            float* o = out + (size_t)(t.row0 + tok) * a.ldo;
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const uint32_t r = t.rb * 64 + tr * 4 + i;
                if (r >= a.rows) continue;
                if constexpr (EPI == EPI_SILU_GLU) {
                    if (i & 1) continue;
                    const float g = acc[i][j] * pre, u = acc[i + 1][j] * pre;
                    o[r >> 1] = g / (1.0f + expf(-g)) * u * post;
                } else if constexpr (EPI == EPI_RELU2) o[r] = relu2(acc[i][j] * pre) * post;
                else if constexpr (EPI == EPI_ADD) o[r] += acc[i][j];
                else if (r >= a.tail_from) a.tail[(size_t)(t.row0 + tok) * a.ldt + r - a.tail_from] = acc[i][j];
                else o[r] = a.cap != 0.f ? a.cap * tanhf(acc[i][j] / a.cap) : acc[i][j];
            }
        }
    }
}

template <int EPI, int NT>
static int32_t launch_tc(runit_ctx* ctx, const char* name, const GemmDesc& d, Args a, uint32_t items) {
    static bool attr_set[64] = {false};
    if (ctx->device >= 0 && ctx->device < 64 && !attr_set[ctx->device]) {
        RUNIT_CUDA_TRY(ctx, cudaFuncSetAttribute(gemm_tc_kernel<EPI, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg<NT>::smem));
        attr_set[ctx->device] = true;
    }
    CUtensorMap map_w, map_x;
    int32_t st = runit_get_tmap(ctx, d.w, (uint64_t)d.n_experts * d.rows, (uint64_t)d.ldw * 2, kRowsTile, 128, &map_w, 1);
    if (st != RUNIT_OK) return st;
    if ((st = runit_get_tmap(ctx, d.x, d.x_rows, (uint64_t)d.ldx * 2, NT, 128, &map_x, 1)) != RUNIT_OK) return st;
    const uint32_t grid = items < (uint32_t)ctx->sm_count ? items : (uint32_t)ctx->sm_count;
    gemm_tc_kernel<EPI, NT><<<grid, kThreads, Cfg<NT>::smem, ctx->stream>>>(map_w, map_x, a);
    return runit_after_launch(ctx, name);
}

template <int NT>
static int32_t dispatch_tc(runit_ctx* ctx, const char* name, const GemmDesc& d, const Args& a, uint32_t items) {
    switch (d.epi) {
        case EPI_F32: return launch_tc<EPI_F32, NT>(ctx, name, d, a, items);
        case EPI_ADD: return launch_tc<EPI_ADD, NT>(ctx, name, d, a, items);
        case EPI_CAST: return launch_tc<EPI_CAST, NT>(ctx, name, d, a, items);
        case EPI_SILU_GLU: return launch_tc<EPI_SILU_GLU, NT>(ctx, name, d, a, items);
        default: return launch_tc<EPI_RELU2, NT>(ctx, name, d, a, items);
    }
}

// Token tile of a dense product: the one with the least (waves of tiles) x (time of a tile).  A tile's time hardly falls with
// its width below 128 tokens (the MMA issue rate bounds it), hence the weights.
static uint32_t dense_tile_tok(const runit_ctx* ctx, uint32_t nb, uint32_t T) {
    const uint32_t nt[3] = {256, 128, 64};
    const float cost[3] = {1.0f, 0.6f, 0.45f};
    uint32_t best = 64;
    float best_c = 1e30f;
    for (int i = 0; i < 3; i++) {
        const uint64_t tiles = (uint64_t)nb * ((T + nt[i] - 1) / nt[i]);
        const float c = (float)((tiles + ctx->sm_count - 1) / ctx->sm_count) * cost[i];
        if (c < best_c) { best_c = c; best = nt[i]; }
    }
    return best;
}

}  // namespace gm

uint32_t gemm_bf16_tile_tok(uint32_t tokens_per_expert, bool exact) {
    if (exact) return 64;
    return tokens_per_expert > 128 ? 256 : (tokens_per_expert > 48 ? 128 : 64);
}

int32_t gemm_bf16(runit_ctx* ctx, const char* name, const GemmDesc& d, bool exact) {
    RUNIT_REQUIRE(ctx, d.w && d.x && d.out && d.rows > 0 && d.K > 0 && d.T > 0, "%s: bad argument", name);
    RUNIT_REQUIRE(ctx, d.ldw % 8 == 0 && d.ldw >= d.K && d.ldx >= d.K, "%s: bad row pitch", name);
    RUNIT_REQUIRE(ctx, d.epi != EPI_SILU_GLU || d.rows % 2 == 0, "%s: a gated product needs pairs of rows", name);
    const bool grouped = d.tile_expert != nullptr;
    gm::Args a{(const __nv_bfloat16*)d.w, (const float*)d.x, d.rows, d.K, d.ldw, d.ldx, 0, d.T, 0, d.tile_expert, d.tile_nvalid, d.tile_row0,
               d.n_tok_tiles, d.out, d.ldo, d.pre, d.post, d.tail, d.tail ? d.tail_from : 0xFFFFFFFFu, d.ldt, d.cap, ctx->d_status};
    RUNIT_REQUIRE(ctx, (!d.tail || d.epi == EPI_CAST) && (d.cap == 0.f || d.epi == EPI_F32), "%s: f32 columns go with EPI_CAST, a cap with EPI_F32", name);
    if (exact) {
        a.nb = (d.rows + 63) / 64;
        a.tile_tok = 64;
        const uint64_t items = (uint64_t)a.nb * (grouped ? d.max_tiles : (d.T + 63) / 64);
        const uint32_t cap = (uint32_t)ctx->sm_count * 8, grid = items < cap ? (uint32_t)items : cap;
        switch (d.epi) {
            case EPI_ADD: gm::gemm_f32_kernel<EPI_ADD><<<grid, 256, 0, ctx->stream>>>(a); break;
            case EPI_SILU_GLU: gm::gemm_f32_kernel<EPI_SILU_GLU><<<grid, 256, 0, ctx->stream>>>(a); break;
            case EPI_RELU2: gm::gemm_f32_kernel<EPI_RELU2><<<grid, 256, 0, ctx->stream>>>(a); break;
            default: gm::gemm_f32_kernel<EPI_F32><<<grid, 256, 0, ctx->stream>>>(a); break;
        }
        return runit_after_launch(ctx, name);
    }
    RUNIT_REQUIRE(ctx, d.ldx % 8 == 0 && runit_aligned(d.x, 16) && runit_aligned(d.w, 16), "%s: operands must be 16-byte aligned", name);
    a.nb = (d.rows + gm::kRowsTile - 1) / gm::kRowsTile;
    a.tile_tok = grouped ? d.tile_tok : gm::dense_tile_tok(ctx, a.nb, d.T);
    const uint64_t items64 = (uint64_t)a.nb * (grouped ? d.max_tiles : (d.T + a.tile_tok - 1) / a.tile_tok);
    const uint32_t items = items64 < 0x7fffffffull ? (uint32_t)items64 : 0x7fffffffu;
    if (a.tile_tok == 256) return gm::dispatch_tc<256>(ctx, name, d, a, items);
    if (a.tile_tok == 128) return gm::dispatch_tc<128>(ctx, name, d, a, items);
    RUNIT_REQUIRE(ctx, a.tile_tok == 64, "%s: token tiles of 64, 128 or 256 only", name);
    return gm::dispatch_tc<64>(ctx, name, d, a, items);
}

}  // namespace runit

using namespace runit;

extern "C" {

int32_t runit_gemm_bf16_rows(runit_ctx_t* ctx, const void* weight, const void* x, void* y, uint32_t ldy, uint32_t T, uint32_t m, uint32_t k,
                             int32_t exact, int32_t epi, const void* pre, const void* post) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, weight && x && y && T > 0 && m > 0 && k > 0 && epi >= RUNIT_EPI_F32 && epi <= RUNIT_EPI_RELU2, "gemm_bf16_rows: bad argument");
    GemmDesc d;
    d.w = weight; d.rows = m; d.K = k; d.ldw = pad8(k); d.x = x; d.ldx = pad8(k); d.x_rows = T; d.T = T; d.epi = epi; d.out = y; d.ldo = ldy;
    d.pre = (const float*)pre; d.post = (const float*)post;
    return gemm_bf16(ctx, "gemm_bf16_rows", d, exact != 0);
}

}  // extern "C"
