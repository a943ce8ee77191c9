// Layers with a decaying linear state per head, S <- decay S + k v^T, o = S^T q: retention (decay fixed per head) and the
// state-space layer (decay and step size per token).  S is f32 and so is everything that enters the recurrence besides the
// projections and the short convolution.  A sequence that starts at position 0 starts from a zero state: the kernels look at
// the position, nothing has to be cleared.
//   * ssm_step_kernel: one token, convolution to gate (the retention's step is in head_attention.cu, beside the attention).
//   * ssm_conv_kernel: convolution, silu and softplus of a portion.
//   * linear_scan_kernel: the recurrence token by token, state in registers.  32-bit runs, short portions, odd sizes.
//   * chunk_state_kernel + chunk_out_kernel: long portions in bf16, in chunks of 128 tokens on tensor cores.  The first walks the
//     chunks of one head and 32 value columns with the state in accumulators and leaves the state at the start of every chunk
//     (as the sum of two bf16 numbers); the second forms all chunks at once: what the starting state contributes, and the masked
//     products within the chunk, weighted by decays in f32.
//   * gated_norm_kernel: gate and norm of groups of the result.
#include "bf16_ops.cuh"
#include "gemv_common.cuh"
#include "linear_state.cuh"
#include "tma.cuh"

namespace runit {
namespace ls {

__device__ __forceinline__ float wsum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// ── one token ──
// Convolved and activated value of channel c at position pos; raw: its projection at pos.
__device__ __forceinline__ float conv_step(const Ssm& m, uint32_t c, float raw, uint32_t pos) {
    const uint32_t ch = m.channels();
    float s = m.conv_b[c];
    for (uint32_t j = 0; j + 1 < m.taps; j++) {
        const uint32_t back = m.taps - 1 - j;
        if (pos >= back) s = fmaf(m.conv_w[(size_t)c * m.taps + j], m.ring[(size_t)((pos - back) % m.taps) * ch + c], s);
    }
    return silu(fmaf(m.conv_w[(size_t)c * m.taps + m.taps - 1], raw, s));
}

// grid (heads, ceil(vdim / 32)).  The ring row of this position is not read by anyone in this launch.
__global__ void __launch_bounds__(256) ssm_step_kernel(const Ssm m, const float* proj, float* y, float* squares, const int32_t* pos_ptr) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[8][33];
    float *qs = sm, *ks = sm + m.state;
    const uint32_t tid = threadIdx.x, lane = tid & 31, h = blockIdx.x, j = blockIdx.y * 32 + lane, inner = m.inner(), ch = m.channels();
    const uint32_t rep = m.heads / m.groups, g = h / rep;
    float* S = m.s + (size_t)h * m.state * m.vdim;
    StateRows st;
    load_rows(st, S, m.state, m.vdim, j, 0);         // the state is that of the last step: final long before this launch
    const float a = m.a[h], bias = m.dt_bias[h], skip = m.skip[h];
    grid_dependency_wait();
    grid_launch_dependents();
    const uint32_t pos = (uint32_t)*pos_ptr;
    float* slot = m.ring + (size_t)(pos % m.taps) * ch;
    const float dt = softplus(proj[2 * inner + 2 * m.groups * m.state + h] + bias);
    const float* xbc = proj + inner;
    const bool writes = blockIdx.y == 0 && h % rep == 0;
    for (uint32_t i = tid; i < 2 * m.state; i += 256) {
        const bool is_c = i >= m.state;
        const uint32_t n = is_c ? i - m.state : i, c = inner + (is_c ? m.groups * m.state : 0) + g * m.state + n;
        const float raw = xbc[c], v = conv_step(m, c, raw, pos);
        if (is_c) qs[n] = v;
        else ks[n] = v * dt;
        if (writes) slot[c] = raw;
    }
    float v = 0.f, z = 0.f;
    if (j < m.vdim) {
        const uint32_t c = h * m.vdim + j;
        const float raw = xbc[c];
        v = conv_step(m, c, raw, pos);
        z = proj[c];
        if (tid < 32) slot[c] = raw;
    }
    __syncthreads();
    const float o = state_step(st, S, m.state, m.vdim, j, qs, ks, v, expf(a * dt), pos == 0, red);
    if (tid < 32) {
        const float r = j < m.vdim ? fmaf(skip, v, o) * silu(z) : 0.f;
        if (j < m.vdim) y[h * m.vdim + j] = r;
        const float sq = wsum(r * r);
        if (tid == 0) squares[h * gridDim.y + blockIdx.y] = sq;
    }
}

// ── many tokens: convolution ──
// grid (channel blocks + 1, token blocks of kConvTok), a thread walks VEC neighbouring channels; the last column of blocks does the
// step sizes.  Only the first token block reads the ring, and each of its threads rewrites it for its channels afterwards.
// TAPS > 0: the window stays in registers.
constexpr uint32_t kConvTok = 32, kConvThreads = 128;
static_assert(kConvTok == 32, "four groups of eight tokens");
template <int VEC, typename TA>
__device__ __forceinline__ void load_vec(const TA* p, float (&v)[VEC]) {
    if constexpr (VEC == 1) {
        v[0] = to_f32(*p);
    } else if constexpr (sizeof(TA) == 2) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        v[0] = __uint_as_float(u.x << 16); v[1] = __uint_as_float(u.x & 0xffff0000u);
        v[2] = __uint_as_float(u.y << 16); v[3] = __uint_as_float(u.y & 0xffff0000u);
    } else {
        const float4 u = *reinterpret_cast<const float4*>(p);
        v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w;
    }
}
template <int VEC, typename TA>
__device__ __forceinline__ void store_vec(TA* p, const float (&v)[VEC]) {
    if constexpr (VEC == 1) {
        put(p, v[0]);
    } else if constexpr (sizeof(TA) == 2) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    } else {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
}
// One token of the window kernel: the window moves on by `in`, y = silu(taps . window + b).
template <typename TA, int TAPS, int VEC>
__device__ __forceinline__ void conv_token(float (&win)[TAPS][VEC], const float (&wr)[TAPS][VEC], const float (&b)[VEC], const float (&in)[VEC],
                                           float (&y)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; e++) {
#pragma unroll
        for (int j = 0; j + 1 < TAPS; j++) win[j][e] = win[j + 1][e];
        win[TAPS - 1][e] = in[e];
        float s = b[e];
#pragma unroll
        for (int j = 0; j < TAPS; j++) s = fmaf(wr[j][e], win[j][e], s);
        y[e] = silu_for<TA>(s);
    }
}
template <typename TA, int TAPS, int VEC>
__global__ void __launch_bounds__(kConvThreads) ssm_conv_kernel(const Ssm m, const TA* __restrict__ proj, uint32_t ld, TA* __restrict__ out,
                                                                 uint32_t ld_out, float* __restrict__ dt, uint32_t T, uint32_t start) {
    const uint32_t t0 = blockIdx.y * kConvTok, t1 = min(T, t0 + kConvTok);
    if (blockIdx.x == gridDim.x - 1) {
        for (uint32_t i = t0 * m.heads + threadIdx.x; i < t1 * m.heads; i += kConvThreads) dt[i] = softplus(dt[i] + m.dt_bias[i % m.heads]);
        return;
    }
    const uint32_t c = (blockIdx.x * kConvThreads + threadIdx.x) * VEC, ch = m.channels(), taps = TAPS ? TAPS : m.taps;
    if (c >= ch) return;
    const TA* x = proj + m.inner() + c;
    float b[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) b[e] = m.conv_b[c + e];
    auto input = [&](int32_t t, float (&v)[VEC]) {           // t relative to the portion
        if (t >= 0) {
            load_vec<VEC>(x + (size_t)t * ld, v);
        } else {
#pragma unroll
            for (int e = 0; e < VEC; e++) v[e] = (int32_t)start + t >= 0 ? m.ring[(size_t)((start + t) % taps) * ch + c + e] : 0.f;
        }
    };
    if constexpr (TAPS > 0) {
        constexpr uint32_t B = 8;                            // tokens requested together
        constexpr bool ASYNC = sizeof(TA) == 2 && VEC == 4;  // all of the block's tokens on their way at once, through shared memory
        extern __shared__ __align__(16) uint2 own[];         // [kConvTok][kConvThreads]: a thread reads what it has requested itself
        if constexpr (ASYNC) {
#pragma unroll
            for (uint32_t i = 0; i < kConvTok; i++) {
                if (t0 + i < t1) cp_async8(smem_u32(own + i * kConvThreads + threadIdx.x), x + (size_t)(t0 + i) * ld);
                if (i % B == B - 1) cp_async_commit();
            }
        }
        float win[TAPS][VEC], wr[TAPS][VEC];
#pragma unroll
        for (int j = 0; j < TAPS; j++)
#pragma unroll
            for (int e = 0; e < VEC; e++) wr[j][e] = m.conv_w[(size_t)(c + e) * TAPS + j];
#pragma unroll
        for (int j = 0; j + 1 < TAPS; j++) input((int32_t)t0 - (TAPS - 1 - j), win[j + 1]);
        if constexpr (ASYNC) {
#pragma unroll
            for (uint32_t q = 0; q < kConvTok / B; q++) {
                if (q == 0) cp_async_wait<3>();
                else if (q == 1) cp_async_wait<2>();
                else if (q == 2) cp_async_wait<1>();
                else cp_async_wait<0>();
#pragma unroll
                for (uint32_t i = q * B; i < q * B + B; i++) {
                    if (t0 + i >= t1) break;
                    float in[VEC], y[VEC];
                    load_vec<VEC>(reinterpret_cast<const TA*>(own + i * kConvThreads + threadIdx.x), in);
                    conv_token<TA, TAPS, VEC>(win, wr, b, in, y);
                    store_vec<VEC>(out + (size_t)(t0 + i) * ld_out + c, y);
                }
            }
        } else {
            for (uint32_t tb = t0; tb < t1; tb += B) {
                float in[B][VEC];
#pragma unroll
                for (uint32_t i = 0; i < B; i++)
                    if (tb + i < t1) load_vec<VEC>(x + (size_t)(tb + i) * ld, in[i]);
#pragma unroll
                for (uint32_t i = 0; i < B; i++) {
                    if (tb + i >= t1) break;
                    float y[VEC];
                    conv_token<TA, TAPS, VEC>(win, wr, b, in[i], y);
                    store_vec<VEC>(out + (size_t)(tb + i) * ld_out + c, y);
                }
            }
        }
    } else {
        for (uint32_t t = t0; t < t1; t++) {
            float s[VEC];
#pragma unroll
            for (int e = 0; e < VEC; e++) s[e] = b[e];
            for (uint32_t j = 0; j < taps; j++) {
                float v[VEC];
                input((int32_t)t - (int32_t)(taps - 1 - j), v);
#pragma unroll
                for (int e = 0; e < VEC; e++) s[e] = fmaf(m.conv_w[(size_t)(c + e) * taps + j], v[e], s[e]);
            }
#pragma unroll
            for (int e = 0; e < VEC; e++) s[e] = silu_for<TA>(s[e]);
            store_vec<VEC>(out + (size_t)t * ld_out + c, s);
        }
    }
    if (blockIdx.y == 0)
        for (uint32_t t = T > taps ? T - taps : 0; t < T; t++) {
            float v[VEC];
            load_vec<VEC>(x + (size_t)t * ld, v);
#pragma unroll
            for (int e = 0; e < VEC; e++) m.ring[(size_t)((start + t) % taps) * ch + c + e] = v[e];
        }
}

// ── many tokens: the recurrence token by token ──
// grid (heads, ceil(dv / 32)), 256 threads: lane = column, warp w keeps rows w, w + 8, ... of the state in registers.
template <typename TA, int NR>
__global__ void __launch_bounds__(256) linear_scan_kernel(const LinearRows d, uint32_t T, uint32_t fresh) {
    __shared__ float qs[2][NR * 8], ks[2][NR * 8], red[2][8][33];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, j = blockIdx.y * 32 + lane, g = h / (d.heads / d.groups);
    const bool live = j < d.dv;
    const TA *q = (const TA*)d.q + g * d.dk, *k = (const TA*)d.k + g * d.dk, *v = (const TA*)d.v + h * d.dv + j;
    float* S = d.state + (size_t)h * d.dk * d.dv;
    TA* out = (TA*)d.out + h * d.dv + j;
    const float skip = d.skip ? d.skip[h] : 0.f, ld = d.log_decay ? d.log_decay[h] : 0.f, fixed = d.decay ? d.decay[h] : 0.f;
    float s[NR];
#pragma unroll
    for (int r = 0; r < NR; r++) {
        const uint32_t i = warp + 8 * r;
        s[r] = (!fresh && i < d.dk && live) ? S[(size_t)i * d.dv + j] : 0.f;
    }
    for (uint32_t t = 0; t < T; t++) {
        const uint32_t b = t & 1;
        const float dt = d.dt ? d.dt[(size_t)t * d.heads + h] : 1.f;
        for (uint32_t i = tid; i < NR * 8; i += 256) {
            qs[b][i] = i < d.dk ? to_f32(q[(size_t)t * d.ldq + i]) : 0.f;
            ks[b][i] = i < d.dk ? to_f32(k[(size_t)t * d.ldk + i]) * dt : 0.f;
        }
        const float vv = live ? to_f32(v[(size_t)t * d.ldv]) : 0.f, decay = d.dt ? expf(ld * dt) : fixed;
        __syncthreads();
        float o = 0.f;
#pragma unroll
        for (int r = 0; r < NR; r++) {
            s[r] = fmaf(ks[b][warp + 8 * r], vv, decay * s[r]);
            o = fmaf(s[r], qs[b][warp + 8 * r], o);
        }
        red[b][warp][lane] = o;
        __syncthreads();
        if (warp == 0 && live) {
            float sum = skip * vv;
#pragma unroll
            for (int w = 0; w < 8; w++) sum += red[b][w][lane];
            put(out + (size_t)t * d.ldo, sum);
        }
    }
#pragma unroll
    for (int r = 0; r < NR; r++) {
        const uint32_t i = warp + 8 * r;
        if (i < d.dk && live) S[(size_t)i * d.dv + j] = s[r];
    }
}

// ── many tokens: chunks ──
constexpr uint32_t kChunk = 128;
static inline uint32_t pad64(uint32_t n) { return (n + 63) & ~63u; }

__device__ __forceinline__ uint32_t pack_bf2(float a, float b) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ float bf_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf_hi(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}
// Rows t0 .. t0 + ROWS - 1 of a bf16 matrix (n of its columns) into shared rows of COLS + 8 elements; rows
// from T on and columns from n on become zero.  Asynchronous where the rows are 16-byte aligned (wide).  256 threads.
template <int ROWS, int COLS>
__device__ __forceinline__ void stage_rows(__nv_bfloat16* dst, const __nv_bfloat16* src, uint32_t ld, uint32_t n, uint32_t t0, uint32_t T, bool wide) {
    constexpr uint32_t CPR = COLS / 8, STEP = 256 / CPR, PITCH = COLS + 8;
    static_assert(256 % CPR == 0 && ROWS % STEP == 0, "whole passes");
    const uint32_t r0 = threadIdx.x / CPR, c = (threadIdx.x % CPR) * 8;
    const __nv_bfloat16* s = src + (size_t)(t0 + r0) * ld + c;
    __nv_bfloat16* p = dst + r0 * PITCH + c;
    const uint32_t rows = t0 + r0 < T ? T - t0 - r0 : 0;       // rows left from this thread's first one
    const bool in = c < n;
#pragma unroll
    for (uint32_t r = 0; r < (uint32_t)ROWS; r += STEP) {
        if (!in || r >= rows) {
            *reinterpret_cast<uint4*>(p + r * PITCH) = make_uint4(0, 0, 0, 0);
        } else if (wide) {
            cp_async16(smem_u32(p + r * PITCH), s);
        } else {
            for (uint32_t e = 0; e < 8; e++) p[r * PITCH + e] = c + e < n ? s[e] : __float2bfloat16_rn(0.f);
        }
        s += (size_t)STEP * ld;
    }
}
// 2^x (the argument is not positive)
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
constexpr float kLog2e = 1.44269504088896341f;
__device__ __forceinline__ bool rows_aligned(const void* p, uint32_t ld, uint32_t n) {
    return (reinterpret_cast<uintptr_t>(p) & 15u) == 0 && (ld & 7u) == 0 && (n & 7u) == 0;
}
// One warp: la[t] = sum of the binary logarithms of the decays of tokens 0 .. t of the chunk (nothing for the tokens past the end),
// w[t] = step size.
__device__ __forceinline__ void chunk_decays(const LinearRows& d, uint32_t h, uint32_t t0, uint32_t T, float* la, float* w) {
    constexpr int P = kChunk / 32;
    const uint32_t lane = threadIdx.x & 31;
    const float ld = d.log_decay[h] * kLog2e;
    float x[P];
#pragma unroll
    for (int i = 0; i < P; i++) {
        const uint32_t t = t0 + P * lane + i;
        const float dt = t < T ? (d.dt ? d.dt[(size_t)t * d.heads + h] : 1.f) : 0.f;
        w[P * lane + i] = dt;
        x[i] = ld * dt + (i ? x[i - 1] : 0.f);
    }
    float s = x[P - 1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float n = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= (uint32_t)o) s += n;
    }
    const float before = s - x[P - 1];
#pragma unroll
    for (int i = 0; i < P; i++) la[P * lane + i] = before + x[i];
}

// The state of one head at the start of a chunk, as the operand fragments the second kernel multiplies: [16 value columns]
// [16 key rows][high, low part][lane] 16 bytes.  A lane's 16 bytes: value column lane / 4, key rows 2 (lane % 4), + 1 and + 8, + 9;
// then the same of value column lane / 4 + 8.
__device__ __forceinline__ size_t state_fragments(uint32_t chunk, uint32_t heads, uint32_t h, uint32_t dkp, uint32_t dvp) {
    return ((size_t)chunk * heads + h) * (dvp / 16) * (dkp / 16) * 64;
}

// The state is carried as its transpose, 16 value columns x 8 key rows per accumulator tile, which is the layout of those
// fragments.  grid (heads, dvp / 32), 8 warps: warp = 16 of the CTA's 32 value columns x every fourth block of 16 key rows.  Keys
// arrive in steps of 64 or 128 tokens, three steps deep; the values are weighted on their way into shared memory.  The decays of all
// chunks are summed up before the walk.  DK >= dk: the rest is zero.
template <int DK>
struct StateCfg {
    static constexpr uint32_t step = DK <= 128 ? 128 : 64, lv = 40;
    static size_t smem(uint32_t nc) { return (size_t)3 * step * (DK + 8) * 2 + (size_t)2 * step * lv * 2 + (size_t)nc * kChunk * 8; }
};
template <int DK>
__global__ void __launch_bounds__(256) chunk_state_kernel(const LinearRows d, uint4* __restrict__ states, uint32_t dvp, uint32_t T, uint32_t fresh) {
    extern __shared__ __align__(16) uint8_t smem[];
    constexpr uint32_t STEP = StateCfg<DK>::step, LV = StateCfg<DK>::lv, LK = DK + 8, NB = DK / 16, NBW = NB / 4, VP = STEP / 64, PER = kChunk / STEP;
    const uint32_t nc = (T + kChunk - 1) / kChunk, ns = (T + STEP - 1) / STEP;
    __nv_bfloat16* kS = reinterpret_cast<__nv_bfloat16*>(smem);       // [3][STEP][LK]
    __nv_bfloat16* vS = kS + 3 * STEP * LK;                           // [2][STEP][LV]
    float* la = reinterpret_cast<float*>(vS + 2 * STEP * LV);         // [nc][kChunk]
    float* wt = la + nc * kChunk;                                     // [nc][kChunk]
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, mt = warp & 1, quarter = warp >> 1;
    const uint32_t h = blockIdx.x, j0 = blockIdx.y * 32, grp = h / (d.heads / d.groups);
    const __nv_bfloat16 *k = (const __nv_bfloat16*)d.k + grp * d.dk, *v = (const __nv_bfloat16*)d.v + h * d.dv + j0;
    float* S = d.state + (size_t)h * d.dk * d.dv;
    const bool wide = rows_aligned(k, d.ldk, d.dk);
    // value rows: thread -> tokens tid / 4 (+ 64) of a step, columns 8 * (tid % 4) ..
    const uint32_t vt = tid >> 2, vc = (tid & 3) * 8;
    const bool vwide = rows_aligned(v, d.ldv, 8) && j0 + vc + 8 <= d.dv;
    uint4 vr[VP];
    auto load_v = [&](uint32_t s) {
#pragma unroll
        for (uint32_t i = 0; i < VP; i++) {
            const uint32_t t = s * STEP + vt + 64 * i;
            const __nv_bfloat16* p = v + (size_t)t * d.ldv + vc;
            if (t < T && vwide) {
                vr[i] = *reinterpret_cast<const uint4*>(p);
            } else {
                uint32_t w[4];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const float x = (t < T && j0 + vc + 2 * e < d.dv) ? __bfloat162float(p[2 * e]) : 0.f;
                    const float y = (t < T && j0 + vc + 2 * e + 1 < d.dv) ? __bfloat162float(p[2 * e + 1]) : 0.f;
                    w[e] = pack_bf2(x, y);
                }
                vr[i] = make_uint4(w[0], w[1], w[2], w[3]);
            }
        }
    };
    auto put_v = [&](uint32_t s) {         // weighted by what is left of it at the end of its chunk
        const float end = la[s / PER * kChunk + kChunk - 1];
#pragma unroll
        for (uint32_t i = 0; i < VP; i++) {
            const uint32_t t = s * STEP + vt + 64 * i;
            const float f = wt[t] * ex2(end - la[t]);
            const uint32_t w[4] = {vr[i].x, vr[i].y, vr[i].z, vr[i].w};
            uint32_t p[4];
#pragma unroll
            for (int e = 0; e < 4; e++) p[e] = pack_bf2(bf_lo(w[e]) * f, bf_hi(w[e]) * f);
            *reinterpret_cast<uint4*>(vS + (size_t)(s & 1) * STEP * LV + (vt + 64 * i) * LV + vc) = make_uint4(p[0], p[1], p[2], p[3]);
        }
    };
    auto stage_k = [&](uint32_t s, uint32_t buf) {
        if (s < ns) stage_rows<STEP, DK>(kS + buf * STEP * LK, k, d.ldk, d.dk, s * STEP, T, wide);
        cp_async_commit();
    };
    stage_k(0, 0);
    stage_k(1, 1);
    load_v(0);
    for (uint32_t c = warp; c < nc; c += 8) chunk_decays(d, h, c * kChunk, T, la + c * kChunk, wt + c * kChunk);
    float acc[NBW][2][4];                                             // blocks quarter, quarter + 4, ...: two tiles of 8 key rows
    auto each = [&](auto f) {
#pragma unroll
        for (uint32_t b = 0; b < NBW; b++)
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const uint32_t i = (quarter + 4 * b) * 16 + n * 8 + 2 * t4 + (e & 1), j = j0 + mt * 16 + g + 8 * (e >> 1);
                    f(acc[b][n][e], i < d.dk && j < d.dv, (size_t)i * d.dv + j);
                }
    };
    each([&](float& x, bool in, size_t at) { x = in && !fresh ? S[at] : 0.f; });
    __syncthreads();
    put_v(0);
    if (ns > 1) load_v(1);
    const uint32_t k_u = smem_u32(kS + (lane & 15) * LK + (lane >> 4) * 8) + quarter * 32;
    // V^T: tiles (tokens 0-7 | 8-15) x (columns 0-7 | 8-15), transposed
    const uint32_t v_u = smem_u32(vS + ((lane >> 4) * 8 + (lane & 7)) * LV + mt * 16 + ((lane >> 3) & 1) * 8);
    uint4* fr = states + state_fragments(0, d.heads, h, DK, dvp) + (size_t)(j0 / 16 + mt) * NB * 64 + quarter * 64 + lane;
    const size_t fr_step = state_fragments(1, d.heads, 0, DK, dvp);
    uint32_t buf = 0;
    for (uint32_t s = 0; s < ns; s++) {
        if (s % PER == 0) {
            // the state at the start of the chunk
            const float e = ex2(la[s / PER * kChunk + kChunk - 1]);
#pragma unroll
            for (uint32_t b = 0; b < NBW; b++) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int i = 0; i < 4; i++) {          // i: value column half (i >> 1), tile (i & 1)
                    float &x = acc[b][i & 1][(i >> 1) * 2], &y = acc[b][i & 1][(i >> 1) * 2 + 1];
                    hi[i] = pack_bf2(x, y);
                    lo[i] = pack_bf2(x - bf_lo(hi[i]), y - bf_hi(hi[i]));
                    x *= e;
                    y *= e;
                }
                fr[b * 4 * 64] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                fr[b * 4 * 64 + 32] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
            fr += fr_step;
        }
        cp_async_wait<1>();
        __syncthreads();          // step s has arrived for everyone, step s - 1 has been read by everyone
        stage_k(s + 2, buf == 0 ? 2 : buf - 1);
        const uint32_t kb_u = k_u + buf * STEP * LK * 2, vb_u = v_u + (s & 1) * STEP * LV * 2;
#pragma unroll
        for (uint32_t kk = 0; kk < STEP / 16; kk++) {
            uint32_t a[4];
            ldsm_x4_trans(a, vb_u + kk * 16 * LV * 2);
#pragma unroll
            for (uint32_t b = 0; b < NBW; b++) {
                uint32_t bk[4];
                ldsm_x4_trans(bk, kb_u + (kk * 16 * LK + b * 64) * 2);
                mma_bf16(acc[b][0], a, bk[0], bk[1]);
                mma_bf16(acc[b][1], a, bk[2], bk[3]);
            }
        }
        if (s + 1 < ns) put_v(s + 1);
        if (s + 2 < ns) load_v(s + 2);
        buf = buf == 2 ? 0 : buf + 1;
    }
    each([&](float& x, bool in, size_t at) { if (in) S[at] = x; });
}

// grid (chunks, heads, dvp / 64), 8 warps of 16 tokens.  DK >= dk: the rest is zero.
template <int DK>
__global__ void __launch_bounds__(256, DK <= 128 ? 2 : 1) chunk_out_kernel(const LinearRows d, const uint4* __restrict__ states, uint32_t dvp, uint32_t T) {
    extern __shared__ __align__(16) uint8_t smem[];
    constexpr uint32_t LV = 72, LK = DK + 8, NB = DK / 16;
    __nv_bfloat16* kS = reinterpret_cast<__nv_bfloat16*>(smem);       // [kChunk][LK]: first the queries, then the keys
    __nv_bfloat16* vS = kS + kChunk * LK;                             // [kChunk][LV]
    uint4* fS = reinterpret_cast<uint4*>(vS + kChunk * LV);           // [4 column blocks][NB][2][32]: the starting state
    __shared__ __align__(8) float la[kChunk], wt[kChunk];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const uint32_t c = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * 64, grp = h / (d.heads / d.groups), t0 = c * kChunk;
    const __nv_bfloat16 *q = (const __nv_bfloat16*)d.q + grp * d.dk, *k = (const __nv_bfloat16*)d.k + grp * d.dk,
                        *v = (const __nv_bfloat16*)d.v + h * d.dv + j0;
    const uint32_t nv = min(64u, d.dv - j0);
    stage_rows<kChunk, DK>(kS, q, d.ldq, d.dk, t0, T, rows_aligned(q, d.ldq, d.dk));
    cp_async_commit();
    {
        const uint4* fr = states + state_fragments(c, d.heads, h, DK, dvp) + (size_t)(j0 / 16) * NB * 64;
#pragma unroll
        for (uint32_t i = 0; i < NB; i++) cp_async16(smem_u32(fS + tid + i * 256), fr + tid + i * 256);
    }
    cp_async_commit();
    stage_rows<kChunk, 64>(vS, v, d.ldv, nv, t0, T, rows_aligned(v, d.ldv, nv));
    if (warp == 0) chunk_decays(d, h, t0, T, la, wt);
    cp_async_wait<1>();
    __syncthreads();
    // a scheduler's two warps: one with many earlier tokens in the chunk, one with few
    const uint32_t rblk = warp < 4 ? warp : 11 - warp;
    uint32_t qa[NB][4];
    {
        const uint32_t q_u = smem_u32(kS + (rblk * 16 + (lane & 15)) * LK + (lane >> 4) * 8);
#pragma unroll
        for (uint32_t ks = 0; ks < NB; ks++) ldsm_x4(qa[ks], q_u + ks * 32);
    }
    float o[8][4];
#pragma unroll
    for (int n = 0; n < 8; n++) { o[n][0] = 0.f; o[n][1] = 0.f; o[n][2] = 0.f; o[n][3] = 0.f; }
    __syncthreads();              // everyone has its queries
    stage_rows<kChunk, DK>(kS, k, d.ldk, d.dk, t0, T, rows_aligned(k, d.ldk, d.dk));
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const uint4* fr = fS + lane;
#pragma unroll
    for (uint32_t ks = 0; ks < NB; ks++) {
        uint4 hi[4], lo[4];
#pragma unroll
        for (int n = 0; n < 4; n++) {
            hi[n] = fr[(n * NB + ks) * 64];
            lo[n] = fr[(n * NB + ks) * 64 + 32];
        }
#pragma unroll
        for (int n = 0; n < 4; n++) {
            mma_bf16(o[2 * n], qa[ks], hi[n].x, hi[n].y);
            mma_bf16(o[2 * n + 1], qa[ks], hi[n].z, hi[n].w);
        }
#pragma unroll
        for (int n = 0; n < 4; n++) {
            mma_bf16(o[2 * n], qa[ks], lo[n].x, lo[n].y);
            mma_bf16(o[2 * n + 1], qa[ks], lo[n].z, lo[n].w);
        }
    }
    // The decay from an earlier token j to token i of this warp's block is cut at the block's first token r: r <- j is a factor
    // of column j, i <- r one of the whole row, which also the starting state's part (decayed up to r) takes.
    const uint32_t ra = rblk * 16 + g, rb = ra + 8;
    const float la_a = la[ra], la_b = la[rb], la_r = la[rblk * 16];
    {
        const float e = ex2(la_r);
#pragma unroll
        for (int n = 0; n < 8; n++) { o[n][0] *= e; o[n][1] *= e; o[n][2] *= e; o[n][3] *= e; }
    }
    cp_async_wait<0>();
    __syncthreads();
    // products within the chunk: 16 tokens at a time up to this warp's own
    const uint32_t k_u = smem_u32(kS + ((lane >> 4) * 8 + (lane & 7)) * LK + ((lane >> 3) & 1) * 8);
    const uint32_t v_u = smem_u32(vS + (lane & 15) * LV + (lane >> 4) * 8);
    auto scores = [&](uint32_t kk, float (&s0)[4], float (&s1)[4]) {
#pragma unroll
        for (int i = 0; i < 4; i++) s0[i] = s1[i] = 0.f;
        float u0[4] = {0.f, 0.f, 0.f, 0.f}, u1[4] = {0.f, 0.f, 0.f, 0.f};       // two chains of half the length
#pragma unroll
        for (uint32_t ks = 0; ks < NB; ks += 2) {
            uint32_t b[4], b2[4];
            ldsm_x4(b, k_u + (kk * 16 * LK + ks * 16) * 2);
            ldsm_x4(b2, k_u + (kk * 16 * LK + ks * 16 + 16) * 2);
            mma_bf16(s0, qa[ks], b[0], b[1]);
            mma_bf16(s1, qa[ks], b[2], b[3]);
            mma_bf16(u0, qa[ks + 1], b2[0], b2[1]);
            mma_bf16(u1, qa[ks + 1], b2[2], b2[3]);
        }
#pragma unroll
        for (int i = 0; i < 4; i++) { s0[i] += u0[i]; s1[i] += u1[i]; }
    };
    auto values = [&](uint32_t kk, const uint32_t (&p)[4]) {
#pragma unroll
        for (int n = 0; n < 8; n += 2) {
            uint32_t b[4];
            ldsm_x4_trans(b, v_u + (kk * 16 * LV + n * 8) * 2);
            mma_bf16(o[n], p, b[0], b[1]);
            mma_bf16(o[n + 1], p, b[2], b[3]);
        }
    };
    for (uint32_t kk = 0; kk < rblk; kk++) {
        float s0[4], s1[4];
        const uint32_t ja = kk * 16 + 2 * t4;
        const float2 l0 = *reinterpret_cast<const float2*>(la + ja), l1 = *reinterpret_cast<const float2*>(la + ja + 8);
        const float2 w0 = *reinterpret_cast<const float2*>(wt + ja), w1 = *reinterpret_cast<const float2*>(wt + ja + 8);
        const float f0 = w0.x * ex2(la_r - l0.x), f1 = w0.y * ex2(la_r - l0.y), f2 = w1.x * ex2(la_r - l1.x), f3 = w1.y * ex2(la_r - l1.y);
        scores(kk, s0, s1);
        const uint32_t p[4] = {pack_bf2(s0[0] * f0, s0[1] * f1), pack_bf2(s0[2] * f0, s0[3] * f1), pack_bf2(s1[0] * f2, s1[1] * f3),
                               pack_bf2(s1[2] * f2, s1[3] * f3)};
        values(kk, p);
    }
    {
        const float e_a = ex2(la_a - la_r), e_b = ex2(la_b - la_r);
#pragma unroll
        for (int n = 0; n < 8; n++) { o[n][0] *= e_a; o[n][1] *= e_a; o[n][2] *= e_b; o[n][3] *= e_b; }
        float s0[4], s1[4];
        scores(rblk, s0, s1);
        auto weigh = [&](float s, uint32_t i, float la_i, uint32_t j) { return j <= i ? s * wt[j] * ex2(la_i - la[j]) : 0.f; };
        const uint32_t ja = rblk * 16 + 2 * t4;
        const uint32_t p[4] = {pack_bf2(weigh(s0[0], ra, la_a, ja), weigh(s0[1], ra, la_a, ja + 1)),
                               pack_bf2(weigh(s0[2], rb, la_b, ja), weigh(s0[3], rb, la_b, ja + 1)),
                               pack_bf2(weigh(s1[0], ra, la_a, ja + 8), weigh(s1[1], ra, la_a, ja + 9)),
                               pack_bf2(weigh(s1[2], rb, la_b, ja + 8), weigh(s1[3], rb, la_b, ja + 9))};
        values(rblk, p);
    }
    const float skip = d.skip ? d.skip[h] : 0.f;
    const bool pairs = (d.dv & 1u) == 0 && (d.ldo & 1u) == 0;
    __nv_bfloat16* out = (__nv_bfloat16*)d.out + h * d.dv + j0;
#pragma unroll
    for (int n = 0; n < 8; n++) {
        const uint32_t j = n * 8 + 2 * t4;
        if (j >= nv) continue;
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const uint32_t r = half ? rb : ra;
            if (t0 + r >= T) continue;
            const float x = fmaf(skip, __bfloat162float(vS[r * LV + j]), o[n][2 * half]), y = fmaf(skip, __bfloat162float(vS[r * LV + j + 1]), o[n][2 * half + 1]);
            __nv_bfloat16* p = out + (size_t)(t0 + r) * d.ldo + j;
            if (pairs) {
                *reinterpret_cast<uint32_t*>(p) = pack_bf2(x, y);
            } else {
                p[0] = __float2bfloat16_rn(x);
                if (j + 1 < nv) p[1] = __float2bfloat16_rn(y);
            }
        }
    }
}

// ── gate and norm ──
// grid (T), 256 threads; the row's values (and their factors) pass through shared memory.
template <typename TA, bool BEFORE>
__global__ void __launch_bounds__(256) gated_norm_kernel(TA* __restrict__ a, uint32_t lda, uint32_t n, uint32_t group, const TA* __restrict__ gate,
                                                          uint32_t ldg, const float* __restrict__ weight, float out_scale, float eps) {
    extern __shared__ __align__(16) float sm[];
    float *v = sm, *fac = sm + n;
    TA* row = a + (size_t)blockIdx.x * lda;
    const TA* gr = gate + (size_t)blockIdx.x * ldg;
    for (uint32_t i = threadIdx.x; i < n; i += 256) {
        float x = to_f32(row[i]);
        if (BEFORE) x *= silu(to_f32(gr[i]));
        v[i] = x;
    }
    __syncthreads();
    const uint32_t groups = n / group, wpg = groups >= 8 ? 1u : (groups >= 3 ? 2u : (groups == 2 ? 4u : 8u));
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = warp % wpg;
    for (uint32_t g = warp / wpg; g < groups; g += 8 / wpg) {
        float sq = 0.f;
        for (uint32_t i = sub * 32 + lane; i < group; i += 32 * wpg) sq = fmaf(v[g * group + i], v[g * group + i], sq);
        sq = wsum(sq);
        if (lane == 0) fac[g * wpg + sub] = sq;
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < n; i += 256) {
        const uint32_t g = i / group;
        float sq = 0.f;
        for (uint32_t k = 0; k < wpg; k++) sq += fac[g * wpg + k];
        float x = v[i] * rsqrtf(sq / (float)group + eps);
        if (BEFORE) x *= weight[i];
        else x *= silu(to_f32(gr[i])) * out_scale;
        put(row + i, x);
    }
}

// The same for bf16 rows of 16-byte pieces: a thread keeps its (at most NC) pieces in registers, only their sums of squares pass
// through shared memory.
template <bool BEFORE, int NC>
__global__ void __launch_bounds__(256) gated_norm_vec_kernel(__nv_bfloat16* __restrict__ a, uint32_t lda, uint32_t n, uint32_t group,
                                                              const __nv_bfloat16* __restrict__ gate, uint32_t ldg, const float* __restrict__ weight,
                                                              float out_scale, float eps) {
    extern __shared__ __align__(16) float sm[];
    const uint32_t pieces = n / 8, per = group / 8, groups = n / group;
    float *sums = sm, *fac = sm + pieces;
    uint4* row = reinterpret_cast<uint4*>(a + (size_t)blockIdx.x * lda);
    const uint4* gr = reinterpret_cast<const uint4*>(gate + (size_t)blockIdx.x * ldg);
    uint4 av[NC], gv[NC];
#pragma unroll
    for (int c = 0; c < NC; c++) {
        const uint32_t i = threadIdx.x + 256 * c;
        if (i < pieces) {
            av[c] = row[i];
            gv[c] = gr[i];
        }
    }
    float v[NC][8];
#pragma unroll
    for (int c = 0; c < NC; c++) {
        const uint32_t i = threadIdx.x + 256 * c;
        if (i >= pieces) break;
        const uint32_t w[4] = {av[c].x, av[c].y, av[c].z, av[c].w}, z[4] = {gv[c].x, gv[c].y, gv[c].z, gv[c].w};
        float sq = 0.f;
#pragma unroll
        for (int e = 0; e < 8; e++) {
            v[c][e] = (e & 1) ? bf_hi(w[e / 2]) : bf_lo(w[e / 2]);
            if (BEFORE) v[c][e] *= silu_for<__nv_bfloat16>((e & 1) ? bf_hi(z[e / 2]) : bf_lo(z[e / 2]));
            sq = fmaf(v[c][e], v[c][e], sq);
        }
        sums[i] = sq;
    }
    __syncthreads();
    const uint32_t wpg = groups >= 8 ? 1u : (groups >= 3 ? 2u : (groups == 2 ? 4u : 8u));
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = warp % wpg;
    for (uint32_t g = warp / wpg; g < groups; g += 8 / wpg) {
        float sq = 0.f;
        for (uint32_t i = sub * 32 + lane; i < per; i += 32 * wpg) sq += sums[g * per + i];
        sq = wsum(sq);
        if (lane == 0) fac[g * wpg + sub] = sq;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < NC; c++) {
        const uint32_t i = threadIdx.x + 256 * c;
        if (i >= pieces) break;
        const uint32_t g = i / per, z[4] = {gv[c].x, gv[c].y, gv[c].z, gv[c].w};
        float sq = 0.f;
        for (uint32_t k = 0; k < wpg; k++) sq += fac[g * wpg + k];
        const float r = rsqrtf(sq / (float)group + eps);
        if (BEFORE) {
            const float4 w0 = *reinterpret_cast<const float4*>(weight + 8 * i), w1 = *reinterpret_cast<const float4*>(weight + 8 * i + 4);
            const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
            for (int e = 0; e < 8; e++) v[c][e] *= r * w[e];
        } else {
#pragma unroll
            for (int e = 0; e < 8; e++) v[c][e] *= r * silu_for<__nv_bfloat16>((e & 1) ? bf_hi(z[e / 2]) : bf_lo(z[e / 2])) * out_scale;
        }
        row[i] = make_uint4(pack_bf2(v[c][0], v[c][1]), pack_bf2(v[c][2], v[c][3]), pack_bf2(v[c][4], v[c][5]), pack_bf2(v[c][6], v[c][7]));
    }
}

template <typename K>
static int32_t allow_smem(runit_ctx* ctx, const char* name, K kern, size_t smem) {
    RUNIT_REQUIRE(ctx, smem <= (size_t)ctx->max_smem_optin - 2048, "%s: the layer's sizes do not fit shared memory", name);
    if (smem > 40 * 1024) RUNIT_CUDA_TRY(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return RUNIT_OK;
}

}  // namespace ls

using namespace ls;

int32_t ssm_step(runit_ctx* ctx, const Ssm& m, const float* proj, float* y, float* squares, const int32_t* pos_ptr) {
    RUNIT_REQUIRE(ctx, m.state <= kMaxKeyDim, "ssm_step: bad sizes");
    runit_launch_chain_smem(ctx, ssm_step_kernel, dim3(m.heads, (m.vdim + 31) / 32), dim3(256), (size_t)m.state * 8, m, proj, y, squares, pos_ptr);
    return runit_after_launch(ctx, "ssm_step");
}

int32_t ssm_conv_rows(runit_ctx* ctx, const Ssm& m, bool exact, const void* proj, uint32_t ld, void* xbc, uint32_t ld_out, float* dt, uint32_t T,
                      uint32_t start) {
    RUNIT_REQUIRE(ctx, m.taps >= 1 && m.taps <= kConvTok, "ssm_conv: %u taps (1 .. %u)", m.taps, kConvTok);
    const size_t es = exact ? 4 : 2;
    const bool wide = m.channels() % 4 == 0 && m.inner() % 4 == 0 && ld % 4 == 0 && ld_out % 4 == 0 && runit_aligned(proj, 4 * es) && runit_aligned(xbc, 4 * es);
    const uint32_t vec = wide ? 4 : 1, per = kConvThreads * vec;
    const dim3 grid((m.channels() + per - 1) / per + 1, (T + kConvTok - 1) / kConvTok);
    auto go = [&](auto kern, auto* p, auto* o) -> int32_t {
        kern<<<grid, kConvThreads, !exact && wide && m.taps == 4 ? kConvTok * kConvThreads * 8 : 0, ctx->stream>>>(m, p, ld, o, ld_out, dt, T, start);
        return runit_after_launch(ctx, "ssm_conv");
    };
#define RUNIT_CONV(TA, TAPS) (wide ? go(ssm_conv_kernel<TA, TAPS, 4>, (const TA*)proj, (TA*)xbc) : go(ssm_conv_kernel<TA, TAPS, 1>, (const TA*)proj, (TA*)xbc))
    if (exact) return m.taps == 4 ? RUNIT_CONV(float, 4) : RUNIT_CONV(float, 0);
    return m.taps == 4 ? RUNIT_CONV(__nv_bfloat16, 4) : RUNIT_CONV(__nv_bfloat16, 0);
#undef RUNIT_CONV
}

// key dimensions of the chunk kernels' variants
static uint32_t chunk_dk(uint32_t dk) { return dk <= 64 ? 64u : (dk <= 128 ? 128u : (dk <= 256 ? 256u : 0u)); }
size_t linear_chunk_bytes(uint32_t heads, uint32_t dk, uint32_t dv, uint32_t T) {
    return (size_t)((T + kChunk - 1) / kChunk) * heads * chunk_dk(dk) * pad64(dv) * 4;
}

int32_t linear_rows(runit_ctx* ctx, const LinearRows& d, bool exact, void* chunk_states, uint32_t T, uint32_t start) {
    RUNIT_REQUIRE(ctx, d.heads > 0 && d.groups > 0 && d.heads % d.groups == 0 && d.dk > 0 && d.dk <= kMaxKeyDim && d.dv > 0, "linear_rows: bad sizes");
    int32_t st;
    if (!exact && T >= 16 && chunk_states && chunk_dk(d.dk)) {
        const uint32_t dvp = pad64(d.dv), nc = (T + kChunk - 1) / kChunk;
        auto go = [&](auto state, auto out, size_t sa, uint32_t dkp) -> int32_t {
            const size_t sb = (size_t)kChunk * (dkp + 8 + 72) * 2 + (size_t)dkp * 64 * 4;
            if ((st = allow_smem(ctx, "chunk_state", state, sa)) != RUNIT_OK) return st;
            state<<<dim3(d.heads, dvp / 32), 256, sa, ctx->stream>>>(d, (uint4*)chunk_states, dvp, T, start == 0);
            if ((st = runit_after_launch(ctx, "chunk_state")) != RUNIT_OK) return st;
            if ((st = allow_smem(ctx, "chunk_out", out, sb)) != RUNIT_OK) return st;
            out<<<dim3(nc, d.heads, dvp / 64), 256, sb, ctx->stream>>>(d, (const uint4*)chunk_states, dvp, T);
            return runit_after_launch(ctx, "chunk_out");
        };
        switch (chunk_dk(d.dk)) {
            case 64: return go(chunk_state_kernel<64>, chunk_out_kernel<64>, StateCfg<64>::smem(nc), 64);
            case 128: return go(chunk_state_kernel<128>, chunk_out_kernel<128>, StateCfg<128>::smem(nc), 128);
            default: return go(chunk_state_kernel<256>, chunk_out_kernel<256>, StateCfg<256>::smem(nc), 256);
        }
    }
    const dim3 grid(d.heads, (d.dv + 31) / 32);
#define RUNIT_SCAN(NR)                                                                                            \
    do {                                                                                                          \
        if (exact) linear_scan_kernel<float, NR><<<grid, 256, 0, ctx->stream>>>(d, T, start == 0);                 \
        else linear_scan_kernel<__nv_bfloat16, NR><<<grid, 256, 0, ctx->stream>>>(d, T, start == 0);               \
    } while (0)
    if (d.dk <= 64) RUNIT_SCAN(8);
    else if (d.dk <= 128) RUNIT_SCAN(16);
    else if (d.dk <= 256) RUNIT_SCAN(32);
    else RUNIT_SCAN(128);
#undef RUNIT_SCAN
    return runit_after_launch(ctx, "linear_scan");
}

int32_t gated_norm_rows(runit_ctx* ctx, bool exact, void* a, uint32_t lda, uint32_t n, uint32_t group, const void* gate, uint32_t ldg, bool before,
                        const float* weight, float out_scale, float eps, uint32_t T) {
    RUNIT_REQUIRE(ctx, group > 0 && n % group == 0 && (!before || weight), "gated_norm: bad groups");
    const size_t smem = ((size_t)n + n / group + 8) * 4;
    int32_t st;
    auto go = [&](auto kern, auto* p, auto* g) -> int32_t {
        if ((st = allow_smem(ctx, "gated_norm", kern, smem)) != RUNIT_OK) return st;
        kern<<<T, 256, smem, ctx->stream>>>(p, lda, n, group, g, ldg, weight, out_scale, eps);
        return runit_after_launch(ctx, "gated_norm");
    };
    if (!exact && n <= 8192 && group % 8 == 0 && lda % 8 == 0 && ldg % 8 == 0 && runit_aligned(a, 16) && runit_aligned(gate, 16) && runit_aligned(weight, 16)) {
        const size_t small = ((size_t)n / 8 + n / group + 8) * 4;
        auto vec = [&](auto kern) -> int32_t {
            kern<<<T, 256, small, ctx->stream>>>((__nv_bfloat16*)a, lda, n, group, (const __nv_bfloat16*)gate, ldg, weight, out_scale, eps);
            return runit_after_launch(ctx, "gated_norm");
        };
        if (n <= 2048) return before ? vec(gated_norm_vec_kernel<true, 1>) : vec(gated_norm_vec_kernel<false, 1>);
        if (n <= 4096) return before ? vec(gated_norm_vec_kernel<true, 2>) : vec(gated_norm_vec_kernel<false, 2>);
        return before ? vec(gated_norm_vec_kernel<true, 4>) : vec(gated_norm_vec_kernel<false, 4>);
    }
    if (exact) return before ? go(gated_norm_kernel<float, true>, (float*)a, (const float*)gate) : go(gated_norm_kernel<float, false>, (float*)a, (const float*)gate);
    return before ? go(gated_norm_kernel<__nv_bfloat16, true>, (__nv_bfloat16*)a, (const __nv_bfloat16*)gate)
                  : go(gated_norm_kernel<__nv_bfloat16, false>, (__nv_bfloat16*)a, (const __nv_bfloat16*)gate);
}

}  // namespace runit

using namespace runit;

namespace {
int32_t ssm_of(runit_ctx* ctx, const char* who, const runit_ssm_cfg* c, Ssm* m) {
    RUNIT_REQUIRE(ctx, c && c->heads > 0 && c->vdim > 0 && c->state_dim > 0 && c->state_dim <= kMaxKeyDim && c->groups > 0 && c->heads % c->groups == 0 &&
                           c->taps > 0 && c->taps <= kConvTok && c->conv && c->conv_b && c->dt_bias && c->a && c->skip && c->state && c->ring,
                  "%s: bad state-space layer", who);
    m->heads = c->heads; m->vdim = c->vdim; m->state = c->state_dim; m->groups = c->groups; m->taps = c->taps;
    m->conv_w = (const float*)c->conv; m->conv_b = (const float*)c->conv_b; m->dt_bias = (const float*)c->dt_bias; m->a = (const float*)c->a;
    m->skip = (const float*)c->skip; m->s = (float*)c->state; m->ring = (float*)c->ring;
    return RUNIT_OK;
}
}  // namespace

extern "C" {

int32_t runit_ssm_step(runit_ctx_t* ctx, const runit_ssm_cfg* cfg, const void* proj, void* y, void* squares, const void* pos) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    Ssm m;
    int32_t st = ssm_of(ctx, "ssm_step", cfg, &m);
    if (st != RUNIT_OK) return st;
    RUNIT_REQUIRE(ctx, proj && y && squares && pos, "ssm_step: null argument");
    return ssm_step(ctx, m, (const float*)proj, (float*)y, (float*)squares, (const int32_t*)pos);
}

int32_t runit_ssm_conv_rows(runit_ctx_t* ctx, const runit_ssm_cfg* cfg, int32_t f32, const void* proj, uint32_t ld, void* xbc, uint32_t ldx, void* dt,
                            uint32_t T, uint32_t start) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    Ssm m;
    int32_t st = ssm_of(ctx, "ssm_conv_rows", cfg, &m);
    if (st != RUNIT_OK) return st;
    RUNIT_REQUIRE(ctx, proj && xbc && dt && T > 0 && ld >= m.inner() + m.channels() && ldx >= m.channels(), "ssm_conv_rows: bad argument");
    return ssm_conv_rows(ctx, m, f32 != 0, proj, ld, xbc, ldx, (float*)dt, T, start);
}

size_t runit_linear_scratch_bytes(uint32_t heads, uint32_t dk, uint32_t dv, uint32_t T) { return linear_chunk_bytes(heads, dk, dv, T); }

int32_t runit_linear_rows(runit_ctx_t* ctx, const runit_linear_cfg* c, int32_t f32, void* scratch, uint32_t T, uint32_t start) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, c && c->q && c->k && c->v && c->log_decay && (c->dt || c->decay) && c->state && c->out && T > 0 && c->groups > 0 &&
                           c->ldq >= c->groups * c->dk && c->ldk >= c->groups * c->dk && c->ldv >= c->heads * c->dv && c->ldo >= c->heads * c->dv &&
                           runit_aligned(scratch, 16), "linear_rows: bad argument");
    LinearRows d;
    d.heads = c->heads; d.groups = c->groups; d.dk = c->dk; d.dv = c->dv; d.q = c->q; d.k = c->k; d.v = c->v; d.ldq = c->ldq; d.ldk = c->ldk; d.ldv = c->ldv;
    d.dt = (const float*)c->dt; d.log_decay = (const float*)c->log_decay; d.decay = (const float*)c->decay; d.skip = (const float*)c->skip;
    d.state = (float*)c->state; d.out = c->out; d.ldo = c->ldo;
    return linear_rows(ctx, d, f32 != 0, scratch, T, start);
}

int32_t runit_gated_norm_rows(runit_ctx_t* ctx, int32_t f32, void* a, uint32_t lda, uint32_t n, uint32_t group, const void* gate, uint32_t ldg,
                              int32_t before, const void* weight, float out_scale, float eps, uint32_t T) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, a && gate && n > 0 && lda >= n && ldg >= n && T > 0, "gated_norm_rows: bad argument");
    return gated_norm_rows(ctx, f32 != 0, a, lda, n, group, gate, ldg, before != 0, (const float*)weight, out_scale, eps, T);
}

}  // extern "C"
