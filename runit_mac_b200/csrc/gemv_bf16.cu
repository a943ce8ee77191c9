// One-token operators of decoders with bf16 weights: GEMV with the norm in front and the activation behind fused in, and the
// row operators of a pass (embedding; norms with one gain for all coordinates, or with one per coordinate on a sublayer's output).
//
// A warp owns 1, 2 or 4 weight rows (rows 2i and 2i+1 together for a gated block) and keeps eight to sixteen 16-byte loads per
// lane in flight; the first group of them does not depend on the previous kernel of the chain and is requested before the dependency
// wait.  The input vector is staged in shared memory as f32; the norm's factor multiplies the dot product (the gain is one
// number), so the vector is read once.  Sums are f32.
#include "bf16_ops.cuh"
#include "model_core.h"
#include "tma.cuh"

namespace runit {
namespace gv {

constexpr int kWarps = 8;

__device__ __forceinline__ float bf_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf_hi(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }
// eight products of one 16-byte piece of a row with x (xa: elements 0..3, xb: 4..7)
__device__ __forceinline__ float dot8(const uint4& w, const float4& xa, const float4& xb, float acc) {
    acc = fmaf(bf_lo(w.x), xa.x, acc); acc = fmaf(bf_hi(w.x), xa.y, acc);
    acc = fmaf(bf_lo(w.y), xa.z, acc); acc = fmaf(bf_hi(w.y), xa.w, acc);
    acc = fmaf(bf_lo(w.z), xb.x, acc); acc = fmaf(bf_hi(w.z), xb.y, acc);
    acc = fmaf(bf_lo(w.w), xb.z, acc); acc = fmaf(bf_hi(w.w), xb.w, acc);
    return acc;
}
__device__ __forceinline__ float warp_add(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float silu_mul(float g, float u) { return g / (1.0f + expf(-g)) * u; }
__device__ __forceinline__ float relu2(float v) {
    v = fmaxf(v, 0.f);
    return v * v;
}

// x (K values) into shared memory as two planes of 16-byte pieces (elements 0..3 and 4..7 of every chunk of eight), zero
// padded; returns the sum of squares of this thread's elements.
__device__ __forceinline__ float stage_x(const float* x, uint32_t K, uint32_t nch, float4* xa, float4* xb) {
    float sq = 0.f;
    const bool vec = (K & 3u) == 0 && (reinterpret_cast<uintptr_t>(x) & 15u) == 0;
    for (uint32_t i = threadIdx.x; i < 2 * nch; i += kWarps * 32) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        const uint32_t e = 4 * i;
        if (vec) {
            if (e < K) v = *reinterpret_cast<const float4*>(x + e);
        } else {
            if (e < K) v.x = x[e];
            if (e + 1 < K) v.y = x[e + 1];
            if (e + 2 < K) v.z = x[e + 2];
            if (e + 3 < K) v.w = x[e + 3];
        }
        sq = fmaf(v.x, v.x, sq); sq = fmaf(v.y, v.y, sq); sq = fmaf(v.z, v.z, sq); sq = fmaf(v.w, v.w, sq);
        ((i & 1u) ? xb : xa)[i >> 1] = v;
    }
    return sq;
}

// sum over the CTA of up to two values at a time (kWarps warps); every thread gets it
__device__ __forceinline__ float cta_sum(float s, float* part) {
    s = warp_add(s);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = s;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int i = 0; i < kWarps; i++) tot += part[i];
    return tot;
}
__device__ __forceinline__ float4 load4(const float* p, uint32_t e, uint32_t n, bool vec) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (vec) {
        if (e < n) v = *reinterpret_cast<const float4*>(p + e);
    } else {
        if (e < n) v.x = p[e];
        if (e + 1 < n) v.y = p[e + 1];
        if (e + 2 < n) v.z = p[e + 2];
        if (e + 3 < n) v.w = p[e + 3];
    }
    return v;
}
__device__ __forceinline__ bool aligned4(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

// The prologues work on two pairs of planes, xa / xb and ya / yb (four neighbouring values each, see stage_x); a thread handles
// the same pieces in every pass.  stage_early runs before the dependency wait.
__device__ __forceinline__ float4 group_factors(const GemvPrologue& p, uint32_t e, uint32_t K, bool vec) {
    if (vec) return e >= p.plain ? load4(p.factor, e - p.plain, K - p.plain, true) : make_float4(1.f, 1.f, 1.f, 1.f);
    auto one = [&](uint32_t j) { return j < p.plain ? 1.f : (j < K ? p.factor[j - p.plain] : 0.f); };
    return make_float4(one(e), one(e + 1), one(e + 2), one(e + 3));
}
__device__ __forceinline__ bool pro_vec(const float* x, const GemvPrologue& p, uint32_t K) {
    return (K & 3u) == 0 && (p.plain & 3u) == 0 && aligned4(x) && aligned4(p.y) && aligned4(p.y_gain) && aligned4(p.gain) && aligned4(p.x_out) && aligned4(p.factor);
}
__device__ __forceinline__ void stage_early(const float* x, const GemvPrologue& p, uint32_t K, uint32_t nch, float4* xa, float4* xb, float4* ya,
                                             float4* yb) {
    const bool vec = pro_vec(x, p, K);
    if (p.kind == GEMV_PRO_RESIDUAL && p.y && p.early) {
        for (uint32_t i = threadIdx.x; i < 2 * nch; i += kWarps * 32) {
            const float4 xv = load4(x, 4 * i, K, vec), g = load4(p.y_gain, 4 * i, K, vec);
            ((i & 1u) ? xb : xa)[i >> 1] = xv;
            ((i & 1u) ? yb : ya)[i >> 1] = g;
        }
    } else if (p.kind == GEMV_PRO_GROUPS && p.factor_early) {
        for (uint32_t i = threadIdx.x; i < 2 * nch; i += kWarps * 32) ((i & 1u) ? yb : ya)[i >> 1] = group_factors(p, 4 * i, K, vec);
    }
}

// GEMV_PRO_RESIDUAL: returns the factor of the products (that of the second norm).
__device__ __forceinline__ float stage_residual(const float* x, const GemvPrologue& p, float eps, uint32_t K, uint32_t nch, float4* xa, float4* xb,
                                                 float4* ya, float4* yb, float* part) {
    const bool vec = pro_vec(x, p, K);
    float r = 0.f;
    if (p.y) {
        float sq = 0.f;
        for (uint32_t i = threadIdx.x; i < 2 * nch; i += kWarps * 32) {
            float4& gs = ((i & 1u) ? yb : ya)[i >> 1];
            float4 y = load4(p.y, 4 * i, K, vec), g;
            if (p.early) {
                g = gs;
            } else {
                g = load4(p.y_gain, 4 * i, K, vec);
                ((i & 1u) ? xb : xa)[i >> 1] = load4(x, 4 * i, K, vec);
            }
            sq = fmaf(y.x, y.x, sq); sq = fmaf(y.y, y.y, sq); sq = fmaf(y.z, y.z, sq); sq = fmaf(y.w, y.w, sq);
            y.x *= g.x; y.y *= g.y; y.z *= g.z; y.w *= g.w;
            gs = y;
        }
        r = rsqrtf(cta_sum(sq, part) / (float)K + eps);
    }
    float sq = 0.f;
    for (uint32_t i = threadIdx.x; i < 2 * nch; i += kWarps * 32) {
        float4& s = ((i & 1u) ? xb : xa)[i >> 1];
        float4 v;
        if (p.y) {
            const float4 y = ((i & 1u) ? yb : ya)[i >> 1];
            v = s;
            v.x = fmaf(y.x, r, v.x); v.y = fmaf(y.y, r, v.y); v.z = fmaf(y.z, r, v.z); v.w = fmaf(y.w, r, v.w);
            if (p.x_out && blockIdx.x == 0) {
                const uint32_t e = 4 * i;
                if (vec) {
                    if (e < K) *reinterpret_cast<float4*>(p.x_out + e) = v;
                } else {
                    if (e < K) p.x_out[e] = v.x;
                    if (e + 1 < K) p.x_out[e + 1] = v.y;
                    if (e + 2 < K) p.x_out[e + 2] = v.z;
                    if (e + 3 < K) p.x_out[e + 3] = v.w;
                }
            }
        } else {
            v = load4(x, 4 * i, K, vec);
        }
        if (p.gain) {
            sq = fmaf(v.x, v.x, sq); sq = fmaf(v.y, v.y, sq); sq = fmaf(v.z, v.z, sq); sq = fmaf(v.w, v.w, sq);
            const float4 g = load4(p.gain, 4 * i, K, vec);
            v.x *= g.x; v.y *= g.y; v.z *= g.z; v.w *= g.w;
        }
        s = v;
    }
    if (!p.gain) return 1.f;
    __syncthreads();           // part is rewritten
    return rsqrtf(cta_sum(sq, part) / (float)K + eps);
}

// GEMV_PRO_GROUPS: the sums of squares of the groups come from the launch that made x (squares), or are formed from the staged
// values.  fac: one word per group and warp of it.  Returns the factor of the products.
__device__ __forceinline__ float stage_groups(const float* x, const GemvPrologue& p, float eps, uint32_t K, uint32_t nch, float4* xa, float4* xb,
                                              float4* ya, float4* yb, float* fac) {
    const bool vec = pro_vec(x, p, K);
    const uint32_t groups = (K - p.plain) / p.group, wpg = groups >= 8 ? 1u : (groups >= 3 ? 2u : (groups == 2 ? 4u : 8u));
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = warp % wpg;
    for (uint32_t i = threadIdx.x; i < 2 * nch; i += kWarps * 32) {
        float4 v = load4(x, 4 * i, K, vec);
        if (p.squares) {
            const float4 f = p.factor_early ? ((i & 1u) ? yb : ya)[i >> 1] : group_factors(p, 4 * i, K, vec);
            v.x *= f.x; v.y *= f.y; v.z *= f.z; v.w *= f.w;
        } else if (!p.factor_early) {
            ((i & 1u) ? yb : ya)[i >> 1] = group_factors(p, 4 * i, K, vec);
        }
        ((i & 1u) ? xb : xa)[i >> 1] = v;
    }
    if (!p.squares) __syncthreads();
    auto at = [&](uint32_t e) -> float { return reinterpret_cast<const float*>(((e >> 2) & 1u) ? xb : xa)[(e >> 3) * 4 + (e & 3u)]; };
    for (uint32_t g = warp / wpg; g < groups; g += kWarps / wpg) {
        float sq = 0.f;
        if (p.squares) {
            for (uint32_t i = sub * 32 + lane; i < p.squares_n; i += 32 * wpg) sq += p.squares[(size_t)g * p.squares_n + i];
        } else {
            const uint32_t lo = p.plain + g * p.group;
            for (uint32_t i = sub * 32 + lane; i < p.group; i += 32 * wpg) {
                const float v = at(lo + i);
                sq = fmaf(v, v, sq);
            }
        }
        sq = warp_add(sq);
        if (lane == 0) fac[g * wpg + sub] = sq;
    }
    __syncthreads();
    auto group_factor = [&](uint32_t g) {
        float sq = 0.f;
        for (uint32_t i = 0; i < wpg; i++) sq += fac[g * wpg + i];
        return rsqrtf(sq / (float)p.group + eps);
    };
    if (p.squares && p.plain == 0 && groups == 1) return group_factor(0);
    const bool whole = (p.group & 3u) == 0 && (p.plain & 3u) == 0;       // four neighbours share a group
    for (uint32_t i = threadIdx.x; i < 2 * nch; i += kWarps * 32) {
        const uint32_t e = 4 * i;
        float4& v = ((i & 1u) ? xb : xa)[i >> 1];
        const float4 f = p.squares ? make_float4(1.f, 1.f, 1.f, 1.f) : ((i & 1u) ? yb : ya)[i >> 1];
        auto r = [&](uint32_t j) { return j < p.plain ? 1.f : (j < K ? group_factor((j - p.plain) / p.group) : 0.f); };
        if (whole) {
            const float s = r(e);
            v.x *= f.x * s; v.y *= f.y * s; v.z *= f.z * s; v.w *= f.w * s;
        } else {
            v.x *= f.x * r(e); v.y *= f.y * r(e + 1); v.z *= f.z * r(e + 2); v.w *= f.w * r(e + 3);
        }
    }
    return 1.f;
}

struct Args {
    const uint8_t* w;
    uint32_t rows, K, ldw;
    const float* x;
    const float* gain;
    float eps;
    float* out;
    const float* res;
    int32_t* argmax;
    unsigned long long* argmax_ctl;
    uint32_t n_routed, slot_stride;
    const int32_t* slot_expert;
    const float* pre;
    const uint8_t* w_extra;
    uint32_t rows_extra;
    const float* post_extra;
    GemvPrologue pro;
    float cap;
};

// RPU: rows of a warp's unit; U: 16-byte loads per lane, row and group
template <int EPI, int RPU, int U, bool SLOTS, bool PRO = false>
__global__ void __launch_bounds__(kWarps * 32, PRO && RPU * U <= 8 ? 4 : 1) gemv_bf16_kernel(const Args a) {
    extern __shared__ __align__(16) float4 smem4[];
    __shared__ float part[kWarps];
    __shared__ unsigned long long best_s[kWarps];
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t nch = (a.K + 7) / 8;
    float4 *xa = smem4, *xb = smem4 + nch;
    const uint32_t slot = SLOTS ? blockIdx.y : 0;
    const bool extra = SLOTS && slot == a.n_routed;
    const uint32_t rows = extra ? a.rows_extra : a.rows;
    const uint32_t units = (rows + RPU - 1) / RPU;
    const uint8_t* w = extra ? a.w_extra : a.w;
    const size_t row_bytes = (size_t)a.ldw * 2;
    uint32_t unit = blockIdx.x * kWarps + warp;
    uint4 v[RPU][U];
    auto load = [&](uint32_t u, uint32_t c0) {
#pragma unroll
        for (int r = 0; r < RPU; r++) {
            const uint8_t* row = w + (size_t)(u * RPU + r) * row_bytes;
#pragma unroll
            for (int i = 0; i < U; i++) {
                const uint32_t c = c0 + 32 * i + lane;
                v[r][i] = (c < nch && u * RPU + r < rows) ? __ldg(reinterpret_cast<const uint4*>(row) + c) : make_uint4(0, 0, 0, 0);
            }
        }
    };
    const bool early = !SLOTS || extra;
    if (early && unit < units) load(unit, 0);
    if constexpr (PRO) stage_early(a.x, a.pro, a.K, nch, xa, xb, xb + nch, xb + 2 * nch);
    grid_dependency_wait();
    grid_launch_dependents();
    float pre = 1.f, post = 1.f;
    if (SLOTS) {
        if (extra) {
            if (a.post_extra) post = *a.post_extra;
        } else {
            const int32_t e = a.slot_expert[slot];
            if (e < 0) return;
            w += (size_t)e * a.rows * row_bytes;
            if (a.pre) pre = a.pre[slot];
        }
    }
    if (!early && unit < units) load(unit, 0);
    float scale = 1.f;
    if constexpr (PRO) {
        float4 *ya = xb + nch, *yb = ya + nch;
        if (a.pro.kind == GEMV_PRO_RESIDUAL) scale = stage_residual(a.x, a.pro, a.eps, a.K, nch, xa, xb, ya, yb, part);
        else scale = stage_groups(a.x, a.pro, a.eps, a.K, nch, xa, xb, ya, yb, reinterpret_cast<float*>(yb + nch));
        __syncthreads();
    } else {
        scale = stage_x(a.x, a.K, nch, xa, xb);
        if (a.gain) {
            scale = warp_add(scale);
            if (lane == 0) part[warp] = scale;
        }
        __syncthreads();
        scale = 1.f;
        if (a.gain) {
            float tot = 0.f;
#pragma unroll
            for (int i = 0; i < kWarps; i++) tot += part[i];
            scale = rsqrtf(tot / (float)a.K + a.eps) * *a.gain;
        }
    }
    unsigned long long best = 0;
    bool first = true;
    for (; unit < units; unit += gridDim.x * kWarps) {
        float acc[RPU];
#pragma unroll
        for (int r = 0; r < RPU; r++) acc[r] = 0.f;
        for (uint32_t c0 = 0; c0 < nch; c0 += 32 * U) {
            if (!first) load(unit, c0);
            first = false;
#pragma unroll
            for (int i = 0; i < U; i++) {
                const uint32_t c = c0 + 32 * i + lane;
                if (c < nch) {
                    const float4 p = xa[c], q = xb[c];
#pragma unroll
                    for (int r = 0; r < RPU; r++) acc[r] = dot8(v[r][i], p, q, acc[r]);
                }
            }
        }
        if (PRO && unit + gridDim.x * kWarps < units) {       // the next unit's first loads go out before this one's sums
            load(unit + gridDim.x * kWarps, 0);
            first = true;
        }
#pragma unroll
        for (int r = 0; r < RPU; r++) acc[r] = warp_add(acc[r]) * scale;
        if (lane == 0) {
            float* out = a.out + (size_t)slot * a.slot_stride;
            if (EPI == EPI_SILU_GLU) {
#pragma unroll
                for (int r = 0; r + 1 < RPU; r += 2)
                    if (unit * RPU + r + 1 < rows) out[(unit * RPU + r) / 2] = silu_mul(acc[r] * pre, acc[r + 1] * pre) * post;
            } else {
#pragma unroll
                for (int r = 0; r < RPU; r++) {
                    const uint32_t row = unit * RPU + r;
                    if (row >= rows) continue;
                    float o;
                    if (EPI == EPI_RELU2) o = relu2(acc[r] * pre) * post;
                    else o = acc[r] + (a.res ? a.res[row] : 0.f);
                    if (EPI == EPI_F32 && a.cap != 0.f) o = a.cap * tanhf(o / a.cap);
                    out[row] = o;
                    if (EPI == EPI_F32 && a.argmax) {
                        uint32_t b = __float_as_uint(o);
                        b = (b & 0x80000000u) ? ~b : (b | 0x80000000u);
                        const unsigned long long key = ((unsigned long long)b << 32) | (0xFFFFFFFFu - row);
                        best = key > best ? key : best;
                    }
                }
            }
        }
    }
    if (EPI == EPI_F32 && a.argmax) {
        if (lane == 0) best_s[warp] = best;
        __syncthreads();
        if (threadIdx.x == 0) {
#pragma unroll
            for (int i = 1; i < kWarps; i++) best = best_s[i] > best ? best_s[i] : best;
            atomicMax(a.argmax_ctl, best);
            __threadfence();
            if (atomicAdd(a.argmax_ctl + 1, 1ull) == gridDim.x - 1) {
                const unsigned long long k = atomicExch(a.argmax_ctl, 0ull);
                a.argmax_ctl[1] = 0;
                *a.argmax = (int32_t)(0xFFFFFFFFu - (uint32_t)k);
            }
        }
    }
}

struct SumArgs {
    const uint8_t* w;
    uint32_t rows, K, ldw, n_routed, x_stride;
    const int32_t* slot_expert;
    const uint8_t* w_extra;
    uint32_t K_extra, ldw_extra;
    const float* x;
    const float* res;
    float* out;
};

// The inputs of all slots lie one after the other in shared memory, each padded to chunks of eight.  A warp walks steps of 32
// chunks of one slot after the other, U steps in flight, so the loads of small blocks overlap across slots.
template <int RPU, int U>
__global__ void __launch_bounds__(kWarps * 32) gemv_bf16_sum_kernel(const SumArgs a) {
    extern __shared__ __align__(16) float4 smem4[];
    __shared__ const uint8_t* base_s[33];
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t chs = (a.K + 7) / 8, routed = a.n_routed * chs, chx = a.w_extra ? (a.K_extra + 7) / 8 : 0, total = routed + chx;
    float4 *xa = smem4, *xb = smem4 + total;
    // The expert ids come from the launch before the one this depends on: that launch has waited for it, so they are final
    // and the first weights can be requested before the wait.
    if (threadIdx.x < a.n_routed) {
        const int32_t e = a.slot_expert ? a.slot_expert[threadIdx.x] : 0;
        base_s[threadIdx.x] = e < 0 ? nullptr : a.w + (size_t)e * a.rows * a.ldw * 2;
    }
    if (threadIdx.x == a.n_routed) base_s[threadIdx.x] = a.w_extra;
    __syncthreads();
    const uint32_t units = (a.rows + RPU - 1) / RPU;
    const uint32_t steps_s = (chs + 31) / 32, steps = a.n_routed * steps_s + (chx + 31) / 32;
    uint32_t unit = blockIdx.x * kWarps + warp;
    uint4 v[RPU][U];
    uint32_t slot = 0, k = 0;                     // position of the next step to load
    uint32_t fslot = 0, fk = 0;                   // and of the next step to multiply
    auto advance = [&](uint32_t& s, uint32_t& kk) {
        if (++kk == steps_s && s < a.n_routed) { kk = 0; s++; }
    };
    auto load = [&](uint32_t u, uint32_t s0) {
#pragma unroll
        for (int i = 0; i < U; i++) {
            const bool extra = slot == a.n_routed;
            const uint32_t c = k * 32 + lane, n = extra ? chx : chs, pitch = (extra ? a.ldw_extra : a.ldw) * 2;
            const uint8_t* p = (s0 + i < steps && c < n) ? base_s[slot] : nullptr;
#pragma unroll
            for (int r = 0; r < RPU; r++) {
                const uint32_t row = u * RPU + r;
                v[r][i] = (p && row < a.rows) ? __ldg(reinterpret_cast<const uint4*>(p + (size_t)row * pitch) + c) : make_uint4(0, 0, 0, 0);
            }
            advance(slot, k);
        }
    };
    if (unit < units) load(unit, 0);
    grid_dependency_wait();
    grid_launch_dependents();
    // inputs: four 16-byte pieces per thread in flight
    {
        const bool vec = (a.K & 3u) == 0 && (a.K_extra & 3u) == 0 && (a.x_stride & 3u) == 0 && (reinterpret_cast<uintptr_t>(a.x) & 15u) == 0;
        for (uint32_t i0 = threadIdx.x; i0 < 2 * total; i0 += 4 * kWarps * 32) {
            float4 t[4];
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const uint32_t i = i0 + j * kWarps * 32;
                t[j] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (i >= 2 * total) continue;
                const uint32_t s = i < 2 * routed ? i / (2 * chs) : a.n_routed, e = 4 * (i - s * 2 * chs), n = s == a.n_routed ? a.K_extra : a.K;
                const float* x = a.x + (size_t)s * a.x_stride + e;
                if (vec) {
                    if (e < n) t[j] = *reinterpret_cast<const float4*>(x);
                } else {
                    if (e < n) t[j].x = x[0];
                    if (e + 1 < n) t[j].y = x[1];
                    if (e + 2 < n) t[j].z = x[2];
                    if (e + 3 < n) t[j].w = x[3];
                }
            }
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const uint32_t i = i0 + j * kWarps * 32;
                if (i < 2 * total) ((i & 1u) ? xb : xa)[i >> 1] = t[j];
            }
        }
    }
    __syncthreads();
    bool first = true;
    for (; unit < units; unit += gridDim.x * kWarps) {
        float acc[RPU];
#pragma unroll
        for (int r = 0; r < RPU; r++) acc[r] = 0.f;
        if (!first) slot = k = 0;
        fslot = fk = 0;
        for (uint32_t s0 = 0; s0 < steps; s0 += U) {
            if (!first) load(unit, s0);
            first = false;
#pragma unroll
            for (int i = 0; i < U; i++) {
                const uint32_t c = fk * 32 + lane, n = fslot == a.n_routed ? chx : chs;
                if (s0 + i < steps && c < n) {
                    const float4 p = xa[fslot * chs + c], q = xb[fslot * chs + c];
#pragma unroll
                    for (int r = 0; r < RPU; r++) acc[r] = dot8(v[r][i], p, q, acc[r]);
                }
                advance(fslot, fk);
            }
        }
#pragma unroll
        for (int r = 0; r < RPU; r++) {
            acc[r] = warp_add(acc[r]);
            const uint32_t row = unit * RPU + r;
            if (lane == 0 && row < a.rows) a.out[row] = (a.res ? a.res[row] : 0.f) + acc[r];
        }
    }
}

// ── rows ──
// sum over the CTA (256 threads)
__device__ __forceinline__ float block_sum(float s) {
    __shared__ float part[8];
    s = warp_add(s);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = s;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) tot += part[i];
    return tot;
}

__global__ void __launch_bounds__(256) embed_norm_kernel(const __nv_bfloat16* __restrict__ emb, uint32_t ld, const int32_t* __restrict__ tokens,
                                                          const int32_t* state, const int32_t* __restrict__ forced, uint32_t n_forced,
                                                          uint32_t vocab, const float* __restrict__ gain, float eps, float* __restrict__ x,
                                                          uint32_t width, float scale) {
    grid_dependency_wait();
    grid_launch_dependents();
    const uint32_t t = blockIdx.x;
    const int32_t tok = tokens ? tokens[t] : model_step_token(state, forced, n_forced, vocab);
    const __nv_bfloat16* row = emb + (size_t)tok * ld;
    float r = scale;
    if (gain) {
        float s = 0.f;
        for (uint32_t i = threadIdx.x; i < width; i += 256) {
            const float v = __bfloat162float(row[i]);
            s = fmaf(v, v, s);
        }
        r = rsqrtf(block_sum(s) / (float)width + eps) * *gain;
    }
    for (uint32_t i = threadIdx.x; i < width; i += 256) x[(size_t)t * width + i] = __bfloat162float(row[i]) * r;
}

template <typename TY>
__global__ void __launch_bounds__(256) norm_rows_kernel(const float* __restrict__ x, const int32_t* __restrict__ row_index,
                                                         const float* __restrict__ gain, float eps, TY* __restrict__ y, uint32_t ldy,
                                                         float* __restrict__ y2, uint32_t width, const float* __restrict__ gate_row,
                                                         float* __restrict__ gate_out) {
    grid_dependency_wait();
    grid_launch_dependents();
    const uint32_t t = blockIdx.x;
    const float* row = x + (size_t)(row_index ? row_index[t] : (int32_t)t) * width;
    float s = 0.f;
    for (uint32_t i = threadIdx.x; i < width; i += 256) s = fmaf(row[i], row[i], s);
    const float r = rsqrtf(block_sum(s) / (float)width + eps) * *gain;
    for (uint32_t i = threadIdx.x; i < ldy; i += 256) {
        const float v = i < width ? row[i] * r : 0.f;
        if constexpr (sizeof(TY) == 2) y[(size_t)t * ldy + i] = __float2bfloat16_rn(v);
        else y[(size_t)t * ldy + i] = v;
        if (y2 && i < width) y2[(size_t)t * width + i] = v;
    }
    if (gate_row) {          // sigmoid of one product of the normed row (the gate of a block that runs for every token)
        float z = 0.f;
        for (uint32_t i = threadIdx.x; i < width; i += 256) z = fmaf(row[i] * r, gate_row[i], z);
        __syncthreads();     // block_sum's partial sums are rewritten
        z = block_sum(z);
        if (threadIdx.x == 0) gate_out[t] = 1.0f / (1.0f + expf(-z));
    }
}

// x += y / rms(y) * gain (y null: x as it is), and y_out = x in the operand type; T rows.  With out_gain the stored row is x
// divided by its own root mean square and multiplied by out_gain (a final norm), and x stays as it is.
template <typename TY>
__global__ void __launch_bounds__(256) add_norm_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ gain, float eps,
                                                        const int32_t* __restrict__ row_index, const float* __restrict__ out_gain,
                                                        TY* __restrict__ out, uint32_t ldo, uint32_t width) {
    grid_dependency_wait();
    grid_launch_dependents();
    const uint32_t t = blockIdx.x;
    float* xr = x + (size_t)(row_index ? row_index[t] : (int32_t)t) * width;
    float r = 0.f, q = 1.f;
    if (y) {
        const float* yr = y + (size_t)t * width;
        float s = 0.f;
        for (uint32_t i = threadIdx.x; i < width; i += 256) s = fmaf(yr[i], yr[i], s);
        r = rsqrtf(block_sum(s) / (float)width + eps);
        for (uint32_t i = threadIdx.x; i < width; i += 256) xr[i] = fmaf(yr[i] * gain[i], r, xr[i]);
    }
    if (out_gain) {
        float s = 0.f;
        for (uint32_t i = threadIdx.x; i < width; i += 256) s = fmaf(xr[i], xr[i], s);      // this thread's own elements
        __syncthreads();
        q = rsqrtf(block_sum(s) / (float)width + eps);
    }
    if (!out) return;
    for (uint32_t i = threadIdx.x; i < ldo; i += 256) {
        const float v = i < width ? (out_gain ? xr[i] * q * out_gain[i] : xr[i]) : 0.f;
        if constexpr (sizeof(TY) == 2) out[(size_t)t * ldo + i] = __float2bfloat16_rn(v);
        else out[(size_t)t * ldo + i] = v;
    }
}

template <int EPI, int RPU, int U, bool SLOTS, bool PRO = false>
static int32_t launch(runit_ctx* ctx, const char* name, const Args& a, uint32_t max_rows, uint32_t slots) {
    size_t smem = (size_t)((a.K + 7) / 8) * 32 * (PRO ? 2 : 1);
    if (PRO && a.pro.kind == GEMV_PRO_GROUPS) smem += ((size_t)(a.K - a.pro.plain) / a.pro.group + 8) * 4;
    RUNIT_REQUIRE(ctx, smem <= (size_t)ctx->max_smem_optin - 1024, "%s: %u columns do not fit shared memory", name, a.K);
    if (smem > 48 * 1024)
        RUNIT_CUDA_TRY(ctx, cudaFuncSetAttribute(gemv_bf16_kernel<EPI, RPU, U, SLOTS, PRO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    // every CTA forms the whole vector: with a prologue that reads several vectors, fewer and longer-lived ones
    const uint32_t units = (max_rows + RPU - 1) / RPU, want = (units + kWarps - 1) / kWarps, cap = (uint32_t)ctx->sm_count * (PRO ? (ctx->tune.gemv_pro_ctas > 0 ? ctx->tune.gemv_pro_ctas : (RPU * U <= 8 ? 4 : 2)) : 8);
    const uint32_t rounds = PRO ? (want + cap - 1) / cap : 1;
    runit_launch_chain_smem(ctx, gemv_bf16_kernel<EPI, RPU, U, SLOTS, PRO>, dim3(PRO ? (want + rounds - 1) / rounds : (want < cap ? want : cap), slots), dim3(kWarps * 32), smem, a);
    return runit_after_launch(ctx, name);
}

}  // namespace gv

int32_t gemv_bf16(runit_ctx* ctx, const char* name, const GemvDesc& d) {
    RUNIT_REQUIRE(ctx, d.w && d.x && d.out && d.rows > 0 && d.K > 0 && d.ldw % 8 == 0 && d.ldw >= d.K, "%s: bad argument", name);
    gv::Args a{(const uint8_t*)d.w, d.rows, d.K, d.ldw, d.x, d.gain, d.eps, d.out, d.res, d.argmax, d.argmax_ctl, d.n_routed, d.slot_stride,
               d.slot_expert, d.pre, (const uint8_t*)d.w_extra, d.rows_extra, d.post_extra, d.pro, d.cap};
    if (d.pro.kind != GEMV_PRO_NONE) {
        RUNIT_REQUIRE(ctx, !d.slot_expert && !d.gain && (d.epi == EPI_F32 || d.epi == EPI_RELU2 || d.epi == EPI_SILU_GLU),
                      "%s: a prologue goes with a plain product", name);
        RUNIT_REQUIRE(ctx, d.pro.kind != GEMV_PRO_GROUPS || (d.pro.group > 0 && d.pro.plain < d.K && (d.K - d.pro.plain) % d.pro.group == 0 && d.pro.factor),
                      "%s: bad groups", name);
        RUNIT_REQUIRE(ctx, d.pro.kind != GEMV_PRO_RESIDUAL || !d.pro.y || d.pro.y_gain, "%s: bad residual", name);
#define RUNIT_GVP(E, R, U) gv::launch<E, R, U, false, true>(ctx, name, a, d.rows, 1)
        if (d.epi == EPI_SILU_GLU) return d.K <= 512 ? RUNIT_GVP(EPI_SILU_GLU, 4, 2) : RUNIT_GVP(EPI_SILU_GLU, 2, 8);
        if (d.epi == EPI_RELU2) return d.K <= 512 ? RUNIT_GVP(EPI_RELU2, 4, 2) : (d.K <= 1024 ? RUNIT_GVP(EPI_RELU2, 2, 4) : RUNIT_GVP(EPI_RELU2, 1, 8));
        if (d.K <= 512) return RUNIT_GVP(EPI_F32, 4, 2);
        return d.K <= 1024 ? RUNIT_GVP(EPI_F32, 2, 4) : (d.K <= 2048 ? RUNIT_GVP(EPI_F32, 1, 8) : RUNIT_GVP(EPI_F32, 1, 16));
#undef RUNIT_GVP
    }
    const bool slots = d.slot_expert != nullptr;
    const uint32_t n_slots = slots ? d.n_routed + (d.w_extra ? 1 : 0) : 1;
    const uint32_t rows = slots && d.w_extra && d.rows_extra > d.rows ? d.rows_extra : d.rows;
    // small rows: several per warp, so that as many loads are in flight; several blocks: fewer, larger CTAs
#define RUNIT_GV(E, R, U) (slots ? gv::launch<E, R, U, true>(ctx, name, a, rows, n_slots) : gv::launch<E, R, U, false>(ctx, name, a, rows, n_slots))
    const bool mid = d.K > 512 && !(slots && d.K > 1024);
    if (d.epi == EPI_SILU_GLU) return d.K <= 512 ? RUNIT_GV(EPI_SILU_GLU, 4, 2) : (mid ? RUNIT_GV(EPI_SILU_GLU, 2, 4) : RUNIT_GV(EPI_SILU_GLU, 2, 8));
    if (d.epi == EPI_RELU2)
        return d.K <= 512 ? RUNIT_GV(EPI_RELU2, 4, 2) : (mid && d.K <= 1024 ? RUNIT_GV(EPI_RELU2, 2, 4) : (slots ? RUNIT_GV(EPI_RELU2, 2, 8) : RUNIT_GV(EPI_RELU2, 1, 8)));
    if (d.K <= 512) return RUNIT_GV(EPI_F32, 4, 2);
    if (d.K <= 1024) return RUNIT_GV(EPI_F32, 2, 4);
    return d.K <= 4096 ? RUNIT_GV(EPI_F32, 1, 8) : RUNIT_GV(EPI_F32, 1, 16);
#undef RUNIT_GV
}

int32_t gemv_bf16_sum(runit_ctx* ctx, const char* name, const GemvSumDesc& d) {
    RUNIT_REQUIRE(ctx, (d.w || d.n_routed == 0) && d.x && d.out && d.rows > 0 && d.n_routed <= 32 && (d.n_routed > 0 || d.w_extra),
                  "%s: bad argument", name);
    gv::SumArgs a{(const uint8_t*)d.w, d.rows, d.K, d.ldw, d.n_routed, d.x_stride, d.slot_expert, (const uint8_t*)d.w_extra, d.K_extra,
                  d.ldw_extra, d.x, d.res, d.out};
    const uint32_t total = d.n_routed * ((d.K + 7) / 8) + (d.w_extra ? (d.K_extra + 7) / 8 : 0);
    const size_t smem = (size_t)total * 32;
    RUNIT_REQUIRE(ctx, smem <= (size_t)ctx->max_smem_optin - 1024, "%s: the slots' inputs do not fit shared memory", name);
    auto go = [&](auto kern, uint32_t rpu) -> int32_t {
        if (smem > 48 * 1024) RUNIT_CUDA_TRY(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        const uint32_t units = (d.rows + rpu - 1) / rpu, want = (units + gv::kWarps - 1) / gv::kWarps, cap = (uint32_t)ctx->sm_count * 8;
        runit_launch_chain_smem(ctx, kern, dim3(want < cap ? want : cap), dim3(gv::kWarps * 32), smem, a);
        return runit_after_launch(ctx, name);
    };
    if (total > 128) return go(gv::gemv_bf16_sum_kernel<1, 12>, 1);
    return go(gv::gemv_bf16_sum_kernel<2, 4>, 2);
}

int32_t embed_norm_rows(runit_ctx* ctx, const void* embed, uint32_t ld, const int32_t* tokens, const int32_t* state, const int32_t* forced,
                        uint32_t n_forced, uint32_t vocab, const float* gain, float eps, float* x, uint32_t T, uint32_t width, float scale) {
    runit_launch_chain(ctx, gv::embed_norm_kernel, dim3(T), dim3(256), (const __nv_bfloat16*)embed, ld, tokens, state, forced, n_forced, vocab,
                       gain, eps, x, width, scale);
    return runit_after_launch(ctx, "embed_norm");
}

int32_t norm_rows(runit_ctx* ctx, const float* x, const int32_t* row_index, const float* gain, float eps, void* y, bool y_f32, uint32_t ldy,
                  float* y2, uint32_t T, uint32_t width, const float* gate_row, float* gate_out) {
    if (y_f32) runit_launch_chain(ctx, gv::norm_rows_kernel<float>, dim3(T), dim3(256), x, row_index, gain, eps, (float*)y, ldy, y2, width, gate_row, gate_out);
    else runit_launch_chain(ctx, gv::norm_rows_kernel<__nv_bfloat16>, dim3(T), dim3(256), x, row_index, gain, eps, (__nv_bfloat16*)y, ldy, y2, width,
                            gate_row, gate_out);
    return runit_after_launch(ctx, "norm_rows");
}

int32_t add_norm_rows(runit_ctx* ctx, float* x, const float* y, const float* gain, float eps, const int32_t* row_index, const float* out_gain,
                      void* out, bool out_f32, uint32_t ldo, uint32_t T, uint32_t width) {
    if (out_f32) runit_launch_chain(ctx, gv::add_norm_kernel<float>, dim3(T), dim3(256), x, y, gain, eps, row_index, out_gain, (float*)out, ldo, width);
    else runit_launch_chain(ctx, gv::add_norm_kernel<__nv_bfloat16>, dim3(T), dim3(256), x, y, gain, eps, row_index, out_gain, (__nv_bfloat16*)out, ldo,
                            width);
    return runit_after_launch(ctx, "add_norm_rows");
}

}  // namespace runit

using namespace runit;

extern "C" {

int32_t runit_gemv_bf16_f32(runit_ctx_t* ctx, const void* weight, const void* x, const void* gain, float eps, void* y, const void* residual,
                            uint32_t m, uint32_t k) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, weight && x && y && m > 0 && k > 0 && runit_aligned(weight, 16), "gemv_bf16_f32: bad argument");
    GemvDesc d;
    d.w = weight; d.rows = m; d.K = k; d.ldw = pad8(k); d.x = (const float*)x; d.gain = (const float*)gain; d.eps = eps; d.out = (float*)y;
    d.res = (const float*)residual;
    return gemv_bf16(ctx, "gemv_bf16_f32", d);
}

int32_t runit_norm_gain_rows(runit_ctx_t* ctx, const void* x, const void* gain, float eps, void* y, int32_t y_f32, uint32_t T, uint32_t width) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, x && gain && y && T > 0 && width > 0, "norm_gain_rows: bad argument");
    return norm_rows(ctx, (const float*)x, nullptr, (const float*)gain, eps, y, y_f32 != 0, pad8(width), nullptr, T, width);
}

int32_t runit_add_norm_rows(runit_ctx_t* ctx, void* x, const void* y, const void* gain, float eps, const void* out_gain, void* out, int32_t out_f32,
                            uint32_t T, uint32_t width) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, x && (!y || gain) && T > 0 && width > 0, "add_norm_rows: bad argument");
    return add_norm_rows(ctx, (float*)x, (const float*)y, (const float*)gain, eps, nullptr, (const float*)out_gain, out, out_f32 != 0, pad8(width), T, width);
}

int32_t runit_gemv_bf16_residual_f32(runit_ctx_t* ctx, const void* weight, const void* x, const void* y, const void* y_gain, const void* gain, void* x_out,
                                     void* out, float eps, float cap, int32_t relu2, uint32_t m, uint32_t k) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, weight && x && out && m > 0 && k > 0 && runit_aligned(weight, 16) && x_out != x, "gemv_bf16_residual_f32: bad argument");
    GemvDesc d;
    d.w = weight; d.rows = m; d.K = k; d.ldw = pad8(k); d.x = (const float*)x; d.eps = eps; d.out = (float*)out; d.cap = cap;
    d.epi = relu2 ? EPI_RELU2 : EPI_F32;
    d.pro.kind = GEMV_PRO_RESIDUAL; d.pro.y = (const float*)y; d.pro.y_gain = (const float*)y_gain; d.pro.gain = (const float*)gain;
    d.pro.x_out = (float*)x_out;
    return gemv_bf16(ctx, "gemv_bf16_residual_f32", d);
}

int32_t runit_gemv_bf16_groups_f32(runit_ctx_t* ctx, const void* weight, const void* x, const void* factor, const void* squares, uint32_t squares_n,
                                   void* out, float eps, uint32_t plain, uint32_t group, uint32_t m, uint32_t k) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(ctx, weight && x && out && m > 0 && k > 0 && runit_aligned(weight, 16), "gemv_bf16_groups_f32: bad argument");
    GemvDesc d;
    d.w = weight; d.rows = m; d.K = k; d.ldw = pad8(k); d.x = (const float*)x; d.eps = eps; d.out = (float*)out;
    d.pro.kind = GEMV_PRO_GROUPS; d.pro.plain = plain; d.pro.group = group; d.pro.factor = (const float*)factor;
    d.pro.squares = (const float*)squares; d.pro.squares_n = squares_n;
    return gemv_bf16(ctx, "gemv_bf16_groups_f32", d);
}

}  // extern "C"
