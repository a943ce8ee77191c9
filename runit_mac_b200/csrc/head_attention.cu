// Attention over cached keys and values per head: grouped queries, an optional sliding window, an optional distance bias,
// optionally queries and keys of unit root mean square.  And the layer that runs it side by side with a retention: one decode
// launch for both (heads_step_kernel), one pass over the projected rows of a portion (heads_rows_kernel).
//
// The cache of a layer is a ring of `cap` rows per key / value head: a window plus the longest portion, or the whole sequence
// without a window.  Scores, softmax, norms and angles are f32.
//   * attn_cta: any sizes, bf16 or f32 cache.  A CTA serves up to eight query heads of one key head for one token; keys in tiles
//     of 64, split over CTAs; the last CTA of a head block to finish merges the splits.  Decoding, short portions, 32-bit runs.
//   * window_prefill_kernel: long portions in bf16, 64 queries of a head per CTA, blocks of 64 keys, mma.sync (the arrangement of
//     latent_prefill_kernel); blocks outside of the window are not visited.
#include <cmath>

#include "bf16_ops.cuh"
#include "gemv_common.cuh"
#include "linear_state.cuh"
#include "tma.cuh"

namespace runit {
namespace ha {

using ls::put;
using ls::to_f32;

__device__ __forceinline__ float wsum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float wmax(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        v[2 * i] = __uint_as_float(w[i] << 16);
        v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void unpack8(const uint4& u, float (&v)[8]) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        v[2 * i] = __uint_as_float(w[i] << 16);
        v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
// element i of a small array in registers
__device__ __forceinline__ uint4 pick(const uint4 (&x)[4], uint32_t i) { return i == 0 ? x[0] : (i == 1 ? x[1] : (i == 2 ? x[2] : x[3])); }
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
// factor that makes a vector's root mean square one (a warp's lanes read it); 1 when the layer leaves q and k as they are
template <typename T>
__device__ __forceinline__ float unit_factor(const HeadAttn& a, const T* p) {
    if (!a.unit_qk) return 1.f;
    float s = 0.f;
    for (uint32_t i = threadIdx.x & 31; i < a.dim; i += 32) {
        const float v = to_f32(p[i]);
        s = fmaf(v, v, s);
    }
    return rsqrtf(wsum(s) / (float)a.dim + a.eps);
}
// one warp writes the cache row of key head g (padding zero); wide: bf16 rows whose heads start at multiples of 4 elements
template <typename TC, typename T>
__device__ __forceinline__ void write_row(const HeadAttn& a, const T* row, uint32_t g, uint32_t pos, bool wide = false) {
    const uint32_t lane = threadIdx.x & 31, slot = pos % a.cap;
    const T *k = row + a.heads * a.dim + g * a.dim, *v = row + (a.heads + a.kv_heads) * a.dim + g * a.vdim;
    TC* kd = reinterpret_cast<TC*>(a.kc) + ((size_t)g * a.cap + slot) * a.kd();
    TC* vd = reinterpret_cast<TC*>(a.vc) + ((size_t)g * a.cap + slot) * a.vd();
    if constexpr (sizeof(T) == 2 && sizeof(TC) == 2) {
        if (wide && a.kd() == a.dim && a.vd() == a.vdim && a.dim <= 256) {
            uint2 u[2];
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const uint32_t c = (lane + 32 * i) * 4;
                u[i] = c < a.dim ? *reinterpret_cast<const uint2*>(k + c) : make_uint2(0, 0);
                const float x[4] = {__uint_as_float(u[i].x << 16), __uint_as_float(u[i].x & 0xffff0000u), __uint_as_float(u[i].y << 16),
                                    __uint_as_float(u[i].y & 0xffff0000u)};
#pragma unroll
                for (int e = 0; e < 4; e++) s = fmaf(x[e], x[e], s);
            }
            for (uint32_t c = lane * 4; c < a.vdim; c += 128) *reinterpret_cast<uint2*>(vd + c) = *reinterpret_cast<const uint2*>(v + c);
            const float f = a.unit_qk ? rsqrtf(wsum(s) / (float)a.dim + a.eps) : 1.f;
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const uint32_t c = (lane + 32 * i) * 4;
                if (c >= a.dim) break;
                const __nv_bfloat162 p = __floats2bfloat162_rn(__uint_as_float(u[i].x << 16) * f, __uint_as_float(u[i].x & 0xffff0000u) * f);
                const __nv_bfloat162 q = __floats2bfloat162_rn(__uint_as_float(u[i].y << 16) * f, __uint_as_float(u[i].y & 0xffff0000u) * f);
                *reinterpret_cast<uint2*>(kd + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&p), *reinterpret_cast<const uint32_t*>(&q));
            }
            return;
        }
    }
    const float f = unit_factor(a, k);
    for (uint32_t i = lane; i < a.kd(); i += 32) put(kd + i, i < a.dim ? to_f32(k[i]) * f : 0.f);
    for (uint32_t i = lane; i < a.vd(); i += 32) put(vd + i, i < a.vdim ? to_f32(v[i]) : 0.f);
}

struct Parts {
    float *o, *ml;             // [T * heads][nsplit][vdim], [T * heads][nsplit][2] (maximum, sum)
    uint32_t* tickets;         // [T][kv_heads][head blocks]
    uint32_t nsplit;
};
constexpr int kTile = 64;
static size_t cta_smem(const HeadAttn& a, int RB) {
    const size_t nv = a.vd() / 8, ng = 256 / nv, red = ng * RB * a.vd(), wts = (size_t)RB * 64;
    return ((size_t)RB * a.kd() + RB * kTile + 4 * 8 + (red > wts ? red : wts)) * 4;
}

// Cached rows of a CTA's first tile, requested before its inputs are known: a thread's pieces of a key row and of the value rows
// it adds up (at most P of each).  bf16 caches only.
constexpr int kPre = 4;
struct FirstTile {
    uint4 k[kPre], v[kPre];
};

// RAW: the token's own key and value are still in the projected row; the CTA whose keys end with it writes the cache row.  With a
// bf16 cache the first tile is requested before the dependency wait (which this function then does).
template <typename TC, typename TQ, typename TO, int RB, bool RAW>
__device__ __forceinline__ void attn_cta(const HeadAttn& a, const TQ* row, TO* out, uint32_t pos, uint32_t g, uint32_t hb, uint32_t nhb,
                                          uint32_t split, uint32_t t, const Parts& pt, float* sm) {
    constexpr bool EARLY = RAW && sizeof(TC) == 2;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t rep = a.heads / a.kv_heads, h0 = g * rep + hb * RB, nr = min((uint32_t)RB, rep - hb * RB), kd = a.kd(), vd = a.vd();
    __shared__ uint32_t last_s;
    __shared__ float slope_s[8];
    float* qs = sm;
    float* ss = qs + RB * kd;
    float *ms = ss + RB * kTile, *lsum = ms + 8, *fs = lsum + 8;
    float* red = fs + 16;
    const uint32_t lo = a.window && pos + 1 > a.window ? pos + 1 - a.window : 0, len = pos + 1 - lo;
    const uint32_t chunk = max(16u, ((len + pt.nsplit - 1) / pt.nsplit + 15) / 16 * 16);
    const uint32_t beg = lo + min(len, split * chunk), end = min(lo + len, beg + chunk);
    const TC* kc = reinterpret_cast<const TC*>(a.kc) + (size_t)g * a.cap * kd;
    const TC* vc = reinterpret_cast<const TC*>(a.vc) + (size_t)g * a.cap * vd;
    const uint32_t nv = vd / 8, ng = 256 / nv, cv = tid % nv, gp = tid / nv;
    const uint32_t fkey = beg + (tid >> 2);
    FirstTile ft;
    if constexpr (EARLY) {
#pragma unroll
        for (int i = 0; i < kPre; i++) {
            const uint32_t ch = (tid & 3) + 4 * i, kk = gp + ng * i;
            if (fkey < end && fkey != pos && ch < kd / 8) ft.k[i] = *reinterpret_cast<const uint4*>(kc + (size_t)(fkey % a.cap) * kd + ch * 8);
            if (gp < ng && kk < (uint32_t)kTile && beg + kk < end && beg + kk != pos)
                ft.v[i] = *reinterpret_cast<const uint4*>(vc + (size_t)((beg + kk) % a.cap) * vd + cv * 8);
        }
    }
    if (tid < nr) slope_s[tid] = a.slopes ? a.slopes[h0 + tid] : 0.f;
    if constexpr (RAW) {
        grid_dependency_wait();
        grid_launch_dependents();
    }
    for (uint32_t r = warp; r < RB; r += 8) {
        if (r < nr) {
            const TQ* q = row + (size_t)(h0 + r) * a.dim;
            const float f = unit_factor(a, q) * a.scale;
            for (uint32_t i = lane; i < kd; i += 32) qs[r * kd + i] = i < a.dim ? to_f32(q[i]) * f : 0.f;
        } else {
            for (uint32_t i = lane; i < kd; i += 32) qs[r * kd + i] = 0.f;
        }
        if (lane == 0) {
            ms[r] = -INFINITY;
            lsum[r] = 0.f;
        }
    }
    if (RAW && beg < end && end == pos + 1 && warp == 7) write_row<TC>(a, row, g, pos);
    __syncthreads();
    float acc[RB][8];
#pragma unroll
    for (int r = 0; r < RB; r++)
#pragma unroll
        for (int i = 0; i < 8; i++) acc[r][i] = 0.f;
    for (uint32_t k0 = beg; k0 < end; k0 += kTile) {
        {
            const uint32_t key = k0 + (tid >> 2), c = tid & 3;
            float s[RB];
#pragma unroll
            for (int r = 0; r < RB; r++) s[r] = 0.f;
            if (key < end) {
                const TC* kr = kc + (size_t)(key % a.cap) * kd;
                const bool have = EARLY && k0 == beg && key != pos;      // the pieces requested early
#pragma unroll 4
                for (uint32_t i = 0; 4 * i + c < kd / 8; i++) {
                    const uint32_t ch = 4 * i + c;
                    float kv[8];
                    if (EARLY && have && i < kPre) unpack8(pick(ft.k, i), kv);
                    else load8(kr + ch * 8, kv);
#pragma unroll
                    for (int r = 0; r < RB; r++) {
                        const float4 x = *reinterpret_cast<const float4*>(qs + r * kd + ch * 8), y = *reinterpret_cast<const float4*>(qs + r * kd + ch * 8 + 4);
                        s[r] = fmaf(kv[0], x.x, s[r]); s[r] = fmaf(kv[1], x.y, s[r]); s[r] = fmaf(kv[2], x.z, s[r]); s[r] = fmaf(kv[3], x.w, s[r]);
                        s[r] = fmaf(kv[4], y.x, s[r]); s[r] = fmaf(kv[5], y.y, s[r]); s[r] = fmaf(kv[6], y.z, s[r]); s[r] = fmaf(kv[7], y.w, s[r]);
                    }
                }
            }
#pragma unroll
            for (int r = 0; r < RB; r++) {
                s[r] += __shfl_xor_sync(0xffffffffu, s[r], 1);
                s[r] += __shfl_xor_sync(0xffffffffu, s[r], 2);
                if (c == (uint32_t)(r & 3) && (uint32_t)r < nr) {
                    ss[r * kTile + (tid >> 2)] = key < end ? s[r] - slope_s[r] * (float)(pos - key) : -INFINITY;
                }
            }
        }
        __syncthreads();
        for (uint32_t r = warp; r < nr; r += 8) {
            const float s0 = ss[r * kTile + lane], s1 = ss[r * kTile + 32 + lane], m = ms[r];
            const float n = fmaxf(m, wmax(fmaxf(s0, s1)));          // the tile's first key is visible: finite
            const float p0 = expf(s0 - n), p1 = expf(s1 - n), f = expf(m - n), l = wsum(p0 + p1);
            ss[r * kTile + lane] = p0;
            ss[r * kTile + 32 + lane] = p1;
            __syncwarp();
            if (lane == 0) {
                ms[r] = n;
                lsum[r] = lsum[r] * f + l;
                fs[r] = f;
            }
        }
        __syncthreads();
        if (gp < ng) {
#pragma unroll
            for (int r = 0; r < RB; r++) {
                const float f = (uint32_t)r < nr ? fs[r] : 0.f;
#pragma unroll
                for (int i = 0; i < 8; i++) acc[r][i] *= f;
            }
            const uint32_t n = min((uint32_t)kTile, end - k0);
#pragma unroll 4
            for (uint32_t i = 0; gp + ng * i < n; i++) {
                const uint32_t kk = gp + ng * i;
                float v[8];
                if (EARLY && k0 == beg && i < kPre && k0 + kk != pos) unpack8(pick(ft.v, i), v);
                else load8(vc + (size_t)((k0 + kk) % a.cap) * vd + cv * 8, v);
#pragma unroll
                for (int r = 0; r < RB; r++) {
                    const float p = (uint32_t)r < nr ? ss[r * kTile + kk] : 0.f;
#pragma unroll
                    for (int i = 0; i < 8; i++) acc[r][i] = fmaf(p, v[i], acc[r][i]);
                }
            }
        }
        __syncthreads();
    }
    if (gp < ng)
#pragma unroll
        for (int r = 0; r < RB; r++)
#pragma unroll
            for (int i = 0; i < 8; i++) red[((size_t)gp * RB + r) * vd + cv * 8 + i] = acc[r][i];
    __syncthreads();
    const bool whole = pt.nsplit == 1;
    for (uint32_t i = tid; i < nr * a.vdim; i += 256) {
        const uint32_t r = i / a.vdim, j = i - r * a.vdim;
        float s = 0.f;
        for (uint32_t k = 0; k < ng; k++) s += red[((size_t)k * RB + r) * vd + j];
        if (whole) put(out + (size_t)(h0 + r) * a.vdim + j, s / lsum[r] * a.out_scale);
        else pt.o[(((size_t)t * a.heads + h0 + r) * pt.nsplit + split) * a.vdim + j] = s;
    }
    if (whole) return;
    if (tid < nr) {
        float* p = pt.ml + (((size_t)t * a.heads + h0 + tid) * pt.nsplit + split) * 2;
        p[0] = ms[tid];
        p[1] = lsum[tid];
    }
    __threadfence();
    __syncthreads();
    uint32_t* ticket = pt.tickets + ((size_t)t * a.kv_heads + g) * nhb + hb;
    if (tid == 0) {
        const uint32_t n = atomicAdd(ticket, 1u);
        last_s = n == pt.nsplit - 1;
        if (n == pt.nsplit - 1) *ticket = 0;
    }
    __syncthreads();
    if (!last_s) return;
    __threadfence();
    float* wt = red;                    // [nr][64]: weight of every split (0 for one without keys)
    for (uint32_t r = warp; r < nr; r += 8) {
        const float* p = pt.ml + ((size_t)t * a.heads + h0 + r) * pt.nsplit * 2;
        const float m0 = lane < pt.nsplit ? __ldcg(p + 2 * lane) : -INFINITY, m1 = lane + 32 < pt.nsplit ? __ldcg(p + 2 * (lane + 32)) : -INFINITY;
        const float l0 = lane < pt.nsplit ? __ldcg(p + 2 * lane + 1) : 0.f, l1 = lane + 32 < pt.nsplit ? __ldcg(p + 2 * (lane + 32) + 1) : 0.f;
        const float M = wmax(fmaxf(m0, m1)), w0 = expf(m0 - M), w1 = expf(m1 - M), L = wsum(w0 * l0 + w1 * l1);
        wt[r * 64 + lane] = w0 / L;
        wt[r * 64 + 32 + lane] = w1 / L;
    }
    __syncthreads();
    const uint32_t live = min(pt.nsplit, (len + chunk - 1) / chunk);      // the splits with keys are the first ones
    for (uint32_t i = tid; i < nr * a.vdim; i += 256) {
        const uint32_t r = i / a.vdim, j = i - r * a.vdim;
        const float* p = pt.o + ((size_t)t * a.heads + h0 + r) * pt.nsplit * a.vdim + j;
        float s = 0.f;
#pragma unroll 8
        for (uint32_t k = 0; k < live; k++) s = fmaf(wt[r * 64 + k], __ldcg(p + (size_t)k * a.vdim), s);
        put(out + (size_t)(h0 + r) * a.vdim + j, s * a.out_scale);
    }
}

// One retention step for columns 32 * jb .. of head h; row: [q | k | v | g] of all heads.
__device__ __forceinline__ void retention_cta(const Retention& r, const float* row, float* out, float* factor, float* squares, uint32_t h, uint32_t jb,
                                               const int32_t* pos_ptr, float* sm) {
    __shared__ float red[8][33];
    const uint32_t tid = threadIdx.x, lane = tid & 31, j = jb * 32 + lane, half = r.rot_dims / 2;
    float *qs = sm, *ks = sm + r.dim;
    float* S = r.state + (size_t)h * r.dim * r.vdim;
    ls::StateRows st;
    ls::load_rows(st, S, r.dim, r.vdim, j, 0);       // the state is that of the last step: final long before this launch
    const float decay = r.decay[h];
    grid_dependency_wait();
    grid_launch_dependents();
    const uint32_t pos = (uint32_t)*pos_ptr;
    const float *q = row + (size_t)h * r.dim, *k = q + (size_t)r.heads * r.dim;
    for (uint32_t i = tid; i < r.dim; i += 256) {
        float qv = q[i], kv = k[i];
        if (i < r.rot_dims) {
            const bool second = i >= half;
            const uint32_t p = second ? i - half : i + half;
            float s, c;
            const uint32_t f = second ? p : i;
            ls::sincos_at(pos, r.freq[f], r.freq[half + f], &s, &c);
            const float qo = q[p], ko = k[p];
            qv = second ? fmaf(qv, c, qo * s) : fmaf(qv, c, -(qo * s));
            kv = second ? fmaf(kv, c, ko * s) : fmaf(kv, c, -(ko * s));
        }
        qs[i] = qv;
        ks[i] = kv * r.k_scale;
    }
    const size_t at = (size_t)h * r.vdim + j;
    const float* vrow = row + (size_t)2 * r.heads * r.dim;
    const float v = j < r.vdim ? vrow[at] : 0.f;
    __syncthreads();
    const float o = ls::state_step(st, S, r.dim, r.vdim, j, qs, ks, v, decay, pos == 0, red);
    if (tid >= 32) return;
    if (j < r.vdim) {
        out[at] = o;
        factor[at] = ls::silu(vrow[(size_t)r.heads * r.vdim + at]) * r.out_scale;
    }
    const float sq = wsum(j < r.vdim ? o * o : 0.f);
    if (tid == 0) squares[h * ((r.vdim + 31) / 32) + jb] = sq;
}

// grid: attention CTAs (kv_heads x head blocks x splits), then retention CTAs (heads x 32-column slices)
template <typename TC, int RB>
__global__ void __launch_bounds__(256) heads_step_kernel(const HeadAttn a, const Retention r, const float* proj, float* ao, float* factor, float* squares, const Parts pt,
                                                          uint32_t n_attn, uint32_t nhb, const int32_t* pos_ptr) {
    extern __shared__ __align__(16) float sm[];
    if (blockIdx.x >= n_attn) {
        const uint32_t i = blockIdx.x - n_attn, nj = (r.vdim + 31) / 32;
        retention_cta(r, proj + (n_attn ? a.in_rows() : 0), ao + (n_attn ? a.out_rows() : 0), factor, squares, i / nj, i % nj, pos_ptr, sm);
        return;
    }
    const uint32_t split = blockIdx.x % pt.nsplit, b = blockIdx.x / pt.nsplit;
    attn_cta<TC, float, float, RB, true>(a, proj, ao, (uint32_t)*pos_ptr, b / nhb, b % nhb, nhb, split, 0, pt, sm);
}

// T tokens whose cache rows are written: grid (kv_heads x head blocks x splits, T)
template <typename TC, int RB>
__global__ void __launch_bounds__(256) attn_rows_kernel(const HeadAttn a, const TC* proj, uint32_t ld, TC* out, uint32_t ldo, const Parts pt, uint32_t nhb,
                                                         uint32_t start) {
    extern __shared__ __align__(16) float sm[];
    const uint32_t split = blockIdx.x % pt.nsplit, b = blockIdx.x / pt.nsplit, t = blockIdx.y;
    attn_cta<TC, TC, TC, RB, false>(a, proj + (size_t)t * ld, out + (size_t)t * ldo, start + t, b / nhb, b % nhb, nhb, split, t, pt, sm);
}

// Projected rows of a portion: cache rows, and the retention's rotated q and k in place.  grid (T), 8 warps; warp items: key
// heads, then q and k of every retention head.
template <typename TC>
__global__ void __launch_bounds__(256) heads_rows_kernel(const HeadAttn a, const Retention r, TC* proj, uint32_t ld, uint32_t start) {
    extern __shared__ __align__(16) float sm[];
    float2* cs = reinterpret_cast<float2*>(sm);
    const uint32_t t = blockIdx.x, pos = start + t, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = r.rot_dims / 2;
    TC* row = proj + (size_t)t * ld;
    for (uint32_t i = threadIdx.x; i < (r.heads ? half : 0); i += 256) ls::sincos_at(pos, r.freq[i], r.freq[half + i], &cs[i].y, &cs[i].x);
    __syncthreads();
    const bool wide = (ld & 3u) == 0 && (a.dim & 3u) == 0 && (a.vdim & 3u) == 0 && (reinterpret_cast<uintptr_t>(proj) & 7u) == 0;
    const bool pairs = sizeof(TC) == 2 && (ld & 1u) == 0 && (r.dim & 1u) == 0 && (half & 1u) == 0 && (a.in_rows() & 1u) == 0 &&
                       (reinterpret_cast<uintptr_t>(proj) & 3u) == 0;
    for (uint32_t item = warp; item < a.kv_heads + 2 * r.heads; item += 8) {
        if (item < a.kv_heads) {
            write_row<TC>(a, row, item, pos, wide);
            continue;
        }
        const uint32_t i0 = item - a.kv_heads;
        TC* p = row + (a.heads ? a.in_rows() : 0) + (size_t)i0 * r.dim;          // q of all heads, then k of all heads
        const float f = i0 < r.heads ? 1.f : r.k_scale;
        if constexpr (sizeof(TC) == 2) {
            for (uint32_t i = 2 * lane; i < (pairs ? half : 0); i += 64) {
                __nv_bfloat162 *pu = reinterpret_cast<__nv_bfloat162*>(p + i), *pv = reinterpret_cast<__nv_bfloat162*>(p + i + half);
                const float2 u = __bfloat1622float2(*pu), v = __bfloat1622float2(*pv), a0 = cs[i], a1 = cs[i + 1];
                *pu = __floats2bfloat162_rn(fmaf(u.x, a0.x, -(v.x * a0.y)) * f, fmaf(u.y, a1.x, -(v.y * a1.y)) * f);
                *pv = __floats2bfloat162_rn(fmaf(v.x, a0.x, u.x * a0.y) * f, fmaf(v.y, a1.x, u.y * a1.y) * f);
            }
        }
        for (uint32_t i = pairs ? half : lane; i < half; i += 32) {
            const float u = to_f32(p[i]), v = to_f32(p[i + half]), c = cs[i].x, s = cs[i].y;
            put(p + i, fmaf(u, c, -(v * s)) * f);
            put(p + i + half, fmaf(v, c, u * s) * f);
        }
        if (i0 >= r.heads)
            for (uint32_t i = r.rot_dims + lane; i < r.dim; i += 32) put(p + i, to_f32(p[i]) * f);
    }
}

// ── prompts ──
__device__ __forceinline__ uint32_t pack_bf2(float a, float b) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&h);
}
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

// grid (heads, ceil(T / 64)), 4 warps of 16 queries.  QK >= dim, VD >= vdim: the rest is zero.
template <int QK, int VD>
__global__ void __launch_bounds__(128) window_prefill_kernel(const HeadAttn a, const __nv_bfloat16* __restrict__ proj, uint32_t ld,
                                                              __nv_bfloat16* __restrict__ out, uint32_t ldo, uint32_t T, uint32_t start) {
    constexpr int LK = QK + 8, LV = VD + 8, KS = QK / 16, ND = VD / 8;
    extern __shared__ __align__(16) uint8_t smem[];
    __nv_bfloat16* const Ks = reinterpret_cast<__nv_bfloat16*>(smem);     // [2][64 * LK]
    __nv_bfloat16* const Vs = Ks + 2 * 64 * LK;                           // [2][64 * LV]
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const uint32_t head = blockIdx.x, kvh = head / (a.heads / a.kv_heads), q0 = (gridDim.y - 1 - blockIdx.y) * 64, kd = a.kd(), vd = a.vd();
    const uint32_t row_a = q0 + warp * 16 + g, row_b = row_a + 8;
    const __nv_bfloat16* kc = reinterpret_cast<const __nv_bfloat16*>(a.kc) + (size_t)kvh * a.cap * kd;
    const __nv_bfloat16* vc = reinterpret_cast<const __nv_bfloat16*>(a.vc) + (size_t)kvh * a.cap * vd;
    const bool pairs = (a.dim & 1u) == 0 && (ld & 1u) == 0;
    auto ldq2 = [&](uint32_t row, uint32_t c) -> float2 {
        float2 v = make_float2(0.f, 0.f);
        if (row >= T || c >= a.dim) return v;
        const __nv_bfloat16* p = proj + (size_t)row * ld + head * a.dim + c;
        if (pairs) return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
        v.x = __bfloat162float(p[0]);
        if (c + 1 < a.dim) v.y = __bfloat162float(p[1]);
        return v;
    };
    uint32_t qa[KS][4];
    {
        float f_a = 1.f, f_b = 1.f;
        if (a.unit_qk) {
            float s_a = 0.f, s_b = 0.f;
#pragma unroll
            for (int ks = 0; ks < 2 * KS; ks++) {
                const float2 x = ldq2(row_a, ks * 8 + 2 * t), y = ldq2(row_b, ks * 8 + 2 * t);
                s_a = fmaf(x.x, x.x, s_a); s_a = fmaf(x.y, x.y, s_a);
                s_b = fmaf(y.x, y.x, s_b); s_b = fmaf(y.y, y.y, s_b);
            }
            s_a += __shfl_xor_sync(0xffffffffu, s_a, 1); s_a += __shfl_xor_sync(0xffffffffu, s_a, 2);
            s_b += __shfl_xor_sync(0xffffffffu, s_b, 1); s_b += __shfl_xor_sync(0xffffffffu, s_b, 2);
            f_a = rsqrtf(s_a / (float)a.dim + a.eps);
            f_b = rsqrtf(s_b / (float)a.dim + a.eps);
        }
#pragma unroll
        for (int ks = 0; ks < 2 * KS; ks++) {
            const float2 x = ldq2(row_a, ks * 8 + 2 * t), y = ldq2(row_b, ks * 8 + 2 * t);
            qa[ks / 2][(ks & 1) * 2] = pack_bf2(x.x * f_a, x.y * f_a);
            qa[ks / 2][(ks & 1) * 2 + 1] = pack_bf2(y.x * f_b, y.y * f_b);
        }
    }
    float o[ND][4];
#pragma unroll
    for (int i = 0; i < ND; i++) { o[i][0] = 0.f; o[i][1] = 0.f; o[i][2] = 0.f; o[i][3] = 0.f; }
    float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.f, l_b = 0.f;
    constexpr float kLog2e = 1.44269504088896341f;
    const float sc = a.scale * kLog2e, slope = a.slopes ? a.slopes[head] * kLog2e : 0.f;      // scores in units of log 2
    const uint32_t first_pos = start + q0, last_pos = start + min(T, q0 + 64) - 1, total = last_pos + 1;
    const uint32_t lo = a.window && first_pos + 1 > a.window ? first_pos + 1 - a.window : 0;
    const uint32_t n_blocks = (last_pos - lo) / 64 + 1;
    auto stage = [&](uint32_t kb, uint32_t buf) {
        constexpr int CK = QK / 8, CV = VD / 8;
        __nv_bfloat16* ks = Ks + buf * 64 * LK;
        __nv_bfloat16* vs = Vs + buf * 64 * LV;
        const uint32_t k0 = lo + kb * 64, base = k0 % a.cap, c_k = kd / 8, c_v = vd / 8;
        auto slot = [&](uint32_t r) { return base + r < a.cap ? base + r : (base + r) % a.cap; };
        for (uint32_t i = tid; i < 64 * CK; i += 128) {
            const uint32_t r = i / CK, c = i % CK;
            __nv_bfloat16* dst = ks + r * LK + c * 8;
            if (k0 + r < total && c < c_k) cp_async16(smem_u32(dst), kc + (size_t)slot(r) * kd + c * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        for (uint32_t i = tid; i < 64 * CV; i += 128) {
            const uint32_t r = i / CV, c = i % CV;
            __nv_bfloat16* dst = vs + r * LV + c * 8;
            if (k0 + r < total && c < c_v) cp_async16(smem_u32(dst), vc + (size_t)slot(r) * vd + c * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
    };
    const uint32_t pos_a = start + row_a, pos_b = start + row_b;
    const uint32_t lo_a = a.window && pos_a + 1 > a.window ? pos_a + 1 - a.window : 0, lo_b = a.window && pos_b + 1 > a.window ? pos_b + 1 - a.window : 0;
    stage(0, 0);
    for (uint32_t kb = 0; kb < n_blocks; kb++) {
        if (kb + 1 < n_blocks) {
            stage(kb + 1, (kb + 1) & 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const uint32_t ks_u = smem_u32(Ks + (kb & 1) * 64 * LK), vs_u = smem_u32(Vs + (kb & 1) * 64 * LV);
        float s[8][4];
#pragma unroll
        for (int n = 0; n < 8; n++) { s[n][0] = 0.f; s[n][1] = 0.f; s[n][2] = 0.f; s[n][3] = 0.f; }
#pragma unroll
        for (int ks = 0; ks < KS; ks++)
#pragma unroll
            for (int n = 0; n < 8; n += 2) {
                uint32_t b[4];
                ldsm_x4(b, ks_u + ((n * 8 + (lane >> 4) * 8 + (lane & 7)) * LK + ks * 16 + ((lane >> 3) & 1) * 8) * 2);
                mma_bf16(s[n], qa[ks], b[0], b[1]);
                mma_bf16(s[n + 1], qa[ks], b[2], b[3]);
            }
        const uint32_t k0 = lo + kb * 64;
        const uint32_t w_first = first_pos + warp * 16, w_last = w_first + 15;       // positions of this warp's rows
        const bool edge = k0 + 63 > w_first || (a.window && k0 + a.window <= w_last);
        float x_a = -INFINITY, x_b = -INFINITY;
#pragma unroll
        for (int n = 0; n < 8; n++) {
            const uint32_t key = k0 + n * 8 + 2 * t;
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const uint32_t kk = key + (j & 1), pos = j < 2 ? pos_a : pos_b;
                s[n][j] = s[n][j] * sc - slope * (float)(int32_t)(pos - kk);
                if (edge && (kk > pos || kk < (j < 2 ? lo_a : lo_b))) s[n][j] = -INFINITY;
            }
            x_a = fmaxf(x_a, fmaxf(s[n][0], s[n][1]));
            x_b = fmaxf(x_b, fmaxf(s[n][2], s[n][3]));
        }
        x_a = fmaxf(x_a, __shfl_xor_sync(0xffffffffu, x_a, 1)); x_a = fmaxf(x_a, __shfl_xor_sync(0xffffffffu, x_a, 2));
        x_b = fmaxf(x_b, __shfl_xor_sync(0xffffffffu, x_b, 1)); x_b = fmaxf(x_b, __shfl_xor_sync(0xffffffffu, x_b, 2));
        const float n_a = fmaxf(m_a, x_a), n_b = fmaxf(m_b, x_b);
        // a row may see none of the first blocks' keys: its maximum stays -inf and its weights are 0
        const float base_a = n_a == -INFINITY ? 0.f : n_a, base_b = n_b == -INFINITY ? 0.f : n_b;
        const float f_a = exp2f(m_a - base_a), f_b = exp2f(m_b - base_b);
        m_a = n_a;
        m_b = n_b;
        float sum_a = 0.f, sum_b = 0.f;
        uint32_t p[8][2];
#pragma unroll
        for (int n = 0; n < 8; n++) {
            const float p0 = exp2f(s[n][0] - base_a), p1 = exp2f(s[n][1] - base_a), p2 = exp2f(s[n][2] - base_b), p3 = exp2f(s[n][3] - base_b);
            sum_a += p0 + p1;
            sum_b += p2 + p3;
            p[n][0] = pack_bf2(p0, p1);
            p[n][1] = pack_bf2(p2, p3);
        }
        l_a = l_a * f_a + sum_a;
        l_b = l_b * f_b + sum_b;
#pragma unroll
        for (int i = 0; i < ND; i++) { o[i][0] *= f_a; o[i][1] *= f_a; o[i][2] *= f_b; o[i][3] *= f_b; }
#pragma unroll
        for (int kk = 0; kk < 4; kk++) {
            const uint32_t pa[4] = {p[2 * kk][0], p[2 * kk][1], p[2 * kk + 1][0], p[2 * kk + 1][1]};
#pragma unroll
            for (int i = 0; i < ND; i += 2) {
                uint32_t v[4];
                ldsm_x4_trans(v, vs_u + ((kk * 16 + (lane & 15)) * LV + i * 8 + (lane >> 4) * 8) * 2);
                mma_bf16(o[i], pa, v[0], v[1]);
                mma_bf16(o[i + 1], pa, v[2], v[3]);
            }
        }
        __syncthreads();
    }
    l_a += __shfl_xor_sync(0xffffffffu, l_a, 1); l_a += __shfl_xor_sync(0xffffffffu, l_a, 2);
    l_b += __shfl_xor_sync(0xffffffffu, l_b, 1); l_b += __shfl_xor_sync(0xffffffffu, l_b, 2);
    const float i_a = a.out_scale / l_a, i_b = a.out_scale / l_b;
    const bool wide = (a.vdim & 1u) == 0 && (ldo & 1u) == 0;
#pragma unroll
    for (int i = 0; i < ND; i++) {
        const uint32_t c = i * 8 + 2 * t;
        if (c >= a.vdim) continue;
        auto store = [&](uint32_t row, float x, float y) {
            __nv_bfloat16* p = out + (size_t)row * ldo + head * a.vdim + c;
            if (wide) {
                *reinterpret_cast<uint32_t*>(p) = pack_bf2(x, y);
            } else {
                p[0] = __float2bfloat16_rn(x);
                if (c + 1 < a.vdim) p[1] = __float2bfloat16_rn(y);
            }
        };
        if (row_a < T) store(row_a, o[i][0] * i_a, o[i][1] * i_a);
        if (row_b < T) store(row_b, o[i][2] * i_b, o[i][3] * i_b);
    }
}

template <typename K>
static int32_t allow_smem(runit_ctx* ctx, const char* name, K kern, size_t smem) {
    RUNIT_REQUIRE(ctx, smem <= (size_t)ctx->max_smem_optin - 2048, "%s: the layer's sizes do not fit shared memory", name);
    if (smem > 40 * 1024) RUNIT_CUDA_TRY(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return RUNIT_OK;
}
static int head_block(const HeadAttn& a) {
    const uint32_t rep = a.kv_heads ? a.heads / a.kv_heads : 1;
    return rep == 1 ? 1 : (rep == 2 ? 2 : (rep <= 4 ? 4 : 8));
}
static uint32_t head_blocks(const HeadAttn& a) { return a.kv_heads ? (a.heads / a.kv_heads + head_block(a) - 1) / head_block(a) : 0; }

}  // namespace ha

using namespace ha;

uint32_t heads_step_splits(const runit_ctx* ctx, const HeadAttn& a, uint32_t T) {
    // a split of 64 keys is one tile; no more CTAs than two per SM
    const uint64_t blocks = (uint64_t)a.kv_heads * head_blocks(a) * T, keys = a.window && a.window < a.cap ? a.window : a.cap;
    uint64_t n = (2ull * ctx->sm_count + blocks - 1) / blocks;
    n = n < (keys + 63) / 64 ? n : (keys + 63) / 64;
    return n < 1 ? 1u : (n > 64 ? 64u : (uint32_t)n);
}
size_t heads_part_floats(const HeadAttn& a, uint32_t nsplit, uint32_t T) { return (size_t)T * a.heads * nsplit * (a.vdim + 2); }

int32_t heads_step(runit_ctx* ctx, const HeadAttn* ap, const Retention* rp, bool exact, const float* proj, float* ao, float* factor, float* squares,
                   float* part, uint32_t* tickets, uint32_t nsplit, const int32_t* pos_ptr) {
    const HeadAttn a = ap ? *ap : HeadAttn();
    const Retention r = rp ? *rp : Retention();
    RUNIT_REQUIRE(ctx, nsplit > 0 && nsplit <= 64 && (a.heads || r.heads) && r.dim <= ls::kMaxKeyDim && a.vd() <= 2048, "heads_step: bad sizes");
    const uint32_t nhb = head_blocks(a), n_attn = a.kv_heads * nhb * nsplit, n_ret = r.heads * ((r.vdim + 31) / 32);
    const Parts pt{part, part + (size_t)a.heads * nsplit * a.vdim, tickets, nsplit};
    auto go = [&](auto kern, int rb) -> int32_t {
        size_t smem = a.heads ? cta_smem(a, rb) : 0;
        smem = smem > (size_t)r.dim * 8 ? smem : (size_t)r.dim * 8;
        int32_t st = allow_smem(ctx, "heads_step", kern, smem);
        if (st != RUNIT_OK) return st;
        runit_launch_chain_smem(ctx, kern, dim3(n_attn + n_ret), dim3(256), smem, a, r, proj, ao, factor, squares, pt, n_attn, nhb, pos_ptr);
        return runit_after_launch(ctx, "heads_step");
    };
#define RUNIT_HS(RB) (exact ? go(heads_step_kernel<float, RB>, RB) : go(heads_step_kernel<__nv_bfloat16, RB>, RB))
    switch (head_block(a)) {
        case 1: return RUNIT_HS(1);
        case 2: return RUNIT_HS(2);
        case 4: return RUNIT_HS(4);
        default: return RUNIT_HS(8);
    }
#undef RUNIT_HS
}

int32_t heads_rows(runit_ctx* ctx, const HeadAttn* ap, const Retention* rp, bool exact, void* proj, uint32_t ld, uint32_t T, uint32_t start) {
    const HeadAttn a = ap ? *ap : HeadAttn();
    const Retention r = rp ? *rp : Retention();
    RUNIT_REQUIRE(ctx, !ap || T <= a.cap, "heads_rows: %u tokens, but the cache holds %u", T, a.cap);
    const size_t smem = (size_t)r.rot_dims * 4 + 16;
    if (exact) heads_rows_kernel<float><<<T, 256, smem, ctx->stream>>>(a, r, (float*)proj, ld, start);
    else heads_rows_kernel<__nv_bfloat16><<<T, 256, smem, ctx->stream>>>(a, r, (__nv_bfloat16*)proj, ld, start);
    return runit_after_launch(ctx, "heads_rows");
}

int32_t head_attention_rows(runit_ctx* ctx, const HeadAttn& a, bool exact, const void* proj, uint32_t ld, void* out, uint32_t ldo, uint32_t T,
                            uint32_t start, float* part, size_t part_cap, uint32_t* tickets) {
    int32_t st;
    if (!exact && T >= 16 && a.dim <= 192 && a.vdim <= 192) {
        auto go = [&](auto kern, int qk, int vd) -> int32_t {
            const size_t smem = (size_t)2 * 64 * (qk + 8 + vd + 8) * 2;
            if ((st = allow_smem(ctx, "window_prefill", kern, smem)) != RUNIT_OK) return st;
            kern<<<dim3(a.heads, (T + 63) / 64), 128, smem, ctx->stream>>>(a, (const __nv_bfloat16*)proj, ld, (__nv_bfloat16*)out, ldo, T, start);
            return runit_after_launch(ctx, "window_prefill");
        };
        const uint32_t m = a.dim > a.vdim ? a.dim : a.vdim;
        if (m <= 64) return go(window_prefill_kernel<64, 64>, 64, 64);
        if (m <= 128) return go(window_prefill_kernel<128, 128>, 128, 128);
        return go(window_prefill_kernel<192, 192>, 192, 192);
    }
    uint32_t ns = heads_step_splits(ctx, a, T);
    const uint32_t nhb = head_blocks(a);
    while (ns > 1 && (heads_part_floats(a, ns, T) > part_cap || (uint64_t)T * a.kv_heads * nhb > 4096)) ns--;
    const Parts pt{part, part + (size_t)T * a.heads * ns * a.vdim, tickets, ns};
    auto go = [&](auto kern, int rb, auto* p, auto* o) -> int32_t {
        const size_t smem = cta_smem(a, rb);
        if ((st = allow_smem(ctx, "attention_rows", kern, smem)) != RUNIT_OK) return st;
        kern<<<dim3(a.kv_heads * nhb * ns, T), 256, smem, ctx->stream>>>(a, p, ld, o, ldo, pt, nhb, start);
        return runit_after_launch(ctx, "attention_rows");
    };
#define RUNIT_AR(RB)                                                                                 \
    (exact ? go(attn_rows_kernel<float, RB>, RB, (const float*)proj, (float*)out)                    \
           : go(attn_rows_kernel<__nv_bfloat16, RB>, RB, (const __nv_bfloat16*)proj, (__nv_bfloat16*)out))
    switch (head_block(a)) {
        case 1: return RUNIT_AR(1);
        case 2: return RUNIT_AR(2);
        case 4: return RUNIT_AR(4);
        default: return RUNIT_AR(8);
    }
#undef RUNIT_AR
}

}  // namespace runit

using namespace runit;

namespace {
int32_t heads_of(runit_ctx* ctx, const char* who, const runit_heads_cfg* c, HeadAttn* a) {
    RUNIT_REQUIRE(ctx, c->heads > 0 && c->kv_heads > 0 && c->heads % c->kv_heads == 0 && c->dim > 0 && c->dim <= 1024 && c->vdim > 0 && c->vdim <= 1024 &&
                           c->cap > 0 && c->k_cache && c->v_cache, "%s: bad attention sizes", who);
    a->heads = c->heads; a->kv_heads = c->kv_heads; a->dim = c->dim; a->vdim = c->vdim; a->window = c->window; a->cap = c->cap; a->unit_qk = c->unit_qk;
    a->scale = c->scale; a->out_scale = c->out_scale; a->eps = c->eps; a->slopes = (const float*)c->slopes; a->kc = c->k_cache; a->vc = c->v_cache;
    return RUNIT_OK;
}
int32_t retention_of(runit_ctx* ctx, const char* who, const runit_retention_cfg* c, Retention* r) {
    RUNIT_REQUIRE(ctx, c->heads > 0 && c->dim > 0 && c->dim <= 1024 && c->vdim > 0 && c->rot_dims <= c->dim && c->rot_dims % 2 == 0 && c->decay && c->state &&
                           (c->freq || c->rot_dims == 0), "%s: bad retention", who);
    r->heads = c->heads; r->dim = c->dim; r->vdim = c->vdim; r->rot_dims = c->rot_dims; r->out_scale = c->out_scale;
    r->k_scale = (float)(1.0 / std::sqrt((double)c->dim)); r->freq = (const float*)c->freq; r->decay = (const float*)c->decay; r->state = (float*)c->state;
    return RUNIT_OK;
}
}  // namespace

extern "C" {

int32_t runit_heads_step(runit_ctx_t* ctx, const runit_heads_cfg* attn, const runit_retention_cfg* ret, int32_t cache_f32, const void* proj, void* ao,
                         void* factor, void* squares, void* part, void* tickets, uint32_t nsplit, const void* pos) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    HeadAttn a;
    Retention r;
    int32_t st;
    if (attn && (st = heads_of(ctx, "heads_step", attn, &a))) return st;
    if (ret && (st = retention_of(ctx, "heads_step", ret, &r))) return st;
    RUNIT_REQUIRE(ctx, proj && ao && pos && (!attn || (part && tickets)) && (!ret || (factor && squares)), "heads_step: null argument");
    return heads_step(ctx, attn ? &a : nullptr, ret ? &r : nullptr, cache_f32 != 0, (const float*)proj, (float*)ao, (float*)factor, (float*)squares, (float*)part,
                      (uint32_t*)tickets, nsplit, (const int32_t*)pos);
}

int32_t runit_heads_rows(runit_ctx_t* ctx, const runit_heads_cfg* attn, const runit_retention_cfg* ret, int32_t cache_f32, void* proj, uint32_t ld,
                         uint32_t T, uint32_t start) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    HeadAttn a;
    Retention r;
    int32_t st;
    if (attn && (st = heads_of(ctx, "heads_rows", attn, &a))) return st;
    if (ret && (st = retention_of(ctx, "heads_rows", ret, &r))) return st;
    RUNIT_REQUIRE(ctx, proj && (attn || ret) && T > 0 && ld >= a.in_rows() + r.in_rows(), "heads_rows: bad argument");
    return heads_rows(ctx, attn ? &a : nullptr, ret ? &r : nullptr, cache_f32 != 0, proj, ld, T, start);
}

int32_t runit_head_attention_rows(runit_ctx_t* ctx, const runit_heads_cfg* attn, int32_t cache_f32, const void* proj, uint32_t ld, void* out,
                                  uint32_t ldo, uint32_t T, uint32_t start, void* part, size_t part_floats, void* tickets) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    HeadAttn a;
    int32_t st;
    RUNIT_REQUIRE(ctx, attn, "head_attention_rows: null argument");
    if ((st = heads_of(ctx, "head_attention_rows", attn, &a))) return st;
    const uint32_t reach = T + (a.window ? a.window - 1 : start);
    RUNIT_REQUIRE(ctx, proj && out && T > 0 && T <= 65535 && ld >= a.in_rows() && ldo >= a.out_rows() && (a.cap >= reach || a.cap >= start + T) && tickets &&
                           (part || part_floats == 0), "head_attention_rows: bad argument");
    return head_attention_rows(ctx, a, cache_f32 != 0, proj, ld, out, ldo, T, start, (float*)part, part_floats, (uint32_t*)tickets);
}

}  // extern "C"
