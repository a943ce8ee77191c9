// One token of a decaying linear state, S <- decay S + k v^T and o = S^T q, for 32 columns of one head's S [dk][dv] (f32): the
// step of retention (head_attention.cu) and of the state-space layer (linear_state.cu).  256 threads: lane = column, warp w owns
// rows w, w + 8, ...; batches of 128 rows, the first one requested before the inputs are known.
#pragma once

#include "bf16_ops.cuh"

namespace runit {
namespace ls {

constexpr uint32_t kMaxKeyDim = 1024;

struct StateRows {
    float s[16];
};
__device__ __forceinline__ void load_rows(StateRows& st, const float* S, uint32_t dk, uint32_t dv, uint32_t j, uint32_t i0) {
    const uint32_t warp = threadIdx.x >> 5;
#pragma unroll
    for (int r = 0; r < 16; r++) {
        const uint32_t i = i0 + warp + 8 * r;
        st.s[r] = (i < dk && j < dv) ? S[(size_t)i * dv + j] : 0.f;
    }
}
// qs, ks [dk] and red [8][33] in shared memory (qs, ks written and synchronised by the caller).  Returns o[j] in warp 0.
__device__ __forceinline__ float state_step(StateRows& st, float* S, uint32_t dk, uint32_t dv, uint32_t j, const float* qs, const float* ks, float v,
                                            float decay, bool fresh, float (*red)[33]) {
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float o = 0.f;
    for (uint32_t i0 = 0; i0 < dk; i0 += 128) {
        if (i0) load_rows(st, S, dk, dv, j, i0);
#pragma unroll
        for (int r = 0; r < 16; r++) {
            const uint32_t i = i0 + warp + 8 * r;
            if (i < dk && j < dv) {
                const float n = fmaf(ks[i], v, fresh ? 0.f : decay * st.s[r]);
                S[(size_t)i * dv + j] = n;
                o = fmaf(n, qs[i], o);
            }
        }
    }
    red[warp][lane] = o;
    __syncthreads();
    if (warp != 0) return 0.f;
    o = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) o += red[w][lane];
    return o;
}
__device__ __forceinline__ float silu(float x) { return x / (1.0f + expf(-x)); }
// where the result is rounded to bf16 anyway (rows of a portion in the operand type TA)
template <typename TA>
__device__ __forceinline__ float silu_for(float x) {
    if constexpr (sizeof(TA) == 2) return __fdividef(x, 1.0f + __expf(-x));
    else return silu(x);
}
__device__ __forceinline__ float softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
// Sine and cosine of pos * (hi + lo), hi + lo a frequency as the sum of two floats: the product's rounding error (which for far
// positions is that of the angle) and the low part turn the result by their small angle e.
__device__ __forceinline__ void sincos_at(uint32_t pos, float hi, float lo, float* s, float* c) {
    const float p = (float)pos, a = p * hi, e = fmaf(p, lo, fmaf(p, hi, -a));
    float s0, c0;
    sincosf(a, &s0, &c0);
    const float h = -0.5f * e * e;
    *s = s0 + fmaf(c0, e, s0 * h);
    *c = c0 + fmaf(-s0, e, c0 * h);
}
__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

}  // namespace ls
}  // namespace runit
