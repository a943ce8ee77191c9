// Attention over a cached latent per position (multi-head latent attention).
//
// The cache holds one row per position: the normed latent c and the rotated key part all heads share, both padded with zeros
// to multiples of 16 (bf16, or f32 in passes that run in 32-bit throughout).  Two arrangements of the same arithmetic:
//   * folded (decoding, short portions, every pass in 32-bit): W_uk moves to the query side, q_eff = [W_uk^T q_un | q_rot], so
//     that all heads attend over the cached rows themselves and W_uv is applied once to the averaged latent.  A tile of 16
//     (token, head) rows shares every key row it reads; keys are split over CTAs and the partial results are merged by the
//     launch that applies W_uv.
//   * expanded (prompts in bf16): keys and values of all heads are formed by one GEMM over the cached latents, then a causal
//     flash-attention kernel runs per head on tensor cores: (dim + rot_dim) + vdim multiply-adds per pair and head instead of
//     (kv_rank + rot_dim) + kv_rank.
// Scores, softmax, norms and angles are f32 in both.  Rotation: coordinates 2i and 2i+1 form a pair, angle = position * freq[i].
#include "bf16_ops.cuh"
#include "gemv_common.cuh"
#include "tma.cuh"

namespace runit {
namespace la {

__device__ __forceinline__ float wsum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float bf_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf_hi(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }
__device__ __forceinline__ uint32_t pack_bf2(float a, float b) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ void rotate_pair(float& u, float& v, uint32_t pos, float f) {
    float s, c;
    sincosf((float)pos * f, &s, &c);
    const float a = u * c - v * s, b = v * c + u * s;
    u = a;
    v = b;
}

struct Dims {
    uint32_t heads, dim, rot, vdim, rank, cp, pitch;
    float scale, eps;
};

// Cache row of one position from the raw projection (kv_rank + rot_dim values): 256 threads.
template <typename TC>
__device__ __forceinline__ void write_cache_row(const Dims& d, const float* __restrict__ raw, const float* __restrict__ kv_norm,
                                                const float* __restrict__ freq, TC* __restrict__ row, uint32_t pos) {
    __shared__ float part[8];
    float s = 0.f;
    for (uint32_t i = threadIdx.x; i < d.rank; i += 256) s = fmaf(raw[i], raw[i], s);
    s = wsum(s);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = s;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) tot += part[i];
    const float r = rsqrtf(tot / (float)d.rank + d.eps);
    for (uint32_t i = threadIdx.x; i < d.rank; i += 256) put(row + i, raw[i] * r * kv_norm[i]);
    for (uint32_t i = threadIdx.x; i < d.rot / 2; i += 256) {
        float u = raw[d.rank + 2 * i], v = raw[d.rank + 2 * i + 1];
        rotate_pair(u, v, pos, freq[i]);
        put(row + d.cp + 2 * i, u);
        put(row + d.cp + 2 * i + 1, v);
    }
}

// Query side with W_uk folded in.  grid (heads * nchunk + own, T), 256 threads: a CTA forms 64 columns of one head's folded
// query (8 columns x 32 shares of the head's unrotated dimensions per thread, shares added in order); the CTA of a head's
// first chunk also rotates its rot_dim part; the last CTA of a token writes its cache row.
template <typename TC>
__global__ void __launch_bounds__(256) latent_query_kernel(const Dims d, const float* __restrict__ qkv, uint32_t ldq,
                                                            const __nv_bfloat16* __restrict__ w_uk, uint32_t ldk, uint32_t nchunk,
                                                            const float* __restrict__ kv_norm, const float* __restrict__ freq,
                                                            TC* __restrict__ cache, void* __restrict__ q_eff, const LatentPos lp) {
    __shared__ float red[32][65];
    const uint32_t t = blockIdx.y;
    const float* q = qkv + (size_t)t * ldq;
    if (blockIdx.x == d.heads * nchunk) {
        grid_dependency_wait();
        grid_launch_dependents();
        const uint32_t pos = (lp.pos_ptr ? (uint32_t)*lp.pos_ptr : lp.start) + t;
        write_cache_row(d, q + d.heads * (d.dim + d.rot), kv_norm, freq, cache + (size_t)pos * d.pitch, pos);
        return;
    }
    const uint32_t h = blockIdx.x / nchunk, ch = blockIdx.x % nchunk;
    const uint32_t cg = threadIdx.x & 7, g = threadIdx.x >> 3, c = ch * 64 + cg * 8;
    const uint8_t* w = reinterpret_cast<const uint8_t*>(w_uk + (size_t)h * d.dim * ldk + c);
    constexpr int P = 4;
    uint4 pre[P];
#pragma unroll
    for (int i = 0; i < P; i++)
        pre[i] = (c < ldk && g + 32 * i < d.dim) ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)(g + 32 * i) * ldk * 2)) : make_uint4(0, 0, 0, 0);
    grid_dependency_wait();
    grid_launch_dependents();
    const float* qh = q + (size_t)h * (d.dim + d.rot);
    float acc[8];
#pragma unroll
    for (int i = 0; i < 8; i++) acc[i] = 0.f;
    auto step = [&](const uint4& v, float x) {
        acc[0] = fmaf(bf_lo(v.x), x, acc[0]); acc[1] = fmaf(bf_hi(v.x), x, acc[1]);
        acc[2] = fmaf(bf_lo(v.y), x, acc[2]); acc[3] = fmaf(bf_hi(v.y), x, acc[3]);
        acc[4] = fmaf(bf_lo(v.z), x, acc[4]); acc[5] = fmaf(bf_hi(v.z), x, acc[5]);
        acc[6] = fmaf(bf_lo(v.w), x, acc[6]); acc[7] = fmaf(bf_hi(v.w), x, acc[7]);
    };
#pragma unroll
    for (int i = 0; i < P; i++)
        if (g + 32 * i < d.dim) step(pre[i], qh[g + 32 * i]);
    if (c < ldk)
        for (uint32_t k = g + 32 * P; k < d.dim; k += 32) step(__ldg(reinterpret_cast<const uint4*>(w + (size_t)k * ldk * 2)), qh[k]);
#pragma unroll
    for (int i = 0; i < 8; i++) red[g][cg * 8 + i] = acc[i];
    __syncthreads();
    // a row of the folded query: f32, or the high and the low bf16 half of every value (same bytes)
    float* out = reinterpret_cast<float*>(q_eff) + ((size_t)t * d.heads + h) * d.pitch;
    auto put_q = [&](uint32_t col, float v) {
        if constexpr (sizeof(TC) == 4) {
            out[col] = v;
        } else {
            __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(out);
            const __nv_bfloat16 hi = __float2bfloat16_rn(v);
            o[col] = hi;
            o[d.pitch + col] = __float2bfloat16_rn(v - __bfloat162float(hi));
        }
    };
    if (threadIdx.x < 64) {
        const uint32_t col = ch * 64 + threadIdx.x;
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < 32; i++) s += red[i][threadIdx.x];
        if (col < d.cp) put_q(col, s);          // columns past kv_rank are zero: so is the padding of W_uk
    } else if (ch == 0) {
        const uint32_t pos = (lp.pos_ptr ? (uint32_t)*lp.pos_ptr : lp.start) + t;
        for (uint32_t i = threadIdx.x - 64; i < (d.pitch - d.cp) / 2; i += 192) {
            float u = 0.f, v = 0.f;
            if (2 * i < d.rot) {
                u = qh[d.dim + 2 * i];
                v = qh[d.dim + 2 * i + 1];
                rotate_pair(u, v, pos, freq[i]);
            }
            put_q(d.cp + 2 * i, u);
            put_q(d.cp + 2 * i + 1, v);
        }
    }
}

// Cache rows of many tokens, and the rotated parts of their queries in place.  grid (T), 256 threads.
template <typename TC>
__global__ void __launch_bounds__(256) latent_rows_kernel(const Dims d, float* __restrict__ qkv, uint32_t ldq, const float* __restrict__ kv_norm,
                                                           const float* __restrict__ freq, TC* __restrict__ cache, uint32_t start) {
    const uint32_t t = blockIdx.x, pos = start + t;
    float* q = qkv + (size_t)t * ldq;
    const uint32_t half = d.rot / 2;
    for (uint32_t i = threadIdx.x; i < d.heads * half; i += 256) {
        float* p = q + (size_t)(i / half) * (d.dim + d.rot) + d.dim + 2 * (i % half);
        float u = p[0], v = p[1];
        rotate_pair(u, v, pos, freq[i % half]);
        p[0] = u;
        p[1] = v;
    }
    if (kv_norm) write_cache_row(d, q + d.heads * (d.dim + d.rot), kv_norm, freq, cache + (size_t)pos * d.pitch, pos);
}

// ── folded attention ──
// The keys of a tile whose last row sees `len` of them, cut for split `split` of `nsplit`.
__device__ __forceinline__ void split_range(uint32_t len, uint32_t split, uint32_t nsplit, uint32_t& beg, uint32_t& end) {
    const uint32_t chunk = max(64u, ((len + nsplit - 1) / nsplit + 63) / 64 * 64);
    beg = min(len, split * chunk);
    end = min(len, beg + chunk);
}

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x2(uint32_t& r0, uint32_t& r1, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}

// Tensor cores, bf16 cache.  grid (ceil(rows / 16), nsplit), 8 warps; blocks of KB keys, two stages (cp.async).  Scores: warp w
// takes keys 8w .. 8w+7 over the whole row; values: warp w takes the 16-column groups w, w+8, ... of the latent for all keys.
// The query is carried as the sum of two bf16 numbers, so that its rounding does not add to the cache's.
// KB = 64, or 32 for rows that would not fit shared memory otherwise.
template <int NG, int KB>      // 16-column groups of the latent per warp, keys per block
__global__ void __launch_bounds__(256) latent_attn_kernel(const Dims d, const __nv_bfloat16* __restrict__ q_eff, const __nv_bfloat16* __restrict__ cache,
                                                           float* __restrict__ part_o, float* __restrict__ part_ml, uint32_t rows,
                                                           const LatentPos lp) {
    extern __shared__ __align__(16) uint8_t smem[];
    constexpr int LP = KB + 8;
    __shared__ float wmax[8][16], wl[8][16];
    const uint32_t ld = d.pitch + 8;                                   // row pitch in shared memory (elements)
    __nv_bfloat16* qh = reinterpret_cast<__nv_bfloat16*>(smem);        // [16][ld] high part
    __nv_bfloat16* ql = qh + 16 * ld;                                  // [16][ld] low part
    __nv_bfloat16* kv = ql + 16 * ld;                                  // [2][KB][ld]
    __nv_bfloat16* ps = kv + 2 * KB * ld;                             // [16][LP]
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const uint32_t r0 = blockIdx.x * 16, split = blockIdx.y, nsplit = gridDim.y;
    grid_dependency_wait();
    grid_launch_dependents();
    const uint32_t start = lp.pos_ptr ? (uint32_t)*lp.pos_ptr : lp.start;
    const uint32_t last = min(rows, r0 + 16) - 1, len = start + last / d.heads + 1;
    uint32_t beg, end;
    split_range(len, split, nsplit, beg, end);
    const uint32_t cpr = d.pitch / 8, nblk = (end - beg + KB - 1) / KB;
    auto stage = [&](uint32_t b) {
        __nv_bfloat16* dst = kv + (b & 1) * KB * ld;
        for (uint32_t i = tid; i < KB * cpr; i += 256) {
            const uint32_t r = i / cpr, c = i - r * cpr, key = beg + b * KB + r;
            if (key < end) cp_async16(smem_u32(dst + r * ld + c * 8), cache + (size_t)key * d.pitch + c * 8);
            else *reinterpret_cast<uint4*>(dst + r * ld + c * 8) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
    };
    if (nblk) {
        for (uint32_t i = tid; i < 32 * cpr; i += 256) {               // the tile's queries: 16 high rows, 16 low rows
            const uint32_t r = i / cpr, c = i - r * cpr, row = r0 + (r & 15);
            __nv_bfloat16* dst = qh + r * ld + c * 8;
            if (row < rows) cp_async16(smem_u32(dst), q_eff + ((size_t)row * 2 + (r >> 4)) * d.pitch + c * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        stage(0);                                                      // one group with the queries
    }
    const uint32_t ra = r0 + g, rb = ra + 8;                           // this thread's two query rows
    const uint32_t lim_a = ra < rows ? start + ra / d.heads : 0, lim_b = rb < rows ? start + rb / d.heads : 0;   // last visible position
    float o[NG][8];
#pragma unroll
    for (int i = 0; i < NG; i++)
#pragma unroll
        for (int j = 0; j < 8; j++) o[i][j] = 0.f;
    float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.f, l_b = 0.f;
    const uint32_t ngroups = d.cp / 16;
    // lane -> row and 8-column half of the 16x16 A tile (ldmatrix x4)
    const uint32_t a_off = (lane & 15) * ld + (lane >> 4) * 8;
    for (uint32_t b = 0; b < nblk; b++) {
        if (b + 1 < nblk) {
            stage(b + 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const __nv_bfloat16* kb = kv + (b & 1) * KB * ld;
        float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
        const bool scores = warp * 8 < KB;
        const uint32_t qh_u = smem_u32(qh + a_off), ql_u = smem_u32(ql + a_off);
        const uint32_t k_u = smem_u32(kb + (warp * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8);
        if (scores)
#pragma unroll 4
        for (uint32_t ks = 0; ks < d.pitch / 16; ks++) {
            uint32_t ah[4], al[4], b0, b1;
            ldsm_x4(ah, qh_u + ks * 32);
            ldsm_x4(al, ql_u + ks * 32);
            ldsm_x2(b0, b1, k_u + ks * 32);
            mma_bf16(s, ah, b0, b1);
            mma_bf16(s2, al, b0, b1);
        }
        const uint32_t key0 = beg + b * KB + warp * 8 + 2 * tq;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const uint32_t key = key0 + (j & 1);
            const bool vis = scores && key < end && key <= (j < 2 ? lim_a : lim_b);
            s[j] = vis ? (s[j] + s2[j]) * d.scale : -INFINITY;
        }
        float xa = fmaxf(s[0], s[1]), xb = fmaxf(s[2], s[3]);
        xa = fmaxf(xa, __shfl_xor_sync(0xffffffffu, xa, 1)); xa = fmaxf(xa, __shfl_xor_sync(0xffffffffu, xa, 2));
        xb = fmaxf(xb, __shfl_xor_sync(0xffffffffu, xb, 1)); xb = fmaxf(xb, __shfl_xor_sync(0xffffffffu, xb, 2));
        if (tq == 0) { wmax[warp][g] = xa; wmax[warp][g + 8] = xb; }
        __syncthreads();
        float n_a = m_a, n_b = m_b;
#pragma unroll
        for (int i = 0; i < 8; i++) {
            n_a = fmaxf(n_a, wmax[i][g]);
            n_b = fmaxf(n_b, wmax[i][g + 8]);
        }
        // a row may see none of the block's keys (and none so far): its maximum stays -inf and its weights are 0
        const float base_a = n_a == -INFINITY ? 0.f : n_a, base_b = n_b == -INFINITY ? 0.f : n_b;
        const float f_a = expf(m_a - base_a), f_b = expf(m_b - base_b);
        const float p0 = expf(s[0] - base_a), p1 = expf(s[1] - base_a), p2 = expf(s[2] - base_b), p3 = expf(s[3] - base_b);
        m_a = n_a;
        m_b = n_b;
        l_a = l_a * f_a + p0 + p1;
        l_b = l_b * f_b + p2 + p3;
        if (scores) {
            *reinterpret_cast<uint32_t*>(ps + g * LP + warp * 8 + 2 * tq) = pack_bf2(p0, p1);
            *reinterpret_cast<uint32_t*>(ps + (g + 8) * LP + warp * 8 + 2 * tq) = pack_bf2(p2, p3);
        }
        __syncthreads();
        uint32_t pa[KB / 16][4];
#pragma unroll
        for (int kk = 0; kk < KB / 16; kk++) ldsm_x4(pa[kk], smem_u32(ps + (lane & 15) * LP + (lane >> 4) * 8 + kk * 16));
#pragma unroll
        for (int i = 0; i < NG; i++) {
            const uint32_t grp = warp + 8 * i;
            if (grp >= ngroups) break;
            o[i][0] *= f_a; o[i][1] *= f_a; o[i][2] *= f_b; o[i][3] *= f_b;
            o[i][4] *= f_a; o[i][5] *= f_a; o[i][6] *= f_b; o[i][7] *= f_b;
#pragma unroll
            for (int kk = 0; kk < KB / 16; kk++) {
                // 16 keys x 16 columns: transposed tiles (keys 0-7 | 8-15) x (columns 0-7 | 8-15)
                uint32_t v[4];
                ldsm_x4_trans(v, smem_u32(kb + (kk * 16 + (lane & 15)) * ld + grp * 16 + (lane >> 4) * 8));
                float (&o0)[4] = *reinterpret_cast<float(*)[4]>(&o[i][0]);
                float (&o1)[4] = *reinterpret_cast<float(*)[4]>(&o[i][4]);
                mma_bf16(o0, pa[kk], v[0], v[1]);
                mma_bf16(o1, pa[kk], v[2], v[3]);
            }
        }
        __syncthreads();       // the stage buffer and ps may be rewritten
    }
    l_a += __shfl_xor_sync(0xffffffffu, l_a, 1); l_a += __shfl_xor_sync(0xffffffffu, l_a, 2);
    l_b += __shfl_xor_sync(0xffffffffu, l_b, 1); l_b += __shfl_xor_sync(0xffffffffu, l_b, 2);
    if (tq == 0) { wl[warp][g] = l_a; wl[warp][g + 8] = l_b; }
    __syncthreads();
    auto sum_l = [&](uint32_t r) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < 8; i++) s += wl[i][r];
        return s;
    };
    if (warp == 0 && tq == 0) {
        if (ra < rows) {
            float* p = part_ml + ((size_t)ra * nsplit + split) * 2;
            p[0] = m_a;
            p[1] = sum_l(g);
        }
        if (rb < rows) {
            float* p = part_ml + ((size_t)rb * nsplit + split) * 2;
            p[0] = m_b;
            p[1] = sum_l(g + 8);
        }
    }
    if (!nblk) return;         // an empty split: its maximum is -inf and its sums are not read
#pragma unroll
    for (int i = 0; i < NG; i++) {
        const uint32_t grp = warp + 8 * i;
        if (grp >= ngroups) break;
        const uint32_t col = grp * 16 + 2 * tq;
        if (ra < rows) {
            float* p = part_o + ((size_t)ra * nsplit + split) * d.cp + col;
            *reinterpret_cast<float2*>(p) = make_float2(o[i][0], o[i][1]);
            *reinterpret_cast<float2*>(p + 8) = make_float2(o[i][4], o[i][5]);
        }
        if (rb < rows) {
            float* p = part_o + ((size_t)rb * nsplit + split) * d.cp + col;
            *reinterpret_cast<float2*>(p) = make_float2(o[i][2], o[i][3]);
            *reinterpret_cast<float2*>(p + 8) = make_float2(o[i][6], o[i][7]);
        }
    }
}

// f32 cache: grid (rows, nsplit), 4 warps, a warp takes every fourth key of the split; lane <-> columns.
template <int CPL>     // latent columns per lane
__global__ void __launch_bounds__(128) latent_attn_f32_kernel(const Dims d, const float* __restrict__ q_eff, const float* __restrict__ cache,
                                                               float* __restrict__ part_o, float* __restrict__ part_ml, const LatentPos lp) {
    extern __shared__ __align__(16) uint8_t smem[];
    float* qs = reinterpret_cast<float*>(smem);            // [pitch]
    float* os = qs + d.pitch;                              // [4][cp]
    __shared__ float sm_m[4], sm_l[4];
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x, split = blockIdx.y, nsplit = gridDim.y;
    grid_dependency_wait();
    grid_launch_dependents();
    const uint32_t len = (lp.pos_ptr ? (uint32_t)*lp.pos_ptr : lp.start) + row / d.heads + 1;
    uint32_t beg, end;
    split_range(len, split, nsplit, beg, end);
    for (uint32_t i = threadIdx.x; i < d.pitch; i += 128) qs[i] = q_eff[(size_t)row * d.pitch + i];
    __syncthreads();
    float m = -INFINITY, l = 0.f, o[CPL];
#pragma unroll
    for (int i = 0; i < CPL; i++) o[i] = 0.f;
    for (uint32_t key = beg + warp; key < end; key += 4) {
        const float* r = cache + (size_t)key * d.pitch;
        float c[CPL], s = 0.f;
#pragma unroll
        for (int i = 0; i < CPL; i++) {
            const uint32_t col = lane + 32 * i;
            c[i] = col < d.cp ? r[col] : 0.f;
            if (col < d.cp) s = fmaf(c[i], qs[col], s);
        }
        for (uint32_t col = d.cp + lane; col < d.pitch; col += 32) s = fmaf(r[col], qs[col], s);
        s = wsum(s) * d.scale;
        const float n = fmaxf(m, s), f = expf(m - n), p = expf(s - n);
        m = n;
        l = l * f + p;
#pragma unroll
        for (int i = 0; i < CPL; i++) o[i] = fmaf(p, c[i], o[i] * f);
    }
    if (lane == 0) { sm_m[warp] = m; sm_l[warp] = l; }
#pragma unroll
    for (int i = 0; i < CPL; i++)
        if (lane + 32 * i < d.cp) os[warp * d.cp + lane + 32 * i] = o[i];
    __syncthreads();
    const float M = fmaxf(fmaxf(sm_m[0], sm_m[1]), fmaxf(sm_m[2], sm_m[3]));
    float f[4], L = 0.f;
#pragma unroll
    for (int w = 0; w < 4; w++) {
        f[w] = sm_m[w] == -INFINITY ? 0.f : expf(sm_m[w] - M);
        L += sm_l[w] * f[w];
    }
    if (threadIdx.x == 0) {
        float* p = part_ml + ((size_t)row * nsplit + split) * 2;
        p[0] = M;
        p[1] = L;
    }
    if (beg == end) return;
    float* po = part_o + ((size_t)row * nsplit + split) * d.cp;
    for (uint32_t i = threadIdx.x; i < d.cp; i += 128)
        po[i] = os[i] * f[0] + os[d.cp + i] * f[1] + os[2 * d.cp + i] * f[2] + os[3 * d.cp + i] * f[3];
}

// Merge of the splits of one (token, head) and its value projection: grid (heads, ceil(vdim / 32), T), 8 warps, a warp takes 4
// rows of W_uv.
template <typename TO>
__global__ void __launch_bounds__(256) latent_value_kernel(const Dims d, const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                            uint32_t nsplit, const __nv_bfloat16* __restrict__ w_uv, uint32_t ldk,
                                                            TO* __restrict__ out, uint32_t ldo) {
    extern __shared__ __align__(16) uint8_t smem[];
    float* c = reinterpret_cast<float*>(smem);             // [max(1024, cp)]: shares of the merged latent
    float* wt = c + (d.cp < 1024 ? 1024 : d.cp);           // [nsplit]
    __shared__ uint32_t live_s;
    const uint32_t h = blockIdx.x, t = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t j0 = blockIdx.y * 32 + warp * 4, nch = (d.rank + 7) / 8;
    const uint4* w = reinterpret_cast<const uint4*>(w_uv + (size_t)(h * d.vdim + j0) * ldk);
    constexpr int P = 2;
    uint4 pre[4][P];
#pragma unroll
    for (int r = 0; r < 4; r++)
#pragma unroll
        for (int i = 0; i < P; i++)
            pre[r][i] = (j0 + r < d.vdim && lane + 32 * i < nch) ? __ldg(w + (size_t)r * (ldk / 8) + lane + 32 * i) : make_uint4(0, 0, 0, 0);
    grid_dependency_wait();
    grid_launch_dependents();
    const size_t row = (size_t)t * d.heads + h;
    if (warp == 0) {
        float M = -INFINITY, L = 0.f;
        uint32_t live = 0;
        for (uint32_t s = lane; s < nsplit; s += 32) {
            const float m = part_ml[(row * nsplit + s) * 2];
            M = fmaxf(M, m);
            if (m != -INFINITY) live = s + 1;         // the splits in which the row sees keys are the first ones
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
            live = max(live, __shfl_xor_sync(0xffffffffu, live, o));
        }
        for (uint32_t s = lane; s < live; s += 32) {
            const float2 ml = *reinterpret_cast<const float2*>(part_ml + (row * nsplit + s) * 2);
            const float f = expf(ml.x - M);
            wt[s] = f;
            L = fmaf(f, ml.y, L);
        }
        L = wsum(L);
        for (uint32_t s = lane; s < live; s += 32) wt[s] /= L;
        if (lane == 0) live_s = live;
    }
    __syncthreads();
    // weighted sum of the splits' rows: thread = 4 columns x every G-th split, eight loads in flight; shares added in order
    const uint32_t c4 = d.cp / 4, G = c4 < 256 ? 256 / c4 : 1, live = live_s;
    for (uint32_t i = threadIdx.x; i < G * c4; i += 256) {
        const uint32_t grp = i / c4, col = i - grp * c4;
        const float4* p = reinterpret_cast<const float4*>(part_o + row * nsplit * d.cp) + col;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        for (uint32_t s0 = grp; s0 < live; s0 += 8 * G) {
            float4 x[8];
#pragma unroll
            for (int k = 0; k < 8; k++) {
                const uint32_t s = s0 + k * G;
                x[k] = s < live ? p[(size_t)s * c4] : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int k = 0; k < 8; k++) {
                const uint32_t s = s0 + k * G;
                const float f = s < live ? wt[s] : 0.f;
                v.x = fmaf(f, x[k].x, v.x); v.y = fmaf(f, x[k].y, v.y); v.z = fmaf(f, x[k].z, v.z); v.w = fmaf(f, x[k].w, v.w);
            }
        }
        reinterpret_cast<float4*>(c)[grp * c4 + col] = v;
    }
    __syncthreads();
    if (G > 1) {
        for (uint32_t i = threadIdx.x; i < d.cp; i += 256) {
            float v = c[i];
            for (uint32_t k = 1; k < G; k++) v += c[k * d.cp + i];
            c[i] = v;
        }
        __syncthreads();
    }
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    auto step = [&](const uint4& v, uint32_t ch, float a) {
        const float4 x0 = *reinterpret_cast<const float4*>(c + ch * 8), x1 = *reinterpret_cast<const float4*>(c + ch * 8 + 4);
        a = fmaf(bf_lo(v.x), x0.x, a); a = fmaf(bf_hi(v.x), x0.y, a); a = fmaf(bf_lo(v.y), x0.z, a); a = fmaf(bf_hi(v.y), x0.w, a);
        a = fmaf(bf_lo(v.z), x1.x, a); a = fmaf(bf_hi(v.z), x1.y, a); a = fmaf(bf_lo(v.w), x1.z, a); a = fmaf(bf_hi(v.w), x1.w, a);
        return a;
    };
#pragma unroll
    for (int i = 0; i < P; i++)
        if (lane + 32 * i < nch)
#pragma unroll
            for (int r = 0; r < 4; r++) acc[r] = step(pre[r][i], lane + 32 * i, acc[r]);
    for (uint32_t ch = lane + 32 * P; ch < nch; ch += 32)
#pragma unroll
        for (int r = 0; r < 4; r++)
            if (j0 + r < d.vdim) acc[r] = step(__ldg(w + (size_t)r * (ldk / 8) + ch), ch, acc[r]);
#pragma unroll
    for (int r = 0; r < 4; r++) {
        acc[r] = wsum(acc[r]);
        if (lane == 0 && j0 + r < d.vdim) put(out + (size_t)t * ldo + h * d.vdim + j0 + r, acc[r]);
    }
}

// ── expanded attention (prompts) ──
// The arrangement of prefill_attn_kernel (prefill.cu) with keys of two sources and separate key and value widths: grid
// (heads, ceil(T / 64)), 4 warps of 16 queries, key blocks of 64 staged two deep by cp.async, mma.sync m16n8k16.
// QK >= dim + rot_dim and VD >= vdim: the rest is zero.
template <int QK, int VD>
__global__ void __launch_bounds__(128) latent_prefill_kernel(const Dims d, const float* __restrict__ q, uint32_t ldq,
                                                              const __nv_bfloat16* __restrict__ kv, uint32_t ldkv,
                                                              const __nv_bfloat16* __restrict__ cache, __nv_bfloat16* __restrict__ out,
                                                              uint32_t ldo, uint32_t T, uint32_t start) {
    constexpr int LK = QK + 8, LV = VD + 8, KS = QK / 16, ND = VD / 8;
    extern __shared__ __align__(16) uint8_t smem[];
    __nv_bfloat16* const Ks = reinterpret_cast<__nv_bfloat16*>(smem);     // [2][64 * LK]
    __nv_bfloat16* const Vs = Ks + 2 * 64 * LK;                           // [2][64 * LV]
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const uint32_t head = blockIdx.x, q0 = (gridDim.y - 1 - blockIdx.y) * 64;      // the blocks that see the most keys first
    const uint32_t row_a = q0 + warp * 16 + g, row_b = row_a + 8, qd = d.dim + d.rot;
    uint32_t qa[KS][4];
    auto ldq2 = [&](uint32_t row, uint32_t c) -> uint32_t {
        float2 v = make_float2(0.f, 0.f);
        if (row < T && c < qd) v = *reinterpret_cast<const float2*>(q + (size_t)row * ldq + head * qd + c);
        return pack_bf2(v.x, v.y);
    };
#pragma unroll
    for (int ks = 0; ks < KS; ks++) {
        const uint32_t c0 = ks * 16 + 2 * t;
        qa[ks][0] = ldq2(row_a, c0);
        qa[ks][1] = ldq2(row_b, c0);
        qa[ks][2] = ldq2(row_a, c0 + 8);
        qa[ks][3] = ldq2(row_b, c0 + 8);
    }
    float o[ND][4];
#pragma unroll
    for (int i = 0; i < ND; i++) { o[i][0] = 0.f; o[i][1] = 0.f; o[i][2] = 0.f; o[i][3] = 0.f; }
    float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.f, l_b = 0.f;
    const uint32_t total = start + T, last_q = min(T, q0 + 64) - 1, n_blocks = (start + last_q) / 64 + 1;
    const float sc = d.scale * 1.44269504088896341f;                      // scores in units of log 2
    auto stage = [&](uint32_t kb, uint32_t buf) {
        constexpr int CK = QK / 8, CV = VD / 8;
        __nv_bfloat16* kd = Ks + buf * 64 * LK;
        __nv_bfloat16* vd = Vs + buf * 64 * LV;
        const uint32_t c_un = d.dim / 8, c_all = qd / 8, c_v = d.vdim / 8;
        for (uint32_t i = tid; i < 64 * CK; i += 128) {
            const uint32_t r = i / CK, c = i % CK, key = kb * 64 + r;
            __nv_bfloat16* dst = kd + r * LK + c * 8;
            if (key < total && c < c_un) cp_async16(smem_u32(dst), kv + (size_t)key * ldkv + head * d.dim + c * 8);
            else if (key < total && c < c_all) cp_async16(smem_u32(dst), cache + (size_t)key * d.pitch + d.cp + (c - c_un) * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        for (uint32_t i = tid; i < 64 * CV; i += 128) {
            const uint32_t r = i / CV, c = i % CV, key = kb * 64 + r;
            __nv_bfloat16* dst = vd + r * LV + c * 8;
            if (key < total && c < c_v) cp_async16(smem_u32(dst), kv + (size_t)key * ldkv + d.heads * d.dim + head * d.vdim + c * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
    };
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
                // keys 8n .. 8n+15, 16 K elements: tiles (keys 0-7, k 0-7), (0-7, 8-15), (8-15, 0-7), (8-15, 8-15)
                uint32_t b[4];
                ldsm_x4(b, ks_u + ((n * 8 + (lane >> 4) * 8 + (lane & 7)) * LK + ks * 16 + ((lane >> 3) & 1) * 8) * 2);
                mma_bf16(s[n], qa[ks], b[0], b[1]);
                mma_bf16(s[n + 1], qa[ks], b[2], b[3]);
            }
        const uint32_t lim_a = start + row_a, lim_b = start + row_b;
        const bool edge = (kb + 1) * 64 > start + q0 + warp * 16 + 1;         // some key of the block is past some query of this warp
        float x_a = -INFINITY, x_b = -INFINITY;
#pragma unroll
        for (int n = 0; n < 8; n++) {
            const uint32_t key = kb * 64 + n * 8 + 2 * t;
#pragma unroll
            for (int j = 0; j < 4; j++) {
                s[n][j] *= sc;
                if (edge && key + (j & 1) > (j < 2 ? lim_a : lim_b)) s[n][j] = -INFINITY;
            }
            x_a = fmaxf(x_a, fmaxf(s[n][0], s[n][1]));
            x_b = fmaxf(x_b, fmaxf(s[n][2], s[n][3]));
        }
        x_a = fmaxf(x_a, __shfl_xor_sync(0xffffffffu, x_a, 1)); x_a = fmaxf(x_a, __shfl_xor_sync(0xffffffffu, x_a, 2));
        x_b = fmaxf(x_b, __shfl_xor_sync(0xffffffffu, x_b, 1)); x_b = fmaxf(x_b, __shfl_xor_sync(0xffffffffu, x_b, 2));
        const float n_a = fmaxf(m_a, x_a), n_b = fmaxf(m_b, x_b);             // key 0 is visible to every row: finite
        const float f_a = exp2f(m_a - n_a), f_b = exp2f(m_b - n_b);
        m_a = n_a;
        m_b = n_b;
        float sum_a = 0.f, sum_b = 0.f;
        uint32_t p[8][2];
#pragma unroll
        for (int n = 0; n < 8; n++) {
            const float p0 = exp2f(s[n][0] - n_a), p1 = exp2f(s[n][1] - n_a), p2 = exp2f(s[n][2] - n_b), p3 = exp2f(s[n][3] - n_b);
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
            const uint32_t a[4] = {p[2 * kk][0], p[2 * kk][1], p[2 * kk + 1][0], p[2 * kk + 1][1]};
#pragma unroll
            for (int i = 0; i < ND; i += 2) {
                uint32_t v[4];
                ldsm_x4_trans(v, vs_u + ((kk * 16 + (lane & 15)) * LV + i * 8 + (lane >> 4) * 8) * 2);
                mma_bf16(o[i], a, v[0], v[1]);
                mma_bf16(o[i + 1], a, v[2], v[3]);
            }
        }
        __syncthreads();
    }
    l_a += __shfl_xor_sync(0xffffffffu, l_a, 1); l_a += __shfl_xor_sync(0xffffffffu, l_a, 2);
    l_b += __shfl_xor_sync(0xffffffffu, l_b, 1); l_b += __shfl_xor_sync(0xffffffffu, l_b, 2);
    const float i_a = 1.0f / l_a, i_b = 1.0f / l_b;
#pragma unroll
    for (int i = 0; i < ND; i++) {
        const uint32_t c = i * 8 + 2 * t;
        if (c >= d.vdim) continue;
        if (row_a < T) *reinterpret_cast<uint32_t*>(out + (size_t)row_a * ldo + head * d.vdim + c) = pack_bf2(o[i][0] * i_a, o[i][1] * i_a);
        if (row_b < T) *reinterpret_cast<uint32_t*>(out + (size_t)row_b * ldo + head * d.vdim + c) = pack_bf2(o[i][2] * i_b, o[i][3] * i_b);
    }
}

static Dims dims_of(const LatentDims& d) { return Dims{d.heads, d.dim, d.rot_dim, d.vdim, d.kv_rank, d.cp(), d.pitch(), d.scale, d.eps}; }

template <typename K>
static int32_t allow_smem(runit_ctx* ctx, const char* name, K kern, size_t smem) {
    RUNIT_REQUIRE(ctx, smem <= (size_t)ctx->max_smem_optin - 1024, "%s: the layer's sizes do not fit shared memory", name);
    if (smem > 40 * 1024) RUNIT_CUDA_TRY(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return RUNIT_OK;
}

}  // namespace la

using namespace la;

int32_t latent_query(runit_ctx* ctx, const LatentDims& d, bool cache_f32, const float* qkv, uint32_t ldq, const void* w_uk, uint32_t ldk,
                     const float* kv_norm, const float* freq, void* cache, void* q_eff, uint32_t T, LatentPos pos) {
    const uint32_t nchunk = (d.cp() + 63) / 64;
    const dim3 grid(d.heads * nchunk + (kv_norm ? 1 : 0), T);
    if (cache_f32)
        runit_launch_chain(ctx, latent_query_kernel<float>, grid, dim3(256), dims_of(d), qkv, ldq, (const __nv_bfloat16*)w_uk, ldk, nchunk, kv_norm,
                           freq, (float*)cache, q_eff, pos);
    else
        runit_launch_chain(ctx, latent_query_kernel<__nv_bfloat16>, grid, dim3(256), dims_of(d), qkv, ldq, (const __nv_bfloat16*)w_uk, ldk, nchunk,
                           kv_norm, freq, (__nv_bfloat16*)cache, q_eff, pos);
    return runit_after_launch(ctx, "latent_query");
}

int32_t latent_rows(runit_ctx* ctx, const LatentDims& d, bool cache_f32, float* qkv, uint32_t ldq, const float* kv_norm, const float* freq,
                    void* cache, uint32_t T, LatentPos pos) {
    RUNIT_REQUIRE(ctx, !pos.pos_ptr, "latent_rows: the position is a host value");
    if (cache_f32) latent_rows_kernel<float><<<T, 256, 0, ctx->stream>>>(dims_of(d), qkv, ldq, kv_norm, freq, (float*)cache, pos.start);
    else latent_rows_kernel<__nv_bfloat16><<<T, 256, 0, ctx->stream>>>(dims_of(d), qkv, ldq, kv_norm, freq, (__nv_bfloat16*)cache, pos.start);
    return runit_after_launch(ctx, "latent_rows");
}

uint32_t latent_splits(const runit_ctx* ctx, const LatentDims& d, bool cache_f32, uint32_t T) {
    const uint64_t rows = (uint64_t)T * d.heads, tiles = cache_f32 ? rows : (rows + 15) / 16;
    const uint64_t want = (uint64_t)ctx->sm_count * (cache_f32 ? 8 : 2), n = want / tiles;
    return n < 1 ? 1u : (n > 64 ? 64u : (uint32_t)n);
}

int32_t latent_attention(runit_ctx* ctx, const LatentDims& d, bool cache_f32, const void* q_eff, const void* cache, float* part_o,
                         float* part_ml, uint32_t nsplit, uint32_t T, LatentPos pos) {
    const uint32_t rows = T * d.heads;
    int32_t st;
    if (cache_f32) {
        const size_t smem = (size_t)(d.pitch() + 4 * d.cp()) * 4;
        auto go = [&](auto kern) -> int32_t {
            if ((st = allow_smem(ctx, "latent_attention", kern, smem)) != RUNIT_OK) return st;
            runit_launch_chain_smem(ctx, kern, dim3(rows, nsplit), dim3(128), smem, dims_of(d), (const float*)q_eff, (const float*)cache, part_o, part_ml, pos);
            return runit_after_launch(ctx, "latent_attention_f32");
        };
        if (d.cp() <= 128) return go(latent_attn_f32_kernel<4>);
        if (d.cp() <= 512) return go(latent_attn_f32_kernel<16>);
        RUNIT_REQUIRE(ctx, d.cp() <= 1024, "latent_attention: a latent of more than 1024 values");
        return go(latent_attn_f32_kernel<32>);
    }
    const size_t ld = d.pitch() + 8;
    auto go = [&](auto kern, size_t kb) -> int32_t {
        const size_t smem = (32 * ld + 2 * kb * ld + 16 * (kb + 8)) * 2;
        if ((st = allow_smem(ctx, "latent_attention", kern, smem)) != RUNIT_OK) return st;
        runit_launch_chain_smem(ctx, kern, dim3((rows + 15) / 16, nsplit), dim3(256), smem, dims_of(d), (const __nv_bfloat16*)q_eff,
                                (const __nv_bfloat16*)cache, (float*)part_o, (float*)part_ml, rows, pos);
        return runit_after_launch(ctx, "latent_attention");
    };
    RUNIT_REQUIRE(ctx, d.cp() <= 1024, "latent_attention: a latent of more than 1024 values");
    if (d.pitch() <= 672) {
        if (d.cp() <= 128) return go(latent_attn_kernel<1, 64>, 64);
        if (d.cp() <= 512) return go(latent_attn_kernel<4, 64>, 64);
        return go(latent_attn_kernel<8, 64>, 64);
    }
    return go(latent_attn_kernel<8, 32>, 32);
}

int32_t latent_value(runit_ctx* ctx, const LatentDims& d, const float* part_o, const float* part_ml, uint32_t nsplit, const void* w_uv,
                     uint32_t ldk, void* out, bool out_f32, uint32_t ldo, uint32_t T) {
    const dim3 grid(d.heads, (d.vdim + 31) / 32, T);
    const size_t smem = (size_t)((d.cp() < 1024 ? 1024 : d.cp()) + nsplit) * 4;
    if (out_f32)
        runit_launch_chain_smem(ctx, latent_value_kernel<float>, grid, dim3(256), smem, dims_of(d), part_o, part_ml, nsplit,
                                (const __nv_bfloat16*)w_uv, ldk, (float*)out, ldo);
    else
        runit_launch_chain_smem(ctx, latent_value_kernel<__nv_bfloat16>, grid, dim3(256), smem, dims_of(d), part_o, part_ml, nsplit,
                                (const __nv_bfloat16*)w_uv, ldk, (__nv_bfloat16*)out, ldo);
    return runit_after_launch(ctx, "latent_value");
}

bool latent_prefill_supported(const LatentDims& d) {
    return d.dim % 8 == 0 && d.rot_dim % 8 == 0 && d.vdim % 8 == 0 && d.dim + d.rot_dim <= 192 && d.vdim <= 128;
}

int32_t latent_prefill(runit_ctx* ctx, const LatentDims& d, const float* q, uint32_t ldq, const void* kv, uint32_t ldkv, const void* cache,
                       void* out_bf16, uint32_t ldo, uint32_t T, uint32_t start) {
    RUNIT_REQUIRE(ctx, latent_prefill_supported(d) && ldq % 2 == 0 && ldkv % 8 == 0 && ldo % 2 == 0, "latent_prefill: sizes not supported");
    int32_t st;
    auto go = [&](auto kern, int qk, int vd) -> int32_t {
        const size_t smem = (size_t)2 * 64 * (qk + 8 + vd + 8) * 2;
        if ((st = allow_smem(ctx, "latent_prefill", kern, smem)) != RUNIT_OK) return st;
        kern<<<dim3(d.heads, (T + 63) / 64), 128, smem, ctx->stream>>>(dims_of(d), q, ldq, (const __nv_bfloat16*)kv, ldkv,
                                                                        (const __nv_bfloat16*)cache, (__nv_bfloat16*)out_bf16, ldo, T, start);
        return runit_after_launch(ctx, "latent_prefill");
    };
    const uint32_t qk = d.dim + d.rot_dim;
    if (d.vdim <= 64) {
        if (qk <= 64) return go(latent_prefill_kernel<64, 64>, 64, 64);
        if (qk <= 96) return go(latent_prefill_kernel<96, 64>, 96, 64);
        if (qk <= 128) return go(latent_prefill_kernel<128, 64>, 128, 64);
    }
    if (qk <= 128) return go(latent_prefill_kernel<128, 128>, 128, 128);
    return go(latent_prefill_kernel<192, 128>, 192, 128);
}

}  // namespace runit

using namespace runit;

static int32_t latent_check(runit_ctx* ctx, const char* who, const runit_latent_cfg* c, LatentDims* d, uint32_t T) {
    RUNIT_REQUIRE(ctx, c && T > 0 && T <= 65535 && c->heads > 0 && c->dim > 0 && c->rot_dim > 0 && c->rot_dim % 2 == 0 && c->vdim > 0 && c->kv_rank > 0 &&
                           c->kv_rank <= 1024, "%s: bad sizes", who);
    *d = LatentDims{c->heads, c->dim, c->rot_dim, c->vdim, c->kv_rank, c->scale, c->eps};
    return RUNIT_OK;
}

extern "C" {

int32_t runit_latent_query(runit_ctx_t* ctx, const runit_latent_cfg* cfg, int32_t cache_f32, const void* qkv, uint32_t ldq, const void* w_uk,
                           const void* kv_norm, const void* freq, void* cache, void* q_eff, uint32_t T, uint32_t start) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    LatentDims d;
    int32_t st = latent_check(ctx, "latent_query", cfg, &d, T);
    if (st != RUNIT_OK) return st;
    RUNIT_REQUIRE(ctx, qkv && w_uk && freq && cache && q_eff && ldq >= d.q_width() + (kv_norm ? d.kv_rank + d.rot_dim : 0), "latent_query: bad argument");
    return latent_query(ctx, d, cache_f32 != 0, (const float*)qkv, ldq, w_uk, pad8(d.kv_rank), (const float*)kv_norm, (const float*)freq, cache,
                        q_eff, T, LatentPos{nullptr, start});
}

int32_t runit_latent_attention(runit_ctx_t* ctx, const runit_latent_cfg* cfg, int32_t cache_f32, const void* q_eff, const void* cache,
                               void* part_o, void* part_ml, uint32_t nsplit, uint32_t T, uint32_t start) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    LatentDims d;
    int32_t st = latent_check(ctx, "latent_attention", cfg, &d, T);
    if (st != RUNIT_OK) return st;
    RUNIT_REQUIRE(ctx, q_eff && cache && part_o && part_ml && nsplit > 0 && nsplit <= 1024, "latent_attention: bad argument");
    return latent_attention(ctx, d, cache_f32 != 0, q_eff, cache, (float*)part_o, (float*)part_ml, nsplit, T, LatentPos{nullptr, start});
}

int32_t runit_latent_value(runit_ctx_t* ctx, const runit_latent_cfg* cfg, const void* part_o, const void* part_ml, uint32_t nsplit,
                           const void* w_uv, void* out, uint32_t T) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    LatentDims d;
    int32_t st = latent_check(ctx, "latent_value", cfg, &d, T);
    if (st != RUNIT_OK) return st;
    RUNIT_REQUIRE(ctx, part_o && part_ml && w_uv && out && nsplit > 0 && nsplit <= 1024, "latent_value: bad argument");
    return latent_value(ctx, d, (const float*)part_o, (const float*)part_ml, nsplit, w_uv, pad8(d.kv_rank), out, true, d.heads * d.vdim, T);
}

int32_t runit_latent_rows(runit_ctx_t* ctx, const runit_latent_cfg* cfg, int32_t cache_f32, void* qkv, uint32_t ldq, const void* kv_norm,
                          const void* freq, void* cache, uint32_t T, uint32_t start) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    LatentDims d;
    int32_t st = latent_check(ctx, "latent_rows", cfg, &d, T);
    if (st != RUNIT_OK) return st;
    RUNIT_REQUIRE(ctx, qkv && freq && cache && ldq >= d.q_width() + (kv_norm ? d.kv_rank + d.rot_dim : 0), "latent_rows: bad argument");
    return latent_rows(ctx, d, cache_f32 != 0, (float*)qkv, ldq, (const float*)kv_norm, (const float*)freq, cache, T, LatentPos{nullptr, start});
}

int32_t runit_latent_prefill_attention(runit_ctx_t* ctx, const runit_latent_cfg* cfg, const void* q, uint32_t ldq, const void* kv, uint32_t ldkv,
                                       const void* cache, void* out, uint32_t ldo, uint32_t T, uint32_t start) {
    if (!ctx) return RUNIT_ERR_BAD_ARG;
    LatentDims d;
    int32_t st = latent_check(ctx, "latent_prefill_attention", cfg, &d, T);
    if (st != RUNIT_OK) return st;
    RUNIT_REQUIRE(ctx, q && kv && cache && out && ldq >= d.q_width() && ldkv >= d.heads * (d.dim + d.vdim) && ldo >= d.heads * d.vdim,
                  "latent_prefill_attention: bad argument");
    return latent_prefill(ctx, d, (const float*)q, ldq, kv, ldkv, cache, out, ldo, T, start);
}

}  // extern "C"
