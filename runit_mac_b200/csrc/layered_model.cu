// Decoders described layer by layer (runit_layer_desc): mixers (latent attention with an optional latent borrowed from an earlier
// layer; attention over keys and values per head and / or retention; state-space layers), dense or mixture-of-experts
// feed-forward with a shared block, norms in front of the sublayers or on their outputs, bf16 weights.
//
// The step bookkeeping, command lists, generate loop and sampler are the shared core's (model_core.cu); routing and token
// permutation are those of the other mixture-of-experts blocks (moe_route.cu, moe_permute.cu).  Here: how one decode step and
// one batched portion are issued.
//   Decode step, latent attention: norm + q | latent projection; folded queries + rotation + cache row; split attention over the
//   cached rows; merge + value projection; output projection + residual; then either norm + gate/up + activation and down +
//   residual (dense), or norm + router + top-k, all selected blocks' up + activation, all their downs + residual.  Vectors are
//   f32, weights bf16.
//   The other mixers: projections; attention and state step, or convolution and state step; output projection with the norm of
//   the mixer's groups in front.  A norm on a sublayer's output and the addition to the residual stream happen in front of the
//   next matrix that reads the stream; the stream then moves to the other one of two buffers.
//   Portion: the same with GEMMs; long portions in bf16 expand keys and values of the whole context per layer, the others use
//   the folded arrangement.  A prompt is cut into portions of at most portion_cap tokens.
#include <algorithm>
#include <cmath>
#include <new>
#include <vector>

#include "bf16_ops.cuh"
#include "decode_ops.cuh"
#include "model_core.h"
#include "moe_internal.h"

namespace runit {

struct Layer {
    runit_layer_desc d;
    LatentDims lat;
    uint32_t q_rows;           // rows of w_q
    const float* freq;         // [rot_dim / 2]
    void* cache;               // its own or the lending layer's
    const void* w_uv;          // inside w_ukv
    uint32_t gates;            // rows of the router past the experts
    HeadAttn at;               // RUNIT_MIX_HEADS
    Retention rt;
    Ssm ss;                    // RUNIT_MIX_SSM
    uint32_t out_k;            // columns of w_o
    const HeadAttn* attn() const { return at.heads ? &at : nullptr; }
    const Retention* ret() const { return rt.heads ? &rt : nullptr; }
    // the recurrence of the layer, without its operands
    uint32_t lin_heads() const { return d.mixer == RUNIT_MIX_SSM ? ss.heads : rt.heads; }
    uint32_t lin_dk() const { return d.mixer == RUNIT_MIX_SSM ? ss.state : rt.dim; }
    uint32_t lin_dv() const { return d.mixer == RUNIT_MIX_SSM ? ss.vdim : rt.vdim; }
};

struct LayeredModel : runit_model {
    runit_layered_cfg cfg;
    runit_layered_weights w;
    std::vector<Layer> layers;
    bool exact = false;
    uint32_t depth = 0;             // layers that run
    uint32_t portion_cap = 0;       // tokens of one batched portion
    uint32_t nsplit1 = 1;           // key splits of a decode step
    bool recurrent = false;         // some layer carries a state
    size_t part_cap = 0;            // floats of part1
    uint32_t* tickets = nullptr;
    unsigned long long* argmax_ctl = nullptr;
    uint32_t* counter = nullptr;    // ticket word of the routing launch
    // one token (f32)
    float *x1 = nullptr, *xn1 = nullptr, *qkv1 = nullptr, *qeff1 = nullptr, *po1 = nullptr, *pml1 = nullptr, *ao1 = nullptr, *act1 = nullptr,
          *rl1 = nullptr, *rw1 = nullptr, *gate1 = nullptr, *x2 = nullptr, *y1 = nullptr, *factor1 = nullptr, *squares1 = nullptr, *part1 = nullptr;
    int32_t* idx1 = nullptr;
    uint32_t act_stride = 0;
    // portions (allocated on first use)
    struct {
        float *x = nullptr, *xf = nullptr, *qkv = nullptr, *qeff = nullptr, *po = nullptr, *pml = nullptr, *rl = nullptr, *rw = nullptr,
              *gate = nullptr, *pre = nullptr, *y = nullptr, *logits = nullptr, *out = nullptr, *dt = nullptr;
        void *proj = nullptr, *xbc = nullptr, *states = nullptr;
        void *h = nullptr, *ao = nullptr, *act = nullptr, *kv = nullptr, *xperm = nullptr, *actp = nullptr;
        int32_t *tokens = nullptr, *idx = nullptr, *want = nullptr;
        MoePermutation perm{};
        uint32_t rows_perm = 0, po_rows = 0;
    } pf;
    static constexpr uint32_t kWantRows = 64;       // rows of one head product

    int32_t issue_step(bool with_logits, uint32_t n_forced, bool sampled) override;
    int32_t prefill(const int32_t* tokens, uint32_t n, int32_t* next_token) override;
    int32_t forward(const int32_t* tokens, uint32_t n, uint32_t start_pos, const uint32_t* want, uint32_t n_want, float* logits_host) override;
    uint64_t launches_per_token() override;
    int32_t check_start(uint32_t pos) override;

    GemvDesc head_product(const float* x) const;
    int32_t alloc_portions();
    int32_t in_rows(const Layer& l, uint32_t T);
    int32_t out_rows(const Layer& l, uint32_t T);
    int32_t heads_mixer_rows(const Layer& l, uint32_t T, uint32_t start);
    int32_t ssm_mixer_rows(const Layer& l, uint32_t T, uint32_t start);
    int32_t portion(const int32_t* tokens, uint32_t T, uint32_t start);
    int32_t latent_mixer_rows(const Layer& l, uint32_t T, uint32_t start);
    int32_t ff_rows(const Layer& l, uint32_t T);
    size_t es() const { return exact ? 4 : 2; }
    uint32_t width() const { return (uint32_t)cfg.width; }
    uint32_t ldw() const { return pad8(width()); }
    // long portions in bf16 expand keys and values; in 32-bit and for short portions the folded form reads less
    bool expands(const Layer& l, uint32_t T) const { return !exact && T >= 32 && latent_prefill_supported(l.lat); }
};

static uint32_t up_rows(const runit_layer_desc& d, uint32_t ff) { return d.ff_act == RUNIT_ACT_SILU_GLU ? 2 * ff : ff; }
static int act_epi(const runit_layer_desc& d) { return d.ff_act == RUNIT_ACT_SILU_GLU ? EPI_SILU_GLU : EPI_RELU2; }

int32_t LayeredModel::issue_step(bool with_logits, uint32_t n_forced, bool sampled) {
    int32_t st;
    const LatentPos pos{state + 1, 0};
    const uint32_t wd = width();
    float *x = x1, *x_other = x2;                     // the residual stream; with norms on the outputs it changes buffers
    const float *y = nullptr, *y_gain = nullptr;      // a sublayer's output that is still to be normed and added
    // the vector a sublayer's first matrix reads
    auto enter = [&](GemvDesc& g, const void* gain) {
        g.x = x;
        g.eps = cfg.eps;
        if (!cfg.post_norm) {
            g.gain = (const float*)gain;
        } else if (y) {
            g.pro.kind = GEMV_PRO_RESIDUAL;
            // the stream was last written two launches or more before this one (by the matrix that entered the sublayer)
            g.pro.y = y; g.pro.y_gain = y_gain; g.pro.x_out = x_other; g.pro.early = true;
            std::swap(x, x_other);
            y = nullptr;
        }
    };
    // where the last matrix of a sublayer leaves its product
    auto leave = [&](float*& out, const float*& res, const void* gain) {
        if (cfg.post_norm) {
            out = y1;
            y = y1;
            y_gain = (const float*)gain;
        } else {
            out = x;
            res = x;
        }
    };
    if ((st = embed_norm_rows(ctx, w.embed, ldw(), nullptr, state, forced, n_forced, (uint32_t)vocab, (const float*)w.embed_norm, cfg.eps, x, 1, wd,
                              cfg.embed_scale)))
        return st;
    for (uint32_t i = 0; i < depth; i++) {
        const Layer& l = layers[i];
        const runit_layer_desc& d = l.d;
        GemvDesc g;
        g.w = d.w_q; g.rows = l.q_rows; g.K = wd; g.ldw = ldw(); g.out = qkv1;
        enter(g, d.norm1);
        if ((st = gemv_bf16(ctx, "layer_qkv", g))) return st;
        g = GemvDesc();
        g.w = d.w_o; g.rows = wd; g.K = l.out_k; g.ldw = pad8(l.out_k); g.x = ao1; g.eps = cfg.eps;
        if (d.mixer == RUNIT_MIX_HEADS) {
            if ((st = heads_step(ctx, l.attn(), l.ret(), exact, qkv1, ao1, factor1, squares1, part1, tickets, l.at.heads ? heads_step_splits(ctx, l.at, 1) : 1,
                                 state + 1)))
                return st;
            if (l.rt.heads) {
                g.pro.kind = GEMV_PRO_GROUPS;
                g.pro.plain = l.at.out_rows(); g.pro.group = l.rt.vdim; g.pro.factor = factor1;
                g.pro.squares = squares1; g.pro.squares_n = (l.rt.vdim + 31) / 32;
            }
        } else if (d.mixer == RUNIT_MIX_SSM) {
            if ((st = ssm_step(ctx, l.ss, qkv1, ao1, squares1, state + 1))) return st;
            g.pro.kind = GEMV_PRO_GROUPS;
            g.pro.group = l.ss.inner() / l.ss.norm_groups; g.pro.factor = l.ss.norm; g.pro.factor_early = true;
            if (g.pro.group % l.ss.vdim == 0) {       // whole heads
                g.pro.squares = squares1; g.pro.squares_n = g.pro.group / l.ss.vdim * ((l.ss.vdim + 31) / 32);
            }
        } else {
            const uint32_t ldk = pad8(l.lat.kv_rank);
            if ((st = latent_query(ctx, l.lat, exact, qkv1, 0, d.w_ukv, ldk, (const float*)d.kv_norm, l.freq, l.cache, qeff1, 1, pos))) return st;
            if ((st = latent_attention(ctx, l.lat, exact, qeff1, l.cache, po1, pml1, nsplit1, 1, pos))) return st;
            if ((st = latent_value(ctx, l.lat, po1, pml1, nsplit1, l.w_uv, ldk, ao1, true, 0, 1))) return st;
        }
        leave(g.out, g.res, d.norm1);
        if ((st = gemv_bf16(ctx, "layer_out", g))) return st;
        if (d.ff_kind == RUNIT_FF_DENSE) {
            g = GemvDesc();
            g.w = d.ff_up; g.rows = up_rows(d, d.ff); g.K = wd; g.ldw = ldw(); g.out = act1; g.epi = act_epi(d);
            enter(g, d.norm2);
            if ((st = gemv_bf16(ctx, "layer_up", g))) return st;
            g = GemvDesc();
            g.w = d.ff_down; g.rows = wd; g.K = d.ff; g.ldw = pad8(d.ff); g.x = act1;
            leave(g.out, g.res, d.norm2);
            if ((st = gemv_bf16(ctx, "layer_down", g))) return st;
        } else if (d.ff_kind == RUNIT_FF_MOE) {
            const uint32_t E = d.n_experts, k = d.top_k;
            if ((st = moe_route_gated(ctx, (const float*)d.router, x, rl1, E + l.gates, E, wd, k, d.score, d.renorm, idx1, rw1, gate1, counter,
                                      (const float*)d.norm2, cfg.eps, xn1)))
                return st;
            g = GemvDesc();
            g.w = d.ff_up; g.rows = up_rows(d, d.ff); g.K = wd; g.ldw = ldw(); g.x = xn1; g.out = act1; g.epi = act_epi(d);
            g.n_routed = k; g.slot_stride = act_stride; g.slot_expert = idx1; g.pre = rw1;
            if (d.shared_ff) { g.w_extra = d.shared_up; g.rows_extra = up_rows(d, d.shared_ff); g.post_extra = gate1; }
            if ((st = gemv_bf16(ctx, "layer_experts_up", g))) return st;
            GemvSumDesc s;
            s.w = d.ff_down; s.rows = wd; s.K = d.ff; s.ldw = pad8(d.ff); s.n_routed = k; s.x_stride = act_stride; s.slot_expert = idx1;
            if (d.shared_ff) { s.w_extra = d.shared_down; s.K_extra = d.shared_ff; s.ldw_extra = pad8(d.shared_ff); }
            s.x = act1; s.res = x; s.out = x;
            if ((st = gemv_bf16_sum(ctx, "layer_experts_down", s))) return st;
        }
    }
    if (with_logits) {
        GemvDesc g = head_product(x);
        if (cfg.post_norm) { g.pro.y = y; g.pro.y_gain = y_gain; g.pro.early = true; }
        if (!sampled) { g.argmax = state + 3; g.argmax_ctl = argmax_ctl; }
        if ((st = gemv_bf16(ctx, "layer_head", g))) return st;
        // the context of the draw: what has been generated so far, out_tokens[state[4] .. state[5])
        if (sampled && (st = runit_sample_f32(ctx, logits, scores, (uint32_t)vocab, &sampler_cfg, out_tokens, state + 4, 0, 0, eos, sampler_n_eos, rng,
                                              state + 3)))
            return st;
    }
    model_issue_advance(this, with_logits);
    return runit_after_launch(ctx, "advance");
}

// Final norm and head on one row of the residual stream.
GemvDesc LayeredModel::head_product(const float* x) const {
    GemvDesc g;
    g.w = w.head; g.rows = (uint32_t)vocab; g.K = width(); g.ldw = ldw(); g.x = x; g.eps = cfg.eps; g.out = logits; g.cap = cfg.logit_cap;
    if (cfg.post_norm) {
        g.pro.kind = GEMV_PRO_RESIDUAL;
        g.pro.gain = (const float*)w.final_norm;
    } else {
        g.gain = (const float*)w.final_norm;
    }
    return g;
}

int32_t LayeredModel::alloc_portions() {
    if (pf.x) return RUNIT_OK;
    int32_t st = RUNIT_OK;
    auto A = [&](void** p, size_t b) {
        if (st == RUNIT_OK && b) st = model_dev_alloc(this, p, b);
        if (st == RUNIT_OK && b) cudaMemsetAsync(*p, 0, b, ctx->stream);       // padding stays finite
    };
    const uint32_t P = portion_cap, wd = width();
    uint32_t q = 0, hv = 0, kvw = 0, ffd = 0, ffe = 0, k = 0, E = 0, heads = 0, cp = 0, pitch = 0, proj = 0, xbc = 0, dt = 0;
    size_t states = 0;
    bool all_expand = true;
    for (const Layer& l : layers) {
        const runit_layer_desc& d = l.d;
        hv = std::max(hv, pad8(l.out_k));
        if (d.mixer == RUNIT_MIX_LATENT) {
            q = std::max(q, l.q_rows);
            kvw = std::max(kvw, pad8(l.lat.heads * (l.lat.dim + l.lat.vdim)));
            heads = std::max(heads, l.lat.heads); cp = std::max(cp, l.lat.cp()); pitch = std::max(pitch, l.lat.pitch());
            all_expand = all_expand && expands(l, 1u << 30);
        } else {
            proj = std::max(proj, pad8(l.q_rows));
            if (l.lin_heads() && !exact) states = std::max(states, linear_chunk_bytes(l.lin_heads(), l.lin_dk(), l.lin_dv(), P));
        }
        if (d.mixer == RUNIT_MIX_SSM) {
            xbc = std::max(xbc, pad8(l.ss.channels()));
            dt = std::max(dt, l.ss.heads);
        }
        if (d.ff_kind == RUNIT_FF_DENSE) ffd = std::max(ffd, pad8(d.ff));
        if (d.ff_kind == RUNIT_FF_MOE) {
            ffe = std::max(ffe, pad8(d.ff)); ffd = std::max(ffd, pad8(d.shared_ff));
            k = std::max(k, (uint32_t)d.top_k); E = std::max(E, (uint32_t)d.n_experts);
        }
    }
    q = (q + 1) & ~1u;
    // rows of the folded arrangement: every portion in 32-bit or with sizes the expanded kernel does not take, else short ones
    const uint32_t fold_T = all_expand ? std::min(P, 32u) : P;
    if (heads) pf.po_rows = fold_T * heads + 16 * (2 * ctx->sm_count + 64);
    A((void**)&pf.tokens, (size_t)P * 4); A((void**)&pf.xf, (size_t)P * wd * 4); A((void**)&pf.qkv, (size_t)P * q * 4);
    A((void**)&pf.qeff, (size_t)fold_T * heads * pitch * 4); A((void**)&pf.po, (size_t)pf.po_rows * cp * 4); A((void**)&pf.pml, (size_t)pf.po_rows * 8);
    A(&pf.h, (size_t)P * ldw() * es()); A(&pf.ao, (size_t)P * hv * es()); A(&pf.act, (size_t)P * ffd * es());
    if (!exact) A(&pf.kv, (size_t)max_seq * kvw * 2);
    A(&pf.proj, (size_t)P * proj * es()); A(&pf.xbc, (size_t)P * xbc * es()); A((void**)&pf.dt, (size_t)P * dt * 4); A(&pf.states, states);
    if (cfg.post_norm) A((void**)&pf.out, (size_t)P * wd * 4);
    A((void**)&pf.logits, (size_t)kWantRows * vocab * 4); A((void**)&pf.want, (size_t)kWantRows * 4);
    if (E) {
        const size_t S = (size_t)P * k;
        pf.rows_perm = ((uint32_t)((S + kMoeRowAlign - 1) / kMoeRowAlign) + E) * kMoeRowAlign;
        const size_t tiles = S / 64 + E + 1;
        A((void**)&pf.rl, (size_t)P * E * 4); A((void**)&pf.idx, S * 4); A((void**)&pf.rw, S * 4); A((void**)&pf.gate, (size_t)P * 4);
        A((void**)&pf.pre, (size_t)pf.rows_perm * 4); A((void**)&pf.y, (size_t)pf.rows_perm * wd * 4);
        A(&pf.xperm, (size_t)pf.rows_perm * ldw() * es()); A(&pf.actp, (size_t)pf.rows_perm * ffe * es());
        A((void**)&pf.perm.counts, 1024); A((void**)&pf.perm.n_tok_tiles, 16); A((void**)&pf.perm.tile_expert, tiles * 4);
        A((void**)&pf.perm.tile_nvalid, tiles * 4); A((void**)&pf.perm.tile_row0, tiles * 4); A((void**)&pf.perm.pos_of_slot, S * 4);
    }
    A((void**)&pf.x, (size_t)P * wd * 4);       // last: its pointer says that all of them are there
    return st;
}

// Projections of the mixer's input (behind the norm in front, when there is one): f32 into pf.qkv for latent attention, else the
// operand type into pf.proj with the step sizes of a state-space layer in f32.
int32_t LayeredModel::in_rows(const Layer& l, uint32_t T) {
    int32_t st;
    const runit_layer_desc& d = l.d;
    if (!cfg.post_norm && (st = norm_rows(ctx, pf.x, nullptr, (const float*)d.norm1, cfg.eps, pf.h, exact, ldw(), nullptr, T, width()))) return st;
    GemmDesc g;
    g.w = d.w_q; g.rows = l.q_rows; g.K = width(); g.ldw = ldw(); g.x = pf.h; g.ldx = ldw(); g.x_rows = portion_cap; g.T = T;
    if (d.mixer == RUNIT_MIX_LATENT) {
        g.out = pf.qkv; g.ldo = (l.q_rows + 1) & ~1u;
    } else {
        g.out = pf.proj; g.ldo = pad8(l.q_rows); g.epi = EPI_CAST;
        if (d.mixer == RUNIT_MIX_SSM) { g.tail = pf.dt; g.tail_from = l.q_rows - l.ss.heads; g.ldt = l.ss.heads; }
    }
    return gemm_bf16(ctx, "rows_qkv", g, exact);
}

// Output projection of the mixer and the residual stream; with a norm on the output also the next matrix's operand rows.
int32_t LayeredModel::out_rows(const Layer& l, uint32_t T) {
    int32_t st;
    const uint32_t wd = width(), ldh = pad8(l.out_k);
    GemmDesc g;
    g.w = l.d.w_o; g.rows = wd; g.K = l.out_k; g.ldw = ldh; g.x = pf.ao; g.ldx = ldh; g.x_rows = portion_cap; g.T = T; g.ldo = wd;
    g.out = cfg.post_norm ? pf.out : pf.x; g.epi = cfg.post_norm ? EPI_F32 : EPI_ADD;
    if ((st = gemm_bf16(ctx, "rows_out", g, exact)) || !cfg.post_norm) return st;
    return add_norm_rows(ctx, pf.x, pf.out, (const float*)l.d.norm1, cfg.eps, nullptr, nullptr, pf.h, exact, ldw(), T, wd);
}

int32_t LayeredModel::heads_mixer_rows(const Layer& l, uint32_t T, uint32_t start) {
    int32_t st;
    const uint32_t ld = pad8(l.q_rows), ldh = pad8(l.out_k);
    auto at = [&](void* p, size_t i) { return (void*)((uint8_t*)p + i * es()); };
    if ((st = heads_rows(ctx, l.attn(), l.ret(), exact, pf.proj, ld, T, start))) return st;
    if (l.at.heads && (st = head_attention_rows(ctx, l.at, exact, pf.proj, ld, pf.ao, ldh, T, start, part1, part_cap, tickets))) return st;
    if (!l.rt.heads) return RUNIT_OK;
    const Retention& r = l.rt;
    const size_t base = l.at.in_rows(), hk = (size_t)r.heads * r.dim, hv = (size_t)r.heads * r.vdim;
    LinearRows d;
    d.heads = d.groups = r.heads; d.dk = r.dim; d.dv = r.vdim;
    d.q = at(pf.proj, base); d.k = at(pf.proj, base + hk); d.v = at(pf.proj, base + 2 * hk); d.ldq = d.ldk = d.ldv = ld;
    d.decay = r.decay; d.log_decay = r.decay + r.heads; d.state = r.state;
    d.out = at(pf.ao, l.at.out_rows()); d.ldo = ldh;
    if ((st = linear_rows(ctx, d, exact, pf.states, T, start))) return st;
    return gated_norm_rows(ctx, exact, d.out, ldh, r.out_rows(), r.vdim, at(pf.proj, base + 2 * hk + hv), ld, false, nullptr, r.out_scale, cfg.eps, T);
}

int32_t LayeredModel::ssm_mixer_rows(const Layer& l, uint32_t T, uint32_t start) {
    int32_t st;
    const Ssm& m = l.ss;
    const uint32_t ld = pad8(l.q_rows), ldx = pad8(m.channels()), ldh = pad8(l.out_k), inner = m.inner();
    auto at = [&](void* p, size_t i) { return (void*)((uint8_t*)p + i * es()); };
    if ((st = ssm_conv_rows(ctx, m, exact, pf.proj, ld, pf.xbc, ldx, pf.dt, T, start))) return st;
    LinearRows d;
    d.heads = m.heads; d.groups = m.groups; d.dk = m.state; d.dv = m.vdim;
    d.v = pf.xbc; d.k = at(pf.xbc, inner); d.q = at(pf.xbc, inner + m.groups * m.state); d.ldq = d.ldk = d.ldv = ldx;
    d.dt = pf.dt; d.log_decay = m.a; d.skip = m.skip; d.state = m.s;
    d.out = pf.ao; d.ldo = ldh;
    if ((st = linear_rows(ctx, d, exact, pf.states, T, start))) return st;
    return gated_norm_rows(ctx, exact, pf.ao, ldh, inner, inner / m.norm_groups, pf.proj, ld, true, m.norm, 1.f, cfg.eps, T);
}

int32_t LayeredModel::latent_mixer_rows(const Layer& l, uint32_t T, uint32_t start) {
    int32_t st;
    const runit_layer_desc& d = l.d;
    const uint32_t ldk = pad8(l.lat.kv_rank), ldh = pad8(l.out_k), ldq = (l.q_rows + 1) & ~1u;
    const LatentPos pos{nullptr, start};
    if (expands(l, T)) {
        if ((st = latent_rows(ctx, l.lat, false, pf.qkv, ldq, (const float*)d.kv_norm, l.freq, l.cache, T, pos))) return st;
        const uint32_t kvw = l.lat.heads * (l.lat.dim + l.lat.vdim), S = start + T;
        GemmDesc g;
        g.w = d.w_ukv; g.rows = kvw; g.K = l.lat.kv_rank; g.ldw = ldk; g.x = l.cache; g.ldx = l.lat.pitch(); g.x_rows = (uint32_t)max_seq; g.T = S;
        g.out = pf.kv; g.ldo = pad8(kvw); g.epi = EPI_CAST;
        if ((st = gemm_bf16(ctx, "rows_expand", g, false))) return st;
        return latent_prefill(ctx, l.lat, pf.qkv, ldq, pf.kv, pad8(kvw), l.cache, pf.ao, ldh, T, start);
    }
    uint32_t ns = latent_splits(ctx, l.lat, exact, T);
    while (ns > 1 && (uint64_t)ns * T * l.lat.heads > pf.po_rows) ns--;
    if ((st = latent_query(ctx, l.lat, exact, pf.qkv, ldq, d.w_ukv, ldk, (const float*)d.kv_norm, l.freq, l.cache, pf.qeff, T, pos))) return st;
    if ((st = latent_attention(ctx, l.lat, exact, pf.qeff, l.cache, pf.po, pf.pml, ns, T, pos))) return st;
    return latent_value(ctx, l.lat, pf.po, pf.pml, ns, l.w_uv, ldk, pf.ao, exact, ldh, T);
}

int32_t LayeredModel::ff_rows(const Layer& l, uint32_t T) {
    const runit_layer_desc& d = l.d;
    if (d.ff_kind == RUNIT_FF_NONE) return RUNIT_OK;
    int32_t st;
    const uint32_t wd = width();
    const bool moe = d.ff_kind == RUNIT_FF_MOE;
    const float* gate_row = moe && d.shared_ff ? (const float*)d.router + (size_t)d.n_experts * wd : nullptr;
    if (!cfg.post_norm &&
        (st = norm_rows(ctx, pf.x, nullptr, (const float*)d.norm2, cfg.eps, pf.h, exact, ldw(), moe ? pf.xf : nullptr, T, wd, gate_row, pf.gate)))
        return st;
    auto block = [&](const void* up, const void* down, uint32_t ff, const float* post) -> int32_t {
        GemmDesc g;
        g.w = up; g.rows = up_rows(d, ff); g.K = wd; g.ldw = ldw(); g.x = pf.h; g.ldx = ldw(); g.x_rows = portion_cap; g.T = T;
        g.out = pf.act; g.ldo = pad8(ff); g.epi = act_epi(d); g.post = post;
        if ((st = gemm_bf16(ctx, "rows_up", g, exact))) return st;
        g = GemmDesc();
        g.w = down; g.rows = wd; g.K = ff; g.ldw = pad8(ff); g.x = pf.act; g.ldx = pad8(ff); g.x_rows = portion_cap; g.T = T; g.ldo = wd;
        g.out = cfg.post_norm ? pf.out : pf.x; g.epi = cfg.post_norm ? EPI_F32 : EPI_ADD;
        if ((st = gemm_bf16(ctx, "rows_down", g, exact)) || !cfg.post_norm) return st;
        return add_norm_rows(ctx, pf.x, pf.out, (const float*)d.norm2, cfg.eps, nullptr, nullptr, pf.h, exact, ldw(), T, wd);
    };
    if (!moe) return block(d.ff_up, d.ff_down, d.ff, nullptr);
    const uint32_t E = d.n_experts, k = d.top_k, S = T * k;
    if ((st = moe_router(ctx, (const float*)d.router, pf.xf, pf.rl, E, wd, T))) return st;
    if ((st = moe_topk_rows(ctx, pf.rl, 0, E, E, k, d.score, d.renorm, T, pf.idx, pf.rw))) return st;
    if (d.shared_ff && (st = block(d.shared_up, d.shared_down, d.shared_ff, pf.gate))) return st;
    const uint32_t tt = gemm_bf16_tile_tok(S / E, exact);
    if ((st = moe_permute(ctx, pf.idx, S, E, tt, pf.perm))) return st;
    if ((st = moe_gather_rows(ctx, pf.h, pf.perm.pos_of_slot, pf.xperm, S, (size_t)ldw() * es(), k))) return st;
    if ((st = moe_gather_values(ctx, pf.rw, pf.perm.pos_of_slot, pf.pre, S))) return st;
    GemmDesc g;
    g.n_experts = E; g.T = S; g.x_rows = pf.rows_perm; g.tile_tok = tt; g.max_tiles = S / tt + E;
    g.tile_expert = pf.perm.tile_expert; g.tile_nvalid = pf.perm.tile_nvalid; g.tile_row0 = pf.perm.tile_row0; g.n_tok_tiles = pf.perm.n_tok_tiles;
    g.w = d.ff_up; g.rows = up_rows(d, d.ff); g.K = wd; g.ldw = ldw(); g.x = pf.xperm; g.ldx = ldw(); g.out = pf.actp; g.ldo = pad8(d.ff);
    g.epi = act_epi(d); g.pre = pf.pre;
    if ((st = gemm_bf16(ctx, "rows_experts_up", g, exact))) return st;
    g.w = d.ff_down; g.rows = wd; g.K = d.ff; g.ldw = pad8(d.ff); g.x = pf.actp; g.ldx = pad8(d.ff); g.out = pf.y; g.ldo = wd; g.epi = EPI_F32; g.pre = nullptr;
    if ((st = gemm_bf16(ctx, "rows_experts_down", g, exact))) return st;
    return moe_grouped_combine(ctx, pf.y, pf.perm.pos_of_slot, nullptr, pf.x, pf.x, T, wd, k);
}

// One batched portion at positions start .. start + T - 1; the residual stream of its tokens is left in pf.x.
int32_t LayeredModel::portion(const int32_t* tokens, uint32_t T, uint32_t start) {
    int32_t st;
    RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(pf.tokens, tokens, (size_t)T * 4, cudaMemcpyHostToDevice, ctx->stream));
    if ((st = embed_norm_rows(ctx, w.embed, ldw(), pf.tokens, nullptr, nullptr, 0, (uint32_t)vocab, (const float*)w.embed_norm, cfg.eps, pf.x, T, width(),
                              cfg.embed_scale)))
        return st;
    if (cfg.post_norm && (st = add_norm_rows(ctx, pf.x, nullptr, nullptr, cfg.eps, nullptr, nullptr, pf.h, exact, ldw(), T, width()))) return st;
    for (uint32_t i = 0; i < depth; i++) {
        const Layer& l = layers[i];
        if ((st = in_rows(l, T))) return st;
        switch (l.d.mixer) {
            case RUNIT_MIX_HEADS: st = heads_mixer_rows(l, T, start); break;
            case RUNIT_MIX_SSM: st = ssm_mixer_rows(l, T, start); break;
            default: st = latent_mixer_rows(l, T, start); break;
        }
        if (st || (st = out_rows(l, T)) || (st = ff_rows(l, T))) return st;
    }
    cached = start + T;
    return RUNIT_OK;
}

int32_t LayeredModel::prefill(const int32_t* tokens, uint32_t n, int32_t* next_token) {
    int32_t st = alloc_portions();
    if (st != RUNIT_OK) return st;
    uint32_t last = 0;
    for (uint32_t i = 0; i < n; i += portion_cap) {
        last = std::min(portion_cap, n - i);
        if ((st = portion(tokens + i, last, i))) return st;
    }
    // final norm + head on the last position only, through the decode path's launch
    GemvDesc g = head_product(pf.x + (size_t)(last - 1) * width());
    g.argmax = state + 3; g.argmax_ctl = argmax_ctl;
    if ((st = gemv_bf16(ctx, "layer_head", g))) return st;
    return model_finish_prefill(this, n, next_token);
}

int32_t LayeredModel::forward(const int32_t* tokens, uint32_t n, uint32_t start_pos, const uint32_t* want, uint32_t n_want, float* logits_host) {
    int32_t st;
    RUNIT_REQUIRE(ctx, start_pos <= cached, "model_forward: position %u, but the cache holds %u", start_pos, cached);
    if (start_pos > 0 && (st = check_start(start_pos))) return st;
    if (n == 1) {       // a decode step: the recorded command list
        if ((st = runit_model_reset(this, tokens[0], (int32_t)start_pos))) return st;
        RUNIT_CUDA_TRY(ctx, cudaMemsetAsync(forced, 0xFF, 4, ctx->stream));     // not forced by an earlier prompt
        RUNIT_CUDA_TRY(ctx, cudaGraphLaunch(n_want ? graph_full : graph_prompt, ctx->stream));
        for (uint32_t i = 0; i < n_want; i++)
            RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(logits_host + (size_t)i * vocab, logits, (size_t)vocab * 4, cudaMemcpyDeviceToHost, ctx->stream));
        cached = start_pos + 1;
        return runit_flush(ctx);
    }
    if ((st = alloc_portions())) return st;
    const uint32_t want_rows = portion_cap < kWantRows ? portion_cap : kWantRows;
    for (uint32_t i = 0; i < n; i += portion_cap) {
        const uint32_t T = std::min(portion_cap, n - i);
        if ((st = portion(tokens + i, T, start_pos + i))) return st;
        // the wanted places of this portion, a few rows at a time (their order in the output is the caller's)
        std::vector<uint32_t> at;
        for (uint32_t j = 0; j < n_want; j++)
            if (want[j] >= i && want[j] < i + T) at.push_back(j);
        for (size_t a = 0; a < at.size(); a += want_rows) {
            const uint32_t m = (uint32_t)std::min<size_t>(want_rows, at.size() - a);
            int32_t rows[kWantRows];
            for (uint32_t j = 0; j < m; j++) rows[j] = (int32_t)(want[at[a + j]] - i);
            RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(pf.want, rows, (size_t)m * 4, cudaMemcpyHostToDevice, ctx->stream));
            if (cfg.post_norm) st = add_norm_rows(ctx, pf.x, nullptr, nullptr, cfg.eps, pf.want, (const float*)w.final_norm, pf.h, exact, ldw(), m, width());
            else st = norm_rows(ctx, pf.x, pf.want, (const float*)w.final_norm, cfg.eps, pf.h, exact, ldw(), nullptr, m, width());
            if (st) return st;
            GemmDesc g;
            g.w = w.head; g.rows = (uint32_t)vocab; g.K = width(); g.ldw = ldw(); g.x = pf.h; g.ldx = ldw(); g.x_rows = portion_cap; g.T = m;
            g.out = pf.logits; g.ldo = (uint32_t)vocab; g.cap = cfg.logit_cap;
            if ((st = gemm_bf16(ctx, "rows_head", g, exact))) return st;
            for (uint32_t j = 0; j < m; j++)
                RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(logits_host + (size_t)at[a + j] * vocab, pf.logits + (size_t)j * vocab, (size_t)vocab * 4,
                                                    cudaMemcpyDeviceToHost, ctx->stream));
            if ((st = runit_flush(ctx))) return st;
        }
    }
    return runit_flush(ctx);
}

uint64_t LayeredModel::launches_per_token() {
    uint64_t n = 1 + 2;      // embed + norm; head with its norm and the argmax, advance
    for (uint32_t i = 0; i < depth; i++) n += (layers[i].d.mixer == RUNIT_MIX_LATENT ? 5 : 3) + (layers[i].d.ff_kind == RUNIT_FF_MOE ? 3 : (layers[i].d.ff_kind == RUNIT_FF_DENSE ? 2 : 0));
    return n;
}

// Positions before the last one are gone from a state; a ring keeps the last `cap` positions.
int32_t LayeredModel::check_start(uint32_t pos) {
    if (pos == cached) return RUNIT_OK;
    RUNIT_REQUIRE(ctx, !recurrent, "position %u: a recurrent state stands at %u and continues there or from 0", pos, cached);
    for (const Layer& l : layers)
        if (l.at.heads && l.at.cap < (uint32_t)max_seq) {
            const uint32_t first = pos + 1 > l.at.window ? pos + 1 - l.at.window : 0;
            RUNIT_REQUIRE(ctx, first + l.at.cap >= cached, "position %u: its window has left the cache, which holds the last %u of %u positions", pos,
                          l.at.cap, cached);
        }
    return RUNIT_OK;
}

static int32_t check_heads(runit_ctx* ctx, const runit_layer_desc& d, int32_t i) {
    RUNIT_REQUIRE(ctx, d.at_heads >= 0 && d.rt_heads >= 0 && (d.at_heads || d.rt_heads), "model_create_layered: layer %d: no heads", i);
    if (d.at_heads)
        RUNIT_REQUIRE(ctx, d.at_kv_heads > 0 && d.at_heads % d.at_kv_heads == 0 && d.at_dim > 0 && d.at_dim <= 1024 && d.at_vdim > 0 && d.at_vdim <= 1024 &&
                               d.at_window >= 0 && d.at_kv_heads * ((d.at_heads / d.at_kv_heads + 7) / 8) <= 4096,
                      "model_create_layered: layer %d: bad attention sizes (heads of at most 1024, query heads a multiple of key heads)", i);
    if (d.rt_heads)
        RUNIT_REQUIRE(ctx, d.rt_dim > 0 && d.rt_dim <= 1024 && d.rt_vdim > 0 && d.rt_rot_dims >= 0 && d.rt_rot_dims <= d.rt_dim && d.rt_rot_dims % 2 == 0 &&
                               (d.rt_rot_dims == 0 || d.rt_rot_base > 0.f) && d.rt_decay,
                      "model_create_layered: layer %d: bad retention (dim <= 1024, an even number of rotated dimensions)", i);
    return RUNIT_OK;
}

static int32_t check_ssm(runit_ctx* ctx, const runit_layer_desc& d, int32_t i) {
    RUNIT_REQUIRE(ctx, d.ss_heads > 0 && d.ss_vdim > 0 && d.ss_state > 0 && d.ss_state <= 1024 && d.ss_groups > 0 && d.ss_heads % d.ss_groups == 0 &&
                           d.ss_taps > 0 && d.ss_taps <= 32 && d.ss_norm_groups > 0 && (d.ss_heads * d.ss_vdim) % d.ss_norm_groups == 0,
                  "model_create_layered: layer %d: bad state-space sizes (state <= 1024, taps <= 32, heads a multiple of groups)", i);
    RUNIT_REQUIRE(ctx, d.ss_conv && d.ss_conv_b && d.ss_dt_bias && d.ss_a && d.ss_skip && d.ss_norm, "model_create_layered: layer %d: null pointer", i);
    return RUNIT_OK;
}

static int32_t check_latent(runit_ctx* ctx, const runit_layer_desc* all, int32_t i) {
    const runit_layer_desc& d = all[i];
    RUNIT_REQUIRE(ctx, d.heads > 0 && d.dim > 0 && d.rot_dim > 0 && d.rot_dim % 2 == 0 && d.vdim > 0 && d.kv_rank > 0 && d.kv_rank <= 1024,
                  "model_create_layered: layer %d: bad attention sizes (rot_dim even, kv_rank <= 1024)", i);
    RUNIT_REQUIRE(ctx, d.rot_base > 0.f && d.w_ukv, "model_create_layered: layer %d: null pointer", i);
    if (d.kv_from >= 0) {
        RUNIT_REQUIRE(ctx, d.kv_from < i && all[d.kv_from].mixer == RUNIT_MIX_LATENT && all[d.kv_from].kv_from < 0, "model_create_layered: layer %d borrows from layer %d, which has no latent of its own before it", i, d.kv_from);
        const runit_layer_desc& s = all[d.kv_from];
        RUNIT_REQUIRE(ctx, s.kv_rank == d.kv_rank && s.rot_dim == d.rot_dim && s.rot_base == d.rot_base,
                      "model_create_layered: layer %d and the layer it borrows from differ in latent size or rotation", i);
    } else {
        RUNIT_REQUIRE(ctx, d.kv_norm, "model_create_layered: layer %d: null latent norm", i);
    }
    return RUNIT_OK;
}

static int32_t check_layer(runit_ctx* ctx, const runit_layer_desc* all, int32_t i, bool post_norm) {
    const runit_layer_desc& d = all[i];
    int32_t st;
    RUNIT_REQUIRE(ctx, d.mixer >= RUNIT_MIX_LATENT && d.mixer <= RUNIT_MIX_SSM, "model_create_layered: layer %d: unknown mixer %d", i, d.mixer);
    RUNIT_REQUIRE(ctx, d.norm1 && d.w_q && d.w_o, "model_create_layered: layer %d: null pointer", i);
    st = d.mixer == RUNIT_MIX_HEADS ? check_heads(ctx, d, i) : (d.mixer == RUNIT_MIX_SSM ? check_ssm(ctx, d, i) : check_latent(ctx, all, i));
    if (st != RUNIT_OK || d.ff_kind == RUNIT_FF_NONE) return st;
    RUNIT_REQUIRE(ctx, !post_norm || d.ff_kind == RUNIT_FF_DENSE, "model_create_layered: layer %d: norms on the outputs go with a dense feed-forward", i);
    RUNIT_REQUIRE(ctx, d.ff_kind == RUNIT_FF_DENSE || d.ff_kind == RUNIT_FF_MOE, "model_create_layered: layer %d: unknown feed-forward kind %d", i, d.ff_kind);
    RUNIT_REQUIRE(ctx, d.ff_act == RUNIT_ACT_SILU_GLU || d.ff_act == RUNIT_ACT_RELU2, "model_create_layered: layer %d: unknown activation %d", i, d.ff_act);
    RUNIT_REQUIRE(ctx, d.ff > 0 && d.norm2 && d.ff_up && d.ff_down, "model_create_layered: layer %d: bad feed-forward", i);
    if (d.ff_kind == RUNIT_FF_DENSE) return RUNIT_OK;
    RUNIT_REQUIRE(ctx, d.n_experts > 0 && d.n_experts <= 256 && d.top_k > 0 && d.top_k <= d.n_experts && d.top_k <= 32 && d.router,
                  "model_create_layered: layer %d: bad experts (at most 256, top_k at most 32)", i);
    RUNIT_REQUIRE(ctx, d.score == RUNIT_SCORE_SOFTMAX || d.score == RUNIT_SCORE_SIGMOID, "model_create_layered: layer %d: unknown scoring function", i);
    RUNIT_REQUIRE(ctx, d.shared_ff == 0 || (d.shared_ff > 0 && d.shared_up && d.shared_down), "model_create_layered: layer %d: bad shared block", i);
    return RUNIT_OK;
}

}  // namespace runit

using namespace runit;

extern "C" {

int32_t runit_model_create_layered(runit_ctx_t* ctx, const runit_layered_cfg* cfg, const runit_layer_desc* layers,
                                   const runit_layered_weights* weights, runit_model_t** out) {
    if (!ctx || !out) return RUNIT_ERR_BAD_ARG;
    *out = nullptr;
    RUNIT_REQUIRE(ctx, cfg && layers && weights && weights->embed && weights->final_norm && weights->head,
                  "model_create_layered: null configuration or weights");
    const runit_layered_cfg& c = *cfg;
    RUNIT_REQUIRE(ctx, c.n_layers > 0 && c.n_layers <= 1024 && c.width > 0 && c.width <= 12000 && c.vocab > 0 && c.max_seq > 0,
                  "model_create_layered: bad width, depth, vocabulary or length");
    int32_t st;
    for (int32_t i = 0; i < c.n_layers; i++)
        if ((st = check_layer(ctx, layers, i, c.post_norm != 0)) != RUNIT_OK) return st;
    LayeredModel* m = new (std::nothrow) LayeredModel();
    if (!m) return RUNIT_ERR_ALLOC;
    m->ctx = ctx;
    m->cfg = c;
    m->w = *weights;
    m->vocab = c.vocab;
    m->max_seq = c.max_seq;
    m->exact = c.exact != 0;
    m->depth = (uint32_t)c.n_layers;
    m->portion_cap = std::min<uint32_t>((uint32_t)c.max_seq, m->exact ? 256u : 2048u);
    st = model_alloc_common(m);
    auto A = [&](void** p, size_t b) {
        if (st == RUNIT_OK && b) st = model_dev_alloc(m, p, b);
        if (st == RUNIT_OK && b) cudaMemsetAsync(*p, 0, b, ctx->stream);
    };
    size_t q = 0, qe = 0, po = 0, hv = 0, rows = 0, act = 0, routers = 0;
    uint32_t splits = 1;
    // frequencies of a rotation; then (pairs) what their rounding to f32 has left
    auto angles = [&](int32_t dims, float base, bool pairs) -> const float* {
        const int32_t half = dims / 2;
        std::vector<float> f(pairs ? 2 * half : half);
        for (int32_t j = 0; j < half; j++) {
            const double x = std::pow((double)base, -2.0 * j / dims);
            f[j] = (float)x;
            if (pairs) f[half + j] = (float)(x - (double)f[j]);
        }
        float* p = nullptr;
        A((void**)&p, f.size() * 4);
        if (st == RUNIT_OK) {
            cudaMemcpyAsync(p, f.data(), f.size() * 4, cudaMemcpyHostToDevice, ctx->stream);
            cudaStreamSynchronize(ctx->stream);      // f lives in this call
        }
        return p;
    };
    for (int32_t i = 0; i < c.n_layers && st == RUNIT_OK; i++) {
        Layer l{};
        l.d = layers[i];
        const runit_layer_desc& d = l.d;
        l.gates = d.ff_kind == RUNIT_FF_MOE && d.shared_ff ? 1 : 0;
        if (d.mixer == RUNIT_MIX_HEADS) {
            if (d.at_heads) {
                HeadAttn& a = l.at;
                a.heads = d.at_heads; a.kv_heads = d.at_kv_heads; a.dim = d.at_dim; a.vdim = d.at_vdim; a.window = d.at_window; a.unit_qk = d.at_unit_qk != 0;
                a.scale = d.at_scale; a.out_scale = d.at_out_scale; a.eps = c.eps; a.slopes = (const float*)d.at_slopes;
                // a window's positions before a portion, and the portion
                const uint64_t ring = (uint64_t)a.window - 1 + m->portion_cap;
                a.cap = a.window && ring < (uint64_t)c.max_seq ? (uint32_t)ring : (uint32_t)c.max_seq;
                A(&a.kc, (size_t)a.kv_heads * a.cap * a.kd() * m->es());
                A(&a.vc, (size_t)a.kv_heads * a.cap * a.vd() * m->es());
                const size_t one = heads_part_floats(a, heads_step_splits(ctx, a, 1), 1);
                m->part_cap = std::max(m->part_cap, std::max(one, heads_part_floats(a, heads_step_splits(ctx, a, 16), 16)));
            }
            if (d.rt_heads) {
                Retention& r = l.rt;
                r.heads = d.rt_heads; r.dim = d.rt_dim; r.vdim = d.rt_vdim; r.rot_dims = d.rt_rot_dims; r.out_scale = d.rt_out_scale; r.eps = c.eps;
                r.k_scale = (float)(1.0 / std::sqrt((double)r.dim));
                if (r.rot_dims) r.freq = angles(d.rt_rot_dims, d.rt_rot_base, true);
                r.decay = (const float*)d.rt_decay;
                A((void**)&r.state, (size_t)r.heads * r.dim * r.vdim * 4);
                m->recurrent = true;
            }
            l.q_rows = l.at.in_rows() + l.rt.in_rows();
            l.out_k = l.at.out_rows() + l.rt.out_rows();
        } else if (d.mixer == RUNIT_MIX_SSM) {
            Ssm& s = l.ss;
            s.heads = d.ss_heads; s.vdim = d.ss_vdim; s.state = d.ss_state; s.groups = d.ss_groups; s.taps = d.ss_taps; s.norm_groups = d.ss_norm_groups;
            s.eps = c.eps; s.conv_w = (const float*)d.ss_conv; s.conv_b = (const float*)d.ss_conv_b; s.dt_bias = (const float*)d.ss_dt_bias;
            s.a = (const float*)d.ss_a; s.skip = (const float*)d.ss_skip; s.norm = (const float*)d.ss_norm;
            A((void**)&s.s, (size_t)s.heads * s.state * s.vdim * 4);
            A((void**)&s.ring, (size_t)s.taps * s.channels() * 4);
            m->recurrent = true;
            l.q_rows = s.in_rows();
            l.out_k = s.inner();
        } else {
            l.lat = LatentDims{(uint32_t)d.heads, (uint32_t)d.dim, (uint32_t)d.rot_dim, (uint32_t)d.vdim, (uint32_t)d.kv_rank, d.scale, c.eps};
            const bool own = d.kv_from < 0;
            l.q_rows = l.lat.q_width() + (own ? d.kv_rank + d.rot_dim : 0);
            l.out_k = l.lat.heads * l.lat.vdim;
            l.w_uv = (const uint8_t*)d.w_ukv + (size_t)d.heads * d.dim * pad8(d.kv_rank) * 2;
            if (own) A(&l.cache, (size_t)c.max_seq * l.lat.pitch() * m->es());
            else l.cache = m->layers[d.kv_from].cache;
            l.freq = angles(d.rot_dim, d.rot_base, false);
            splits = std::max(splits, latent_splits(ctx, l.lat, m->exact, 1));
            qe = std::max<size_t>(qe, (size_t)d.heads * l.lat.pitch());
            po = std::max<size_t>(po, (size_t)d.heads * l.lat.cp());
            rows = std::max<size_t>(rows, d.heads);
        }
        q = std::max<size_t>(q, l.q_rows);
        hv = std::max<size_t>(hv, l.out_k);
        if (d.ff_kind == RUNIT_FF_DENSE) act = std::max<size_t>(act, d.ff);
        if (d.ff_kind == RUNIT_FF_MOE) {
            const uint32_t stride = pad8((uint32_t)std::max(d.ff, d.shared_ff));
            m->act_stride = std::max(m->act_stride, stride);
            act = std::max<size_t>(act, (size_t)m->act_stride * 34);
            routers = std::max<size_t>(routers, d.n_experts + l.gates);
        }
        m->layers.push_back(l);
    }
    m->nsplit1 = splits;
    A((void**)&m->x1, (size_t)c.width * 4); A((void**)&m->xn1, (size_t)c.width * 4); A((void**)&m->qkv1, q * 4); A((void**)&m->qeff1, qe * 4);
    A((void**)&m->po1, po * splits * 4); A((void**)&m->pml1, rows * splits * 8); A((void**)&m->ao1, hv * 4); A((void**)&m->act1, (act + 8) * 4);
    A((void**)&m->rl1, (routers + 1) * 4); A((void**)&m->rw1, 128); A((void**)&m->gate1, 16); A((void**)&m->idx1, 128); A((void**)&m->counter, 16);
    A((void**)&m->argmax_ctl, 16);
    A((void**)&m->x2, (size_t)c.width * 4); A((void**)&m->y1, (size_t)c.width * 4); A((void**)&m->factor1, hv * 4); A((void**)&m->squares1, hv * 4);
    A((void**)&m->part1, m->part_cap * 4); A((void**)&m->tickets, 4096 * 4);
    if (st == RUNIT_OK) st = model_record(m);
    if (st != RUNIT_OK) {
        runit_model_destroy(m);
        return st;
    }
    *out = m;
    return RUNIT_OK;
}

void* runit_model_residual(runit_model_t* model) {
    LayeredModel* m = dynamic_cast<LayeredModel*>(model);
    return m ? (void*)m->pf.x : nullptr;
}

int32_t runit_model_set_depth(runit_model_t* model, int32_t n_layers) {
    if (!model) return RUNIT_ERR_BAD_ARG;
    LayeredModel* m = dynamic_cast<LayeredModel*>(model);
    RUNIT_REQUIRE(model->ctx, m && n_layers <= m->cfg.n_layers, "model_set_depth: not a layered decoder, or more layers than it has");
    m->depth = n_layers < 0 ? (uint32_t)m->cfg.n_layers : (uint32_t)n_layers;
    return RUNIT_OK;
}

}  // extern "C"
