// The part of a decoder that does not depend on its architecture: step bookkeeping on the device, recorded command lists,
// the greedy / sampled generate loop and the C entry points that take any runit_model_t (decode_model.cu: OLMoE-shaped with
// Q4_K matrices; layered_model.cu: decoders described layer by layer).
#include "model_core.h"

#include "gemv_stream_host.h"
#include "tma.cuh"

namespace runit {

// After the step: record the produced token, advance position and step.
__global__ void advance_kernel(int32_t* state, const int32_t* argmax_result, int32_t* out_tokens, uint32_t out_cap,
                               int has_logits) {
    grid_dependency_wait();      // inputs come from the previous kernel of the chain
    grid_launch_dependents();
    if (threadIdx.x == 0 && blockIdx.x == 0) {
        const uint32_t step = (uint32_t)state[2];
        if (has_logits) {
            state[0] = argmax_result[0];
            if (step < out_cap) out_tokens[step] = argmax_result[0];
        } else if (step < out_cap) {
            out_tokens[step] = -1;
        }
        state[1] += 1;
        state[2] += 1;
        state[5] = state[2];   // end of the sampler's context range {state[4], state[5]} inside out_tokens
    }
}

int32_t model_dev_alloc(runit_model* m, void** p, size_t bytes) {
    cudaError_t e = cudaMalloc(p, bytes);
    if (e != cudaSuccess) {
        cudaGetLastError();
        return runit_fail(m->ctx, RUNIT_ERR_ALLOC, "model: allocation of %zu bytes failed: %s", bytes, cudaGetErrorString(e));
    }
    m->owned.push_back(*p);
    return RUNIT_OK;
}

static int32_t record_graph(runit_model* m, bool with_logits, cudaGraphExec_t* out, bool sampled = false) {
    runit_ctx* ctx = m->ctx;
    RUNIT_CUDA_TRY(ctx, cudaStreamBeginCapture(ctx->stream, cudaStreamCaptureModeThreadLocal));
    ctx->capturing = true;
    stream_rec_begin(ctx);
    int32_t st = m->issue_step(with_logits, m->forced_cap, sampled);
    ctx->capturing = false;
    cudaGraph_t g = nullptr;
    cudaError_t e = cudaStreamEndCapture(ctx->stream, &g);
    if (st != RUNIT_OK) {
        stream_rec_discard(ctx);
        if (g) cudaGraphDestroy(g);
        return st;
    }
    if (e != cudaSuccess || !g) {
        cudaGetLastError();
        stream_rec_discard(ctx);
        return runit_fail(ctx, RUNIT_ERR_LAUNCH, "model: stream capture failed: %s", cudaGetErrorString(e));
    }
    // adjacent GEMVs of the step (none today: every GEMV of this model is followed by another kind of operator) would share
    // one persistent launch, as in any recorded command list
    st = stream_rec_fuse(ctx, g, &m->owned, nullptr);
    stream_rec_discard(ctx);
    if (st != RUNIT_OK) {
        cudaGraphDestroy(g);
        return st;
    }
    e = cudaGraphInstantiate(out, g, 0);
    cudaGraphDestroy(g);
    if (e != cudaSuccess) return runit_fail(ctx, RUNIT_ERR_LAUNCH, "model: graph instantiate failed: %s", cudaGetErrorString(e));
    return RUNIT_OK;
}

int32_t model_alloc_common(runit_model* m) {
    int32_t st = RUNIT_OK;
    auto A = [&](void** p, size_t b) { if (st == RUNIT_OK) st = model_dev_alloc(m, p, b); };
    m->forced_cap = (uint32_t)m->max_seq;
    m->out_cap = (uint32_t)m->max_seq;
    A((void**)&m->logits, (size_t)m->vocab * 4);
    A((void**)&m->scores, (size_t)m->vocab * 4); A((void**)&m->eos, 64); A((void**)&m->rng, 8);
    A((void**)&m->state, 64); A((void**)&m->forced, (size_t)m->forced_cap * 4); A((void**)&m->out_tokens, (size_t)m->out_cap * 4);
    if (st != RUNIT_OK) return st;
    cudaMemsetAsync(m->forced, 0xFF, (size_t)m->forced_cap * 4, m->ctx->stream);   // nothing forced
    return model_clear_state(m);
}

int32_t model_clear_state(runit_model* m) {
    RUNIT_CUDA_TRY(m->ctx, cudaMemsetAsync(m->state, 0, 64, m->ctx->stream));
    return RUNIT_OK;
}

int32_t model_record(runit_model* m) {
    int32_t st = m->issue_step(true, 0, false);
    if (st == RUNIT_OK) st = runit_flush(m->ctx);
    if (st == RUNIT_OK) st = model_clear_state(m);
    if (st == RUNIT_OK) st = record_graph(m, true, &m->graph_full);
    if (st == RUNIT_OK) st = record_graph(m, false, &m->graph_prompt);
    return st;
}

void model_issue_advance(runit_model* m, bool with_logits) {
    runit_launch_chain(m->ctx, advance_kernel, dim3(1), dim3(32), m->state, m->state + 3, m->out_tokens, m->out_cap, with_logits ? 1 : 0);
}

int32_t model_check_tokens(runit_model* m, const char* who, const int32_t* tokens, uint32_t n) {
    for (uint32_t i = 0; i < n; i++)
        RUNIT_REQUIRE(m->ctx, tokens[i] >= 0 && tokens[i] < m->vocab, "%s: token id %d out of range", who, tokens[i]);
    return RUNIT_OK;
}

// After a batched prefill: the decoder stands at position n with the token the last position produced.
__global__ void prefill_finish_kernel(int32_t* state, int32_t n) {
    if (threadIdx.x == 0) {
        state[0] = state[3];
        state[1] = n;
        state[2] = 0;
        state[5] = 0;
    }
}

int32_t model_finish_prefill(runit_model* m, uint32_t n, int32_t* next_token) {
    runit_ctx* ctx = m->ctx;
    m->cached = n;
    prefill_finish_kernel<<<1, 32, 0, ctx->stream>>>(m->state, (int32_t)n);
    int32_t st = runit_after_launch(ctx, "prefill_finish");
    if (st != RUNIT_OK) return st;
    RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(next_token, m->state, 4, cudaMemcpyDeviceToHost, ctx->stream));
    return runit_flush(ctx);
}

}  // namespace runit

using namespace runit;

int32_t runit_model::forward(const int32_t*, uint32_t, uint32_t, const uint32_t*, uint32_t, float*) {
    return runit_fail(ctx, RUNIT_ERR_UNSUPPORTED, "model_forward: not available on this decoder");
}

int32_t runit_model::check_start(uint32_t) { return RUNIT_OK; }

extern "C" {

int32_t runit_model_destroy(runit_model_t* m) {
    if (!m) return RUNIT_ERR_BAD_ARG;
    cudaStreamSynchronize(m->ctx->stream);
    if (m->graph_full) cudaGraphExecDestroy(m->graph_full);
    if (m->graph_prompt) cudaGraphExecDestroy(m->graph_prompt);
    if (m->graph_sampled) cudaGraphExecDestroy(m->graph_sampled);
    for (void* p : m->owned) cudaFree(p);
    delete m;
    return RUNIT_OK;
}

int32_t runit_model_prefill(runit_model_t* m, const int32_t* tokens, uint32_t n, int32_t* next_token) {
    if (!m) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(m->ctx, tokens && n > 0 && next_token, "model_prefill: null or empty prompt");     // prefill.rs:35-37
    RUNIT_REQUIRE(m->ctx, n <= (uint32_t)m->max_seq, "model_prefill: %u tokens exceed max_seq %d", n, m->max_seq);
    int32_t st = model_check_tokens(m, "model_prefill", tokens, n);                                   // prefill.rs:55-57
    return st == RUNIT_OK ? m->prefill(tokens, n, next_token) : st;
}

int32_t runit_model_forward(runit_model_t* m, const int32_t* tokens, uint32_t n, uint32_t start_pos, const uint32_t* want, uint32_t n_want,
                            float* logits) {
    if (!m) return RUNIT_ERR_BAD_ARG;
    RUNIT_REQUIRE(m->ctx, tokens && n > 0 && (n_want == 0 || (want && logits)), "model_forward: null or empty portion");
    RUNIT_REQUIRE(m->ctx, (uint64_t)start_pos + n <= (uint64_t)m->max_seq, "model_forward: %u tokens from position %u exceed max_seq %d", n,
                  start_pos, m->max_seq);
    for (uint32_t i = 0; i < n_want; i++) RUNIT_REQUIRE(m->ctx, want[i] < n, "model_forward: wanted place %u outside the portion", want[i]);
    int32_t st = model_check_tokens(m, "model_forward", tokens, n);
    return st == RUNIT_OK ? m->forward(tokens, n, start_pos, want, n_want, logits) : st;
}

// Clear the KV position: the next step runs at `pos` with input token `token`.
int32_t runit_model_reset(runit_model_t* m, int32_t token, int32_t pos) {
    if (!m) return RUNIT_ERR_BAD_ARG;
    runit_ctx* ctx = m->ctx;
    RUNIT_REQUIRE(ctx, token >= 0 && token < m->vocab, "model_reset: token id %d out of range", token);   // forward.rs:1804-1806
    RUNIT_REQUIRE(ctx, pos >= 0 && pos < m->max_seq, "model_reset: position %d out of range", pos);
    const int32_t init[4] = {token, pos, 0, 0};
    RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(m->state, init, sizeof(init), cudaMemcpyHostToDevice, ctx->stream));
    RUNIT_CUDA_TRY(ctx, cudaStreamSynchronize(ctx->stream));   // `init` lives on this stack frame
    return RUNIT_OK;
}

// Executor::forward_greedy(token_id, pos, kv) -> next token (forward.rs:1795-1975): one step, synchronous.
int32_t runit_model_forward_greedy(runit_model_t* m, int32_t token_id, int32_t pos, int32_t* next_token) {
    if (!m) return RUNIT_ERR_BAD_ARG;
    runit_ctx* ctx = m->ctx;
    int32_t st = pos > 0 ? m->check_start((uint32_t)pos) : RUNIT_OK;
    if (st == RUNIT_OK) st = runit_model_reset(m, token_id, pos);
    if (st != RUNIT_OK) return st;
    // step 0 must not be forced by a prompt left over from runit_model_generate_greedy
    RUNIT_CUDA_TRY(ctx, cudaMemsetAsync(m->forced, 0xFF, 4, ctx->stream));
    RUNIT_CUDA_TRY(ctx, cudaGraphLaunch(m->graph_full, ctx->stream));
    int32_t tok = -1;
    RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(&tok, m->state, 4, cudaMemcpyDeviceToHost, ctx->stream));
    st = runit_flush(ctx);
    if (st != RUNIT_OK) return st;
    m->cached = (uint32_t)pos + 1;
    if (next_token) *next_token = tok;
    return RUNIT_OK;
}

// Run a prompt of n_prompt known tokens followed by n_gen greedy steps, starting at position start_pos,
// entirely on the device.  out_tokens (host, n_prompt + n_gen entries): out_tokens[i] is the arg-max token
// after step i; prompt steps before the last give -1 when skip_prompt_logits is set (their logits are not
// computed).  The generated continuation is out_tokens[n_prompt-1 ...].  One synchronisation at the end.
static int32_t generate_impl(runit_model_t* m, const int32_t* prompt, uint32_t n_prompt, uint32_t n_gen, int32_t start_pos,
                             int32_t skip_prompt_logits, int32_t* out_tokens, cudaGraphExec_t graph_step);

int32_t runit_model_generate_greedy(runit_model_t* m, const int32_t* prompt, uint32_t n_prompt, uint32_t n_gen,
                                    int32_t start_pos, int32_t skip_prompt_logits, int32_t* out_tokens) {
    if (!m) return RUNIT_ERR_BAD_ARG;
    return generate_impl(m, prompt, n_prompt, n_gen, start_pos, skip_prompt_logits, out_tokens, m->graph_full);
}

int32_t runit_model_generate_sampled(runit_model_t* m, const int32_t* prompt, uint32_t n_prompt, uint32_t n_gen, int32_t start_pos,
                                     const runit_sampler_cfg* cfg, uint64_t seed, const int32_t* eos_ids, uint32_t n_eos,
                                     int32_t* out_tokens) {
    if (!m) return RUNIT_ERR_BAD_ARG;
    runit_ctx* ctx = m->ctx;
    RUNIT_REQUIRE(ctx, cfg && n_eos <= 16 && (eos_ids || n_eos == 0) && n_prompt > 0, "model_generate_sampled: null configuration or more than 16 eos ids");
    RUNIT_REQUIRE(ctx, m->can_sample(), "model_generate_sampled: the expert-parallel decoder is greedy only");
    const bool same = m->graph_sampled && memcmp(&m->sampler_cfg, cfg, sizeof(*cfg)) == 0 && m->sampler_n_eos == n_eos;
    if (!same) {
        RUNIT_CUDA_TRY(ctx, cudaStreamSynchronize(ctx->stream));
        if (m->graph_sampled) cudaGraphExecDestroy(m->graph_sampled);
        m->graph_sampled = nullptr;
        m->sampler_cfg = *cfg;
        m->sampler_n_eos = n_eos;
        // an eager launch of the sampler checks the configuration before it is recorded (its result is discarded)
        int32_t st = runit_sample_f32(ctx, m->logits, m->scores, (uint32_t)m->vocab, &m->sampler_cfg, m->out_tokens, nullptr, 0, 0,
                                      m->eos, 0, m->rng, m->state + 3);
        if (st == RUNIT_OK) st = runit_flush(ctx);
        if (st == RUNIT_OK) st = record_graph(m, true, &m->graph_sampled, true);
        if (st != RUNIT_OK) return st;
    }
    const unsigned long long state0 = runit_sampler_seed_state(seed);
    int32_t eos_host[16] = {0};
    for (uint32_t i = 0; i < n_eos; i++) eos_host[i] = eos_ids[i];
    RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(m->rng, &state0, 8, cudaMemcpyHostToDevice, ctx->stream));
    RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(m->eos, eos_host, 64, cudaMemcpyHostToDevice, ctx->stream));
    RUNIT_CUDA_TRY(ctx, cudaStreamSynchronize(ctx->stream));   // the sources live on this stack frame
    return generate_impl(m, prompt, n_prompt, n_gen, start_pos, 1, out_tokens, m->graph_sampled);
}

static int32_t generate_impl(runit_model_t* m, const int32_t* prompt, uint32_t n_prompt, uint32_t n_gen, int32_t start_pos,
                             int32_t skip_prompt_logits, int32_t* out_tokens, cudaGraphExec_t graph_step) {
    runit_ctx* ctx = m->ctx;
    RUNIT_REQUIRE(ctx, prompt && n_prompt > 0 && out_tokens, "model_generate_greedy: null or empty prompt");
    const uint32_t n_steps = n_prompt + n_gen;
    RUNIT_REQUIRE(ctx, start_pos >= 0 && (uint64_t)start_pos + n_steps <= (uint64_t)m->max_seq,
                  "model_generate_greedy: %u steps from position %d exceed max_seq %d", n_steps, start_pos, m->max_seq);   // kv_cache.rs:63
    RUNIT_REQUIRE(ctx, n_prompt <= m->forced_cap && n_steps <= m->out_cap, "model_generate_greedy: too many steps");
    for (uint32_t i = 0; i < n_prompt; i++)
        RUNIT_REQUIRE(ctx, prompt[i] >= 0 && prompt[i] < m->vocab, "model_generate_greedy: token id %d out of range", prompt[i]);
    if (start_pos > 0) {
        const int32_t ok = m->check_start((uint32_t)start_pos);
        if (ok != RUNIT_OK) return ok;
    }
    RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(m->forced, prompt, (size_t)n_prompt * 4, cudaMemcpyHostToDevice, ctx->stream));
    // the sampler's context range inside out_tokens: from the step that produces the first generated token to the current step
    const int32_t range[2] = {(int32_t)n_prompt - 1, 0};
    RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(m->state + 4, range, sizeof(range), cudaMemcpyHostToDevice, ctx->stream));
    int32_t st = runit_model_reset(m, prompt[0], start_pos);   // synchronises: `range` lives on this stack frame
    if (st != RUNIT_OK) return st;
    // Steps past the prompt are not forced: their entries are negative and the step takes the previous argmax.
    RUNIT_CUDA_TRY(ctx, cudaMemsetAsync(m->forced + n_prompt, 0xFF, (size_t)(m->forced_cap - n_prompt) * 4, ctx->stream));
    for (uint32_t i = 0; i < n_steps; i++) {
        const bool prompt_step = i + 1 < n_prompt;
        cudaGraphExec_t g = (prompt_step && skip_prompt_logits) ? m->graph_prompt : graph_step;
        RUNIT_CUDA_TRY(ctx, cudaGraphLaunch(g, ctx->stream));
        // a bounded wait already gave up (e.g. a rank of the expert-parallel group is missing): stop feeding the stream,
        // the flush below reports it
        if (ctx->h_status && *reinterpret_cast<volatile int32_t*>(ctx->h_status) != 0) break;
    }
    m->cached = (uint32_t)start_pos + n_steps;
    RUNIT_CUDA_TRY(ctx, cudaMemcpyAsync(out_tokens, m->out_tokens, (size_t)n_steps * 4, cudaMemcpyDeviceToHost, ctx->stream));
    return runit_flush(ctx);
}

void* runit_model_logits(runit_model_t* m) { return m ? (void*)m->logits : nullptr; }
uint64_t runit_model_launches_per_token(runit_model_t* m) { return m ? m->launches_per_token() : 0; }

}  // extern "C"
