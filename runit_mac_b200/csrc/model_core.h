// What every decoder of the library shares: the device-resident token / position / step words, the forced-token list, the
// output list, the recorded command lists of one step, the sampler's state and the generate loop (model_core.cu).  A model
// class adds its weights and cache and says how one step and one batched pass are issued.
#pragma once

#include <vector>

#include "runit_internal.h"

struct runit_model {
    runit_ctx* ctx = nullptr;
    int32_t vocab = 0, max_seq = 0;
    int32_t* state = nullptr;   // [0] = token, [1] = pos, [2] = step counter, [3] = argmax, [4..5] = the sampler's context range
    int32_t* forced = nullptr;  // forced input tokens (prompt), n_forced entries
    int32_t* out_tokens = nullptr;
    uint32_t forced_cap = 0, out_cap = 0;
    float* logits = nullptr;    // [vocab] of the last step
    cudaGraphExec_t graph_full = nullptr;    // step with lm_head + argmax
    cudaGraphExec_t graph_prompt = nullptr;  // step without them (prompt positions whose logits nobody reads)
    // sampled decoding: the step with lm_head + sampler, recorded on first use and when the configuration changes
    cudaGraphExec_t graph_sampled = nullptr;
    runit_sampler_cfg sampler_cfg{};
    uint32_t sampler_n_eos = 0;
    float* scores = nullptr;                 // [vocab]
    int32_t* eos = nullptr;                  // [16]
    unsigned long long* rng = nullptr;
    uint32_t cached = 0;                     // positions the cache holds
    std::vector<void*> owned;

    virtual ~runit_model() {}
    // Issue the launches of one decode step on the context's stream.
    virtual int32_t issue_step(bool with_logits, uint32_t n_forced, bool sampled) = 0;
    // The whole prompt in one batched pass from an empty cache.
    virtual int32_t prefill(const int32_t* tokens, uint32_t n, int32_t* next_token) = 0;
    // A portion of a sequence at positions start_pos .. start_pos + n - 1; logits (host) of the wanted places.
    virtual int32_t forward(const int32_t* tokens, uint32_t n, uint32_t start_pos, const uint32_t* want, uint32_t n_want, float* logits_host);
    virtual uint64_t launches_per_token() = 0;
    virtual bool can_sample() const { return true; }
    // Whether the cache and state allow a pass that starts at `pos` (0 always does).
    virtual int32_t check_start(uint32_t pos);
};

namespace runit {
int32_t model_dev_alloc(runit_model* m, void** p, size_t bytes);
// Buffers of the shared part (m->ctx, vocab and max_seq are set).
int32_t model_alloc_common(runit_model* m);
int32_t model_clear_state(runit_model* m);
// One eager step configures every kernel (shared-memory attributes, tensor maps), then the two command lists are recorded.
int32_t model_record(runit_model* m);
// The end of a step: record the produced token, advance position and step (the caller checks the launch).
void model_issue_advance(runit_model* m, bool with_logits);
// The end of a batched pass: the decoder stands at position n with the token in state[3].
int32_t model_finish_prefill(runit_model* m, uint32_t n, int32_t* next_token);
int32_t model_check_tokens(runit_model* m, const char* who, const int32_t* tokens, uint32_t n);

// Input token of a step: from the forced list while it is not negative there, else the last produced one.
__device__ __forceinline__ int32_t model_step_token(const int32_t* state, const int32_t* __restrict__ forced, uint32_t n_forced, uint32_t vocab) {
    const uint32_t step = (uint32_t)state[2];
    int32_t tok = state[0];
    if (step < n_forced) {
        const int32_t f = forced[step];   // negative = this step is not forced
        if (f >= 0) tok = f;
    }
    return (tok < 0 || (uint32_t)tok >= vocab) ? 0 : tok;   // ids are validated on the host; never index out of range
}
}  // namespace runit
