// The token loop of the decoders that keep logits, ids and step state on the device: generate_cancellable
// (ferrum_core/src/llm.rs:733-754) from the logits of a fed prompt on. Shared by every decoder family.
#pragma once
#include "fc_common.cuh"
#include "llama_ops.cuh"

namespace fc {

struct GenCtx {
    cudaStream_t st;
    float* logits; int vocab;
    int* queue; int queue_cap;
    StepState* state;
    unsigned long long* rng_d;     // holds the generator state already
    cudaEvent_t ev0, ev1;
    int* host_pos;
    float* last_ms;
};

// step() runs one decode step with the head; read(StepState*) fetches and checks the device state. n: ids in the queue
// (the prompt); max_new tokens at most. On success *n_out tokens are in out.
template <class Step, class Read>
int generate_tokens(const GenCtx& g, int n, int max_new, const fc_sampling* params, const int32_t* stops, int n_stops, uint64_t* rng_state,
                    const volatile int32_t* cancel, int32_t* out, int* n_out, Step step, Read read) {
    // greedy without a penalty needs neither the sampler's sort nor, without stop ids, the host
    const bool plain_greedy = params->temperature <= 0.0f && params->repetition_penalty == 1.0f;
    const bool free_run = plain_greedy && n_stops == 0 && !cancel;
    FC_CUDA(cudaEventRecord(g.ev0, g.st));
    int made = 0;
    int rc = FC_OK;
    bool cancelled = false, timed = false;
    while (made < max_new) {
        if (cancel && *cancel) { cancelled = true; break; }
        // recent = prompt + tokens so far = the queue (llm.rs:740-751)
        rc = plain_greedy ? launch_llama_pick(g.logits, g.vocab, g.queue, g.queue_cap, g.state, g.st)
                          : launch_sample(g.logits, g.vocab, 0, *params, g.queue, 0, g.rng_d, g.queue, g.queue_cap, g.state,
                                          nullptr, g.st);
        if (rc != FC_OK) break;
        ++made;
        bool stop = false;
        if (!free_run) {
            int32_t tok = 0;
            if (cudaMemcpyAsync(&tok, g.queue + n + made - 1, 4, cudaMemcpyDeviceToHost, g.st) != cudaSuccess ||
                cudaStreamSynchronize(g.st) != cudaSuccess) { rc = fail(FC_E_CUDA, "token download failed"); break; }
            out[made - 1] = tok;
            for (int i = 0; i < n_stops; ++i) stop |= stops[i] == tok;
        }
        if (stop) break;                                     // a stop id is kept in out and not fed (llm.rs:747-749)
        // the forward of the last requested token keeps the cache continuable (llm.rs:750-751); its logits are not used
        // here, so it stays outside the timed region
        if (made == max_new) { FC_CUDA(cudaEventRecord(g.ev1, g.st)); timed = true; }
        rc = step();                                 // forward_one(next), the last token included (llm.rs:750-751)
        if (rc != FC_OK) break;
        *g.host_pos += 1;
    }
    if (rc == FC_OK) {
        if (!timed) FC_CUDA(cudaEventRecord(g.ev1, g.st));
        if (free_run && made > 0) FC_CUDA(cudaMemcpyAsync(out, g.queue + n, (size_t)made * 4, cudaMemcpyDeviceToHost, g.st));
        StepState hs;
        rc = read(&hs);
        if (rc == FC_OK && hs.error) rc = fail(hs.error, "the decode step rejected a token or position on the device");
        if (rc == FC_OK) FC_CUDA(cudaEventElapsedTime(g.last_ms, g.ev0, g.ev1));
    }
    FC_CUDA(cudaMemcpy(rng_state, g.rng_d, 8, cudaMemcpyDeviceToHost));
    if (rc != FC_OK) return rc;
    *n_out = made;
    if (cancelled) return fail(FC_E_CANCELLED, "generation cancelled after %d tokens", made);
    return FC_OK;
}

}  // namespace fc
