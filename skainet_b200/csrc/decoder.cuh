// The decoder runtime every model design runs on: sequences and their positions, one CUDA graph per decode step and
// context-length bucket, chunked prompts, greedy sampling on the device, logits, the bounded-wait flag. A design derives
// from Decoder, owns its weights and caches, and enqueues its layers; the entry points of include/skainet_cuda_llama.h that
// take a model handle work on any of them.
#pragma once
#include "common.cuh"
#include "comm.cuh"
#include "../../include/skainet_cuda_llama.h"

#include <map>
#include <vector>

namespace sk {

struct Decoder {
    // set by the design before decoder_init
    int vocab = 0, d_model = 0, max_seq = 0, max_batch = 0;
    int max_rows = 0;              // rows of one prompt pass (and at least max_batch)
    int tp_rank = 0, tp_world = 1, vocab_l = 0;

    float* logits = nullptr;       // [logits_rows][vocab_l]
    float* logits_full = nullptr;
    int logits_rows = 0;           // rows one enqueue_head call may ask for
    float2* pairs = nullptr;       // arg-max records
    int32_t *cur_token = nullptr, *pos = nullptr, *kv_len = nullptr, *log = nullptr, *log_cursor = nullptr;
    int log_cap = 4096;
    std::vector<int> host_pos;
    cudaStream_t stream = nullptr;
    std::map<std::pair<int, int>, cudaGraphExec_t> graphs;   // (batch, bucket) -> step graph
    bool finalized = false;
    Comm* comm = nullptr;
    bool comm_broken = false;      // a peer wait ran out: the group's inboxes are out of step, the model refuses further steps
    int device = 0;
    int* d_flag = nullptr;         // the device's bounded-wait flag (owned by the library, not by the model)
    int* h_flag = nullptr;         // pinned host copy read after every synchronising call
    uint64_t magic = 0;
    std::vector<void*> owned;      // device allocations freed with the model

    // Zeroed: the tails of activation rows and cache rows are read as zeros and never written.
    int32_t alloc(void** p, size_t bytes);
    template <typename T> int32_t alloc(T** p, size_t count) { return alloc((void**) p, count * sizeof(T)); }

    virtual ~Decoder();
    virtual int32_t finalize() = 0;
    // Row b = next token (cur_token[b]) of sequence b at pos[b]; leaves logits[b]. kv_bound bounds every sequence's length after the step.
    virtual int32_t enqueue_decode(int batch, int kv_bound, cudaStream_t s) = 0;
    // Rows = consecutive tokens (cur_token[0..rows)) of sequence seq from pos[seq].
    virtual int32_t begin_prompt(int seq, cudaStream_t s) { (void) seq; (void) s; return SKAINET_CUDA_OK; }
    virtual int32_t enqueue_prompt(int rows, int seq, int kv_bound, cudaStream_t s) = 0;
    // Logits of n <= logits_rows rows of the prompt pass just enqueued, in the order of `rows` (host), into logits[0..n).
    virtual int32_t enqueue_head(const int32_t* rows, int n, cudaStream_t s) = 0;
    // Seeded noise as the first n positions of a sequence's cache.
    virtual int32_t fill_context(int seq, int n, uint64_t seed) = 0;
    virtual int64_t step_bytes(int batch) const = 0;
    virtual const float* buffer(int which) const = 0;
};

int32_t decoder_init(Decoder* m);                     // allocates what the base owns and registers the handle
skainet_model_t decoder_handle(Decoder* m);
void decoder_destroy(Decoder* m);                     // unregisters and deletes
Decoder* decoder_from_handle(skainet_model_t h);      // nullptr (+ error set) when unknown
int32_t decoder_require_ready(Decoder* m, const char* who);
int32_t flag_fetch(Decoder& m, cudaStream_t s);
int32_t flag_check(Decoder& m);

// A handle of one particular design.
template <typename M>
M* design_from_handle(skainet_model_t h, const char* who) {
    Decoder* d = decoder_from_handle(h);
    M* m = dynamic_cast<M*>(d);
    if (d && !m) set_error("%s: the model handle is of another design", who);
    return m;
}

template <typename T>
inline int32_t dalloc(T** p, size_t count) {
    *p = nullptr;
    if (count == 0) return SKAINET_CUDA_OK;
    SK_CUDA(cudaMalloc((void**) p, count * sizeof(T)));
    return SKAINET_CUDA_OK;
}

}  // namespace sk
