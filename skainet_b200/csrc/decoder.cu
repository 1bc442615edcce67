// The decoder runtime shared by every model design (contract: decoder.cuh, include/skainet_cuda_llama.h): the step graph with
// greedy sampling, chunked prompts, logits of chosen positions, generation on the device. What a layer computes is the
// design's (llama.cu, tivazen.cu, fomalix.cu).
#include "decoder.cuh"
#include "tma.cuh"

#include <algorithm>
#include <cmath>
#include <cstring>
#include <mutex>
#include <unordered_set>

namespace sk {

// Arg max per row (lowest index on ties) + bookkeeping of the step: the token becomes the next
// step's input, is recorded in the output log, and the sequence position advances.
__global__ void __launch_bounds__(1024)
argmax_advance_kernel(const float* __restrict__ logits, int cols, int32_t* __restrict__ cur_token, int32_t* __restrict__ pos,
                      int32_t* __restrict__ log, int32_t* __restrict__ log_cursor, int batch) {
    __shared__ float sv[32];
    __shared__ int si[32];
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const float* r = logits + (size_t) blockIdx.x * cols;
    float best = -INFINITY; int bi = 0x7fffffff;
    for (int i = threadIdx.x; i < cols; i += blockDim.x) {
        const float v = r[i];
        if (v > best || (v == best && i < bi)) { best = v; bi = i; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(~0u, best, o); const int oi = __shfl_xor_sync(~0u, bi, o);
        if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (lane == 0) { sv[warp] = best; si[warp] = bi; }
    __syncthreads();
    if (warp == 0) {
        const int nw = blockDim.x >> 5;
        best = lane < nw ? sv[lane] : -INFINITY; bi = lane < nw ? si[lane] : 0x7fffffff;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(~0u, best, o); const int oi = __shfl_xor_sync(~0u, bi, o);
            if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
        }
        if (lane == 0) {
            const int tok = bi == 0x7fffffff ? 0 : bi;
            cur_token[blockIdx.x] = tok;
            pos[blockIdx.x] += 1;
            if (log) log[(size_t) log_cursor[0] * batch + blockIdx.x] = tok;
        }
    }
}
__global__ void bump_cursor_kernel(int32_t* cursor) { skd::pdl_launch_dependents(); skd::pdl_wait(); cursor[0] += 1; }

// Row-wise arg max of a vocabulary shard -> (value, global index) pairs, for the TP merge.
__global__ void __launch_bounds__(1024)
argmax_pairs_kernel(const float* __restrict__ logits, int cols, int idx_offset, float* __restrict__ vals, int32_t* __restrict__ idxs) {
    __shared__ float sv[32];
    __shared__ int si[32];
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const float* r = logits + (size_t) blockIdx.x * cols;
    float best = -INFINITY; int bi = 0x7fffffff;
    for (int i = threadIdx.x; i < cols; i += blockDim.x) {
        const float v = r[i];
        if (v > best || (v == best && i < bi)) { best = v; bi = i; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(~0u, best, o); const int oi = __shfl_xor_sync(~0u, bi, o);
        if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (lane == 0) { sv[warp] = best; si[warp] = bi; }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int w = 1; w < (int) (blockDim.x >> 5); ++w)
            if (sv[w] > best || (sv[w] == best && si[w] < bi)) { best = sv[w]; bi = si[w]; }
        vals[blockIdx.x] = best; idxs[blockIdx.x] = (bi == 0x7fffffff ? 0 : bi) + idx_offset;
    }
}
// Arg max of one chunk of a row's logits -> out[chunk][row] as a (value, index) record: with a vocabulary of 128256 one
// CTA per row would scan for tens of microseconds at the end of every step; the chunks of all rows run side by side and
// finish_step_kernel picks among them (lowest index on ties, as the reference's arg max does).
constexpr int ARGMAX_CHUNKS = 32;
__global__ void __launch_bounds__(256)
argmax_chunks_kernel(const float* __restrict__ logits, int cols, int chunk_cols, float2* __restrict__ out, int batch) {
    __shared__ float sv[8];
    __shared__ int si[8];
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int row = blockIdx.x, c0 = blockIdx.y * chunk_cols, c1 = min(cols, c0 + chunk_cols);
    const float* r = logits + (size_t) row * cols;
    float best = -INFINITY; int bi = 0x7fffffff;
    for (int i = c0 + threadIdx.x; i < c1; i += 256) {
        const float v = r[i];
        if (v > best || (v == best && i < bi)) { best = v; bi = i; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(~0u, best, o); const int oi = __shfl_xor_sync(~0u, bi, o);
        if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (lane == 0) { sv[warp] = best; si[warp] = bi; }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int w = 1; w < 8; ++w)
            if (sv[w] > best || (sv[w] == best && si[w] < bi)) { best = sv[w]; bi = si[w]; }
        out[(size_t) blockIdx.y * batch + row] = make_float2(best, __int_as_float(bi));
    }
}
// pairs[world][batch] as (float, int) interleaved 8-byte records -> token per row, then the step's bookkeeping
__global__ void finish_step_kernel(const float2* __restrict__ pairs, int world, int batch, int32_t* __restrict__ cur_token,
                                   int32_t* __restrict__ pos, int32_t* __restrict__ log, const int32_t* __restrict__ log_cursor) {
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b >= batch) return;
    float best = -INFINITY; int bi = 0x7fffffff;
    for (int r = 0; r < world; ++r) {
        const float2 p = pairs[(size_t) r * batch + b];
        const int idx = __float_as_int(p.y);
        if (p.x > best || (p.x == best && idx < bi)) { best = p.x; bi = idx; }
    }
    if (bi == 0x7fffffff) bi = 0;               // no finite logit in the row
    cur_token[b] = bi; pos[b] += 1;
    if (log) log[(size_t) log_cursor[0] * batch + b] = bi;
}
__global__ void pack_pairs_kernel(const float* vals, const int32_t* idxs, float2* out, int n) {
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = make_float2(vals[i], __int_as_float(idxs[i]));
}

__global__ void begin_step_kernel(const int32_t* __restrict__ pos, int32_t* __restrict__ kv_len, int batch) {
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b < batch) kv_len[b] = pos[b] + 1;
}

// ================================================================================================
// handles
// ================================================================================================
static const uint64_t MODEL_MAGIC = 0x534b4d4f44454cull;
static std::mutex g_model_mu;
static std::unordered_set<Decoder*> g_models;

Decoder* decoder_from_handle(skainet_model_t h) {
    Decoder* m = reinterpret_cast<Decoder*>(h);
    std::lock_guard<std::mutex> lk(g_model_mu);
    if (!m || g_models.find(m) == g_models.end() || m->magic != MODEL_MAGIC) {
        set_error("unknown or freed model handle %lld", (long long) h);
        return nullptr;
    }
    return m;
}
skainet_model_t decoder_handle(Decoder* m) { return (skainet_model_t) reinterpret_cast<intptr_t>(m); }

constexpr int HEAD_ROWS = 32;      // positions whose logits one head pass computes

int32_t decoder_init(Decoder* m) {
    SK_REQUIRE(m->max_seq >= 1 && m->max_batch >= 1, "model: max_seq and max_batch must be positive");
    cudaGetDevice(&m->device);
    m->d_flag = device_timeout_flag();          // allocate the per-device flag now: not allowed later inside stream capture
    if (cudaMallocHost((void**) &m->h_flag, sizeof(int)) == cudaSuccess) *m->h_flag = 0; else { cudaGetLastError(); m->h_flag = nullptr; }
    m->host_pos.assign(m->max_batch, 0);
    m->logits_rows = std::max(m->max_batch, HEAD_ROWS);
    m->magic = MODEL_MAGIC;
    { std::lock_guard<std::mutex> lk(g_model_mu); g_models.insert(m); }
    SK_TRY(dalloc(&m->logits, (size_t) m->logits_rows * m->vocab_l));
    if (m->tp_world > 1) SK_TRY(dalloc(&m->logits_full, (size_t) m->max_batch * m->vocab));
    SK_TRY(dalloc(&m->pairs, (size_t) (std::max(ARGMAX_CHUNKS, m->tp_world) + 2) * m->max_batch));
    SK_TRY(dalloc(&m->cur_token, (size_t) std::max(m->max_rows, m->max_batch)));
    SK_TRY(dalloc(&m->pos, m->max_batch)); SK_TRY(dalloc(&m->kv_len, m->max_batch));
    SK_TRY(dalloc(&m->log, (size_t) m->log_cap * m->max_batch)); SK_TRY(dalloc(&m->log_cursor, 1));
    SK_CUDA(cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking));
    SK_CUDA(cudaMemset(m->pos, 0, sizeof(int32_t) * m->max_batch));
    SK_CUDA(cudaMemset(m->log_cursor, 0, sizeof(int32_t)));
    return SKAINET_CUDA_OK;
}

int32_t Decoder::alloc(void** p, size_t bytes) {
    SK_CUDA(cudaMalloc(p, std::max<size_t>(bytes, 16)));
    owned.push_back(*p);
    SK_CUDA(cudaMemset(*p, 0, std::max<size_t>(bytes, 16)));
    return SKAINET_CUDA_OK;
}

Decoder::~Decoder() {
    for (void* p : owned) cudaFree(p);
    for (auto& kv : graphs) cudaGraphExecDestroy(kv.second);
    for (void* p : {(void*) logits, (void*) logits_full, (void*) pairs, (void*) cur_token, (void*) pos, (void*) kv_len, (void*) log, (void*) log_cursor})
        if (p) cudaFree(p);
    comm_destroy(comm);
    if (h_flag) cudaFreeHost(h_flag);
    if (stream) { scratch_release(stream); cudaStreamDestroy(stream); }
    magic = 0;
}

void decoder_destroy(Decoder* m) {
    { std::lock_guard<std::mutex> lk(g_model_mu); g_models.erase(m); }
    delete m;
}

// ================================================================================================
// steps
// ================================================================================================
static int bucket_of(const Decoder& m, int len) {
    int b = 256;
    while (b < len) b <<= 1;
    return std::min(b, m.max_seq);
}

// Enqueues one greedy decode step for sequences 0..batch-1 on s.
static int32_t enqueue_step(Decoder& m, int batch, int kv_bound, cudaStream_t s) {
    begin_step_kernel<<<(batch + 255) / 256, 256, 0, s>>>(m.pos, m.kv_len, batch);
    SK_TRY(m.enqueue_decode(batch, kv_bound, s));
    if (m.tp_world > 1) {
        float* vals = (float*) m.pairs; int32_t* idxs = (int32_t*) (vals + batch);
        float2 *mine = m.pairs + batch, *all = mine + batch;
        SK_CUDA(launch_pdl(argmax_pairs_kernel, dim3(batch), dim3(1024), 0, s, (const float*) m.logits, m.vocab_l, m.tp_rank * m.vocab_l, vals, idxs));
        SK_CUDA(launch_pdl(pack_pairs_kernel, dim3((batch + 255) / 256), dim3(256), 0, s, (const float*) vals, (const int32_t*) idxs, mine, batch));
        SK_TRY(comm_all_gather(m.comm, mine, all, (int64_t) batch * 8, s));
        SK_CUDA(launch_pdl(finish_step_kernel, dim3((batch + 255) / 256), dim3(256), 0, s, (const float2*) all, m.tp_world, batch, m.cur_token, m.pos, m.log, (const int32_t*) m.log_cursor));
    } else if (m.vocab >= 8192) {
        float2* pairs = m.pairs;
        const int chunk_cols = (m.vocab + ARGMAX_CHUNKS - 1) / ARGMAX_CHUNKS;
        SK_CUDA(launch_pdl(argmax_chunks_kernel, dim3(batch, ARGMAX_CHUNKS), dim3(256), 0, s, (const float*) m.logits, m.vocab, chunk_cols, pairs, batch));
        SK_CUDA(launch_pdl(finish_step_kernel, dim3((batch + 255) / 256), dim3(256), 0, s, (const float2*) pairs, ARGMAX_CHUNKS, batch, m.cur_token, m.pos, m.log, (const int32_t*) m.log_cursor));
    } else {
        SK_CUDA(launch_pdl(argmax_advance_kernel, dim3(batch), dim3(1024), 0, s, (const float*) m.logits, m.vocab, m.cur_token, m.pos, m.log, m.log_cursor, batch));
    }
    SK_CUDA(launch_pdl(bump_cursor_kernel, dim3(1), dim3(1), 0, s, m.log_cursor));
    SK_CUDA(cudaGetLastError());
    return SKAINET_CUDA_OK;
}

static int32_t step_graph(Decoder& m, int batch, int bucket, cudaGraphExec_t* out) {
    auto key = std::make_pair(batch, bucket);
    auto it = m.graphs.find(key);
    if (it != m.graphs.end()) { *out = it->second; return SKAINET_CUDA_OK; }
    cudaGraph_t g = nullptr;
    SK_CUDA(cudaStreamBeginCapture(m.stream, cudaStreamCaptureModeThreadLocal));
    const int32_t st = enqueue_step(m, batch, bucket, m.stream);
    cudaError_t e = cudaStreamEndCapture(m.stream, &g);
    if (st != SKAINET_CUDA_OK) { if (g) cudaGraphDestroy(g); return st; }
    if (e != cudaSuccess) return cuda_fail(e, "cudaStreamEndCapture(step)", __FILE__, __LINE__);
    cudaGraphExec_t ge = nullptr;
    e = cudaGraphInstantiate(&ge, g, 0);
    cudaGraphDestroy(g);
    if (e != cudaSuccess) return cuda_fail(e, "cudaGraphInstantiate(step)", __FILE__, __LINE__);
    m.graphs[key] = ge;
    *out = ge;
    return SKAINET_CUDA_OK;
}

static int max_host_pos(const Decoder& m, int batch) {
    int p = 0;
    for (int b = 0; b < batch; ++b) p = std::max(p, m.host_pos[b]);
    return p;
}

static int32_t run_steps(Decoder& m, int batch, int n_steps) {
    for (int i = 0; i < n_steps; ++i) {
        const int need = max_host_pos(m, batch) + 1;
        SK_REQUIRE(need <= m.max_seq, "decode: sequence would exceed max_seq %d", m.max_seq);
        cudaGraphExec_t ge;
        SK_TRY(step_graph(m, batch, bucket_of(m, need), &ge));
        SK_CUDA(cudaGraphLaunch(ge, m.stream));
        for (int b = 0; b < batch; ++b) m.host_pos[b] += 1;
    }
    return SKAINET_CUDA_OK;
}

// The model's device becomes the calling thread's device (flag, SM count and scratch follow it).
static int32_t set_device_of(Decoder& m) { return set_thread_device(m.device); }

// Copies the bounded-wait flag next to the results a call is about to wait for ...
int32_t flag_fetch(Decoder& m, cudaStream_t s) {
    if (m.d_flag && m.h_flag) SK_CUDA(cudaMemcpyAsync(m.h_flag, m.d_flag, sizeof(int), cudaMemcpyDeviceToHost, s));
    return SKAINET_CUDA_OK;
}
// ... and, after the stream has been synchronised, turns a raised flag into SKAINET_CUDA_ERR_TIMEOUT (clearing it).
// A peer wait that ran out leaves the group's inboxes out of step, so the model refuses further steps.
int32_t flag_check(Decoder& m) {
    if (!m.d_flag || !m.h_flag) return SKAINET_CUDA_OK;
    const int v = *m.h_flag;
    if (v == 0) return SKAINET_CUDA_OK;
    *m.h_flag = 0;
    cudaMemsetAsync(m.d_flag, 0, sizeof(int), m.stream);
    if (v == 2) m.comm_broken = true;
    return timeout_status(v);
}

int32_t decoder_require_ready(Decoder* m, const char* who) {
    SK_REQUIRE(m->finalized, "%s: call llama_finalize first", who);
    SK_REQUIRE(m->tp_world == 1 || m->comm != nullptr, "%s: tensor-parallel model without a communicator", who);
    if (m->comm_broken) { set_error("%s: an earlier step gave up waiting for a tensor-parallel peer; rebuild the group (llama_tp_init) before running again", who); return SKAINET_CUDA_ERR_COMM; }
    return set_device_of(*m);
}

// Greedy token after row `row` of the prompt pass just enqueued (no position bookkeeping).
static int32_t sample_row(Decoder& m, int row, int32_t* token_host) {
    cudaStream_t s = m.stream;
    SK_TRY(m.enqueue_head(&row, 1, s));
    const float* full = m.logits;
    if (m.tp_world > 1) {
        SK_TRY(comm_all_gather(m.comm, m.logits, m.logits_full, (int64_t) m.vocab_l * 4, s));
        full = m.logits_full;
    }
    SK_TRY(launch_argmax(full, 1, m.vocab, m.cur_token, s));
    SK_CUDA(cudaMemcpyAsync(token_host, m.cur_token, sizeof(int32_t), cudaMemcpyDeviceToHost, s));
    SK_TRY(flag_fetch(m, s));
    SK_CUDA(cudaStreamSynchronize(s));
    return flag_check(m);
}

static int32_t check_tokens(const Decoder& m, const int32_t* tokens, int n, const char* who) {
    for (int i = 0; i < n; ++i) SK_REQUIRE(tokens[i] >= 0 && tokens[i] < m.vocab, "%s: token %d outside the vocabulary of %d", who, tokens[i], m.vocab);
    return SKAINET_CUDA_OK;
}

// n prompt tokens of a sequence in passes of at most max_rows; after_pass(first token of the pass, rows) runs with the pass
// enqueued and the position not yet advanced on the host.
template <typename F>
static int32_t run_prompt(Decoder* m, int seq, const int32_t* tokens_host, int n, F&& after_pass) {
    cudaStream_t s = m->stream;
    SK_TRY(m->begin_prompt(seq, s));
    for (int done = 0; done < n;) {
        const int rows = std::min(n - done, m->max_rows);
        SK_CUDA(cudaMemcpyAsync(m->cur_token, tokens_host + done, sizeof(int32_t) * rows, cudaMemcpyHostToDevice, s));
        SK_TRY(m->enqueue_prompt(rows, seq, m->host_pos[seq] + rows, s));
        SK_TRY(after_pass(done, rows));
        m->host_pos[seq] += rows;
        SK_CUDA(cudaMemcpyAsync(m->pos + seq, &m->host_pos[seq], sizeof(int32_t), cudaMemcpyHostToDevice, s));
        SK_TRY(flag_fetch(*m, s));
        SK_CUDA(cudaStreamSynchronize(s));     // host_pos/tokens buffers are reused by the next chunk
        SK_TRY(flag_check(*m));
        done += rows;
    }
    return SKAINET_CUDA_OK;
}

}  // namespace sk

using namespace sk;

extern "C" {

int32_t skainet_cuda_llama_free(skainet_model_t h) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    set_device_of(*m);
    cudaStreamSynchronize(m->stream);
    decoder_destroy(m);
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_llama_finalize(skainet_model_t h) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    if (m->finalized) return SKAINET_CUDA_OK;
    SK_TRY(set_device_of(*m));
    SK_TRY(m->finalize());
    SK_CUDA(cudaDeviceSynchronize());
    m->finalized = true;
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_llama_reset(skainet_model_t h) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_TRY(set_device_of(*m));
    SK_CUDA(cudaMemsetAsync(m->pos, 0, sizeof(int32_t) * m->max_batch, m->stream));
    std::fill(m->host_pos.begin(), m->host_pos.end(), 0);
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_llama_prefill(skainet_model_t h, int32_t seq, const int32_t* tokens_host, int32_t n, int32_t* next_token_host) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_TRY(decoder_require_ready(m, "llama_prefill"));
    SK_REQUIRE(seq >= 0 && seq < m->max_batch, "llama_prefill: sequence %d out of range", seq);
    SK_REQUIRE(n >= 0 && (n == 0 || tokens_host), "llama_prefill: bad token array");
    SK_REQUIRE(m->host_pos[seq] + n <= m->max_seq, "llama_prefill: %d + %d tokens exceed max_seq %d", m->host_pos[seq], n, m->max_seq);
    SK_TRY(check_tokens(*m, tokens_host, n, "llama_prefill"));
    int last_rows = 0;
    SK_TRY(run_prompt(m, seq, tokens_host, n, [&](int, int rows) { last_rows = rows; return SKAINET_CUDA_OK; }));
    if (next_token_host && n > 0) SK_TRY(sample_row(*m, last_rows - 1, next_token_host));
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_llama_forward(skainet_model_t h, int32_t seq, const int32_t* tokens_host, int32_t n, const int32_t* want_host, int32_t n_want,
                                   float* logits_host) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_TRY(decoder_require_ready(m, "llama_forward"));
    SK_REQUIRE(m->tp_world == 1, "llama_forward: single-GPU models only");
    SK_REQUIRE(seq >= 0 && seq < m->max_batch, "llama_forward: sequence %d out of range", seq);
    SK_REQUIRE(n >= 0 && (n == 0 || tokens_host), "llama_forward: bad token array");
    SK_REQUIRE(n_want >= 0 && (n_want == 0 || (want_host && logits_host)), "llama_forward: bad list of wanted positions");
    for (int i = 0; i < n_want; ++i) SK_REQUIRE(want_host[i] >= 0 && want_host[i] < n, "llama_forward: wanted position %d outside the %d tokens", want_host[i], n);
    SK_REQUIRE(m->host_pos[seq] + n <= m->max_seq, "llama_forward: %d + %d tokens exceed max_seq %d", m->host_pos[seq], n, m->max_seq);
    SK_TRY(check_tokens(*m, tokens_host, n, "llama_forward"));
    cudaStream_t s = m->stream;
    const size_t V = m->vocab;
    if (n == 1 && seq == 0 && m->host_pos[0] > 0) {          // a decoded token of the first sequence: the captured step
        SK_CUDA(cudaMemcpyAsync(m->cur_token, tokens_host, sizeof(int32_t), cudaMemcpyHostToDevice, s));
        SK_CUDA(cudaMemsetAsync(m->log_cursor, 0, sizeof(int32_t), s));
        SK_TRY(run_steps(*m, 1, 1));
        for (int i = 0; i < n_want; ++i) SK_CUDA(cudaMemcpyAsync(logits_host + i * V, m->logits, sizeof(float) * V, cudaMemcpyDeviceToHost, s));
        SK_TRY(flag_fetch(*m, s));
        SK_CUDA(cudaStreamSynchronize(s));
        return flag_check(*m);
    }
    return run_prompt(m, seq, tokens_host, n, [&](int first, int rows) -> int32_t {
        std::vector<int32_t> at, row;                        // places in want_host that fall into this pass, and their rows
        for (int i = 0; i < n_want; ++i)
            if (want_host[i] >= first && want_host[i] < first + rows) { at.push_back(i); row.push_back(want_host[i] - first); }
        for (size_t b = 0; b < at.size(); b += m->logits_rows) {
            const int k = (int) std::min(at.size() - b, (size_t) m->logits_rows);
            SK_TRY(m->enqueue_head(row.data() + b, k, s));
            for (int i = 0; i < k; ++i)
                SK_CUDA(cudaMemcpyAsync(logits_host + at[b + i] * V, m->logits + i * V, sizeof(float) * V, cudaMemcpyDeviceToHost, s));
            SK_CUDA(cudaStreamSynchronize(s));
        }
        return SKAINET_CUDA_OK;
    });
}

int32_t skainet_cuda_llama_reset_seq(skainet_model_t h, int32_t seq) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_REQUIRE(seq >= 0 && seq < m->max_batch, "llama_reset_seq: sequence %d out of range", seq);
    SK_TRY(set_device_of(*m));
    SK_CUDA(cudaMemsetAsync(m->pos + seq, 0, sizeof(int32_t), m->stream));
    m->host_pos[seq] = 0;
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_llama_fake_prefill(skainet_model_t h, int32_t seq, int32_t n, uint64_t seed) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_TRY(decoder_require_ready(m, "llama_fake_prefill"));
    SK_REQUIRE(seq >= 0 && seq < m->max_batch, "llama_fake_prefill: sequence %d out of range", seq);
    SK_REQUIRE(n >= 0 && n <= m->max_seq, "llama_fake_prefill: %d tokens exceed max_seq %d", n, m->max_seq);
    SK_TRY(m->fill_context(seq, n, seed));
    m->host_pos[seq] = n;
    SK_CUDA(cudaMemcpyAsync(m->pos + seq, &m->host_pos[seq], sizeof(int32_t), cudaMemcpyHostToDevice, m->stream));
    SK_CUDA(cudaStreamSynchronize(m->stream));
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_llama_decode(skainet_model_t h, int32_t batch, const int32_t* tokens_in_host, int32_t* tokens_out_host) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_TRY(decoder_require_ready(m, "llama_decode"));
    SK_REQUIRE(batch >= 1 && batch <= m->max_batch, "llama_decode: batch %d out of range (max %d)", batch, m->max_batch);
    SK_REQUIRE(tokens_in_host && tokens_out_host, "llama_decode: null token array");
    SK_TRY(check_tokens(*m, tokens_in_host, batch, "llama_decode"));
    cudaStream_t s = m->stream;
    SK_CUDA(cudaMemcpyAsync(m->cur_token, tokens_in_host, sizeof(int32_t) * batch, cudaMemcpyHostToDevice, s));
    SK_CUDA(cudaMemsetAsync(m->log_cursor, 0, sizeof(int32_t), s));
    SK_TRY(run_steps(*m, batch, 1));
    SK_CUDA(cudaMemcpyAsync(tokens_out_host, m->cur_token, sizeof(int32_t) * batch, cudaMemcpyDeviceToHost, s));
    SK_TRY(flag_fetch(*m, s));
    SK_CUDA(cudaStreamSynchronize(s));
    return flag_check(*m);
}

int32_t skainet_cuda_llama_generate(skainet_model_t h, int32_t batch, const int32_t* first_tokens_host, int32_t n_steps, int32_t* out_tokens_host) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_TRY(decoder_require_ready(m, "llama_generate"));
    SK_REQUIRE(batch >= 1 && batch <= m->max_batch, "llama_generate: batch %d out of range (max %d)", batch, m->max_batch);
    SK_REQUIRE(n_steps >= 0 && n_steps <= m->log_cap, "llama_generate: %d steps (max %d per call)", n_steps, m->log_cap);
    SK_REQUIRE(first_tokens_host && (n_steps == 0 || out_tokens_host), "llama_generate: null token array");
    SK_TRY(check_tokens(*m, first_tokens_host, batch, "llama_generate"));
    cudaStream_t s = m->stream;
    SK_CUDA(cudaMemcpyAsync(m->cur_token, first_tokens_host, sizeof(int32_t) * batch, cudaMemcpyHostToDevice, s));
    SK_CUDA(cudaMemsetAsync(m->log_cursor, 0, sizeof(int32_t), s));
    SK_TRY(run_steps(*m, batch, n_steps));
    if (n_steps > 0) SK_CUDA(cudaMemcpyAsync(out_tokens_host, m->log, sizeof(int32_t) * (size_t) n_steps * batch, cudaMemcpyDeviceToHost, s));
    SK_TRY(flag_fetch(*m, s));
    SK_CUDA(cudaStreamSynchronize(s));
    return flag_check(*m);
}

int32_t skainet_cuda_llama_logits(skainet_model_t h, int32_t batch, float* logits_host) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_TRY(decoder_require_ready(m, "llama_logits"));
    SK_REQUIRE(batch >= 1 && batch <= m->max_batch && logits_host, "llama_logits: bad arguments");
    cudaStream_t s = m->stream;
    if (m->tp_world == 1) {
        SK_CUDA(cudaMemcpyAsync(logits_host, m->logits, sizeof(float) * (size_t) batch * m->vocab, cudaMemcpyDeviceToHost, s));
        SK_CUDA(cudaStreamSynchronize(s));
        return SKAINET_CUDA_OK;
    }
    SK_TRY(comm_all_gather(m->comm, m->logits, m->logits_full, (int64_t) batch * m->vocab_l * 4, s));
    std::vector<float> tmp((size_t) batch * m->vocab);
    SK_CUDA(cudaMemcpyAsync(tmp.data(), m->logits_full, sizeof(float) * tmp.size(), cudaMemcpyDeviceToHost, s));
    SK_CUDA(cudaStreamSynchronize(s));
    for (int r = 0; r < m->tp_world; ++r)
        for (int b = 0; b < batch; ++b)
            memcpy(logits_host + (size_t) b * m->vocab + (size_t) r * m->vocab_l, tmp.data() + ((size_t) r * batch + b) * m->vocab_l, sizeof(float) * m->vocab_l);
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_llama_step_cost(skainet_model_t h, int32_t batch, int64_t* out2) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_TRY(decoder_require_ready(m, "llama_step_cost"));
    SK_REQUIRE(batch >= 1 && batch <= m->max_batch && out2, "llama_step_cost: bad arguments");
    out2[0] = m->step_bytes(batch);
    cudaGraphExec_t ge;
    SK_TRY(step_graph(*m, batch, bucket_of(*m, max_host_pos(*m, batch) + 1), &ge));
    // kernel nodes of the step graph = launches per step
    cudaGraph_t g = nullptr;
    size_t n = 0;
    int64_t kernels = 0;
#if CUDART_VERSION >= 12000
    (void) g;
#endif
    // Count by re-capturing into a throw-away graph (cheap; the exec graph does not expose its nodes).
    SK_CUDA(cudaStreamBeginCapture(m->stream, cudaStreamCaptureModeThreadLocal));
    const int32_t st = enqueue_step(*m, batch, bucket_of(*m, max_host_pos(*m, batch) + 1), m->stream);
    cudaError_t e = cudaStreamEndCapture(m->stream, &g);
    if (st != SKAINET_CUDA_OK) { if (g) cudaGraphDestroy(g); return st; }
    if (e != cudaSuccess) return cuda_fail(e, "cudaStreamEndCapture(count)", __FILE__, __LINE__);
    SK_CUDA(cudaGraphGetNodes(g, nullptr, &n));
    std::vector<cudaGraphNode_t> nodes(n);
    SK_CUDA(cudaGraphGetNodes(g, nodes.data(), &n));
    for (size_t i = 0; i < n; ++i) {
        cudaGraphNodeType t;
        if (cudaGraphNodeGetType(nodes[i], &t) == cudaSuccess && t == cudaGraphNodeTypeKernel) ++kernels;
    }
    cudaGraphDestroy(g);
    out2[1] = kernels;
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_llama_peek(skainet_model_t h, int32_t which, float* host_out, int64_t n) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_REQUIRE(host_out && n >= 0, "llama_peek: bad arguments");
    SK_TRY(set_device_of(*m));
    const float* src = m->buffer(which);
    SK_REQUIRE(src != nullptr, "llama_peek: unknown buffer %d", which);
    SK_CUDA(cudaStreamSynchronize(m->stream));
    SK_CUDA(cudaMemcpy(host_out, src, sizeof(float) * (size_t) n, cudaMemcpyDeviceToHost));
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_llama_stream(skainet_model_t h, skainet_stream_t* out) {
    Decoder* m = decoder_from_handle(h);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_REQUIRE(out != nullptr, "llama_stream: null output");
    *out = (skainet_stream_t) m->stream;
    return SKAINET_CUDA_OK;
}

}  // extern "C"
