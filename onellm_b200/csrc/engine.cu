// The generation engine shared by the model designs (see engine.h), and its C entry points.
//
// The reference leaves its model class unwritten: src/models/llama/llama.h is empty and
// src/models/llama/llama.cpp:1-50 is a comment outline.  The design-independent part of that outline is here: one
// arena per model, the batch state of a generation (step counter, per-sequence offsets, finished flags), the context
// pass and the decode step around the layers of a design, top-K sampling, the generate loop.
//
// A decode step is captured once per (row-bucket, mode) as a CUDA graph and replayed: the attention and sampling
// kernels read the step counter from device memory.
#include <string.h>

#include <algorithm>

#include "engine.h"

namespace onellm {

// ---- small kernels of the driver ---------------------------------------------------------------------------
// First kernel of every step, launched with a full stream dependency: everything after it sees
// the new step.
__global__ void advance_step_kernel(int* step) { *step += 1; }

// ids[b] = prompt[b * prompt_len + (*step - 1)]; launched with a full stream dependency
__global__ void gather_prompt_ids_kernel(const int* __restrict__ prompt, int prompt_len, const int* __restrict__ step,
                                         int* __restrict__ ids, int B)
{
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b < B) ids[b] = prompt[(size_t)b * prompt_len + (*step - 1)];
}

__device__ __forceinline__ uint64_t splitmix64(uint64_t x)
{
    x += 0x9E3779B97F4A7C15ull;
    x = (x ^ (x >> 30)) * 0xBF58476D1CE4E5B9ull;
    x = (x ^ (x >> 27)) * 0x94D049BB133111EBull;
    return x ^ (x >> 31);
}
// w[i] = mean + std * N(0,1), counter-based (seed, tensor tag, index) so that any slice of a
// tensor can be generated independently: `row_stride`/`col0` describe the slice of a
// [rows, full_cols] tensor this buffer holds.
template <typename T>
__global__ void init_normal_kernel(T* __restrict__ w, size_t rows, size_t cols, size_t full_cols, size_t row0,
                                   size_t col0, uint64_t seed, uint64_t tag, float mean, float std)
{
    const size_t n = rows * cols;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const size_t r = i / cols, c = i % cols;
        const uint64_t gi = (row0 + r) * full_cols + col0 + c;
        const uint64_t h = splitmix64(seed * 0x100000001B3ull + tag * 0x9E3779B1ull + gi);
        const float u1 = ((float)(uint32_t)(h >> 40) + 1.0f) * (1.0f / 16777217.0f);  // (0,1]
        const float u2 = (float)(uint32_t)((h >> 8) & 0xFFFFFFu) * (1.0f / 16777216.0f);
        const float z = sqrtf(-2.0f * logf(u1)) * cospif(2.0f * u2);
        w[i] = from_float<T>(mean + std * z);
    }
}

int init_normal(int dtype, void* w, size_t rows, size_t cols, size_t full_cols, size_t row0, size_t col0, uint64_t seed, uint64_t tag,
                float mean, float std, cudaStream_t st)
{
    const int nb = blocks_for(rows * cols);
    if (dtype == ONELLM_F16) init_normal_kernel<<<nb, 256, 0, st>>>((__half*)w, rows, cols, full_cols, row0, col0, seed, tag, mean, std);
    else if (dtype == ONELLM_BF16) init_normal_kernel<<<nb, 256, 0, st>>>((__nv_bfloat16*)w, rows, cols, full_cols, row0, col0, seed, tag, mean, std);
    else init_normal_kernel<<<nb, 256, 0, st>>>((float*)w, rows, cols, full_cols, row0, col0, seed, tag, mean, std);
    ONELLM_CHECK_LAUNCH();
    return ONELLM_OK;
}

__global__ void half_to_float_kernel(const __half* in, float* out, size_t n)
{
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        out[i] = __half2float(in[i]);
}

// ---- memory ------------------------------------------------------------------------------------------------
void Engine::carve_common(Carver& cv)
{
    const size_t B = max_batch;
    d_ids = cv.take<int>(B);
    d_prompt = cv.take<int>(B * (size_t)max_seq_len);
    d_step = cv.take<int>(4);
    d_step_off = cv.take<int>(B);
    d_out_ids = cv.take<int>(B);
    d_seqlen = cv.take<int>(B);
    d_topk_id = cv.take<int>(B * 64);
    d_bad_id = cv.take<int>(4);
    d_finished = cv.take<unsigned char>(B);
    d_topk_val = cv.take<float>(B * 64);
    d_u = cv.take<float>(B);
    d_skip = cv.take<uint32_t>(skip_table_words((int)B));
    d_cu = cv.take<int>(B + 1);
    d_hist = cv.take<int>(B);
    logits = cv.take_bytes(B * (size_t)vocab * dtype_size(logits_dtype));
}

int Engine::allocate()
{
    Carver sizing{nullptr};
    carve_common(sizing);
    carve(sizing);
    arena_bytes = align_up(sizing.off, 256);
    cudaError_t e = cudaMalloc(&arena, arena_bytes);
    ONELLM_REQUIRE(e == cudaSuccess, ONELLM_ERR_CUDA, "%s: cudaMalloc of %zu bytes failed: %s", design(), arena_bytes, cudaGetErrorString(e));
    Carver real{arena};
    carve_common(real);
    carve(real);
    ONELLM_CUDA(cudaStreamCreateWithFlags(&stream, cudaStreamNonBlocking));
    ONELLM_CUDA(cudaMemsetAsync(arena, 0, arena_bytes, stream));
    ONELLM_CUDA(cudaStreamSynchronize(stream));
    return build_skip_table(d_skip, max_batch, &skip_ok, stream);
}

Engine::~Engine()
{
    if (stream) cudaStreamSynchronize(stream);
    drop_graphs();
    if (stream) cudaStreamDestroy(stream);
    if (arena) cudaFree(arena);
    if (scratch) cudaFree(scratch);
    if (row_logits) cudaFree(row_logits);
    if (d_rows) cudaFree(d_rows);
}

int Engine::ensure_scratch(size_t bytes)
{
    if (bytes <= scratch_bytes) return ONELLM_OK;
    ONELLM_CUDA(cudaStreamSynchronize(stream));
    if (scratch) cudaFree(scratch);
    scratch = nullptr;
    scratch_bytes = 0;
    const cudaError_t e = cudaMalloc(&scratch, bytes);
    ONELLM_REQUIRE(e == cudaSuccess, ONELLM_ERR_CUDA, "%s: cannot allocate %zu bytes of context scratch: %s", design(), bytes, cudaGetErrorString(e));
    scratch_bytes = bytes;
    return ONELLM_OK;
}

void Engine::drop_graphs()
{
    for (auto& kv : graphs) cudaGraphExecDestroy(kv.second);
    graphs.clear();
    graph_nodes.clear();
    warmed.clear();
}

// ---- one decode step ---------------------------------------------------------------------------------------
int Engine::sample(const void* rows)
{
    if (top_k < 1) return ONELLM_OK;
    RC(onellm_topk(logits_dtype, rows, batch, vocab, top_k, d_topk_val, d_topk_id, 0, (void*)stream));
    return topk_sample_launch(d_topk_id, d_topk_val, batch, top_k, temperature, 0, d_step, vocab, eos_id, literal_walk, d_out_ids,
                              d_seqlen, d_finished, d_u, d_ids, /*early_seed=*/true, skip_ok ? d_skip : nullptr, stream);
}

// Enqueues one decode step for `batch` sequences on the stream.  `step_bound` sizes the attention grid; the real
// step is read from d_step on the device.
int Engine::enqueue_step(int mode, int step_bound, int prompt_len)
{
    // The step counter advances first.  This kernel, the id gather and the embedding are
    // launched with full stream dependencies; every later kernel of the step may overlap its
    // predecessor's tail (programmatic dependent launch) and therefore starts after these.
    note_launch();
    (void)prefer_max_shared((const void*)advance_step_kernel);  // same L1 / shared-memory split as every kernel behind it
    (void)prefer_max_shared((const void*)gather_prompt_ids_kernel);
    advance_step_kernel<<<1, 1, 0, stream>>>(d_step);
    if (mode & MODE_GATHER) {
        note_launch();
        gather_prompt_ids_kernel<<<(batch + 127) / 128, 128, 0, stream>>>(d_prompt, prompt_len, d_step, d_ids, batch);
    }
    RC(decode_layers(step_bound, (mode & MODE_HEAD) != 0));
    if (mode & MODE_HEAD) RC(sample(logits));
    ONELLM_CHECK_LAUNCH();
    return ONELLM_OK;
}

// Runs one step (attending cur_len + 1 rows) and advances cur_len.
int Engine::run_step(int mode, int prompt_len)
{
    const int step = cur_len + 1;
    last_logits = logits;
    ONELLM_REQUIRE(step <= max_seq_len, ONELLM_ERR_STATE, "decode: sequence length %d exceeds max_seq_len %d", step,
                   max_seq_len);
    int bound = (step + 255) / 256 * 256;
    bound = std::min({bound, max_seq_len, span_cap});
    if (!use_graphs) {
        const long before = launches_noted();
        RC(enqueue_step(mode, bound, prompt_len));
        launches += launches_noted() - before;
        cur_len++;
        return ONELLM_OK;
    }
    const long key = ((long)bound << 20) | ((long)batch << 8) | ((long)mode << 4) | (top_k > 1 ? 1 : 0);
    // prompt_len, top_k, temperature are baked into the captured nodes: changing them drops the cache
    auto it = graphs.find(key);
    if (it == graphs.end() && !warmed.count(key)) {
        // first step of this shape runs eagerly: the launch planners query occupancy and set
        // function attributes once per kernel, which must not happen inside a stream capture
        warmed[key] = 1;
        const long before = launches_noted();
        RC(enqueue_step(mode, bound, prompt_len));
        launches += launches_noted() - before;
        cur_len++;
        return ONELLM_OK;
    }
    if (it == graphs.end()) {
        const long before = launches_noted();  // what the capture records = the nodes of one replay
        cudaGraph_t g = nullptr;
        ONELLM_CUDA(cudaStreamBeginCapture(stream, cudaStreamCaptureModeThreadLocal));
        const int rc = enqueue_step(mode, bound, prompt_len);
        const cudaError_t e = cudaStreamEndCapture(stream, &g);
        if (rc) {
            if (g) cudaGraphDestroy(g);
            return rc;
        }
        ONELLM_REQUIRE(e == cudaSuccess && g, ONELLM_ERR_CUDA, "graph capture failed: %s", cudaGetErrorString(e));
        cudaGraphExec_t ge = nullptr;
        const cudaError_t e2 = cudaGraphInstantiate(&ge, g, 0);
        cudaGraphDestroy(g);
        ONELLM_REQUIRE(e2 == cudaSuccess, ONELLM_ERR_CUDA, "graph instantiate failed: %s", cudaGetErrorString(e2));
        graph_nodes[key] = (int)(launches_noted() - before);
        it = graphs.emplace(key, ge).first;
    }
    ONELLM_CUDA(cudaGraphLaunch(it->second, stream));
    launches += graph_nodes[key];
    cur_len++;
    return ONELLM_OK;
}

// ---- context phase -----------------------------------------------------------------------------------------
// lens[b] new tokens of sequence b (packed in d_prompt in sequence order) behind the cur_len + seq_off[b] positions it
// has cached: all tokens at once through the design's context kernels, then sampling from the last token of every
// sequence.
int Engine::prefill_context(int B, const int* lens)
{
    ContextBatch c;
    c.B = B;
    std::vector<int> cu(B + 1, 0), hist(B), off(B);
    seq_off.resize(max_batch, 0);
    int new_max = 0;
    for (int b = 0; b < B; b++) {
        hist[b] = cur_len + seq_off[b];
        cu[b + 1] = cu[b] + lens[b];
        c.T += (size_t)lens[b];
        c.P = std::max(c.P, lens[b]);
        new_max = std::max(new_max, hist[b] + lens[b]);
    }
    for (int b = 0; b < B; b++) off[b] = hist[b] + lens[b] - new_max;
    // the rows whose logits are computed: the last one of every sequence, then the ones asked for
    std::vector<int> rows;
    for (int b = 0; b < B; b++) rows.push_back(cu[b + 1] - 1);
    for (int r : want_rows) {
        ONELLM_REQUIRE(r >= 0 && (size_t)r < c.T, ONELLM_ERR_ARG, "want_logits: row %d outside the %zu tokens of this call", r, c.T);
        rows.push_back(r);
    }
    row_have = want_rows.size();
    want_rows.clear();
    c.n_rows = (int)rows.size();
    if (rows.size() > row_cap || !d_rows) {
        ONELLM_CUDA(cudaStreamSynchronize(stream));
        if (d_rows) cudaFree(d_rows);
        if (row_logits) cudaFree(row_logits);
        d_rows = nullptr;
        row_logits = nullptr;
        row_cap = std::max(rows.size(), (size_t)max_batch);
        ONELLM_CUDA(cudaMalloc(&d_rows, row_cap * sizeof(int)));
        if (row_have) ONELLM_CUDA(cudaMalloc(&row_logits, row_cap * vocab * dtype_size(logits_dtype)));
    } else if (row_have && !row_logits) {
        ONELLM_CUDA(cudaMalloc(&row_logits, row_cap * vocab * dtype_size(logits_dtype)));
    }
    c.logits = row_have ? row_logits : logits;
    last_logits = c.logits;
    c.cu = d_cu;
    c.hist = d_hist;
    c.host_hist = hist.data();
    c.rows = d_rows;
    ONELLM_CUDA(cudaMemcpyAsync(d_step_off, off.data(), B * sizeof(int), cudaMemcpyHostToDevice, stream));
    ONELLM_CUDA(cudaMemcpyAsync(d_cu, cu.data(), (B + 1) * sizeof(int), cudaMemcpyHostToDevice, stream));
    ONELLM_CUDA(cudaMemcpyAsync(d_hist, hist.data(), B * sizeof(int), cudaMemcpyHostToDevice, stream));
    ONELLM_CUDA(cudaMemcpyAsync(d_rows, rows.data(), rows.size() * sizeof(int), cudaMemcpyHostToDevice, stream));
    ONELLM_CUDA(cudaStreamSynchronize(stream));  // the host arrays live on this stack frame
    const long before = launches_noted();
    RC(context_layers(c));
    RC(sample(c.logits));  // seeded with the step counter, as the position-by-position path does
    launches += launches_noted() - before;
    for (int b = 0; b < B; b++) seq_off[b] = off[b];
    cur_len = new_max;
    return ONELLM_OK;
}

// The host's side of a context pass: first tokens out, then what the kernels recorded.
int Engine::finish_context(int* host_first_ids, const char* where)
{
    if (host_first_ids) ONELLM_CUDA(cudaMemcpyAsync(host_first_ids, d_out_ids, (size_t)batch * sizeof(int), cudaMemcpyDeviceToHost, stream));
    RC(queue_comm_check());
    ONELLM_CUDA(cudaStreamSynchronize(stream));
    RC(comm_check(where));
    int bad[2] = {0, 0};
    ONELLM_CUDA(cudaMemcpy(bad, d_bad_id, 2 * sizeof(int), cudaMemcpyDeviceToHost));
    ONELLM_REQUIRE(bad[0] == 0, ONELLM_ERR_ARG, "%s: token id outside [0, vocab_size)", where);
    ONELLM_REQUIRE(bad[1] == 0, ONELLM_ERR_STATE, "%s: a position beyond max_seq_len was refused by the cache", where);
    ONELLM_REQUIRE(onellm_gemm_timeout_flag() <= 0, ONELLM_ERR_CUDA, "%s: a tensor-core GEMM block timed out", where);
    return ONELLM_OK;
}

}  // namespace onellm

using namespace onellm;

static Engine* engine_of(onellm_llama* h) { return reinterpret_cast<Engine*>(h); }
static const Engine* engine_of(const onellm_llama* h) { return reinterpret_cast<const Engine*>(h); }

extern "C" int onellm_llama_last_draws(onellm_llama* h, float* host_u, int* host_step, int* table_in_use)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m && host_u, ONELLM_ERR_ARG, "llama_last_draws: null pointer");
    ONELLM_CUDA(cudaMemcpyAsync(host_u, m->d_u, (size_t)m->max_batch * sizeof(float), cudaMemcpyDeviceToHost,
                                m->stream));
    int step = 0;
    ONELLM_CUDA(cudaMemcpyAsync(&step, m->d_step, sizeof(int), cudaMemcpyDeviceToHost, m->stream));
    ONELLM_CUDA(cudaStreamSynchronize(m->stream));
    if (host_step) *host_step = step;
    if (table_in_use) *table_in_use = m->skip_ok;
    return ONELLM_OK;
}

extern "C" void onellm_llama_destroy(onellm_llama* h) { delete engine_of(h); }

extern "C" const char* onellm_model_design(const onellm_llama* h) { return h ? engine_of(h)->design() : ""; }

extern "C" size_t onellm_llama_device_bytes(const onellm_llama* h) { return h ? engine_of(h)->arena_bytes : 0; }

extern "C" void* onellm_llama_stream(onellm_llama* h) { return h ? (void*)engine_of(h)->stream : nullptr; }

extern "C" int onellm_llama_init_random(onellm_llama* h, uint64_t seed, float std)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m, ONELLM_ERR_ARG, "llama_init_random: null handle");
    return m->init_random(seed, std);
}

extern "C" int onellm_llama_set_sampling(onellm_llama* h, int top_k, float temperature, int literal_walk)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m, ONELLM_ERR_ARG, "llama_set_sampling: null handle");
    ONELLM_REQUIRE(top_k >= 0 && top_k <= 64 && temperature > 0.f, ONELLM_ERR_ARG,
                   "llama_set_sampling: top_k in [1,64] (0: logits only), temperature > 0");
    if (top_k != m->top_k || temperature != m->temperature || literal_walk != m->literal_walk) {
        cudaStreamSynchronize(m->stream);
        m->drop_graphs();
    }
    m->top_k = top_k;
    m->temperature = temperature;
    m->literal_walk = literal_walk;
    return ONELLM_OK;
}

extern "C" int onellm_llama_set_prefill_by_decode(onellm_llama* h, int enabled)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m, ONELLM_ERR_ARG, "llama_set_prefill_by_decode: null handle");
    if ((enabled == 2) != m->plain_kernels) {
        ONELLM_CUDA(cudaStreamSynchronize(m->stream));
        m->drop_graphs();
    }
    m->prefill_by_decode = enabled == 1;
    m->plain_kernels = enabled == 2;
    return ONELLM_OK;
}

extern "C" int onellm_llama_set_graphs(onellm_llama* h, int enabled)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m, ONELLM_ERR_ARG, "llama_set_graphs: null handle");
    m->use_graphs = enabled != 0;
    return ONELLM_OK;
}

extern "C" int onellm_llama_prefill(onellm_llama* h, const int* host_ids, int batch, int prompt_len, int* host_first_ids)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m && host_ids, ONELLM_ERR_ARG, "llama_prefill: null pointer");
    ONELLM_REQUIRE(m->weights_ready, ONELLM_ERR_STATE, "llama_prefill: weights not loaded");
    ONELLM_REQUIRE(batch >= 1 && batch <= m->max_batch, ONELLM_ERR_ARG, "llama_prefill: batch %d outside [1,%d]", batch, m->max_batch);
    ONELLM_REQUIRE(prompt_len >= 1 && prompt_len <= m->max_seq_len, ONELLM_ERR_ARG, "llama_prefill: prompt_len %d outside [1,%d]", prompt_len, m->max_seq_len);
    cudaStream_t st = m->stream;
    if (batch != m->batch || prompt_len != m->graph_prompt_len) {
        // batch and prompt length are baked into the captured launches
        ONELLM_CUDA(cudaStreamSynchronize(st));
        m->drop_graphs();
    }
    m->batch = batch;
    m->graph_prompt_len = prompt_len;
    m->cur_len = 0;
    m->seq_off.assign(m->max_batch, 0);
    ONELLM_CUDA(cudaMemsetAsync(m->d_step_off, 0, (size_t)m->max_batch * sizeof(int), st));
    const int first_step = m->prefill_by_decode ? 0 : prompt_len;  // the step kernels increment before use
    ONELLM_CUDA(cudaMemcpyAsync(m->d_prompt, host_ids, (size_t)batch * prompt_len * sizeof(int), cudaMemcpyHostToDevice, st));
    ONELLM_CUDA(cudaMemcpyAsync(m->d_step, &first_step, sizeof(int), cudaMemcpyHostToDevice, st));
    ONELLM_CUDA(cudaMemsetAsync(m->d_seqlen, 0, (size_t)batch * sizeof(int), st));
    ONELLM_CUDA(cudaMemsetAsync(m->d_finished, 0, (size_t)batch, st));
    ONELLM_CUDA(cudaMemsetAsync(m->d_bad_id, 0, 4 * sizeof(int), st));
    ONELLM_CUDA(cudaStreamSynchronize(st));  // `first_step` lives on this stack frame
    if (m->prefill_by_decode) {
        ONELLM_REQUIRE(m->want_rows.empty(), ONELLM_ERR_STATE, "llama_prefill: logits of single rows need the context-phase kernels");
        // one position at a time through the decode kernels; only the last position needs the LM head
        for (int p = 0; p < prompt_len; p++)
            RC(m->run_step(MODE_GATHER | (p == prompt_len - 1 ? MODE_HEAD : 0), prompt_len));
    } else {
        const std::vector<int> lens(batch, prompt_len);
        RC(m->prefill_context(batch, lens.data()));
    }
    return m->finish_context(host_first_ids, "llama_prefill");
}

// Prompts of different lengths: host_ids holds them packed one after the other, lens[b] tokens each.  Sequence b is
// cached in rows 0 .. lens[b]-1 of its cache; the step counter follows the longest sequence and the decode attention
// gives every other sequence its own, shorter, row count and position.
extern "C" int onellm_llama_prefill_ragged(onellm_llama* h, const int* host_ids, const int* lens, int batch, int* host_first_ids)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m && host_ids && lens, ONELLM_ERR_ARG, "llama_prefill_ragged: null pointer");
    ONELLM_REQUIRE(m->weights_ready, ONELLM_ERR_STATE, "llama_prefill_ragged: weights not loaded");
    ONELLM_REQUIRE(batch >= 1 && batch <= m->max_batch, ONELLM_ERR_ARG, "llama_prefill_ragged: batch %d outside [1,%d]", batch, m->max_batch);
    size_t total = 0;
    int longest = 0;
    for (int b = 0; b < batch; b++) {
        ONELLM_REQUIRE(lens[b] >= 1 && lens[b] <= m->max_seq_len, ONELLM_ERR_ARG, "llama_prefill_ragged: lens[%d] = %d outside [1,%d]", b,
                       lens[b], m->max_seq_len);
        total += (size_t)lens[b];
        longest = lens[b] > longest ? lens[b] : longest;
    }
    cudaStream_t st = m->stream;
    ONELLM_CUDA(cudaStreamSynchronize(st));
    if (batch != m->batch) m->drop_graphs();
    m->batch = batch;
    m->cur_len = 0;
    m->seq_off.assign(m->max_batch, 0);
    ONELLM_CUDA(cudaMemcpyAsync(m->d_prompt, host_ids, total * sizeof(int), cudaMemcpyHostToDevice, st));
    ONELLM_CUDA(cudaMemcpyAsync(m->d_step, &longest, sizeof(int), cudaMemcpyHostToDevice, st));
    ONELLM_CUDA(cudaMemsetAsync(m->d_seqlen, 0, (size_t)batch * sizeof(int), st));
    ONELLM_CUDA(cudaMemsetAsync(m->d_finished, 0, (size_t)batch, st));
    ONELLM_CUDA(cudaMemsetAsync(m->d_bad_id, 0, 4 * sizeof(int), st));
    ONELLM_CUDA(cudaStreamSynchronize(st));  // `longest` lives on this stack frame
    RC(m->prefill_context(batch, lens));
    return m->finish_context(host_first_ids, "llama_prefill_ragged");
}

// A further turn: n_new more tokens per sequence behind the cur_len positions already cached (history),
// through the context-phase kernels; the sampler is seeded with the new length, as after a prefill.
extern "C" int onellm_llama_extend(onellm_llama* h, const int* host_ids, int n_new, int* host_first_ids)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m && host_ids, ONELLM_ERR_ARG, "llama_extend: null pointer");
    ONELLM_REQUIRE(m->batch > 0 && m->cur_len > 0, ONELLM_ERR_STATE, "llama_extend: call prefill first");
    ONELLM_REQUIRE(n_new >= 1 && m->cur_len + n_new <= m->max_seq_len, ONELLM_ERR_ARG,
                   "llama_extend: %d cached + %d new positions exceed max_seq_len %d", m->cur_len, n_new, m->max_seq_len);
    cudaStream_t st = m->stream;
    const int batch = m->batch, new_len = m->cur_len + n_new;
    ONELLM_CUDA(cudaMemcpyAsync(m->d_prompt, host_ids, (size_t)batch * n_new * sizeof(int), cudaMemcpyHostToDevice, st));
    ONELLM_CUDA(cudaMemcpyAsync(m->d_step, &new_len, sizeof(int), cudaMemcpyHostToDevice, st));
    ONELLM_CUDA(cudaStreamSynchronize(st));  // `new_len` lives on this stack frame
    const std::vector<int> lens(batch, n_new);
    RC(m->prefill_context(batch, lens.data()));
    return m->finish_context(host_first_ids, "llama_extend");
}

// The next prefill / extend call also computes the logits of these token rows (packed order of that call).
extern "C" int onellm_llama_want_logits(onellm_llama* h, const int* rows, int n_rows)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m && n_rows >= 0 && (rows || n_rows == 0), ONELLM_ERR_ARG, "llama_want_logits: bad argument");
    m->want_rows.assign(rows, rows + n_rows);
    return ONELLM_OK;
}

// Declares `cur_len` positions of `batch` sequences as already cached (whatever the cache holds)
// and `host_ids` as the next input tokens: resumes decoding on a cache filled elsewhere, and lets
// profiling runs skip the context phase.
extern "C" int onellm_llama_seek(onellm_llama* h, int batch, int cur_len, const int* host_ids)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m && host_ids, ONELLM_ERR_ARG, "llama_seek: null pointer");
    ONELLM_REQUIRE(m->weights_ready, ONELLM_ERR_STATE, "llama_seek: weights not loaded");
    ONELLM_REQUIRE(batch >= 1 && batch <= m->max_batch && cur_len >= 1 && cur_len < m->max_seq_len, ONELLM_ERR_ARG,
                   "llama_seek: batch or position out of range");
    cudaStream_t st = m->stream;
    ONELLM_CUDA(cudaStreamSynchronize(st));
    if (batch != m->batch) m->drop_graphs();
    m->batch = batch;
    m->cur_len = cur_len;
    m->seq_off.assign(m->max_batch, 0);
    ONELLM_CUDA(cudaMemsetAsync(m->d_step_off, 0, (size_t)m->max_batch * sizeof(int), st));
    ONELLM_CUDA(cudaMemcpyAsync(m->d_step, &cur_len, sizeof(int), cudaMemcpyHostToDevice, st));
    ONELLM_CUDA(cudaMemcpyAsync(m->d_ids, host_ids, (size_t)batch * sizeof(int), cudaMemcpyHostToDevice, st));
    ONELLM_CUDA(cudaMemsetAsync(m->d_seqlen, 0, (size_t)batch * sizeof(int), st));
    ONELLM_CUDA(cudaMemsetAsync(m->d_finished, 0, (size_t)batch, st));
    ONELLM_CUDA(cudaStreamSynchronize(st));
    return ONELLM_OK;
}

extern "C" int onellm_llama_decode_step(onellm_llama* h, const int* host_in_ids, int* host_out_ids)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m, ONELLM_ERR_ARG, "llama_decode_step: null handle");
    ONELLM_REQUIRE(m->batch > 0 && m->cur_len > 0, ONELLM_ERR_STATE, "llama_decode_step: call prefill first");
    cudaStream_t st = m->stream;
    if (host_in_ids)
        ONELLM_CUDA(cudaMemcpyAsync(m->d_ids, host_in_ids, (size_t)m->batch * sizeof(int), cudaMemcpyHostToDevice, st));
    RC(m->run_step(MODE_HEAD, 0));
    if (host_out_ids) {
        ONELLM_CUDA(cudaMemcpyAsync(host_out_ids, m->d_out_ids, (size_t)m->batch * sizeof(int), cudaMemcpyDeviceToHost, st));
        RC(m->queue_comm_check());
        ONELLM_CUDA(cudaStreamSynchronize(st));
        RC(m->comm_check("llama_decode_step"));
    }
    return ONELLM_OK;
}

extern "C" int onellm_llama_sync(onellm_llama* h)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m, ONELLM_ERR_ARG, "llama_sync: null handle");
    RC(m->queue_comm_check());
    ONELLM_CUDA(cudaStreamSynchronize(m->stream));
    return m->comm_check("llama_sync");
}

extern "C" int onellm_llama_generate(onellm_llama* h, const int* host_prompt, int batch, int prompt_len, int n_new, int* host_out)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m && host_prompt && host_out && n_new >= 1, ONELLM_ERR_ARG, "llama_generate: bad argument");
    std::vector<int> ids(batch);
    RC(onellm_llama_prefill(h, host_prompt, batch, prompt_len, ids.data()));
    for (int b = 0; b < batch; b++) host_out[(size_t)b * n_new] = ids[b];
    for (int t = 1; t < n_new; t++) {
        RC(onellm_llama_decode_step(h, nullptr, ids.data()));
        for (int b = 0; b < batch; b++) host_out[(size_t)b * n_new + t] = ids[b];
    }
    return ONELLM_OK;
}

// n rows of logits from row `first` of the last pass, as float on the host.
static int copy_logits(Engine* m, size_t first, size_t rows, float* host_logits)
{
    const size_t n = rows * m->vocab;
    const char* src = static_cast<const char*>(m->last_logits) + first * m->vocab * dtype_size(m->logits_dtype);
    cudaError_t e;
    float* tmp = nullptr;
    if (m->logits_dtype == ONELLM_F32) {
        e = cudaMemcpyAsync(host_logits, src, n * sizeof(float), cudaMemcpyDeviceToHost, m->stream);
    } else {
        ONELLM_CUDA(cudaMalloc(&tmp, n * sizeof(float)));
        half_to_float_kernel<<<blocks_for(n), 256, 0, m->stream>>>(reinterpret_cast<const __half*>(src), tmp, n);
        e = cudaMemcpyAsync(host_logits, tmp, n * sizeof(float), cudaMemcpyDeviceToHost, m->stream);
    }
    const int qrc = m->queue_comm_check();
    if (e == cudaSuccess) e = cudaStreamSynchronize(m->stream);
    if (tmp) cudaFree(tmp);
    ONELLM_REQUIRE(e == cudaSuccess, ONELLM_ERR_CUDA, "llama_get_logits: %s", cudaGetErrorString(e));
    RC(qrc);
    return m->comm_check("llama_get_logits");
}

extern "C" int onellm_llama_get_logits(onellm_llama* h, float* host_logits)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m && host_logits, ONELLM_ERR_ARG, "llama_get_logits: null pointer");
    ONELLM_REQUIRE(m->batch > 0 && m->last_logits, ONELLM_ERR_STATE, "llama_get_logits: nothing computed yet");
    return copy_logits(m, 0, m->batch, host_logits);
}

extern "C" int onellm_llama_get_row_logits(onellm_llama* h, float* host_logits, int n_rows)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m && host_logits && n_rows >= 1, ONELLM_ERR_ARG, "llama_get_row_logits: bad argument");
    ONELLM_REQUIRE(m->row_have == (size_t)n_rows && m->last_logits == m->row_logits, ONELLM_ERR_STATE,
                   "llama_get_row_logits: the last pass was not a context pass with %d wanted rows", n_rows);
    return copy_logits(m, m->batch, n_rows, host_logits);
}

extern "C" int onellm_llama_get_state(onellm_llama* h, int* cur_len, long* kernel_launches, int* host_seqlen, unsigned char* host_finished)
{
    Engine* m = engine_of(h);
    ONELLM_REQUIRE(m, ONELLM_ERR_ARG, "llama_get_state: null handle");
    if (cur_len) *cur_len = m->cur_len;
    if (kernel_launches) *kernel_launches = m->launches;
    if (host_seqlen && m->batch) ONELLM_CUDA(cudaMemcpy(host_seqlen, m->d_seqlen, (size_t)m->batch * sizeof(int), cudaMemcpyDeviceToHost));
    if (host_finished && m->batch) ONELLM_CUDA(cudaMemcpy(host_finished, m->d_finished, (size_t)m->batch, cudaMemcpyDeviceToHost));
    return ONELLM_OK;
}

extern "C" int onellm_model_limits(const onellm_llama* h, int* vocab_size, int* max_seq_len, int* max_batch)
{
    ONELLM_REQUIRE(h, ONELLM_ERR_ARG, "model_limits: null handle");
    const Engine* m = engine_of(h);
    if (vocab_size) *vocab_size = m->vocab;
    if (max_seq_len) *max_seq_len = m->max_seq_len;
    if (max_batch) *max_batch = m->max_batch;
    return ONELLM_OK;
}
