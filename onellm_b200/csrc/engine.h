// The generation engine behind every onellm_llama handle: device memory, sequence state, step counter, CUDA graphs,
// sampling and the generate loop.  A model design (llama.cu, finuvik.cu) derives from it and supplies its weights, its
// per-sequence memory (KV cache, recurrent state) and the kernels of a decode step and of a context pass.
#pragma once
#include <map>
#include <string>
#include <vector>

#include "common.cuh"

namespace onellm {

inline size_t align_up(size_t x, size_t a) { return (x + a - 1) / a * a; }
inline int blocks_for(size_t n) { return (int)((n + 255) / 256 < 4096 ? (n + 255) / 256 : 4096); }

// Hands out 256-byte aligned pieces of one allocation; with base == nullptr it only adds up the size.
struct Carver {
    char* base;
    size_t off = 0;
    template <typename T>
    T* take(size_t n)
    {
        off = align_up(off, 256);
        T* p = base ? reinterpret_cast<T*>(base + off) : nullptr;
        off += n * sizeof(T);
        return p;
    }
    void* take_bytes(size_t n) { return take<char>(n); }
};

enum StepMode { MODE_GATHER = 1, MODE_HEAD = 2 };

// One context pass: T new tokens of B sequences, packed in sequence order in Engine::d_prompt.
struct ContextBatch {
    int B = 0, P = 0;          // sequences; most new tokens of one sequence
    size_t T = 0;              // tokens
    const int* cu = nullptr;   // device [B + 1]: token offsets of the sequences
    const int* hist = nullptr; // device [B]: positions a sequence has cached
    const int* host_hist = nullptr;  // the same on the host
    const int* rows = nullptr; // device [n_rows]: packed token rows whose logits are wanted, the last one of every
    int n_rows = 0;            // sequence first (those B rows are sampled from)
    void* logits = nullptr;    // device [n_rows, vocab] of Engine::logits_dtype
};

struct Engine {
    // capacity and vocabulary, set by the design's constructor
    int vocab = 0, max_seq_len = 0, max_batch = 0, eos_id = 2;
    int span_cap = 0x7fffffff;  // most positions a launch of a decode step depends on (the longest window of a windowed design)
    int logits_dtype = ONELLM_F16;
    // memory
    char* arena = nullptr;
    size_t arena_bytes = 0;
    char* scratch = nullptr;  // context pass, grown on demand
    size_t scratch_bytes = 0;
    int *d_ids = nullptr, *d_prompt = nullptr, *d_step = nullptr, *d_out_ids = nullptr, *d_seqlen = nullptr,
        *d_topk_id = nullptr, *d_bad_id = nullptr, *d_cu = nullptr, *d_hist = nullptr;
    // per sequence: cached length minus cur_len (<= 0; all zero unless the prompts had different lengths)
    int* d_step_off = nullptr;
    std::vector<int> seq_off;  // host copy
    unsigned char* d_finished = nullptr;
    float *d_topk_val = nullptr, *d_u = nullptr;
    uint32_t* d_skip = nullptr;  // the sampler's per-row skip-ahead table (sampling.cu)
    int skip_ok = 0;             // 1 once the table is built and has matched the direct draws
    void* logits = nullptr;      // [max_batch, vocab]
    // logits of further rows of the next context pass (onellm_llama_want_logits)
    std::vector<int> want_rows;
    int* d_rows = nullptr;
    void* row_logits = nullptr;  // [max_batch + wanted, vocab]
    size_t row_cap = 0, row_have = 0;
    const void* last_logits = nullptr;
    // state
    int batch = 0, cur_len = 0, graph_prompt_len = 0;
    int top_k = 1, literal_walk = 0;  // top_k 0: logits only, nothing is sampled
    float temperature = 1.0f;
    bool weights_ready = false, use_graphs = true;
    bool prefill_by_decode = false;  // true: run the context phase one position at a time (reference path for tests)
    bool plain_kernels = false;      // true: the design's unfused kernels where it has fused ones (comparison)
    cudaStream_t stream = nullptr;
    std::map<long, cudaGraphExec_t> graphs;
    long launches = 0;  // kernels enqueued by this model (graph replays count their nodes)
    std::map<long, int> graph_nodes;
    std::map<long, int> warmed;  // keys whose first step already ran outside a capture

    virtual ~Engine();
    // Allocates the arena (twice through carve: size, then pointers), the stream and the sampler's table.
    int allocate();
    int ensure_scratch(size_t bytes);
    void drop_graphs();

    // ---- what a design supplies
    virtual const char* design() const = 0;
    virtual void carve(Carver& cv) = 0;
    // From the batch ids in d_ids (and, for every sequence b, its position *d_step - 1 + d_step_off[b]) through all
    // layers; with_head also the logits of every sequence into `logits`.  `step_bound` is an upper bound of
    // min(*d_step, span_cap).
    virtual int decode_layers(int step_bound, bool with_head) = 0;
    // All tokens of a context pass through all layers, and the logits of c.rows into c.logits.
    virtual int context_layers(const ContextBatch& c) = 0;
    virtual int init_random(uint64_t seed, float std) = 0;
    // Around every point where the host waits for the stream (see llama.cu: tensor-parallel peers).
    virtual int queue_comm_check() { return ONELLM_OK; }
    virtual int comm_check(const char*) { return ONELLM_OK; }

    // ---- the generation loop
    int sample(const void* row_logits);
    int enqueue_step(int mode, int step_bound, int prompt_len);
    int run_step(int mode, int prompt_len);
    int prefill_context(int B, const int* lens);
    int finish_context(int* host_first_ids, const char* where);

  private:
    void carve_common(Carver& cv);
};

// ---- model registry: a design is found by the name its configuration file gives -----------------------------
struct ModelOptions {
    int dtype = ONELLM_BF16;
    int max_batch = 1, max_seq_len = 0;
};
struct Json;
using ModelFactory = int (*)(const Json& config, const std::string& folder, const ModelOptions& opt, Engine** out);
struct ModelRegistration {
    ModelRegistration(const char* architecture, ModelFactory make);
};

// ---- kernels and launchers of other files --------------------------------------------------------------------
size_t skip_table_words(int rows);  // sampling.cu
int build_skip_table(uint32_t* table, int rows, int* usable, cudaStream_t st);
int topk_sample_launch(const int* topk_id, const float* topk_val, int B, int K, float temperature, int rng_step,
                       const int* rng_step_dev, int vocab_size, int end_id, int literal_walk, int* output_id,
                       int* seqlen, unsigned char* finished, float* u_out, int* output_id2, bool early_seed,
                       const uint32_t* skip_table, cudaStream_t st);
int embedding_launch(int dtype, const int* ids, void* out, void* out2, const void* table, int n_tokens, int hidden,
                     int vocab, int* bad_id_flag, bool pdl, cudaStream_t st);
// w[i] = mean + std * N(0,1) of element type dtype, counter-based (seed, tensor tag, index); see engine.cu
int init_normal(int dtype, void* w, size_t rows, size_t cols, size_t full_cols, size_t row0, size_t col0, uint64_t seed, uint64_t tag,
                float mean, float std, cudaStream_t st);

}  // namespace onellm
