// Sequence-mixing mechanisms the model designs are put together from, with everything a design fixes as parameters:
//   - attention with its own key and value sizes, a score factor per query position and a score penalty per head and
//     distance (biased_attn.cu, biased_attn_tc.cu);
//   - a gated outer-product recurrence with a float state (gated_recurrence.cu);
// and the norm and embedding kernels of designs that keep the residual stream in float (norm.cu, elementwise.cu).
// Element type T of projections, caches and outputs: bfloat16 (ONELLM_BF16) or float (ONELLM_F32).
#pragma once
#include "common.cuh"

namespace onellm {

// Where the tokens of a launch belong.  Context pass: cu / hist as in ContextBatch, token t is packed.  Decode step (cu
// NULL): one token per sequence, at position *step - 1 + off[t].
struct TokenPositions {
    const int* cu;
    const int* hist;
    int B;
    const int* step;
    const int* off;

    __device__ __forceinline__ void locate(int t, int& b, int& pos) const
    {
        if (cu) {
            b = 0;
            while (b + 1 < B && t >= cu[b + 1]) b++;
            pos = hist[b] + t - cu[b];
        } else {
            b = t;
            pos = *step - 1 + off[t];
        }
    }
};

struct BiasedAttn {
    int dtype;
    int H, G, dk, dv;        // query heads, key/value heads, sizes (multiples of 16, at most 256); head h reads h / (H / G)
    const void *q, *k, *v;   // the tokens' projections: token t at + t * ld; heads dk (q, k) / dv (v) apart
    long ld;
    void *k_cache, *v_cache; // one layer: [B, G, S, dk] and [B, G, S, dv]
    int S;
    // score of a key `d` positions back for a query at position p, in units of log2:
    //     (q . k) * q_factor[p] - penalty[h * S + d]
    const float* q_factor;   // [S]
    const float* penalty;    // [H, S]
    void* out;               // token t, head h at + t * out_ld + h * dv
    long out_ld;
    float out_scale;
};

// Keys and values of `tokens` tokens into the cache (not needed in front of biased_attn_decode).
int biased_attn_store(const BiasedAttn& a, const TokenPositions& tp, int tokens, int* overflow, cudaStream_t st);
// Context pass over the cache (keys and values stored before): tensor cores for bfloat16, plain float otherwise or when
// `plain` asks for it.  max_new: most tokens of one sequence.
int biased_attn_context(const BiasedAttn& a, const TokenPositions& tp, int tokens, int max_new, bool plain, cudaStream_t st);
// Decode step of B sequences (bfloat16): stores the new key and value and attends.  step_bound: upper bound of *tp.step.
size_t biased_attn_decode_workspace(int B, int H, int dv);
int biased_attn_decode(const BiasedAttn& a, const TokenPositions& tp, int step_bound, void* workspace, cudaStream_t st);
// q_factor[p] = scale * (1 + coef * ln(floor((p + 1) / every) + 1)) * log2(e)
int build_query_factor(float* out, int S, double scale, double coef, double every, cudaStream_t st);
// penalty[h, d] = r1[h] * ln(1 + r2[h] * d) * log2(e)
int build_distance_penalty(float* out, const float* r1, const float* r2, int H, int S, cudaStream_t st);

// Per head h, with the gates of a token  f = l + (1 - l) * sigmoid(z + zb)  (dk values) and  q' = silu(q):
//     state = diag(f) state + (1 - f) v^T        o = state^T q'
//     out   = o * rsqrt(mean(o^2) + eps) * w * out_scale
struct GatedRecurrence {
    int dtype;
    int H, dk, dv;           // dk a multiple of 16, dv of 32, at most 256
    const void *q, *z, *v;   // token t at + t * ld; heads dk / dk / dv apart
    long ld;
    const float *zb, *lower; // [H * dk]
    const float* w;          // [dv]
    float eps;
    int norm_width;          // the mean is taken over this many channels (dv without padding)
    float* state;            // [B, H, dk, dv]; ignored (zero) for a sequence whose history is empty
    void* out;               // token t, head h at + t * out_ld + h * dv
    long out_ld;
    float out_scale;
};
int gated_recurrence(const GatedRecurrence& g, const TokenPositions& tp, int B, cudaStream_t st);

// norm.cu
int norm_pair(int dtype, const float* x, const int* rows, int n_rows, const float* w1, const float* w2, void* out1, void* out2, float eps,
              int width, int ld, cudaStream_t st);
// elementwise.cu
int embedding_pos_launch(int dtype, const int* ids, float* out, const void* table, const void* pos_table, int n_tokens, int ld, int vocab,
                         int max_pos, const TokenPositions& tp, int* bad, cudaStream_t st);

}  // namespace onellm
