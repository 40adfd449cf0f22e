// Sequence-mixing mechanisms the model designs are put together from, with everything a design fixes as parameters:
//   - attention with its own key and value sizes, a score factor per query position and a score penalty per head and
//     distance (biased_attn.cu, biased_attn_tc.cu);
//   - attention over cached latents in a sliding window (latent_attn.cu; whole prompts: biased_attn_tc.cu);
//   - a gated outer-product recurrence with a float state, in two kinds (gated_recurrence.cu);
//   - the routing of a mixture of experts (route.cu; its products are projections in row groups, project.h);
// and the norm and embedding kernels of designs that keep the residual stream in float (norm.cu, elementwise.cu).
// Element type T of projections, caches and outputs: bfloat16 (ONELLM_BF16) or float (ONELLM_F32).  The parameter
// structures and what the functions compute are described in onellm_b200.h.
#pragma once
#include "common.cuh"

namespace onellm {

using TokenPositions = onellm_token_positions;
using BiasedAttn = onellm_biased_attn;
using GatedRecurrence = onellm_gated_recurrence;
using LatentAttn = onellm_latent_attn;
using WindowAttn = onellm_window_attn;
using NormRows = onellm_norm_rows;
using Route = onellm_route;

// sequence and position of token t
__device__ __forceinline__ void locate(const TokenPositions& tp, int t, int& b, int& pos)
{
    if (tp.cu) {
        b = 0;
        while (b + 1 < tp.B && t >= tp.cu[b + 1]) b++;
        pos = tp.hist[b] + t - tp.cu[b];
    } else {
        b = t;
        pos = *tp.step - 1 + tp.off[t];
    }
}

int biased_attn_store(const BiasedAttn& a, const TokenPositions& tp, int tokens, int* overflow, cudaStream_t st);
int biased_attn_context(const BiasedAttn& a, const TokenPositions& tp, int tokens, int max_new, bool plain, cudaStream_t st);
size_t biased_attn_decode_workspace(int B, int H, int dv);
int biased_attn_decode(const BiasedAttn& a, const TokenPositions& tp, int step_bound, void* workspace, cudaStream_t st);
int build_query_factor(float* out, int S, double scale, double coef, double every, cudaStream_t st);
int build_distance_penalty(float* out, const float* r1, const float* r2, int H, int S, cudaStream_t st);
// value size padded to what the recurrence kernels take: 32 columns for every 256
inline int gated_recurrence_pad_dv(int dv)
{
    const int m = 32 * ((dv + 255) / 256);
    return (dv + m - 1) / m * m;
}
size_t gated_recurrence_workspace(int kind, int tokens, int H, int dk, int dv);
int gated_recurrence(const GatedRecurrence& g, const TokenPositions& tp, int B, int tokens, cudaStream_t st);

// max_hist: most positions a sequence has before this pass; max_new: most new tokens of one
inline int latent_pad(int rank) { return (rank + 63) / 64 * 64; }
int latent_store(const LatentAttn& a, const TokenPositions& tp, int tokens, int max_hist, cudaStream_t st);
int latent_keep(const LatentAttn& a, const TokenPositions& tp, int max_new, cudaStream_t st);
size_t latent_attn_workspace(int tokens, int H, int rank);
int latent_attn(const LatentAttn& a, const TokenPositions& tp, int tokens, int span_bound, bool plain, void* workspace, cudaStream_t st);
int window_attn(const WindowAttn& a, const TokenPositions& tp, int max_new, cudaStream_t st);

// route.cu
int route_max_tiles(int T, int experts, int top);
int route(const Route& r, cudaStream_t st);
// norm.cu
int norm_rows(const NormRows& n, cudaStream_t st);
// elementwise.cu
int embedding_norm_launch(int dtype, const int* ids, float* out, const void* table, const float* w, float eps, int n_tokens, int width, int ld,
                          int vocab, int* bad, cudaStream_t st);
int softcap(const float* in, long ld, float* out, int rows, int cols, float cap, cudaStream_t st);
int embedding_pos_launch(int dtype, const int* ids, float* out, const void* table, const void* pos_table, int n_tokens, int ld, int vocab,
                         int max_pos, const TokenPositions& tp, int* bad, cudaStream_t st);

}  // namespace onellm
