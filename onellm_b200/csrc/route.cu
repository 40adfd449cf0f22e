// Routing of a mixture of experts: the best experts of every token by the sigmoid of its router logits, and the tokens in
// expert order, so that the expert products are projections in row groups (project.h).
//
// Up to 64 tokens (a decode step) one block does everything in shared memory.  A context pass takes three launches: the
// choice with a count per expert, the offsets and the 128-row tiles of every expert, the copy of the rows into expert
// order.  Which of the equal places of an expert's block of rows a token gets depends on the order the blocks run in; what
// is computed for it does not.
#include <algorithm>

#include "mixers.h"

namespace onellm {

constexpr int kRtThreads = 256, kRtMaxExperts = 1024, kRtSmall = 64, kRtTile = 128;

// The `top` largest of z[0 .. E) by one warp, best first, the lower index on a tie; lane 0 reports each through emit(k, e, z).
template <typename Emit>
__device__ __forceinline__ void best_of(const float* __restrict__ z, int E, int top, Emit emit)
{
    const int lane = threadIdx.x & 31;
    float last = INFINITY;
    int last_e = -1;
    for (int k = 0; k < top; k++) {
        // the best one behind (last, last_e) in the order of value down, index up
        float best = -INFINITY;
        int be = E;
        for (int e = lane; e < E; e += 32) {
            const float v = z[e];
            if ((v < last || (v == last && e > last_e)) && (v > best || be == E)) {
                best = v;
                be = e;
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float v = __shfl_xor_sync(0xffffffffu, best, o);
            const int e = __shfl_xor_sync(0xffffffffu, be, o);
            if (e < E && (be == E || v > best || (v == best && e < be))) {
                best = v;
                be = e;
            }
        }
        if (be == E) be = min(last_e + 1, E - 1);  // logits that do not compare (NaN): still a valid expert
        if (lane == 0) emit(k, be, best);
        last = best;
        last_e = be;
    }
}
__device__ __forceinline__ float score(float z) { return 1.f / (1.f + expf(-z)); }

// Offsets of the experts, the list of those with rows and their tiles, from counts in shared memory; one warp.
__device__ __forceinline__ void lay_out(const int* count, int* off_s, const Route& r)
{
    const int lane = threadIdx.x & 31, E = r.experts;
    int rows = 0, used = 0, tiles = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
        const int e = e0 + lane, n = e < E ? count[e] : 0, nt = (n + kRtTile - 1) / kRtTile;
        int a = n, b = n > 0, c = nt;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int pa = __shfl_up_sync(0xffffffffu, a, o), pb = __shfl_up_sync(0xffffffffu, b, o), pc = __shfl_up_sync(0xffffffffu, c, o);
            if (lane >= o) {
                a += pa;
                b += pb;
                c += pc;
            }
        }
        if (e < E) {
            const int first = rows + a - n;
            off_s[e] = first;
            r.off[e] = first;
            if (n > 0) r.used[used + b - 1] = e;
            for (int i = 0; i < nt; i++) {
                r.tile_group[tiles + c - nt + i] = e;
                r.tile_row[tiles + c - nt + i] = first + i * kRtTile;
            }
        }
        rows += __shfl_sync(0xffffffffu, a, 31);
        used += __shfl_sync(0xffffffffu, b, 31);
        tiles += __shfl_sync(0xffffffffu, c, 31);
    }
    if (lane == 0) {
        r.off[E] = rows;
        *r.n_used = used;
        *r.n_tiles = tiles;
    }
}

__global__ void __launch_bounds__(kRtThreads) route_small_kernel(const Route r)
{
    __shared__ int count[kRtMaxExperts], off[kRtMaxExperts];
    extern __shared__ int choice[];  // [T * top], then the places of the rows inside their experts
    const int warp = threadIdx.x >> 5, n = r.T * r.top;
    int* place = choice + n;
    float* weight = reinterpret_cast<float*>(place + n);
    for (int e = threadIdx.x; e < r.experts; e += kRtThreads) count[e] = 0;
    __syncthreads();
    pdl_launch_dependents();
    pdl_wait();
    for (int t = warp; t < r.T; t += kRtThreads / 32)
        best_of(r.logits + (size_t)t * r.ld, r.experts, r.top, [&](int k, int e, float z) {
            choice[t * r.top + k] = e;
            weight[t * r.top + k] = score(z);
            place[t * r.top + k] = atomicAdd(&count[e], 1);
        });
    __syncthreads();
    if (warp == 0) lay_out(count, off, r);
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += kRtThreads) {
        const int s = off[choice[i]] + place[i];
        r.slot[i] = s;
        r.slot_token[s] = i / r.top;
        r.slot_weight[s] = weight[i];
    }
}

// one warp per token
__global__ void __launch_bounds__(kRtThreads) route_choose_kernel(const Route r)
{
    __shared__ int count[kRtMaxExperts];
    for (int e = threadIdx.x; e < r.experts; e += kRtThreads) count[e] = 0;
    __syncthreads();
    pdl_launch_dependents();
    pdl_wait();
    const int per = kRtThreads / 32 * 4, t0 = blockIdx.x * per;
    for (int t = t0 + (threadIdx.x >> 5); t < min(t0 + per, r.T); t += kRtThreads / 32)
        best_of(r.logits + (size_t)t * r.ld, r.experts, r.top, [&](int k, int e, float z) {
            r.choice[(size_t)t * r.top + k] = e;
            r.choice_weight[(size_t)t * r.top + k] = score(z);
            atomicAdd(&count[e], 1);
        });
    __syncthreads();
    for (int e = threadIdx.x; e < r.experts; e += kRtThreads)
        if (count[e]) atomicAdd(&r.count[e], count[e]);
}

__global__ void __launch_bounds__(kRtThreads) route_lay_out_kernel(const Route r)
{
    __shared__ int count[kRtMaxExperts], off[kRtMaxExperts];
    pdl_launch_dependents();
    pdl_wait();
    for (int e = threadIdx.x; e < r.experts; e += kRtThreads) count[e] = r.count[e];
    __syncthreads();
    if (threadIdx.x < 32) lay_out(count, off, r);
    __syncthreads();
    for (int e = threadIdx.x; e < r.experts; e += kRtThreads) r.count[e] = 0;  // the next kernel counts the places with it
}

// one block per token: its places, and its row into each of them
__global__ void __launch_bounds__(128) route_copy_kernel(const Route r, int row_bytes)
{
    __shared__ int at[64];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    for (int k = threadIdx.x; k < r.top; k += blockDim.x) {
        const int i = t * r.top + k, e = r.choice[i], s = r.off[e] + atomicAdd(&r.count[e], 1);
        r.slot[i] = s;
        r.slot_token[s] = t;
        r.slot_weight[s] = r.choice_weight[i];
        at[k] = s;
    }
    __syncthreads();
    if (!r.xs) return;
    const uint4* src = reinterpret_cast<const uint4*>(static_cast<const char*>(r.x) + (size_t)t * row_bytes);
    for (int i = threadIdx.x; i < row_bytes / 16; i += blockDim.x) {
        const uint4 v = src[i];
        for (int k = 0; k < r.top; k++) reinterpret_cast<uint4*>(static_cast<char*>(r.xs) + (size_t)at[k] * row_bytes)[i] = v;
    }
}
// the counts are zero between calls
__global__ void __launch_bounds__(kRtThreads) route_clear_kernel(int* count, int E)
{
    pdl_launch_dependents();
    pdl_wait();
    for (int e = threadIdx.x; e < E; e += kRtThreads) count[e] = 0;
}

int route_max_tiles(int T, int experts, int top) { return T * top / kRtTile + std::min(experts, T * top); }

int route(const Route& r, cudaStream_t st)
{
    ONELLM_REQUIRE(r.logits && r.slot && r.slot_token && r.slot_weight && r.off && r.used && r.n_used && r.tile_group && r.tile_row && r.n_tiles,
                   ONELLM_ERR_ARG, "route: null pointer");
    ONELLM_REQUIRE(r.T >= 0 && r.experts > 0 && r.experts <= kRtMaxExperts && r.top > 0 && r.top <= r.experts && r.top <= 64 && r.ld >= r.experts,
                   ONELLM_ERR_UNSUPPORTED, "route: %d of %d experts (at most 64 of %d)", r.top, r.experts, kRtMaxExperts);
    if (r.T == 0) return ONELLM_OK;
    if (r.T <= kRtSmall) {
        const size_t smem = (size_t)r.T * r.top * 12;
        ONELLM_CUDA(launch_pdl(route_small_kernel, dim3(1), dim3(kRtThreads), smem, st, r));
        return ONELLM_OK;
    }
    ONELLM_REQUIRE(r.choice && r.choice_weight && r.count, ONELLM_ERR_ARG, "route: null pointer");
    const size_t es = r.dtype == ONELLM_F32 ? 4 : 2;
    ONELLM_REQUIRE(!r.xs || (r.x && r.ld_x * es % 16 == 0 && aligned16(r.x) && aligned16(r.xs)), ONELLM_ERR_ARG, "route: rows of whole 16-byte vectors");
    const int per = kRtThreads / 32 * 4;
    ONELLM_CUDA(launch_pdl(route_choose_kernel, dim3((r.T + per - 1) / per), dim3(kRtThreads), 0, st, r));
    ONELLM_CUDA(launch_pdl(route_lay_out_kernel, dim3(1), dim3(kRtThreads), 0, st, r));
    ONELLM_CUDA(launch_pdl(route_copy_kernel, dim3(r.T), dim3(128), 0, st, r, (int)(r.ld_x * es)));
    ONELLM_CUDA(launch_pdl(route_clear_kernel, dim3(1), dim3(kRtThreads), 0, st, r.count, r.experts));
    return ONELLM_OK;
}

}  // namespace onellm

extern "C" int onellm_route_max_tiles(int T, int experts, int top) { return onellm::route_max_tiles(T, experts, top); }

extern "C" int onellm_route_run(const onellm_route* r, void* stream)
{
    ONELLM_REQUIRE(r, ONELLM_ERR_ARG, "route: null pointer");
    return onellm::route(*r, reinterpret_cast<cudaStream_t>(stream));
}
