// Gated outer-product recurrence (the HGRN2 form of linear attention: the forget gate also decides what is written);
// gates, recurrence and the per-head RMS norm of the output are computed in float.  With g = 1 - f a state element
// moves as
//     s <- s + g (v - s)
// which needs one multiply-add and keeps the digits of a gate near one (g comes from the complementary sigmoid).
//
// Context pass (gated_recurrence_kernel).  A thread block owns 32 value columns of one (sequence, head) and keeps that
// part of the state, dk x 32 floats, in registers over all tokens of the call: columns of the state never meet, only the
// dk rows are summed into the output.  Eight warps do nothing but the recurrence: a thread holds R rows x 4 columns as
// pairs of rows for the packed fma.rn.f32x2; the 8 lanes of a row group cover the 32 columns, the 4 row groups of each
// warp and the warps the dk <= 32 R rows; tokens are taken four at a time so that their sums over the row groups overlap.
// Four more warps feed and drain them, a block of tokens ahead and behind: they copy the projections (cp.async), turn
// them into g and silu(q), add the partial outputs of the eight warps, and norm and store the result.  The blocks of a
// head form a cluster: the RMS norm needs all value columns, and the sums of squares of a token block are exchanged
// through distributed shared memory.  One cluster barrier per token block orders everything.
//
// Decode step (gated_recurrence_step_kernel).  One token per sequence: the state is streamed once through registers,
// HBM-bound; its first rows are requested before the dependency wait, because they do not depend on the kernel in front.
#include <cooperative_groups.h>

#include "mixers.h"

namespace cg = cooperative_groups;

namespace onellm {

constexpr int kGrCols = 32, kGrWarps = 8, kGrFeed = 128;  // value columns of a block; recurrence warps; feeding threads
constexpr int kGrThreads = kGrWarps * 32 + kGrFeed;

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack_f2(float lo, float hi)
{
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float sum_f2(f32x2 v)
{
    float lo, hi;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
    return lo + hi;
}
__device__ __forceinline__ f32x2 fma_f2(f32x2 a, f32x2 b, f32x2 c)
{
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f32x2 sub_f2(f32x2 a, f32x2 b)
{
    f32x2 r;
    asm("sub.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// sigmoid(x) and 1 - sigmoid(x), both with full relative precision; the fast exponential and division where the
// projections are bfloat16 (their error is far below the rounding of x)
template <typename T>
__device__ __forceinline__ void sigmoid_pair(float x, float& s, float& c)
{
    float e, r;
    if constexpr (sizeof(T) == 2) {
        e = __expf(-fabsf(x));
        r = __fdividef(1.f, 1.f + e);
    } else {
        e = expf(-fabsf(x));
        r = 1.f / (1.f + e);
    }
    s = x >= 0.f ? r : e * r;
    c = x >= 0.f ? e * r : r;
}
// 1 - f and silu(q) of one channel
template <typename T>
__device__ __forceinline__ void gate(float q, float z, float zb, float lower, float& g, float& qs)
{
    float s, c;
    sigmoid_pair<T>(z + zb, s, c);
    g = (1.f - lower) * c;
    sigmoid_pair<T>(q, s, c);
    qs = q * s;
}

struct GrParams {
    GatedRecurrence g;
    TokenPositions tp;
};

// bytes of one raw token block: q and z rows of dk, v rows of 32 columns
template <typename T, int TOK>
__host__ __device__ constexpr size_t gr_raw_bytes(int dk) { return (size_t)TOK * (2 * dk + kGrCols) * sizeof(T); }
// floats of one prepared token block
template <int R, int TOK>
__host__ __device__ constexpr int gr_block_floats() { return TOK * (2 * 32 * R + kGrCols); }
template <typename T, int R, int TOK>
static size_t gr_smem_bytes(int dk)
{
    return 2 * gr_raw_bytes<T, TOK>(dk) + sizeof(float) * 2 * ((size_t)gr_block_floats<R, TOK>() + kGrWarps * TOK * kGrCols + TOK);
}

template <typename T, int R, int TOK>
__global__ void __launch_bounds__(kGrThreads) gated_recurrence_kernel(const GrParams pp)
{
    constexpr int DKP = 32 * R;  // dk padded to whole thread tiles; the extra rows have zero gates and queries
    constexpr int VEC = Vec16<T>::N;
    constexpr int BLK = gr_block_floats<R, TOK>(), PART = kGrWarps * TOK * kGrCols;
    const GatedRecurrence& p = pp.g;
    extern __shared__ __align__(16) unsigned char smem[];
    const int dk = p.dk, h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * kGrCols;
    const size_t raw = gr_raw_bytes<T, TOK>(dk);
    float* ready = reinterpret_cast<float*>(smem + 2 * raw);  // two blocks of g [TOK][DKP], silu(q) [TOK][DKP], v [TOK][32]
    float* part = ready + 2 * BLK;                            // two blocks of [warp][TOK][32]
    float* ssq = part + 2 * PART;                             // [2][TOK]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    cg::cluster_group cluster = cg::this_cluster();

    const int tok0 = pp.tp.cu[b], n_tok = pp.tp.cu[b + 1] - tok0;
    const int n_blk = (n_tok + TOK - 1) / TOK;
    if (warp < kGrWarps) {
        // ---- the recurrence
        const int k0 = (warp * 4 + (lane >> 3)) * R, col = (lane & 7) * 4;
        const bool fresh = pp.tp.hist[b] == 0;
        float4* st = reinterpret_cast<float4*>(p.state + (((size_t)b * p.H + h) * dk) * p.dv + c0 + col);
        const size_t st_row = (size_t)p.dv / 4;
        f32x2 S[R / 2][4];
#pragma unroll
        for (int r = 0; r < R; r += 2) {
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f), c = a;
            if (!fresh && k0 + r < dk) a = st[(size_t)(k0 + r) * st_row];
            if (!fresh && k0 + r + 1 < dk) c = st[(size_t)(k0 + r + 1) * st_row];
            S[r / 2][0] = pack_f2(a.x, c.x);
            S[r / 2][1] = pack_f2(a.y, c.y);
            S[r / 2][2] = pack_f2(a.z, c.z);
            S[r / 2][3] = pack_f2(a.w, c.w);
        }
        pdl_wait();
        pdl_launch_dependents();
        const bool hi2 = lane & 16, hi1 = lane & 8;
        const int my_col = col + (hi2 ? 2 : 0) + (hi1 ? 1 : 0);
        cluster.sync();  // block 0 is prepared
        for (int it = 0; it < n_blk + 2; it++) {
            if (it < n_blk) {
                const float* sg = ready + (it & 1) * BLK + k0;
                const float* sq = sg + TOK * DKP;
                const float* sv = ready + (it & 1) * BLK + 2 * TOK * DKP + col;
                float* dst = part + (it & 1) * PART + warp * TOK * kGrCols + my_col;
                const int n4 = (min(TOK, n_tok - it * TOK) + 3) & ~3;  // tokens behind the end have g = q = v = 0
                for (int t = 0; t < n4; t += 4) {
                    f32x2 o2[4][4];
#pragma unroll
                    for (int u = 0; u < 4; u++) {
                        const float4 v4 = *reinterpret_cast<const float4*>(sv + (t + u) * kGrCols);
                        const f32x2 vv[4] = {pack_f2(v4.x, v4.x), pack_f2(v4.y, v4.y), pack_f2(v4.z, v4.z), pack_f2(v4.w, v4.w)};
                        f32x2 g2[R / 2], q2[R / 2];
                        const float *gt = sg + (t + u) * DKP, *qt = sq + (t + u) * DKP;
                        if constexpr (R >= 4) {
#pragma unroll
                            for (int r = 0; r < R / 2; r += 2) {
                                *reinterpret_cast<ulonglong2*>(&g2[r]) = *reinterpret_cast<const ulonglong2*>(gt + 2 * r);
                                *reinterpret_cast<ulonglong2*>(&q2[r]) = *reinterpret_cast<const ulonglong2*>(qt + 2 * r);
                            }
                        } else {
                            g2[0] = *reinterpret_cast<const f32x2*>(gt);
                            q2[0] = *reinterpret_cast<const f32x2*>(qt);
                        }
#pragma unroll
                        for (int c = 0; c < 4; c++) o2[u][c] = 0ull;
#pragma unroll
                        for (int r = 0; r < R / 2; r++)
#pragma unroll
                            for (int c = 0; c < 4; c++) {
                                S[r][c] = fma_f2(g2[r], sub_f2(vv[c], S[r][c]), S[r][c]);
                                o2[u][c] = fma_f2(q2[r], S[r][c], o2[u][c]);
                            }
                    }
                    // sum over the row groups of the warp; a lane keeps one column: halves first (columns 0-1 | 2-3), then
                    // one of two
#pragma unroll
                    for (int u = 0; u < 4; u++) {
                        const float o[4] = {sum_f2(o2[u][0]), sum_f2(o2[u][1]), sum_f2(o2[u][2]), sum_f2(o2[u][3])};
                        float a0 = hi2 ? o[2] : o[0], a1 = hi2 ? o[3] : o[1];
                        a0 += __shfl_xor_sync(0xffffffffu, hi2 ? o[0] : o[2], 16);
                        a1 += __shfl_xor_sync(0xffffffffu, hi2 ? o[1] : o[3], 16);
                        dst[(t + u) * kGrCols] = (hi1 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, hi1 ? a0 : a1, 8);
                    }
                }
            }
            cluster.sync();
        }
        if (n_tok > 0) {
#pragma unroll
            for (int r = 0; r < R; r += 2) {
                float a[4], c[4];
#pragma unroll
                for (int j = 0; j < 4; j++) asm("mov.b64 {%0, %1}, %2;" : "=f"(a[j]), "=f"(c[j]) : "l"(S[r / 2][j]));
                if (k0 + r < dk) st[(size_t)(k0 + r) * st_row] = make_float4(a[0], a[1], a[2], a[3]);
                if (k0 + r + 1 < dk) st[(size_t)(k0 + r + 1) * st_row] = make_float4(c[0], c[1], c[2], c[3]);
            }
        }
    } else {
        // ---- feed and drain
        const int ft = tid - kGrWarps * 32, fw = ft >> 5;
        const int n_peers = gridDim.x;
        // the channels whose gates this thread makes: ft % DKP of tokens ft / DKP, + 128 / DKP, ... (two channels when there
        // are more of them than threads)
        constexpr int KPT = DKP > kGrFeed ? DKP / kGrFeed : 1, TSTEP = DKP > kGrFeed ? 1 : kGrFeed / DKP;
        float zb[KPT], lower[KPT];
#pragma unroll
        for (int i = 0; i < KPT; i++) {
            const int k = min(ft % DKP + i * kGrFeed, dk - 1);
            zb[i] = p.zb[h * dk + k];
            lower[i] = p.lower[h * dk + k];
        }
        const float wn = p.w[c0 + lane] * p.out_scale;
        pdl_wait();
        pdl_launch_dependents();
        const T* q = reinterpret_cast<const T*>(p.q) + (size_t)h * dk;
        const T* z = reinterpret_cast<const T*>(p.z) + (size_t)h * dk;
        const T* v = reinterpret_cast<const T*>(p.v) + (size_t)h * p.dv + c0;
        const int kc = dk / VEC, per_tok = 2 * kc + kGrCols / VEC;
        const uint32_t raw_base = (uint32_t)__cvta_generic_to_shared(smem);
        auto issue = [&](int blk) {  // a warp copies whole tokens
            if (blk < n_blk) {
                const int t0 = blk * TOK, n = min(TOK, n_tok - t0);
                for (int t = fw; t < n; t += kGrFeed / 32) {
                    const size_t row = (size_t)(tok0 + t0 + t) * p.ld;
                    const uint32_t dst = raw_base + (uint32_t)((blk & 1) * raw) + (uint32_t)(t * per_tok) * 16u;
                    for (int c = lane; c < per_tok; c += 32) {
                        const T* src = c < kc ? q + row + c * VEC : c < 2 * kc ? z + row + (c - kc) * VEC : v + row + (c - 2 * kc) * VEC;
                        cp_async16(dst + c * 16u, src, 16);
                    }
                }
            }
            cp_async_commit();
        };
        auto prepare = [&](int blk) {  // the copies of this block were issued one call ago
            cp_async_wait<0>();
            asm volatile("bar.sync 1, %0;" ::"n"(kGrFeed) : "memory");  // the feeding threads' copies of the block, and their reads of the one before
            issue(blk + 1);
            if (blk >= n_blk) return;
            const int n = min(TOK, n_tok - blk * TOK), n4 = (n + 3) & ~3;
            const T* rb = reinterpret_cast<const T*>(smem + (size_t)(blk & 1) * raw);
            const int row_el = 2 * dk + kGrCols;
            float* sg = ready + (blk & 1) * BLK;
            float* sq = sg + TOK * DKP;
            float* sv = sq + TOK * DKP;
#pragma unroll
            for (int i = 0; i < KPT; i++) {
                const int k = ft % DKP + i * kGrFeed, kk = min(k, dk - 1);
#pragma unroll 4
                for (int t = ft / DKP; t < n4; t += TSTEP) {
                    const T* row = rb + min(t, n - 1) * row_el + kk;
                    float g, qs;
                    gate<T>(to_float(row[0]), to_float(row[dk]), zb[i], lower[i], g, qs);
                    const bool real = k < dk && t < n;
                    sg[t * DKP + k] = real ? g : 0.f;
                    sq[t * DKP + k] = real ? qs : 0.f;
                }
            }
#pragma unroll 4
            for (int t = fw; t < n4; t += kGrFeed / 32) {
                const float x = to_float(rb[min(t, n - 1) * row_el + 2 * dk + lane]);
                sv[t * kGrCols + lane] = t < n ? x : 0.f;
            }
        };
        issue(0);
        prepare(0);
        cluster.sync();
        float o[TOK / 4];  // outputs of token fw + 4 i, column `lane`, of the block summed last
        for (int it = 0; it < n_blk + 2; it++) {
            prepare(it + 1);
            if (it >= 2) {
                // norm and store block it - 2: every block of the cluster left its sums before the last barrier, and writes
                // that buffer again behind the next one
                const int blk = it - 2, n = min(TOK, n_tok - blk * TOK);
                float inv = 0.f;
                if (lane < TOK) {
                    float* mine = ssq + (blk & 1) * TOK;
                    float s[8];
#pragma unroll
                    for (int r = 0; r < 8; r++) s[r] = r < n_peers ? cluster.map_shared_rank(mine, r)[lane] : 0.f;
                    inv = 1.0f / sqrtf((((s[0] + s[1]) + (s[2] + s[3])) + ((s[4] + s[5]) + (s[6] + s[7]))) / (float)p.norm_width + p.eps);
                }
                T* dst = reinterpret_cast<T*>(p.out) + (size_t)(tok0 + blk * TOK) * p.out_ld + (size_t)h * p.dv + c0 + lane;
#pragma unroll
                for (int i = 0; i < TOK / 4; i++) {
                    const int t = fw + 4 * i;
                    const float f = __shfl_sync(0xffffffffu, inv, t);
                    if (t < n) dst[(size_t)t * p.out_ld] = from_float<T>(o[i] * f * wn);
                }
            }
            if (it >= 1 && it <= n_blk) {
                // add the warps' partial outputs of block it - 1 (rows behind its end are whatever was there: never stored)
                const float* src = part + ((it - 1) & 1) * PART + lane;
                float* mine = ssq + ((it - 1) & 1) * TOK;
#pragma unroll
                for (int i = 0; i < TOK / 4; i++) {
                    o[i] = 0.f;
#pragma unroll
                    for (int w = 0; w < kGrWarps; w++) o[i] += src[(w * TOK + fw + 4 * i) * kGrCols];
                }
#pragma unroll
                for (int i = 0; i < TOK / 4; i++) {
                    const float s = warp_sum(o[i] * o[i]);
                    if (lane == 0) mine[fw + 4 * i] = s;
                }
            }
            cluster.sync();
        }
        cp_async_wait<0>();
    }
}

// One token per sequence.  A block owns `cols` value columns of one (sequence, head); cols / 4 threads share a row and
// every thread walks the rows of its column group, kGsBatch at a time.
constexpr int kGsThreads = 256, kGsBatch = 8;

template <typename T>
__global__ void __launch_bounds__(kGsThreads) gated_recurrence_step_kernel(const GrParams pp, int cols)
{
    const GatedRecurrence& p = pp.g;
    __shared__ float sg[256], sq[256];
    __shared__ __align__(16) float part[kGsThreads * 4];
    __shared__ float ssq, wsum[kGsThreads / 32];
    const int dk = p.dk, h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * cols, tid = threadIdx.x;
    const int tpr = cols / 4, rows_par = kGsThreads / tpr;  // threads per row, rows at a time
    const int r0 = tid / tpr, col = (tid % tpr) * 4;
    const bool works = r0 < rows_par;  // 256 need not be a multiple of tpr
    const bool fresh = *pp.tp.step - 1 + pp.tp.off[b] == 0;
    float* base = p.state + (((size_t)b * p.H + h) * dk) * p.dv + c0 + col;
    float4 s[kGsBatch];
    auto fetch = [&](int first) {
#pragma unroll
        for (int i = 0; i < kGsBatch; i++) {
            const int r = first + i * rows_par;
            s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (works && !fresh && r < dk) s[i] = *reinterpret_cast<const float4*>(base + (size_t)r * p.dv);
        }
    };
    fetch(r0);
    float zb = 0.f, lower = 0.f;
    if (tid < dk) {
        zb = p.zb[h * dk + tid];
        lower = p.lower[h * dk + tid];
    }
    pdl_wait();
    pdl_launch_dependents();
    if (tid < dk) {
        const T* q = reinterpret_cast<const T*>(p.q) + (size_t)b * p.ld + (size_t)h * dk;
        const T* z = reinterpret_cast<const T*>(p.z) + (size_t)b * p.ld + (size_t)h * dk;
        gate<T>(to_float(q[tid]), to_float(z[tid]), zb, lower, sg[tid], sq[tid]);
    }
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (works) {
        const T* vp = reinterpret_cast<const T*>(p.v) + (size_t)b * p.ld + (size_t)h * p.dv + c0 + col;
#pragma unroll
        for (int i = 0; i < 4; i++) v[i] = to_float(vp[i]);
    }
    __syncthreads();
    float o[4] = {0.f, 0.f, 0.f, 0.f};
    for (int first = r0; first < dk; first += kGsBatch * rows_par) {
        if (first != r0) fetch(first);
#pragma unroll
        for (int i = 0; i < kGsBatch; i++) {
            const int r = first + i * rows_par;
            if (works && r < dk) {
                const float g = sg[r], q = sq[r];
                s[i].x = fmaf(g, v[0] - s[i].x, s[i].x);
                s[i].y = fmaf(g, v[1] - s[i].y, s[i].y);
                s[i].z = fmaf(g, v[2] - s[i].z, s[i].z);
                s[i].w = fmaf(g, v[3] - s[i].w, s[i].w);
                o[0] = fmaf(q, s[i].x, o[0]);
                o[1] = fmaf(q, s[i].y, o[1]);
                o[2] = fmaf(q, s[i].z, o[2]);
                o[3] = fmaf(q, s[i].w, o[3]);
                *reinterpret_cast<float4*>(base + (size_t)r * p.dv) = s[i];
            }
        }
    }
    if (works) *reinterpret_cast<float4*>(&part[r0 * cols + col]) = make_float4(o[0], o[1], o[2], o[3]);  // rows_par * cols <= 1024
    __syncthreads();
    float y = 0.f;
    if (tid < cols)
        for (int r = 0; r < rows_par; r++) y += part[r * cols + tid];
    const float sq1 = warp_sum(y * y);
    if ((tid & 31) == 0) wsum[tid >> 5] = sq1;
    __syncthreads();
    if (tid == 0) {
        float t = 0.f;
        for (int i = 0; i < kGsThreads / 32; i++) t += wsum[i];
        ssq = t;
    }
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();  // a barrier of the block too when it is alone
    float t = 0.f;
    for (int r = 0; r < (int)gridDim.x; r++) t += *cluster.map_shared_rank(&ssq, r);
    if (tid < cols) {
        const float inv = 1.0f / sqrtf(t / (float)p.norm_width + p.eps);
        reinterpret_cast<T*>(p.out)[(size_t)b * p.out_ld + (size_t)h * p.dv + c0 + tid] = from_float<T>(y * inv * p.w[c0 + tid] * p.out_scale);
    }
    cluster.sync();  // peers may still be reading this block's sum
}

template <typename Kernel, typename... Args>
static int launch_cluster(Kernel kern, dim3 grid, int threads, size_t smem, cudaStream_t st, Args... args)
{
    (void)prefer_max_shared((const void*)kern);
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = grid.x;
    at[0].val.clusterDim.y = 1;
    at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.gridDim = grid;
    cfg.blockDim = dim3(threads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cfg.attrs = at;
    cfg.numAttrs = 2;
    note_launch();
    ONELLM_CUDA(cudaLaunchKernelEx(&cfg, kern, args...));
    return ONELLM_OK;
}

template <typename T, int R, int TOK>
static int launch_gr(const GrParams& p, int B, cudaStream_t st)
{
    auto kern = gated_recurrence_kernel<T, R, TOK>;
    static DeviceOnce attr;
    ONELLM_CUDA(attr.run([kern] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024); }));
    return launch_cluster(kern, dim3(p.g.dv / kGrCols, p.g.H, B), kGrThreads, gr_smem_bytes<T, R, TOK>(p.g.dk), st, p);
}

template <typename T>
static int dispatch_gr(const GrParams& p, int B, cudaStream_t st)
{
    if (!p.tp.cu) {
        // columns of a head over several blocks only while whole heads leave SMs without work
        int cols = p.g.dv;
        for (int n = 2; n <= 8 && (long)B * p.g.H * (p.g.dv / cols) < 2L * num_sms(); n *= 2)
            if (p.g.dv % (32 * n) == 0) cols = p.g.dv / n;
        return launch_cluster(gated_recurrence_step_kernel<T>, dim3(p.g.dv / cols, p.g.H, B), kGsThreads, 0, st, p, cols);
    }
    // token blocks of 32 where one thread block per SM is all there is, else of 16 (two thread blocks share an SM)
    const int dk = p.g.dk;
    if constexpr (sizeof(T) == 2) {
        if (dk <= 128 && (long)B * p.g.H * (p.g.dv / kGrCols) <= num_sms())
            return dk <= 64 ? launch_gr<T, 2, 32>(p, B, st) : launch_gr<T, 4, 32>(p, B, st);
    }
    if (dk <= 64) return launch_gr<T, 2, 16>(p, B, st);
    if (dk <= 128) return launch_gr<T, 4, 16>(p, B, st);
    return launch_gr<T, 8, 16>(p, B, st);
}

int gated_recurrence(const GatedRecurrence& g, const TokenPositions& tp, int B, cudaStream_t st)
{
    ONELLM_REQUIRE(g.q && g.z && g.v && g.zb && g.lower && g.w && g.state && g.out, ONELLM_ERR_ARG, "gated_recurrence: null pointer");
    ONELLM_REQUIRE(g.dk > 0 && g.dk % 16 == 0 && g.dk <= 256 && g.dv > 0 && g.dv % kGrCols == 0 && g.dv <= 8 * kGrCols, ONELLM_ERR_UNSUPPORTED,
                   "gated_recurrence: key size %d must be a multiple of 16 and value size %d of 32, both at most 256", g.dk, g.dv);
    ONELLM_REQUIRE(g.H > 0 && g.H <= 65535 && B > 0 && B <= 65535 && g.ld % 8 == 0 && (tp.cu ? tp.hist != nullptr : tp.step && tp.off),
                   ONELLM_ERR_ARG, "gated_recurrence: bad argument");
    const GrParams p = {g, tp};
    return g.dtype == ONELLM_F32 ? dispatch_gr<float>(p, B, st) : dispatch_gr<__nv_bfloat16>(p, B, st);
}

}  // namespace onellm

extern "C" int onellm_gated_recurrence_run(const onellm_gated_recurrence* g, const onellm_token_positions* tp, int B, void* stream)
{
    ONELLM_REQUIRE(g && tp, ONELLM_ERR_ARG, "gated_recurrence: null pointer");
    return onellm::gated_recurrence(*g, *tp, B, reinterpret_cast<cudaStream_t>(stream));
}
