// Gated outer-product recurrence (the HGRN2 form of linear attention: the forget gate also decides what is written),
// for a context pass of any length and for one decode step; gates, recurrence and the per-head RMS norm of the
// output are computed in float.
//
// A thread block owns 32 value columns of one (sequence, head) and keeps that part of the state, dk x 32 floats, in
// registers over all tokens of the call: columns of the state never meet, only the dk rows are summed into the output.
// A thread holds R rows x 4 columns; the 8 lanes of a row group cover the 32 columns, the 4 row groups of each of
// the 4 warps the dk = 16 R rows.  Tokens come in blocks of 32 through a double-buffered cp.async ring, are turned
// into f, 1 - f and silu(q) once per block (1 - f from the complementary sigmoid, so that a gate near one keeps its
// digits), and each warp leaves its partial outputs in shared memory; one reduction per token block adds the warps.
// The blocks of a head form a cluster: its RMS norm needs all value columns, and the sums of squares of a token block
// are exchanged through distributed shared memory.
#include <cooperative_groups.h>

#include "mixers.h"

namespace cg = cooperative_groups;

namespace onellm {

constexpr int kGrThreads = 128, kGrCols = 32;
// tokens of a block: 32, fewer where the widest float heads would not fit shared memory
template <typename T, int R>
constexpr int gr_tok() { return sizeof(T) == 4 && R > 8 ? 16 : 32; }

struct GrParams {
    const void *q, *z, *v;
    long ld;
    const float *zb, *lower, *w;
    float eps;
    int H, dk, dv, norm_width;
    float* state;
    void* out;
    long out_ld;
    float out_scale;
    TokenPositions tp;
};

// bytes of one raw token block: q and z rows of dk, v rows of 32 columns
template <typename T, int R>
__host__ __device__ constexpr size_t gr_raw_bytes(int dk) { return (size_t)gr_tok<T, R>() * (2 * dk + kGrCols) * sizeof(T); }
template <typename T, int R>
static size_t gr_smem_bytes(int dk)
{
    constexpr int kGrTok = gr_tok<T, R>();
    return 2 * gr_raw_bytes<T, R>(dk) + sizeof(float) * ((size_t)kGrTok * (3 * 16 * R + kGrCols) + 4 * kGrTok * kGrCols + 2 * kGrTok);
}

template <typename T, int R>
__global__ void __launch_bounds__(kGrThreads) gated_recurrence_kernel(const GrParams p)
{
    constexpr int kGrTok = gr_tok<T, R>();
    constexpr int DKP = 16 * R;  // dk padded to whole thread tiles; the extra rows have zero gates and queries
    constexpr int VEC = Vec16<T>::N;
    extern __shared__ __align__(16) unsigned char smem[];
    const int dk = p.dk, h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * kGrCols;
    const size_t raw = gr_raw_bytes<T, R>(dk);
    float* sf = reinterpret_cast<float*>(smem + 2 * raw);
    float* sg = sf + kGrTok * DKP;
    float* sq = sg + kGrTok * DKP;
    float* sv = sq + kGrTok * DKP;
    float* part = sv + kGrTok * kGrCols;        // [4 warps][kGrTok][32]
    float* ssq = part + 4 * kGrTok * kGrCols;   // [2][kGrTok]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int k0 = (warp * 4 + (lane >> 3)) * R, col = (lane & 7) * 4;
    cg::cluster_group cluster = cg::this_cluster();
    const int n_peers = gridDim.x;

    const int tok0 = p.tp.cu ? p.tp.cu[b] : b;
    const int n_tok = p.tp.cu ? p.tp.cu[b + 1] - tok0 : 1;
    const bool fresh = p.tp.cu && p.tp.hist[b] == 0;
    float4* st = reinterpret_cast<float4*>(p.state + (((size_t)b * p.H + h) * dk) * p.dv + c0 + col);
    const size_t st_row = (size_t)p.dv / 4;

    // The state was written by the same layer of an earlier step: it does not depend on the kernel before this one.
    float S[R][4];
#pragma unroll
    for (int r = 0; r < R; r++) {
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && k0 + r < dk) s = st[(size_t)(k0 + r) * st_row];
        S[r][0] = s.x;
        S[r][1] = s.y;
        S[r][2] = s.z;
        S[r][3] = s.w;
    }
    pdl_wait();
    pdl_launch_dependents();

    const T* q = reinterpret_cast<const T*>(p.q) + (size_t)h * dk;
    const T* z = reinterpret_cast<const T*>(p.z) + (size_t)h * dk;
    const T* v = reinterpret_cast<const T*>(p.v) + (size_t)h * p.dv + c0;
    const int kc = dk / VEC, vc = kGrCols / VEC, per_tok = 2 * kc + vc;
    const uint32_t raw_base = (uint32_t)__cvta_generic_to_shared(smem);
    auto issue = [&](int blk) {
        const int t0 = blk * kGrTok, n = min(kGrTok, n_tok - t0);
        const uint32_t dst = raw_base + (uint32_t)((blk & 1) * raw);
        for (int i = tid; i < n * per_tok; i += kGrThreads) {
            const int t = i / per_tok, c = i % per_tok;
            const size_t row = (size_t)(tok0 + t0 + t) * p.ld;
            const T* src = c < kc ? q + row + c * VEC : c < 2 * kc ? z + row + (c - kc) * VEC : v + row + (c - 2 * kc) * VEC;
            cp_async16(dst + (uint32_t)i * 16u, src, 16);
        }
    };
    const int n_blk = (n_tok + kGrTok - 1) / kGrTok;
    if (n_blk > 0) issue(0);
    cp_async_commit();
    for (int blk = 0; blk < n_blk; blk++) {
        if (blk + 1 < n_blk) issue(blk + 1);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const int n = min(kGrTok, n_tok - blk * kGrTok);
        const T* rb = reinterpret_cast<const T*>(smem + (size_t)(blk & 1) * raw);
        const int row_el = 2 * dk + kGrCols;
        for (int i = tid; i < n * DKP; i += kGrThreads) {
            const int t = i / DKP, k = i % DKP;
            float f = 0.f, g = 0.f, qs = 0.f;
            if (k < dk) {
                const float qv = to_float(rb[t * row_el + k]);
                const float zv = to_float(rb[t * row_el + dk + k]) + p.zb[h * dk + k];
                const float l = p.lower[h * dk + k];
                const float e = expf(-fabsf(zv)), s = 1.f / (1.f + e), es = e * s;
                f = l + (1.f - l) * (zv >= 0.f ? s : es);
                g = (1.f - l) * (zv >= 0.f ? es : s);
                const float eq = expf(-fabsf(qv)), sg1 = 1.f / (1.f + eq);
                qs = qv * (qv >= 0.f ? sg1 : eq * sg1);
            }
            sf[i] = f;
            sg[i] = g;
            sq[i] = qs;
        }
        for (int i = tid; i < n * kGrCols; i += kGrThreads) sv[i] = to_float(rb[(i / kGrCols) * row_el + 2 * dk + i % kGrCols]);
        __syncthreads();
#pragma unroll 2
        for (int t = 0; t < n; t++) {
            const float4 v4 = *reinterpret_cast<const float4*>(sv + t * kGrCols + col);
            const float vv[4] = {v4.x, v4.y, v4.z, v4.w};
            float o[4] = {0.f, 0.f, 0.f, 0.f};
            const float *ft = sf + t * DKP + k0, *gt = sg + t * DKP + k0, *qt = sq + t * DKP + k0;
            float f[R], g[R], qq[R];
            if constexpr (R % 4 == 0) {
#pragma unroll
                for (int r = 0; r < R; r += 4) {
                    *reinterpret_cast<float4*>(&f[r]) = *reinterpret_cast<const float4*>(ft + r);
                    *reinterpret_cast<float4*>(&g[r]) = *reinterpret_cast<const float4*>(gt + r);
                    *reinterpret_cast<float4*>(&qq[r]) = *reinterpret_cast<const float4*>(qt + r);
                }
            } else {
#pragma unroll
                for (int r = 0; r < R; r++) {
                    f[r] = ft[r];
                    g[r] = gt[r];
                    qq[r] = qt[r];
                }
            }
#pragma unroll
            for (int r = 0; r < R; r++)
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    S[r][c] = fmaf(f[r], S[r][c], g[r] * vv[c]);
                    o[c] = fmaf(qq[r], S[r][c], o[c]);
                }
            // sum over the four row groups of the warp; lane keeps one column: first halves (columns 0-1 | 2-3), then one of two
            const bool hi2 = lane & 16, hi1 = lane & 8;
            float a0 = hi2 ? o[2] : o[0], a1 = hi2 ? o[3] : o[1], b0 = hi2 ? o[0] : o[2], b1 = hi2 ? o[1] : o[3];
            a0 += __shfl_xor_sync(0xffffffffu, b0, 16);
            a1 += __shfl_xor_sync(0xffffffffu, b1, 16);
            float a = hi1 ? a1 : a0;
            const float bb = hi1 ? a0 : a1;
            a += __shfl_xor_sync(0xffffffffu, bb, 8);
            part[(warp * kGrTok + t) * kGrCols + col + (hi2 ? 2 : 0) + (hi1 ? 1 : 0)] = a;
        }
        __syncthreads();
        // one warp per token row: add the warps' partial sums, sum of squares of the 32 columns
        float o[kGrTok / 4];
        float* ss_now = ssq + (blk & 1) * kGrTok;
#pragma unroll
        for (int i = 0; i < kGrTok / 4; i++) {
            const int t = warp + 4 * i;
            o[i] = 0.f;
            if (t < n) {
                for (int w = 0; w < 4; w++) o[i] += part[(w * kGrTok + t) * kGrCols + lane];
                const float s = warp_sum(o[i] * o[i]);
                if (lane == 0) ss_now[t] = s;
            }
        }
        // Every block of the cluster has written its sums; they stay valid for one more round (two buffers), and a block
        // that writes that buffer again has passed the next round's barrier, behind everyone's reads of this one.
        cluster.sync();
#pragma unroll
        for (int i = 0; i < kGrTok / 4; i++) {
            const int t = warp + 4 * i;
            if (t < n) {
                float s = 0.f;
                for (int r = 0; r < n_peers; r++) s += cluster.map_shared_rank(ss_now, r)[t];
                const float inv = 1.0f / sqrtf(s / (float)p.norm_width + p.eps);
                T* dst = reinterpret_cast<T*>(p.out) + (size_t)(tok0 + blk * kGrTok + t) * p.out_ld + (size_t)h * p.dv + c0 + lane;
                *dst = from_float<T>(o[i] * inv * p.w[c0 + lane] * p.out_scale);
            }
        }
    }
    cp_async_wait<0>();
    if (n_tok > 0) {
#pragma unroll
        for (int r = 0; r < R; r++)
            if (k0 + r < dk) st[(size_t)(k0 + r) * st_row] = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
    }
    cluster.sync();  // peers may still be reading this block's sums
}

template <typename T, int R>
static int launch_gr(const GrParams& p, int B, cudaStream_t st)
{
    auto kern = gated_recurrence_kernel<T, R>;
    static DeviceOnce attr;
    ONELLM_CUDA(attr.run([kern] {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
        return e != cudaSuccess ? e : prefer_max_shared((const void*)kern);
    }));
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = p.dv / kGrCols;
    at[0].val.clusterDim.y = 1;
    at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.gridDim = dim3(p.dv / kGrCols, p.H, B);
    cfg.blockDim = dim3(kGrThreads);
    cfg.dynamicSmemBytes = gr_smem_bytes<T, R>(p.dk);
    cfg.stream = st;
    cfg.attrs = at;
    cfg.numAttrs = 2;
    note_launch();
    ONELLM_CUDA(cudaLaunchKernelEx(&cfg, kern, p));
    return ONELLM_OK;
}

template <typename T>
static int dispatch_gr(const GrParams& p, int B, cudaStream_t st)
{
    const int R = p.dk / 16;
    if (R <= 1) return launch_gr<T, 1>(p, B, st);
    if (R <= 2) return launch_gr<T, 2>(p, B, st);
    if (R <= 4) return launch_gr<T, 4>(p, B, st);
    if (R <= 8) return launch_gr<T, 8>(p, B, st);
    return launch_gr<T, 16>(p, B, st);
}

int gated_recurrence(const GatedRecurrence& g, const TokenPositions& tp, int B, cudaStream_t st)
{
    ONELLM_REQUIRE(g.q && g.z && g.v && g.zb && g.lower && g.w && g.state && g.out, ONELLM_ERR_ARG, "gated_recurrence: null pointer");
    ONELLM_REQUIRE(g.dk > 0 && g.dk % 16 == 0 && g.dk <= 256 && g.dv > 0 && g.dv % kGrCols == 0 && g.dv <= 8 * kGrCols, ONELLM_ERR_UNSUPPORTED,
                   "gated_recurrence: key size %d must be a multiple of 16 and value size %d of 32, both at most 256", g.dk, g.dv);
    ONELLM_REQUIRE(g.H > 0 && g.H <= 65535 && B > 0 && B <= 65535 && g.ld % 8 == 0, ONELLM_ERR_ARG, "gated_recurrence: bad size");
    const GrParams p = {g.q, g.z, g.v, g.ld, g.zb, g.lower, g.w, g.eps, g.H, g.dk, g.dv, g.norm_width, g.state, g.out, g.out_ld, g.out_scale, tp};
    return g.dtype == ONELLM_F32 ? dispatch_gr<float>(p, B, st) : dispatch_gr<__nv_bfloat16>(p, B, st);
}

}  // namespace onellm

extern "C" int onellm_gated_recurrence_run(const onellm_gated_recurrence* g, const onellm_token_positions* tp, int B, void* stream)
{
    ONELLM_REQUIRE(g && tp, ONELLM_ERR_ARG, "gated_recurrence: null pointer");
    return onellm::gated_recurrence(*g, *tp, B, reinterpret_cast<cudaStream_t>(stream));
}
