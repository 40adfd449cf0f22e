// Gated outer-product recurrences; gates, recurrence and the per-head RMS norm of the output are computed in float.  Two
// kinds (onellm_gr_kind):
//   TIED (HGRN2): what a channel forgets of its state is the share it takes of the new value.  With g = 1 - f
//         s <- s + g (v - s)
//     which needs one multiply-add and keeps the digits of a gate near one (g comes from the complementary sigmoid).
//   KEYED (gated linear attention): the new value comes in through a key of its own.  With g = f - 1
//         s <- s + k v + g s
//     which keeps the digits of a gate near one as well; the gate's logit comes through a low-rank projection, whose
//     second matrix is applied in float here.
//
// Context pass, three launches:
//   1. the prepare kernel turns the projections into the vectors of the recurrence (g and silu(q); or g, k and q), in
//      float and head by head, so that the tokens of a head lie behind each other.
//   2. gated_recurrence_scan_kernel.  A thread block owns 32 value columns of one (sequence, head) and keeps that part of
//      the state, dk x 32 floats, in registers over all tokens of the call: columns of the state never meet, only the dk
//      rows are summed into the output.  A thread holds R rows x 4 columns as pairs of rows for the packed fma.rn.f32x2;
//      the 8 lanes of a row group cover the 32 columns, the 4 row groups of each of the 8 warps the dk <= 32 R rows;
//      tokens are taken four at a time so that their sums over the row groups overlap.  Blocks of tokens arrive by bulk
//      copies (one for g and q, one for v) in two stages; one block barrier per token block, behind which the warps add
//      their partial outputs.
//   3. gated_recurrence_norm_kernel: RMS norm per head and the output gate, output in the element type.
// (One launch that made the gates itself, once per value tile, and normed through a cluster spent two thirds of its time
// outside the recurrence.)
//
// Decode step (gated_recurrence_step_kernel).  One token per sequence: the state is streamed once through registers,
// HBM-bound; its first rows are requested before the dependency wait, because they do not depend on the kernel in front.
#include <cooperative_groups.h>

#include <algorithm>

#include "mixers.h"
#include "tc_common.cuh"

namespace cg = cooperative_groups;

namespace onellm {

constexpr int kGrCols = 32, kGrWarps = 8;  // value columns of a block; warps
constexpr int kGrThreads = kGrWarps * 32;

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
template <typename T>
__device__ __forceinline__ float silu_of(float x)
{
    float s, c;
    sigmoid_pair<T>(x, s, c);
    return x * s;
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

// sigmoid(z) ^ inv_tau - 1 from the logarithm of the sigmoid
__device__ __forceinline__ float decay(float z, float inv_tau) { return expm1f(inv_tau * (fminf(z, 0.f) - log1pf(expf(-fabsf(z))))); }

struct GrParams {
    GatedRecurrence g;
    TokenPositions tp;
};

// Layout of the work space of T tokens: the vectors of a head [H][T][n * dkp] (TIED n = 2: g, silu(q); KEYED n = 3: g, q, k),
// v [H][dv / 32][T][32], outputs before the norm [T][H][dv]; all float, dkp = dk padded to the rows of a block.
static int gr_dkp(int dk) { return dk <= 64 ? 64 : dk <= 128 ? 128 : dk <= 256 ? 256 : 512; }
static int gr_vectors(int kind) { return kind == ONELLM_GR_KEYED ? 3 : 2; }

template <typename T>
__device__ __forceinline__ void gr_load4(const T* src, float (&f)[4])
{
    if constexpr (sizeof(T) == 4) {
        const float4 x = *reinterpret_cast<const float4*>(src);
        f[0] = x.x; f[1] = x.y; f[2] = x.z; f[3] = x.w;
    } else {
        const uint2 x = *reinterpret_cast<const uint2*>(src);
        const float2 a = unpack2<T>(x.x), b = unpack2<T>(x.y);
        f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
    }
}
// the values of one token, 32-column tile by tile
template <typename T>
__device__ __forceinline__ void gr_values(const GatedRecurrence& p, int t, int tokens, float* __restrict__ vf)
{
    const T* v = reinterpret_cast<const T*>(p.v) + (size_t)t * p.ld;
    for (int i = threadIdx.x; i < p.H * (p.dv / 4); i += blockDim.x) {
        const int c = i * 4, tile = c / kGrCols;  // tiles of all heads in a row: h * (dv / 32) + tile of the head
        float x[4];
        gr_load4(v + c, x);
        *reinterpret_cast<float4*>(vf + ((size_t)tile * tokens + t) * kGrCols + c % kGrCols) = make_float4(x[0], x[1], x[2], x[3]);
    }
}

// KEYED: a block prepares kGrPrepTok tokens, so that the second gate matrix is read once for all of them.
constexpr int kGrPrepTok = 8;
template <typename T>
__global__ void __launch_bounds__(256) gated_recurrence_prepare_keyed_kernel(const GrParams pp, int tokens, int dkp, float* __restrict__ gq, float* __restrict__ vf)
{
    const GatedRecurrence& p = pp.g;
    extern __shared__ float sr[];  // [kGrPrepTok][rank]
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = blockIdx.x * kGrPrepTok, nt = min(kGrPrepTok, tokens - t0), dk = p.dk, rank = p.rank;
    for (int i = threadIdx.x; i < kGrPrepTok * rank; i += blockDim.x) {
        const int tt = i / rank;
        sr[i] = tt < nt ? to_float(reinterpret_cast<const T*>(p.r)[(size_t)(t0 + tt) * p.ld + i % rank]) : 0.f;
    }
    __syncthreads();
    const int nq = p.H * (dkp / 4);
    for (int i = threadIdx.x; i < nq; i += blockDim.x) {
        const int h = i / (dkp / 4), k = (i % (dkp / 4)) * 4, c = h * dk + k;
        const bool in = k < dk;
        float z[kGrPrepTok][4];
        if (in) {
            const float4 zb = *reinterpret_cast<const float4*>(p.zb + c);
#pragma unroll
            for (int tt = 0; tt < kGrPrepTok; tt++) {
                z[tt][0] = zb.x; z[tt][1] = zb.y; z[tt][2] = zb.z; z[tt][3] = zb.w;
            }
            const float* A = p.A + (size_t)c * rank;
            for (int j = 0; j < rank; j++) {
                const float a0 = A[j], a1 = A[rank + j], a2 = A[2 * rank + j], a3 = A[3 * rank + j];
#pragma unroll
                for (int tt = 0; tt < kGrPrepTok; tt++) {
                    const float r = sr[tt * rank + j];
                    z[tt][0] = fmaf(a0, r, z[tt][0]);
                    z[tt][1] = fmaf(a1, r, z[tt][1]);
                    z[tt][2] = fmaf(a2, r, z[tt][2]);
                    z[tt][3] = fmaf(a3, r, z[tt][3]);
                }
            }
        }
#pragma unroll
        for (int tt = 0; tt < kGrPrepTok; tt++) {
            if (tt >= nt) break;
            float f[4] = {0.f, 0.f, 0.f, 0.f}, q[4] = {0.f, 0.f, 0.f, 0.f}, kk[4] = {0.f, 0.f, 0.f, 0.f};
            if (in) {
                gr_load4(reinterpret_cast<const T*>(p.q) + (size_t)(t0 + tt) * p.ld + c, q);
                gr_load4(reinterpret_cast<const T*>(p.k) + (size_t)(t0 + tt) * p.ld + c, kk);
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    f[e] = decay(z[tt][e], p.inv_tau);
                    q[e] *= p.q_scale;
                }
            }
            float* dst = gq + ((size_t)h * tokens + t0 + tt) * 3 * dkp + k;
            *reinterpret_cast<float4*>(dst) = make_float4(f[0], f[1], f[2], f[3]);
            *reinterpret_cast<float4*>(dst + dkp) = make_float4(q[0], q[1], q[2], q[3]);
            *reinterpret_cast<float4*>(dst + 2 * dkp) = make_float4(kk[0], kk[1], kk[2], kk[3]);
        }
    }
    for (int tt = 0; tt < nt; tt++) gr_values<T>(p, t0 + tt, tokens, vf);
}

template <typename T>
__global__ void __launch_bounds__(256) gated_recurrence_prepare_kernel(const GrParams pp, int tokens, int dkp, float* __restrict__ gq, float* __restrict__ vf)
{
    const GatedRecurrence& p = pp.g;
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, dk = p.dk;
    const T* q = reinterpret_cast<const T*>(p.q) + (size_t)t * p.ld;
    const T* z = reinterpret_cast<const T*>(p.z) + (size_t)t * p.ld;
    const int nq = p.H * (dkp / 4);
    for (int i = threadIdx.x; i < nq; i += blockDim.x) {
        const int h = i / (dkp / 4), k = (i % (dkp / 4)) * 4;
        float g[4] = {0.f, 0.f, 0.f, 0.f}, qs[4] = {0.f, 0.f, 0.f, 0.f};  // rows behind dk change nothing
        if (k < dk) {
            const int c = h * dk + k;
            float qv[4], zv[4];
            gr_load4(q + c, qv);
            gr_load4(z + c, zv);
            const float4 zb = *reinterpret_cast<const float4*>(p.zb + c), lo = *reinterpret_cast<const float4*>(p.lower + c);
            gate<T>(qv[0], zv[0], zb.x, lo.x, g[0], qs[0]);
            gate<T>(qv[1], zv[1], zb.y, lo.y, g[1], qs[1]);
            gate<T>(qv[2], zv[2], zb.z, lo.z, g[2], qs[2]);
            gate<T>(qv[3], zv[3], zb.w, lo.w, g[3], qs[3]);
        }
        float* dst = gq + ((size_t)h * tokens + t) * 2 * dkp + k;
        *reinterpret_cast<float4*>(dst) = make_float4(g[0], g[1], g[2], g[3]);
        *reinterpret_cast<float4*>(dst + dkp) = make_float4(qs[0], qs[1], qs[2], qs[3]);
    }
    gr_values<T>(p, t, tokens, vf);
}

__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar)
{
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar)
                 : "memory");
}

template <int NV, int R, int TOK>
constexpr size_t gr_smem_bytes() { return sizeof(float) * 2 * ((size_t)TOK * (NV * 32 * R + kGrCols) + (size_t)kGrWarps * TOK * kGrCols); }

// NV: vectors per token (gr_vectors), which tells the kind
template <int NV, int R, int TOK>
__global__ void __launch_bounds__(kGrThreads)
gated_recurrence_scan_kernel(const GrParams pp, int tokens, const float* __restrict__ gq, const float* __restrict__ vf, float* __restrict__ of)
{
    constexpr int DKP = 32 * R;
    constexpr bool KEYED = NV == 3;
    constexpr int STAGE = TOK * (NV * DKP + kGrCols), PART = kGrWarps * TOK * kGrCols;  // floats
    const GatedRecurrence& p = pp.g;
    extern __shared__ __align__(128) float smem_f[];
    float* part = smem_f + 2 * STAGE;
    __shared__ __align__(8) uint64_t bars[2];
    const int dk = p.dk, h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * kGrCols;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int k0 = (warp * 4 + (lane >> 3)) * R, col = (lane & 7) * 4;
    const int tok0 = pp.tp.cu[b], n_tok = pp.tp.cu[b + 1] - tok0, n_blk = (n_tok + TOK - 1) / TOK;
    const bool fresh = pp.tp.hist[b] == 0;
    if (tid == 0) {
        mbar_init(smem_u32(&bars[0]), 1);
        mbar_init(smem_u32(&bars[1]), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    // the state was written by an earlier call: it does not depend on the kernel in front of this one
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
    __syncthreads();
    pdl_wait();
    pdl_launch_dependents();
    const float* gq_src = gq + ((size_t)h * tokens + tok0) * NV * DKP;
    const float* v_src = vf + ((size_t)(h * (p.dv / kGrCols) + blockIdx.x) * tokens + tok0) * kGrCols;
    auto load = [&](int blk) {
        const int s = blk & 1, n = min(TOK, n_tok - blk * TOK);
        const uint32_t dst = smem_u32(smem_f + s * STAGE), bar = smem_u32(&bars[s]);
        const uint32_t gq_bytes = (uint32_t)n * NV * DKP * 4, v_bytes = (uint32_t)n * kGrCols * 4;
        mbar_expect_tx(bar, gq_bytes + v_bytes);
        bulk_load(dst, gq_src + (size_t)blk * TOK * NV * DKP, gq_bytes, bar);
        bulk_load(dst + TOK * NV * DKP * 4, v_src + (size_t)blk * TOK * kGrCols, v_bytes, bar);
    };
    if (tid == 0) {
        if (n_blk > 0) load(0);
        if (n_blk > 1) load(1);
    }
    const bool hi2 = lane & 16, hi1 = lane & 8;
    const int my_col = col + (hi2 ? 2 : 0) + (hi1 ? 1 : 0);
    bool ok = true;
    for (int blk = 0; blk < n_blk; blk++) {
        const int s = blk & 1, n = min(TOK, n_tok - blk * TOK);
        ok = mbar_wait(smem_u32(&bars[s]), (uint32_t)(blk >> 1) & 1u);
        const float* sg = smem_f + s * STAGE + k0;
        const float* sv = smem_f + s * STAGE + TOK * NV * DKP + col;
        float* dst = part + s * PART + warp * TOK * kGrCols + my_col;
        if (ok) {
            int t = 0;
            auto token = [&](int tt, f32x2 (&o2)[4]) {
                const float4 v4 = *reinterpret_cast<const float4*>(sv + tt * kGrCols);
                const f32x2 vv[4] = {pack_f2(v4.x, v4.x), pack_f2(v4.y, v4.y), pack_f2(v4.z, v4.z), pack_f2(v4.w, v4.w)};
                f32x2 g2[R / 2], q2[R / 2], k2[KEYED ? R / 2 : 1];
                const float *gt = sg + tt * NV * DKP, *qt = gt + DKP, *kt = qt + DKP;
                if constexpr (R >= 4) {
#pragma unroll
                    for (int r = 0; r < R / 2; r += 2) {
                        *reinterpret_cast<ulonglong2*>(&g2[r]) = *reinterpret_cast<const ulonglong2*>(gt + 2 * r);
                        *reinterpret_cast<ulonglong2*>(&q2[r]) = *reinterpret_cast<const ulonglong2*>(qt + 2 * r);
                        if constexpr (KEYED) *reinterpret_cast<ulonglong2*>(&k2[r]) = *reinterpret_cast<const ulonglong2*>(kt + 2 * r);
                    }
                } else {
                    g2[0] = *reinterpret_cast<const f32x2*>(gt);
                    q2[0] = *reinterpret_cast<const f32x2*>(qt);
                    if constexpr (KEYED) k2[0] = *reinterpret_cast<const f32x2*>(kt);
                }
#pragma unroll
                for (int c = 0; c < 4; c++) o2[c] = 0ull;
#pragma unroll
                for (int r = 0; r < R / 2; r++)
#pragma unroll
                    for (int c = 0; c < 4; c++) {
                        if constexpr (KEYED) S[r][c] = fma_f2(g2[r], S[r][c], fma_f2(k2[r], vv[c], S[r][c]));
                        else S[r][c] = fma_f2(g2[r], sub_f2(vv[c], S[r][c]), S[r][c]);
                        o2[c] = fma_f2(q2[r], S[r][c], o2[c]);
                    }
            };
            // sum over the row groups of the warp; a lane keeps one column: halves first (columns 0-1 | 2-3), then one of two
            auto reduce = [&](int tt, const f32x2 (&o2)[4]) {
                const float o[4] = {sum_f2(o2[0]), sum_f2(o2[1]), sum_f2(o2[2]), sum_f2(o2[3])};
                float a0 = hi2 ? o[2] : o[0], a1 = hi2 ? o[3] : o[1];
                a0 += __shfl_xor_sync(0xffffffffu, hi2 ? o[0] : o[2], 16);
                a1 += __shfl_xor_sync(0xffffffffu, hi2 ? o[1] : o[3], 16);
                dst[tt * kGrCols] = (hi1 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, hi1 ? a0 : a1, 8);
            };
            for (; t + 4 <= n; t += 4) {
                f32x2 o2[4][4];
#pragma unroll
                for (int u = 0; u < 4; u++) token(t + u, o2[u]);
#pragma unroll
                for (int u = 0; u < 4; u++) reduce(t + u, o2[u]);
            }
            for (; t < n; t++) {
                f32x2 o2[4];
                token(t, o2);
                reduce(t, o2);
            }
        }
        // everyone is done with the stage and has left its partial outputs (two buffers of them: a warp writes this one again
        // behind the next barrier, which everybody reaches after the sums below)
        ok = __syncthreads_and(ok);
        if (!ok) break;
        if (tid == 0 && blk + 2 < n_blk) load(blk + 2);
        float* out = of + ((size_t)(tok0 + blk * TOK) * p.H + h) * p.dv + c0 + lane;
        const float* src = part + s * PART + lane;
#pragma unroll
        for (int i = 0; i < TOK / kGrWarps; i++) {
            const int t = warp + kGrWarps * i;
            if (t < n) {
                float o = 0.f;
#pragma unroll
                for (int w = 0; w < kGrWarps; w++) o += src[(w * TOK + t) * kGrCols];
                out[(size_t)t * p.H * p.dv] = o;
            }
        }
    }
    if (ok && n_tok > 0) {
#pragma unroll
        for (int r = 0; r < R; r += 2) {
            float a[4], c[4];
#pragma unroll
            for (int j = 0; j < 4; j++) asm("mov.b64 {%0, %1}, %2;" : "=f"(a[j]), "=f"(c[j]) : "l"(S[r / 2][j]));
            if (k0 + r < dk) st[(size_t)(k0 + r) * st_row] = make_float4(a[0], a[1], a[2], a[3]);
            if (k0 + r + 1 < dk) st[(size_t)(k0 + r + 1) * st_row] = make_float4(c[0], c[1], c[2], c[3]);
        }
    }
}
static const TimeoutFlag timeout_flag(tc_flag_read_clear);

// one warp per (token, head), at most 32 NJ columns
template <typename T, int NJ>
__global__ void __launch_bounds__(256) gated_recurrence_norm_kernel(const GrParams pp, int tokens, const float* __restrict__ of)
{
    const GatedRecurrence& p = pp.g;
    pdl_launch_dependents();
    pdl_wait();
    const long i = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (i >= (long)tokens * p.H) return;
    const int t = (int)(i / p.H), h = (int)(i % p.H);
    const float* src = of + (size_t)i * p.dv;
    float o[NJ], ss = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; j++) {
        o[j] = lane + 32 * j < p.dv ? src[lane + 32 * j] : 0.f;
        ss = fmaf(o[j], o[j], ss);
    }
    const float inv = p.out_scale / sqrtf(warp_sum(ss) / (float)p.norm_width + p.eps);
    T* dst = reinterpret_cast<T*>(p.out) + (size_t)t * p.out_ld + (size_t)h * p.dv;
    const T* gate = p.g ? reinterpret_cast<const T*>(p.g) + (size_t)t * p.ld + (size_t)h * p.dv : nullptr;
#pragma unroll
    for (int j = 0; j < NJ; j++)
        if (lane + 32 * j < p.dv) {
            const int c = lane + 32 * j;
            float y = o[j] * inv * p.w[c];
            if (gate) y *= silu_of<T>(to_float(gate[c]));
            dst[c] = from_float<T>(y);
        }
}

// One token per sequence.  A block owns `cols` value columns of one (sequence, head); cols / 4 threads share a row and
// every thread walks the rows of its column group, kGsBatch at a time.
constexpr int kGsThreads = 256, kGsBatch = 8;

template <typename T, bool KEYED>
__global__ void __launch_bounds__(kGsThreads) gated_recurrence_step_kernel(const GrParams pp, int cols)
{
    const GatedRecurrence& p = pp.g;
    __shared__ float sg[512], sq[512], sk[KEYED ? 512 : 1];
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
    const float zb0 = tid < dk ? p.zb[h * dk + tid] : 0.f, lower0 = !KEYED && tid < dk ? p.lower[h * dk + tid] : 0.f;
    pdl_wait();
    pdl_launch_dependents();
    const T* q = reinterpret_cast<const T*>(p.q) + (size_t)b * p.ld + (size_t)h * dk;
    for (int i = tid; i < dk; i += kGsThreads) {
        if constexpr (KEYED) {
            const T* r = reinterpret_cast<const T*>(p.r) + (size_t)b * p.ld;
            const float* A = p.A + (size_t)(h * dk + i) * p.rank;
            float z = i == tid ? zb0 : p.zb[h * dk + i];
            for (int j = 0; j < p.rank; j++) z = fmaf(A[j], to_float(r[j]), z);
            sg[i] = decay(z, p.inv_tau);
            sq[i] = to_float(q[i]) * p.q_scale;
            sk[i] = to_float(reinterpret_cast<const T*>(p.k)[(size_t)b * p.ld + (size_t)h * dk + i]);
        } else {
            const T* z = reinterpret_cast<const T*>(p.z) + (size_t)b * p.ld + (size_t)h * dk;
            gate<T>(to_float(q[i]), to_float(z[i]), i == tid ? zb0 : p.zb[h * dk + i], i == tid ? lower0 : p.lower[h * dk + i], sg[i], sq[i]);
        }
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
                if constexpr (KEYED) {
                    const float k = sk[r];
                    s[i].x = fmaf(g, s[i].x, fmaf(k, v[0], s[i].x));
                    s[i].y = fmaf(g, s[i].y, fmaf(k, v[1], s[i].y));
                    s[i].z = fmaf(g, s[i].z, fmaf(k, v[2], s[i].z));
                    s[i].w = fmaf(g, s[i].w, fmaf(k, v[3], s[i].w));
                } else {
                    s[i].x = fmaf(g, v[0] - s[i].x, s[i].x);
                    s[i].y = fmaf(g, v[1] - s[i].y, s[i].y);
                    s[i].z = fmaf(g, v[2] - s[i].z, s[i].z);
                    s[i].w = fmaf(g, v[3] - s[i].w, s[i].w);
                }
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
        y *= inv * p.w[c0 + tid] * p.out_scale;
        if (p.g) y *= silu_of<T>(to_float(reinterpret_cast<const T*>(p.g)[(size_t)b * p.ld + (size_t)h * p.dv + c0 + tid]));
        reinterpret_cast<T*>(p.out)[(size_t)b * p.out_ld + (size_t)h * p.dv + c0 + tid] = from_float<T>(y);
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

template <int NV, int R, int TOK>
static int launch_scan(const GrParams& p, int B, int tokens, const float* gq, const float* vf, float* of, cudaStream_t st)
{
    auto kern = gated_recurrence_scan_kernel<NV, R, TOK>;
    static DeviceOnce attr;
    ONELLM_CUDA(attr.run([kern] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)gr_smem_bytes<NV, R, TOK>()); }));
    ONELLM_CUDA(launch_pdl(kern, dim3(p.g.dv / kGrCols, p.g.H, B), dim3(kGrThreads), gr_smem_bytes<NV, R, TOK>(), st, p, tokens, gq, vf, of));
    return ONELLM_OK;
}

template <int NV>
static int dispatch_scan(const GrParams& p, int B, int tokens, const float* gq, const float* vf, float* of, cudaStream_t st)
{
    // long token blocks where one thread block per SM is all there is, short ones (more thread blocks per SM) otherwise
    const bool few = (long)B * p.g.H * (p.g.dv / kGrCols) <= num_sms();
    switch (gr_dkp(p.g.dk)) {
        case 64: return few ? launch_scan<NV, 2, 32>(p, B, tokens, gq, vf, of, st) : launch_scan<NV, 2, 16>(p, B, tokens, gq, vf, of, st);
        case 128: return few ? launch_scan<NV, 4, 32>(p, B, tokens, gq, vf, of, st) : launch_scan<NV, 4, 16>(p, B, tokens, gq, vf, of, st);
        case 256: return launch_scan<NV, 8, 16>(p, B, tokens, gq, vf, of, st);
        default: return launch_scan<NV, 16, 8>(p, B, tokens, gq, vf, of, st);
    }
}

template <typename T>
static int dispatch_gr(const GrParams& p, int B, int tokens, cudaStream_t st)
{
    const bool keyed = p.g.kind == ONELLM_GR_KEYED;
    if (!p.tp.cu) {
        // columns of a head over several blocks where one block cannot hold them and while whole heads leave SMs without work
        int cols = p.g.dv;
        for (int n = 1; n <= 8; n++)
            if (p.g.dv % (32 * n) == 0 && (cols > 256 || (long)B * p.g.H * (p.g.dv / cols) < 2L * num_sms())) cols = p.g.dv / n;
        const dim3 grid(p.g.dv / cols, p.g.H, B);
        return keyed ? launch_cluster(gated_recurrence_step_kernel<T, true>, grid, kGsThreads, 0, st, p, cols)
                     : launch_cluster(gated_recurrence_step_kernel<T, false>, grid, kGsThreads, 0, st, p, cols);
    }
    if (tokens <= 0) return ONELLM_OK;
    const int dkp = gr_dkp(p.g.dk), nv = gr_vectors(p.g.kind);
    float* gq = static_cast<float*>(p.g.work);
    float* vf = gq + (size_t)tokens * p.g.H * nv * dkp;
    float* of = vf + (size_t)tokens * p.g.H * p.g.dv;
    if (keyed)
        ONELLM_CUDA(launch_pdl(gated_recurrence_prepare_keyed_kernel<T>, dim3((tokens + kGrPrepTok - 1) / kGrPrepTok), dim3(256),
                               (size_t)kGrPrepTok * p.g.rank * sizeof(float), st, p, tokens, dkp, gq, vf));
    else
        ONELLM_CUDA(launch_pdl(gated_recurrence_prepare_kernel<T>, dim3(tokens), dim3(256), 0, st, p, tokens, dkp, gq, vf));
    const int rc = keyed ? dispatch_scan<3>(p, B, tokens, gq, vf, of, st) : dispatch_scan<2>(p, B, tokens, gq, vf, of, st);
    if (rc) return rc;
    const dim3 grid((unsigned)(((long)tokens * p.g.H + 7) / 8));
    if (p.g.dv <= 256) ONELLM_CUDA(launch_pdl(gated_recurrence_norm_kernel<T, 8>, grid, dim3(256), 0, st, p, tokens, of));
    else if (p.g.dv <= 512) ONELLM_CUDA(launch_pdl(gated_recurrence_norm_kernel<T, 16>, grid, dim3(256), 0, st, p, tokens, of));
    else ONELLM_CUDA(launch_pdl(gated_recurrence_norm_kernel<T, 64>, grid, dim3(256), 0, st, p, tokens, of));
    return ONELLM_OK;
}

size_t gated_recurrence_workspace(int kind, int tokens, int H, int dk, int dv)
{
    return (size_t)tokens * H * (gr_vectors(kind) * gr_dkp(dk) + 2 * dv) * sizeof(float);
}

int gated_recurrence(const GatedRecurrence& g, const TokenPositions& tp, int B, int tokens, cudaStream_t st)
{
    const bool keyed = g.kind == ONELLM_GR_KEYED;
    ONELLM_REQUIRE(g.kind == ONELLM_GR_TIED || keyed, ONELLM_ERR_ARG, "gated_recurrence: kind %d", g.kind);
    ONELLM_REQUIRE(g.q && g.v && g.zb && g.w && g.state && g.out && (keyed ? g.k && g.r && g.A : g.z && g.lower), ONELLM_ERR_ARG,
                   "gated_recurrence: null pointer");
    ONELLM_REQUIRE(g.dk > 0 && g.dk % 16 == 0 && g.dk <= 512 && g.dv > 0 && g.dv == gated_recurrence_pad_dv(g.dv) && g.dv <= 2048, ONELLM_ERR_UNSUPPORTED,
                   "gated_recurrence: key size %d must be a multiple of 16 up to 512, value size %d of 32 per 256 columns up to 2048", g.dk, g.dv);
    ONELLM_REQUIRE(!keyed || (g.rank > 0 && g.rank <= 1024), ONELLM_ERR_UNSUPPORTED, "gated_recurrence: gate rank %d", g.rank);
    ONELLM_REQUIRE(g.H > 0 && g.H <= 65535 && B > 0 && B <= 65535 && g.ld % 8 == 0 && (tp.cu ? tp.hist && g.work && aligned16(g.work) : tp.step && tp.off),
                   ONELLM_ERR_ARG, "gated_recurrence: bad argument");
    const GrParams p = {g, tp};
    return g.dtype == ONELLM_F32 ? dispatch_gr<float>(p, B, tokens, st) : dispatch_gr<__nv_bfloat16>(p, B, tokens, st);
}

}  // namespace onellm

extern "C" size_t onellm_gated_recurrence_workspace(int kind, int tokens, int H, int dk, int dv)
{
    return tokens > 0 && H > 0 && dk > 0 && dv > 0 ? onellm::gated_recurrence_workspace(kind, tokens, H, dk, dv) : 0;
}

extern "C" int onellm_gated_recurrence_run(const onellm_gated_recurrence* g, const onellm_token_positions* tp, int tokens, void* stream)
{
    ONELLM_REQUIRE(g && tp && tokens >= 0, ONELLM_ERR_ARG, "gated_recurrence: bad argument");
    return onellm::gated_recurrence(*g, *tp, tp->B, tokens, reinterpret_cast<cudaStream_t>(stream));
}
