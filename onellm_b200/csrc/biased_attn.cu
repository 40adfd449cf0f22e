// Attention with its own key and value sizes, a score factor per query position and a penalty per head and distance
// (mixers.h: BiasedAttn): the cache store, a plain float form of any phase, and the decode kernel for bfloat16.  The
// tcgen05 form of the context pass is in biased_attn_tc.cu.
//
// Factor and penalty come as tables over positions and distances, in units of log2, built once from the model's
// constants in double precision: a kernel then spends one load and one multiply-add per score on them whatever their
// formula, and every kernel sees the same numbers.
#include <math.h>

#include <algorithm>

#include "mixers.h"

namespace onellm {

// ---- tables ------------------------------------------------------------------------------------------------
__global__ void query_factor_kernel(float* __restrict__ out, int S, double scale, double coef, double every)
{
    for (int p = blockIdx.x * blockDim.x + threadIdx.x; p < S; p += gridDim.x * blockDim.x)
        out[p] = (float)(scale * (1.0 + coef * log(floor((double)(p + 1) / every) + 1.0)) * 1.4426950408889634);
}
__global__ void distance_penalty_kernel(float* __restrict__ out, const float* __restrict__ r1, const float* __restrict__ r2, int S)
{
    const int h = blockIdx.y;
    const double a = r1[h], b = r2[h];
    for (int d = blockIdx.x * blockDim.x + threadIdx.x; d < S; d += gridDim.x * blockDim.x)
        out[(size_t)h * S + d] = (float)(a * log(1.0 + b * (double)d) * 1.4426950408889634);
}

int build_query_factor(float* out, int S, double scale, double coef, double every, cudaStream_t st)
{
    query_factor_kernel<<<(S + 255) / 256, 256, 0, st>>>(out, S, scale, coef, every);
    ONELLM_CHECK_LAUNCH();
    return ONELLM_OK;
}
int build_distance_penalty(float* out, const float* r1, const float* r2, int H, int S, cudaStream_t st)
{
    distance_penalty_kernel<<<dim3((S + 255) / 256, H), 256, 0, st>>>(out, r1, r2, S);
    ONELLM_CHECK_LAUNCH();
    return ONELLM_OK;
}

// ---- cache store -------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128) biased_attn_store_kernel(const BiasedAttn a, const TokenPositions tp, int* __restrict__ overflow)
{
    constexpr int VEC = Vec16<T>::N;
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    int b, pos;
    locate(tp, t, b, pos);
    if (pos < 0 || pos >= a.S) {
        if (threadIdx.x == 0 && overflow) atomicExch(overflow, 1);
        return;
    }
    const int nk = a.G * a.dk / VEC, nv = a.G * a.dv / VEC;
    for (int i = threadIdx.x; i < nk + nv; i += blockDim.x) {
        const bool is_k = i < nk;
        const int e = (is_k ? i : i - nk) * VEC, d = is_k ? a.dk : a.dv, g = e / d, c = e % d;
        const T* src = reinterpret_cast<const T*>(is_k ? a.k : a.v) + (size_t)t * a.ld + e;
        T* dst = reinterpret_cast<T*>(is_k ? a.k_cache : a.v_cache) + (((size_t)b * a.G + g) * a.S + pos) * d + c;
        *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src);
    }
}

int biased_attn_store(const BiasedAttn& a, const TokenPositions& tp, int tokens, int* overflow, cudaStream_t st)
{
    if (tokens <= 0) return ONELLM_OK;
    if (a.dtype == ONELLM_F32)
        ONELLM_CUDA(launch_pdl(biased_attn_store_kernel<float>, dim3(tokens), dim3(128), 0, st, a, tp, overflow));
    else
        ONELLM_CUDA(launch_pdl(biased_attn_store_kernel<__nv_bfloat16>, dim3(tokens), dim3(128), 0, st, a, tp, overflow));
    return ONELLM_OK;
}

// ---- plain form: one warp per (token, head), 32 keys at a time, everything in float ----------------------------
template <typename T>
__global__ void __launch_bounds__(128) biased_attn_plain_kernel(const BiasedAttn a, const TokenPositions tp)
{
    constexpr int VEC = Vec16<T>::N;
    __shared__ __align__(16) float qs[4][256];
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x, h = blockIdx.y * 4 + warp;
    if (h >= a.H) return;
    int b, pos;
    locate(tp, t, b, pos);
    if (pos < 0 || pos >= a.S) return;
    const int g = h / (a.H / a.G);
    const T* q = reinterpret_cast<const T*>(a.q) + (size_t)t * a.ld + (size_t)h * a.dk;
    for (int c = lane; c < a.dk; c += 32) qs[warp][c] = to_float(q[c]);
    __syncwarp();
    const T* kc = reinterpret_cast<const T*>(a.k_cache) + ((size_t)b * a.G + g) * a.S * a.dk;
    const T* vc = reinterpret_cast<const T*>(a.v_cache) + ((size_t)b * a.G + g) * a.S * a.dv;
    const float factor = a.q_factor[pos];
    const float* pen = a.penalty + (size_t)h * a.S;
    float m = -INFINITY, l = 0.f, o[8];
#pragma unroll
    for (int i = 0; i < 8; i++) o[i] = 0.f;
    for (int j0 = 0; j0 <= pos; j0 += 32) {
        const int j = j0 + lane;
        float s = -INFINITY;
        if (j <= pos) {
            const T* kr = kc + (size_t)j * a.dk;
            float acc = 0.f;
            for (int c = 0; c < a.dk; c += VEC) {
                float kf[VEC];
                Vec16<T>::load(kr + c, kf);
#pragma unroll
                for (int e = 0; e < VEC; e++) acc = fmaf(qs[warp][c + e], kf[e], acc);
            }
            s = acc * factor - pen[pos - j];
        }
        const float mn = fmaxf(m, warp_max(s));
        const float corr = exp2f(m - mn), w = exp2f(s - mn);  // key 0 is always visible: mn is finite
        m = mn;
        l = l * corr + w;  // this lane's share
#pragma unroll
        for (int i = 0; i < 8; i++) o[i] *= corr;
        const int n = min(32, pos + 1 - j0);
        for (int jj = 0; jj < n; jj++) {
            const float wj = __shfl_sync(0xffffffffu, w, jj);
            const T* vr = vc + (size_t)(j0 + jj) * a.dv;
#pragma unroll
            for (int i = 0; i < 8; i++)
                if (lane + 32 * i < a.dv) o[i] = fmaf(wj, to_float(vr[lane + 32 * i]), o[i]);
        }
    }
    const float inv = a.out_scale / warp_sum(l);
    T* out = reinterpret_cast<T*>(a.out) + (size_t)t * a.out_ld + (size_t)h * a.dv;
#pragma unroll
    for (int i = 0; i < 8; i++)
        if (lane + 32 * i < a.dv) out[lane + 32 * i] = from_float<T>(o[i] * inv);
}

static int check_attn(const BiasedAttn& a)
{
    ONELLM_REQUIRE(a.q && a.k_cache && a.v_cache && a.q_factor && a.penalty && a.out, ONELLM_ERR_ARG, "biased_attn: null pointer");
    ONELLM_REQUIRE(a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.S > 0, ONELLM_ERR_ARG, "biased_attn: bad size");
    ONELLM_REQUIRE(a.dk > 0 && a.dv > 0 && a.dk % 16 == 0 && a.dv % 16 == 0 && a.dk <= 256 && a.dv <= 256, ONELLM_ERR_UNSUPPORTED,
                   "biased_attn: key size %d and value size %d must be multiples of 16, at most 256", a.dk, a.dv);
    ONELLM_REQUIRE(a.ld % 8 == 0 && a.out_ld % 8 == 0, ONELLM_ERR_ARG, "biased_attn: row strides must be multiples of 8");
    return ONELLM_OK;
}

int biased_attn_tc_launch(const BiasedAttn& a, const TokenPositions& tp, int max_new, cudaStream_t st);  // biased_attn_tc.cu

int biased_attn_context(const BiasedAttn& a, const TokenPositions& tp, int tokens, int max_new, bool plain, cudaStream_t st)
{
    const int rc = check_attn(a);
    if (rc || tokens <= 0) return rc;
    if (a.dtype == ONELLM_BF16 && !plain && tp.cu) return biased_attn_tc_launch(a, tp, max_new, st);
    const dim3 grid(tokens, (a.H + 3) / 4);
    if (a.dtype == ONELLM_F32) ONELLM_CUDA(launch_pdl(biased_attn_plain_kernel<float>, grid, dim3(128), 0, st, a, tp));
    else ONELLM_CUDA(launch_pdl(biased_attn_plain_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, a, tp));
    return ONELLM_OK;
}

// ---- decode step -------------------------------------------------------------------------------------------
// Split-KV, HBM-bound, after the pattern of decode_attn_mma_kernel (decode_attn.cu): a block owns up to 8 query heads
// of one key/value head and one range of cache rows; each warp streams a contiguous part of it through its own cp.async
// ring of 16-row tiles (no block barrier in the loop) and runs q.K^T and P.V on mma.m16n8k16 with the query heads as the
// 8 used rows of the M operand.  Rows in shared memory are padded by 16 bytes (an odd number of 16-byte units, so
// ldmatrix reads any row size without bank conflicts).  The block of the last range takes the new key and value from the
// projection output instead of the cache and stores them.
// DKT / DVT: sizes known at compile time, or 0 for any multiple of 16 up to 256.
constexpr int kBdWarps = 4, kBdRows = 16;

struct BdParams {
    BiasedAttn a;
    TokenPositions tp;
    int heads;       // query heads per block
    int n_split, chunk, nst;
    float* part_o;   // [B, H, n_split, dv]
    float* part_ml;  // [B, H, n_split, 2]
};

__device__ __forceinline__ int bd_splits(int n_cached, int chunk)
{
    const int s = (n_cached + chunk - 1) / chunk;
    return s < 1 ? 1 : s;
}

template <int DKT, int DVT>
__global__ void __launch_bounds__(kBdWarps * 32) biased_attn_decode_kernel(const BdParams p)
{
    typedef __nv_bfloat16 bf16;
    const int dk = DKT ? DKT : p.a.dk, dv = DVT ? DVT : p.a.dv;
    constexpr int KSM = (DKT ? DKT : 256) / 16, VSM = (DVT ? DVT : 256) / 16;  // k steps of q.K^T, column pairs of P.V
    const int krow = dk * 2 + 16, vrow = dv * 2 + 16;                          // bytes per row in shared memory
    const int tile = kBdRows * (krow + vrow);
    extern __shared__ __align__(16) unsigned char ring[];
    __shared__ __align__(16) bf16 q_s[8][256 + 8];
    __shared__ float sm_m[kBdWarps][8], sm_l[kBdWarps][8];

    const int group = p.a.H / p.a.G, per_g = (group + p.heads - 1) / p.heads;
    const int split = blockIdx.x, hk = blockIdx.y / per_g, h_in = (blockIdx.y % per_g) * p.heads, b = blockIdx.z;
    const int h0 = hk * group + h_in, nh = min(p.heads, group - h_in);
    const bool writes_cache = h_in == 0;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;

    int bb, n_cached;  // the query's position = rows already in the cache
    locate(p.tp, b, bb, n_cached);
    const int n_split = bd_splits(n_cached, p.chunk);
    if (split >= n_split || n_cached < 0 || n_cached >= p.a.S) {
        pdl_launch_dependents();
        pdl_wait();
        return;
    }
    const bool owns_new = split == n_split - 1;
    const int row0 = split * p.chunk;
    const int row1 = min(row0 + p.chunk, n_cached) + (owns_new ? 1 : 0);
    int per_warp = (row1 - row0 + kBdWarps - 1) / kBdWarps;
    per_warp = (per_warp + kBdRows - 1) / kBdRows * kBdRows;
    const int wr0 = min(row0 + warp * per_warp, row1), wr1 = min(wr0 + per_warp, row1);
    const int n_tiles = (wr1 - wr0 + kBdRows - 1) / kBdRows;

    bf16* kc = reinterpret_cast<bf16*>(p.a.k_cache) + ((size_t)b * p.a.G + hk) * p.a.S * dk;
    bf16* vc = reinterpret_cast<bf16*>(p.a.v_cache) + ((size_t)b * p.a.G + hk) * p.a.S * dv;
    const int nst = p.nst;
    const uint32_t ring_base = (uint32_t)__cvta_generic_to_shared(ring) + (uint32_t)(warp * nst * tile);
    unsigned char* ring_gen = ring + (size_t)warp * nst * tile;

    // rows at or beyond n_cached are not in the cache yet: zero-filled
    const int kch = dk / 8, vch = dv / 8;
    auto issue = [&](int it, int buf) {
        if (it < n_tiles) {
            const int r0 = wr0 + it * kBdRows;
            const uint32_t sb = ring_base + (uint32_t)(buf * tile);
#pragma unroll
            for (int i = 0; i < KSM; i++) {  // 16 rows * dk / 8 chunks over 32 lanes = dk / 16 rounds
                if (!DKT && i >= dk / 16) break;
                const int id = lane + 32 * i, row = id / kch, c = id % kch, rr = r0 + row;
                const bool ok = rr < wr1 && rr < n_cached;
                cp_async16(sb + row * krow + c * 16, kc + (ok ? (size_t)rr * dk + c * 8 : 0), ok ? 16 : 0);
            }
            const uint32_t vb = sb + kBdRows * krow;
#pragma unroll
            for (int i = 0; i < VSM; i++) {
                if (!DVT && i >= dv / 16) break;
                const int id = lane + 32 * i, row = id / vch, c = id % vch, rr = r0 + row;
                const bool ok = rr < wr1 && rr < n_cached;
                cp_async16(vb + row * vrow + c * 16, vc + (ok ? (size_t)rr * dv + c * 8 : 0), ok ? 16 : 0);
            }
        }
        cp_async_commit();
    };
    for (int s = 0; s < nst - 1; s++) issue(s, s);

    // penalties of the four keys this thread scores for head g, one tile ahead
    const float* pen = p.a.penalty + (size_t)(h0 + min(g, nh - 1)) * p.a.S;
    float pn[4];
    auto load_pen = [&](int it) {
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int j = wr0 + it * kBdRows + 2 * t + (e & 1) + (e & 2) * 4;
            pn[e] = pen[max(n_cached - j, 0)];
        }
    };
    load_pen(0);
    const float factor = p.a.q_factor[n_cached];
    pdl_wait();

    for (int i = threadIdx.x; i < 8 * kch; i += kBdWarps * 32) {
        const int head = i / kch, c = i % kch;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (head < nh)
            v = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(p.a.q) + (size_t)b * p.a.ld + (size_t)(h0 + head) * dk + c * 8);
        *reinterpret_cast<uint4*>(&q_s[head][c * 8]) = v;
    }
    __syncthreads();
    uint32_t qa[KSM][2];  // (head g, d 16ks + 2t ..) and (head g, d 16ks + 8 + 2t ..)
#pragma unroll
    for (int ks = 0; ks < KSM; ks++) {
        qa[ks][0] = qa[ks][1] = 0u;
        if (DKT || ks < dk / 16) {
            qa[ks][0] = *reinterpret_cast<const uint32_t*>(&q_s[g][16 * ks + 2 * t]);
            qa[ks][1] = *reinterpret_cast<const uint32_t*>(&q_s[g][16 * ks + 8 + 2 * t]);
        }
    }
    float O[2 * VSM][2];
#pragma unroll
    for (int j = 0; j < 2 * VSM; j++) O[j][0] = O[j][1] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;

    const int mi = lane >> 3, lr = lane & 7;
    const uint32_t k_off = (uint32_t)((lr + (mi >> 1) * 8) * krow + (mi & 1) * 16);
    const uint32_t v_off = (uint32_t)(kBdRows * krow + (lr + (mi & 1) * 8) * vrow + (mi >> 1) * 16);
    int buf = 0, fill = nst - 1;
    for (int it = 0; it < n_tiles; it++) {
        cp_async_wait_dyn(nst - 2);
        __syncwarp();
        const int r0 = wr0 + it * kBdRows;
        const uint32_t sb = ring_base + (uint32_t)(buf * tile);
        if (owns_new && n_cached >= r0 && n_cached < r0 + kBdRows && n_cached < wr1) {
            // the new row: projection output -> tile and cache
            const int row = n_cached - r0;
            for (int c = lane; c < kch + vch; c += 32) {
                const bool is_k = c < kch;
                const int cc = is_k ? c : c - kch;
                const bf16* src = reinterpret_cast<const bf16*>(is_k ? p.a.k : p.a.v) + (size_t)b * p.a.ld + (size_t)hk * (is_k ? dk : dv) + cc * 8;
                const uint4 v = *reinterpret_cast<const uint4*>(src);
                unsigned char* sm = ring_gen + (size_t)buf * tile + (is_k ? row * krow : kBdRows * krow + row * vrow) + cc * 16;
                *reinterpret_cast<uint4*>(sm) = v;
                if (writes_cache) *reinterpret_cast<uint4*>(is_k ? kc + (size_t)n_cached * dk + cc * 8 : vc + (size_t)n_cached * dv + cc * 8) = v;
            }
            __syncwarp();
        }
        issue(it + nst - 1, fill);
        buf = buf + 1 == nst ? 0 : buf + 1;
        fill = fill + 1 == nst ? 0 : fill + 1;
        float cur[4] = {pn[0], pn[1], pn[2], pn[3]};
        load_pen(it + 1);

        float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int ks = 0; ks < KSM; ks++) {
            if (!DKT && ks >= dk / 16) break;
            uint32_t kb[4];
            ldsm_x4(kb, sb + k_off + ks * 32);
            mma_bf16(s0, qa[ks][0], 0u, qa[ks][1], 0u, kb[0], kb[1]);
            mma_bf16(s1, qa[ks][0], 0u, qa[ks][1], 0u, kb[2], kb[3]);
        }
        const int valid = wr1 - r0;
        float sc[4];
        sc[0] = (2 * t < valid) ? fmaf(s0[0], factor, -cur[0]) : -INFINITY;
        sc[1] = (2 * t + 1 < valid) ? fmaf(s0[1], factor, -cur[1]) : -INFINITY;
        sc[2] = (8 + 2 * t < valid) ? fmaf(s1[0], factor, -cur[2]) : -INFINITY;
        sc[3] = (9 + 2 * t < valid) ? fmaf(s1[1], factor, -cur[3]) : -INFINITY;
        float mx = fmaxf(fmaxf(sc[0], sc[1]), fmaxf(sc[2], sc[3]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m_run, mx);
        const float ms = (m_new == -INFINITY) ? 0.f : m_new;
        const float corr = fast_exp2(m_run - ms);
        m_run = m_new;
        float pr[4];
#pragma unroll
        for (int e = 0; e < 4; e++) pr[e] = fast_exp2(sc[e] - ms);
        l_run = l_run * corr + (pr[0] + pr[1] + pr[2] + pr[3]);
        const uint32_t pa0 = pack2<bf16>(pr[0], pr[1]), pa2 = pack2<bf16>(pr[2], pr[3]);
#pragma unroll
        for (int j = 0; j < 2 * VSM; j++) {
            O[j][0] *= corr;
            O[j][1] *= corr;
        }
#pragma unroll
        for (int jp = 0; jp < VSM; jp++) {
            if (!DVT && jp >= dv / 16) break;
            uint32_t vb[4];
            ldsm_x4_t(vb, sb + v_off + jp * 32);
            float o0[4] = {O[2 * jp][0], O[2 * jp][1], 0.f, 0.f}, o1[4] = {O[2 * jp + 1][0], O[2 * jp + 1][1], 0.f, 0.f};
            mma_bf16(o0, pa0, 0u, pa2, 0u, vb[0], vb[1]);
            mma_bf16(o1, pa0, 0u, pa2, 0u, vb[2], vb[3]);
            O[2 * jp][0] = o0[0];
            O[2 * jp][1] = o0[1];
            O[2 * jp + 1][0] = o1[0];
            O[2 * jp + 1][1] = o1[1];
        }
    }
    cp_async_wait<0>();
    pdl_launch_dependents();
    __syncthreads();  // every warp is done with its ring before it is reused below

    l_run += __shfl_xor_sync(0xffffffffu, l_run, 1);
    l_run += __shfl_xor_sync(0xffffffffu, l_run, 2);
    float* sm_o = reinterpret_cast<float*>(ring);  // [warps][8][dv]
#pragma unroll
    for (int j = 0; j < 2 * VSM; j++) {
        if (!DVT && j >= dv / 8) break;
        *reinterpret_cast<float2*>(&sm_o[(warp * 8 + g) * dv + 8 * j + 2 * t]) = make_float2(O[j][0], O[j][1]);
    }
    if (t == 0) {
        sm_m[warp][g] = m_run;
        sm_l[warp][g] = l_run;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nh * dv; i += kBdWarps * 32) {
        const int gg = i / dv, d = i % dv, h = h0 + gg;
        float M = -INFINITY;
#pragma unroll
        for (int w = 0; w < kBdWarps; w++) M = fmaxf(M, sm_m[w][gg]);
        float L = 0.f, Ov = 0.f;
#pragma unroll
        for (int w = 0; w < kBdWarps; w++) {
            const float c = fast_exp2(sm_m[w][gg] - M);  // warps without rows: exp2(-inf) = 0
            L = fmaf(sm_l[w][gg], c, L);
            Ov = fmaf(sm_o[(w * 8 + gg) * dv + d], c, Ov);
        }
        if (n_split == 1) {
            reinterpret_cast<bf16*>(p.a.out)[(size_t)b * p.a.out_ld + (size_t)h * dv + d] = __float2bfloat16_rn(Ov / L * p.a.out_scale);
        } else {
            const size_t base = ((size_t)b * p.a.H + h) * p.n_split + split;
            p.part_o[base * dv + d] = Ov;
            if (d == 0) {
                p.part_ml[base * 2] = M;
                p.part_ml[base * 2 + 1] = L;
            }
        }
    }
}

// Merges the per-split partials: out = sum_i O_i 2^(m_i - M) / sum_i L_i 2^(m_i - M).
__global__ void __launch_bounds__(128) biased_attn_merge_kernel(const BdParams p)
{
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, b = blockIdx.y, dv = p.a.dv;
    int bb, n_cached;
    locate(p.tp, b, bb, n_cached);
    const int n_split = bd_splits(n_cached, p.chunk);
    if (n_split == 1) return;  // the attention kernel wrote the output itself
    const size_t base = ((size_t)b * p.a.H + h) * p.n_split;
    float M = -INFINITY;
    for (int i = 0; i < n_split; i++) M = fmaxf(M, p.part_ml[(base + i) * 2]);
    float L = 0.f;
    for (int i = 0; i < n_split; i++) L = fmaf(p.part_ml[(base + i) * 2 + 1], fast_exp2(p.part_ml[(base + i) * 2] - M), L);
    const float inv = p.a.out_scale / L;
    for (int d = threadIdx.x; d < dv; d += blockDim.x) {
        float O = 0.f;
        for (int i = 0; i < n_split; i++) O = fmaf(p.part_o[(base + i) * dv + d], fast_exp2(p.part_ml[(base + i) * 2] - M), O);
        reinterpret_cast<__nv_bfloat16*>(p.a.out)[(size_t)b * p.a.out_ld + (size_t)h * dv + d] = __float2bfloat16_rn(O * inv);
    }
}

constexpr int kBdMaxSplits = 32;

size_t biased_attn_decode_workspace(int B, int H, int dv) { return (size_t)B * H * kBdMaxSplits * (dv + 2) * sizeof(float); }

template <int DKT, int DVT>
static int launch_bd(const BdParams& p, dim3 grid, size_t smem, cudaStream_t st)
{
    auto kern = biased_attn_decode_kernel<DKT, DVT>;
    static DeviceOnce attr;
    ONELLM_CUDA(attr.run([kern] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024); }));
    ONELLM_CUDA(launch_pdl(kern, grid, dim3(kBdWarps * 32), smem, st, p));
    return ONELLM_OK;
}

int biased_attn_decode(const BiasedAttn& a, const TokenPositions& tp, int step_bound, void* workspace, cudaStream_t st)
{
    const int rc = check_attn(a);
    if (rc) return rc;
    ONELLM_REQUIRE(a.dtype == ONELLM_BF16 && a.k && a.v && workspace && !tp.cu && tp.step && tp.B >= 1, ONELLM_ERR_ARG, "biased_attn_decode: bad argument");
    const int group = a.H / a.G, heads = std::min(group, 8), per_g = (group + heads - 1) / heads;
    const long pairs = (long)tp.B * a.G * per_g;
    const size_t tile = (size_t)kBdRows * ((a.dk + a.dv) * 2 + 32);
    // Two blocks per SM share its memory when their rings are at least three tiles deep, else one.
    const size_t merge = (size_t)kBdWarps * 8 * a.dv * sizeof(float);
    int per_sm = 2;
    int nst = (int)((size_t)108 * 1024 / (kBdWarps * tile));
    if (nst < 3) {
        per_sm = 1;
        nst = (int)((size_t)216 * 1024 / (kBdWarps * tile));
    }
    nst = std::min(nst, 8);
    ONELLM_REQUIRE(nst >= 2, ONELLM_ERR_UNSUPPORTED, "biased_attn_decode: key size %d + value size %d", a.dk, a.dv);
    // Ranges per (sequence, head) pair: the count with the least estimated time, from the rows a block streams at its
    // share of the memory rate, a fixed cost per wave of blocks and the merge launch behind a split.
    const int rows = std::max(step_bound - 1, 1);
    const long slots = (long)per_sm * num_sms();
    const double row_us = (double)(a.dk + a.dv) * 2.0 / (6.5e6 / (double)slots);
    int best = 1, best_chunk = (rows + 63) / 64 * 64;
    double best_t = 1e300;
    for (int n = 1; n <= kBdMaxSplits; n++) {
        const int c = ((rows + n - 1) / n + 63) / 64 * 64, ns = (rows + c - 1) / c;
        const long waves = (pairs * ns + slots - 1) / slots;
        // a block alone on the chip cannot use the whole rate: about four times its even share
        const double share = std::max(0.25, std::min(1.0, (double)(pairs * ns) / (double)slots));
        const double t = (double)waves * (c * row_us * share + 1.5) + (ns > 1 ? 4.0 : 0.0);
        if (t < best_t - 1e-9) {
            best_t = t;
            best = ns;
            best_chunk = c;
        }
    }
    BdParams p = {a, tp, heads, best, best_chunk, nst, (float*)workspace, nullptr};
    p.part_ml = p.part_o + (size_t)tp.B * a.H * kBdMaxSplits * a.dv;
    const dim3 grid(best, a.G * per_g, tp.B);
    const size_t smem = std::max((size_t)kBdWarps * nst * tile, merge);
    int e;
    if (a.dk == 128 && a.dv == 128) e = launch_bd<128, 128>(p, grid, smem, st);
    else if (a.dk == 64 && a.dv == 128) e = launch_bd<64, 128>(p, grid, smem, st);
    else if (a.dk == 64 && a.dv == 64) e = launch_bd<64, 64>(p, grid, smem, st);
    else e = launch_bd<0, 0>(p, grid, smem, st);
    if (e) return e;
    if (best > 1) ONELLM_CUDA(launch_pdl(biased_attn_merge_kernel, dim3(a.H, tp.B), dim3(128), 0, st, p));
    return ONELLM_OK;
}

}  // namespace onellm

using namespace onellm;

extern "C" int onellm_query_factor(float* out, int S, double scale, double coef, double every, void* stream)
{
    ONELLM_REQUIRE(out && S > 0 && every > 0.0, ONELLM_ERR_ARG, "query_factor: bad argument");
    return build_query_factor(out, S, scale, coef, every, reinterpret_cast<cudaStream_t>(stream));
}

extern "C" int onellm_distance_penalty(float* out, const float* r1, const float* r2, int H, int S, void* stream)
{
    ONELLM_REQUIRE(out && r1 && r2 && H > 0 && H <= 65535 && S > 0, ONELLM_ERR_ARG, "distance_penalty: bad argument");
    return build_distance_penalty(out, r1, r2, H, S, reinterpret_cast<cudaStream_t>(stream));
}

extern "C" int onellm_biased_attn_store(const onellm_biased_attn* a, const onellm_token_positions* tp, int tokens, int* overflow, void* stream)
{
    ONELLM_REQUIRE(a && tp && a->k && a->v, ONELLM_ERR_ARG, "biased_attn_store: null pointer");
    const int rc = check_attn(*a);
    if (rc) return rc;
    return biased_attn_store(*a, *tp, tokens, overflow, reinterpret_cast<cudaStream_t>(stream));
}

extern "C" int onellm_biased_attn_context(const onellm_biased_attn* a, const onellm_token_positions* tp, int tokens, int max_new, int plain,
                                          void* stream)
{
    ONELLM_REQUIRE(a && tp && tokens >= 0 && max_new >= 0, ONELLM_ERR_ARG, "biased_attn_context: bad argument");
    return biased_attn_context(*a, *tp, tokens, max_new, plain != 0, reinterpret_cast<cudaStream_t>(stream));
}

extern "C" size_t onellm_biased_attn_decode_workspace(int B, int H, int dv) { return biased_attn_decode_workspace(B, H, dv); }

extern "C" int onellm_biased_attn_decode(const onellm_biased_attn* a, const onellm_token_positions* tp, int step_bound, void* workspace,
                                         void* stream)
{
    ONELLM_REQUIRE(a && tp && step_bound >= 1, ONELLM_ERR_ARG, "biased_attn_decode: bad argument");
    return biased_attn_decode(*a, *tp, step_bound, workspace, reinterpret_cast<cudaStream_t>(stream));
}
