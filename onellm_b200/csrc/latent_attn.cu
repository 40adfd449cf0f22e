// Attention over latents in a sliding window (mixers.h: LatentAttn): the norms in front of it with the cache store, and the
// attention itself in latent space.
//
// Keys and values of all heads are linear in one latent per token, so with the queries turned into latent space beforehand
// (q' = W_uk^T q, a per-head projection) a head's score is q' . c and its output is W_uv applied to the weighted latent:
// every head reads the same rows and only those are cached.  They lie in a ring as long as the window, so a sequence's
// memory does not grow with its length.
//
// Decode steps run on tcgen05 (latent_attn_tc.cu).  The kernel here (short portions of a prompt, at most 64 tokens, and
// decode steps with latents above 512) owns up to 16 heads of one token and one range of its keys: 16 is the row operand of
// mma.m16n8k16, so heads beyond the first are free.  Tiles of 32 latents go
// through a cp.async ring; the eight warps first share the scores out by keys and halves of the rank, then the outputs by
// 16-column groups of the same tile, which is key and value at once.  Tiles that hold no token of this very pass are
// requested before the dependency wait.  Whole prompts are cheaper with the keys and values formed once per token
// (biased_attn_tc.cu, window_attn).
#include <math.h>

#include <algorithm>

#include "mixers.h"

namespace onellm {

// positions a sequence brings along from its ring into a joined buffer
__device__ __forceinline__ int kept_rows(const LatentAttn& a, int hist) { return min(hist, a.window - 1); }
// first row of sequence b in a joined buffer
__device__ __forceinline__ int joined_base(const LatentAttn& a, const TokenPositions& tp, int b)
{
    int base = tp.cu[b];
    for (int i = 0; i < b; i++) base += kept_rows(a, tp.hist[i]);
    return base;
}
// row of local token i of sequence b in the fresh buffer of a context pass
__device__ __forceinline__ int fresh_row(const LatentAttn& a, const TokenPositions& tp, int b, int i)
{
    return a.joined ? joined_base(a, tp, b) + kept_rows(a, tp.hist[b]) + i : tp.cu[b] + i;
}

// ---- norms and store ---------------------------------------------------------------------------------------
constexpr int kLsThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kLsThreads) latent_store_kernel(const LatentAttn a, const TokenPositions tp, int rank_p)
{
    constexpr int VEC = Vec16<T>::N;
    __shared__ float part[2][kLsThreads / 32];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    int b, pos;
    locate(tp, t, b, pos);
    T* dst;
    if (tp.cu) dst = static_cast<T*>(a.fresh) + (size_t)fresh_row(a, tp, b, t - tp.cu[b]) * rank_p;
    else dst = static_cast<T*>(a.ring) + ((size_t)b * a.R + pos % a.R) * rank_p;
    const T* qs = static_cast<const T*>(a.q_src) + (size_t)t * a.ld;
    const T* ks = static_cast<const T*>(a.kv_src) + (size_t)t * a.ld;
    const int nq = a.q_ld / VEC, nk = rank_p / VEC;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < nq + nk; i += kLsThreads) {
        float f[VEC], s = 0.f;
        Vec16<T>::load(i < nq ? qs + (size_t)i * VEC : ks + (size_t)(i - nq) * VEC, f);
#pragma unroll
        for (int e = 0; e < VEC; e++) s = fmaf(f[e], f[e], s);
        if (i < nq) sq += s;
        else sk += s;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) {
        part[0][threadIdx.x >> 5] = sq;
        part[1][threadIdx.x >> 5] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < kLsThreads / 32; i++) {
        sq += part[0][i];
        sk += part[1][i];
    }
    const float iq = 1.f / sqrtf(sq / (float)a.q_width + a.eps), ik = 1.f / sqrtf(sk / (float)a.rank + a.eps);
    for (int i = threadIdx.x; i < nq + nk; i += kLsThreads) {
        const bool q = i < nq;
        const int c = (q ? i : i - nq) * VEC;
        float f[VEC];
        Vec16<T>::load((q ? qs : ks) + c, f);
        const float* w = (q ? a.q_w : a.kv_w) + c;
        const float inv = q ? iq : ik;
#pragma unroll
        for (int e = 0; e < VEC; e++) f[e] *= inv * w[e];
        *reinterpret_cast<uint4*>(q ? static_cast<T*>(a.q_out) + (size_t)t * a.q_ld + c : dst + c) = Vec16<T>::pack(f);
    }
}

// Rows between a ring and the fresh buffer of a context pass, one warp per row: TO_RING: the last latents of every sequence
// into its ring; else the rows a joined buffer brings along.
template <typename T, bool TO_RING>
__global__ void __launch_bounds__(256) latent_rows_kernel(const LatentAttn a, const TokenPositions tp, int rank_p)
{
    constexpr int VEC = Vec16<T>::N;
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.y, i = blockIdx.x * 8 + (threadIdx.x >> 5), hist = tp.hist[b];
    T *ring, *fresh;
    if (TO_RING) {
        const int n_new = tp.cu[b + 1] - tp.cu[b];
        if (i >= min(n_new, a.R)) return;
        const int local = n_new - 1 - i;
        ring = static_cast<T*>(a.ring) + ((size_t)b * a.R + (hist + local) % a.R) * rank_p;
        fresh = static_cast<T*>(a.fresh) + (size_t)fresh_row(a, tp, b, local) * rank_p;
    } else {
        const int kept = kept_rows(a, hist);
        if (i >= kept) return;
        ring = static_cast<T*>(a.ring) + ((size_t)b * a.R + (hist - kept + i) % a.R) * rank_p;
        fresh = static_cast<T*>(a.fresh) + (size_t)(joined_base(a, tp, b) + i) * rank_p;
    }
    const uint4* src = reinterpret_cast<const uint4*>(TO_RING ? fresh : ring);
    uint4* dst = reinterpret_cast<uint4*>(TO_RING ? ring : fresh);
    for (int c = threadIdx.x & 31; c < rank_p / VEC; c += 32) dst[c] = src[c];
}

static int check_latent(const LatentAttn& a)
{
    ONELLM_REQUIRE(a.H > 0 && a.rank > 0 && a.window > 0 && a.R > 0, ONELLM_ERR_ARG, "latent_attn: bad size");
    ONELLM_REQUIRE(a.dtype == ONELLM_BF16 || a.dtype == ONELLM_F32, ONELLM_ERR_UNSUPPORTED, "latent_attn: dtype %d", a.dtype);
    ONELLM_REQUIRE(a.rank <= 1024, ONELLM_ERR_UNSUPPORTED, "latent_attn: latents of %d elements (at most 1024)", a.rank);
    ONELLM_REQUIRE(a.ring && aligned16(a.ring), ONELLM_ERR_ARG, "latent_attn: ring");
    return ONELLM_OK;
}

template <bool TO_RING>
static int latent_rows(const LatentAttn& a, const TokenPositions& tp, int rows, cudaStream_t st)
{
    if (rows <= 0) return ONELLM_OK;
    const dim3 grid((rows + 7) / 8, tp.B);
    if (a.dtype == ONELLM_F32) ONELLM_CUDA(launch_pdl(latent_rows_kernel<float, TO_RING>, grid, dim3(256), 0, st, a, tp, latent_pad(a.rank)));
    else ONELLM_CUDA(launch_pdl(latent_rows_kernel<__nv_bfloat16, TO_RING>, grid, dim3(256), 0, st, a, tp, latent_pad(a.rank)));
    return ONELLM_OK;
}

int latent_store(const LatentAttn& a, const TokenPositions& tp, int tokens, int max_hist, cudaStream_t st)
{
    RC(check_latent(a));
    ONELLM_REQUIRE(a.q_src && a.kv_src && a.q_w && a.kv_w && a.q_out && a.q_width > 0 && a.q_ld % 8 == 0 && a.ld % 8 == 0 && (!tp.cu || (a.fresh && tp.hist)),
                   ONELLM_ERR_ARG, "latent_store: bad argument");
    if (tokens <= 0) return ONELLM_OK;
    if (a.dtype == ONELLM_F32)
        ONELLM_CUDA(launch_pdl(latent_store_kernel<float>, dim3(tokens), dim3(kLsThreads), 0, st, a, tp, latent_pad(a.rank)));
    else
        ONELLM_CUDA(launch_pdl(latent_store_kernel<__nv_bfloat16>, dim3(tokens), dim3(kLsThreads), 0, st, a, tp, latent_pad(a.rank)));
    return tp.cu && a.joined ? latent_rows<false>(a, tp, std::min(max_hist, a.window - 1), st) : ONELLM_OK;
}

int latent_keep(const LatentAttn& a, const TokenPositions& tp, int max_new, cudaStream_t st)
{
    RC(check_latent(a));
    ONELLM_REQUIRE(tp.cu && tp.hist && a.fresh, ONELLM_ERR_ARG, "latent_keep: needs a context pass");
    return latent_rows<true>(a, tp, std::min(max_new, a.R), st);
}

// ---- attention ---------------------------------------------------------------------------------------------
// where the latent of position j of sequence b lies
template <typename T>
__device__ __forceinline__ const T* latent_at(const LatentAttn& a, const TokenPositions& tp, int rank_p, int b, int fresh0, int first, int j)
{
    return j >= fresh0 ? static_cast<const T*>(a.fresh) + (size_t)(first + j - fresh0) * rank_p
                       : static_cast<const T*>(a.ring) + ((size_t)b * a.R + j % a.R) * rank_p;
}
__device__ __forceinline__ float sigmoid_of(float x) { return 1.f / (1.f + expf(-x)); }

template <typename T>
__device__ __forceinline__ float out_factor(const LatentAttn& a, int t, int h)
{
    return a.out_scale * (a.gate ? sigmoid_of(to_float(static_cast<const T*>(a.gate)[(size_t)t * a.gate_ld + h])) : 1.f);
}

// Plain form: one warp per (token, head), 32 keys at a time, everything in float.
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_plain_kernel(const LatentAttn a, const TokenPositions tp, int rank_p)
{
    constexpr int VEC = Vec16<T>::N;
    __shared__ __align__(16) float qs[4][1024];
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x, h = blockIdx.y * 4 + warp;
    if (h >= a.H) return;
    int b, pos;
    locate(tp, t, b, pos);
    const int fresh0 = tp.cu ? tp.hist[b] : pos + 1, first = tp.cu ? fresh_row(a, tp, b, 0) : 0;
    const T* q = static_cast<const T*>(a.q) + ((size_t)t * a.H + h) * rank_p;
    for (int c = lane; c < rank_p; c += 32) qs[warp][c] = to_float(q[c]) * a.scale;
    __syncwarp();
    const int lo = max(0, pos - a.window + 1);
    float m = -INFINITY, l = 0.f, o[32];
#pragma unroll
    for (int i = 0; i < 32; i++) o[i] = 0.f;
    for (int j0 = lo; j0 <= pos; j0 += 32) {
        const int j = j0 + lane;
        float s = -INFINITY;
        if (j <= pos) {
            const T* c = latent_at<T>(a, tp, rank_p, b, fresh0, first, j);
            s = 0.f;
            for (int e0 = 0; e0 < rank_p; e0 += VEC) {
                float f[VEC];
                Vec16<T>::load(c + e0, f);
#pragma unroll
                for (int e = 0; e < VEC; e++) s = fmaf(qs[warp][e0 + e], f[e], s);
            }
        }
        const float mn = fmaxf(m, warp_max(s));
        const float corr = expf(m - mn), w = expf(s - mn);  // the first key is visible: mn is finite
        m = mn;
        l = l * corr + w;  // this lane's share
#pragma unroll
        for (int i = 0; i < 32; i++) o[i] *= corr;
        const int n = min(32, pos + 1 - j0);
        for (int jj = 0; jj < n; jj++) {
            const float wj = __shfl_sync(0xffffffffu, w, jj);
            const T* c = latent_at<T>(a, tp, rank_p, b, fresh0, first, j0 + jj);
#pragma unroll
            for (int i = 0; i < 32; i++)
                if (lane + 32 * i < rank_p) o[i] = fmaf(wj, to_float(c[lane + 32 * i]), o[i]);
        }
    }
    const float f = out_factor<T>(a, t, h) / warp_sum(l);
    T* out = static_cast<T*>(a.out) + ((size_t)t * a.H + h) * rank_p;
#pragma unroll
    for (int i = 0; i < 32; i++)
        if (lane + 32 * i < rank_p) out[lane + 32 * i] = from_float<T>(o[i] * f);
}

constexpr int kLaWarps = 8, kLaKeys = 32, kLaHeads = 16;

struct LaParams {
    LatentAttn a;
    TokenPositions tp;
    int rank_p, nst, n_split, chunk;
    float* part_o;   // [T, H, n_split, rank_p]
    float* part_ml;  // [T, H, n_split, 2]
};

__device__ __forceinline__ void ldsm_x2(uint32_t (&r)[2], uint32_t addr)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}

// bytes of the fixed part of the shared memory: queries, scores, weights, row factors
static size_t la_fixed_bytes(int rank_p)
{
    return (size_t)kLaHeads * (rank_p * 2 + 16) + 2 * kLaHeads * (kLaKeys + 1) * 4 + kLaHeads * (kLaKeys + 8) * 2 + 2 * kLaHeads * 4;
}
static size_t la_tile_bytes(int rank_p) { return (size_t)kLaKeys * (rank_p * 2 + 16); }

// NP: 16-column groups of a warp, rank_p <= 128 NP
template <int NP>
__global__ void __launch_bounds__(kLaWarps * 32) latent_attn_kernel(const LaParams p)
{
    typedef __nv_bfloat16 bf16;
    const LatentAttn& a = p.a;
    const int rank_p = p.rank_p, row_bytes = rank_p * 2 + 16, tile = kLaKeys * row_bytes, nst = p.nst;
    extern __shared__ __align__(16) unsigned char smem[];
    const uint32_t ring = (uint32_t)__cvta_generic_to_shared(smem), q_base = ring + nst * tile;
    unsigned char* q_gen = smem + (size_t)nst * tile;
    float* S = reinterpret_cast<float*>(q_gen + kLaHeads * row_bytes);  // [2][16][33]: the two halves of the rank
    bf16* P = reinterpret_cast<bf16*>(S + 2 * kLaHeads * (kLaKeys + 1));  // [16][40]
    float* corr_s = reinterpret_cast<float*>(P + kLaHeads * (kLaKeys + 8));
    float* l_s = corr_s + kLaHeads;
    const uint32_t p_base = (uint32_t)__cvta_generic_to_shared(P);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
    const int split = blockIdx.x, h0 = blockIdx.y * kLaHeads, t = blockIdx.z, nh = min(kLaHeads, a.H - h0);

    int b, pos;
    locate(p.tp, t, b, pos);
    const int lo = max(0, pos - a.window + 1), n_keys = pos + 1 - lo;
    const int used = max(1, (n_keys + p.chunk - 1) / p.chunk);
    if (split >= used || n_keys <= 0) {
        pdl_launch_dependents();
        pdl_wait();
        return;
    }
    // latents of this pass: from fresh0 on, in the fresh buffer (a decode step has put its one into the ring)
    const int fresh0 = p.tp.cu ? p.tp.hist[b] : pos + 1, first = p.tp.cu ? fresh_row(a, p.tp, b, 0) : 0;
    const int new0 = p.tp.cu ? p.tp.hist[b] : pos;
    const int k0 = lo + split * p.chunk, k1 = min(k0 + p.chunk, pos + 1);
    const int n_tiles = (k1 - k0 + kLaKeys - 1) / kLaKeys;
    const int chunks = rank_p / 8;
    auto issue = [&](int it) {
        if (it < n_tiles) {
            const uint32_t dst = ring + (uint32_t)((it % nst) * tile);
#pragma unroll
            for (int r = 0; r < kLaKeys / kLaWarps; r++) {
                const int row = warp * (kLaKeys / kLaWarps) + r, j = k0 + it * kLaKeys + row;
                const bool ok = j < k1;  // rows behind the range are zero: they take part in no sum
                const bf16* src = latent_at<bf16>(a, p.tp, rank_p, b, fresh0, first, ok ? j : k0);
                for (int c = lane; c < chunks; c += 32) cp_async16(dst + row * row_bytes + c * 16, src + c * 8, ok ? 16 : 0);
            }
        }
        cp_async_commit();
    };
    int early = 0;
    while (early < nst - 1 && k0 + (early + 1) * kLaKeys <= new0) issue(early++);
    pdl_wait();
    for (int it = early; it < nst - 1; it++) issue(it);
    for (int i = threadIdx.x; i < kLaHeads * chunks; i += kLaWarps * 32) {
        const int head = i / chunks, c = i % chunks;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (head < nh) v = reinterpret_cast<const uint4*>(static_cast<const bf16*>(a.q) + ((size_t)t * a.H + h0 + head) * rank_p)[c];
        *reinterpret_cast<uint4*>(q_gen + head * row_bytes + c * 16) = v;
    }
    const float scale = a.scale * 1.4426950408889634f;
    float O[NP][2][4];
#pragma unroll
    for (int i = 0; i < NP; i++)
#pragma unroll
        for (int n = 0; n < 2; n++) O[i][n][0] = O[i][n][1] = O[i][n][2] = O[i][n][3] = 0.f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};  // rows 2 warp, 2 warp + 1
    // scores: this warp's eight keys and half of the rank
    const int key8 = warp & 3, half = warp >> 2, n_ks = rank_p / 16, ks0 = half ? (n_ks + 1) / 2 : 0, ks1 = half ? n_ks : (n_ks + 1) / 2;
    const uint32_t qa_off = q_base + (uint32_t)((lane & 15) * row_bytes + (lane >> 4) * 16);
    const uint32_t kb_off = (uint32_t)((key8 * 8 + (lane & 7)) * row_bytes + ((lane >> 3) & 1) * 16);
    // outputs: 16 keys x 16 columns per ldmatrix
    const int mi = lane >> 3, lr = lane & 7;
    const uint32_t v_off = (uint32_t)((lr + (mi & 1) * 8) * row_bytes + (mi >> 1) * 16);
    const uint32_t pa_off = p_base + (uint32_t)((lane & 15) * (kLaKeys + 8) * 2 + (lane >> 4) * 16);
    for (int it = 0; it < n_tiles; it++) {
        cp_async_wait_dyn(nst - 2);
        __syncthreads();
        issue(it + nst - 1);
        const uint32_t sb = ring + (uint32_t)((it % nst) * tile);
        {
            float s[4] = {0.f, 0.f, 0.f, 0.f};
            for (int ks = ks0; ks < ks1; ks++) {
                uint32_t qa[4], kb[2];
                ldsm_x4(qa, qa_off + ks * 32);
                ldsm_x2(kb, sb + kb_off + ks * 32);
                mma_bf16(s, qa[0], qa[1], qa[2], qa[3], kb[0], kb[1]);
            }
            float* dst = S + (half * kLaHeads + g) * (kLaKeys + 1) + key8 * 8 + 2 * tq;
            dst[0] = s[0];
            dst[1] = s[1];
            dst[8 * (kLaKeys + 1)] = s[2];
            dst[8 * (kLaKeys + 1) + 1] = s[3];
        }
        __syncthreads();
        const bool valid = k0 + it * kLaKeys + lane < k1;
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int row = 2 * warp + r;
            float s = (S[row * (kLaKeys + 1) + lane] + S[(kLaHeads + row) * (kLaKeys + 1) + lane]) * scale;
            if (!valid) s = -INFINITY;
            const float mn = fmaxf(m_run[r], warp_max(s));  // a tile has at least one key
            const float corr = fast_exp2(m_run[r] - mn), w = fast_exp2(s - mn);
            m_run[r] = mn;
            l_run[r] = l_run[r] * corr + warp_sum(w);
            P[row * (kLaKeys + 8) + lane] = __float2bfloat16_rn(w);
            if (lane == 0) corr_s[row] = corr;
        }
        __syncthreads();
        const float c0 = corr_s[g], c1 = corr_s[g + 8];
        uint32_t pa[2][4];
        ldsm_x4(pa[0], pa_off);
        ldsm_x4(pa[1], pa_off + 32);
#pragma unroll
        for (int i = 0; i < NP; i++) {
            const int cg = warp + kLaWarps * i;  // column group
            if (cg * 16 >= rank_p) break;
#pragma unroll
            for (int n = 0; n < 2; n++) {
                O[i][n][0] *= c0;
                O[i][n][1] *= c0;
                O[i][n][2] *= c1;
                O[i][n][3] *= c1;
            }
#pragma unroll
            for (int ks = 0; ks < 2; ks++) {
                uint32_t vb[4];
                ldsm_x4_t(vb, sb + v_off + ks * 16 * row_bytes + cg * 32);
                mma_bf16(O[i][0], pa[ks][0], pa[ks][1], pa[ks][2], pa[ks][3], vb[0], vb[1]);
                mma_bf16(O[i][1], pa[ks][0], pa[ks][1], pa[ks][2], pa[ks][3], vb[2], vb[3]);
            }
        }
    }
    cp_async_wait<0>();
    pdl_launch_dependents();
    if (lane < 2) {
        const int row = 2 * warp + lane;
        l_s[row] = lane ? l_run[1] : l_run[0];
        if (used > 1 && row < nh) {
            float* ml = p.part_ml + (((size_t)t * a.H + h0 + row) * p.n_split + split) * 2;
            ml[0] = lane ? m_run[1] : m_run[0];
            ml[1] = l_s[row];
        }
    }
    __syncthreads();
#pragma unroll
    for (int hh = 0; hh < 2; hh++) {
        const int row = g + 8 * hh;
        if (row >= nh) continue;
        const float f = used > 1 ? 1.f : out_factor<bf16>(a, t, h0 + row) / l_s[row];
#pragma unroll
        for (int i = 0; i < NP; i++) {
            const int cg = warp + kLaWarps * i;
            if (cg * 16 >= rank_p) break;
#pragma unroll
            for (int n = 0; n < 2; n++) {
                const int c = cg * 16 + n * 8 + 2 * tq;
                const float x = O[i][n][2 * hh] * f, y = O[i][n][2 * hh + 1] * f;
                if (used > 1)
                    *reinterpret_cast<float2*>(p.part_o + (((size_t)t * a.H + h0 + row) * p.n_split + split) * rank_p + c) = make_float2(x, y);
                else
                    *reinterpret_cast<uint32_t*>(static_cast<bf16*>(a.out) + ((size_t)t * a.H + h0 + row) * rank_p + c) = pack2<bf16>(x, y);
            }
        }
    }
}

// Sum of the ranges of a head, weighted by their maxima.
__global__ void __launch_bounds__(128) latent_attn_merge_kernel(const LaParams p)
{
    typedef __nv_bfloat16 bf16;
    pdl_launch_dependents();
    pdl_wait();
    const LatentAttn& a = p.a;
    const int h = blockIdx.x, t = blockIdx.y;
    int b, pos;
    locate(p.tp, t, b, pos);
    const int n_keys = pos + 1 - max(0, pos - a.window + 1), used = max(1, (n_keys + p.chunk - 1) / p.chunk);
    if (used == 1) return;  // the attention kernel wrote the output itself
    const size_t base = ((size_t)t * a.H + h) * p.n_split;
    float M = -INFINITY, L = 0.f;
    for (int i = 0; i < used; i++) M = fmaxf(M, p.part_ml[(base + i) * 2]);
    for (int i = 0; i < used; i++) L = fmaf(p.part_ml[(base + i) * 2 + 1], fast_exp2(p.part_ml[(base + i) * 2] - M), L);
    const float f = out_factor<bf16>(a, t, h) / L;
    bf16* out = static_cast<bf16*>(a.out) + ((size_t)t * a.H + h) * p.rank_p;
    for (int c = threadIdx.x; c < p.rank_p; c += blockDim.x) {
        float O = 0.f;
        for (int i = 0; i < used; i++) O = fmaf(p.part_o[(base + i) * p.rank_p + c], fast_exp2(p.part_ml[(base + i) * 2] - M), O);
        out[c] = __float2bfloat16_rn(O * f);
    }
}

constexpr int kLaMaxSplits = 16;
// latent_attn_tc.cu: decode steps
bool latent_attn_tc_takes(const LatentAttn& a, const TokenPositions& tp);
size_t latent_attn_tc_workspace(int tokens, int H, int rank);
int latent_attn_tc(const LatentAttn& a, const TokenPositions& tp, int tokens, int span_bound, void* workspace, cudaStream_t st);

size_t latent_attn_workspace(int tokens, int H, int rank)
{
    return std::max((size_t)std::min(tokens, 64) * H * kLaMaxSplits * (latent_pad(rank) + 2) * sizeof(float), latent_attn_tc_workspace(tokens, H, rank));
}

template <int NP>
static int launch_la(const LaParams& p, dim3 grid, size_t smem, cudaStream_t st)
{
    auto kern = latent_attn_kernel<NP>;
    static DeviceOnce attr;
    ONELLM_CUDA(attr.run([kern] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024); }));
    ONELLM_CUDA(launch_pdl(kern, grid, dim3(kLaWarps * 32), smem, st, p));
    return ONELLM_OK;
}

int latent_attn(const LatentAttn& a, const TokenPositions& tp, int tokens, int span_bound, bool plain, void* workspace, cudaStream_t st)
{
    RC(check_latent(a));
    ONELLM_REQUIRE(a.q && a.out && span_bound >= 1 && (tp.cu ? tp.hist && a.fresh : tp.step && tp.off), ONELLM_ERR_ARG, "latent_attn: bad argument");
    if (tokens <= 0) return ONELLM_OK;
    const int rank_p = latent_pad(a.rank);
    if (plain || a.dtype == ONELLM_F32) {
        const dim3 grid(tokens, (a.H + 3) / 4);
        if (a.dtype == ONELLM_F32) ONELLM_CUDA(launch_pdl(latent_attn_plain_kernel<float>, grid, dim3(128), 0, st, a, tp, rank_p));
        else ONELLM_CUDA(launch_pdl(latent_attn_plain_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, a, tp, rank_p));
        return ONELLM_OK;
    }
    ONELLM_REQUIRE(workspace, ONELLM_ERR_ARG, "latent_attn: no workspace");
    if (latent_attn_tc_takes(a, tp)) return latent_attn_tc(a, tp, tokens, span_bound, workspace, st);
    ONELLM_REQUIRE(tokens <= 64, ONELLM_ERR_UNSUPPORTED, "latent_attn: %d tokens, at most 64 in latent space", tokens);
    const size_t tile = la_tile_bytes(rank_p), fixed = la_fixed_bytes(rank_p);
    const int nst = (int)std::max<size_t>(2, std::min<size_t>(6, (108 * 1024 - std::min<size_t>(fixed, 64 * 1024)) / tile));
    // ranges: enough blocks for the SMs, of at least four tiles each
    const int groups = (a.H + kLaHeads - 1) / kLaHeads, span = std::min(span_bound, a.window);
    int n = (int)std::min<long>(kLaMaxSplits, (2L * num_sms()) / std::max(1L, (long)tokens * groups));
    n = std::max(1, std::min(n, span / (4 * kLaKeys)));
    const int chunk = ((span + n - 1) / n + kLaKeys - 1) / kLaKeys * kLaKeys;
    n = (span + chunk - 1) / chunk;
    LaParams p = {a, tp, rank_p, nst, n, chunk, (float*)workspace, nullptr};
    p.part_ml = p.part_o + (size_t)tokens * a.H * n * rank_p;
    const dim3 grid(n, groups, tokens);
    const size_t smem = nst * tile + fixed;
    if (rank_p <= 128) RC(launch_la<1>(p, grid, smem, st));
    else if (rank_p <= 256) RC(launch_la<2>(p, grid, smem, st));
    else if (rank_p <= 512) RC(launch_la<4>(p, grid, smem, st));
    else RC(launch_la<8>(p, grid, smem, st));
    if (n > 1) ONELLM_CUDA(launch_pdl(latent_attn_merge_kernel, dim3(a.H, tokens), dim3(128), 0, st, p));
    return ONELLM_OK;
}

}  // namespace onellm

using namespace onellm;

extern "C" int onellm_latent_store(const onellm_latent_attn* a, const onellm_token_positions* tp, int tokens, int max_hist, void* stream)
{
    ONELLM_REQUIRE(a && tp, ONELLM_ERR_ARG, "latent_store: null pointer");
    return latent_store(*a, *tp, tokens, max_hist, reinterpret_cast<cudaStream_t>(stream));
}

extern "C" int onellm_latent_keep(const onellm_latent_attn* a, const onellm_token_positions* tp, int max_new, void* stream)
{
    ONELLM_REQUIRE(a && tp, ONELLM_ERR_ARG, "latent_keep: null pointer");
    return latent_keep(*a, *tp, max_new, reinterpret_cast<cudaStream_t>(stream));
}

extern "C" size_t onellm_latent_attn_workspace(int tokens, int H, int rank)
{
    return tokens > 0 && H > 0 && rank > 0 ? latent_attn_workspace(tokens, H, rank) : 0;
}

extern "C" int onellm_latent_attn_run(const onellm_latent_attn* a, const onellm_token_positions* tp, int tokens, int span_bound, int plain,
                                      void* workspace, void* stream)
{
    ONELLM_REQUIRE(a && tp, ONELLM_ERR_ARG, "latent_attn: null pointer");
    return latent_attn(*a, *tp, tokens, span_bound, plain != 0, workspace, reinterpret_cast<cudaStream_t>(stream));
}
