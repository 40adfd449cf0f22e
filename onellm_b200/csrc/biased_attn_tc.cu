// Context pass of BiasedAttn and WindowAttn (mixers.h) on the 5th-generation tensor cores: bfloat16, key and value sizes of
// their own; the scores of the one take a factor per query position and a penalty per head and distance, those of the other
// a constant scale and a sliding window.
//
// The schedule is the one of context_attn_tc_kernel (context_attn_tc.cu): a block owns 128 query rows of one
// (sequence, head) and walks the cache in 64-row tiles; S = Q.K^T and O += P.V by tcgen05.mma with S, P and O in tensor
// memory, four softmax warps with one query row per thread, a fifth warp that issues TMA loads and MMAs.  What differs:
//   - sizes are run-time numbers of 64-column chunks (key chunks in Q and K, value chunks in V and O; a size that is not
//     a multiple of 64 is zero-filled by TMA and by the threads that write Q);
//   - the scores of a row are turned into log2 units by the factor of its position and lose the penalty of their
//     distance before the maximum is taken.  A tile of scores spans 191 distances: the threads read the table of the
//     head directly, consecutive rows at consecutive addresses;
//   - WINDOWED: keys and values of all heads lie beside each other in one buffer that a sequence's rows are packed into, so
//     a head is a range of columns; the tiles of a block start at the first key its first query sees, masks apply on both
//     sides, a row may see nothing in its block's first tiles, and the output takes the gate of its token and head.
// Every mbarrier wait is bounded; on expiry the block raises the time-out flag, stops, frees its tensor memory and
// returns.
#include <math.h>

#include "mixers.h"
#include "tc_common.cuh"

namespace onellm {

constexpr int kBaQ = 128, kBaKV = 64;
constexpr int kBaSoftmaxThreads = 128;
constexpr int kBaThreads = kBaSoftmaxThreads + 32;
constexpr int kBaQChunk = kBaQ * 128;    // 16 KB: 128 rows x 64 columns
constexpr int kBaKVChunk = kBaKV * 128;  // 8 KB: 64 rows x 64 columns
constexpr uint32_t kBaO = 128;           // tensor-memory column of O; S0 at 0, S1 at 64

struct BaParams {
    BiasedAttn a;
    const int *cu, *hist;
    int kch, vch;         // 64-column chunks of a key / value
    uint32_t tmem_cols;   // 256 or 512
    int window;           // WINDOWED from here on
    float scale_log2;
    const void* gate;
    long gate_ld;
};

__device__ __forceinline__ void ba_umma_ta(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc, uint32_t accumulate)
{
    asm volatile(
        "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n}" ::"r"(tmem_d),
        "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}

template <bool WINDOWED>
__global__ void __launch_bounds__(kBaThreads, 2)
biased_attn_tc_kernel(const BaParams p, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v)
{
    typedef __nv_bfloat16 bf16;
    extern __shared__ __align__(1024) unsigned char smem_raw[];  // the 128-byte swizzle works on shared-window address bits
    const int kch = p.kch, vch = p.vch;
    const int k_tile = kch * kBaKVChunk, v_tile = vch * kBaKVChunk;
    unsigned char* sQ = smem_raw;
    unsigned char* sK = sQ + kch * kBaQChunk;  // two buffers
    unsigned char* sV = sK + 2 * k_tile;       // two buffers
    uint64_t* bars = reinterpret_cast<uint64_t*>(sV + 2 * v_tile);
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 11);
    // per-tile barriers come in pairs: tile j uses slot j & 1, phase (j >> 1) & 1, so that a producer two tiles ahead
    // of a waiter cannot be taken for the tile waited for
    const uint32_t q_full = smem_u32(bars), k_full0 = smem_u32(bars + 1), s_full0 = smem_u32(bars + 3), v_full0 = smem_u32(bars + 5),
                   p_full0 = smem_u32(bars + 7), o_full0 = smem_u32(bars + 9);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int b = blockIdx.z, h = blockIdx.y, hk = h / (p.a.H / p.a.G);

    if (smem_u32(smem_raw) & 1023u) {  // the tiles would be read with the wrong swizzle
        if (threadIdx.x == 0) atomicExch(&g_tc_timeout_flag, 1);
        return;
    }
    if (threadIdx.x == 0) {
        mbar_init(q_full, kBaSoftmaxThreads);
        for (int s = 0; s < 2; s++) {
            mbar_init(k_full0 + 8 * s, 1);
            mbar_init(s_full0 + 8 * s, 1);
            mbar_init(v_full0 + 8 * s, 1);
            mbar_init(p_full0 + 8 * s, kBaSoftmaxThreads);
            mbar_init(o_full0 + 8 * s, 1);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(p.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem_base = *tmem_slot;

    pdl_launch_dependents();
    pdl_wait();
    const int tok0 = p.cu[b], q_len = p.cu[b + 1] - tok0, hist = p.hist[b];
    const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kBaQ;  // the blocks with the most cache tiles first
    const bool active = q0 < q_len && (WINDOWED || hist + q_len <= p.a.S);
    const int q_rows = active ? min(kBaQ, q_len - q0) : 0;
    const int kv_end = hist + q0 + q_rows;
    const int key0 = WINDOWED ? max(0, hist + q0 - p.window + 1) : 0;  // first key of the first tile
    const int n_tiles = active ? (kv_end - key0 + kBaKV - 1) / kBaKV : 0;
    // row of key0 and columns of the head
    int cache_row0 = (b * p.a.G + hk) * p.a.S, k_col = 0, v_col = 0;
    if (WINDOWED) {
        int base = tok0;
        for (int i = 0; i < b; i++) base += min(p.hist[i], p.window - 1);
        cache_row0 = base + key0 - (hist - min(hist, p.window - 1));
        k_col = h * p.a.dk;
        v_col = p.a.H * p.a.dk + h * p.a.dv;
    }

    if (warp == 4 && active) {
        // ---- control: the whole warp runs this code, one elected lane issues (warp-uniform control flow keeps the
        // operands of the MMAs in uniform registers)
        uint32_t leader;
        asm volatile("{\n .reg .pred p;\n elect.sync _|p, 0xffffffff;\n selp.u32 %0, 1, 0, p;\n}" : "=r"(leader));
        bool ok = true;
        auto load = [&](const CUtensorMap* map, unsigned char* base, int tile_bytes, int chunks, uint32_t full0, int j, int col) {
            const int s = j & 1;
            if (leader) {
                mbar_expect_tx(full0 + 8 * s, tile_bytes);
                for (int c = 0; c < chunks; c++)
                    tma_load_2d(smem_u32(base + s * tile_bytes + c * kBaKVChunk), map, col + 64 * c, cache_row0 + j * kBaKV, full0 + 8 * s);
            }
        };
        auto load_k = [&](int j) { load(&map_k, sK, k_tile, kch, k_full0, j, k_col); };
        auto load_v = [&](int j) { load(&map_v, sV, v_tile, vch, v_full0, j, v_col); };
        auto wait_all = [&](uint32_t bar, uint32_t parity) { return __all_sync(0xffffffffu, mbar_wait(bar, parity)); };
        const uint32_t types = (1u << 4) | umma_operand_bits<bf16>() | ((uint32_t)(kBaQ >> 4) << 24);
        const uint32_t idesc_s = types | ((uint32_t)(kBaKV >> 3) << 17);
        const uint32_t idesc_o = types | (1u << 16) | ((uint32_t)(vch * 8) << 17);
        const uint64_t dq = umma_desc(smem_u32(sQ), 16, 1024), dk = umma_desc(smem_u32(sK), 16, 1024),
                       dv = umma_desc(smem_u32(sV), kBaKVChunk, 1024);
        auto issue_s = [&](int j) {  // S_j = Q . K_j^T into accumulator j & 1
            const int s = j & 1;
            if (!wait_all(k_full0 + 8 * s, (uint32_t)(j >> 1) & 1u)) return false;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint64_t dks = dk + (uint64_t)((s * k_tile) >> 4);
            const uint32_t acc = tmem_base + (uint32_t)(s * kBaKV);
            if (leader) {
                for (int c = 0; c < kch; c++)
#pragma unroll
                    for (int kk = 0; kk < 4; kk++)
                        umma_f16(acc, dq + (uint64_t)((c * kBaQChunk + kk * 32) >> 4), dks + (uint64_t)((c * kBaKVChunk + kk * 32) >> 4), idesc_s,
                                 (c | kk) ? 1u : 0u);
                umma_commit(s_full0 + 8 * s);
            }
            __syncwarp();
            return true;
        };
        load_k(0);
        load_v(0);
        if (n_tiles > 1) {
            load_k(1);
            load_v(1);
        }
        ok = wait_all(q_full, 0) && issue_s(0);
        for (int j = 0; j < n_tiles && ok; j++) {
            const int s = j & 1;
            if (j + 1 < n_tiles) ok = issue_s(j + 1);
            ok = ok && wait_all(s_full0 + 8 * s, (uint32_t)(j >> 1) & 1u);  // K buffer s is free
            if (ok && j + 2 < n_tiles) load_k(j + 2);
            ok = ok && wait_all(p_full0 + 8 * s, (uint32_t)(j >> 1) & 1u) && wait_all(v_full0 + 8 * s, (uint32_t)(j >> 1) & 1u);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint64_t dvs = dv + (uint64_t)((s * v_tile) >> 4);
            if (leader) {
#pragma unroll
                for (int kk = 0; kk < kBaKV / 16; kk++)
                    ba_umma_ta(tmem_base + kBaO, tmem_base + (uint32_t)(s * kBaKV + kk * 8), dvs + (uint64_t)((kk * 2048) >> 4), idesc_o,
                               (j > 0 || kk > 0) ? 1u : 0u);
                umma_commit(o_full0 + 8 * s);
            }
            __syncwarp();
            if (j + 2 < n_tiles) {
                ok = wait_all(o_full0 + 8 * s, (uint32_t)(j >> 1) & 1u);  // V buffer s is free again
                if (ok) load_v(j + 2);
            }
        }
    } else if (warp < 4 && active) {
        // ---- softmax and output, one query row per thread
        const int r = threadIdx.x;
        const int pos = hist + q0 + r;
        const bool row_ok = r < q_rows;
        const uint32_t t_lane = tmem_base + ((uint32_t)(warp * 32) << 16);
        const uint32_t t_o = t_lane + kBaO;
        const uint32_t row_off = (r >> 3) * 1024 + (r & 7) * 128;
        const float factor = WINDOWED ? p.scale_log2 : row_ok ? p.a.q_factor[pos] : 0.f;
        const float* pen = WINDOWED ? nullptr : p.a.penalty + (size_t)h * p.a.S;
        const int pos_c = row_ok ? pos : hist + q0;  // rows behind the end of the sequence read the penalties of its first row
        float m_ref = -INFINITY, l_run = 0.f;
        bool ok = true;
        {
            const bf16* qrow = reinterpret_cast<const bf16*>(p.a.q) + (size_t)(tok0 + q0 + (row_ok ? r : 0)) * p.a.ld + (size_t)h * p.a.dk;
            for (int u = 0; u < kch * 8; u++) {
                const uint4 v = (row_ok && u * 8 < p.a.dk) ? *reinterpret_cast<const uint4*>(qrow + u * 8) : make_uint4(0u, 0u, 0u, 0u);
                *reinterpret_cast<uint4*>(sQ + (u >> 3) * kBaQChunk + row_off + (((u & 7) ^ (r & 7)) << 4)) = v;
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            mbar_arrive(q_full);
        }
        for (int j = 0; j < n_tiles && ok; j++) {
            ok = mbar_wait(s_full0 + 8 * (j & 1), (uint32_t)(j >> 1) & 1u);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int kv0 = key0 + j * kBaKV;
            const bool need_mask = kv0 + kBaKV - 1 > hist + q0 || (WINDOWED && kv0 <= hist + q0 + q_rows - 1 - p.window);
            uint32_t sv[64];
            tmem_ld32(t_lane + (uint32_t)((j & 1) * kBaKV), *reinterpret_cast<uint32_t(*)[32]>(&sv[0]));
            tmem_ld32(t_lane + (uint32_t)((j & 1) * kBaKV + 32), *reinterpret_cast<uint32_t(*)[32]>(&sv[32]));
            asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
            float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            const float* pd = pen + (pos_c - kv0);  // penalty of the tile's first key; key i: pd[-i]
            if constexpr (WINDOWED) {
                if (need_mask) {
                    const int last = pos_c - kv0, before = last - p.window;  // visible: before < i <= last
#pragma unroll
                    for (int i = 0; i < 64; i++)
                        if (i > last || i <= before) sv[i] = __float_as_uint(-INFINITY);
                }
#pragma unroll
                for (int i = 0; i < 64; i++) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sv[i]));
            } else if (need_mask) {
#pragma unroll
                for (int i = 0; i < 64; i++) {
                    float s = -INFINITY;
                    if (kv0 + i <= pos_c) s = fmaf(__uint_as_float(sv[i]), factor, -__ldg(pd - i));
                    sv[i] = __float_as_uint(s);
                    mx4[i & 3] = fmaxf(mx4[i & 3], s);
                }
            } else {
#pragma unroll
                for (int i = 0; i < 64; i++) {
                    const float s = fmaf(__uint_as_float(sv[i]), factor, -__ldg(pd - i));
                    sv[i] = __float_as_uint(s);
                    mx4[i & 3] = fmaxf(mx4[i & 3], s);
                }
            }
            float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
            if (WINDOWED) mx *= factor;  // a positive scale commutes with the maximum
            const bool grow = mx > m_ref + 8.f;  // always on the first tile with a key the row sees
            float alpha = 1.f;
            if (grow) {
                alpha = fast_exp2(m_ref - mx);
                m_ref = mx;
                l_run *= alpha;
            }
            float sum4[4] = {0.f, 0.f, 0.f, 0.f};
            const float ref = WINDOWED && m_ref == -INFINITY ? 0.f : m_ref;  // nothing seen so far: all weights zero
#pragma unroll
            for (int i = 0; i < 64; i++) {
                const float pv = fast_exp2(WINDOWED ? fmaf(__uint_as_float(sv[i]), factor, -ref) : __uint_as_float(sv[i]) - ref);
                sum4[i & 3] += pv;
                sv[i] = __float_as_uint(pv);
            }
            l_run += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
            if (j > 0 && __any_sync(0xffffffffu, grow)) {
                ok = mbar_wait(o_full0 + 8 * ((j - 1) & 1), (uint32_t)((j - 1) >> 1) & 1u);  // P.V of the tile before: O is at rest
                ok = __all_sync(0xffffffffu, ok);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                uint32_t ov[32];
#pragma unroll 1
                for (int c = 0; c < vch * 64; c += 32) {
                    tmem_ld32(t_o + (uint32_t)c, ov);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int i = 0; i < 32; i++) ov[i] = __float_as_uint(__uint_as_float(ov[i]) * alpha);
                    tmem_st32(t_o + (uint32_t)c, ov);
                }
                asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            }
            {
                uint32_t pk[32];
#pragma unroll
                for (int i = 0; i < 32; i++) pk[i] = pack2<bf16>(__uint_as_float(sv[2 * i]), __uint_as_float(sv[2 * i + 1]));
                tmem_st32(t_lane + (uint32_t)((j & 1) * kBaKV), pk);
            }
            if (kv0 + kBaKV > kv_end) {
                // rows of the tile beyond the ones that exist hold anything (0 x NaN would poison the product): clear them
                ok = mbar_wait(v_full0 + 8 * (j & 1), (uint32_t)(j >> 1) & 1u);
                ok = __all_sync(0xffffffffu, ok);
                if (!ok) break;
                if (r < kBaKV && kv0 + r >= kv_end)
                    for (int u = 0; u < vch * 8; u++)
                        *reinterpret_cast<uint4*>(sV + (j & 1) * v_tile + (u >> 3) * kBaKVChunk + row_off + (u & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(p_full0 + 8 * (j & 1));
        }
        ok = ok && mbar_wait(o_full0 + 8 * ((n_tiles - 1) & 1), (uint32_t)((n_tiles - 1) >> 1) & 1u);
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            float inv = l_run > 0.f ? p.a.out_scale / l_run : 0.f;
            if (WINDOWED && p.gate && row_ok)
                inv *= 1.f / (1.f + expf(-__bfloat162float(static_cast<const bf16*>(p.gate)[(size_t)(tok0 + q0 + r) * p.gate_ld + h])));
            bf16* dst = reinterpret_cast<bf16*>(p.a.out) + (size_t)(tok0 + q0 + r) * p.a.out_ld + (size_t)h * p.a.dv;
#pragma unroll 1
            for (int c0 = 0; c0 < vch * 64; c0 += 32) {
                uint32_t ov[32];
                tmem_ld32(t_o + (uint32_t)c0, ov);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                if (row_ok) {
#pragma unroll
                    for (int c = 0; c < 32; c += 8)
                        if (c0 + c < p.a.dv)
                            *reinterpret_cast<uint4*>(dst + c0 + c) = make_uint4(
                                pack2<bf16>(__uint_as_float(ov[c]) * inv, __uint_as_float(ov[c + 1]) * inv),
                                pack2<bf16>(__uint_as_float(ov[c + 2]) * inv, __uint_as_float(ov[c + 3]) * inv),
                                pack2<bf16>(__uint_as_float(ov[c + 4]) * inv, __uint_as_float(ov[c + 5]) * inv),
                                pack2<bf16>(__uint_as_float(ov[c + 6]) * inv, __uint_as_float(ov[c + 7]) * inv));
                }
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 0)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(p.tmem_cols) : "memory");
}

static const TimeoutFlag timeout_flag(tc_flag_read_clear);

template <bool WINDOWED>
static int ba_launch(const BaParams& p, int B, int max_new, const CUtensorMap& map_k, const CUtensorMap& map_v, cudaStream_t st)
{
    const int smem = p.kch * kBaQChunk + 2 * (p.kch + p.vch) * kBaKVChunk + 256;
    static DeviceOnce attr;
    ONELLM_CUDA(attr.run([] { return cudaFuncSetAttribute(biased_attn_tc_kernel<WINDOWED>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); }));
    ONELLM_CUDA(launch_pdl(biased_attn_tc_kernel<WINDOWED>, dim3((max_new + kBaQ - 1) / kBaQ, p.a.H, B), dim3(kBaThreads), smem, st, p, map_k, map_v));
    return ONELLM_OK;
}

int biased_attn_tc_launch(const BiasedAttn& a, const TokenPositions& tp, int max_new, cudaStream_t st)
{
    BaParams p = {a, tp.cu, tp.hist, (a.dk + 63) / 64, (a.dv + 63) / 64, 256u, 0, 0.f, nullptr, 0};
    if (p.vch > 2) p.tmem_cols = 512u;
    const uint64_t rows = (uint64_t)tp.B * a.G * a.S;
    ONELLM_REQUIRE(rows < (1ull << 31), ONELLM_ERR_UNSUPPORTED, "biased_attn: cache of %llu rows", (unsigned long long)rows);
    CUtensorMap map_k, map_v;
    int rc = make_map(&map_k, a.k_cache, (uint64_t)a.dk, rows, kBaKV);
    if (!rc) rc = make_map(&map_v, a.v_cache, (uint64_t)a.dv, rows, kBaKV);
    if (rc) return rc;
    return ba_launch<false>(p, tp.B, max_new, map_k, map_v, st);
}

int window_attn(const WindowAttn& a, const TokenPositions& tp, int max_new, cudaStream_t st)
{
    ONELLM_REQUIRE(a.q && a.kv && a.out && tp.cu && tp.hist && tp.B > 0, ONELLM_ERR_ARG, "window_attn: null pointer");
    ONELLM_REQUIRE(a.H > 0 && a.dk > 0 && a.dv > 0 && a.dk % 16 == 0 && a.dv % 16 == 0 && a.dk <= 256 && a.dv <= 256, ONELLM_ERR_UNSUPPORTED,
                   "window_attn: key size %d and value size %d must be multiples of 16, at most 256", a.dk, a.dv);
    ONELLM_REQUIRE(a.window > 0 && a.scale > 0.f && a.q_ld % 8 == 0 && a.out_ld % 8 == 0 && a.kv_ld % 8 == 0 && a.kv_ld >= (long)a.H * (a.dk + a.dv) &&
                       a.kv_rows > 0 && a.kv_rows < (1l << 31),
                   ONELLM_ERR_ARG, "window_attn: bad argument");
    if (max_new <= 0) return ONELLM_OK;
    BiasedAttn base = {};
    base.H = base.G = a.H;
    base.dk = a.dk;
    base.dv = a.dv;
    base.q = a.q;
    base.ld = a.q_ld;
    base.out = a.out;
    base.out_ld = a.out_ld;
    base.out_scale = a.out_scale;
    BaParams p = {base, tp.cu, tp.hist, (a.dk + 63) / 64, (a.dv + 63) / 64, 256u, a.window, a.scale * 1.4426950408889634f, a.gate, a.gate_ld};
    if (p.vch > 2) p.tmem_cols = 512u;
    CUtensorMap map;
    RC(make_map(&map, a.kv, (uint64_t)a.kv_ld, (uint64_t)a.kv_rows, kBaKV));
    return ba_launch<true>(p, tp.B, max_new, map, map, st);
}

}  // namespace onellm

extern "C" int onellm_window_attn_run(const onellm_window_attn* a, const onellm_token_positions* tp, int max_new, void* stream)
{
    ONELLM_REQUIRE(a && tp, ONELLM_ERR_ARG, "window_attn: null pointer");
    return onellm::window_attn(*a, *tp, max_new, reinterpret_cast<cudaStream_t>(stream));
}
