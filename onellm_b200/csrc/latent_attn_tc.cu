// Decode step of LatentAttn (mixers.h) on the 5th-generation tensor cores: bfloat16, latents of up to 512 elements.
//
// A latent is key and value of every head at once, so the latents are the large operand of both products and the heads the
// small one.  A block owns 32 heads of one sequence and a range of 64-row tiles of its ring,
//     S^T[64 latents, 32 heads] = C . Q'^T            A = the tile as it lies in memory (K-major), B = the queries
//     O^T[rank, 32 heads]      += C^T . P^T           A = the same tile read the other way (MN-major), B = the weights
// both tcgen05.mma N32 K16 with accumulators in tensor memory; no row of an operand is padding but for heads beyond the
// last.  One thread issues TMA loads: eight whole latents at a time, contiguous in memory, which a three-dimensional tensor
// map lays out as eight rows of every 64-element chunk, so that the tile is an operand of either product; a tile's buffer
// is refilled in groups of 16 latents as the second product is done with them.  One warp issues the MMAs, the first
// product of the next tile ahead of the second of this one where it has arrived; eight warps take the softmax: a thread has one
// latent and the scores of half of the heads,
// the maximum over a warp's latents is one redux per head, the sums stay in registers until the end, and the accumulator is
// only rescaled when a maximum has grown by more than 2^8.
//
// Attention does not depend on the order of the keys, so tiles are ranges of ring rows, whatever positions they hold; rows
// that hold none the query sees (not written yet, or out of the window) get the weight zero and are cleared before the
// second product.  A sequence alone in its range writes its output; the results of several ranges go through L2 to a merge
// kernel (adding them through the shared memory of a thread-block cluster took longer).  Tiles
// without the row that this step has stored are requested before the dependency wait.  (Chunk by chunk, as 128-byte pieces
// of 64 rows, the loads did not get beyond 4 TB/s.)
// Every mbarrier wait is bounded; on expiry the block raises the time-out flag, writes zeros, frees its tensor memory and
// returns.
#include <math.h>

#include <algorithm>

#include "mixers.h"
#include "tc_common.cuh"

namespace onellm {

constexpr int kLtRows = 64, kLtHeads = 32, kLtSoftmaxWarps = 8, kLtThreads = 64 + 32 * kLtSoftmaxWarps;
constexpr int kLtCols = kLtHeads / 2;          // heads of a softmax warp: two warps share the lanes of a quarter of tensor memory
constexpr int kLtUnitRows = 8;                 // latents of a load
constexpr int kLtChunk = kLtUnitRows * 128;    // 1 KB: eight latents x 64 elements
constexpr int kLtGroups = kLtRows / 16;        // refill units of a tile
constexpr int kLtQChunk = kLtHeads * 128;      // 4 KB: 32 heads x 64 elements
constexpr int kLtPChunk = kLtHeads * 128;      // 4 KB: 32 heads x 64 latents
constexpr int kLtMaxPairs = 4, kLtMaxBufs = 4, kLtMaxSplits = 16;
constexpr uint32_t kLtTmem = 256, kLtO = 64;   // S of even and odd tiles at columns 0 and 32, O behind them, 32 columns per pair

struct LtParams {
    LatentAttn a;
    TokenPositions tp;
    int rank_p, n_pair, n_buf;  // elements, pairs of 64-element chunks, tile buffers
    int n_split, tiles_per_split;
    float* part_o;   // [T, groups of heads, n_split, 32, 128 n_pair]
    float2* part_ml; // [T, groups of heads, n_split, 32]: reference (log2), sum
};

__device__ __forceinline__ int lt_ranges(const LtParams& p, int pos)
{
    const int tiles = (min(pos + 1, p.a.R) + kLtRows - 1) / kLtRows;
    return (tiles + p.tiles_per_split - 1) / p.tiles_per_split;
}
__device__ __forceinline__ float lt_out_factor(const LatentAttn& a, int t, int h)
{
    const float g = a.gate ? __bfloat162float(static_cast<const __nv_bfloat16*>(a.gate)[(size_t)t * a.gate_ld + h]) : 0.f;
    return a.out_scale * (a.gate ? 1.f / (1.f + expf(-g)) : 1.f);
}

__device__ __forceinline__ float redux_max(float v)
{
    float r;
    asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(r) : "f"(v));
    return r;
}

// barrier of the softmax warps that share heads
__device__ __forceinline__ bool all_of_four_warps(int half, bool v)
{
    uint32_t r;
    asm volatile(
        "{\n .reg .pred p, q;\n setp.ne.u32 q, %1, 0;\n barrier.cta.red.and.pred p, %2, 128, q;\n selp.u32 %0, 1, 0, p;\n}"
        : "=r"(r)
        : "r"((uint32_t)v), "r"(1 + half)
        : "memory");
    return r != 0;
}

__global__ void __launch_bounds__(kLtThreads, 1)
latent_attn_tc_kernel(const LtParams p, const __grid_constant__ CUtensorMap map_c, const __grid_constant__ CUtensorMap map_q)
{
    typedef __nv_bfloat16 bf16;
    const LatentAttn& a = p.a;
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int unit_bytes = 2 * p.n_pair * kLtChunk, tile_bytes = kLtRows / kLtUnitRows * unit_bytes;
    unsigned char* sQ = smem + (size_t)p.n_buf * tile_bytes;
    unsigned char* sP = sQ + 2 * p.n_pair * kLtQChunk;  // two buffers
    __shared__ __align__(8) uint64_t bars[(1 + kLtGroups) * kLtMaxBufs + 7];
    __shared__ uint32_t tmem_slot;
    __shared__ __align__(16) float s_max[4][kLtHeads], s_ref[4][kLtHeads], s_alpha[4][kLtHeads], s_sum[4][kLtHeads];
    const uint32_t full0 = smem_u32(bars), empty0 = smem_u32(bars + kLtMaxBufs), q_full = smem_u32(bars + (1 + kLtGroups) * kLtMaxBufs),
                   s_full0 = q_full + 8, p_full0 = q_full + 24, o_full0 = q_full + 40;  // in pairs: tile j uses slot j & 1, phase (j >> 1) & 1
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int split = blockIdx.x, h0 = blockIdx.y * kLtHeads, t = blockIdx.z, nh = min(kLtHeads, a.H - h0);

    int b, pos;
    locate(p.tp, t, b, pos);
    const int n_rows = min(pos + 1, a.R);  // ring rows in use
    const int tile0 = split * p.tiles_per_split, n_tiles = max(0, min(p.tiles_per_split, (n_rows + kLtRows - 1) / kLtRows - tile0));
    if (n_tiles == 0) {
        pdl_launch_dependents();
        pdl_wait();
        return;
    }
    if (threadIdx.x == 0) {
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_c));
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_q));
        for (int i = 0; i < p.n_buf; i++) {
            mbar_init(full0 + 8 * i, 1);
            for (int g = 0; g < kLtGroups; g++) mbar_init(empty0 + 8 * (i * kLtGroups + g), 1);
        }
        mbar_init(q_full, 1);
        for (int i = 0; i < 2; i++) {
            mbar_init(s_full0 + 8 * i, 1);
            mbar_init(p_full0 + 8 * i, 32 * kLtSoftmaxWarps);
            mbar_init(o_full0 + 8 * i, 1);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 2) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(kLtTmem) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_slot;
    const int new_tile = (pos % a.R) / kLtRows;
    pdl_launch_dependents();  // the merge kernel (or what follows) may wait for this one beside it
    if (warp == 0) {
        if (lane == 0) {
            auto load = [&](int j, int g) {  // 16 latents of tile j
                const int buf = j % p.n_buf, r0 = (tile0 + j) * kLtRows + 16 * g;
                const uint32_t dst = smem_u32(smem + (size_t)buf * tile_bytes) + (uint32_t)(2 * g * unit_bytes), bar = full0 + 8 * buf;
                if (g == 0) mbar_expect_tx(bar, (uint32_t)tile_bytes);
                tma_load_3d(dst, &map_c, 0, b * a.R + r0, 0, bar);
                tma_load_3d(dst + unit_bytes, &map_c, 0, b * a.R + r0 + kLtUnitRows, 0, bar);
            };
            int j = 0;
            for (; j < min(n_tiles, p.n_buf) && tile0 + j != new_tile; j++)
                for (int g = 0; g < kLtGroups; g++) load(j, g);
            pdl_wait();
            mbar_expect_tx(q_full, 2 * p.n_pair * kLtQChunk);
            for (int c = 0; c < 2 * p.n_pair; c++) tma_load_2d(smem_u32(sQ + c * kLtQChunk), &map_q, 64 * c, t * a.H + h0, q_full);
            bool ok = true;
            for (; j < n_tiles && ok; j++)
                for (int g = 0; g < kLtGroups && ok; g++) {
                    if (j >= p.n_buf) ok = mbar_wait(empty0 + 8 * (j % p.n_buf * kLtGroups + g), ((j / p.n_buf) - 1) & 1);
                    if (ok) load(j, g);
                }
        } else {
            pdl_wait();
        }
    } else if (warp == 1) {
        pdl_wait();
        // the whole warp runs this code, one elected lane issues: warp-uniform control flow keeps the descriptors in uniform
        // registers (issued from a divergent branch, an MMA this small took 110 cycles)
        uint32_t leader;
        asm volatile("{\n .reg .pred p;\n elect.sync _|p, 0xffffffff;\n selp.u32 %0, 1, 0, p;\n}" : "=r"(leader));
        auto wait_all = [&](uint32_t bar, uint32_t parity) { return __all_sync(0xffffffffu, mbar_wait(bar, parity)); };
        // D f32, A and B bfloat16, N = 32, B K-major; first product: M = 64, A K-major; second: M = 128, A MN-major
        const uint32_t types = (1u << 4) | umma_operand_bits<bf16>() | ((uint32_t)(kLtHeads >> 3) << 17);
        const uint32_t idesc_s = types | ((uint32_t)(kLtRows >> 4) << 24), idesc_o = types | (1u << 15) | (8u << 24);
        const uint64_t dk = umma_desc(smem_u32(smem), 16, (uint32_t)unit_bytes), dv = umma_desc(smem_u32(smem), kLtChunk, (uint32_t)unit_bytes),
                       dq = umma_desc(smem_u32(sQ), 16, 1024), dp = umma_desc(smem_u32(sP), 16, 1024);
        auto issue_s = [&](int j) {
            const int buf = j % p.n_buf;
            if (!wait_all(full0 + 8 * buf, (uint32_t)(j / p.n_buf) & 1u)) return false;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint64_t c = dk + (uint64_t)((buf * tile_bytes) >> 4);
            if (leader) {
                for (int i = 0; i < p.n_pair; i++) {
                    const uint64_t ci = c + (uint64_t)((2 * i * kLtChunk) >> 4), qi = dq + (uint64_t)((2 * i * kLtQChunk) >> 4);
#pragma unroll
                    for (int k = 0; k < 8; k++)
                        umma_f16(tmem + 32u * (j & 1), ci + (uint64_t)(((k >> 2) * kLtChunk + (k & 3) * 32) >> 4),
                                 qi + (uint64_t)(((k >> 2) * kLtQChunk + (k & 3) * 32) >> 4), idesc_s, (i | k) ? 1u : 0u);
                }
                umma_commit(s_full0 + 8 * (j & 1));
            }
            __syncwarp();
            return true;
        };
        bool ok = wait_all(q_full, 0) && issue_s(0);
        for (int j = 0; j < n_tiles && ok; j++) {
            const bool more = j + 1 < n_tiles;
            const bool arrived = more && mbar_test(full0 + 8 * ((j + 1) % p.n_buf), (uint32_t)((j + 1) / p.n_buf) & 1u);
            const bool ahead = __all_sync(0xffffffffu, arrived);
            if (ahead) ok = issue_s(j + 1);
            ok = ok && wait_all(p_full0 + 8 * (j & 1), (j >> 1) & 1);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int buf = j % p.n_buf;
            const uint64_t c = dv + (uint64_t)((buf * tile_bytes) >> 4), pd = dp + (uint64_t)(((j & 1) * kLtPChunk) >> 4);
            if (leader) {
#pragma unroll
                for (int k = 0; k < kLtGroups; k++) {  // 16 latents: two units of eight rows
                    const uint64_t ck = c + (uint64_t)((2 * k * unit_bytes) >> 4);
                    for (int i = 0; i < p.n_pair; i++)
                        umma_f16(tmem + kLtO + 32u * i, ck + (uint64_t)((2 * i * kLtChunk) >> 4), pd + (uint64_t)((k * 32) >> 4), idesc_o, (j | k) ? 1u : 0u);
                    umma_commit(empty0 + 8 * (buf * kLtGroups + k));
                }
                umma_commit(o_full0 + 8 * (j & 1));
            }
            __syncwarp();
            if (more && !ahead) ok = issue_s(j + 1);
        }
    } else {
        pdl_wait();
        // an accumulator of 64 rows lies in the first 16 lanes of every warp's 32; one of 128 rows in all of them
        const int q = warp & 3, half = (warp - 2) >> 2, c0 = half * kLtCols, row = 16 * q + lane, own = c0 + (lane & 15);
        const uint32_t t_lane = tmem + ((uint32_t)(32 * q) << 16);
        const float scale = a.scale * 1.4426950408889634f;
        float ref = -INFINITY;  // lanes h and h + 16: reference of head c0 + h
        float l[kLtCols];
#pragma unroll
        for (int h = 0; h < kLtCols; h++) l[h] = 0.f;
        bool ok = true;
        for (int j = 0; j < n_tiles; j++) {
            const int slot = (tile0 + j) * kLtRows + row;
            const int back = (pos - slot) % a.R, dist = back < 0 ? back + a.R : back;  // how far back the row's position lies
            const bool seen = lane < 16 && slot < n_rows && dist < a.window;
            ok = ok && mbar_wait(s_full0 + 8 * (j & 1), (j >> 1) & 1);
            ok = __all_sync(0xffffffffu, ok);
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            uint32_t s[kLtCols];
            tmem_ld16(t_lane + 32u * (j & 1) + c0, s);
            asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
            float mine = -INFINITY;  // maximum of head `own` over this warp's latents
#pragma unroll
            for (int h = 0; h < kLtCols; h++) {
                const float v = seen ? __uint_as_float(s[h]) * scale : -INFINITY;
                s[h] = __float_as_uint(v);
                const float m = redux_max(v);
                if ((lane & 15) == h) mine = m;
            }
            s_max[q][own] = mine;
            ok = all_of_four_warps(half, ok);  // the four go on or give up together, here and nowhere else
            if (!ok) break;
            const float mx = fmaxf(fmaxf(s_max[0][own], s_max[1][own]), fmaxf(s_max[2][own], s_max[3][own]));
            const bool grow = mx > ref + 8.f;  // always when a head sees its first latents
            const float alpha = grow ? fast_exp2(ref - mx) : 1.f;
            if (grow) ref = mx;
            s_ref[q][own] = ref == -INFINITY ? 0.f : ref;
            const bool any = __any_sync(0xffffffffu, grow) && j > 0;
            if (any) s_alpha[q][own] = alpha;
            __syncwarp();
            if (any) {
                ok = mbar_wait(o_full0 + 8 * ((j - 1) & 1), ((j - 1) >> 1) & 1);  // the second product of the tile before: O is at rest
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                for (int i = 0; i < p.n_pair; i++) {
                    uint32_t o[kLtCols];
                    tmem_ld16(t_lane + kLtO + 32u * i + c0, o);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int h = 0; h < kLtCols; h++) o[h] = __float_as_uint(__uint_as_float(o[h]) * s_alpha[q][c0 + h]);
                    tmem_st16(t_lane + kLtO + 32u * i + c0, o);
                }
                asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
#pragma unroll
                for (int h = 0; h < kLtCols; h++) l[h] *= s_alpha[q][c0 + h];
            }
            unsigned char* dst = sP + (j & 1) * kLtPChunk + c0 * 128 + (row & 7) * 2;
            const int unit = row >> 3;
#pragma unroll
            for (int h = 0; h < kLtCols; h += 4) {  // every reference is read before the first store
                const float4 r = *reinterpret_cast<const float4*>(&s_ref[q][c0 + h]);
                s[h] = __float_as_uint(fast_exp2(__uint_as_float(s[h]) - r.x));
                s[h + 1] = __float_as_uint(fast_exp2(__uint_as_float(s[h + 1]) - r.y));
                s[h + 2] = __float_as_uint(fast_exp2(__uint_as_float(s[h + 2]) - r.z));
                s[h + 3] = __float_as_uint(fast_exp2(__uint_as_float(s[h + 3]) - r.w));
            }
#pragma unroll
            for (int h = 0; h < kLtCols; h++) {
                l[h] += __uint_as_float(s[h]);
                if (lane < 16) *reinterpret_cast<bf16*>(dst + h * 128 + ((unit ^ (h & 7)) << 4)) = __float2bfloat16_rn(__uint_as_float(s[h]));
            }
            if (lane < 16 && !seen && half == 0) {  // the row holds anything (0 x NaN would poison the product): clear it
                unsigned char* r = smem + (size_t)(j % p.n_buf) * tile_bytes + (size_t)(row >> 3) * unit_bytes + (row & 7) * 128;
                for (int c = 0; c < 2 * p.n_pair; c++)
#pragma unroll
                    for (int u = 0; u < 8; u++) *reinterpret_cast<uint4*>(r + c * kLtChunk + u * 16) = make_uint4(0u, 0u, 0u, 0u);
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(p_full0 + 8 * (j & 1));
        }
        // sums of the heads; the four warps hold the same references.  (Only the first 16 lanes have weights; a lane hands half
        // of its heads to its partner at every step and ends with the whole sum of one.)
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) {
            const bool hi = lane & o;
#pragma unroll
            for (int h = 0; h < o; h++) {
                const float give = hi ? l[h] : l[h + o], keep = hi ? l[h + o] : l[h];
                l[h] = keep + __shfl_xor_sync(0xffffffffu, give, o);
            }
        }
        if (lane < 16) s_sum[q][own] = l[0];
        ok = ok && mbar_wait(o_full0 + 8 * ((n_tiles - 1) & 1), ((n_tiles - 1) >> 1) & 1);
        ok = all_of_four_warps(half, ok);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const float total_l = s_sum[0][own] + s_sum[1][own] + s_sum[2][own] + s_sum[3][own];
        const int ranges = lt_ranges(p, pos);
        const size_t part = ((size_t)t * gridDim.y + blockIdx.y) * p.n_split + split;
        const int el = 32 * q + lane, ld = p.n_pair * 128;
        if (ranges > 1) {
            if (q == 0 && lane < 16) p.part_ml[part * kLtHeads + own] = make_float2(ref, total_l);
            float* dst = p.part_o + (part * kLtHeads + c0) * ld + el;
            for (int i = 0; i < p.n_pair; i++, dst += 128) {
                uint32_t o[kLtCols];
                tmem_ld16(t_lane + kLtO + 32u * i + c0, o);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                for (int h = 0; h < kLtCols; h++) dst[h * ld] = ok ? __uint_as_float(o[h]) : 0.f;
            }
        } else {
            // through shared memory as [head][element] (every MMA and load has run, the tiles are free)
            s_ref[q][own] = own < nh && total_l > 0.f ? lt_out_factor(a, t, h0 + own) / total_l : 0.f;
            float* so = reinterpret_cast<float*>(smem) + c0 * ld;
            for (int i = 0; i < p.n_pair; i++) {
                uint32_t o[kLtCols];
                tmem_ld16(t_lane + kLtO + 32u * i + c0, o);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                for (int h = 0; h < kLtCols; h++) so[h * ld + i * 128 + el] = ok ? __uint_as_float(o[h]) : 0.f;
            }
            (void)all_of_four_warps(half, true);
            const int quads = p.rank_p / 4, mine = min(kLtCols, nh - c0);  // heads of this half
            for (int i = 32 * q + lane; i < mine * quads; i += 128) {
                const int h = i / quads, c = 4 * (i % quads);
                const float4 v = *reinterpret_cast<const float4*>(so + h * ld + c);
                const float f = s_ref[q][c0 + h];
                *reinterpret_cast<uint2*>(static_cast<bf16*>(a.out) + ((size_t)t * a.H + h0 + c0 + h) * p.rank_p + c) =
                    make_uint2(pack2<bf16>(v.x * f, v.y * f), pack2<bf16>(v.z * f, v.w * f));
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 2) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kLtTmem) : "memory");
    }
}

// Sum of the ranges of a head, weighted by their references; a thread has four elements.
__global__ void __launch_bounds__(128) latent_attn_tc_merge_kernel(const LtParams p, int groups)
{
    const LatentAttn& a = p.a;
    const int h = blockIdx.x, t = blockIdx.y, e = 4 * threadIdx.x, ld = p.n_pair * 128;
    pdl_launch_dependents();
    pdl_wait();
    int b, pos;
    locate(p.tp, t, b, pos);
    const int ranges = lt_ranges(p, pos);
    if (ranges <= 1 || e >= p.rank_p) return;  // one range: the attention kernel wrote the output itself
    const size_t part = ((size_t)t * groups + h / kLtHeads) * p.n_split;
    const float* src = p.part_o + (part * kLtHeads + h % kLtHeads) * ld + e;
    const float2* mls = p.part_ml + part * kLtHeads + h % kLtHeads;
    const size_t step = (size_t)kLtHeads * ld;
    float4 v[kLtMaxSplits];
    float2 ml[kLtMaxSplits];
#pragma unroll
    for (int r = 0; r < kLtMaxSplits; r++)
        if (r < ranges) {
            ml[r] = mls[r * kLtHeads];
            v[r] = *reinterpret_cast<const float4*>(src + r * step);
        }
    float M = -INFINITY, L = 0.f;
#pragma unroll
    for (int r = 0; r < kLtMaxSplits; r++)
        if (r < ranges) M = fmaxf(M, ml[r].x);
    if (M == -INFINITY) M = 0.f;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < kLtMaxSplits; r++)
        if (r < ranges) {
            const float w = fast_exp2(ml[r].x - M);
            L = fmaf(ml[r].y, w, L);
            o.x = fmaf(w, v[r].x, o.x);
            o.y = fmaf(w, v[r].y, o.y);
            o.z = fmaf(w, v[r].z, o.z);
            o.w = fmaf(w, v[r].w, o.w);
        }
    const float f = L > 0.f ? lt_out_factor(a, t, h) / L : 0.f;
    *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(a.out) + ((size_t)t * a.H + h) * p.rank_p + e) =
        make_uint2(pack2<__nv_bfloat16>(o.x * f, o.y * f), pack2<__nv_bfloat16>(o.z * f, o.w * f));
}

static const TimeoutFlag timeout_flag(tc_flag_read_clear);

bool latent_attn_tc_takes(const LatentAttn& a, const TokenPositions& tp)
{
    return !tp.cu && a.dtype == ONELLM_BF16 && a.rank <= 64 * 2 * kLtMaxPairs && (long)tp.B * a.R < (1l << 31);
}

size_t latent_attn_tc_workspace(int tokens, int H, int rank)
{
    const size_t groups = (H + kLtHeads - 1) / kLtHeads, elements = (size_t)(rank + 127) / 128 * 128;
    // n_split * tokens * groups stays below the number of SMs unless there is one range only, which needs none
    const size_t parts = std::min<size_t>((size_t)tokens * groups * kLtMaxSplits, 512);
    return parts * kLtHeads * (elements * sizeof(float) + sizeof(float2));
}

int latent_attn_tc(const LatentAttn& a, const TokenPositions& tp, int tokens, int span_bound, void* workspace, cudaStream_t st)
{
    LtParams p = {a, tp};
    p.rank_p = latent_pad(a.rank);
    p.n_pair = (p.rank_p + 127) / 128;
    const int rows = a.R > a.window ? a.R : std::min(span_bound, a.R);
    const int tiles = (rows + kLtRows - 1) / kLtRows, groups = (a.H + kLtHeads - 1) / kLtHeads;
    const int n = std::max(1, std::min({kLtMaxSplits, tiles, std::min(num_sms(), 512) / (tokens * groups)}));
    p.tiles_per_split = (tiles + n - 1) / n;
    p.n_split = (tiles + p.tiles_per_split - 1) / p.tiles_per_split;
    const size_t tile_bytes = (size_t)2 * p.n_pair * kLtChunk * (kLtRows / kLtUnitRows), rest = 1024 + 2 * p.n_pair * kLtQChunk + 2 * kLtPChunk;
    p.n_buf = std::min({kLtMaxBufs, p.tiles_per_split, (int)((220 * 1024 - rest) / tile_bytes)});
    p.part_o = static_cast<float*>(workspace);
    p.part_ml = reinterpret_cast<float2*>(p.part_o + (size_t)tokens * groups * p.n_split * p.n_pair * 128 * kLtHeads);
    CUtensorMap map_c, map_q;
    RC(make_chunk_map(&map_c, a.ring, (uint64_t)p.rank_p, (uint64_t)tp.B * a.R, kLtUnitRows, 2 * p.n_pair));
    RC(make_map(&map_q, a.q, (uint64_t)p.rank_p, (uint64_t)tokens * a.H, kLtHeads));
    const size_t smem = rest + (size_t)p.n_buf * tile_bytes;
    static DeviceOnce attr;
    ONELLM_CUDA(attr.run([] { return cudaFuncSetAttribute(latent_attn_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024); }));
    ONELLM_CUDA(launch_pdl(latent_attn_tc_kernel, dim3(p.n_split, groups, tokens), dim3(kLtThreads), smem, st, p, map_c, map_q));
    if (p.n_split > 1) ONELLM_CUDA(launch_pdl(latent_attn_tc_merge_kernel, dim3(a.H, tokens), dim3(128), 0, st, p, groups));
    return ONELLM_OK;
}

}  // namespace onellm
