// Context-phase projections (M > 64 tokens) on the 5th-generation tensor cores of sm_100a.
//
// Replaces the cuBLAS GEMM behind launchLinearGemm (src/kernels/qkv_linear.cu:8-65,
// src/kernels/cublas_wrapper.cc:45-90 of the reference) for prefill shapes: y[M,N] = x[M,K] . W with
// W [K,N] (the layer weights, N contiguous) or W [N,K] (the LM head), fp16 in, fp32 accumulate.
//
// Persistent: one block per SM walks 128 x 256 output tiles (with 128 x 128 tiles the operand traffic from L2
// into shared memory, 15.6 KB per MFLOP, was what bounded the kernel; the wider tile needs 11.7) in an order
// that keeps the tiles in flight on a near-square patch of the output.  Warp 0 streams 64-deep K slices of
// both operands into a ring of four shared-memory stages with TMA (cp.async.bulk.tensor, 128-byte swizzle; no
// cluster multicast anywhere); one thread of warp 1 issues tcgen05.mma (M = 128, N = 256, K = 16, kind::f16)
// and releases each stage with tcgen05.commit; tensor memory holds two 256-column accumulators, so warps 2-5
// (tcgen05.ld, convert, store) drain tile i while the MMAs of tile i + 1 run.
// The [K,N] weight is used as it lies in memory: it is the "MN-major" B operand of the MMA
// (four 64-column TMA boxes per stage), so no transposed copy of the weights is ever made.
// Every wait on an mbarrier is bounded; on a time-out the block records it in a device flag,
// skips its stores, frees its tensor memory and exits.
#include <cuda.h>

#include <algorithm>
#include <mutex>

#include "project.h"
#include "tc_common.cuh"

namespace onellm {

constexpr int kTcBM = 128, kTcBN = 256, kTcBK = 64;
constexpr int kTcStages = 4;
constexpr int kTcBand = 16;  // row tiles per band of the tile order
constexpr int kTcThreads = 192;      // producer warp, MMA warp, four epilogue warps
constexpr int kTcEpiThreads = 128;
constexpr int kTcATile = kTcBM * kTcBK * 2;        // 16 KB: 128 rows x 128 bytes
constexpr int kTcBTile = kTcBN * kTcBK * 2;        // 32 KB: [K,N] four boxes of 64 k-rows x 128 bytes; [N,K] 256 rows x 128 bytes
constexpr int kTcBChunk = 64 * kTcBK * 2;          // 8 KB: one 64-column chunk of a [K,N] stage
constexpr int kTcStageBytes = kTcATile + kTcBTile;
constexpr int kTcSmemBytes = kTcStages * kTcStageBytes + 1024 /* alignment slack */ + 256 /* barriers, TMEM address */;

// W_NK = false: W [K,N] (B operand MN-major);  W_NK = true: W [N,K] (B operand K-major).
// Persistent: grid = min(tiles, SMs) blocks of six warps; block c works on tiles c, c + grid, ... in band
// order (see below).  Warp 0 (one thread) is the TMA producer, warp 1 (one thread) issues the MMAs,
// warps 2-5 are the epilogue.  Tensor memory holds TWO 128 x 256 accumulators, so the MMAs of the next
// tile run while the epilogue warps drain the previous one.
// MODE 2: two [K,N] weights; the 256 accumulator columns of a tile are 128 columns of x.W (gate) beside the
// same 128 columns of x.W2 (up), and the epilogue stores silu(gate) * up: the gate GEMM, the up GEMM and
// launchAct of src/layers/ffn/ffn.cpp:62-66 in one pass, without the [T, 2, I] buffer.
// Epilogue options that let the context phase run without norm kernels, as the decode step does (the norm's gamma
// is multiplied into the weight rows beforehand):
//   row_ss:  sums of squares of the rows of x, as ss_parts partial sums per row; the result rows are scaled by
//            rsqrt(sum / K + eps), i.e. this is the projection of RMSNorm(x)
//   resid:   y = resid + bias + result (resid may be y itself: an element is read and written by the same thread)
//   ss_out:  [M, ceil(N / tile columns)]: the sum of squares of the stored (rounded) values of each row inside this
//            tile's columns -- the row_ss of the projection that reads y next.  Every entry is written by exactly
//            one block, so the sums do not depend on the order the blocks run in.
//   act:     gate function of MODE 2
//   ldy:     row stride of y (and of resid); 0: N
//   f32:     y and resid are float instead of the element type (no ss_out then)
//   scale:   with f32, factor on the result in front of the residual
//   limit:   bound of the clamped gate function
// GROUPED: the rows of x and y lie in groups with weights of their own (onellm_row_groups: the experts of a mixture).  The
// row tiles come from a table, 128 rows of one group each; the weights are stacked, so that a tile reads K rows of W from
// row group * K on.  Columns of x behind K are zero-filled, so that a last K slice that reaches into the next weight adds
// nothing.
struct TcEpilogue {
    const float* row_ss;
    int ss_parts;
    float eps;
    const void* resid;
    const void* bias;
    float* ss_out;
    int act;
    long ldy;
    int f32;
    float scale = 1.f, limit = 0.f;
};

template <typename T, int MODE, bool GROUPED = false>
__global__ void __launch_bounds__(kTcThreads)
gemm_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b,
               const __grid_constant__ CUtensorMap map_b2, T* y, int M, int N, int K, const TcEpilogue epi, const RowGroups grp)
{
    constexpr bool W_NK = MODE == 1;
    constexpr bool DUAL = MODE == 2;
    constexpr int kOutN = DUAL ? kTcBN / 2 : kTcBN;  // output columns per tile
    extern __shared__ unsigned char smem_raw[];
    // 1024-byte alignment for the 128-byte swizzle pattern
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + kTcStages * kTcStageBytes);
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * kTcStages + 4);
    const uint32_t full0 = smem_u32(bars), empty0 = smem_u32(bars + kTcStages);
    const uint32_t acc_full0 = smem_u32(bars + 2 * kTcStages), acc_empty0 = smem_u32(bars + 2 * kTcStages + 2);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // Tile order: the linear tile index walks down a band of kTcBand row tiles, then moves one column
    // tile to the right, so the tiles in flight at one time (one per SM) cover a near-square patch
    // of the output and share their A row blocks and B column blocks in L2.  (Row-major order made every
    // wave touch all column tiles of B: operands were read from DRAM seven times over.)
    int tiles_m = (M + kTcBM - 1) / kTcBM;
    const int tiles_n = (N + kOutN - 1) / kOutN;
    int n_tiles = tiles_m * tiles_n;
    // first row and column of a tile, the row of the stacked weights it starts at, the end of its rows
    auto tile_origin = [&](int t, int& m0, int& n0, int& k0, int& m_end) {
        const int per_band = kTcBand * tiles_n;
        const int band = t / per_band, in_band = t % per_band;
        const int band_rows = min(kTcBand, tiles_m - band * kTcBand);
        const int mt = band * kTcBand + in_band % band_rows;
        n0 = (in_band / band_rows) * kOutN;
        if constexpr (GROUPED) {
            const int g = grp.tile_group[mt];
            m0 = grp.tile_row[mt];
            k0 = g * K;
            m_end = grp.off[g + 1];
        } else {
            m0 = mt * kTcBM;
            k0 = 0;
            m_end = M;
        }
    };
    const int k_steps = (K + kTcBK - 1) / kTcBK;

    if (threadIdx.x == 0) {
        for (int s = 0; s < kTcStages; s++) {
            mbar_init(full0 + 8 * s, 1);
            mbar_init(empty0 + 8 * s, 1);
        }
        for (int a = 0; a < 2; a++) {
            mbar_init(acc_full0 + 8 * a, 1);
            mbar_init(acc_empty0 + 8 * a, kTcEpiThreads);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 2) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(2u * kTcBN)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem_base = *tmem_slot;

    pdl_wait();  // x comes from the previous kernel in the stream
    if constexpr (GROUPED) {
        tiles_m = *grp.n_tiles;
        n_tiles = tiles_m * tiles_n;
    }

    if (warp == 0 && lane == 0) {
        // producer: one 64-deep slice of A and of B per stage, tile after tile
        int it = 0;
        bool ok = true;
        for (int t = blockIdx.x; t < n_tiles && ok; t += gridDim.x) {
            int m0, n0, k0, m_end;
            tile_origin(t, m0, n0, k0, m_end);
            for (int ks = 0; ks < k_steps; ks++, it++) {
                const int s = it % kTcStages;
                if (it >= kTcStages) ok = mbar_wait(empty0 + 8 * s, ((it / kTcStages) - 1) & 1);
                if (!ok) break;
                const uint32_t a_dst = smem_u32(smem + s * kTcStageBytes), b_dst = a_dst + kTcATile;
                mbar_expect_tx(full0 + 8 * s, kTcStageBytes);
                tma_load_2d(a_dst, &map_a, ks * kTcBK, m0, full0 + 8 * s);
                if (W_NK) {
                    tma_load_2d(b_dst, &map_b, ks * kTcBK, n0, full0 + 8 * s);
                } else if (DUAL) {
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        tma_load_2d(b_dst + c * kTcBChunk, &map_b, n0 + 64 * c, k0 + ks * kTcBK, full0 + 8 * s);
                        tma_load_2d(b_dst + (2 + c) * kTcBChunk, &map_b2, n0 + 64 * c, k0 + ks * kTcBK, full0 + 8 * s);
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < kTcBN / 64; c++)
                        tma_load_2d(b_dst + c * kTcBChunk, &map_b, n0 + 64 * c, k0 + ks * kTcBK, full0 + 8 * s);
                }
            }
        }
    } else if (warp == 1 && lane == 0) {
        // instruction descriptor: D = f32, A and B of type T, A K-major, B MN-major unless W_NK, N = 256, M = 128
        const uint32_t idesc = (1u << 4) | umma_operand_bits<T>() | ((W_NK ? 0u : 1u) << 16) | ((uint32_t)(kTcBN >> 3) << 17) | ((uint32_t)(kTcBM >> 4) << 24);
        int it = 0, lt = 0;
        bool ok = true;
        for (int t = blockIdx.x; t < n_tiles && ok; t += gridDim.x, lt++) {
            const int acc = lt & 1, use = lt >> 1;
            // the accumulator must have been drained by the epilogue of the tile that used it before
            if (use >= 1) ok = mbar_wait(acc_empty0 + 8 * acc, (use - 1) & 1);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t tmem_d = tmem_base + (uint32_t)(acc * kTcBN);
            for (int ks = 0; ks < k_steps; ks++, it++) {
                const int s = it % kTcStages;
                ok = mbar_wait(full0 + 8 * s, (it / kTcStages) & 1);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t a_addr = smem_u32(smem + s * kTcStageBytes), b_addr = a_addr + kTcATile;
#pragma unroll
                for (int kk = 0; kk < kTcBK / 16; kk++) {
                    // A: K-major, rows of 128 bytes, 8-row groups 1024 bytes apart; 16 k = 32 bytes further in the row
                    const uint64_t adesc = umma_desc(a_addr + kk * 32, 16, 1024);
                    // B [N,K]: same form.  B [K,N]: MN-major, 64-column chunks 8192 bytes apart (LBO), 8-row k groups
                    // 1024 bytes apart (SBO); 16 k = two groups further
                    const uint64_t bdesc = W_NK ? umma_desc(b_addr + kk * 32, 16, 1024) : umma_desc(b_addr + kk * 2048, kTcBChunk, 1024);
                    umma_f16(tmem_d, adesc, bdesc, idesc, (ks > 0 || kk > 0) ? 1u : 0u);
                }
                umma_commit(empty0 + 8 * s);  // frees the stage when these MMAs have read it
            }
            if (ok) umma_commit(acc_full0 + 8 * acc);  // the tile is complete when everything issued so far has run
        }
        pdl_launch_dependents();
    } else if (warp >= 2) {
        // epilogue: warp w may touch TMEM lanes 32 * (w % 4) .. + 31, which are the tile rows of the same numbers
        const int q = warp & 3;
        const size_t ldy = epi.ldy ? (size_t)epi.ldy : (size_t)N;
        int lt = 0;
        bool ok = true;
        for (int t = blockIdx.x; t < n_tiles && ok; t += gridDim.x, lt++) {
            const int acc = lt & 1, use = lt >> 1;
            int m0, n0, k0, m_end;
            tile_origin(t, m0, n0, k0, m_end);
            ok = mbar_wait(acc_full0 + 8 * acc, use & 1);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int row = m0 + q * 32 + lane;
            const bool row_ok = row < m_end;
            float inv = 1.f, sq = 0.f;
            const bool scaled = GROUPED ? grp.row_scale != nullptr : epi.row_ss != nullptr;
            if (GROUPED && scaled && row_ok) inv = grp.row_scale[row];
            if (epi.row_ss && row_ok) {
                float ssum = 0.f;
                for (int pp = 0; pp < epi.ss_parts; pp++) ssum += epi.row_ss[(size_t)row * epi.ss_parts + pp];
                inv = rsqrtf(ssum / (float)K + epi.eps);
            }
#pragma unroll 1
            for (int c0 = 0; c0 < kOutN; c0 += 32) {
                uint32_t r[32];
                tmem_ld32(tmem_base + ((uint32_t)(q * 32) << 16) + (uint32_t)(acc * kTcBN + c0), r);
                if (DUAL) {
                    uint32_t u[32];
                    tmem_ld32(tmem_base + ((uint32_t)(q * 32) << 16) + (uint32_t)(acc * kTcBN + kOutN + c0), u);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int i = 0; i < 32; i++) {
                        const float g = __uint_as_float(r[i]) * inv;
                        r[i] = __float_as_uint(gate_pair(g, __uint_as_float(u[i]) * inv, epi.act, epi.limit));
                    }
                } else {
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                    if (scaled) {
#pragma unroll
                        for (int i = 0; i < 32; i++) r[i] = __float_as_uint(__uint_as_float(r[i]) * inv);
                    }
                }
                if (row_ok) {
                    const size_t at = (size_t)row * ldy + n0 + c0;
#pragma unroll
                    for (int j = 0; j < 4; j++) {
                        if (n0 + c0 + 8 * j < N) {  // N is a multiple of 8
                            float v[8];
#pragma unroll
                            for (int e = 0; e < 8; e++) v[e] = __uint_as_float(r[8 * j + e]);
                            float a[8];
                            if (epi.bias) {
                                Vec16<T>::load(static_cast<const T*>(epi.bias) + n0 + c0 + 8 * j, a);
#pragma unroll
                                for (int e = 0; e < 8; e++) v[e] += a[e];
                            }
                            if (epi.f32) {
                                float4* dst = reinterpret_cast<float4*>(reinterpret_cast<float*>(y) + at + 8 * j);
                                if (epi.resid) {
                                    const float4* rs = reinterpret_cast<const float4*>(static_cast<const float*>(epi.resid) + at + 8 * j);
                                    const float4 r0 = rs[0], r1 = rs[1];
                                    const float sc = epi.scale;
                                    v[0] = fmaf(v[0], sc, r0.x); v[1] = fmaf(v[1], sc, r0.y); v[2] = fmaf(v[2], sc, r0.z); v[3] = fmaf(v[3], sc, r0.w);
                                    v[4] = fmaf(v[4], sc, r1.x); v[5] = fmaf(v[5], sc, r1.y); v[6] = fmaf(v[6], sc, r1.z); v[7] = fmaf(v[7], sc, r1.w);
                                }
                                dst[0] = make_float4(v[0], v[1], v[2], v[3]);
                                dst[1] = make_float4(v[4], v[5], v[6], v[7]);
                                continue;
                            }
                            if (epi.resid) {
                                Vec16<T>::load(static_cast<const T*>(epi.resid) + at + 8 * j, a);
#pragma unroll
                                for (int e = 0; e < 8; e++) v[e] += a[e];
                            }
                            const uint4 packed = Vec16<T>::pack(v);
                            *reinterpret_cast<uint4*>(y + at + 8 * j) = packed;
                            if (epi.ss_out) {
                                Vec16<T>::unpack(packed, v);  // what the next projection will read
#pragma unroll
                                for (int e = 0; e < 8; e++) sq = fmaf(v[e], v[e], sq);
                            }
                        }
                    }
                }
            }
            if (epi.ss_out && row_ok) epi.ss_out[(size_t)row * tiles_n + n0 / kOutN] = sq;
            // this thread's reads of the accumulator are over: hand it back to the MMA warp
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(acc_empty0 + 8 * acc);
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 2) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(2u * kTcBN) : "memory");
    }
}

// ---- host side -----------------------------------------------------------------------------------
using EncodeTiledFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                   const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static EncodeTiledFn encode_tiled()
{
    static EncodeTiledFn fn = nullptr;
    static std::mutex mu;
    std::lock_guard<std::mutex> lock(mu);
    if (!fn) {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess &&
            q == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<EncodeTiledFn>(p);
    }
    return fn;
}

// 2-D tensor map of 16-bit elements: `inner` contiguous elements, `outer` rows of `inner` elements; box {64, box_outer}; 128-byte swizzle
int make_map(CUtensorMap* map, const void* base, uint64_t inner, uint64_t outer, uint32_t box_outer)
{
    EncodeTiledFn enc = encode_tiled();
    ONELLM_REQUIRE(enc, ONELLM_ERR_CUDA, "gemm: cuTensorMapEncodeTiled is not available from the driver");
    const cuuint64_t dims[2] = {inner, outer};
    const cuuint64_t strides[1] = {inner * sizeof(__half)};
    const cuuint32_t box[2] = {64, box_outer};
    const cuuint32_t estr[2] = {1, 1};
    const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    ONELLM_REQUIRE(r == CUDA_SUCCESS, ONELLM_ERR_CUDA, "gemm: cuTensorMapEncodeTiled failed with %d", (int)r);
    return ONELLM_OK;
}

int make_chunk_map(CUtensorMap* map, const void* base, uint64_t inner, uint64_t outer, uint32_t box_rows, uint32_t box_chunks)
{
    EncodeTiledFn enc = encode_tiled();
    ONELLM_REQUIRE(enc, ONELLM_ERR_CUDA, "cuTensorMapEncodeTiled is not available from the driver");
    const cuuint64_t dims[3] = {64, outer, inner / 64};
    const cuuint64_t strides[2] = {inner * 2, 128};
    const cuuint32_t box[3] = {64, box_rows, box_chunks};
    const cuuint32_t estr[3] = {1, 1, 1};
    const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                           CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    ONELLM_REQUIRE(r == CUDA_SUCCESS, ONELLM_ERR_CUDA, "cuTensorMapEncodeTiled failed with %d", (int)r);
    return ONELLM_OK;
}

int gemm_f16_skinny(const __half* x, const __half* W, __half* y, int M, int N, int K, int w_layout, cudaStream_t st);

// mode 0: W [K,N]; 1: W [N,K]; 2: W and W2 [K,N], y = silu(x.W) * (x.W2)
template <typename T>
static int gemm_tc_launch(const T* x, const T* W, const T* W2, T* y, int M, int N, int K, int mode, cudaStream_t st,
                          const TcEpilogue& epi = TcEpilogue{})
{
    ONELLM_REQUIRE(K % 8 == 0 && N % 8 == 0, ONELLM_ERR_UNSUPPORTED, "gemm: M > 64 needs K %% 8 == 0 and N %% 8 == 0 (K=%d N=%d)",
                   K, N);
    CUtensorMap map_a, map_b, map_b2;
    int rc = make_map(&map_a, x, (uint64_t)K, (uint64_t)M, kTcBM);
    if (rc) return rc;
    rc = mode == 1 ? make_map(&map_b, W, (uint64_t)K, (uint64_t)N, kTcBN) : make_map(&map_b, W, (uint64_t)N, (uint64_t)K, kTcBK);
    if (rc) return rc;
    map_b2 = map_b;
    if (mode == 2) {
        rc = make_map(&map_b2, W2, (uint64_t)N, (uint64_t)K, kTcBK);
        if (rc) return rc;
    }
    static DeviceOnce smem_attr[3];
    {
        const void* fn = mode == 0 ? (const void*)gemm_tc_kernel<T, 0> : mode == 1 ? (const void*)gemm_tc_kernel<T, 1> : (const void*)gemm_tc_kernel<T, 2>;
        ONELLM_CUDA(smem_attr[mode].run([fn] { return cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, kTcSmemBytes); }));
    }
    const int out_n = mode == 2 ? kTcBN / 2 : kTcBN;
    const long tiles = (long)((N + out_n - 1) / out_n) * ((M + kTcBM - 1) / kTcBM);
    ONELLM_REQUIRE(tiles <= 0x7fffffffL, ONELLM_ERR_UNSUPPORTED, "gemm: too many tiles");
    const dim3 grid((unsigned)std::min<long>(tiles, num_sms()));  // persistent: one block per SM (shared memory allows no more)
    if (mode == 0)
        ONELLM_CUDA(launch_pdl(gemm_tc_kernel<T, 0>, grid, dim3(kTcThreads), kTcSmemBytes, st, map_a, map_b, map_b2, y, M, N, K, epi, RowGroups{}));
    else if (mode == 1)
        ONELLM_CUDA(launch_pdl(gemm_tc_kernel<T, 1>, grid, dim3(kTcThreads), kTcSmemBytes, st, map_a, map_b, map_b2, y, M, N, K, epi, RowGroups{}));
    else
        ONELLM_CUDA(launch_pdl(gemm_tc_kernel<T, 2>, grid, dim3(kTcThreads), kTcSmemBytes, st, map_a, map_b, map_b2, y, M, N, K, epi, RowGroups{}));
    return ONELLM_OK;
}

// Row groups (bfloat16): x has g.rows rows in group order, the weights are stacked.
static int gemm_tc_grouped(const onellm_projection& p, const TcEpilogue& epi, cudaStream_t st)
{
    typedef __nv_bfloat16 T;
    const RowGroups& g = *p.groups;
    ONELLM_REQUIRE(g.off && g.tile_group && g.tile_row && g.n_tiles && g.max_tiles > 0 && g.rows > 0 && g.weights > 0 && !g.x_rows && !g.x_stride &&
                       !g.y_stride && g.w_stride == (long)p.K * p.N && !p.ldw && !p.ldx && !p.resid,
                   ONELLM_ERR_UNSUPPORTED, "project: more than 64 rows per group need a tile table, rows in group order and stacked weights");
    CUtensorMap map_a, map_b, map_b2;
    int rc = make_map(&map_a, p.x, (uint64_t)p.K, (uint64_t)g.rows, kTcBM);
    if (!rc) rc = make_map(&map_b, p.W, (uint64_t)p.N, (uint64_t)p.K * g.weights, kTcBK);
    map_b2 = map_b;
    if (!rc && p.W2) rc = make_map(&map_b2, p.W2, (uint64_t)p.N, (uint64_t)p.K * g.weights, kTcBK);
    if (rc) return rc;
    const void* fn = p.W2 ? (const void*)gemm_tc_kernel<T, 2, true> : (const void*)gemm_tc_kernel<T, 0, true>;
    static DeviceOnce attr[2];
    ONELLM_CUDA(attr[p.W2 ? 1 : 0].run([fn] { return cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, kTcSmemBytes); }));
    const int out_n = p.W2 ? kTcBN / 2 : kTcBN;
    const long tiles = (long)((p.N + out_n - 1) / out_n) * g.max_tiles;
    ONELLM_REQUIRE(tiles <= 0x7fffffffL, ONELLM_ERR_UNSUPPORTED, "gemm: too many tiles");
    const dim3 grid((unsigned)std::min<long>(tiles, num_sms()));
    if (p.W2)
        ONELLM_CUDA(launch_pdl(gemm_tc_kernel<T, 2, true>, grid, dim3(kTcThreads), kTcSmemBytes, st, map_a, map_b, map_b2, (T*)p.y, p.M, p.N, p.K, epi, g));
    else
        ONELLM_CUDA(launch_pdl(gemm_tc_kernel<T, 0, true>, grid, dim3(kTcThreads), kTcSmemBytes, st, map_a, map_b, map_b2, (T*)p.y, p.M, p.N, p.K, epi, g));
    return ONELLM_OK;
}

int gemm_f16_large(const __half* x, const __half* W, __half* y, int M, int N, int K, int w_layout, cudaStream_t st)
{
    return gemm_tc_launch<__half>(x, W, nullptr, y, M, N, K, w_layout == ONELLM_W_NK ? 1 : 0, st);
}

// Gate and up projections with SwiGLU in the epilogue, M > 64.
int gemm_swiglu_f16_large(const __half* x, const __half* Wg, const __half* Wu, __half* out, int M, int I, int K, cudaStream_t st)
{
    return gemm_tc_launch<__half>(x, Wg, Wu, out, M, I, K, 2, st);
}

// Column tiles of a projection with N outputs (two weights: gate and up share a tile): the second extent of the
// [M, parts] array of partial row sums that onellm_gemm_rows writes.
int gemm_rows_parts(int N, bool dual)
{
    const int out_n = dual ? kTcBN / 2 : kTcBN;
    return (N + out_n - 1) / out_n;
}

// The large-M form of the norm-free projections (see TcEpilogue).
int gemm_rows_f16(const __half* x, const __half* W, const __half* W2, __half* y, int M, int N, int K, const float* row_ss, int ss_parts,
                  float eps, const __half* resid, const __half* bias, float* ss_out, cudaStream_t st)
{
    TcEpilogue epi = {};
    epi.row_ss = row_ss;
    epi.ss_parts = ss_parts;
    epi.eps = eps;
    epi.resid = resid;
    epi.bias = resid ? bias : nullptr;
    epi.ss_out = ss_out;
    return gemm_tc_launch<__half>(x, W, W2, y, M, N, K, W2 ? 2 : 0, st, epi);
}

// The bfloat16 form (more than 64 tokens, or rows in one group) behind project().
int gemm_bf16_large(const onellm_projection& p, cudaStream_t st)
{
    typedef __nv_bfloat16 bf16;
    TcEpilogue epi = {};
    epi.resid = p.resid;
    epi.act = p.act;
    epi.limit = p.limit;
    epi.scale = p.scale;
    epi.ldy = p.ldy;
    epi.f32 = p.f32;
    if (p.groups) return gemm_tc_grouped(p, epi, st);
    return gemm_tc_launch<bf16>((const bf16*)p.x, (const bf16*)p.W, (const bf16*)p.W2, static_cast<bf16*>(p.y), p.M, p.N, p.K, p.W2 ? 2 : 0, st, epi);
}

static const TimeoutFlag timeout_flag(tc_flag_read_clear);

}  // namespace onellm
