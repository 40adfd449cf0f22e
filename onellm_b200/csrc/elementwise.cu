// Small HBM-bound kernels: SwiGLU on a packed [tokens, 2, I] buffer, the embedding gather, and the embedding with learned
// positions of designs that keep their residual stream in float.
//
// The first two replace silu_and_mul_kernel (src/kernels/activation_kernel.cu:10-21) and embeddingFunctor
// (src/kernels/input_embedding.cu:7-20) of the reference with 16-byte vectorised versions.
#include "mixers.h"

namespace onellm {

template <typename T>
__global__ void __launch_bounds__(256)
swiglu_kernel(const T* __restrict__ in, T* __restrict__ out, int inter)
{
    constexpr int VEC = Vec16<T>::N;
    pdl_launch_dependents();
    pdl_wait();
    const T* gate = in + (size_t)blockIdx.y * 2 * inter;
    const T* up = gate + inter;
    T* o = out + (size_t)blockIdx.y * inter;
    const int nvec = inter / VEC;
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < nvec; i += gridDim.x * blockDim.x) {
        float g[VEC], u[VEC], r[VEC];
        Vec16<T>::load(gate + (size_t)i * VEC, g);
        Vec16<T>::load(up + (size_t)i * VEC, u);
#pragma unroll
        for (int e = 0; e < VEC; e++) r[e] = (g[e] / (1.0f + expf(-g[e]))) * u[e];
        *reinterpret_cast<uint4*>(o + (size_t)i * VEC) = Vec16<T>::pack(r);
    }
}

template <typename T>
__global__ void __launch_bounds__(256)
embedding_kernel(const int* __restrict__ ids, T* __restrict__ out, T* __restrict__ out2, const T* __restrict__ table,
                 int hidden, int vocab, int* __restrict__ bad_id_flag)
{
    constexpr int VEC = Vec16<T>::N;
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && bad_id_flag && threadIdx.x == 0) atomicExch(bad_id_flag, 1);
    const uint4* src = reinterpret_cast<const uint4*>(table + (size_t)(ok ? id : 0) * hidden);
    uint4* dst = reinterpret_cast<uint4*>(out + (size_t)t * hidden);
    uint4* dst2 = out2 ? reinterpret_cast<uint4*>(out2 + (size_t)t * hidden) : nullptr;
    for (int i = threadIdx.x; i < hidden / VEC; i += blockDim.x) {
        const uint4 v = ok ? src[i] : make_uint4(0, 0, 0, 0);
        dst[i] = v;
        if (dst2) dst2[i] = v;
    }
}

}  // namespace onellm

using namespace onellm;

extern "C" int onellm_swiglu(int dtype, const void* input, void* out, int tokens, int inter, void* stream)
{
    ONELLM_REQUIRE(input && out, ONELLM_ERR_ARG, "swiglu: null pointer");
    ONELLM_REQUIRE(tokens >= 0 && inter > 0, ONELLM_ERR_ARG, "swiglu: bad size");
    const size_t es = dtype_size(dtype);
    ONELLM_REQUIRE(es != 0, ONELLM_ERR_UNSUPPORTED, "swiglu: dtype %d", dtype);
    ONELLM_REQUIRE(((size_t)inter * es) % 16 == 0 && aligned16(input) && aligned16(out), ONELLM_ERR_ARG,
                   "swiglu: rows must be 16-byte aligned");
    ONELLM_REQUIRE(tokens <= 65535, ONELLM_ERR_UNSUPPORTED, "swiglu: more than 65535 tokens per call");
    if (tokens == 0) return ONELLM_OK;
    cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
    const int nvec = inter / (int)(16 / es);
    const dim3 grid((nvec + 255) / 256, tokens);
    note_launch();
    if (dtype == ONELLM_F16)
        swiglu_kernel<__half><<<grid, 256, 0, st>>>((const __half*)input, (__half*)out, inter);
    else
        swiglu_kernel<float><<<grid, 256, 0, st>>>((const float*)input, (float*)out, inter);
    ONELLM_CHECK_LAUNCH();
    return ONELLM_OK;
}

namespace onellm {
// Shared by the C entry point and the model driver; out2 (may be NULL) receives a second copy
// of the rows (the residual stream).  `pdl` = false launches with a full stream dependency.
int embedding_launch(int dtype, const int* ids, void* out, void* out2, const void* table, int n_tokens, int hidden,
                     int vocab, int* bad_id_flag, bool pdl, cudaStream_t st)
{
    ONELLM_REQUIRE(ids && out && table, ONELLM_ERR_ARG, "embedding: null pointer");
    ONELLM_REQUIRE(n_tokens >= 0 && hidden > 0 && vocab > 0, ONELLM_ERR_ARG, "embedding: bad size");
    const size_t es = dtype_size(dtype);
    ONELLM_REQUIRE(es != 0, ONELLM_ERR_UNSUPPORTED, "embedding: dtype %d", dtype);
    ONELLM_REQUIRE(((size_t)hidden * es) % 16 == 0 && aligned16(out) && aligned16(table) && (!out2 || aligned16(out2)),
                   ONELLM_ERR_ARG, "embedding: rows must be 16-byte aligned");
    if (n_tokens == 0) return ONELLM_OK;
    if (!pdl) note_launch();  // launch_pdl counts its own
    if (dtype == ONELLM_F16) {
        if (pdl)
            ONELLM_CUDA(launch_pdl(embedding_kernel<__half>, dim3(n_tokens), dim3(256), 0, st, ids, (__half*)out,
                                   (__half*)out2, (const __half*)table, hidden, vocab, bad_id_flag));
        else
            embedding_kernel<__half><<<n_tokens, 256, 0, st>>>(ids, (__half*)out, (__half*)out2, (const __half*)table,
                                                               hidden, vocab, bad_id_flag);
    } else {
        if (pdl)
            ONELLM_CUDA(launch_pdl(embedding_kernel<float>, dim3(n_tokens), dim3(256), 0, st, ids, (float*)out,
                                   (float*)out2, (const float*)table, hidden, vocab, bad_id_flag));
        else
            embedding_kernel<float><<<n_tokens, 256, 0, st>>>(ids, (float*)out, (float*)out2, (const float*)table, hidden,
                                                              vocab, bad_id_flag);
    }
    ONELLM_CHECK_LAUNCH();
    return ONELLM_OK;
}
}  // namespace onellm

extern "C" int onellm_embedding(int dtype, const int* ids, void* out, const void* table, int n_tokens, int hidden,
                                int vocab, int* bad_id_flag, void* stream)
{
    return embedding_launch(dtype, ids, out, nullptr, table, n_tokens, hidden, vocab, bad_id_flag, true,
                            reinterpret_cast<cudaStream_t>(stream));
}

namespace onellm {
// Token embedding plus a learned position vector into a float residual stream:
//     out[t] = table[id] + pos_table[position],   both tables [.., ld] of element type T
// The position of token t: hist[b] + its index in sequence b (context pass: cu, hist), or step - 1 + off[t] (decode
// step: one token per sequence).  Ids outside [0, vocab) raise bad[0], positions outside [0, max_pos) bad[1]; both give a
// zero row.
template <typename T>
__global__ void __launch_bounds__(256)
embedding_pos_kernel(const int* __restrict__ ids, float* __restrict__ out, const T* __restrict__ table, const T* __restrict__ pos_table, int ld,
                     int vocab, int max_pos, const TokenPositions tp, int* __restrict__ bad)
{
    constexpr int VEC = Vec16<T>::N;
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, id = ids[t];
    int b, pos;
    locate(tp, t, b, pos);
    const bool id_ok = id >= 0 && id < vocab, pos_ok = pos >= 0 && pos < max_pos;
    if (threadIdx.x == 0) {
        if (!id_ok) atomicExch(bad, 1);
        if (!pos_ok) atomicExch(bad + 1, 1);
    }
    for (int i = threadIdx.x; i < ld / VEC; i += blockDim.x) {
        float a[VEC], p[VEC];
#pragma unroll
        for (int e = 0; e < VEC; e++) a[e] = p[e] = 0.f;
        if (id_ok && pos_ok) {
            Vec16<T>::load(table + (size_t)id * ld + (size_t)i * VEC, a);
            Vec16<T>::load(pos_table + (size_t)pos * ld + (size_t)i * VEC, p);
        }
        float4* dst = reinterpret_cast<float4*>(out + (size_t)t * ld + (size_t)i * VEC);
#pragma unroll
        for (int e = 0; e < VEC; e += 4) dst[e / 4] = make_float4(a[e] + p[e], a[e + 1] + p[e + 1], a[e + 2] + p[e + 2], a[e + 3] + p[e + 3]);
    }
}

// Launched with a full stream dependency (first kernel behind the step counter / the id upload).
int embedding_pos_launch(int dtype, const int* ids, float* out, const void* table, const void* pos_table, int n_tokens, int ld, int vocab,
                         int max_pos, const TokenPositions& tp, int* bad, cudaStream_t st)
{
    ONELLM_REQUIRE(ids && out && table && pos_table && bad && ld % 8 == 0, ONELLM_ERR_ARG, "embedding_pos: bad argument");
    if (n_tokens <= 0) return ONELLM_OK;
    note_launch();
    if (dtype == ONELLM_F32) {
        (void)prefer_max_shared((const void*)embedding_pos_kernel<float>);
        embedding_pos_kernel<float><<<n_tokens, 256, 0, st>>>(ids, out, (const float*)table, (const float*)pos_table, ld, vocab, max_pos, tp, bad);
    } else {
        (void)prefer_max_shared((const void*)embedding_pos_kernel<__nv_bfloat16>);
        embedding_pos_kernel<__nv_bfloat16><<<n_tokens, 256, 0, st>>>(ids, out, (const __nv_bfloat16*)table, (const __nv_bfloat16*)pos_table, ld,
                                                                     vocab, max_pos, tp, bad);
    }
    ONELLM_CHECK_LAUNCH();
    return ONELLM_OK;
}
}  // namespace onellm

extern "C" int onellm_embedding_pos(int dtype, const int* ids, float* out, const void* table, const void* pos_table, int n_tokens, int ld,
                                    int vocab, int max_pos, const onellm_token_positions* tp, int* bad, void* stream)
{
    ONELLM_REQUIRE(tp, ONELLM_ERR_ARG, "embedding_pos: null pointer");
    ONELLM_REQUIRE(dtype == ONELLM_BF16 || dtype == ONELLM_F32, ONELLM_ERR_UNSUPPORTED, "embedding_pos: dtype %d", dtype);
    return embedding_pos_launch(dtype, ids, out, table, pos_table, n_tokens, ld, vocab, max_pos, *tp, bad, reinterpret_cast<cudaStream_t>(stream));
}

namespace onellm {
// Token embedding through an RMSNorm into a float residual stream: out[t] = norm(table[id]) * w over `width` of ld columns.
template <typename T>
__global__ void __launch_bounds__(256)
embedding_norm_kernel(const int* __restrict__ ids, float* __restrict__ out, const T* __restrict__ table, const float* __restrict__ w, float eps,
                      int width, int ld, int vocab, int* __restrict__ bad)
{
    constexpr int VEC = Vec16<T>::N;
    __shared__ float part[8];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    if (threadIdx.x == 0 && !ok) atomicExch(bad, 1);
    const T* src = table + (size_t)(ok ? id : 0) * ld;
    float ss = 0.f;
    for (int i = threadIdx.x; i < ld / VEC; i += blockDim.x) {
        float a[VEC];
        Vec16<T>::load(src + (size_t)i * VEC, a);
#pragma unroll
        for (int e = 0; e < VEC; e++) ss = fmaf(a[e], a[e], ss);
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) total += part[i];
    const float inv = ok ? 1.0f / sqrtf(total / (float)width + eps) : 0.f;
    for (int i = threadIdx.x; i < ld / VEC; i += blockDim.x) {
        float a[VEC];
        Vec16<T>::load(src + (size_t)i * VEC, a);
        const float4* g = reinterpret_cast<const float4*>(w + (size_t)i * VEC);
        float4* dst = reinterpret_cast<float4*>(out + (size_t)t * ld + (size_t)i * VEC);
#pragma unroll
        for (int e = 0; e < VEC; e += 4) {
            const float4 k = g[e / 4];
            dst[e / 4] = make_float4(a[e] * inv * k.x, a[e + 1] * inv * k.y, a[e + 2] * inv * k.z, a[e + 3] * inv * k.w);
        }
    }
}

// Launched with a full stream dependency, as embedding_pos_launch.
int embedding_norm_launch(int dtype, const int* ids, float* out, const void* table, const float* w, float eps, int n_tokens, int width, int ld,
                          int vocab, int* bad, cudaStream_t st)
{
    ONELLM_REQUIRE(ids && out && table && w && bad && ld % 8 == 0 && width > 0 && width <= ld, ONELLM_ERR_ARG, "embedding_norm: bad argument");
    ONELLM_REQUIRE(dtype == ONELLM_BF16 || dtype == ONELLM_F32, ONELLM_ERR_UNSUPPORTED, "embedding_norm: dtype %d", dtype);
    if (n_tokens <= 0) return ONELLM_OK;
    note_launch();
    if (dtype == ONELLM_F32) {
        (void)prefer_max_shared((const void*)embedding_norm_kernel<float>);
        embedding_norm_kernel<float><<<n_tokens, 256, 0, st>>>(ids, out, (const float*)table, w, eps, width, ld, vocab, bad);
    } else {
        (void)prefer_max_shared((const void*)embedding_norm_kernel<__nv_bfloat16>);
        embedding_norm_kernel<__nv_bfloat16><<<n_tokens, 256, 0, st>>>(ids, out, (const __nv_bfloat16*)table, w, eps, width, ld, vocab, bad);
    }
    ONELLM_CHECK_LAUNCH();
    return ONELLM_OK;
}

// out[r, c] = cap * tanh(in[r, c] / cap), rows of ld elements into dense rows
__global__ void __launch_bounds__(256) softcap_kernel(const float* __restrict__ in, long ld, float* __restrict__ out, int cols, float cap)
{
    pdl_launch_dependents();
    pdl_wait();
    const float* src = in + (size_t)blockIdx.y * ld;
    float* dst = out + (size_t)blockIdx.y * cols;
    for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < cols; c += gridDim.x * blockDim.x) dst[c] = cap * tanhf(src[c] / cap);
}

int softcap(const float* in, long ld, float* out, int rows, int cols, float cap, cudaStream_t st)
{
    ONELLM_REQUIRE(in && out && ld >= cols && cols > 0 && cap > 0.f, ONELLM_ERR_ARG, "softcap: bad argument");
    for (int r = 0; r < rows; r += 65535) {
        const int n = rows - r < 65535 ? rows - r : 65535;
        ONELLM_CUDA(launch_pdl(softcap_kernel, dim3((cols + 1023) / 1024, n), dim3(256), 0, st, in + (size_t)r * ld, ld, out + (size_t)r * cols, cols, cap));
    }
    return ONELLM_OK;
}
}  // namespace onellm

extern "C" int onellm_embedding_norm(int dtype, const int* ids, float* out, const void* table, const float* w, float eps, int n_tokens, int width,
                                     int ld, int vocab, int* bad, void* stream)
{
    return embedding_norm_launch(dtype, ids, out, table, w, eps, n_tokens, width, ld, vocab, bad, reinterpret_cast<cudaStream_t>(stream));
}

extern "C" int onellm_softcap(const float* in, long ld, float* out, int rows, int cols, float cap, void* stream)
{
    return softcap(in, ld, out, rows, cols, cap, reinterpret_cast<cudaStream_t>(stream));
}
