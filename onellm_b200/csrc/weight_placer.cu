#include "weight_placer.h"

#include "engine.h"

namespace onellm {

template <typename T>
__global__ void place_kernel(T* __restrict__ dst, int ld, const __nv_bfloat16* __restrict__ src, int out, int in, int out_d, int out_p, int in_d,
                             int in_p, int transposed)
{
    const size_t n = (size_t)out * in;
    for (size_t e = blockIdx.x * (size_t)blockDim.x + threadIdx.x; e < n; e += (size_t)gridDim.x * blockDim.x) {
        const int o = (int)(e / in), i = (int)(e % in);
        const size_t r = (size_t)(i / in_d) * in_p + i % in_d, col = (size_t)(o / out_d) * out_p + o % out_d;
        dst[transposed ? r * ld + col : col * ld + r] = from_float<T>(__bfloat162float(src[e]));
    }
}

WeightPlacer::~WeightPlacer()
{
    if (stage_) cudaFree(stage_);
}

// the tensor's raw bfloat16 data in the stage
int WeightPlacer::fetch(const std::string& name, int64_t rows, int64_t cols)
{
    const SafeTensor* t = file.find(name);
    ONELLM_REQUIRE(t, ONELLM_ERR_IO, "no tensor %s", name.c_str());
    const std::vector<int64_t> want = cols > 0 ? std::vector<int64_t>{rows, cols} : std::vector<int64_t>{rows};
    ONELLM_REQUIRE(t->shape == want && t->dtype == "BF16", ONELLM_ERR_IO, "tensor %s: expected bfloat16 [%lld%s%s]", name.c_str(), (long long)rows,
                   cols > 0 ? ", " : "", cols > 0 ? std::to_string(cols).c_str() : "");
    std::vector<char> raw;
    RC(file.read(*t, &raw));
    ONELLM_REQUIRE(raw.size() == (size_t)rows * (cols > 0 ? cols : 1) * 2, ONELLM_ERR_IO, "tensor %s: wrong number of bytes", name.c_str());
    if (raw.size() > stage_bytes_) {
        if (stage_) cudaFree(stage_);
        stage_ = nullptr;
        stage_bytes_ = 0;
        ONELLM_CUDA(cudaMalloc(&stage_, raw.size()));
        stage_bytes_ = raw.size();
    }
    ONELLM_CUDA(cudaMemcpyAsync(stage_, raw.data(), raw.size(), cudaMemcpyHostToDevice, stream));
    ONELLM_CUDA(cudaStreamSynchronize(stream));  // `raw` goes away, the stage is used again
    return ONELLM_OK;
}

int WeightPlacer::place(const std::string& name, void* dst, int ld, int row, int col, int out, int out_d, int out_p, int in, int in_d, int in_p,
                        bool transposed)
{
    RC(fetch(name, out, in));
    const size_t at = transposed ? (size_t)row * ld + col : (size_t)col * ld + row;
    const int nb = blocks_for((size_t)out * in);
    const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(stage_);
    if (dtype == ONELLM_F32)
        place_kernel<float><<<nb, 256, 0, stream>>>(static_cast<float*>(dst) + at, ld, src, out, in, out_d, out_p, in_d, in_p, transposed);
    else
        place_kernel<__nv_bfloat16><<<nb, 256, 0, stream>>>(static_cast<__nv_bfloat16*>(dst) + at, ld, src, out, in, out_d, out_p, in_d, in_p, transposed);
    ONELLM_CHECK_LAUNCH();
    ONELLM_CUDA(cudaStreamSynchronize(stream));
    return ONELLM_OK;
}

int WeightPlacer::rows_f32(const std::string& name, float* dst, int ld, int out, int out_d, int out_p, int in)
{
    RC(fetch(name, out, in));
    place_kernel<float><<<blocks_for((size_t)out * in), 256, 0, stream>>>(dst, ld, static_cast<const __nv_bfloat16*>(stage_), out, in, out_d, out_p, in, in, 0);
    ONELLM_CHECK_LAUNCH();
    ONELLM_CUDA(cudaStreamSynchronize(stream));
    return ONELLM_OK;
}

int WeightPlacer::vec(const std::string& name, float* dst, int n, int d, int p)
{
    RC(fetch(name, n, 0));
    place_kernel<float><<<blocks_for(n), 256, 0, stream>>>(dst, 1, static_cast<const __nv_bfloat16*>(stage_), n, 1, d, p, 1, 1, 0);
    ONELLM_CHECK_LAUNCH();
    ONELLM_CUDA(cudaStreamSynchronize(stream));
    return ONELLM_OK;
}

}  // namespace onellm
