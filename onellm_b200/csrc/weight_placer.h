// Places the bfloat16 tensors of a model.safetensors file in a design's device memory: transposed into the [in, out] layout
// the projections take, as columns of a packed matrix, heads padded to the sizes the kernels take.
#pragma once
#include <string>

#include "model_files.h"

namespace onellm {

inline int pad_to(int x, int m) { return (x + m - 1) / m * m; }

struct WeightPlacer {
    int dtype;  // element type of the matrices placed: ONELLM_BF16 or ONELLM_F32
    cudaStream_t stream;
    SafeTensors file;

    WeightPlacer(int dtype_, cudaStream_t stream_) : dtype(dtype_), stream(stream_) {}
    ~WeightPlacer();
    WeightPlacer(const WeightPlacer&) = delete;
    WeightPlacer& operator=(const WeightPlacer&) = delete;

    // A tensor [out, in] into dst, a matrix with rows of ld elements, its first element at (row, col); transposed: element
    // (o, i) goes to row (i / in_d) * in_p + i % in_d and column (o / out_d) * out_p + o % out_d behind them, else to the
    // mirrored place.  What lies between stays as it is.
    int place(const std::string& name, void* dst, int ld, int row, int col, int out, int out_d, int out_p, int in, int in_d, int in_p,
              bool transposed = true);
    // The whole of a plain matrix: [in, out] columns from `col` on.
    int columns(const std::string& name, void* dst, int ld, int col, int out, int in) { return place(name, dst, ld, 0, col, out, out, out, in, in, in); }
    // A matrix [out, in] kept as it is, in float, rows of ld elements, groups of out_d rows padded to out_p.
    int rows_f32(const std::string& name, float* dst, int ld, int out, int out_d, int out_p, int in);
    // A vector kept in float, groups of d elements padded to p.
    int vec(const std::string& name, float* dst, int n, int d, int p);
    int vec(const std::string& name, float* dst, int n) { return vec(name, dst, n, n, n); }

  private:
    int fetch(const std::string& name, int64_t rows, int64_t cols);
    void* stage_ = nullptr;  // raw bfloat16 data of a tensor
    size_t stage_bytes_ = 0;
};

}  // namespace onellm
