// One projection of a model design, whatever the number of tokens: picks the weight-streaming, tcgen05 or fp32 kernel.
#pragma once
#include "common.cuh"

namespace onellm {

using RowGroups = onellm_row_groups;
// The parameters are described in onellm_b200.h; everything not set is zero, the scale of the product one.
struct Projection : onellm_projection {
    Projection() : onellm_projection() { scale = 1.f; }
};
int project(const onellm_projection& p, cudaStream_t st);

}  // namespace onellm
