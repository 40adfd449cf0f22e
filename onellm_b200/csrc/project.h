// One projection of a model design, whatever the number of tokens: picks the weight-streaming, tcgen05 or fp32 kernel.
#pragma once
#include "common.cuh"

namespace onellm {

//   y[M,N] = x[M,K] . W                        W, W2 [K,N] of element type dtype (ONELLM_BF16 or ONELLM_F32)
//   y      = act(x . W) * (x . W2)             W2 given
//   y      = resid + x . W                     resid given (float, row stride ldy; may be y; with f32 or dtype F32)
// f32: y is float although x and W are bfloat16.  ldy 0: N.  bfloat16: K % 16 == 0, N and ldy % 8 == 0.
struct Projection {
    int dtype;
    const void *x, *W, *W2;
    void* y;
    long ldy;
    int M, N, K;
    int act;  // GateAct
    int f32;
    const float* resid;
};
int project(const Projection& p, cudaStream_t st);

}  // namespace onellm
