// act.cuh -- the activations of include/crabml_seqops.h (cc_activation) as device functions, in 32-bit floats (expf / tanhf of the CUDA math
// library); shared by the sequence ops, the routed feed-forward and the operand conversion of the dense products.
#pragma once
#include "../../include/crabml_seqops.h"

__device__ __forceinline__ float act_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float act_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float act_gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }
__device__ __forceinline__ float act_relu_squared(float z) { const float r = fmaxf(z, 0.0f); return r * r; }
// alpha: CC_ACT_SWISH only
__device__ __forceinline__ float act_apply(float z, int act, float alpha = 1.0f) {
    switch (act) {
    case CC_ACT_SILU: return act_silu(z);
    case CC_ACT_GELU_TANH: return act_gelu_tanh(z);
    case CC_ACT_SWISH: return z / (1.0f + expf(-(alpha * z)));
    case CC_ACT_SIGMOID: return act_sigmoid(z);
    case CC_ACT_RELU_SQUARED: return act_relu_squared(z);
    }
    return z;
}
// the gated unit: act(min(g, limit)) * (clamp(u, -limit, limit) + up_shift); limit <= 0 clamps nothing
__device__ __forceinline__ float glu_apply(float g, float u, const cc_glu_params P) {
    if (P.limit > 0.0f) { g = fminf(g, P.limit); u = fminf(fmaxf(u, -P.limit), P.limit); }
    return act_apply(g, P.act, P.alpha) * (u + P.up_shift);
}
