// The activations that a product may apply to its result before it is stored as bfloat16, shared by the one-block product
// (gemm_tc.cu) and the product on pairs of SMs (gemm_tc_pair.cu).  All are 32-bit, with the fast exponential and
// reciprocal (a few units in the last place, far below the bfloat16 rounding that follows): with short inner widths the
// epilogue, not the products, sets the kernel's time.
#pragma once
#include <cuda_runtime.h>

namespace {

// SWIGLU  silu(g) * u                                                        of two products (gate rows, then up rows)
// CLAMPED g' sigmoid(alpha g') (u' + 1), g' = min(g, limit), u' = clamp(u, -limit, limit)    of two products
// RELU2   max(x, 0)^2                                                        of one product
enum : int { ACT_SWIGLU = 0, ACT_CLAMPED = 1, ACT_RELU2 = 2 };

struct ActEpilogue {
    int kind;
    float limit, alpha;
};

__device__ __forceinline__ float act_gated(const ActEpilogue& a, float g, float u) {
    if (a.kind == ACT_CLAMPED) {
        g = fminf(g, a.limit);
        u = fminf(fmaxf(u, -a.limit), a.limit);
        return __fdividef(g, 1.0f + __expf(-a.alpha * g)) * (u + 1.0f);
    }
    return __fdividef(g, 1.0f + __expf(-g)) * u;
}

__device__ __forceinline__ float act_single(float x) {
    const float m = fmaxf(x, 0.0f);
    return m * m;
}

}  // namespace
