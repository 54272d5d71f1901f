// Gates of the matrix-memory layers, shared by the token-by-token and the chunked form.
#pragma once

#include "common.cuh"

namespace lumen {

__device__ __forceinline__ float rsqrtf_exact(float x) { return __fdiv_rn(1.0f, sqrtf(x)); }

// Log input gate cap * tanh((z_i + b_i) / cap) and log forget gate logsigmoid(cap * tanh((z_f + b_f) / cap)) of head h.
__device__ __forceinline__ void log_gates(const float *z, const float *bias, int H, int h, float cap, float &li, float &lf) {
    li = cap * tanhf(__fdiv_rn(z[h] + bias[h], cap));
    const float x = cap * tanhf(__fdiv_rn(z[H + h] + bias[H + h], cap));
    lf = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}

}  // namespace lumen
