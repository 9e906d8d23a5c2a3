// Activations by number, shared by the kernels that take one as a parameter (accurate expf / tanhf / log1pf):
// 0 identity, 1 silu z / (1 + e^-z), 2 relu(z)^2, 3 sigmoid, 4 tanh, 5 softplus.
#pragma once
#include <math.h>

enum : int { ACT_NONE = 0, ACT_SILU = 1, ACT_RELU2 = 2, ACT_SIGMOID = 3, ACT_TANH = 4, ACT_SOFTPLUS = 5 };

__device__ __forceinline__ float act_apply(float z, int act) {
    switch (act) {
        case ACT_SILU: return z / (1.0f + expf(-z));
        case ACT_RELU2: { const float r = fmaxf(z, 0.f); return r * r; }
        case ACT_SIGMOID: return 1.0f / (1.0f + expf(-z));
        case ACT_TANH: return tanhf(z);
        case ACT_SOFTPLUS: return z > 20.f ? z : log1pf(expf(z));
        default: return z;
    }
}
