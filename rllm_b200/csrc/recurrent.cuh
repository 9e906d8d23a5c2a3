// Element functions that the kernels of layers with a recurrent state share; accurate expf / log1pf.
#pragma once
#include <math.h>

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
