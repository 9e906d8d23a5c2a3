// Kernels of layers whose sublayers stand side by side behind one norm, of Dynamic Tanh norms, and of a
// per-token input from a second table.  float32 arithmetic whatever the storage type; accurate tanhf /
// sqrtf (no fast-math).
//
//   dyt_rows        v = x[t] (+ s * delta[t]);  out[r] = tanh(alpha * v) * w + b  (Dynamic Tanh: no mean, no
//                   variance); the sum is written back to x on request; rows may be gathered.
//   join_sum_rows   v = sa * norm_a(a[t]) + sb * norm_b(b[t]) + c[t], norm_a(a) = a / rms(a) * wa (no weight:
//                   a itself); x[t] = (x[t]) + mult * v; low[t] = x[t] in the activation type.  b, c and low
//                   are optional; without `add` the old x is not read.
//   join_dyt_rows   x[t] += mult * y[t] / rms(y[t]) * wy;  out[t] = tanh(alpha * x[t]) * w + b: a norm on what
//                   joins the stream followed by the Dynamic Tanh in front of the next layer, in one pass.
//   token_gate      out[t, c] = gelu_tanh(z[t, c]) * table[token[t], c]  (c < dim; 0 in the padding columns)
//
// The row kernels come in a form with four columns a thread and the row in registers (float32 rows whose
// width and strides are multiples of 4) and a scalar form; which of the two runs depends on sizes and
// addresses only, never on the batch.
#include "common.cuh"
#include <math.h>

template <typename T> __device__ __forceinline__ void store4(T* p, const float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, const float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, const float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
}
__device__ __forceinline__ float sq4(const float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// Two block-wide sums in one round of barriers, in a fixed order; `red` holds 66 floats.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    if (lane == 0) { red[warp] = a; red[33 + warp] = b; }
    __syncthreads();
    float ta = 0.f, tb = 0.f;
    for (int i = 0; i < nw; ++i) { ta += red[i]; tb += red[33 + i]; }
    return make_float2(ta, tb);
}

static inline bool al(const void* p, int bytes) { return ((uintptr_t)p & (bytes - 1)) == 0; }
// few rows (a decode step) get more threads each, since the row's sums keep it in one block
static inline int row_threads(int n, int per_row) {
    int threads = n < 128 ? 1024 : 256;
    while (threads > 32 && threads / 2 >= per_row) threads >>= 1;
    return threads;
}

// ------------------------------------------------------------------ Dynamic Tanh
template <typename TO, int V>
__global__ void __launch_bounds__(1024)
dyt_rows_kernel(float* x, const float* delta, float s, const int* rows, float alpha, const float* __restrict__ w,
                const float* __restrict__ b, TO* out, int d, int write_x) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t src = rows ? (size_t)rows[blockIdx.x] : blockIdx.x;
    for (int i = threadIdx.x * V; i < d; i += blockDim.x * V) {
        float v[V];
        if constexpr (V == 4) {
            const float4 q = *reinterpret_cast<const float4*>(x + src * d + i);
            v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
        } else {
            v[0] = x[src * d + i];
        }
        if (delta) {
#pragma unroll
            for (int e = 0; e < V; ++e) {
                v[e] += s * delta[src * d + i + e];
                if (write_x) x[src * d + i + e] = v[e];
            }
        }
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = tanhf(alpha * v[e]) * w[i + e] + b[i + e];
        TO* o = out + (size_t)blockIdx.x * d + i;
        if constexpr (V == 4) store4<TO>(o, make_float4(v[0], v[1], v[2], v[3]));
        else o[0] = from_f<TO>(v[0]);
    }
}

RLLM_API int rllm_dyt_rows(float* x, const float* delta, float s, const int* rows, float alpha, const float* w,
                           const float* b, void* out, int out_dt, int n, int d, int write_x, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (d <= 0) return (int)cudaErrorInvalidValue;
    const bool vec = (d & 3) == 0 && al(x, 16) && al(out, 16);
    const dim3 grid(n), block(row_threads(n, vec ? d / 4 : d));
#define LAUNCH(TO, V) \
    return rllm_launch(dyt_rows_kernel<TO, V>, grid, block, 0, stream, x, delta, s, rows, alpha, w, b, (TO*)out, d, write_x)
    if (out_dt == RLLM_F32) {
        if (vec) { LAUNCH(float, 4); }
        LAUNCH(float, 1);
    }
    if (vec) { LAUNCH(bf16, 4); }
    LAUNCH(bf16, 1);
#undef LAUNCH
}

// ------------------------------------------------------------------ two outputs, normed, and a third, joined
struct JoinSum {
    const float *a, *wa, *b, *wb, *c;      // b, c: null when there is none; wa, wb: null for no norm
    long long ld_a, ld_b, ld_c;
    float sa, sb, eps_a, eps_b, mult;
    float* x;
    int add;
};

template <typename TL>
__global__ void __launch_bounds__(1024)
join_sum_rows_kernel(const JoinSum p, TL* low, int d) {
    __shared__ float red[66];
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const float* a = p.a + t * p.ld_a;
    const float* b = p.b ? p.b + t * p.ld_b : nullptr;
    const float* c = p.c ? p.c + t * p.ld_c : nullptr;
    float ra = p.sa, rb = p.sb;
    if (p.wa || p.wb) {
        float qa = 0.f, qb = 0.f;
        for (int i = threadIdx.x; i < d; i += blockDim.x) {
            qa += a[i] * a[i];
            if (b) qb += b[i] * b[i];
        }
        const float2 q = block_sum2(qa, qb, red);
        if (p.wa) ra *= 1.0f / sqrtf(q.x / (float)d + p.eps_a);
        if (p.wb) rb *= 1.0f / sqrtf(q.y / (float)d + p.eps_b);
    }
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        float v = a[i] * ra * (p.wa ? p.wa[i] : 1.f);
        if (b) v += b[i] * rb * (p.wb ? p.wb[i] : 1.f);
        if (c) v += c[i];
        v = p.mult * v + (p.add ? p.x[t * d + i] : 0.f);
        p.x[t * d + i] = v;
        if (low) low[t * d + i] = from_f<TL>(v);
    }
}

template <typename TL, int NV>
__global__ void __launch_bounds__(256)
join_sum_rows_vec_kernel(const JoinSum p, TL* low, int d) {
    __shared__ float red[66];
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int d4 = d >> 2;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4* a4 = reinterpret_cast<const float4*>(p.a + t * p.ld_a);
    const float4* b4 = reinterpret_cast<const float4*>(p.b + t * p.ld_b);
    const float4* c4 = reinterpret_cast<const float4*>(p.c + t * p.ld_c);
    float4* x4 = reinterpret_cast<float4*>(p.x + t * d);
    float4 va[NV], vb[NV];
    float qa = 0.f, qb = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = k * blockDim.x + threadIdx.x;
        va[k] = i < d4 ? a4[i] : zero;
        vb[k] = (p.b && i < d4) ? b4[i] : zero;
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        qa += sq4(va[k]);
        qb += sq4(vb[k]);
    }
    float ra = p.sa, rb = p.sb;
    if (p.wa || p.wb) {
        const float2 q = block_sum2(qa, qb, red);
        if (p.wa) ra *= 1.0f / sqrtf(q.x / (float)d + p.eps_a);
        if (p.wb) rb *= 1.0f / sqrtf(q.y / (float)d + p.eps_b);
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = k * blockDim.x + threadIdx.x;
        if (i >= d4) continue;
        const float4 one = make_float4(1.f, 1.f, 1.f, 1.f);
        const float4 wa = p.wa ? reinterpret_cast<const float4*>(p.wa)[i] : one;
        const float4 wb = p.wb ? reinterpret_cast<const float4*>(p.wb)[i] : one;
        const float4 c = p.c ? c4[i] : zero;
        const float4 o = p.add ? x4[i] : zero;
        float4 v;
        v.x = p.mult * (va[k].x * ra * wa.x + vb[k].x * rb * wb.x + c.x) + o.x;
        v.y = p.mult * (va[k].y * ra * wa.y + vb[k].y * rb * wb.y + c.y) + o.y;
        v.z = p.mult * (va[k].z * ra * wa.z + vb[k].z * rb * wb.z + c.z) + o.z;
        v.w = p.mult * (va[k].w * ra * wa.w + vb[k].w * rb * wb.w + c.w) + o.w;
        x4[i] = v;
        if (low) store4<TL>(low + t * d + 4 * (size_t)i, v);
    }
}

template <typename TL>
static int launch_join_sum(const JoinSum& p, TL* low, int n, int d, cudaStream_t stream) {
    const bool vec = d >= 256 && d <= 8192 && (d & 3) == 0 && ((p.ld_a | p.ld_b | p.ld_c) & 3) == 0 && al(p.a, 16) && al(p.b, 16) &&
                     al(p.c, 16) && al(p.wa, 16) && al(p.wb, 16) && al(p.x, 16) && al(low, 4 * (int)sizeof(TL));
    if (!vec) return rllm_launch(join_sum_rows_kernel<TL>, dim3(n), dim3(row_threads(n, d)), 0, stream, p, low, d);
#define JV(NV) return rllm_launch(join_sum_rows_vec_kernel<TL, NV>, dim3(n), dim3(256), 0, stream, p, low, d)
    const int nv = (d / 4 + 255) / 256;
    if (nv <= 1) { JV(1); }
    if (nv <= 2) { JV(2); }
    if (nv <= 4) { JV(4); }
    JV(8);
#undef JV
}

RLLM_API int rllm_join_sum_rows(const float* a, long long ld_a, const float* wa, float eps_a, float sa, const float* b,
                                long long ld_b, const float* wb, float eps_b, float sb, const float* c, long long ld_c,
                                float mult, float* x, int add, void* low, int low_dt, int n, int d, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (d <= 0 || !a || !x || ld_a < d || (b && ld_b < d) || (c && ld_c < d)) return (int)cudaErrorInvalidValue;
    const JoinSum p = {a, wa, b, b ? wb : nullptr, c, ld_a, b ? ld_b : 0, c ? ld_c : 0, sa, sb, eps_a, eps_b, mult, x, add};
    if (!low || low_dt == RLLM_F32) return launch_join_sum<float>(p, (float*)low, n, d, stream);
    return launch_join_sum<bf16>(p, (bf16*)low, n, d, stream);
}

// ------------------------------------------------------------------ a normed row joins, Dynamic Tanh of the sum
template <typename TO>
__global__ void __launch_bounds__(1024)
join_dyt_rows_kernel(const float* y, long long ld_y, const float* __restrict__ wy, float eps, float mult, float* x,
                     float alpha, const float* __restrict__ w, const float* __restrict__ b, TO* out, int d) {
    __shared__ float red[66];
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const float* row = y + t * ld_y;
    float q = 0.f;
    for (int i = threadIdx.x; i < d; i += blockDim.x) q += row[i] * row[i];
    q = block_sum2(q, 0.f, red).x;
    const float r = mult / sqrtf(q / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        const float v = x[t * d + i] + row[i] * r * wy[i];
        x[t * d + i] = v;
        out[t * d + i] = from_f<TO>(tanhf(alpha * v) * w[i] + b[i]);
    }
}

template <typename TO, int NV>
__global__ void __launch_bounds__(256)
join_dyt_rows_vec_kernel(const float* y, long long ld_y, const float* __restrict__ wy, float eps, float mult, float* x,
                         float alpha, const float* __restrict__ w, const float* __restrict__ b, TO* out, int d) {
    __shared__ float red[66];
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int d4 = d >> 2;
    const float4* y4 = reinterpret_cast<const float4*>(y + t * ld_y);
    float4* x4 = reinterpret_cast<float4*>(x + t * d);
    float4 v[NV], o[NV];
    float q = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = k * blockDim.x + threadIdx.x;
        v[k] = i < d4 ? y4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        o[k] = i < d4 ? x4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) q += sq4(v[k]);
    q = block_sum2(q, 0.f, red).x;
    const float r = mult / sqrtf(q / (float)d + eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = k * blockDim.x + threadIdx.x;
        if (i >= d4) continue;
        const float4 g = reinterpret_cast<const float4*>(wy)[i], ww = reinterpret_cast<const float4*>(w)[i],
                     bb = reinterpret_cast<const float4*>(b)[i];
        const float4 s = make_float4(o[k].x + v[k].x * r * g.x, o[k].y + v[k].y * r * g.y, o[k].z + v[k].z * r * g.z,
                                     o[k].w + v[k].w * r * g.w);
        x4[i] = s;
        store4<TO>(out + t * d + 4 * (size_t)i,
                   make_float4(tanhf(alpha * s.x) * ww.x + bb.x, tanhf(alpha * s.y) * ww.y + bb.y,
                               tanhf(alpha * s.z) * ww.z + bb.z, tanhf(alpha * s.w) * ww.w + bb.w));
    }
}

template <typename TO>
static int launch_join_dyt(const float* y, long long ld_y, const float* wy, float eps, float mult, float* x, float alpha,
                           const float* w, const float* b, TO* out, int n, int d, cudaStream_t stream) {
    const bool vec = d >= 256 && d <= 8192 && (d & 3) == 0 && (ld_y & 3) == 0 && al(y, 16) && al(wy, 16) && al(x, 16) &&
                     al(w, 16) && al(b, 16) && al(out, 4 * (int)sizeof(TO));
    if (!vec)
        return rllm_launch(join_dyt_rows_kernel<TO>, dim3(n), dim3(row_threads(n, d)), 0, stream, y, ld_y, wy, eps, mult, x,
                           alpha, w, b, out, d);
#define JV(NV)                                                                                                            \
    return rllm_launch(join_dyt_rows_vec_kernel<TO, NV>, dim3(n), dim3(256), 0, stream, y, ld_y, wy, eps, mult, x, alpha, w, \
                       b, out, d)
    const int nv = (d / 4 + 255) / 256;
    if (nv <= 1) { JV(1); }
    if (nv <= 2) { JV(2); }
    if (nv <= 4) { JV(4); }
    JV(8);
#undef JV
}

RLLM_API int rllm_join_dyt_rows(const float* y, long long ld_y, const float* wy, float eps, float mult, float* x,
                                float alpha, const float* w, const float* b, void* out, int out_dt, int n, int d,
                                cudaStream_t stream) {
    if (n <= 0) return 0;
    if (d <= 0 || ld_y < d || !y || !wy || !x || !w || !b || !out) return (int)cudaErrorInvalidValue;
    if (out_dt == RLLM_F32)
        return launch_join_dyt<float>(y, ld_y, wy, eps, mult, x, alpha, w, b, (float*)out, n, d, stream);
    return launch_join_dyt<bf16>(y, ld_y, wy, eps, mult, x, alpha, w, b, (bf16*)out, n, d, stream);
}

// ------------------------------------------------------------------ a gate on a row of a token table
template <typename T>
__global__ void token_gate_kernel(const float* z, long long ld_z, const T* __restrict__ table, const int* tokens, T* out,
                                  int dim, int padded, int vocab, size_t total, int* err) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const size_t t = i / padded;
    const int c = (int)(i - t * padded);
    const int tok = tokens[t];
    float v = 0.f;
    if (tok < 0 || tok >= vocab) {
        if (err && c == 0) atomicExch(err, RLLM_ERR_TOKEN);
    } else if (c < dim) {
        const float g = z[t * ld_z + c];
        v = 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * to_f<T>(table[(size_t)tok * dim + c]);
    }
    out[i] = from_f<T>(v);
}

RLLM_API int rllm_token_gate(const float* z, long long ld_z, const void* table, const int* tokens, void* out, int dt, int n,
                             int dim, int padded, int vocab, int* err, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (dim <= 0 || padded < dim || ld_z < dim || vocab <= 0) return (int)cudaErrorInvalidValue;
    const size_t total = (size_t)n * padded;
    const dim3 grid((unsigned)((total + 127) / 128)), block(128);
    if (dt == RLLM_F32)
        return rllm_launch(token_gate_kernel<float>, grid, block, 0, stream, z, ld_z, (const float*)table, tokens, (float*)out,
                           dim, padded, vocab, total, err);
    return rllm_launch(token_gate_kernel<bf16>, grid, block, 0, stream, z, ld_z, (const bf16*)table, tokens, (bf16*)out, dim,
                       padded, vocab, total, err);
}

RLLM_PACKED(rllm_dyt_rows)
RLLM_PACKED(rllm_join_sum_rows)
RLLM_PACKED(rllm_join_dyt_rows)
RLLM_PACKED(rllm_token_gate)
