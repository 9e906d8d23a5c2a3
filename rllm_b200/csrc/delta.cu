// The gated delta rule behind short causal convolutions: a matrix memory per head that is decayed by one
// number per token and corrected towards the token's value along its key.
//
// A token's projection row (float32) holds q, k ([G * dk] each), v ([H * dv]), an output gate ([H * dv]) and two
// numbers per head, b and a.  Head h uses the q/k head h / (H / G).  With conv(.) the causal convolution of
// every channel over `taps` tokens (no bias, the last tap weighs the current token, zeros before the start):
//   q = unit(silu(conv(q))) * q_scale,  k = unit(silu(conv(k))),  v = silu(conv(v)),  unit(x) = x / sqrt(sum x^2 + unit_eps)
//   beta = sigmoid(b),  g = exp(-A * softplus(a + dt_bias))                        (A = exp(A_log), one per head)
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   out = o / rms(o) * norm_w * act(gate)                                          (rms over the head's dv entries)
// Everything here is float32; sums run in a fixed order, and who owns a state element is fixed by the sizes.
//
// State slot of a request (floats): S of every head (DK * dvp floats a head, DK the key size rounded up to 32,
// 64, 128, 256 or 512, dvp the value size rounded up to a multiple of 8), then per head the last taps - 1 inputs
// of its convolutions, [2 dk + dv][taps - 1], oldest first (q and k channels are kept once per value head, so
// that every head's block reads and moves on a copy of its own).  S lies in the threads' order: eight lanes
// (parts) share a pair of value columns; part p holds the key rows 32 m + 4 p + e (m < DK / 32, e < 4) of both;
// entry (row register ii, column c) of thread `gt` (column pair * 8 + part) is at (2 ii + c) * (dvp * 4) + gt.
//
// Two ways through a step, chosen from its shape alone:
//   delta_step    (few tokens per request: decode) one block per (head, request) does all of the above, the
//                 recurrence token by token with S in registers.
//   delta_prep, delta_chunk, delta_out  (prompt portions) chunks of 8 tokens, counted from the portion's start.
//                 prep: a block per (chunk, q/k head): convolutions and unit vectors of q and k, the products
//                 k_i . k_j and q_i . k_j inside the chunk, beta and g.  chunk: a block per (tile of value
//                 columns, head, request) walks the request's chunks with its part of S in registers.  With
//                 c_i = g_1 .. g_i and d_ij = g_(j+1) .. g_i (products taken factor by factor, from 1):
//                     u_i = beta_i (v_i - c_i S0^T k_i) - sum_(j<i) beta_i d_ij (k_i . k_j) u_j
//                     o_i = c_i S0^T q_i + sum_(j<=i) d_ij (q_i . k_j) u_j
//                     S   = c_8 S0 + sum_j d_8j k_j u_j^T
//                 which is the recurrence with the memory read once per chunk: the eight tokens' products with
//                 S0 are independent of one another, and only the small triangular system is a chain.
//                 out: norm, weight and gate per (token, head).
#include "common.cuh"
#include "recurrent.cuh"

#define DELTA_TOK 8            // tokens of a chunk
#define DELTA_PARTS 8          // lanes that share a pair of value columns

struct DeltaArgs {
    const float* rows;         // [n, ld]
    long long ld;
    int q_off, k_off, v_off, g_off, b_off, a_off;
    const float* conv;         // [2 G dk + H dv][taps]: q channels, k channels, v channels
    const float* A;            // [H] exp(A_log)
    const float* dt_bias;      // [H]
    const float* norm_w;       // [dv]
    float q_scale, unit_eps, eps;
    float* state;
    long long slot_stride, conv_base;
    const int* cu_q;
    const int* slots;
    int H, G, dk, dv, dvp, taps, gate, n_requests;
};

__device__ __forceinline__ float delta_gate_act(float z, int gate) {
    return gate == 1 ? silu_f(z) : gate == 2 ? 1.0f / (1.0f + expf(-z)) : 1.0f;
}
__device__ __forceinline__ float head_decay(const DeltaArgs& p, int h, float a) {
    return expf(-p.A[h] * softplus_f(a + p.dt_bias[h]));
}
// The convolution of one channel at the portion's token i: `x` the channel's column at the portion's first row,
// `kept` the channel's taps - 1 kept inputs.
__device__ __forceinline__ float conv_at(const float* x, long long ld, const float* kept, const float* __restrict__ w, int taps,
                                         int i) {
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {
        const int s = i - (taps - 1) + j;
        acc += w[j] * (s >= 0 ? x[(size_t)s * ld] : kept[taps - 1 + s]);
    }
    return silu_f(acc);
}
// The kept inputs of a channel after `len` more tokens (its own thread reads and writes them).
__device__ __forceinline__ void move_kept(const float* x, long long ld, float* kept, int taps, int len) {
    for (int j = 0; j < taps - 1; ++j) {
        const int s = len - (taps - 1) + j;
        kept[j] = s >= 0 ? x[(size_t)s * ld] : kept[j + len];
    }
}
// column of the projection row and row of the convolution weights for channel c of head h ([q | k | v])
__device__ __forceinline__ void head_channel(const DeltaArgs& p, int h, int c, int& col, int& wrow) {
    const int kh = h / (p.H / p.G);
    if (c < p.dk) { col = p.q_off + kh * p.dk + c; wrow = kh * p.dk + c; }
    else if (c < 2 * p.dk) { col = p.k_off + kh * p.dk + c - p.dk; wrow = p.G * p.dk + kh * p.dk + c - p.dk; }
    else { col = p.v_off + h * p.dv + c - 2 * p.dk; wrow = 2 * p.G * p.dk + h * p.dv + c - 2 * p.dk; }
}

// ------------------------------------------------------------------ few tokens: one block per (head, request)
template <typename TA, int DK>
__global__ void __launch_bounds__(512)
delta_step_kernel(const DeltaArgs p, TA* out) {
    constexpr int IPT = DK / DELTA_PARTS;
    extern __shared__ __align__(16) float sm_step[];
    float* s_q = sm_step;                            // [TOK][DK]
    float* s_k = s_q + DELTA_TOK * DK;               // [TOK][DK]
    float* s_v = s_k + DELTA_TOK * DK;               // [TOK][dvp]
    float* s_o = s_v + DELTA_TOK * p.dvp;            // [TOK][dvp]
    float* s_n = s_o + DELTA_TOK * p.dvp;            // [TOK][4]: beta, g, q . k
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x, NT = blockDim.x;
    const int warp = tid >> 5, lane = tid & 31, part = tid & 7;
    const int t0 = p.cu_q[r], len = p.cu_q[r + 1] - t0;
    const int C = 2 * p.dk + p.dv, pairs = p.dvp / 2, tile = NT / DELTA_PARTS;
    float* slot = p.state + (size_t)p.slots[r] * p.slot_stride;
    float* Sg = slot + (size_t)h * DK * p.dvp;
    float* kept = slot + p.conv_base + (size_t)h * C * (p.taps - 1);
    const float* x0 = p.rows + (size_t)t0 * p.ld;
    const size_t stride = (size_t)p.dvp * 4;
    float S0[IPT], S1[IPT];
    auto load = [&](int gt) {
#pragma unroll
        for (int ii = 0; ii < IPT; ++ii) {
            S0[ii] = Sg[(size_t)(2 * ii) * stride + gt];
            S1[ii] = Sg[(size_t)(2 * ii + 1) * stride + gt];
        }
    };
    const bool one_tile = pairs <= tile;
    if (one_tile && tid / DELTA_PARTS < pairs) load(tid);        // on its way while the convolutions run
    for (int c0 = 0; c0 < len; c0 += DELTA_TOK) {
        const int cnt = min(DELTA_TOK, len - c0);
        // q, k (zero rows behind dk) and v of the chunk
        for (int e = tid; e < cnt * 2 * DK; e += NT) {
            const int i = e / (2 * DK), c = e - i * 2 * DK, half = c >= DK, cc = half ? c - DK : c;
            float v = 0.f;
            if (cc < p.dk) {
                int col, wrow;
                head_channel(p, h, half * p.dk + cc, col, wrow);
                v = conv_at(x0 + col, p.ld, kept + (size_t)(half * p.dk + cc) * (p.taps - 1), p.conv + (size_t)wrow * p.taps,
                            p.taps, c0 + i);
            }
            (half ? s_k : s_q)[i * DK + cc] = v;
        }
        for (int e = tid; e < cnt * p.dvp; e += NT) {
            const int i = e / p.dvp, c = e - i * p.dvp;
            float v = 0.f;
            if (c < p.dv) {
                int col, wrow;
                head_channel(p, h, 2 * p.dk + c, col, wrow);
                v = conv_at(x0 + col, p.ld, kept + (size_t)(2 * p.dk + c) * (p.taps - 1), p.conv + (size_t)wrow * p.taps, p.taps,
                            c0 + i);
            }
            s_v[e] = v;
        }
        __syncthreads();
        for (int i = warp; i < cnt; i += NT >> 5) {
            float qq = 0.f, kk = 0.f, qk = 0.f;
            for (int c = lane; c < DK; c += 32) {
                const float a = s_q[i * DK + c], b = s_k[i * DK + c];
                qq += a * a;
                kk += b * b;
                qk += a * b;
            }
            qq = warp_sum(qq);
            kk = warp_sum(kk);
            qk = warp_sum(qk);
            const float rq = p.q_scale / sqrtf(qq + p.unit_eps), rk = 1.0f / sqrtf(kk + p.unit_eps);
            for (int c = lane; c < DK; c += 32) {
                s_q[i * DK + c] *= rq;
                s_k[i * DK + c] *= rk;
            }
            if (lane == 0) {
                const float* row = x0 + (size_t)(c0 + i) * p.ld;
                s_n[4 * i] = 1.0f / (1.0f + expf(-row[p.b_off + h]));
                s_n[4 * i + 1] = head_decay(p, h, row[p.a_off + h]);
                s_n[4 * i + 2] = qk * rq * rk;
            }
        }
        __syncthreads();
        for (int pair = tid / DELTA_PARTS; pair < pairs; pair += tile) {
            const int gt = pair * DELTA_PARTS + part;
            if (!one_tile) load(gt);
            for (int i = 0; i < cnt; ++i) {
                const float4* k4 = reinterpret_cast<const float4*>(s_k + i * DK) + part;
                const float4* q4 = reinterpret_cast<const float4*>(s_q + i * DK) + part;
                float ka = 0.f, kb = 0.f, qa = 0.f, qb = 0.f;
#pragma unroll
                for (int m = 0; m < IPT / 4; ++m) {
                    const float4 k = k4[8 * m], q = q4[8 * m];
                    ka += k.x * S0[4 * m] + k.y * S0[4 * m + 1] + k.z * S0[4 * m + 2] + k.w * S0[4 * m + 3];
                    kb += k.x * S1[4 * m] + k.y * S1[4 * m + 1] + k.z * S1[4 * m + 2] + k.w * S1[4 * m + 3];
                    qa += q.x * S0[4 * m] + q.y * S0[4 * m + 1] + q.z * S0[4 * m + 2] + q.w * S0[4 * m + 3];
                    qb += q.x * S1[4 * m] + q.y * S1[4 * m + 1] + q.z * S1[4 * m + 2] + q.w * S1[4 * m + 3];
                }
#pragma unroll
                for (int o = 4; o > 0; o >>= 1) {
                    ka += __shfl_xor_sync(0xffffffffu, ka, o);
                    kb += __shfl_xor_sync(0xffffffffu, kb, o);
                    qa += __shfl_xor_sync(0xffffffffu, qa, o);
                    qb += __shfl_xor_sync(0xffffffffu, qb, o);
                }
                const float beta = s_n[4 * i], g = s_n[4 * i + 1], qk = s_n[4 * i + 2];
                const float2 v = *reinterpret_cast<const float2*>(s_v + i * p.dvp + 2 * pair);
                const float ua = beta * (v.x - g * ka), ub = beta * (v.y - g * kb);
                if (part == 0)
                    *reinterpret_cast<float2*>(s_o + i * p.dvp + 2 * pair) = make_float2(g * qa + qk * ua, g * qb + qk * ub);
#pragma unroll
                for (int m = 0; m < IPT / 4; ++m) {
                    const float4 k = k4[8 * m];
                    const float kv[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        S0[4 * m + e] = g * S0[4 * m + e] + kv[e] * ua;
                        S1[4 * m + e] = g * S1[4 * m + e] + kv[e] * ub;
                    }
                }
            }
            if (!one_tile || c0 + DELTA_TOK >= len) {
#pragma unroll
                for (int ii = 0; ii < IPT; ++ii) {
                    Sg[(size_t)(2 * ii) * stride + gt] = S0[ii];
                    Sg[(size_t)(2 * ii + 1) * stride + gt] = S1[ii];
                }
            }
        }
        __syncthreads();
        for (int i = warp; i < cnt; i += NT >> 5) {
            float ss = 0.f;
            for (int c = lane; c < p.dv; c += 32) ss += s_o[i * p.dvp + c] * s_o[i * p.dvp + c];
            ss = warp_sum(ss);
            const float rs = 1.0f / sqrtf(ss / (float)p.dv + p.eps);
            const size_t t = t0 + c0 + i;
            const float* gate = p.rows + t * p.ld + p.g_off + (size_t)h * p.dv;
            for (int c = lane; c < p.dv; c += 32) {
                float v = s_o[i * p.dvp + c] * rs * p.norm_w[c];
                if (p.gate) v *= delta_gate_act(gate[c], p.gate);
                out[(t * p.H + h) * p.dv + c] = from_f<TA>(v);
            }
        }
        __syncthreads();
    }
    for (int c = tid; c < C; c += NT) {
        int col, wrow;
        head_channel(p, h, c, col, wrow);
        move_kept(x0 + col, p.ld, kept + (size_t)c * (p.taps - 1), p.taps, len);
    }
}

// ------------------------------------------------------------------ portions: what a chunk needs beside the memory
// qn, kn [n, G * dk]: the unit vectors (q times q_scale).  prods [n, G, 16]: token i of a chunk has k_i . k_j at
// [j] and q_i . k_j at [8 + j] for j <= i.  bg [n, H, 2]: beta and g.
__global__ void __launch_bounds__(256)
delta_prep_kernel(const DeltaArgs p, float* qn, float* kn, float* prods, float* bg) {
    extern __shared__ __align__(16) float sm_prep[];
    float* s_q = sm_prep;                            // [TOK][dk]
    float* s_k = s_q + DELTA_TOK * p.dk;
    pdl_launch_dependents();
    pdl_wait();
    int chunk = blockIdx.x, r = 0, len = 0;
    for (; r < p.n_requests; ++r) {
        len = p.cu_q[r + 1] - p.cu_q[r];
        const int c = (len + DELTA_TOK - 1) / DELTA_TOK;
        if (chunk < c) break;
        chunk -= c;
    }
    if (r >= p.n_requests) return;
    const int kh = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rep = p.H / p.G;
    const int t0 = p.cu_q[r], c0 = chunk * DELTA_TOK, cnt = min(DELTA_TOK, len - c0);
    const float* x0 = p.rows + (size_t)t0 * p.ld;
    const int C = 2 * p.dk + p.dv;
    const float* kept = p.state + (size_t)p.slots[r] * p.slot_stride + p.conv_base + (size_t)kh * rep * C * (p.taps - 1);
    for (int c = tid; c < 2 * p.dk; c += blockDim.x) {       // a thread takes a channel's tokens
        const bool is_k = c >= p.dk;
        const int cc = is_k ? c - p.dk : c;
        const float* x = x0 + (is_k ? p.k_off : p.q_off) + kh * p.dk + cc;
        const float* w = p.conv + (size_t)((is_k ? p.G * p.dk : 0) + kh * p.dk + cc) * p.taps;
        const float* kp = kept + (size_t)c * (p.taps - 1);
        float* dst = (is_k ? s_k : s_q) + cc;
        if (p.taps == 4) {
            float v[DELTA_TOK + 3];
#pragma unroll
            for (int j = 0; j < DELTA_TOK + 3; ++j) {
                const int s = c0 + j - 3;
                v[j] = s >= len ? 0.f : s >= 0 ? x[(size_t)s * p.ld] : kp[3 + s];
            }
            const float w0 = w[0], w1 = w[1], w2 = w[2], w3 = w[3];
#pragma unroll
            for (int i = 0; i < DELTA_TOK; ++i)
                dst[i * p.dk] = silu_f(w0 * v[i] + w1 * v[i + 1] + w2 * v[i + 2] + w3 * v[i + 3]);
        } else {
            for (int i = 0; i < cnt; ++i) dst[i * p.dk] = conv_at(x, p.ld, kp, w, p.taps, c0 + i);
        }
    }
    __syncthreads();
    for (int i = warp; i < cnt; i += 8) {
        float qq = 0.f, kk = 0.f;
        for (int c = lane; c < p.dk; c += 32) {
            qq += s_q[i * p.dk + c] * s_q[i * p.dk + c];
            kk += s_k[i * p.dk + c] * s_k[i * p.dk + c];
        }
        const float rq = p.q_scale / sqrtf(warp_sum(qq) + p.unit_eps), rk = 1.0f / sqrtf(warp_sum(kk) + p.unit_eps);
        const size_t row = ((size_t)(t0 + c0 + i) * p.G + kh) * p.dk;
        for (int c = lane; c < p.dk; c += 32) {
            const float a = s_q[i * p.dk + c] * rq, b = s_k[i * p.dk + c] * rk;
            s_q[i * p.dk + c] = qn[row + c] = a;
            s_k[i * p.dk + c] = kn[row + c] = b;
        }
    }
    __syncthreads();
    for (int i = warp; i < cnt; i += 8) {
        float kk[DELTA_TOK], qk[DELTA_TOK];
#pragma unroll
        for (int j = 0; j < DELTA_TOK; ++j) kk[j] = qk[j] = 0.f;
        for (int c = lane; c < p.dk; c += 32) {
            const float a = s_q[i * p.dk + c], b = s_k[i * p.dk + c];
#pragma unroll
            for (int j = 0; j < DELTA_TOK; ++j) {
                const float o = j <= i ? s_k[j * p.dk + c] : 0.f;
                kk[j] += b * o;
                qk[j] += a * o;
            }
        }
        float* dst = prods + ((size_t)(t0 + c0 + i) * p.G + kh) * 2 * DELTA_TOK;
#pragma unroll
        for (int j = 0; j < DELTA_TOK; ++j) {
            const float a = warp_sum(kk[j]), b = warp_sum(qk[j]);
            if (lane == 0) { dst[j] = a; dst[DELTA_TOK + j] = b; }
        }
    }
    for (int e = tid; e < cnt * rep; e += blockDim.x) {
        const int i = e / rep, h = kh * rep + e % rep;
        const size_t t = t0 + c0 + i;
        const float* row = p.rows + t * p.ld;
        bg[(t * p.H + h) * 2] = 1.0f / (1.0f + expf(-row[p.b_off + h]));
        bg[(t * p.H + h) * 2 + 1] = head_decay(p, h, row[p.a_off + h]);
    }
}

// ------------------------------------------------------------------ portions: the walk through the chunks
__device__ __forceinline__ void delta_cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void delta_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
// Sums of eight values over the eight lanes of a group; lane `part` ends with the sum of value number `part`.
__device__ __forceinline__ float reduce8(const float (&a)[DELTA_TOK], int part) {
    float b[4], c[2];
    const bool h4 = part & 4, h2 = part & 2, h1 = part & 1;
#pragma unroll
    for (int j = 0; j < 4; ++j) b[j] = (h4 ? a[4 + j] : a[j]) + __shfl_xor_sync(0xffffffffu, h4 ? a[j] : a[4 + j], 4);
#pragma unroll
    for (int j = 0; j < 2; ++j) c[j] = (h2 ? b[2 + j] : b[j]) + __shfl_xor_sync(0xffffffffu, h2 ? b[j] : b[2 + j], 2);
    return (h1 ? c[1] : c[0]) + __shfl_xor_sync(0xffffffffu, h1 ? c[0] : c[1], 1);
}

#define DELTA_NT 128
#define DELTA_COLS (2 * DELTA_NT / DELTA_PARTS)      // value columns of a block

template <int DK>
__global__ void __launch_bounds__(DELTA_NT)
delta_chunk_kernel(const DeltaArgs p, const float* qn, const float* kn, const float* prods, const float* bg, float* o) {
    constexpr int IPT = DK / DELTA_PARTS, T = DELTA_TOK, NC = DELTA_COLS;
    extern __shared__ __align__(16) float sm_chunk[];
    const int W = T + p.taps - 1;                    // rows of the values' window
    const int stage = 2 * T * DK + T * 16 + 2 * T + (W * NC + 3) / 4 * 4;
    float* s_kk = sm_chunk + 2 * stage;              // [T][T] beta_i d_ij (k_i . k_j), j < i
    float* s_qk = s_kk + T * T;                      // [T][T] d_ij (q_i . k_j), j <= i, else 0
    float* s_c = s_qk + T * T;                       // [T] c_i
    float* s_d = s_c + T;                            // [T] d_8j
    const int tid = threadIdx.x, part = tid & 7, lane = tid & 31;
    const int n_tiles = (p.dvp + NC - 1) / NC, h = blockIdx.x / n_tiles, tile = blockIdx.x % n_tiles, r = blockIdx.y;
    const int kh = h / (p.H / p.G), C = 2 * p.dk + p.dv;
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = p.cu_q[r], len = p.cu_q[r + 1] - t0;
    if (len <= 0) return;
    float* slot = p.state + (size_t)p.slots[r] * p.slot_stride;
    float* Sg = slot + (size_t)h * DK * p.dvp;
    float* kept = slot + p.conv_base + (size_t)h * C * (p.taps - 1);
    const float* kept_v = kept + (size_t)2 * p.dk * (p.taps - 1);
    const float* x0 = p.rows + (size_t)t0 * p.ld;
    const int col0 = tile * NC, pair = col0 / 2 + tid / DELTA_PARTS, gt = pair * DELTA_PARTS + part, cl = 2 * (tid / DELTA_PARTS);
    const bool live = 2 * pair < p.dvp;
    const size_t stride = (size_t)p.dvp * 4;
    const bool vec = (p.dk & 3) == 0;
    float S0[IPT], S1[IPT];
#pragma unroll
    for (int ii = 0; ii < IPT; ++ii) {
        S0[ii] = live ? Sg[(size_t)(2 * ii) * stride + gt] : 0.f;
        S1[ii] = live ? Sg[(size_t)(2 * ii + 1) * stride + gt] : 0.f;
    }
    // both stages start as zeros: the columns behind dk and behind the last token's rows are never filled
    for (int e = tid; e < 2 * stage; e += DELTA_NT) sm_chunk[e] = 0.f;
    __syncthreads();
    auto fetch = [&](int c0, float* st) {
        const int cnt = min(T, len - c0);
        float *q = st, *k = st + T * DK, *pr = k + T * DK, *b = pr + T * 16, *v = b + 2 * T;
        const size_t t = t0 + c0;
        if (vec) {
            const int d4 = p.dk >> 2;
            for (int e = tid; e < cnt * d4; e += DELTA_NT) {
                const int i = e / d4, c = 4 * (e - i * d4);
                const size_t src = ((t + i) * p.G + kh) * p.dk + c;
                delta_cp16(q + i * DK + c, qn + src);
                delta_cp16(k + i * DK + c, kn + src);
            }
        } else {
            for (int e = tid; e < cnt * p.dk; e += DELTA_NT) {
                const int i = e / p.dk, c = e - i * p.dk;
                const size_t src = ((t + i) * p.G + kh) * p.dk + c;
                delta_cp4(q + i * DK + c, qn + src);
                delta_cp4(k + i * DK + c, kn + src);
            }
        }
        if (tid < 4 * cnt) delta_cp16(pr + 4 * tid, prods + ((t + tid / 4) * p.G + kh) * 16 + 4 * (tid & 3));
        if (tid < 2 * cnt) delta_cp4(b + tid, bg + ((t + tid / 2) * p.H + h) * 2 + (tid & 1));
        for (int e = tid; e < (cnt + p.taps - 1) * NC; e += DELTA_NT) {
            const int i = e / NC, c = col0 + e % NC;
            if (c >= p.dv) continue;
            const int s = c0 + i - (p.taps - 1);
            delta_cp4(v + e, s >= 0 ? x0 + (size_t)s * p.ld + p.v_off + (size_t)h * p.dv + c
                                    : kept_v + (size_t)c * (p.taps - 1) + p.taps - 1 + s);
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    const float* wv0 = p.conv + (size_t)(2 * p.G * p.dk + h * p.dv + min(col0 + cl, p.dv - 1)) * p.taps;
    const float* wv1 = p.conv + (size_t)(2 * p.G * p.dk + h * p.dv + min(col0 + cl + 1, p.dv - 1)) * p.taps;
    fetch(0, sm_chunk);
    int buf = 0;
    for (int c0 = 0; c0 < len; c0 += T, buf ^= 1) {
        const int cnt = min(T, len - c0);
        float* st = sm_chunk + buf * stage;
        asm volatile("cp.async.wait_group 0;\n" ::);
        __syncthreads();
        float *s_q = st, *s_k = st + T * DK, *s_pr = s_k + T * DK, *s_b = s_pr + T * 16, *s_v = s_b + 2 * T;
        if (cnt < T) {                               // the last, short chunk: rows that an earlier chunk left here are cleared
            for (int e = tid; e < (T - cnt) * DK; e += DELTA_NT) s_q[cnt * DK + e] = s_k[cnt * DK + e] = 0.f;
            for (int e = tid; e < (T - cnt) * 16; e += DELTA_NT) s_pr[cnt * 16 + e] = 0.f;
            if (tid < T - cnt) { s_b[2 * (cnt + tid)] = 0.f; s_b[2 * (cnt + tid) + 1] = 1.f; }
            __syncthreads();
        }
        {                                            // thread (i, j) of 64 twice: the chunk's small matrices
            const int e = tid & 63, i = e >> 3, j = e & 7;
            float d = 1.f;
            for (int m = j + 1; m <= i; ++m) d *= s_b[2 * m + 1];
            if (tid < 64) {
                s_kk[e] = j < i ? s_b[2 * i] * d * s_pr[i * 16 + j] : 0.f;
                if (i == T - 1) s_d[j] = d;
            } else {
                s_qk[e] = j <= i ? d * s_pr[i * 16 + 8 + j] : 0.f;
                if (j == 0) s_c[i] = d * s_b[1];
            }
        }
        float va = 0.f, vb = 0.f;                    // this lane's token's values
        for (int j = 0; j < p.taps; ++j) {
            const float2 x = *reinterpret_cast<const float2*>(s_v + (part + j) * NC + cl);
            va += wv0[j] * x.x;
            vb += wv1[j] * x.y;
        }
        va = silu_f(va);
        vb = silu_f(vb);
        float ka[T], kb[T], qa[T], qb[T];
#pragma unroll
        for (int i = 0; i < T; ++i) ka[i] = kb[i] = qa[i] = qb[i] = 0.f;
#pragma unroll
        for (int m = 0; m < IPT / 4; ++m) {
#pragma unroll
            for (int i = 0; i < T; ++i) {
                const float4 k = *(reinterpret_cast<const float4*>(s_k + i * DK + 32 * m) + part);
                ka[i] += k.x * S0[4 * m] + k.y * S0[4 * m + 1] + k.z * S0[4 * m + 2] + k.w * S0[4 * m + 3];
                kb[i] += k.x * S1[4 * m] + k.y * S1[4 * m + 1] + k.z * S1[4 * m + 2] + k.w * S1[4 * m + 3];
                const float4 q = *(reinterpret_cast<const float4*>(s_q + i * DK + 32 * m) + part);
                qa[i] += q.x * S0[4 * m] + q.y * S0[4 * m + 1] + q.z * S0[4 * m + 2] + q.w * S0[4 * m + 3];
                qb[i] += q.x * S1[4 * m] + q.y * S1[4 * m + 1] + q.z * S1[4 * m + 2] + q.w * S1[4 * m + 3];
            }
        }
        const float ksa = reduce8(ka, part), ksb = reduce8(kb, part), qsa = reduce8(qa, part), qsb = reduce8(qb, part);
        __syncthreads();                             // the small matrices are there, and the other stage is free
        if (c0 + T < len) fetch(c0 + T, sm_chunk + (buf ^ 1) * stage);
        const float c = s_c[part], beta = s_b[2 * part];
        const float ra = beta * (va - c * ksa), rb = beta * (vb - c * ksb);
        float ua[T], ub[T];
#pragma unroll
        for (int i = 0; i < T; ++i) {
            ua[i] = __shfl_sync(0xffffffffu, ra, (lane & 24) | i);
            ub[i] = __shfl_sync(0xffffffffu, rb, (lane & 24) | i);
        }
#pragma unroll
        for (int i = 1; i < T; ++i)
#pragma unroll
            for (int j = 0; j < i; ++j) {
                ua[i] -= s_kk[i * T + j] * ua[j];
                ub[i] -= s_kk[i * T + j] * ub[j];
            }
        float oa = c * qsa, ob = c * qsb;
#pragma unroll
        for (int j = 0; j < T; ++j) {
            const float w = s_qk[part * T + j];
            oa += w * ua[j];
            ob += w * ub[j];
        }
        if (part < cnt && live) {
            float* dst = o + ((size_t)(t0 + c0 + part) * p.H + h) * p.dv + col0 + cl;
            if (col0 + cl < p.dv) dst[0] = oa;
            if (col0 + cl + 1 < p.dv) dst[1] = ob;
        }
        const float cT = s_c[T - 1];
#pragma unroll
        for (int j = 0; j < T; ++j) {
            const float w = s_d[j];
            ua[j] *= w;
            ub[j] *= w;
        }
#pragma unroll
        for (int m = 0; m < IPT / 4; ++m) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                S0[4 * m + e] *= cT;
                S1[4 * m + e] *= cT;
            }
#pragma unroll
            for (int j = 0; j < T; ++j) {
                const float4 k = *(reinterpret_cast<const float4*>(s_k + j * DK + 32 * m) + part);
                S0[4 * m] += k.x * ua[j];
                S0[4 * m + 1] += k.y * ua[j];
                S0[4 * m + 2] += k.z * ua[j];
                S0[4 * m + 3] += k.w * ua[j];
                S1[4 * m] += k.x * ub[j];
                S1[4 * m + 1] += k.y * ub[j];
                S1[4 * m + 2] += k.z * ub[j];
                S1[4 * m + 3] += k.w * ub[j];
            }
        }
        __syncthreads();                             // the small matrices and this stage may be written again
    }
    if (live) {
#pragma unroll
        for (int ii = 0; ii < IPT; ++ii) {
            Sg[(size_t)(2 * ii) * stride + gt] = S0[ii];
            Sg[(size_t)(2 * ii + 1) * stride + gt] = S1[ii];
        }
    }
    // the kept inputs move on: this tile's value channels, and with the first tile the head's q and k channels
    // (every read of the old ones, here and in the prep kernel, is done)
    for (int e = tid; e < NC; e += DELTA_NT)
        if (col0 + e < p.dv)
            move_kept(x0 + p.v_off + (size_t)h * p.dv + col0 + e, p.ld, kept + (size_t)(2 * p.dk + col0 + e) * (p.taps - 1), p.taps,
                      len);
    if (tile == 0)
        for (int e = tid; e < 2 * p.dk; e += DELTA_NT) {
            int col, wrow;
            head_channel(p, h, e, col, wrow);
            move_kept(x0 + col, p.ld, kept + (size_t)e * (p.taps - 1), p.taps, len);
        }
}

// ------------------------------------------------------------------ portions: unit norm per head, weight, gate
template <typename TA>
__global__ void __launch_bounds__(256)
delta_out_kernel(const DeltaArgs p, const float* o, TA* out, int n) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t unit = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (unit >= (size_t)n * p.H) return;
    const size_t t = unit / p.H;
    const int h = (int)(unit - t * p.H);
    const float* row = o + unit * p.dv;
    const float* gate = p.rows + t * p.ld + p.g_off + (size_t)h * p.dv;
    float ss = 0.f;
    for (int c = lane; c < p.dv; c += 32) ss += row[c] * row[c];
    const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
    for (int c = lane; c < p.dv; c += 32) {
        float v = row[c] * rs * p.norm_w[c];
        if (p.gate) v *= delta_gate_act(gate[c], p.gate);
        out[unit * p.dv + c] = from_f<TA>(v);
    }
}

// ------------------------------------------------------------------ launchers
static inline int delta_dk(int dk) { return dk <= 32 ? 32 : dk <= 64 ? 64 : dk <= 128 ? 128 : dk <= 256 ? 256 : 512; }
static inline int delta_dvp(int dv) { return (dv + 7) / 8 * 8; }

// Floats of a request's state for H heads of dk x dv behind convolutions of `taps` tokens (no device needed).
RLLM_API long long rllm_delta_state_floats(int H, int dk, int dv, int taps) {
    return (long long)H * delta_dk(dk) * delta_dvp(dv) + (long long)H * (2 * dk + dv) * (taps - 1);
}

template <typename K>
static int raise_smem(K kern, size_t smem, size_t& raised) {
    if (smem <= 48 * 1024 || smem <= raised) return 0;
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess) raised = smem;
    return (int)e;
}

template <typename TA, int DK>
static int launch_delta_step(const DeltaArgs& p, TA* out, cudaStream_t stream) {
    static size_t raised = 0;
    const size_t smem = (size_t)DELTA_TOK * (2 * DK + 2 * p.dvp + 4) * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    const int st = raise_smem(delta_step_kernel<TA, DK>, smem, raised);
    if (st) return st;
    const int threads = p.dvp * 4 > 512 ? 512 : p.dvp * 4;              // a multiple of 32: dvp is a multiple of 8
    return rllm_launch(delta_step_kernel<TA, DK>, dim3(p.H, p.n_requests), dim3(threads), smem, stream, p, out);
}

template <int DK>
static int launch_delta_chunk(const DeltaArgs& p, const float* qn, const float* kn, const float* prods, const float* bg,
                              float* o, cudaStream_t stream) {
    static size_t raised = 0;
    const int W = DELTA_TOK + p.taps - 1;
    const size_t stage = 2 * DELTA_TOK * DK + DELTA_TOK * 16 + 2 * DELTA_TOK + (size_t)(W * DELTA_COLS + 3) / 4 * 4;
    const size_t smem = (2 * stage + 2 * DELTA_TOK * DELTA_TOK + 2 * DELTA_TOK) * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    const int st = raise_smem(delta_chunk_kernel<DK>, smem, raised);
    if (st) return st;
    const int n_tiles = (p.dvp + DELTA_COLS - 1) / DELTA_COLS;
    return rllm_launch(delta_chunk_kernel<DK>, dim3(p.H * n_tiles, p.n_requests), dim3(DELTA_NT), smem, stream, p, qn, kn, prods,
                       bg, o);
}

// portion 0: delta_step, the scratch arrays are not used; 1: prep, chunk, out (qn, kn [n, G * dk], prods [n, G, 16],
// bg [n, H, 2], o [n, H * dv]).
RLLM_API int rllm_gated_delta(const float* rows, long long ld, int q_off, int k_off, int v_off, int g_off, int b_off,
                              int a_off, const float* conv, const float* A, const float* dt_bias, const float* norm_w,
                              float q_scale, float unit_eps, float eps, float* state, long long slot_stride,
                              const int* cu_q, const int* slots, void* out, int act_dt, int n, int n_requests, int H, int G,
                              int dk, int dv, int taps, int gate_kind, int portion, float* qn, float* kn, float* prods,
                              float* bg, float* o, cudaStream_t stream) {
    if (n <= 0 || n_requests <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > 512 || dv <= 0 || taps < 1 || taps > 64 || ld < (long long)q_off + G * dk)
        return (int)cudaErrorInvalidValue;
    const int DK = delta_dk(dk), dvp = delta_dvp(dv);
    const DeltaArgs p = {rows, ld, q_off, k_off, v_off, g_off, b_off, a_off, conv, A, dt_bias, norm_w, q_scale, unit_eps, eps,
                         state, slot_stride, (long long)H * DK * dvp, cu_q, slots, H, G, dk, dv, dvp, taps, gate_kind, n_requests};
#define BY_DK(CALL)                       \
    do {                                  \
        if (DK == 32) return CALL(32);    \
        if (DK == 64) return CALL(64);    \
        if (DK == 128) return CALL(128);  \
        if (DK == 256) return CALL(256);  \
        return CALL(512);                 \
    } while (0)
    if (!portion) {
        if (act_dt == RLLM_F32) {
#define STEP(D) launch_delta_step<float, D>(p, (float*)out, stream)
            BY_DK(STEP);
#undef STEP
        }
#define STEP(D) launch_delta_step<bf16, D>(p, (bf16*)out, stream)
        BY_DK(STEP);
#undef STEP
    }
    if (!qn || !kn || !prods || !bg || !o) return (int)cudaErrorInvalidValue;
    const size_t smem = (size_t)2 * DELTA_TOK * dk * sizeof(float);
    int st = rllm_launch(delta_prep_kernel, dim3(n / DELTA_TOK + n_requests, G), dim3(256), smem, stream, p, qn, kn, prods, bg);
    if (st) return st;
    const auto chunks = [&]() -> int {
#define CHUNK(D) launch_delta_chunk<D>(p, qn, kn, prods, bg, o, stream)
        BY_DK(CHUNK);
#undef CHUNK
    };
    st = chunks();
    if (st) return st;
    const dim3 grid((unsigned)(((size_t)n * H + 7) / 8));
    if (act_dt == RLLM_F32) return rllm_launch(delta_out_kernel<float>, grid, dim3(256), 0, stream, p, (const float*)o, (float*)out, n);
    return rllm_launch(delta_out_kernel<bf16>, grid, dim3(256), 0, stream, p, (const float*)o, (bf16*)out, n);
}
#undef BY_DK

RLLM_PACKED(rllm_gated_delta)
