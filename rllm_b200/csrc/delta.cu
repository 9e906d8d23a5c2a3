// The gated delta rule behind short causal convolutions: a matrix memory per head that is decayed by one
// number per token and corrected towards the token's value along its key.
//
// A token's projection row (float32) holds q, k ([G * dk] each), v ([H * dv]), an output gate ([H * dv]) and two
// numbers per head, b and a.  Head h uses the q/k head h / (H / G).  With conv(.) the causal convolution of
// every channel over `taps` tokens (no bias, the last tap weighs the current token, zeros before the start):
//   q = unit(silu(conv(q))) * q_scale,  k = unit(silu(conv(k))),  v = silu(conv(v)),  unit(x) = x / sqrt(sum x^2 + unit_eps)
//   beta = sigmoid(b),  g = exp(-A * softplus(a + dt_bias))                        (A = exp(A_log), one per head)
//   w_t = beta_t (v_t - g_t M_(t-1)^T k_t),  M_t = g_t M_(t-1) + k_t w_t^T,  o_t = M_t^T q_t         (the code's S is M, its u is w)
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
//                 prep: a block per (chunk, q/k head): convolutions and unit vectors of q and k, and the small
//                 matrices below.  chunk: a block per (tile of value columns, head, request) walks the
//                 request's chunks with its part of S in registers.  With c_i = g_1 .. g_i and d_ij =
//                 g_(j+1) .. g_i (products taken factor by factor, never as a quotient):
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
constexpr int delta_step_threads(int DK) { return DK > 256 ? 256 : 512; }

template <typename TA, int DK>
__global__ void __launch_bounds__(delta_step_threads(DK), DK <= 128 ? 2 : 1)
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
// Chunks are numbered through the step's requests in order; a chunk's rows lie together, eight of them whatever
// the chunk holds, so that the chunk kernel fetches runs of memory.  qk [chunks, G, 2, 8, DK]: the unit vectors of q (times
// q_scale) and k, zeros behind dk.  vals [chunks, H, 8, dvp]: the values behind their convolution.  mats [chunks, H, DELTA_MAT]: -beta_i d_ij (k_i . k_j) at [8 i + j], every entry twice (a pair that
// multiplies two columns at once); d_ij (q_i . k_j) at [128 + 8 i + j] (0 for j > i); beta_i, c_i, d_8i at [192 + i], [200 + i],
// [208 + i].  Tokens behind the last one of a short chunk have k = q = 0, beta = 0 and g = 1.
#define DELTA_MAT 216

// Sixteen values summed over a warp; lane l ends with the sum of value number l / 2.
__device__ __forceinline__ float reduce16(const float (&a)[16], int lane) {
    float b[8], c[4], d[2];
    const bool h4 = lane & 16, h3 = lane & 8, h2 = lane & 4, h1 = lane & 2;
#pragma unroll
    for (int j = 0; j < 8; ++j) b[j] = (h4 ? a[8 + j] : a[j]) + __shfl_xor_sync(0xffffffffu, h4 ? a[j] : a[8 + j], 16);
#pragma unroll
    for (int j = 0; j < 4; ++j) c[j] = (h3 ? b[4 + j] : b[j]) + __shfl_xor_sync(0xffffffffu, h3 ? b[j] : b[4 + j], 8);
#pragma unroll
    for (int j = 0; j < 2; ++j) d[j] = (h2 ? c[2 + j] : c[j]) + __shfl_xor_sync(0xffffffffu, h2 ? c[j] : c[2 + j], 4);
    const float e = (h1 ? d[1] : d[0]) + __shfl_xor_sync(0xffffffffu, h1 ? d[0] : d[1], 2);
    return e + __shfl_xor_sync(0xffffffffu, e, 1);
}

// A channel's eight tokens behind its convolution (zeros behind the request's end): put(token, value).
template <typename F>
__device__ __forceinline__ void conv_chunk(const float* x, long long ld, const float* kept, const float* __restrict__ w,
                                           int taps, int c0, int len, F put) {
    if (taps == 4) {
        float v[DELTA_TOK + 3];
#pragma unroll
        for (int j = 0; j < DELTA_TOK + 3; ++j) {
            const int s = c0 + j - 3;
            v[j] = s >= len ? 0.f : s >= 0 ? x[(size_t)s * ld] : kept[3 + s];
        }
        const float w0 = w[0], w1 = w[1], w2 = w[2], w3 = w[3];
#pragma unroll
        for (int i = 0; i < DELTA_TOK; ++i)
            put(i, c0 + i < len ? silu_f(w0 * v[i] + w1 * v[i + 1] + w2 * v[i + 2] + w3 * v[i + 3]) : 0.f);
    } else {
        for (int i = 0; i < DELTA_TOK; ++i) put(i, c0 + i < len ? conv_at(x, ld, kept, w, taps, c0 + i) : 0.f);
    }
}

__global__ void __launch_bounds__(256)
delta_prep_kernel(const DeltaArgs p, float* qk, float* vals, float* mats, int DK) {
    extern __shared__ __align__(16) float sm_prep[];
    float* s_q = sm_prep;                            // [TOK][DK]
    float* s_k = s_q + DELTA_TOK * DK;
    float* s_bg = s_k + DELTA_TOK * DK;              // [rep][2][TOK]: beta, g
    __shared__ float s_pr[DELTA_TOK][2 * DELTA_TOK]; // k_i . k_j, q_i . k_j
    // (no early launch of what follows: the chunk kernel's few, long-lived blocks are to spread over idle SMs)
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
    for (int e = tid; e < DELTA_TOK * rep; e += blockDim.x) {
        const int i = e & 7, hh = e >> 3, h = kh * rep + hh;
        float beta = 0.f, g = 1.f;
        if (i < cnt) {
            const float* row = x0 + (size_t)(c0 + i) * p.ld;
            beta = 1.0f / (1.0f + expf(-row[p.b_off + h]));
            g = head_decay(p, h, row[p.a_off + h]);
        }
        s_bg[hh * 2 * DELTA_TOK + i] = beta;
        s_bg[hh * 2 * DELTA_TOK + DELTA_TOK + i] = g;
    }
    for (int e = tid; e < 2 * DK; e += blockDim.x) {         // a thread takes a channel's tokens
        const bool is_k = e >= DK;
        const int cc = is_k ? e - DK : e;
        float* dst = (is_k ? s_k : s_q) + cc;
        if (cc < p.dk) {
            conv_chunk(x0 + (is_k ? p.k_off : p.q_off) + kh * p.dk + cc, p.ld, kept + (size_t)(is_k * p.dk + cc) * (p.taps - 1),
                       p.conv + (size_t)((is_k ? p.G * p.dk : 0) + kh * p.dk + cc) * p.taps, p.taps, c0, len,
                       [&](int i, float v) { dst[i * DK] = v; });
        } else {
            for (int i = 0; i < DELTA_TOK; ++i) dst[i * DK] = 0.f;
        }
    }
    for (int e = tid; e < rep * p.dvp; e += blockDim.x) {
        const int hh = e / p.dvp, c = e - hh * p.dvp, h = kh * rep + hh;
        float* dst = vals + ((size_t)blockIdx.x * p.H + h) * DELTA_TOK * p.dvp + c;
        if (c < p.dv) {
            conv_chunk(x0 + p.v_off + (size_t)h * p.dv + c, p.ld, kept + (size_t)(hh * C + 2 * p.dk + c) * (p.taps - 1),
                       p.conv + (size_t)(2 * p.G * p.dk + h * p.dv + c) * p.taps, p.taps, c0, len,
                       [&](int i, float v) { dst[(size_t)i * p.dvp] = v; });
        } else {
            for (int i = 0; i < DELTA_TOK; ++i) dst[(size_t)i * p.dvp] = 0.f;
        }
    }
    __syncthreads();
    {                                                // warp i: token i's lengths
        const int i = warp;
        float qq = 0.f, kk = 0.f;
        for (int c = lane; c < DK; c += 32) {
            qq += s_q[i * DK + c] * s_q[i * DK + c];
            kk += s_k[i * DK + c] * s_k[i * DK + c];
        }
        const float rq = p.q_scale / sqrtf(warp_sum(qq) + p.unit_eps), rk = 1.0f / sqrtf(warp_sum(kk) + p.unit_eps);
        float* row = qk + (((size_t)blockIdx.x * p.G + kh) * 2 * DELTA_TOK + i) * DK;
        for (int c = lane; c < DK; c += 32) {
            const float a = s_q[i * DK + c] * rq, b = s_k[i * DK + c] * rk;
            s_q[i * DK + c] = row[c] = a;
            s_k[i * DK + c] = row[(size_t)DELTA_TOK * DK + c] = b;
        }
    }
    __syncthreads();
    {                                                // and its products with the keys up to it
        const int i = warp;
        float pr[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) pr[j] = 0.f;
        for (int c = lane; c < DK; c += 32) {
            const float a = s_q[i * DK + c], b = s_k[i * DK + c];
#pragma unroll
            for (int j = 0; j < DELTA_TOK; ++j) {
                const float o = j <= i ? s_k[j * DK + c] : 0.f;
                pr[j] += b * o;
                pr[DELTA_TOK + j] += a * o;
            }
        }
        const float v = reduce16(pr, lane);
        if (!(lane & 1)) s_pr[i][lane >> 1] = v;
    }
    __syncthreads();
    for (int e = tid; e < rep * 64; e += blockDim.x) {
        const int hh = e >> 6, i = (e >> 3) & 7, j = e & 7;
        const float *beta = s_bg + hh * 2 * DELTA_TOK, *g = beta + DELTA_TOK;
        float d = 1.f;
#pragma unroll
        for (int m = 1; m < DELTA_TOK; ++m) d *= (m > j && m <= i) ? g[m] : 1.f;
        float* dst = mats + ((size_t)blockIdx.x * p.H + kh * rep + hh) * DELTA_MAT;
        const float kk = j < i ? -beta[i] * d * s_pr[i][j] : 0.f;
        *reinterpret_cast<float2*>(dst + 2 * (8 * i + j)) = make_float2(kk, kk);
        dst[128 + 8 * i + j] = j <= i ? d * s_pr[i][DELTA_TOK + j] : 0.f;
        if (j == 0) {
            dst[192 + i] = beta[i];
            dst[200 + i] = d * g[0];
        }
        if (i == DELTA_TOK - 1) dst[208 + j] = d;
    }
}

// ------------------------------------------------------------------ portions: the walk through the chunks
__device__ __forceinline__ void delta_cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void delta_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
// Pairs of floats in one 64-bit register: two multiply-adds an instruction (each rounded as a single one is).
typedef unsigned long long f2;
__device__ __forceinline__ f2 f2_make(float a, float b) {
    f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void f2_split(f2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f2 f2_fma(f2 a, f2 b, f2 c) {
    f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f2 f2_mul(f2 a, f2 b) {
    f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
// Keeps the compiler from requesting the operands of later work here: they would not fit the registers.
__device__ __forceinline__ void hold_loads() { asm volatile("" ::: "memory"); }
__device__ __forceinline__ float f2_sum(f2 v) {
    float a, b;
    f2_split(v, a, b);
    return a + b;
}
// Sums of eight values over the eight lanes of a group; lane `part` ends with the sum of value number `part`.
__device__ __forceinline__ float reduce8(const f2 (&v)[DELTA_TOK], int part) {
    float a[8], b[4], c[2];
    const bool h4 = part & 4, h2 = part & 2, h1 = part & 1;
#pragma unroll
    for (int j = 0; j < 8; ++j) a[j] = f2_sum(v[j]);
#pragma unroll
    for (int j = 0; j < 4; ++j) b[j] = (h4 ? a[4 + j] : a[j]) + __shfl_xor_sync(0xffffffffu, h4 ? a[j] : a[4 + j], 4);
#pragma unroll
    for (int j = 0; j < 2; ++j) c[j] = (h2 ? b[2 + j] : b[j]) + __shfl_xor_sync(0xffffffffu, h2 ? b[j] : b[2 + j], 2);
    return (h1 ? c[1] : c[0]) + __shfl_xor_sync(0xffffffffu, h1 ? c[0] : c[1], 1);
}

// A block of NT threads takes NT / 4 value columns.
template <int DK, int NT>
__global__ void __launch_bounds__(NT)
delta_chunk_kernel(const DeltaArgs p, const float* qk, const float* vals, const float* mats, float* o) {
    constexpr int IPT = DK / DELTA_PARTS, T = DELTA_TOK, NC = 2 * NT / DELTA_PARTS;
    constexpr int QK4 = 2 * T * DK / 4, MAT4 = DELTA_MAT / 4, V4 = T * NC / 4, stage = 4 * (QK4 + MAT4 + V4);
    extern __shared__ __align__(16) float sm_chunk[];
    const int tid = threadIdx.x, part = tid & 7, lane = tid & 31;
    const int n_tiles = (p.dvp + NC - 1) / NC, h = blockIdx.x / n_tiles, tile = blockIdx.x % n_tiles, r = blockIdx.y;
    const int kh = h / (p.H / p.G), C = 2 * p.dk + p.dv;
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = p.cu_q[r], len = p.cu_q[r + 1] - t0;
    if (len <= 0) return;
    int chunk0 = 0;                                  // the number of the request's first chunk
    for (int i = 0; i < r; ++i) chunk0 += (p.cu_q[i + 1] - p.cu_q[i] + T - 1) / T;
    float* slot = p.state + (size_t)p.slots[r] * p.slot_stride;
    float* Sg = slot + (size_t)h * DK * p.dvp;
    float* kept = slot + p.conv_base + (size_t)h * C * (p.taps - 1);
    const float* x0 = p.rows + (size_t)t0 * p.ld;
    const int col0 = tile * NC, pair = col0 / 2 + tid / DELTA_PARTS, gt = pair * DELTA_PARTS + part, cl = 2 * (tid / DELTA_PARTS);
    const bool live = 2 * pair < p.dvp;
    const size_t stride = (size_t)p.dvp * 4;
    f2 S0[IPT / 2], S1[IPT / 2];                     // rows ii, ii + 1 of the pair's two columns
#pragma unroll
    for (int m = 0; m < IPT / 2; ++m) {
        const float* at = Sg + (size_t)(4 * m) * stride + gt;
        S0[m] = live ? f2_make(at[0], at[2 * stride]) : 0ull;
        S1[m] = live ? f2_make(at[stride], at[3 * stride]) : 0ull;
    }
    // a chunk's q and k, small matrices and values of this tile's columns: runs of 16 bytes
    const float* qk_src = qk + ((size_t)chunk0 * p.G + kh) * 2 * T * DK + 4 * tid;
    const float* mat_src = mats + ((size_t)chunk0 * p.H + h) * DELTA_MAT + 4 * tid;
    const float* v_src = vals + ((size_t)chunk0 * p.H + h) * T * p.dvp + col0;
    auto fetch = [&](float* st) {
#pragma unroll
        for (int e = 0; e < QK4; e += NT) delta_cp16(st + 4 * (e + tid), qk_src + 4 * e);
#pragma unroll
        for (int e = 0; e < MAT4; e += NT)
            if (e + tid < MAT4) delta_cp16(st + 4 * (QK4 + e + tid), mat_src + 4 * e);
#pragma unroll
        for (int e = tid; e < V4; e += NT) {
            const int i = e / (NC / 4), c = 4 * (e % (NC / 4));
            if (col0 + c < p.dvp) delta_cp16(st + 4 * (QK4 + MAT4 + e), v_src + (size_t)i * p.dvp + c);
        }
        asm volatile("cp.async.commit_group;\n" ::);
        qk_src += (size_t)p.G * 2 * T * DK;
        mat_src += (size_t)p.H * DELTA_MAT;
        v_src += (size_t)p.H * T * p.dvp;
    };
    float* dst = o + ((size_t)(t0 + part) * p.H + h) * p.dv + col0 + cl;
    const bool st_a = col0 + cl < p.dv, st_b = col0 + cl + 1 < p.dv;
    fetch(sm_chunk);
    int buf = 0;
    for (int c0 = 0; c0 < len; c0 += T, buf ^= 1) {
        const int cnt = min(T, len - c0);
        float* st = sm_chunk + buf * stage;
        asm volatile("cp.async.wait_group 0;\n" ::);
        __syncthreads();                             // this chunk is there, and everybody is done with the other stage
        if (c0 + T < len) fetch(sm_chunk + (buf ^ 1) * stage);
        float *s_q = st, *s_k = st + T * DK, *s_m = s_k + T * DK, *s_v = s_m + DELTA_MAT;
        f2 ka[T], kb[T], qa[T], qb[T];
#pragma unroll
        for (int i = 0; i < T; ++i) ka[i] = kb[i] = qa[i] = qb[i] = 0ull;
        // four tokens at a time: their operands first, then sixteen independent multiply-adds, then the other halves
#pragma unroll
        for (int m = 0; m < IPT / 4; ++m) {
#pragma unroll
            for (int i0 = 0; i0 < T; i0 += 4) {
                ulonglong2 k[4], q[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    k[i] = *(reinterpret_cast<const ulonglong2*>(s_k + (i0 + i) * DK + 32 * m) + part);
                    q[i] = *(reinterpret_cast<const ulonglong2*>(s_q + (i0 + i) * DK + 32 * m) + part);
                }
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    ka[i0 + i] = f2_fma(k[i].x, S0[2 * m], ka[i0 + i]);
                    kb[i0 + i] = f2_fma(k[i].x, S1[2 * m], kb[i0 + i]);
                    qa[i0 + i] = f2_fma(q[i].x, S0[2 * m], qa[i0 + i]);
                    qb[i0 + i] = f2_fma(q[i].x, S1[2 * m], qb[i0 + i]);
                }
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    ka[i0 + i] = f2_fma(k[i].y, S0[2 * m + 1], ka[i0 + i]);
                    kb[i0 + i] = f2_fma(k[i].y, S1[2 * m + 1], kb[i0 + i]);
                    qa[i0 + i] = f2_fma(q[i].y, S0[2 * m + 1], qa[i0 + i]);
                    qb[i0 + i] = f2_fma(q[i].y, S1[2 * m + 1], qb[i0 + i]);
                }
            }
        }
        const float2 v = *reinterpret_cast<const float2*>(s_v + part * NC + cl);      // this lane's token's values
        const float ksa = reduce8(ka, part), ksb = reduce8(kb, part), qsa = reduce8(qa, part), qsb = reduce8(qb, part);
        const float beta = s_m[192 + part], c = s_m[200 + part];
        const float ra = beta * (v.x - c * ksa), rb = beta * (v.y - c * ksb);
        f2 u[T];                                     // the tokens' corrections of the two columns
#pragma unroll
        for (int i = 0; i < T; ++i)
            u[i] = f2_make(__shfl_sync(0xffffffffu, ra, (lane & 24) | i), __shfl_sync(0xffffffffu, rb, (lane & 24) | i));
        const f2* kk = reinterpret_cast<const f2*>(s_m);
#pragma unroll
        for (int j = 0; j < T - 1; ++j)
#pragma unroll
            for (int i = j + 1; i < T; ++i) u[i] = f2_fma(kk[i * T + j], u[j], u[i]);
        float oa = c * qsa, ob = c * qsb;
#pragma unroll
        for (int j = 0; j < T; ++j) {
            const float w = s_m[128 + part * T + j];
            float a, b;
            f2_split(u[j], a, b);
            oa += w * a;
            ob += w * b;
        }
        if (part < cnt) {
            if (st_a) dst[0] = oa;
            if (st_b) dst[1] = ob;
        }
        dst += (size_t)T * p.H * p.dv;
        const f2 cT = f2_make(s_m[200 + T - 1], s_m[200 + T - 1]);
        f2 ua[T], ub[T];
#pragma unroll
        for (int j = 0; j < T; ++j) {
            const float w = s_m[208 + j];
            float a, b;
            f2_split(u[j], a, b);
            ua[j] = f2_make(a * w, a * w);
            ub[j] = f2_make(b * w, b * w);
        }
        hold_loads();
#pragma unroll
        for (int m = 0; m < IPT / 2; ++m) {
            S0[m] = f2_mul(S0[m], cT);
            S1[m] = f2_mul(S1[m], cT);
        }
#pragma unroll
        for (int j = 0; j < T; ++j)
#pragma unroll
            for (int m = 0; m < IPT / 4; ++m) {
                const ulonglong2 k = *(reinterpret_cast<const ulonglong2*>(s_k + j * DK + 32 * m) + part);
                S0[2 * m] = f2_fma(k.x, ua[j], S0[2 * m]);
                S1[2 * m] = f2_fma(k.x, ub[j], S1[2 * m]);
                S0[2 * m + 1] = f2_fma(k.y, ua[j], S0[2 * m + 1]);
                S1[2 * m + 1] = f2_fma(k.y, ub[j], S1[2 * m + 1]);
            }
    }
    if (live) {
#pragma unroll
        for (int m = 0; m < IPT / 2; ++m) {
            float* at = Sg + (size_t)(4 * m) * stride + gt;
            f2_split(S0[m], at[0], at[2 * stride]);
            f2_split(S1[m], at[stride], at[3 * stride]);
        }
    }
    // the kept inputs move on: this tile's value channels, and with the first tile the head's q and k channels
    // (every read of the old ones, here and in the prep kernel, is done)
    for (int e = tid; e < NC; e += NT)
        if (col0 + e < p.dv)
            move_kept(x0 + p.v_off + (size_t)h * p.dv + col0 + e, p.ld, kept + (size_t)(2 * p.dk + col0 + e) * (p.taps - 1), p.taps, len);
    if (tile == 0)
        for (int e = tid; e < 2 * p.dk; e += NT) {
            int col, wrow;
            head_channel(p, h, e, col, wrow);
            move_kept(x0 + col, p.ld, kept + (size_t)e * (p.taps - 1), p.taps, len);
        }
}

// ------------------------------------------------------------------ portions: unit norm per head, weight, gate
template <typename TA>
__global__ void __launch_bounds__(256)
delta_out_kernel(const DeltaArgs p, const float* o, TA* out, int n, int vec) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t unit = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (unit >= (size_t)n * p.H) return;
    const size_t t = unit / p.H;
    const int h = (int)(unit - t * p.H);
    const float* row = o + unit * p.dv;
    const float* gate = p.rows + t * p.ld + p.g_off + (size_t)h * p.dv;
    if (vec) {                                       // one group of four columns a lane
        const int c = 4 * lane;
        const bool in = c < p.dv;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        float4 v = in ? *reinterpret_cast<const float4*>(row + c) : zero;
        const float4 g = in && p.gate ? *reinterpret_cast<const float4*>(gate + c) : zero;
        const float rs = 1.0f / sqrtf(warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w) / (float)p.dv + p.eps);
        if (!in) return;
        const float4 w = *reinterpret_cast<const float4*>(p.norm_w + c);
        v.x *= rs * w.x * delta_gate_act(g.x, p.gate);
        v.y *= rs * w.y * delta_gate_act(g.y, p.gate);
        v.z *= rs * w.z * delta_gate_act(g.z, p.gate);
        v.w *= rs * w.w * delta_gate_act(g.w, p.gate);
        TA* dst = out + unit * p.dv + c;
        if constexpr (sizeof(TA) == 4) {
            *reinterpret_cast<float4*>(dst) = v;
        } else {
            __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
            uint2 q;
            q.x = *reinterpret_cast<uint32_t*>(&a);
            q.y = *reinterpret_cast<uint32_t*>(&b);
            *reinterpret_cast<uint2*>(dst) = q;
        }
        return;
    }
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
    const int most = delta_step_threads(DK), threads = p.dvp * 4 > most ? most : p.dvp * 4;      // a multiple of 32
    return rllm_launch(delta_step_kernel<TA, DK>, dim3(p.H, p.n_requests), dim3(threads), smem, stream, p, out);
}

template <int DK>
static int launch_delta_chunk(const DeltaArgs& p, const float* qk, const float* vals, const float* mats, float* o,
                              cudaStream_t stream) {
    constexpr int NT = 64, NC = 2 * NT / DELTA_PARTS;           // measured: 64 threads ahead of 32 and 128 at every size
    static size_t raised = 0;
    const size_t smem = 2 * (2 * DELTA_TOK * DK + DELTA_MAT + DELTA_TOK * NC) * sizeof(float);
    const int st = raise_smem(delta_chunk_kernel<DK, NT>, smem, raised);
    if (st) return st;
    const int n_tiles = (p.dvp + NC - 1) / NC;
    return rllm_launch(delta_chunk_kernel<DK, NT>, dim3(p.H * n_tiles, p.n_requests), dim3(NT), smem, stream, p, qk, vals, mats, o);
}

// portion 0: delta_step, the scratch arrays are not used; 1: prep, chunk, out, with n / 8 + n_requests chunks in qk, vals
// and mats (see the prep kernel) and o [n, H * dv]; all 16-byte aligned.
RLLM_API int rllm_gated_delta(const float* rows, long long ld, int q_off, int k_off, int v_off, int g_off, int b_off,
                              int a_off, const float* conv, const float* A, const float* dt_bias, const float* norm_w,
                              float q_scale, float unit_eps, float eps, float* state, long long slot_stride,
                              const int* cu_q, const int* slots, void* out, int act_dt, int n, int n_requests, int H, int G,
                              int dk, int dv, int taps, int gate_kind, int portion, float* qk, float* vals, float* mats,
                              float* o, cudaStream_t stream) {
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
    if (!qk || !vals || !mats || !o) return (int)cudaErrorInvalidValue;
    static size_t raised = 0;
    const size_t smem = (size_t)DELTA_TOK * (2 * DK + 2 * (H / G)) * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    int st = raise_smem(delta_prep_kernel, smem, raised);
    if (st) return st;
    st = rllm_launch(delta_prep_kernel, dim3(n / DELTA_TOK + n_requests, G), dim3(256), smem, stream, p, qk, vals, mats, DK);
    if (st) return st;
    const auto chunks = [&]() -> int {
#define CHUNK(D) launch_delta_chunk<D>(p, qk, vals, mats, o, stream)
        BY_DK(CHUNK);
#undef CHUNK
    };
    st = chunks();
    if (st) return st;
    const dim3 grid((unsigned)(((size_t)n * H + 7) / 8));
    const int vec = dv <= 128 && (dv & 3) == 0 && (ld & 3) == 0 && (g_off & 3) == 0 && ((uintptr_t)rows & 15) == 0 &&
                    ((uintptr_t)out & 15) == 0 && ((uintptr_t)norm_w & 15) == 0 && ((uintptr_t)o & 15) == 0;
    if (act_dt == RLLM_F32) return rllm_launch(delta_out_kernel<float>, grid, dim3(256), 0, stream, p, (const float*)o, (float*)out, n, vec);
    return rllm_launch(delta_out_kernel<bf16>, grid, dim3(256), 0, stream, p, (const float*)o, (bf16*)out, n, vec);
}
#undef BY_DK

RLLM_PACKED(rllm_gated_delta)
