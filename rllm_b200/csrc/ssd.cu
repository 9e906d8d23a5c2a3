// State spaces with one decay per head (the recurrence of Mamba-2) behind a short causal convolution.
//
// A token's projection row (float32) holds z [H * P], then x [H * P], B [G * N], C [G * N] side by side (the
// convolution's channels), and one number dt per head.  Head h uses B and C of group h / (H / G).  With conv(.) the
// causal convolution of every channel over `taps` tokens plus a bias (the last tap weighs the current token, zeros
// before the start):
//   x, B, C = silu(conv(x, B, C));  d_t = softplus(dt + dt_bias);  a_t = exp(-A d_t)         (A = exp(A_log), one per head)
//   S_t = a_t S_(t-1) + d_t x_t B_t^T  (S is P x N);  y_t = S_t C_t + D x_t
//   out = rms_parts(y * silu(z)) * norm_w      (every one of `parts` equal runs of columns by its own root mean square)
// Everything but the storage of x, B, C and y is float32 (the activation type holds those in bfloat16 mode).
//
// State slot of a request (floats): S of every head, [H][P][N], then a ring of the last inputs of the convolution:
// the input of channel c at position p lies at ring[(p % R) * channels + c], R = taps - 1 + SSD_STEP.  A step of at most
// SSD_STEP tokens never writes a ring entry that it reads, so blocks need no order among themselves.
//
//   ssd_conv    (prompt portions) the convolution of all channels and the step sizes of all heads, a thread walking
//               along the tokens with its channels' window in registers.  x, B and C rows are padded to a multiple of 8
//               entries per head and group.
//   ssd_step    token by token, a block per (head, request), rows of S spread over groups of lanes: steps of few tokens
//               (then with the convolution and the step sizes in the same kernel), float32 portions, and sizes that
//               the kernel below does not take.
//   ssd_chunk   bfloat16 portions on the tensor cores, in chunks of 64 tokens counted from the portion's start: a block
//               per (head, 16 to 64 rows of S, request) walks the request's chunks with S^T in the accumulators of
//               mma.sync (two warps, the halves of N, per 16 rows).  Long portions are also cut along time: pass 1 works
//               out what every segment's tokens leave, pass 2 the outputs from the states that follow, all segments side
//               by side.  With L_i = log(a_1 .. a_i) of a chunk:
//                   y_i = e^(L_i) S0 C_i + sum_(j<=i) (C_i . B_j) e^(L_i - L_j) d_j x_j
//                   S   = e^(L_64) S0 + sum_j e^(L_64 - L_j) d_j x_j B_j^T
//               x, B and C are bfloat16 as stored; every other operand (S0, the weighted scores, the weighted x) goes into
//               its product as the sum of two bfloat16 numbers (16 bits of mantissa), with float32 accumulation.
//   ssd_norm    the norm of the gated rows, in place.
#include "common.cuh"
#include "recurrent.cuh"

#define SSD_STEP 8             // tokens of a request that ssd_step takes at a time
#define SSD_CHUNK 64           // tokens of a chunk

struct SsdArgs {
    const float* rows;         // [n, ld]
    long long ld;
    int z_off, c_off, dt_off;  // columns of z, of the convolution's channels, of dt
    const float* conv;         // [taps][channels]
    const float* conv_b;       // [channels]
    const float* dt_bias;      // [H]
    const float* A;            // [H] exp(A_log)
    const float* D;            // [H]
    float* state;
    long long slot_stride, ring_base;
    const int* positions;
    const int* seq_ids;
    const int* cu_q;
    const int* slots;
    int H, G, P, N, taps;
};

__device__ __forceinline__ int ssd_channels(const SsdArgs& p) { return p.H * p.P + 2 * p.G * p.N; }
__device__ __forceinline__ int ssd_ring(const SsdArgs& p) { return p.taps - 1 + SSD_STEP; }
__host__ __device__ __forceinline__ int ssd_pad8(int n) { return (n + 7) / 8 * 8; }

// The ring entries of the request's last tokens, for the channels c0 .. c0 + count - 1.
__device__ __forceinline__ void ssd_keep(const SsdArgs& p, float* ring, int t0, int len, int c0, int count, int tid, int nt) {
    const int m = min(len, p.taps - 1), C = ssd_channels(p), R = ssd_ring(p);
    for (int e = tid; e < m * count; e += nt) {
        const int i = len - m + e / count, c = c0 + e % count;
        ring[(size_t)(p.positions[t0 + i] % R) * C + c] = p.rows[(size_t)(t0 + i) * p.ld + p.c_off + c];
    }
}

// ------------------------------------------------------------------ portions: convolution and step sizes
#define SSD_CONV_TOK 16        // tokens in a row per thread

template <int VEC> struct SsdVec { float v[VEC]; };
template <int VEC> __device__ __forceinline__ SsdVec<VEC> ssd_load(const float* p) {
    SsdVec<VEC> r;
    if constexpr (VEC == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int VEC> __device__ __forceinline__ void ssd_put(float* o, const SsdVec<VEC>& r) {
#pragma unroll
    for (int q = 0; q < VEC; ++q) o[q] = r.v[q];
}
template <int VEC> __device__ __forceinline__ void ssd_put(bf16* o, const SsdVec<VEC>& r) {
    if constexpr (VEC == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 u;
        u.x = *reinterpret_cast<const uint32_t*>(&a);
        u.y = *reinterpret_cast<const uint32_t*>(&b);
        *reinterpret_cast<uint2*>(o) = u;
    } else {
        o[0] = __float2bfloat16_rn(r.v[0]);
    }
}

// TAPS 0: any number of taps (every input read again for every token); else that many, the window in registers.
template <typename TA, int VEC, int TAPS>
__global__ void __launch_bounds__(256)
ssd_conv_kernel(const SsdArgs p, TA* xbc, long long ldx, float* dts, int n) {
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = blockIdx.x * SSD_CONV_TOK, t1 = min(n, t0 + SSD_CONV_TOK), C = ssd_channels(p), R = ssd_ring(p);
    if (blockIdx.y == gridDim.y - 1) {                        // step sizes: dts[0] = d, dts[1] = log a, [H][n] each
        for (int e = threadIdx.x; e < (t1 - t0) * p.H; e += blockDim.x) {
            const int t = t0 + e / p.H, h = e % p.H;
            const float d = softplus_f(p.rows[(size_t)t * p.ld + p.dt_off + h] + p.dt_bias[h]);
            dts[(size_t)h * n + t] = d;
            dts[(size_t)(p.H + h) * n + t] = -p.A[h] * d;
        }
        return;
    }
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    if (c >= C) return;
    const int inner = p.H * p.P, gn = p.G * p.N, P8 = ssd_pad8(p.P), N8 = ssd_pad8(p.N);
    int col;                                                  // the channel's place in the padded row
    if (c < inner) col = c / p.P * P8 + c % p.P;
    else if (c < inner + gn) col = p.H * P8 + (c - inner) / p.N * N8 + (c - inner) % p.N;
    else col = p.H * P8 + p.G * N8 + (c - inner - gn) / p.N * N8 + (c - inner - gn) % p.N;
    const float* src = p.rows + p.c_off + c;
    const SsdVec<VEC> bias = ssd_load<VEC>(p.conv_b + c);
    auto input = [&](const float* ring, int t, int i, int pos, int back) {
        SsdVec<VEC> r;
        if (back <= i) return ssd_load<VEC>(src + (size_t)(t - back) * p.ld);
        if (back <= pos) return ssd_load<VEC>(ring + (size_t)((pos - back) % R) * C + c);
#pragma unroll
        for (int q = 0; q < VEC; ++q) r.v[q] = 0.f;
        return r;
    };
    if constexpr (TAPS > 0) {
        SsdVec<VEC> w[TAPS], win[TAPS];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = ssd_load<VEC>(p.conv + (size_t)j * C + c);
        int req = -1;
        auto open_window = [&](int t, int r) {                // a request's first token here: its window from the row or the ring
            const int i = t - p.cu_q[r], pos = p.positions[t];
            const float* ring = p.state + (size_t)p.slots[r] * p.slot_stride + p.ring_base;
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) win[j + 1] = input(ring, t, i, pos, TAPS - 1 - j);
            req = r;
        };
        auto token = [&](int t, const SsdVec<VEC>& x) {
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) win[j] = win[j + 1];
            win[TAPS - 1] = x;
            SsdVec<VEC> acc = bias;
#pragma unroll
            for (int j = 0; j < TAPS; ++j)
#pragma unroll
                for (int q = 0; q < VEC; ++q) acc.v[q] += w[j].v[q] * win[j].v[q];
#pragma unroll
            for (int q = 0; q < VEC; ++q) acc.v[q] = silu_f(acc.v[q]);
            ssd_put<VEC>(xbc + (size_t)t * ldx + col, acc);
        };
        if (t1 - t0 == SSD_CONV_TOK && p.seq_ids[t0] == p.seq_ids[t1 - 1]) {      // one request: the inputs of eight tokens in flight
            open_window(t0, p.seq_ids[t0]);
            for (int t = t0; t < t1; t += 8) {
                SsdVec<VEC> x[8];
#pragma unroll
                for (int u = 0; u < 8; ++u) x[u] = ssd_load<VEC>(src + (size_t)(t + u) * p.ld);
#pragma unroll
                for (int u = 0; u < 8; ++u) token(t + u, x[u]);
            }
            return;
        }
        for (int t = t0; t < t1; ++t) {
            const int r = p.seq_ids[t];
            if (r != req) open_window(t, r);
            token(t, ssd_load<VEC>(src + (size_t)t * p.ld));
        }
    } else {
        for (int t = t0; t < t1; ++t) {
            const int r = p.seq_ids[t], i = t - p.cu_q[r], pos = p.positions[t];
            const float* ring = p.state + (size_t)p.slots[r] * p.slot_stride + p.ring_base;
            SsdVec<VEC> acc = bias;
            for (int j = 0; j < p.taps; ++j) {
                const SsdVec<VEC> v = input(ring, t, i, pos, p.taps - 1 - j), w = ssd_load<VEC>(p.conv + (size_t)j * C + c);
#pragma unroll
                for (int q = 0; q < VEC; ++q) acc.v[q] += w.v[q] * v.v[q];
            }
#pragma unroll
            for (int q = 0; q < VEC; ++q) acc.v[q] = silu_f(acc.v[q]);
            ssd_put<VEC>(xbc + (size_t)t * ldx + col, acc);
        }
    }
}

// ------------------------------------------------------------------ token by token
// LN lanes share a row of S (KV runs of VEC entries a lane); RU rows a lane group at a time.  FUSED: the step has at
// most SSD_STEP tokens a request and the kernel does the convolution and the step sizes itself; else xbc and dts.
template <typename TA, int VEC, int KV, bool FUSED>
__global__ void __launch_bounds__(256, 3)
ssd_step_kernel(const SsdArgs p, const TA* xbc, long long ldx, const float* dts, int n, TA* out, long long ldo, int LN) {
    constexpr int RU = 8 / KV;
    extern __shared__ __align__(16) float sm_ssd[];
    const int N4 = (p.N + 3) / 4 * 4, tid = threadIdx.x;
    float* s_b = sm_ssd;                             // [STEP][N4]
    float* s_c = s_b + SSD_STEP * N4;
    float* s_x = s_c + SSD_STEP * N4;                // [STEP][P]
    float* s_y = s_x + SSD_STEP * p.P;
    float* s_d = s_y + SSD_STEP * p.P;               // [STEP] step size, [STEP] decay
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, r = blockIdx.y, g = h / (p.H / p.G);
    const int t0 = p.cu_q[r], len = p.cu_q[r + 1] - t0;
    float* slot = p.state + (size_t)p.slots[r] * p.slot_stride;
    float* Sg = slot + (size_t)h * p.P * p.N;
    float* ring = slot + p.ring_base;
    const int inner = p.H * p.P, gn = p.G * p.N, P8 = ssd_pad8(p.P), N8 = ssd_pad8(p.N);
    const int ln = tid % LN, grp = tid / LN, groups = blockDim.x / LN;
    float S[RU][KV][VEC];
    auto load = [&](int p0) {
#pragma unroll
        for (int u = 0; u < RU; ++u) {
            const int row = p0 + u * groups;
#pragma unroll
            for (int k = 0; k < KV; ++k) {
                const int c = (ln + LN * k) * VEC;
                if (row < p.P && c < p.N) {
                    const SsdVec<VEC> f = ssd_load<VEC>(Sg + (size_t)row * p.N + c);
#pragma unroll
                    for (int q = 0; q < VEC; ++q) S[u][k][q] = f.v[q];
                } else {
#pragma unroll
                    for (int q = 0; q < VEC; ++q) S[u][k][q] = 0.f;
                }
            }
        }
    };
    for (int c0 = 0; c0 < len; c0 += SSD_STEP) {
        const int cnt = min(SSD_STEP, len - c0);
        load(grp);                                   // on its way while the convolutions run
        const int per = p.P + 2 * p.N;
        float z_first = 0.f;                         // the gate of the thread's first output, on its way
        if (tid < cnt * p.P) z_first = p.rows[(size_t)(t0 + c0 + tid / p.P) * p.ld + p.z_off + (size_t)h * p.P + tid % p.P];
        for (int e = tid; e < cnt * per; e += blockDim.x) {
            const int i = e / per, c = e - i * per, t = t0 + c0 + i;
            float v;
            if constexpr (FUSED) {
                const int ch = c < p.P ? h * p.P + c : c < p.P + p.N ? inner + g * p.N + c - p.P : inner + gn + g * p.N + c - p.P - p.N;
                const int C = ssd_channels(p), pos = p.positions[t];
                float acc = p.conv_b[ch];
                for (int j0 = 0; j0 < p.taps; j0 += 4) {          // four inputs and their weights in flight
                    float in[4], w[4];
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const int back = p.taps - 1 - j0 - j;
                        const float* at = back <= i ? p.rows + (size_t)(t - back) * p.ld + p.c_off + ch
                                                    : ring + (size_t)((pos - back + ssd_ring(p)) % ssd_ring(p)) * C + ch;
                        const bool ok = back >= 0 && back <= pos;
                        in[j] = ok ? *at : 0.f;
                        w[j] = back >= 0 ? p.conv[(size_t)(j0 + j) * C + ch] : 0.f;
                    }
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc += w[j] * in[j];
                }
                v = to_f<TA>(from_f<TA>(silu_f(acc)));          // as stored where a kernel of its own does this
            } else {
                const int col = c < p.P ? h * P8 + c : c < p.P + p.N ? p.H * P8 + g * N8 + c - p.P
                                                                     : p.H * P8 + p.G * N8 + g * N8 + c - p.P - p.N;
                v = to_f<TA>(xbc[(size_t)t * ldx + col]);
            }
            if (c < p.P) s_x[i * p.P + c] = v;
            else if (c < p.P + p.N) s_b[i * N4 + c - p.P] = v;
            else s_c[i * N4 + c - p.P - p.N] = v;
        }
        if (tid < cnt) {
            const int t = t0 + c0 + tid;
            float d, la;
            if constexpr (FUSED) {
                d = softplus_f(p.rows[(size_t)t * p.ld + p.dt_off + h] + p.dt_bias[h]);
                la = -p.A[h] * d;
            } else {
                d = dts[(size_t)h * n + t];
                la = dts[(size_t)(p.H + h) * n + t];
            }
            s_d[tid] = d;
            s_d[SSD_STEP + tid] = expf(la);
        }
        __syncthreads();
        // every lane goes through every round, also one whose rows lie beyond P: the sums below are warp-wide
        for (int base = 0; base < p.P; base += groups * RU) {
            const int p0 = base + grp;
            if (base) load(p0);
            for (int i = 0; i < cnt; ++i) {
                const float d = s_d[i], a = s_d[SSD_STEP + i];
                SsdVec<VEC> b[KV], cc[KV];
#pragma unroll
                for (int k = 0; k < KV; ++k) {
                    const int c = (ln + LN * k) * VEC;
                    if (c < p.N) {
                        b[k] = ssd_load<VEC>(s_b + i * N4 + c);
                        cc[k] = ssd_load<VEC>(s_c + i * N4 + c);
                    } else {
#pragma unroll
                        for (int q = 0; q < VEC; ++q) b[k].v[q] = cc[k].v[q] = 0.f;
                    }
                }
                float acc[RU];
#pragma unroll
                for (int u = 0; u < RU; ++u) {
                    const int row = p0 + u * groups;
                    const float dx = row < p.P ? d * s_x[i * p.P + row] : 0.f;
                    acc[u] = 0.f;
#pragma unroll
                    for (int k = 0; k < KV; ++k)
#pragma unroll
                        for (int q = 0; q < VEC; ++q) {
                            S[u][k][q] = a * S[u][k][q] + dx * b[k].v[q];
                            acc[u] += S[u][k][q] * cc[k].v[q];
                        }
                }
#pragma unroll
                for (int u = 0; u < RU; ++u)
                    for (int o = LN >> 1; o > 0; o >>= 1) acc[u] += __shfl_xor_sync(0xffffffffu, acc[u], o);
#pragma unroll
                for (int u = 0; u < RU; ++u)
                    if (ln == 0 && p0 + u * groups < p.P) s_y[i * p.P + p0 + u * groups] = acc[u];
            }
#pragma unroll
            for (int u = 0; u < RU; ++u) {
                const int row = p0 + u * groups;
#pragma unroll
                for (int k = 0; k < KV; ++k) {
                    const int c = (ln + LN * k) * VEC;
                    if (row < p.P && c < p.N) {
                        float* at = Sg + (size_t)row * p.N + c;
                        if constexpr (VEC == 4)
                            *reinterpret_cast<float4*>(at) = make_float4(S[u][k][0], S[u][k][1], S[u][k][2], S[u][k][3]);
                        else
                            *at = S[u][k][0];
                    }
                }
            }
        }
        __syncthreads();
        const float Dh = p.D[h];
        for (int e = tid; e < cnt * p.P; e += blockDim.x) {
            const int i = e / p.P, c = e - i * p.P;
            const size_t t = t0 + c0 + i;
            const float z = e == tid ? z_first : p.rows[t * p.ld + p.z_off + (size_t)h * p.P + c];
            out[t * ldo + (size_t)h * p.P + c] = from_f<TA>((s_y[e] + Dh * s_x[e]) * silu_f(z));
        }
        __syncthreads();
    }
    ssd_keep(p, ring, t0, len, h * p.P, p.P, tid, blockDim.x);
    if (h % (p.H / p.G) == 0) {
        ssd_keep(p, ring, t0, len, inner + g * p.N, p.N, tid, blockDim.x);
        ssd_keep(p, ring, t0, len, inner + gn + g * p.N, p.N, tid, blockDim.x);
    }
}

// ------------------------------------------------------------------ bfloat16 portions in chunks, on the tensor cores
__device__ __forceinline__ uint32_t ssd_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ssd_cp16(void* dst, const void* src, int bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(ssd_smem(dst)), "l"(src), "r"(bytes));
}
__device__ __forceinline__ void ssd_ldsm(const bf16* at, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(ssd_smem(at)));
}
__device__ __forceinline__ void ssd_ldsm_t(const bf16* at, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(ssd_smem(at)));
}
__device__ __forceinline__ void ssd_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// a pair of floats as the sum of two pairs of bfloat16 numbers
__device__ __forceinline__ void ssd_split(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 ssd_pair(uint32_t u) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u)); }

// Segments of the step's requests along time (all null: every request is one item).
struct SsdSegments {
    const int* t0;        // [items] first flat token
    const int* t1;        // [items] one past the last
    const int* req;       // [items] the request's row in the step
    const int* flags;     // [items] bit 0: first segment of its request, bit 1: last
    const int* item0;     // [requests] a request's first item
    const int* items;     // [requests] how many it has
    float* carry;         // [items][H][P][N], of a request with several: the state behind its first segment, what the tokens of a
                          // middle one leave from an empty state, and (at its last) the state it came with
    float* decay;         // [items][H]: the sum of the segment's log decays
};

template <int NK, int PW> struct SsdTile {           // N padded to 16 * NK, 16 * PW rows of S^T
    static constexpr int NT = PW * 64;               // threads: two warps (halves of N) per 16 rows
    static constexpr int NS = NK * 16 + 8;           // row stride of B and C (a shift of 16 bytes a row: ldmatrix without conflicts)
    static constexpr int MS = SSD_CHUNK + 8;         // of the weighted scores
    static constexpr int PS = 16 * PW + 8;           // of x
    static constexpr int YS = 16 * PW + 4;           // of the outputs (over the weighted scores)
    static constexpr size_t stage = (size_t)SSD_CHUNK * (2 * NS + PS) * sizeof(bf16);
    static constexpr size_t m_bytes = 2 * SSD_CHUNK * MS * sizeof(bf16), y_bytes = (size_t)SSD_CHUNK * YS * sizeof(float);
    static constexpr size_t bytes = 2 * stage + (m_bytes > y_bytes ? m_bytes : y_bytes) + 2 * 2 * SSD_CHUNK * sizeof(float);
};

// PASS 0: whole requests.  1: what SsdSegments says of carry, and a segment's decay; no output.  2: segments from the state they
// start from (put together from carry: the blocks of a request's last segment overwrite its slot), with output.
template <int NK, int PW, int PASS>
__global__ void __launch_bounds__(PW * 64, NK <= 8 ? 8 / PW : 4 / PW)
ssd_chunk_kernel(const SsdArgs p, const bf16* xbc, long long ldx, const float* dts, int n, bf16* out, long long ldo,
                 const SsdSegments seg) {
    using Tile = SsdTile<NK, PW>;
    constexpr int Q = SSD_CHUNK, NS = Tile::NS, MS = Tile::MS, PS = Tile::PS, YS = Tile::YS, NT = Tile::NT, NH = NK / 2, NW = NT / 32;
    extern __shared__ __align__(128) unsigned char sm_raw[];
    bf16* s_m = reinterpret_cast<bf16*>(sm_raw + 2 * Tile::stage);            // [2][Q][MS]: high and low parts
    float* s_y = reinterpret_cast<float*>(s_m);                               // [Q][YS], when the scores have been read
    float* s_d = reinterpret_cast<float*>(sm_raw + Tile::bytes) - 4 * Q;      // [2 stages][2][Q]: step sizes, sums of log decays
    // (no early launch of what follows while the long-lived blocks are still to be placed)
    pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, c2 = (lane & 3) * 2;
    const int mi = lane >> 3, ri = lane & 7, pw = warp >> 1, half = warp & 1;
    const int tiles = (p.P + 16 * PW - 1) / (16 * PW), h = blockIdx.x / tiles, p0 = (blockIdx.x % tiles) * 16 * PW;
    const int item = blockIdx.y, r = PASS == 0 ? item : seg.req[item];
    const int t0 = PASS == 0 ? p.cu_q[r] : seg.t0[item], len = (PASS == 0 ? p.cu_q[r + 1] : seg.t1[item]) - t0;
    const bool first = PASS == 0 || (seg.flags[item] & 1), last = PASS == 0 || (seg.flags[item] & 2);
    if (len <= 0 || (PASS == 1 && first && last)) return;
    const int grp = h / (p.H / p.G), P8 = ssd_pad8(p.P), N8 = ssd_pad8(p.N);
    float* slot = p.state + (size_t)p.slots[r] * p.slot_stride;
    float* Sg = slot + (size_t)h * p.P * p.N;
    float* Sc = PASS == 0 ? nullptr : seg.carry + ((size_t)item * p.H + h) * p.P * p.N;        // (pass 1)
    float* ring = slot + p.ring_base;
    const int per = p.P * p.N, rows_here = min(16 * PW, p.P - p0);
    if (PASS == 1 && last) {
        for (int e = tid; e < rows_here * p.N; e += NT) Sc[(size_t)p0 * p.N + e] = Sg[(size_t)p0 * p.N + e];
        return;
    }

    const bf16* x_src = xbc + (size_t)t0 * ldx + (size_t)h * P8 + p0;
    const bf16* b_src = xbc + (size_t)t0 * ldx + (size_t)p.H * P8 + (size_t)grp * N8;
    const bf16* c_src = b_src + (size_t)p.G * N8;
    const int x_runs = min(P8 - p0, 16 * PW) / 8, n_runs = N8 / 8;
    auto fetch = [&](int buf, int c0) {
        bf16* s_b = reinterpret_cast<bf16*>(sm_raw + buf * Tile::stage);
        bf16 *s_c = s_b + Q * NS, *s_x = s_c + Q * NS;
        for (int e = tid; e < Q * 2 * NK; e += NT) {
            const int i = e / (2 * NK), q = e % (2 * NK);
            const bool ok = c0 + i < len && q < n_runs;
            const size_t off = ok ? (size_t)(c0 + i) * ldx + 8 * q : 0;
            ssd_cp16(s_b + i * NS + 8 * q, b_src + off, ok ? 16 : 0);
            if (PASS != 1) ssd_cp16(s_c + i * NS + 8 * q, c_src + off, ok ? 16 : 0);
        }
        for (int e = tid; e < Q * 2 * PW; e += NT) {
            const int i = e / (2 * PW), q = e % (2 * PW);
            const bool ok = c0 + i < len && q < x_runs;
            ssd_cp16(s_x + i * PS + 8 * q, x_src + (ok ? (size_t)(c0 + i) * ldx + 8 * q : 0), ok ? 16 : 0);
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    // step sizes and running sums of the log decays of a chunk, by the last warp (two tokens a lane)
    auto scan = [&](int buf, int c0) {
        const int i = 2 * lane, t = t0 + c0 + i;
        const bool ok0 = c0 + i < len, ok1 = c0 + i + 1 < len;
        const float *d = dts + (size_t)h * n, *l = dts + (size_t)(p.H + h) * n;
        const float d0 = ok0 ? d[t] : 0.f, d1 = ok1 ? d[t + 1] : 0.f, l0 = ok0 ? l[t] : 0.f, l1 = ok1 ? l[t + 1] : 0.f;
        float run = l0 + l1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, run, o);
            if (lane >= o) run += up;
        }
        float* s = s_d + buf * 2 * Q;
        s[i] = d0;
        s[i + 1] = d1;
        s[Q + i] = run - l1;
        s[Q + i + 1] = run;
    };
    fetch(0, 0);
    if (warp == NW - 1) scan(0, 0);

    // S^T: rows row0 and row0 + 8 of this lane, columns n0 + 8 j + c2, + 1 (the warp's half of N)
    const int row0 = p0 + pw * 16 + g8, n0 = half * NH * 16;
    float S[2 * NH][4];
    // S <- decay * S + what lies at `from`
    auto take = [&](const float* from, float decay) {
#pragma unroll
        for (int j = 0; j < 2 * NH; ++j)
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const int row = row0 + (q >> 1) * 8, c = n0 + 8 * j + c2 + (q & 1);
                S[j][q] = decay * S[j][q] + (row < p.P && c < p.N ? from[(size_t)row * p.N + c] : 0.f);
            }
    };
#pragma unroll
    for (int j = 0; j < 2 * NH; ++j) S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.f;
    if (PASS != 2 || (first && last)) {
        if (PASS != 1 || first) take(Sg, 0.f);
    } else {
        const int i0 = seg.item0[r];
        auto at = [&](int i) { return seg.carry + ((size_t)i * p.H + h) * per; };
        if (first) {
            take(at(i0 + seg.items[r] - 1), 0.f);
        } else {
            take(at(i0), 0.f);
            for (int i = i0 + 1; i < item; ++i) take(at(i), expf(seg.decay[(size_t)i * p.H + h]));
        }
    }
    const float Dh = p.D[h];
    const bool vec = p.P % 8 == 0 && p.ld % 4 == 0 && p.z_off % 4 == 0 && ldo % 8 == 0 && ((uintptr_t)p.rows & 15) == 0 &&
                     ((uintptr_t)out & 15) == 0;
    float total_all = 0.f;

    int buf = 0;
    for (int c0 = 0; c0 < len; c0 += Q, buf ^= 1) {
        const int cnt = min(Q, len - c0), it16 = (cnt + 15) / 16;        // runs of 16 tokens that hold something
        asm volatile("cp.async.wait_group 0;\n" ::);
        __syncthreads();                             // this chunk is there, and everybody is done with the other stage and the outputs
        if (c0 + Q < len) fetch(buf ^ 1, c0 + Q);
        const bf16* s_b = reinterpret_cast<const bf16*>(sm_raw + buf * Tile::stage);
        const bf16 *s_c = s_b + Q * NS, *s_x = s_c + Q * NS;
        const float *s_dt = s_d + buf * 2 * Q, *s_l = s_dt + Q;
        const float total = s_l[Q - 1], carry = expf(total);
        float y[8][4];

        if (PASS != 1) {
            // weighted scores: a warp takes a run of 16 tokens i against 32 tokens j at a time
            for (int task = warp; task < 8; task += NW) {
                const int ti = task >> 1, jh = task & 1;
                if (ti >= it16 || (jh && ti < 2)) continue;
                float acc[4][4];
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
                for (int k = 0; k < NK; ++k) {
                    uint32_t a[4];
                    ssd_ldsm(s_c + (ti * 16 + (mi & 1) * 8 + ri) * NS + k * 16 + (mi >> 1) * 8, a);
#pragma unroll
                    for (int jq = 0; jq < 2; ++jq) {
                        const int jp = 2 * jh + jq;
                        if (jp <= ti) {
                            uint32_t b[4];
                            ssd_ldsm(s_b + (jp * 16 + (mi >> 1) * 8 + ri) * NS + k * 16 + (mi & 1) * 8, b);
                            ssd_mma(acc[2 * jq], a, b[0], b[1]);
                            ssd_mma(acc[2 * jq + 1], a, b[2], b[3]);
                        }
                    }
                }
                const int i0 = ti * 16 + g8, i1 = i0 + 8;
                const float li0 = s_l[i0], li1 = s_l[i1];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int jc = 32 * jh + 8 * j + c2;
                    if (2 * jh + (j >> 1) <= ti) {
                        const float2 lj = *reinterpret_cast<const float2*>(s_l + jc), dj = *reinterpret_cast<const float2*>(s_dt + jc);
                        const float v00 = jc <= i0 ? acc[j][0] * expf(li0 - lj.x) * dj.x : 0.f;
                        const float v01 = jc + 1 <= i0 ? acc[j][1] * expf(li0 - lj.y) * dj.y : 0.f;
                        const float v10 = jc <= i1 ? acc[j][2] * expf(li1 - lj.x) * dj.x : 0.f;
                        const float v11 = jc + 1 <= i1 ? acc[j][3] * expf(li1 - lj.y) * dj.y : 0.f;
                        uint32_t hi, lo;
                        ssd_split(v00, v01, hi, lo);
                        *reinterpret_cast<uint32_t*>(s_m + i0 * MS + jc) = hi;
                        *reinterpret_cast<uint32_t*>(s_m + (Q + i0) * MS + jc) = lo;
                        ssd_split(v10, v11, hi, lo);
                        *reinterpret_cast<uint32_t*>(s_m + i1 * MS + jc) = hi;
                        *reinterpret_cast<uint32_t*>(s_m + (Q + i1) * MS + jc) = lo;
                    }
                }
            }
            __syncthreads();

            // y^T: what the warp's half of the state before the chunk gives, times e^(L_i), then half of the chunk's own tokens
#pragma unroll
            for (int j = 0; j < 8; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
#pragma unroll
            for (int k = 0; k < NH; ++k) {
                uint32_t ah[4], al[4];
                ssd_split(S[2 * k][0], S[2 * k][1], ah[0], al[0]);
                ssd_split(S[2 * k][2], S[2 * k][3], ah[1], al[1]);
                ssd_split(S[2 * k + 1][0], S[2 * k + 1][1], ah[2], al[2]);
                ssd_split(S[2 * k + 1][2], S[2 * k + 1][3], ah[3], al[3]);
#pragma unroll
                for (int ip = 0; ip < 4; ++ip) {
                    if (ip < it16) {
                        uint32_t b[4];
                        ssd_ldsm(s_c + (ip * 16 + (mi >> 1) * 8 + ri) * NS + n0 + k * 16 + (mi & 1) * 8, b);
                        ssd_mma(y[2 * ip], ah, b[0], b[1]);
                        ssd_mma(y[2 * ip + 1], ah, b[2], b[3]);
                        ssd_mma(y[2 * ip], al, b[0], b[1]);
                        ssd_mma(y[2 * ip + 1], al, b[2], b[3]);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float2 l = *reinterpret_cast<const float2*>(s_l + 8 * j + c2);
                const float e0 = expf(l.x), e1 = expf(l.y);
                y[j][0] *= e0;
                y[j][1] *= e1;
                y[j][2] *= e0;
                y[j][3] *= e1;
            }
        }
#pragma unroll
        for (int j = 0; j < 2 * NH; ++j) {
            S[j][0] *= carry;
            S[j][1] *= carry;
            S[j][2] *= carry;
            S[j][3] *= carry;
        }
#pragma unroll
        for (int kj = 0; kj < 4; ++kj) {
            if (kj < it16) {
                uint32_t x[4];
                ssd_ldsm_t(s_x + (kj * 16 + (mi >> 1) * 8 + ri) * PS + pw * 16 + (mi & 1) * 8, x);
                if (PASS != 1 && (kj & 1) == half) {
#pragma unroll
                    for (int ip = 0; ip < 4; ++ip) {
                        if (ip >= kj && ip < it16) {
                            uint32_t b[4];
                            const bf16* at = s_m + (ip * 16 + (mi >> 1) * 8 + ri) * MS + kj * 16 + (mi & 1) * 8;
                            ssd_ldsm(at, b);
                            ssd_mma(y[2 * ip], x, b[0], b[1]);
                            ssd_mma(y[2 * ip + 1], x, b[2], b[3]);
                            ssd_ldsm(at + Q * MS, b);
                            ssd_mma(y[2 * ip], x, b[0], b[1]);
                            ssd_mma(y[2 * ip + 1], x, b[2], b[3]);
                        }
                    }
                }
                // the tokens' part of the new state: x weighted by e^(L_64 - L_j) d_j
                const int j0 = kj * 16 + c2;
                const float2 la = *reinterpret_cast<const float2*>(s_l + j0), lb = *reinterpret_cast<const float2*>(s_l + j0 + 8);
                const float2 da = *reinterpret_cast<const float2*>(s_dt + j0), db = *reinterpret_cast<const float2*>(s_dt + j0 + 8);
                const float w0 = expf(total - la.x) * da.x, w1 = expf(total - la.y) * da.y;
                const float w2 = expf(total - lb.x) * db.x, w3 = expf(total - lb.y) * db.y;
                uint32_t xh[4], xl[4];
                float2 f = ssd_pair(x[0]);
                ssd_split(f.x * w0, f.y * w1, xh[0], xl[0]);
                f = ssd_pair(x[1]);
                ssd_split(f.x * w0, f.y * w1, xh[1], xl[1]);
                f = ssd_pair(x[2]);
                ssd_split(f.x * w2, f.y * w3, xh[2], xl[2]);
                f = ssd_pair(x[3]);
                ssd_split(f.x * w2, f.y * w3, xh[3], xl[3]);
#pragma unroll
                for (int k = 0; k < NH; ++k) {
                    uint32_t b[4];
                    ssd_ldsm_t(s_b + (kj * 16 + (mi & 1) * 8 + ri) * NS + n0 + k * 16 + (mi >> 1) * 8, b);
                    ssd_mma(S[2 * k], xh, b[0], b[1]);
                    ssd_mma(S[2 * k + 1], xh, b[2], b[3]);
                    ssd_mma(S[2 * k], xl, b[0], b[1]);
                    ssd_mma(S[2 * k + 1], xl, b[2], b[3]);
                }
            }
        }
        total_all += total;
        if (warp == NW - 1 && c0 + Q < len) scan(buf ^ 1, c0 + Q);
        if (PASS == 1) continue;
        // out: the halves added in shared memory (in the order of the halves), then eight columns of a token at a time
        __syncthreads();                             // the weighted scores have been read
        if (half == 0) {
#pragma unroll
            for (int j = 0; j < 8; ++j)
#pragma unroll
                for (int q = 0; q < 4; ++q) s_y[(8 * j + c2 + (q & 1)) * YS + pw * 16 + g8 + (q >> 1) * 8] = y[j][q];
        }
        __syncthreads();
        if (half == 1) {
#pragma unroll
            for (int j = 0; j < 8; ++j)
#pragma unroll
                for (int q = 0; q < 4; ++q) s_y[(8 * j + c2 + (q & 1)) * YS + pw * 16 + g8 + (q >> 1) * 8] += y[j][q];
        }
        __syncthreads();
        for (int e = tid; e < cnt * 2 * PW; e += NT) {
            const int i = e / (2 * PW), c = (e % (2 * PW)) * 8, col = p0 + c;
            if (col >= p.P) continue;
            const size_t t = t0 + c0 + i;
            const float* zp = p.rows + t * p.ld + p.z_off + (size_t)h * p.P + col;
            bf16* o = out + t * ldo + (size_t)h * p.P + col;
            const uint4 xu = *reinterpret_cast<const uint4*>(s_x + i * PS + c);
            const float2 x0 = ssd_pair(xu.x), x1 = ssd_pair(xu.y), x2 = ssd_pair(xu.z), x3 = ssd_pair(xu.w);
            const float xs[8] = {x0.x, x0.y, x1.x, x1.y, x2.x, x2.y, x3.x, x3.y};
            float z[8], v[8];
            if (vec) {
                const float4 za = *reinterpret_cast<const float4*>(zp), zb = *reinterpret_cast<const float4*>(zp + 4);
                z[0] = za.x; z[1] = za.y; z[2] = za.z; z[3] = za.w;
                z[4] = zb.x; z[5] = zb.y; z[6] = zb.z; z[7] = zb.w;
            } else {
#pragma unroll
                for (int q = 0; q < 8; ++q) z[q] = col + q < p.P ? zp[q] : 0.f;
            }
            const float4 ya = *reinterpret_cast<const float4*>(s_y + i * YS + c), yb = *reinterpret_cast<const float4*>(s_y + i * YS + c + 4);
            const float ys[8] = {ya.x, ya.y, ya.z, ya.w, yb.x, yb.y, yb.z, yb.w};
#pragma unroll
            for (int q = 0; q < 8; ++q) v[q] = (ys[q] + Dh * xs[q]) * silu_f(z[q]);
            if (vec) {
                uint4 u;
                const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
                const __nv_bfloat162 cc = __floats2bfloat162_rn(v[4], v[5]), d = __floats2bfloat162_rn(v[6], v[7]);
                u.x = *reinterpret_cast<const uint32_t*>(&a);
                u.y = *reinterpret_cast<const uint32_t*>(&b);
                u.z = *reinterpret_cast<const uint32_t*>(&cc);
                u.w = *reinterpret_cast<const uint32_t*>(&d);
                *reinterpret_cast<uint4*>(o) = u;
            } else {
#pragma unroll
                for (int q = 0; q < 8; ++q)
                    if (col + q < p.P) o[q] = __float2bfloat16_rn(v[q]);
            }
        }
    }
    pdl_launch_dependents();
    if (PASS != 2 || last) {
        float* S_to = PASS == 1 ? Sc : Sg;
#pragma unroll
        for (int j = 0; j < 2 * NH; ++j)
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const int row = row0 + (q >> 1) * 8, c = n0 + 8 * j + c2 + (q & 1);
                if (row < p.P && c < p.N) S_to[(size_t)row * p.N + c] = S[j][q];
            }
    }
    if (PASS == 1) {
        if (tid == 0 && p0 == 0) seg.decay[(size_t)item * p.H + h] = total_all;
        return;
    }
    if (!last) return;
    ssd_keep(p, ring, p.cu_q[r], p.cu_q[r + 1] - p.cu_q[r], h * p.P + p0, min(16 * PW, p.P - p0), tid, NT);
    if (h % (p.H / p.G) == 0 && p0 == 0) {
        const int inner = p.H * p.P, q0 = p.cu_q[r], ql = p.cu_q[r + 1] - q0;
        ssd_keep(p, ring, q0, ql, inner + grp * p.N, p.N, tid, NT);
        ssd_keep(p, ring, q0, ql, inner + p.G * p.N + grp * p.N, p.N, tid, NT);
    }
}

// ------------------------------------------------------------------ norm of the gated rows
// One block per (token, part): v[t, part] /= rms(v[t, part]), times w; in place.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
ssd_norm_kernel(T* v, long long ld, const float* __restrict__ w, int size, float eps) {
    __shared__ float red[33];
    pdl_launch_dependents();
    pdl_wait();
    T* row = v + (size_t)blockIdx.x * ld + (size_t)blockIdx.y * size;
    const float* wp = w + (size_t)blockIdx.y * size;
    float ss = 0.f;
    if constexpr (VEC == 8) {
        for (int i = threadIdx.x * 8; i < size; i += blockDim.x * 8) {
            const uint4 u = *reinterpret_cast<const uint4*>(row + i);
            const uint32_t a[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float2 f = ssd_pair(a[q]);
                ss += f.x * f.x + f.y * f.y;
            }
        }
    } else {
        for (int i = threadIdx.x; i < size; i += blockDim.x) {
            const float f = to_f<T>(row[i]);
            ss += f * f;
        }
    }
    ss = block_sum(ss, red);
    const float rs = 1.0f / sqrtf(ss / (float)size + eps);
    if constexpr (VEC == 8) {
        for (int i = threadIdx.x * 8; i < size; i += blockDim.x * 8) {
            uint4 u = *reinterpret_cast<const uint4*>(row + i);
            uint32_t a[4] = {u.x, u.y, u.z, u.w};
            const float4 w0 = *reinterpret_cast<const float4*>(wp + i), w1 = *reinterpret_cast<const float4*>(wp + i + 4);
            const float ww[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float2 f = ssd_pair(a[q]);
                const __nv_bfloat162 o = __floats2bfloat162_rn(f.x * rs * ww[2 * q], f.y * rs * ww[2 * q + 1]);
                a[q] = *reinterpret_cast<const uint32_t*>(&o);
            }
            *reinterpret_cast<uint4*>(row + i) = make_uint4(a[0], a[1], a[2], a[3]);
        }
    } else {
        for (int i = threadIdx.x; i < size; i += blockDim.x) row[i] = from_f<T>(to_f<T>(row[i]) * rs * wp[i]);
    }
}

// ------------------------------------------------------------------ launchers
static SsdArgs ssd_args(const float* rows, long long ld, int z_off, int c_off, int dt_off, const float* conv, const float* conv_b,
                        const float* dt_bias, const float* A, const float* D, float* state, long long slot_stride,
                        const int* positions, const int* seq_ids, const int* cu_q, const int* slots, int H, int G, int P, int N,
                        int taps) {
    SsdArgs p;
    p.rows = rows; p.ld = ld; p.z_off = z_off; p.c_off = c_off; p.dt_off = dt_off;
    p.conv = conv; p.conv_b = conv_b; p.dt_bias = dt_bias; p.A = A; p.D = D;
    p.state = state; p.slot_stride = slot_stride; p.ring_base = (long long)H * P * N;
    p.positions = positions; p.seq_ids = seq_ids; p.cu_q = cu_q; p.slots = slots;
    p.H = H; p.G = G; p.P = P; p.N = N; p.taps = taps;
    return p;
}

template <typename TA>
static int ssd_run_conv(const SsdArgs& p, TA* xbc, long long ldx, float* dts, int n, cudaStream_t stream) {
    const int C = p.H * p.P + 2 * p.G * p.N;
    const auto al16 = [](const void* q) { return ((uintptr_t)q & 15) == 0; };
    const bool vec = p.P % 8 == 0 && p.N % 8 == 0 && p.ld % 4 == 0 && p.c_off % 4 == 0 && p.slot_stride % 4 == 0 &&
                     p.ring_base % 4 == 0 && al16(p.rows) && al16(p.state) && al16(p.conv) && al16(p.conv_b) && al16(xbc);
    const int per = 256 * (vec ? 4 : 1);
    const dim3 grid((n + SSD_CONV_TOK - 1) / SSD_CONV_TOK, (C + per - 1) / per + 1);
    if (p.taps == 4)
        return vec ? rllm_launch(ssd_conv_kernel<TA, 4, 4>, grid, dim3(256), 0, stream, p, xbc, ldx, dts, n)
                   : rllm_launch(ssd_conv_kernel<TA, 1, 4>, grid, dim3(256), 0, stream, p, xbc, ldx, dts, n);
    return vec ? rllm_launch(ssd_conv_kernel<TA, 4, 0>, grid, dim3(256), 0, stream, p, xbc, ldx, dts, n)
               : rllm_launch(ssd_conv_kernel<TA, 1, 0>, grid, dim3(256), 0, stream, p, xbc, ldx, dts, n);
}

template <typename TA, int VEC, int KV>
static int ssd_run_step_kv(const SsdArgs& p, const TA* xbc, long long ldx, const float* dts, int n, int n_requests, TA* out,
                           long long ldo, int LN, bool fused, cudaStream_t stream) {
    const size_t smem = sizeof(float) * SSD_STEP * (2 * ((p.N + 3) / 4 * 4) + 2 * p.P + 2);
    auto kern = fused ? ssd_step_kernel<TA, VEC, KV, true> : ssd_step_kernel<TA, VEC, KV, false>;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    return rllm_launch(kern, dim3(p.H, n_requests), dim3(256), smem, stream, p, xbc, ldx, dts, n, out, ldo, LN);
}

template <typename TA>
static int ssd_run_step(const SsdArgs& p, const TA* xbc, long long ldx, const float* dts, int n, int n_requests, TA* out,
                        long long ldo, bool fused, cudaStream_t stream) {
    const bool vec = p.N % 4 == 0 && p.slot_stride % 4 == 0 && ((uintptr_t)p.state & 15) == 0;
    const int units = vec ? p.N / 4 : p.N;
    int LN = 1;
    while (LN < units && LN < 32) LN *= 2;
    const int kv = (units + LN - 1) / LN;
#define SSD_KV(V, K) return ssd_run_step_kv<TA, V, K>(p, xbc, ldx, dts, n, n_requests, out, ldo, LN, fused, stream)
    if (vec) {
        if (kv <= 1) SSD_KV(4, 1);
        if (kv <= 2) SSD_KV(4, 2);
        if (kv <= 8) SSD_KV(4, 8);
    } else {
        if (kv <= 1) SSD_KV(1, 1);
        if (kv <= 2) SSD_KV(1, 2);
        if (kv <= 8) SSD_KV(1, 8);
    }
#undef SSD_KV
    return (int)cudaErrorInvalidValue;
}

template <int NK, int PW, int PASS>
static int ssd_run_pass(const SsdArgs& p, const bf16* xbc, long long ldx, const float* dts, int n, int items, bf16* out, long long ldo,
                        const SsdSegments& seg, cudaStream_t stream) {
    using Tile = SsdTile<NK, PW>;
    static bool raised = false;
    if (!raised) {
        const cudaError_t e = cudaFuncSetAttribute(ssd_chunk_kernel<NK, PW, PASS>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                   (int)Tile::bytes);
        if (e != cudaSuccess) return (int)e;
        raised = true;
    }
    const int tiles = (p.P + 16 * PW - 1) / (16 * PW);
    return rllm_launch(ssd_chunk_kernel<NK, PW, PASS>, dim3(p.H * tiles, items), dim3(Tile::NT), Tile::bytes, stream, p, xbc, ldx, dts, n,
                       out, ldo, seg);
}
template <int NK, int PW>
static int ssd_run_chunk_w(const SsdArgs& p, const bf16* xbc, long long ldx, const float* dts, int n, int n_requests, bf16* out,
                           long long ldo, const SsdSegments& seg, int n_items, cudaStream_t stream) {
    if (n_items <= 0) return ssd_run_pass<NK, PW, 0>(p, xbc, ldx, dts, n, n_requests, out, ldo, seg, stream);
    const int st = ssd_run_pass<NK, PW, 1>(p, xbc, ldx, dts, n, n_items, out, ldo, seg, stream);
    if (st) return st;
    return ssd_run_pass<NK, PW, 2>(p, xbc, ldx, dts, n, n_items, out, ldo, seg, stream);
}
template <int NK>
static int ssd_run_chunk(const SsdArgs& p, const bf16* xbc, long long ldx, const float* dts, int n, int n_requests, bf16* out,
                         long long ldo, const SsdSegments& seg, int n_items, cudaStream_t stream) {
    if (p.P <= 16) return ssd_run_chunk_w<NK, 1>(p, xbc, ldx, dts, n, n_requests, out, ldo, seg, n_items, stream);
    if (p.P <= 32) return ssd_run_chunk_w<NK, 2>(p, xbc, ldx, dts, n, n_requests, out, ldo, seg, n_items, stream);
    return ssd_run_chunk_w<NK, 4>(p, xbc, ldx, dts, n, n_requests, out, ldo, seg, n_items, stream);
}

// mode 0: a step of at most SSD_STEP tokens a request, everything in one kernel; 1: portions, token by token; 2: portions
// (bfloat16, N up to 256) in chunks.  xbc [n, H * P8 + 2 G * N8] (activation type) and dts [2, H, n]: scratch of modes 1 and 2.
// out (activation type, rows ldo apart): y * silu(z), before the norm.  seg_*, n_items: the step's requests cut along time (mode 2;
// n_items 0: not cut), carry [n_items, H, P, N] and decay [n_items, H] scratch.
RLLM_API int rllm_ssd(const float* rows, long long ld, int z_off, int c_off, int dt_off, const float* conv, const float* conv_b,
                      const float* dt_bias, const float* A, const float* D, float* state, long long slot_stride,
                      const int* positions, const int* seq_ids, const int* cu_q, const int* slots, int H, int G, int P, int N,
                      int taps, int n, int n_requests, int mode, void* xbc, long long ldx, float* dts, void* out, int out_dt,
                      long long ldo, const int* seg_t0, const int* seg_t1, const int* seg_req, const int* seg_flags,
                      const int* req_item0, const int* req_items, int n_items, float* carry, float* decay, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || P <= 0 || N <= 0 || taps < 1 || n_requests <= 0 || mode < 0 || mode > 2 ||
        (mode > 0 && (!xbc || !dts || ldx < (long long)H * ssd_pad8(P) + 2LL * G * ssd_pad8(N))))
        return (int)cudaErrorInvalidValue;
    const SsdArgs p = ssd_args(rows, ld, z_off, c_off, dt_off, conv, conv_b, dt_bias, A, D, state, slot_stride, positions, seq_ids,
                               cu_q, slots, H, G, P, N, taps);
    if (mode > 0) {
        const int st = out_dt == RLLM_F32 ? ssd_run_conv<float>(p, (float*)xbc, ldx, dts, n, stream)
                                          : ssd_run_conv<bf16>(p, (bf16*)xbc, ldx, dts, n, stream);
        if (st) return st;
    }
    if (mode < 2)
        return out_dt == RLLM_F32
            ? ssd_run_step<float>(p, (const float*)xbc, ldx, dts, n, n_requests, (float*)out, ldo, mode == 0, stream)
            : ssd_run_step<bf16>(p, (const bf16*)xbc, ldx, dts, n, n_requests, (bf16*)out, ldo, mode == 0, stream);
    if (out_dt != RLLM_BF16 || N > 256 || ldx % 8 || ((uintptr_t)xbc & 15)) return (int)cudaErrorInvalidValue;
    if (n_items > 0 && (!seg_t0 || !seg_t1 || !seg_req || !seg_flags || !req_item0 || !req_items || !carry || !decay))
        return (int)cudaErrorInvalidValue;
    const bf16* x = (const bf16*)xbc;
    const SsdSegments seg = {seg_t0, seg_t1, seg_req, seg_flags, req_item0, req_items, carry, decay};
#define SSD_CHUNKS(NK) return ssd_run_chunk<NK>(p, x, ldx, dts, n, n_requests, (bf16*)out, ldo, seg, n_items, stream)
    if (N <= 32) SSD_CHUNKS(2);
    if (N <= 64) SSD_CHUNKS(4);
    if (N <= 128) SSD_CHUNKS(8);
    SSD_CHUNKS(16);
#undef SSD_CHUNKS
}

RLLM_API int rllm_ssd_norm(void* v, int dt, long long ld, const float* w, int n, int parts, int size, float eps,
                           cudaStream_t stream) {
    if (n <= 0) return 0;
    if (parts <= 0 || size <= 0 || ld < (long long)parts * size) return (int)cudaErrorInvalidValue;
    const bool vec = dt == RLLM_BF16 && size % 8 == 0 && ld % 8 == 0 && ((uintptr_t)v & 15) == 0 && ((uintptr_t)w & 15) == 0;
    const int units = vec ? size / 8 : size, threads = units > 128 ? 256 : units > 64 ? 128 : units > 32 ? 64 : 32;
    const dim3 grid(n, parts);
    if (dt == RLLM_F32)
        return rllm_launch(ssd_norm_kernel<float, 1>, grid, dim3(threads), 0, stream, (float*)v, ld, w, size, eps);
    if (vec) return rllm_launch(ssd_norm_kernel<bf16, 8>, grid, dim3(threads), 0, stream, (bf16*)v, ld, w, size, eps);
    return rllm_launch(ssd_norm_kernel<bf16, 1>, grid, dim3(threads), 0, stream, (bf16*)v, ld, w, size, eps);
}

RLLM_PACKED(rllm_ssd)
RLLM_PACKED(rllm_ssd_norm)
