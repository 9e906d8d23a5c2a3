// Products of routed experts on the Blackwell tensor cores in one launch: the rows of A [rows, K] lie in expert order (expert e's
// rows are offsets[e] .. offsets[e + 1] - 1, known on the device only), B [E * N, K] holds the experts' matrices one after another,
//     C[r, n] = f(row_scale[r] * (B[e N + n, :] . A[r, :]))          (row_scale optional; f an activation by number)
// bfloat16 operands, float32 accumulation in tensor memory.  A plain product is the case of one expert (offsets null: all rows).
//
// The machinery of gemm_tc.cu: persistent CTAs over 128 x 256 tiles, a ring of stages filled by TMA, one thread that issues
// tcgen05.mma, two accumulators so that a tile's epilogue overlaps the next tile's products, every mbarrier wait bounded.  The
// tiles are counted from the offsets by every CTA itself: expert e has ceil(rows_e / 128) row tiles; a tile's rows
// behind its expert's last one and columns behind N belong to a neighbour and are dropped at the store.  So the host needs not
// know how many rows an expert has, and the step's launches do not depend on it.
#include "tcgen05.cuh"
#include "activations.cuh"

#define GG_BM 128
#define GG_BN 256
#define GG_BK 64
#define GG_STAGES 4
#define GG_THREADS 192
#define GG_MAX_E 1024

enum { GG_ERR_FULL = 21, GG_ERR_EMPTY = 22, GG_ERR_ACC = 23 };

template <typename TC> __device__ __forceinline__ void gg_store32(TC* dst, const float (&v)[32], int n_valid) {
    if (n_valid >= 32 && ((uintptr_t)dst & 15) == 0) {
        if constexpr (sizeof(TC) == 4) {
#pragma unroll
            for (int j = 0; j < 8; ++j)
                reinterpret_cast<float4*>(dst)[j] = make_float4(v[4 * j], v[4 * j + 1], v[4 * j + 2], v[4 * j + 3]);
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                uint32_t u[4];
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const __nv_bfloat162 b = __floats2bfloat162_rn(v[8 * j + 2 * q], v[8 * j + 2 * q + 1]);
                    u[q] = *reinterpret_cast<const uint32_t*>(&b);
                }
                reinterpret_cast<uint4*>(dst)[j] = make_uint4(u[0], u[1], u[2], u[3]);
            }
        }
    } else {
#pragma unroll
        for (int j = 0; j < 32; ++j)
            if (j < n_valid) dst[j] = from_f<TC>(v[j]);
    }
}

// ACT: the activation's number, or -1: `act` decides (a switch per element in the epilogue's loop costs more than the products)
template <typename TC, int ACT>
__global__ void __launch_bounds__(GG_THREADS, 1)
gemm_group_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB, TC* C, long long ldc, const int* offsets,
                  int E, int rows, int N, int K, const float* row_scale, int act, int* err) {
    constexpr int A_BYTES = GG_BM * GG_BK * 2, B_BYTES = GG_BN * GG_BK * 2, STAGE_BYTES = A_BYTES + B_BYTES;
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    __shared__ __align__(8) uint64_t full_bar[GG_STAGES];
    __shared__ __align__(8) uint64_t empty_bar[GG_STAGES];
    __shared__ __align__(8) uint64_t acc_full[2];
    __shared__ __align__(8) uint64_t acc_empty[2];
    __shared__ uint32_t tmem_base_slot;
    __shared__ volatile int abort_flag;
    __shared__ int s_row[GG_MAX_E + 1];              // an expert's first row
    __shared__ int s_tile[GG_MAX_E + 1];             // its first row tile

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nkb = (K + GG_BK - 1) / GG_BK, n_tiles = (N + GG_BN - 1) / GG_BN;
    if (tid == 0) {
        asm volatile("prefetch.tensormap [%0];" ::"l"(&tmA) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&tmB) : "memory");
        for (int s = 0; s < GG_STAGES; ++s) { mbar_init(&full_bar[s], 1); mbar_init(&empty_bar[s], 1); }
        for (int b = 0; b < 2; ++b) { mbar_init(&acc_full[b], 1); mbar_init(&acc_empty[b], 128); }
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        tmem_alloc(&tmem_base_slot, 2 * GG_BN);
        tmem_relinquish();
    }
    pdl_wait();                                      // rows and offsets are written by the kernels before
    if (warp == 2) {                                 // first rows and first row tiles of the experts, 32 at a time
        int run = 0;
        for (int e0 = 0; e0 <= E; e0 += 32) {
            const int e = e0 + lane;
            const int first = e > E ? 0 : offsets ? min(max(offsets[e], 0), rows) : (e == 0 ? 0 : rows);
            const int next = e >= E ? first : offsets ? min(max(offsets[e + 1], 0), rows) : rows;
            const int t = e < E ? (max(next - first, 0) + GG_BM - 1) / GG_BM : 0;
            int incl = t;
#pragma unroll
            for (int m = 1; m < 32; m <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, incl, m);
                if (lane >= m) incl += up;
            }
            if (e <= E) {
                s_row[e] = first;
                s_tile[e] = run + incl - t;
            }
            run += __shfl_sync(0xffffffffu, incl, 31);
        }
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = tmem_base_slot;
    const int m_tiles = s_tile[E], total_tiles = m_tiles * n_tiles;
    // tile -> its expert, first row, rows of the expert from there on, first column (row tiles fastest)
    auto place = [&](int tile, int& e, int& m0, int& m_end, int& n0) {
        const int mt = tile % m_tiles;
        int lo = 0, hi = E;                          // the last expert whose first tile is <= mt (and that has tiles)
        while (hi - lo > 1) {
            const int mid = (lo + hi) >> 1;
            if (s_tile[mid] <= mt) lo = mid; else hi = mid;
        }
        e = lo;
        m0 = s_row[lo] + (mt - s_tile[lo]) * GG_BM;
        m_end = s_row[lo + 1];
        n0 = tile / m_tiles * GG_BN;
    };

    if (warp == 0 && lane == 0) {
        // ---- TMA producer: one continuous ring over all of this CTA's tiles
        int it = 0, issued = 0;
        bool ok = true;
        for (int tile = blockIdx.x; tile < total_tiles && ok; tile += gridDim.x) {
            int e, m0, m_end, n0;
            place(tile, e, m0, m_end, n0);
            for (int kb = 0; kb < nkb; ++kb, ++it) {
                const int s = it % GG_STAGES;
                const uint32_t ph = (it / GG_STAGES) & 1;
                if (!mbar_wait(&empty_bar[s], ph ^ 1, &abort_flag)) {
                    if (!abort_flag) { atomicExch(err, GG_ERR_EMPTY); abort_flag = 1; }
                    ok = false;
                    break;
                }
                unsigned char* a_s = smem + (size_t)s * STAGE_BYTES;
                mbar_expect_tx(&full_bar[s], STAGE_BYTES);
                tma_load_2d(a_s, &tmA, kb * GG_BK, m0, &full_bar[s]);
                tma_load_2d(a_s + A_BYTES, &tmB, kb * GG_BK, e * N + n0, &full_bar[s]);
                issued = it + 1;
            }
        }
        if (abort_flag) {
            // copies already issued must land before the CTA's shared memory goes away
            volatile int no_abort = 0;
            for (int i = max(0, issued - GG_STAGES); i < issued; ++i)
                mbar_wait(&full_bar[i % GG_STAGES], (i / GG_STAGES) & 1, &no_abort);
        }
    } else if (warp == 1 && lane == 0) {
        // ---- MMA issuer
        constexpr uint32_t idesc = idesc_bf16(GG_BM, GG_BN);
        int it = 0, local = 0;
        bool ok = true;
        for (int tile = blockIdx.x; tile < total_tiles && ok; tile += gridDim.x, ++local) {
            const int buf = local & 1;
            if (!mbar_wait(&acc_empty[buf], ((local >> 1) & 1) ^ 1, &abort_flag)) {
                if (!abort_flag) { atomicExch(err, GG_ERR_ACC); abort_flag = 1; }
                break;
            }
            tc_fence_after();
            const uint32_t d_tmem = tmem_base + buf * GG_BN;
            for (int kb = 0; kb < nkb; ++kb, ++it) {
                const int s = it % GG_STAGES;
                const uint32_t ph = (it / GG_STAGES) & 1;
                if (!mbar_wait(&full_bar[s], ph, &abort_flag)) {
                    if (!abort_flag) { atomicExch(err, GG_ERR_FULL); abort_flag = 1; }
                    ok = false;
                    break;
                }
                tc_fence_after();
                const uint32_t a_addr = s_addr(smem + (size_t)s * STAGE_BYTES);
                const uint64_t a_desc = smem_desc_sw128(a_addr), b_desc = smem_desc_sw128(a_addr + A_BYTES);
#pragma unroll
                for (int kk = 0; kk < GG_BK / 16; ++kk)
                    umma_bf16(d_tmem, a_desc + 2 * kk, b_desc + 2 * kk, idesc, (kb | kk) != 0);
                umma_commit(&empty_bar[s]);
            }
            if (ok) umma_commit(&acc_full[buf]);
        }
    } else if (warp >= 2) {
        // ---- epilogue: warp w may touch TMEM lanes 32 * (w % 4) .. + 31
        const int quarter = warp & 3, row = quarter * 32 + lane;
        int local = 0;
        for (int tile = blockIdx.x; tile < total_tiles; tile += gridDim.x, ++local) {
            const int buf = local & 1;
            int e, m0, m_end, n0;
            place(tile, e, m0, m_end, n0);
            const int gm = m0 + row;
            const float scale = row_scale && gm < m_end ? row_scale[gm] : 1.f;
            bool ok = mbar_wait(&acc_full[buf], (local >> 1) & 1, &abort_flag);
            if (!ok && !abort_flag) { atomicExch(err, GG_ERR_ACC); abort_flag = 1; }
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
            const uint32_t taddr = tmem_base + buf * GG_BN + ((uint32_t)(quarter * 32) << 16);
#pragma unroll 1
            for (int c0 = 0; c0 < GG_BN; c0 += 32) {
                uint32_t r[32];
                float v[32];
                tmem_ld32(taddr + c0, r);
                tmem_ld_wait();
                if (c0 + 32 >= GG_BN) {              // all of this thread's TMEM reads of the tile are done
                    tc_fence_before();
                    mbar_arrive(&acc_empty[buf]);
                }
                const int gn = n0 + c0;
                if (gm < m_end && gn < N) {
#pragma unroll
                    for (int j = 0; j < 32; ++j) v[j] = act_apply(scale * __uint_as_float(r[j]), ACT >= 0 ? ACT : act);
                    gg_store32<TC>(C + (size_t)gm * ldc + gn, v, min(32, N - gn));
                }
            }
        }
        pdl_launch_dependents();
    }
    __syncwarp();          // the lanes that had no role meet the elected one: the barrier below wants whole warps
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem_base, 2 * GG_BN);
}

static int gg_tmap(CUtensorMap* map, const void* base, long long rows, int cols, int box_rows) {
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)cols * 2};
    const cuuint32_t box[2] = {GG_BK, (cuuint32_t)box_rows};
    return tmap_encode_bf16(map, base, 2, dims, strides, box);
}

// A [rows, K], B [E * N, K], both bfloat16, contiguous, 16-byte aligned, K a multiple of 8; offsets int32 [E + 1] on the device (null: E is
// 1 and all rows are its); C in float32 or bfloat16, rows ldc apart.  Returns 0, a cudaError_t or 30000 + CUresult of the
// tensor-map encoder.
RLLM_API int rllm_gemm_group(const void* A, const void* B, void* C, int c_dtype, long long ldc, const int* offsets, int E, int rows,
                             int N, int K, const float* row_scale, int act, int* err, cudaStream_t stream) {
    if (rows <= 0 || N <= 0) return 0;
    if (E <= 0 || E > GG_MAX_E || (!offsets && E != 1) || K <= 0 || (K & 7) || ((uintptr_t)A & 15) || ((uintptr_t)B & 15) || !err ||
        ldc < N || (long long)E * N > 0x7fffffffLL)
        return (int)cudaErrorInvalidValue;
    CUtensorMap ta, tb;
    int st = gg_tmap(&ta, A, rows, K, GG_BM);
    if (st) return st;
    st = gg_tmap(&tb, B, (long long)E * N, K, GG_BN);
    if (st) return st;
    constexpr int smem = GG_STAGES * (GG_BM + GG_BN) * GG_BK * 2 + 1024;
    auto run = [&](auto kern, auto* out, int grid) -> int {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return (int)e;
        return rllm_launch(kern, dim3(grid), dim3(GG_THREADS), smem, stream, ta, tb, out, ldc, offsets, E, rows, N, K, row_scale, act, err);
    };
    static int n_sm = 0;
    if (!n_sm) {
        int dev = 0;
        cudaGetDevice(&dev);
        cudaDeviceGetAttribute(&n_sm, cudaDevAttrMultiProcessorCount, dev);
        if (n_sm <= 0) n_sm = 148;
    }
    const long long most = ((long long)(rows + GG_BM - 1) / GG_BM + (offsets ? E : 0)) * ((N + GG_BN - 1) / GG_BN);
    const int grid = (int)(most < n_sm ? most : n_sm);
#define GG_RUN(T)                                                                          \
    if (act == ACT_NONE) return run(gemm_group_kernel<T, ACT_NONE>, (T*)C, grid);          \
    if (act == ACT_RELU2) return run(gemm_group_kernel<T, ACT_RELU2>, (T*)C, grid);        \
    return run(gemm_group_kernel<T, -1>, (T*)C, grid);
    if (c_dtype == RLLM_F32) { GG_RUN(float) }
    GG_RUN(bf16)
#undef GG_RUN
}

TC_DEFINE_WAIT_CONTROLS(rllm_gemm_group)

RLLM_PACKED(rllm_gemm_group)
