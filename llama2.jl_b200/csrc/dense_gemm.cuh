// Matrix products of many-token passes of layer-stack models: bf16 weights x n activation vectors.
//   bf16_gemm_kernel  bf16 activations on the 5th-generation tensor cores (tcgen05 + TMA + tensor memory);
//   f32_gemm_kernel   f32 activations on the CUDA cores in f32 (the 32-bit mode: bf16 weights are exact in f32).
//
// bf16_gemm_kernel: one block = 128 weight rows x BN tokens, times NA weight tiles that share the token tile (NA = 2: the next 128
// rows, or the same rows of a second matrix, so that gate and up of a feed-forward unit meet in one thread).  Weight rows
// are the M dimension: a thread of the epilogue owns one row, and consecutive lanes store consecutive results of a token.
//   warp 0     producer: TMA tiled copies of 64-value wide operand tiles (128-byte swizzle) into a ring of stages
//   warp 1     MMA issue: four K = 16 steps per stage and weight tile into NA x BN columns of tensor memory
//   warps 2-5  epilogue: tcgen05.ld, then what follows the product (dense_epilogue)
// Every mbarrier wait is bounded; a wait that runs out sets the status word, and the block still frees its tensor memory.
#pragma once
#include "dense_ops.cuh"
#include "tcgen05.cuh"

namespace l2b {

constexpr int BG_THREADS = 192, BG_KB = 64, BG_MAX_STAGES = 8;

struct GemmDenseParams {
    int rows;      // weight rows (results per token)
    int n_tok;
    int k;
    int row2;      // distance of the second weight tile's rows (128: next rows; 0: the same rows of the second matrix)
    int stages;
    DenseEpilogue epi;
    int* status;
};
__host__ __device__ constexpr int bg_stage_bytes(int BN, int NA) { return (NA * 128 + BN) * BG_KB * 2; }

template <int BN, int NA>
__global__ void __launch_bounds__(BG_THREADS) bf16_gemm_kernel(const __grid_constant__ GemmDenseParams p, const __grid_constant__ CUtensorMap map_a,
                                                               const __grid_constant__ CUtensorMap map_a2, const __grid_constant__ CUtensorMap map_b) {
    extern __shared__ __align__(1024) uint8_t bg_raw[];
    __shared__ __align__(8) uint64_t s_full[BG_MAX_STAGES], s_free[BG_MAX_STAGES], s_done;
    __shared__ uint32_t s_tmem;
    uint8_t* smem = bg_raw + ((1024u - (smem_u32(bg_raw) & 1023u)) & 1023u);
    constexpr int COLS = NA * BN < 32 ? 32 : NA * BN;
    constexpr int STAGE = bg_stage_bytes(BN, NA);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row0 = (int)blockIdx.x * (p.row2 ? 128 * NA : 128), tok0 = (int)blockIdx.y * BN;
    const int nk = (p.k + BG_KB - 1) / BG_KB;
    if (threadIdx.x == 0) {
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(s_full + i, 1);
            mbar_init(s_free + i, 1);
        }
        mbar_init(&s_done, 1);
        fence_barrier_init();
        fence_proxy_async();
    }
    if (warp == 1) tmem_alloc(&s_tmem, COLS);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;

    if (warp == 0) {
        if (lane == 0) {
            bool ok = true;
            for (int j = 0; j < nk && ok; ++j) {
                const int s = j % p.stages, use = j / p.stages;
                if (use > 0 && !mbar_wait_bounded(s_free + s, (uint32_t)((use - 1) & 1))) {
                    ok = false;
                    break;
                }
                uint8_t* st = smem + (size_t)s * STAGE;
                mbar_arrive_expect_tx(s_full + s, (uint32_t)STAGE);
                tma_load_2d(st, &map_a, j * BG_KB, row0, s_full + s);
                if (NA == 2) tma_load_2d(st + 128 * BG_KB * 2, &map_a2, j * BG_KB, row0 + p.row2, s_full + s);
                tma_load_2d(st + NA * 128 * BG_KB * 2, &map_b, j * BG_KB, tok0, s_full + s);
            }
            if (!ok) {
                atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
                for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = umma_idesc_bf16(128, BN);
            bool ok = true;
            for (int j = 0; j < nk; ++j) {
                const int s = j % p.stages;
                if (!mbar_wait_bounded(s_full + s, (uint32_t)((j / p.stages) & 1))) {
                    ok = false;
                    break;
                }
                tc_fence_after();
                const uint8_t* st = smem + (size_t)s * STAGE;
                const uint8_t* bt = st + NA * 128 * BG_KB * 2;
#pragma unroll
                for (int kk = 0; kk < BG_KB / 16; ++kk)
#pragma unroll
                    for (int a = 0; a < NA; ++a)
                        umma_bf16(tmem + (uint32_t)(a * BN), umma_desc_sw128(st + a * 128 * BG_KB * 2, kk * 32), umma_desc_sw128(bt, kk * 32), idesc,
                                  (j | kk) ? 1u : 0u);
                umma_commit(s_free + s);
            }
            if (ok) umma_commit(&s_done);
            else atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
        }
    } else {
        const int qd = warp & 3;
        const int r = 32 * qd + lane;
        const bool ok = __all_sync(0xffffffffu, mbar_wait_bounded(&s_done, 0u));
        if (!ok) {
            if (lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
        } else {
            tc_fence_after();
            const uint32_t ta = tmem + ((uint32_t)(32 * qd) << 16);
            const bool dual = NA == 2 && p.row2 == 0;
#pragma unroll 1
            for (int c = 0; c < BN; c += 32) {
                if (tok0 + c >= p.n_tok) break;
                __syncwarp();
                float v[32], v2[32];
                tmem_ld32f(ta + (uint32_t)c, v);
                if (NA == 2) tmem_ld32f(ta + (uint32_t)(BN + c), v2);
                const int n = min(32, p.n_tok - tok0 - c);
                if (p.epi.kind == DE_STORE_T && n == 32 && (p.epi.ld & 7) == 0) {  // a thread's 32 tokens are contiguous
#pragma unroll
                    for (int a = 0; a < NA; ++a) {
                        const int f = row0 + a * 128 + r;
                        if (f >= p.rows) continue;
                        bf16* dst = static_cast<bf16*>(p.epi.act) + (size_t)f * p.epi.ld + tok0 + c;
#pragma unroll
                        for (int k = 0; k < 32; k += 2) {
                            const float x0 = a ? v2[k] : v[k], x1 = a ? v2[k + 1] : v[k + 1];
                            *reinterpret_cast<__nv_bfloat162*>(dst + k) = __floats2bfloat162_rn(x0, x1);
                        }
                    }
                    continue;
                }
                const int f = row0 + r;
#pragma unroll
                for (int k = 0; k < 32; ++k)
                    if (k < n && f < p.rows) dense_epilogue<bf16>(p.epi, tok0 + c + k, f, v[k], NA == 2 ? v2[k] : 0.f);
                if (NA == 2 && !dual) {
#pragma unroll
                    for (int k = 0; k < 32; ++k)
                        if (k < n && f + 128 < p.rows) dense_epilogue<bf16>(p.epi, tok0 + c + k, f + 128, v2[k], 0.f);
                }
            }
        }
    }
    // every path ends here; the tensor memory is freed by the warp that allocated it
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, COLS);
}

// ---- f32 --------------------------------------------------------------------------------------------
// One block = 64 weight rows x 64 tokens, thread = 4 x 4 results; DUAL: two weight rows per result (rows f and f of the second
// matrix).  x [n_tok][ldx] f32, w rows wstride elements apart.
struct GemmF32Params {
    const bf16* w;
    const bf16* w2;
    size_t wstride;
    const float* x;
    int ldx;
    int rows, n_tok, k;
    DenseEpilogue epi;
};
template <bool DUAL>
__global__ void __launch_bounds__(256) f32_gemm_kernel(const __grid_constant__ GemmF32Params p) {
    constexpr int T = 64, KB = 16;
    __shared__ float sw[DUAL ? 2 : 1][KB][T + 4], sx[KB][T + 4];
    const int tid = threadIdx.x, fr = tid & 15, tr = tid >> 4;
    const int f0 = (int)blockIdx.x * T, n0 = (int)blockIdx.y * T;
    float acc[4][4], acc2[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = acc2[i][j] = 0.f;
    for (int k0 = 0; k0 < p.k; k0 += KB) {
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int i = tid + u * 256, k = i & 15, r = i >> 4;
            const bool kin = k0 + k < p.k;
            sw[0][k][r] = kin && f0 + r < p.rows ? __bfloat162float(p.w[(size_t)(f0 + r) * p.wstride + k0 + k]) : 0.f;
            if (DUAL) sw[DUAL ? 1 : 0][k][r] = kin && f0 + r < p.rows ? __bfloat162float(p.w2[(size_t)(f0 + r) * p.wstride + k0 + k]) : 0.f;
            sx[k][r] = kin && n0 + r < p.n_tok ? p.x[(size_t)(n0 + r) * p.ldx + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < KB; ++k) {
            float w[4], w2[4], x[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                w[i] = sw[0][k][fr + 16 * i];
                w2[i] = DUAL ? sw[DUAL ? 1 : 0][k][fr + 16 * i] : 0.f;
                x[i] = sx[k][tr + 16 * i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][j] = fmaf(w[i], x[j], acc[i][j]);
                    if (DUAL) acc2[i][j] = fmaf(w2[i], x[j], acc2[i][j]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int f = f0 + fr + 16 * i, t = n0 + tr + 16 * j;
            if (f < p.rows && t < p.n_tok) dense_epilogue<float>(p.epi, t, f, acc[i][j], acc2[i][j]);
        }
}

}  // namespace l2b
