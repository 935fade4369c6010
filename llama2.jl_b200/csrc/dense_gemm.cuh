// Matrix products of many-token passes of layer-stack models: bf16 weights x n activation vectors.
//   bf16_gemm_kernel  bf16 activations on the 5th-generation tensor cores (tcgen05 + TMA + tensor memory);
//   f32_gemm_kernel   f32 activations on the CUDA cores in f32 (the 32-bit mode: bf16 weights are exact in f32).
//
// bf16_gemm_kernel: a tile = 128 weight rows x BN tokens, times NA weight tiles that share the token tile (NA = 2: the next 128
// rows, or the same rows of a second matrix, so that gate and up of a feed-forward unit meet in one thread).  Weight rows
// are the M dimension: a thread of the epilogue owns one row, and consecutive lanes store consecutive results of a token.
// Persistent: one block per SM walks tiles (token tiles innermost, so that a weight tile is read from L2 after its first use), with
// two sets of NA x BN accumulator columns in tensor memory, so that a tile's epilogue runs beside the next tile's products.
//   warp 0     producer: TMA tiled copies of 64-value wide operand tiles (128-byte swizzle) into a ring of stages
//   warp 1     MMA issue: four K = 16 steps per stage and weight tile
//   warps 2-5  epilogue: tcgen05.ld, then what follows the product
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
    int mtiles, ntiles;
    int stages;
    DenseEpilogue epi;
    int* status;
};
__host__ __device__ constexpr int bg_stage_bytes(int BN, int NA) { return (NA * 128 + BN) * BG_KB * 2; }

// 32 consecutive tokens (n of them exist) of one result row.  What has to be read is read for all of them first.
template <int KIND>
__device__ __forceinline__ void epilogue_tokens(const DenseEpilogue& e, int t0, int n, int f, const float (&v)[32], const float (&v2)[32]) {
    bf16* const act = static_cast<bf16*>(e.act);
    if (KIND == DE_RESIDUAL) {
        float r[32];
#pragma unroll
        for (int k = 0; k < 32; ++k) r[k] = e.y[(size_t)(t0 + min(k, n - 1)) * e.ld + f];
#pragma unroll
        for (int k = 0; k < 32; ++k)
            if (k < n) e.y[(size_t)(t0 + k) * e.ld + f] = r[k] + v[k];
    } else if (KIND == DE_SIDE) {
        float r[32];
#pragma unroll
        for (int k = 0; k < 32; ++k) r[k] = side_value(e, t0 + min(k, n - 1), f);
#pragma unroll
        for (int k = 0; k < 32; ++k)
            if (k < n) put(act + (size_t)(t0 + k) * e.ld + f, gelu_tanh(v[k]) * r[k]);
    } else if (KIND == DE_STORE_T && n == 32 && (e.ld & 7) == 0) {  // a thread's 32 tokens are contiguous
        uint4* dst = reinterpret_cast<uint4*>(act + (size_t)f * e.ld + t0);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            uint32_t w[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const __nv_bfloat162 pk = __floats2bfloat162_rn(v[8 * k + 2 * i], v[8 * k + 2 * i + 1]);
                w[i] = *reinterpret_cast<const uint32_t*>(&pk);
            }
            dst[k] = make_uint4(w[0], w[1], w[2], w[3]);
        }
    } else {
        const float bias = KIND == DE_AFFINE && e.bias ? __ldg(e.bias + f) : 0.f;
#pragma unroll
        for (int k = 0; k < 32; ++k) {
            if (k >= n) continue;
            if (KIND == DE_STORE) e.y[(size_t)(t0 + k) * e.ld + f] = v[k];
            if (KIND == DE_AFFINE) e.y[(size_t)(t0 + k) * e.ld + f] = fmaf(v[k], e.mul, bias);
            if (KIND == DE_SWIGLU) put(act + (size_t)(t0 + k) * e.ld + f, silu(v[k]) * v2[k]);
            if (KIND == DE_GEGLU) put(act + (size_t)(t0 + k) * e.ld + f, gelu_tanh(v[k]) * v2[k]);
            if (KIND == DE_STORE_ACT) put(act + (size_t)(t0 + k) * e.ld + f, v[k]);
            if (KIND == DE_STORE_T) put(act + (size_t)f * e.ld + t0 + k, v[k]);
        }
    }
}
__device__ __forceinline__ void epilogue_tokens(const DenseEpilogue& e, int t0, int n, int f, const float (&v)[32], const float (&v2)[32]) {
    switch (e.kind) {
        case DE_RESIDUAL: epilogue_tokens<DE_RESIDUAL>(e, t0, n, f, v, v2); break;
        case DE_GEGLU: epilogue_tokens<DE_GEGLU>(e, t0, n, f, v, v2); break;
        case DE_SWIGLU: epilogue_tokens<DE_SWIGLU>(e, t0, n, f, v, v2); break;
        case DE_AFFINE: epilogue_tokens<DE_AFFINE>(e, t0, n, f, v, v2); break;
        case DE_SIDE: epilogue_tokens<DE_SIDE>(e, t0, n, f, v, v2); break;
        case DE_STORE_ACT: epilogue_tokens<DE_STORE_ACT>(e, t0, n, f, v, v2); break;
        case DE_STORE_T: epilogue_tokens<DE_STORE_T>(e, t0, n, f, v, v2); break;
        default: epilogue_tokens<DE_STORE>(e, t0, n, f, v, v2); break;
    }
}

template <int BN, int NA>
__global__ void __launch_bounds__(BG_THREADS) bf16_gemm_kernel(const __grid_constant__ GemmDenseParams p, const __grid_constant__ CUtensorMap map_a,
                                                               const __grid_constant__ CUtensorMap map_a2, const __grid_constant__ CUtensorMap map_b) {
    extern __shared__ __align__(1024) uint8_t bg_raw[];
    __shared__ __align__(8) uint64_t s_full[BG_MAX_STAGES], s_free[BG_MAX_STAGES], s_acc[2], s_acc_free[2];
    __shared__ uint32_t s_tmem;
    uint8_t* smem = bg_raw + ((1024u - (smem_u32(bg_raw) & 1023u)) & 1023u);
    constexpr int COLS = 2 * NA * BN;  // 64 .. 512, a power of two
    constexpr int STAGE = bg_stage_bytes(BN, NA);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int tile_rows = p.row2 ? 128 * NA : 128;
    const int nk = (p.k + BG_KB - 1) / BG_KB, tiles = p.mtiles * p.ntiles;
    if (threadIdx.x == 0) {
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(s_full + i, 1);
            mbar_init(s_free + i, 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(s_acc + i, 1);
            mbar_init(s_acc_free + i, 4);
        }
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
            int s = 0, use = 0;
            for (int tile = (int)blockIdx.x; tile < tiles && ok; tile += (int)gridDim.x) {
                const int row0 = tile / p.ntiles * tile_rows, tok0 = tile % p.ntiles * BN;
                for (int j = 0; j < nk; ++j) {
                    if (use > 0 && !mbar_wait_bounded(s_free + s, (uint32_t)((use - 1) & 1))) {
                        ok = false;
                        break;
                    }
                    uint8_t* st = smem + (size_t)s * STAGE;
                    mbar_arrive_expect_tx(s_full + s, (uint32_t)STAGE);
                    tma_load_2d(st, &map_a, j * BG_KB, row0, s_full + s);
                    if (NA == 2) tma_load_2d(st + 128 * BG_KB * 2, &map_a2, j * BG_KB, row0 + p.row2, s_full + s);
                    tma_load_2d(st + NA * 128 * BG_KB * 2, &map_b, j * BG_KB, tok0, s_full + s);
                    if (++s == p.stages) s = 0, ++use;
                }
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
            int s = 0, n = 0;
            uint32_t par = 0;
            for (int tile = (int)blockIdx.x; tile < tiles && ok; tile += (int)gridDim.x, ++n) {
                const int buf = n & 1;
                if (n >= 2 && !mbar_wait_bounded(s_acc_free + buf, (uint32_t)(((n - 2) >> 1) & 1))) {
                    ok = false;
                    break;
                }
                tc_fence_after();
                for (int j = 0; j < nk; ++j) {
                    if (!mbar_wait_bounded(s_full + s, par)) {
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
                            umma_bf16(tmem + (uint32_t)((buf * NA + a) * BN), umma_desc_sw128(st + a * 128 * BG_KB * 2, kk * 32), umma_desc_sw128(bt, kk * 32), idesc,
                                      (j | kk) ? 1u : 0u);
                    umma_commit(s_free + s);
                    if (++s == p.stages) s = 0, par ^= 1u;
                }
                if (ok) umma_commit(s_acc + buf);
            }
            if (!ok) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
        }
    } else {
        const int qd = warp & 3;
        const int r = 32 * qd + lane;
        const bool dual = NA == 2 && p.row2 == 0;
        int n = 0;
        bool ok = true;
        for (int tile = (int)blockIdx.x; tile < tiles; tile += (int)gridDim.x, ++n) {
            const int buf = n & 1, f = tile / p.ntiles * tile_rows + r, tok0 = tile % p.ntiles * BN;
            if (!__all_sync(0xffffffffu, mbar_wait_bounded(s_acc + buf, (uint32_t)((n >> 1) & 1)))) {
                ok = false;
                break;
            }
            tc_fence_after();
            const uint32_t ta = tmem + ((uint32_t)(32 * qd) << 16) + (uint32_t)(buf * NA * BN);
#pragma unroll 1
            for (int c = 0; c < BN; c += 32) {
                const int left = min(32, p.n_tok - tok0 - c);
                if (left <= 0) break;
                __syncwarp();
                float v[32], v2[32];
                tmem_ld32f(ta + (uint32_t)c, v);
                if (NA == 2) tmem_ld32f(ta + (uint32_t)(BN + c), v2);
                if (f < p.rows) epilogue_tokens(p.epi, tok0 + c, left, f, v, v2);
                if (NA == 2 && !dual && f + 128 < p.rows) epilogue_tokens(p.epi, tok0 + c, left, f + 128, v2, v2);
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(s_acc_free + buf);
        }
        if (!ok && lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
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
