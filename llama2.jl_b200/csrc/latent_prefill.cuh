// Latent attention of a long portion of a prompt, on the 5th-generation tensor cores: the keys and values of every position are
// expanded from the cached latents by two GEMMs (K = W_uk c as [position][head][dp], V = W_uv c transposed as
// [head][vp][position]), then this kernel runs softmax attention over 128-query x 128-key tiles.  The rotated key part is read from
// the cache, shared by all heads.
//
// One block = 128 queries of one head:
//   warp 0     producer: TMA tiled copies of Q (once), [K | kr] and V per key tile
//   warp 1     MMA issue: S_j = Q K_j^T into one of two 128-column buffers of tensor memory, one tile ahead of O += P_j V_j
//   warps 2-9  two threads per query, each with half of the tile's keys: scores from tensor memory, scale, causal mask, running
//              maximum (shared between the two) and sum in f32 (exp2 domain); P_j as bf16 into shared memory in operand
//              layout.  The scores are read twice, for the maximum and for the exponentials, in short loops: with all of them in
//              registers the unrolled code no longer fits the instruction cache.  O is rescaled in tensor memory only when a row's maximum has
//              grown by more than 2^8 since it was last taken; the end divides by sum + exp(sink), applies the output gate
//              and stores the operand of the output projection.
// Every mbarrier wait is bounded, as in the GEMM.
#pragma once
#include "latent_attention.cuh"
#include "tcgen05.cuh"

namespace l2b {

constexpr int LP_TILE = 128, LP_WARPS = 8, LP_THREADS = 64 + LP_WARPS * 32, LP_SUB = 128 * 128;  // bytes of a 128-row x 64-value operand tile

struct LatentPrefillParams {
    int n, pos0;              // queries at positions pos0 .. pos0 + n - 1
    int dim, rot, vdim;
    int dp, dq, vp;           // stored dims per head: K; Q (unrotated then rotated, each rounded up to 16); V rows
    int kstages;
    float scale2;
    const float* sink;
    const float* gate;        // gate of (row, head, v) at gate[row * ld + head * vdim + v]
    int ld;
    bf16* out;                // [n][ldo]
    int ldo;
    int* status;
};
struct LpSmem {
    int q, k, v, p, total, kbytes, vbytes;
};
__host__ __device__ inline LpSmem lp_smem_layout(int dim, int rot, int vp, int kstages) {
    LpSmem s;
    const int pieces = (dim + 63) / 64 + (rot + 63) / 64;
    s.kbytes = pieces * LP_SUB;
    s.vbytes = 2 * vp * 128;
    s.vbytes = (s.vbytes + 1023) & ~1023;
    s.q = 0;
    s.k = s.q + pieces * LP_SUB;
    s.v = s.k + kstages * s.kbytes;
    s.p = s.v + s.vbytes;
    s.total = s.p + 2 * LP_SUB;
    return s;
}

__global__ void __launch_bounds__(LP_THREADS) latent_prefill_kernel(const __grid_constant__ LatentPrefillParams p, const __grid_constant__ CUtensorMap map_q,
                                                                    const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_kr,
                                                                    const __grid_constant__ CUtensorMap map_v) {
    extern __shared__ __align__(1024) uint8_t lp_raw[];
    __shared__ __align__(8) uint64_t s_q, s_k[2], s_kfree[2], s_v, s_s[2], s_sfree[2], s_p, s_o;
    __shared__ uint32_t s_tmem;
    __shared__ float s_row[2][2][LP_TILE];  // [tile parity][half][query]: the halves' maxima (at the end: sums)
    uint8_t* smem = lp_raw + ((1024u - (smem_u32(lp_raw) & 1023u)) & 1023u);
    const LpSmem L = lp_smem_layout(p.dim, p.rot, p.vp, p.kstages);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = (int)blockIdx.y, q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * LP_TILE;  // longest tiles first
    const int nt = (p.pos0 + min(p.n, q0 + LP_TILE) - 1) / LP_TILE + 1;                    // key tiles
    const int nd = (p.dim + 63) / 64, nr = (p.rot + 63) / 64;
    if (threadIdx.x == 0) {
        mbar_init(&s_q, 1);
        mbar_init(&s_v, 1);
        mbar_init(&s_p, LP_WARPS);
        mbar_init(&s_o, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(s_k + i, 1);
            mbar_init(s_kfree + i, 1);
            mbar_init(s_s + i, 1);
            mbar_init(s_sfree + i, LP_WARPS);
        }
        fence_barrier_init();
        fence_proxy_async();
    }
    if (warp == 1) tmem_alloc(&s_tmem, 512);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem, tmem_o = tmem + 256;

    if (warp == 0) {
        if (lane == 0) {
            bool ok = true;
            mbar_arrive_expect_tx(&s_q, (uint32_t)((nd + nr) * LP_SUB));
            for (int i = 0; i < nd; ++i) tma_load_2d(smem + L.q + i * LP_SUB, &map_q, h * p.dq + 64 * i, q0, &s_q);
            for (int i = 0; i < nr; ++i) tma_load_2d(smem + L.q + (nd + i) * LP_SUB, &map_q, h * p.dq + p.dp + 64 * i, q0, &s_q);
            for (int j = 0; j < nt && ok; ++j) {
                const int s = p.kstages == 2 ? (j & 1) : 0, use = p.kstages == 2 ? j >> 1 : j;
                if (use > 0 && !mbar_wait_bounded(s_kfree + s, (uint32_t)((use - 1) & 1))) {
                    ok = false;
                    break;
                }
                uint8_t* kt = smem + L.k + s * L.kbytes;
                mbar_arrive_expect_tx(s_k + s, (uint32_t)((nd + nr) * LP_SUB));
                for (int i = 0; i < nd; ++i) tma_load_2d(kt + i * LP_SUB, &map_k, h * p.dp + 64 * i, j * LP_TILE, s_k + s);
                for (int i = 0; i < nr; ++i) tma_load_2d(kt + (nd + i) * LP_SUB, &map_kr, 64 * i, j * LP_TILE, s_k + s);
                if (j > 0 && !mbar_wait_bounded(&s_o, (uint32_t)((j - 1) & 1))) {  // P V of the tile before has read V
                    ok = false;
                    break;
                }
                mbar_arrive_expect_tx(&s_v, (uint32_t)(2 * p.vp * 128));
                tma_load_2d(smem + L.v, &map_v, j * LP_TILE, h * p.vp, &s_v);
                tma_load_2d(smem + L.v + p.vp * 128, &map_v, j * LP_TILE + 64, h * p.vp, &s_v);
            }
            if (!ok) {
                atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
                for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_s = umma_idesc_bf16(128, 128), idesc_o = umma_idesc_bf16(128, p.vp);
            bool ok = mbar_wait_bounded(&s_q, 0u);
            auto pv = [&](int j) {
                if (!mbar_wait_bounded(&s_v, (uint32_t)(j & 1)) || !mbar_wait_bounded(&s_p, (uint32_t)(j & 1))) {
                    ok = false;
                    return;
                }
                tc_fence_after();
                for (int t = 0; t < 2; ++t)
                    for (int kk = 0; kk < 4; ++kk)
                        umma_bf16(tmem_o, umma_desc_sw128(smem + L.p + t * LP_SUB, kk * 32), umma_desc_sw128(smem + L.v + t * p.vp * 128, kk * 32), idesc_o,
                                  (j | t | kk) ? 1u : 0u);
                umma_commit(&s_o);
            };
            for (int j = 0; j < nt && ok; ++j) {
                const int s = p.kstages == 2 ? (j & 1) : 0, use = p.kstages == 2 ? j >> 1 : j, b = j & 1;
                if (!mbar_wait_bounded(s_k + s, (uint32_t)(use & 1)) || (j >= 2 && !mbar_wait_bounded(s_sfree + b, (uint32_t)(((j - 2) >> 1) & 1)))) {
                    ok = false;
                    break;
                }
                tc_fence_after();
                const uint8_t* kt = smem + L.k + s * L.kbytes;
                uint32_t acc = 0u;
                for (int i = 0; i < nd + nr; ++i) {
                    const int left = i < nd ? p.dim - 64 * i : p.rot - 64 * (i - nd);
                    for (int kk = 0; kk < 4 && 16 * kk < left; ++kk, acc = 1u)
                        umma_bf16(tmem + (uint32_t)(b * 128), umma_desc_sw128(smem + L.q + i * LP_SUB, kk * 32), umma_desc_sw128(kt + i * LP_SUB, kk * 32), idesc_s, acc);
                }
                umma_commit(s_s + b);
                umma_commit(s_kfree + s);
                if (j > 0) pv(j - 1);
            }
            if (ok) pv(nt - 1);
            if (!ok) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
        }
    } else {
        const int qd = warp & 3, half = (warp - 2) >> 2, r = 32 * qd + lane;
        const uint32_t lane_off = (uint32_t)(32 * qd) << 16;
        const int qi = q0 + r, qpos = p.pos0 + qi;
        float m = -INFINITY, l = 0.f;
        bool ok = true;
        for (int j = 0; j < nt; ++j) {
            const int b = j & 1;
            if (ok && !__all_sync(0xffffffffu, mbar_wait_bounded(s_s + b, (uint32_t)((j >> 1) & 1)))) ok = false;
            tc_fence_after();
            const uint32_t ts = tmem + lane_off + (uint32_t)(b * 128 + half * 64);
            const int lim = qpos - j * LP_TILE - half * 64;                       // keys 0 .. lim of this half are seen
            const bool masked = j * LP_TILE + LP_TILE - 1 > p.pos0 + q0;           // (the last tiles only)
            float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll 1
            for (int c = 0; c < 64; c += 32) {
                float s[32];
                tmem_ld32f(ts + (uint32_t)c, s);
                if (masked) {
#pragma unroll
                    for (int k = 0; k < 32; ++k)
                        if (c + k > lim) s[k] = -INFINITY;
                }
#pragma unroll
                for (int k = 0; k < 32; ++k) m4[k & 3] = fmaxf(m4[k & 3], s[k]);
            }
            s_row[b][half][r] = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
            partial_sync_2(LP_WARPS * 32);
            const float mx = fmaxf(s_row[b][0][r], s_row[b][1][r]) * p.scale2;  // (scale2 > 0; key 0 is seen, so the first is finite)
            if (ok && j > 0 && !__all_sync(0xffffffffu, mbar_wait_bounded(&s_o, (uint32_t)((j - 1) & 1)))) ok = false;  // P and O are free
            tc_fence_after();
            if (j == 0) {
                m = mx;
            } else if (__any_sync(0xffffffffu, mx > m + 8.f)) {  // (the same decision in both halves)
                const float mn = mx > m + 8.f ? mx : m, corr = fast_exp2(m - mn);
                l *= corr;
                m = mn;
#pragma unroll 1
                for (int c = 32 * half; c < p.vp; c += 64) {
                    float o[32];
                    tmem_ld32f(tmem_o + lane_off + (uint32_t)c, o);
#pragma unroll
                    for (int k = 0; k < 32; ++k) o[k] *= corr;
                    tmem_st32f(tmem_o + lane_off + (uint32_t)c, o);
                }
            }
            float l4[4] = {0.f, 0.f, 0.f, 0.f};
            uint8_t* const pr = smem + L.p + half * LP_SUB + r * 128;
#pragma unroll 1
            for (int c = 0; c < 64; c += 32) {
                float s[32];
                tmem_ld32f(ts + (uint32_t)c, s);
#pragma unroll
                for (int k = 0; k < 32; ++k) s[k] = fast_exp2(fmaf(s[k], p.scale2, -m));
                if (masked) {
#pragma unroll
                    for (int k = 0; k < 32; ++k)
                        if (c + k > lim) s[k] = 0.f;
                }
#pragma unroll
                for (int k = 0; k < 32; ++k) l4[k & 3] += s[k];
#pragma unroll
                for (int g = 0; g < 4; ++g) {  // 8 keys = one 16-byte chunk of the operand row, chunk index xor row (128-byte swizzle)
                    uint32_t w[4];
#pragma unroll
                    for (int k = 0; k < 4; ++k) {
                        const __nv_bfloat162 pk = __floats2bfloat162_rn(s[8 * g + 2 * k], s[8 * g + 2 * k + 1]);
                        w[k] = *reinterpret_cast<const uint32_t*>(&pk);
                    }
                    *reinterpret_cast<uint4*>(pr + (((c >> 3) + g) ^ (r & 7)) * 16) = make_uint4(w[0], w[1], w[2], w[3]);
                }
            }
            l += (l4[0] + l4[1]) + (l4[2] + l4[3]);
            fence_proxy_async();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) {
                mbar_arrive(s_sfree + b);
                mbar_arrive(&s_p);
            }
        }
        if (ok && !__all_sync(0xffffffffu, mbar_wait_bounded(&s_o, (uint32_t)((nt - 1) & 1)))) ok = false;
        s_row[nt & 1][half][r] = l;
        partial_sync_2(LP_WARPS * 32);
        if (!ok) {
            if (lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
        } else {
            tc_fence_after();
            l = s_row[nt & 1][0][r] + s_row[nt & 1][1][r];
            const float inv = 1.f / (l + exp2f(__ldg(p.sink + h) * 1.4426950408889634f - m));  // the sink: a term of the denominator only
            bf16* out = p.out + (size_t)qi * p.ldo + h * p.vdim;
            const bool wide = ((p.vdim | p.ldo) & 7) == 0;
            // gates of this warp's 32 queries, 32 values at a time, through the shared memory that held Q and K (all products are done)
            float* const sg = reinterpret_cast<float*>(smem + L.q) + (warp - 2) * (32 * 33);
#pragma unroll 1
            for (int c = 32 * half; c < p.vdim; c += 64) {
                float o[32];
                __syncwarp();
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    const int t = q0 + 32 * qd + i;
                    o[i] = t < p.n && c + lane < p.vdim ? __ldg(p.gate + (size_t)t * p.ld + h * p.vdim + c + lane) : 0.f;
                }
#pragma unroll
                for (int i = 0; i < 32; ++i) sg[i * 33 + lane] = sigmoid(o[i]);
                __syncwarp();
                tmem_ld32f(tmem_o + lane_off + (uint32_t)c, o);
                const int nv = qi < p.n ? p.vdim - c : 0;  // values of this query to store
#pragma unroll
                for (int k = 0; k < 32; ++k) o[k] *= inv * sg[lane * 33 + k];
                if (wide) {
#pragma unroll
                    for (int g = 0; g < 4; ++g)
                        if (8 * g < nv) {
                            uint32_t w[4];
#pragma unroll
                            for (int k = 0; k < 4; ++k) {
                                const __nv_bfloat162 pk = __floats2bfloat162_rn(o[8 * g + 2 * k], o[8 * g + 2 * k + 1]);
                                w[k] = *reinterpret_cast<const uint32_t*>(&pk);
                            }
                            *reinterpret_cast<uint4*>(out + c + 8 * g) = make_uint4(w[0], w[1], w[2], w[3]);
                        }
                } else {
#pragma unroll
                    for (int k = 0; k < 32; ++k)
                        if (k < nv) put(out + c + k, o[k]);
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, 512);
}

// Query operand of the kernel above: [row][head][dq] = unrotated part rounded up to 16 (zeros), rotated part rounded up to 16.
// Grid (rows, heads); a thread makes two values.
__global__ void __launch_bounds__(128) latent_queries_kernel(const float* __restrict__ qdg, int ld, const float2* __restrict__ rope, int pos0, LatentShape s, int dq,
                                                            bf16* __restrict__ out) {
    const int row = (int)blockIdx.x, h = (int)blockIdx.y;
    const float2* cs = rope + (size_t)(pos0 + row) * (s.rdims >> 1);
    const float* q = qdg + (size_t)row * ld + h * (s.dim + s.rot);
    bf16* dst = out + ((size_t)row * s.heads + h) * dq;
    for (int d = 2 * threadIdx.x; d < dq; d += 256) {
        float v0 = 0.f, v1 = 0.f;
        if (d < s.dp) {
            v0 = d < s.dim ? q[d] : 0.f;
            v1 = d + 1 < s.dim ? q[d + 1] : 0.f;
        } else {
            const int r = d - s.dp;  // even: a whole pair, or two unrotated values
            if (r < s.rot) {
                v0 = rotary_element(r, s.rdims, cs, [&](int j) { return q[s.dim + j]; });
                v1 = rotary_element(r + 1, s.rdims, cs, [&](int j) { return q[s.dim + j]; });
            }
        }
        *reinterpret_cast<__nv_bfloat162*>(dst + d) = __floats2bfloat162_rn(v0, v1);
    }
}

}  // namespace l2b
