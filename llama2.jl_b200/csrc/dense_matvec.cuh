// Matrix-vector product of the decode path of layer-stack models: bf16 weights, f32 activations and accumulation.  The counterpart
// of fused_matvec_kernel for matrices stored in bf16.
//
// One block per SM, 16 warps, every block a contiguous range of rows.
//   before the wait on the previous kernel (programmatic dependent launch): the block's rows are prefetched into L2 with a few
//       bulk prefetches and every warp loads its first step of weights into registers -- weights are constants;
//   prologue : the input vector goes to shared memory as f32, after the pending changes of the residual stream (the normalised
//       per-layer token input, the step vector of a loop pass) and the norm; block 0 writes the changed residual stream back
//       to its other buffer, because the other blocks still read this one;
//   weights  : a warp takes items of 4 rows x a range of 256-value chunks, the next step's loads in flight during the arithmetic;
//       four row sums are reduced over the lanes together (6 shuffles);
//   epilogue : the range sums of a row are added in a fixed order by one thread: store | residual add | gelu(gate) * up (rows
//       2u and 2u+1 of an interleaved matrix) | gelu * token embedding | logits with the block's first maximum.
#pragma once
#include "dense_ops.cuh"

namespace l2b {

constexpr int DMV_WARPS = 16, DMV_THREADS = DMV_WARPS * 32, DMV_ROWS = 4;

struct DmvParams {
    const bf16* w;          // [rows][kp], kp a multiple of 8
    int kp, k;              // stored and logical row length
    int unit;               // rows per result: 1, or 2 (interleaved gate / up)
    int per_lo, per_rem;    // results of block b: per_lo + (b < per_rem), contiguous
    int nchunk;             // 256-value chunks per row
    int nslice, cps;        // a row is summed in nslice ranges of cps chunks
    int prefetch;           // bytes of the block's rows to prefetch into L2
    const float* x;         // input vector [k]
    ResidualUpdate upd;
    float* x_out;           // block 0 writes the updated vector here (null: no update)
    NormParams norm;
    DenseEpilogue epi;      // t = 0
    float* amax_val;        // DE_LOGITS: per block
    int* amax_idx;
};
inline size_t dmv_smem_bytes(const DmvParams& p) {
    const int rows = p.unit * (p.per_lo + (p.per_rem ? 1 : 0));
    return ((size_t)p.nchunk * 256 + (size_t)((rows + DMV_ROWS - 1) / DMV_ROWS * DMV_ROWS) * p.nslice) * 4;
}

__global__ void __launch_bounds__(DMV_THREADS, 2) dense_matvec_kernel(const __grid_constant__ DmvParams p) {
    extern __shared__ __align__(16) float dmv_smem[];
    __shared__ float s_red[DMV_WARPS];
    __shared__ int s_idx[DMV_WARPS];
    float* const xf = dmv_smem;
    float* const part = dmv_smem + p.nchunk * 256;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    pdl_launch_dependents();
    const int b = (int)blockIdx.x;
    const int u0 = b * p.per_lo + min(b, p.per_rem), nu = p.per_lo + (b < p.per_rem ? 1 : 0);
    const int nr = nu * p.unit;
    const bf16* const wb = p.w + (size_t)u0 * p.unit * p.kp;

    if (warp == DMV_WARPS - 1) {
        const size_t total = min((size_t)p.prefetch, (size_t)nr * p.kp * 2);
        for (size_t o = (size_t)lane * 4096; o < total; o += 32 * 4096)
            asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(reinterpret_cast<const char*>(wb) + o), "r"((uint32_t)min((size_t)4096, total - o)) : "memory");
    }
    const int nitems = (nr + DMV_ROWS - 1) / DMV_ROWS * p.nslice;
    int it = warp, g = 0, c = 0, c1 = 0;
    uint4 nxt[DMV_ROWS];
    auto begin_item = [&]() {
        g = it / p.nslice;
        c = (it - g * p.nslice) * p.cps;
        c1 = min(p.nchunk, c + p.cps);
    };
    auto load = [&]() {
        const int e = c * 256 + lane * 8;
        const bf16* src = wb + (size_t)g * DMV_ROWS * p.kp + e;
        const int lim = nr - 1 - g * DMV_ROWS;
#pragma unroll
        for (int i = 0; i < DMV_ROWS; ++i) {
            nxt[i] = make_uint4(0u, 0u, 0u, 0u);
            if (e < p.kp) nxt[i] = __ldg(reinterpret_cast<const uint4*>(src + (size_t)min(i, lim) * p.kp));
        }
    };
    bool have = it < nitems;
    if (have) {
        begin_item();
        load();
    }

    pdl_wait();
    {
        constexpr int U = 4;
        const int k = p.k, kc = p.nchunk * 256;
        float scale = 0.f;
        if (p.upd.y) {
            float ss = 0.f;
            for (int i0 = threadIdx.x; i0 < k; i0 += U * DMV_THREADS) {
                float v[U];
#pragma unroll
                for (int u = 0; u < U; ++u) v[u] = i0 + u * DMV_THREADS < k ? __ldcg(p.upd.y + i0 + u * DMV_THREADS) : 0.f;
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    ss = fmaf(v[u], v[u], ss);
                    if (i0 + u * DMV_THREADS < k) xf[i0 + u * DMV_THREADS] = v[u];
                }
            }
            scale = 1.f / sqrtf(block_sum_all<DMV_WARPS>(ss, s_red) / (float)k + p.upd.eps);
        }
        for (int i0 = threadIdx.x; i0 < kc; i0 += U * DMV_THREADS) {
            float v[U];
#pragma unroll
            for (int u = 0; u < U; ++u) v[u] = i0 + u * DMV_THREADS < k ? __ldcg(p.x + i0 + u * DMV_THREADS) : 0.f;
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * DMV_THREADS;
                if (i < k) {
                    float t = v[u];
                    if (p.upd.y) t = fmaf(xf[i] * scale, __ldg(p.upd.side_w + i), t);
                    if (p.upd.step) t += __ldg(p.upd.step + i);
                    if (p.x_out && b == 0) p.x_out[i] = t;
                    xf[i] = apply_norm(p.norm, t, i);
                } else if (i < kc) {
                    xf[i] = 0.f;
                }
            }
        }
    }
    __syncthreads();

    float acc[DMV_ROWS];
#pragma unroll
    for (int i = 0; i < DMV_ROWS; ++i) acc[i] = 0.f;
    while (have) {
        uint4 cur[DMV_ROWS];
#pragma unroll
        for (int i = 0; i < DMV_ROWS; ++i) cur[i] = nxt[i];
        const int ccur = c, itcur = it, gcur = g;
        const bool last = c + 1 == c1;
        if (last) {
            it += DMV_WARPS;
            have = it < nitems;
            if (have) begin_item();
        } else {
            ++c;
        }
        if (have) load();
        const float4 xa = *reinterpret_cast<const float4*>(xf + ccur * 256 + lane * 8), xb = *reinterpret_cast<const float4*>(xf + ccur * 256 + lane * 8 + 4);
#pragma unroll
        for (int i = 0; i < DMV_ROWS; ++i) {
            const Vec8 w = unpack8(cur[i]);
            float a = acc[i];
            a = fmaf(w.v[0], xa.x, a); a = fmaf(w.v[1], xa.y, a); a = fmaf(w.v[2], xa.z, a); a = fmaf(w.v[3], xa.w, a);
            a = fmaf(w.v[4], xb.x, a); a = fmaf(w.v[5], xb.y, a); a = fmaf(w.v[6], xb.z, a); a = fmaf(w.v[7], xb.w, a);
            acc[i] = a;
        }
        if (last) {
            // four sums over the lanes at once: lanes 8q .. 8q+7 end up with row q
            const bool hi = lane & 16, mid = lane & 8;
            float v0 = (hi ? acc[2] : acc[0]) + __shfl_xor_sync(0xffffffffu, hi ? acc[0] : acc[2], 16);
            float v1 = (hi ? acc[3] : acc[1]) + __shfl_xor_sync(0xffffffffu, hi ? acc[1] : acc[3], 16);
            float v = (mid ? v1 : v0) + __shfl_xor_sync(0xffffffffu, mid ? v0 : v1, 8);
            v += __shfl_xor_sync(0xffffffffu, v, 4);
            v += __shfl_xor_sync(0xffffffffu, v, 2);
            v += __shfl_xor_sync(0xffffffffu, v, 1);
            if ((lane & 7) == 0) part[(gcur * DMV_ROWS + (lane >> 3)) * p.nslice + (itcur - gcur * p.nslice)] = v;
#pragma unroll
            for (int i = 0; i < DMV_ROWS; ++i) acc[i] = 0.f;
        }
    }
    __syncthreads();

    float best = -INFINITY;
    int best_i = 0x7fffffff;
    for (int u = threadIdx.x; u < nu; u += DMV_THREADS) {
        float v = 0.f, v2 = 0.f;
        const float* pr = part + u * p.unit * p.nslice;
        for (int s = 0; s < p.nslice; ++s) v += pr[s];
        if (p.unit == 2)
            for (int s = 0; s < p.nslice; ++s) v2 += pr[p.nslice + s];
        dense_epilogue<float>(p.epi, 0, u0 + u, v, v2);
        if (v > best) {
            best = v;
            best_i = u0 + u;
        }
    }
    if (p.epi.kind != DE_LOGITS) return;
    auto better = [](float v, int i, float w, int j) { return v > w || (v == w && i < j); };
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, best_i, o);
        if (better(ov, oi, best, best_i)) best = ov, best_i = oi;
    }
    if (lane == 0) s_red[warp] = best, s_idx[warp] = best_i;
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int w = 1; w < DMV_WARPS; ++w)
            if (better(s_red[w], s_idx[w], best, best_i)) best = s_red[w], best_i = s_idx[w];
        p.amax_val[b] = best;
        p.amax_idx[b] = best_i;
    }
}

}  // namespace l2b
