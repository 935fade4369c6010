// Matrix-vector product of the decode path of layer-stack models: bf16 weights, f32 activations and accumulation.  The counterpart
// of fused_matvec_kernel for matrices stored in bf16.
//
// One block per SM, 8 consumer warps and a producer warp, every block a contiguous range of rows.
//   producer : a stage is 4 * gs rows x cs 256-value chunks (16 KiB at most); stages come into a ring with bulk asynchronous copies
//       (one copy of adjacent whole rows, or one per row when rows are longer than a stage).  Weights are constants, so
//       the ring is filled BEFORE the wait on the previous kernel (programmatic dependent launch);
//   prologue : the input vector goes to shared memory as f32, after the pending changes of the residual stream (the normalised
//       per-layer token input or sublayer result, the step vector of a loop pass) and the norm; block 0 writes the changed
//       residual stream back to its other buffer, because the other blocks still read this one.  The scalar 1 / rms(x) of an rms
//       norm is applied to the results, so that its reduction needs no barrier of its own;
//   weights  : two groups of four consumer warps take alternate stages (a stage's chain of waits, loads and lane reductions is long
//       beside the time its bytes take); a warp works on up to two units (4 rows x 1 chunk) of a stage and adds over the
//       stages of its rows in registers; eight row sums are then reduced over the lanes together;
//   epilogue : the chunk sums of a row are added in a fixed order by one thread: store | residual add | gelu(gate) * up or silu(gate) *
//       up (rows 2u and 2u+1 of an interleaved matrix) | gelu * token embedding | logits with the block's first maximum.
// Every mbarrier wait is bounded, as everywhere in the library.
#pragma once
#include <algorithm>

#include "dense_ops.cuh"

namespace l2b {

constexpr int DMV_WARPS = 8, DMV_CONSUMERS = DMV_WARPS * 32, DMV_THREADS = DMV_CONSUMERS + 32, DMV_ROWS = 4;
constexpr int DMV_GROUPS = 2, DMV_GROUP_WARPS = DMV_WARPS / DMV_GROUPS;
constexpr int DMV_STAGE = DMV_WARPS * DMV_ROWS * 512, DMV_MAX_STAGES = 11;

struct DmvParams {
    const bf16* w;          // [rows][kp], kp a multiple of 8
    int kp, k;              // stored and logical row length
    int unit;               // rows per result: 1, or 2 (interleaved gate / up)
    int per_lo, per_rem;    // results of block b: per_lo + (b < per_rem), contiguous
    int nchunk;             // 256-value chunks per row
    int gs, cs, nseg;       // a stage: 4 * gs rows x cs chunks (gs * cs <= 8); nseg stages per row group, gs = 1 when nseg > 1
    int stages;             // ring slots
    const float* x;         // input vector [k]
    ResidualUpdate upd;
    float* x_out;           // block 0 writes the updated vector here (null: no update)
    NormParams norm;
    DenseEpilogue epi;      // t = 0
    float* amax_val;        // DE_LOGITS, DE_AFFINE_LOGITS: per block
    int* amax_idx;
    int* status;
};
// Shared memory beside the ring, and ring slots: as many as fit and are of use (bytes in flight are what the HBM rate needs: with
// 64 KiB per SM the stream stays below 4.2 TB/s).
inline size_t dmv_fixed_bytes(const DmvParams& p) {
    const int rows = p.unit * (p.per_lo + (p.per_rem ? 1 : 0)), per_stage = DMV_ROWS * p.gs;
    return ((size_t)p.nchunk * 256 + (size_t)((rows + per_stage - 1) / per_stage * per_stage) * p.cs) * 4;
}
inline int dmv_choose_stages(const DmvParams& p, size_t max_smem) {
    const int rows = p.unit * (p.per_lo + (p.per_rem ? 1 : 0)), per_stage = DMV_ROWS * p.gs;
    const long fit = ((long)max_smem - (long)dmv_fixed_bytes(p)) / DMV_STAGE, use = (long)((rows + per_stage - 1) / per_stage) * p.nseg;
    return (int)std::min<long>(DMV_MAX_STAGES, std::min<long>(fit, std::max<long>(use, 2)));
}

// RMS: the norm in front is an rms norm (else none, or dynamic tanh).  KINDS: one of the sets of epilogues below.
constexpr unsigned DMV_KINDS_GELU = 1u << DE_STORE | 1u << DE_RESIDUAL | 1u << DE_LOGITS | 1u << DE_GEGLU | 1u << DE_SIDE;
constexpr unsigned DMV_KINDS_SILU = 1u << DE_STORE | 1u << DE_RESIDUAL | 1u << DE_LOGITS | 1u << DE_SWIGLU | 1u << DE_AFFINE | 1u << DE_AFFINE_LOGITS;
template <bool RMS, unsigned KINDS>
__global__ void __launch_bounds__(DMV_THREADS, 2) dense_matvec_kernel(const __grid_constant__ DmvParams p) {
    extern __shared__ __align__(128) uint8_t dmv_smem[];
    __shared__ __align__(8) uint64_t s_full[DMV_MAX_STAGES], s_empty[DMV_MAX_STAGES];
    __shared__ float s_red[DMV_WARPS], s_ss[DMV_WARPS];
    __shared__ int s_idx[DMV_WARPS];
    float* const xf = reinterpret_cast<float*>(dmv_smem + p.stages * DMV_STAGE);
    float* const part = xf + p.nchunk * 256;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const bool logits = p.epi.kind == DE_LOGITS || ((KINDS >> DE_AFFINE_LOGITS & 1) && p.epi.kind == DE_AFFINE_LOGITS);
    pdl_launch_dependents();
    if (threadIdx.x == 0) {
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(s_full + i, 1);
            mbar_init(s_empty + i, DMV_GROUP_WARPS);
        }
        fence_barrier_init();
        fence_proxy_async();
    }
    __syncthreads();
    const int b = (int)blockIdx.x;
    const int u0 = b * p.per_lo + min(b, p.per_rem), nu = p.per_lo + (b < p.per_rem ? 1 : 0);
    const int nr = nu * p.unit;
    const bf16* const wb = p.w + (size_t)u0 * p.unit * p.kp;
    const int per_stage = DMV_ROWS * p.gs, nrs = (nr + per_stage - 1) / per_stage;  // row stages; group g takes g, g + 2, ...
    const int seg_vals = p.cs * 256, pitch = p.nseg == 1 ? p.kp : seg_vals;  // values between the rows of a stage
    bool dead = false;

    if (warp == DMV_WARPS) {
        const uint64_t policy = policy_evict_first();
        const int nstage = nrs * p.nseg;
        int s = 0, use = 0;
        int rs = 0, seg = 0;  // order: a pair of row stages at a time, their segments in turn
        for (int j = 0; j < nstage; ++j) {
            if (use > 0 && !mbar_wait_bounded(s_empty + s, (uint32_t)((use - 1) & 1))) {
                dead = true;
                break;
            }
            __syncwarp();
            const int row = rs * per_stage, rows = min(per_stage, nr - row), vals = p.nseg == 1 ? p.kp : min(seg_vals, p.kp - seg * seg_vals);
            uint8_t* const dst = dmv_smem + s * DMV_STAGE;
            if (lane == 0) mbar_arrive_expect_tx(s_full + s, (uint32_t)(rows * vals * 2));
            __syncwarp();
            const bf16* const src = wb + (size_t)row * p.kp + seg * seg_vals;
            if (p.nseg == 1) {
                if (lane == 0) bulk_g2s(dst, src, (uint32_t)(rows * vals * 2), s_full + s, policy);
            } else if (lane < rows) {
                bulk_g2s(dst + lane * seg_vals * 2, src + (size_t)lane * p.kp, (uint32_t)(vals * 2), s_full + s, policy);
            }
            if (!(rs & 1) && rs + 1 < nrs) {
                ++rs;
            } else if (++seg < p.nseg) {
                rs &= ~1;
            } else {
                seg = 0;
                ++rs;
            }
            if (++s == p.stages) s = 0, ++use;
        }
        if (dead) {
            if (lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
            for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
        }
        __syncthreads();
        if (logits) __syncthreads();
        return;
    }

    pdl_wait();
    {
        constexpr int U = 8;
        const int k = p.k, kc = p.nchunk * 256;
        float scale = 0.f;
        if (p.upd.y) {
            float ss = 0.f;
            for (int i0 = threadIdx.x; i0 < k; i0 += U * DMV_CONSUMERS) {
                float v[U];
#pragma unroll
                for (int u = 0; u < U; ++u) v[u] = i0 + u * DMV_CONSUMERS < k ? __ldcg(p.upd.y + i0 + u * DMV_CONSUMERS) : 0.f;
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    ss = fmaf(v[u], v[u], ss);
                    if (i0 + u * DMV_CONSUMERS < k) xf[lane_major(i0 + u * DMV_CONSUMERS)] = v[u];
                }
            }
            scale = 1.f / sqrtf(block_sum_all<DMV_WARPS>(ss, s_red) / (float)k + p.upd.eps);
        }
        float xs = 0.f;
        for (int i0 = threadIdx.x; i0 < kc; i0 += U * DMV_CONSUMERS) {
            float v[U];
#pragma unroll
            for (int u = 0; u < U; ++u) v[u] = i0 + u * DMV_CONSUMERS < k ? __ldcg(p.x + i0 + u * DMV_CONSUMERS) : 0.f;
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * DMV_CONSUMERS, at = lane_major(i);
                if (i < k) {
                    float t = v[u];
                    if (p.upd.y) t = fmaf(xf[at] * scale, __ldg(p.upd.w + i), t);
                    if (p.upd.step) t += __ldg(p.upd.step + i);
                    if (p.x_out && b == 0) p.x_out[i] = t;
                    if (RMS) xs = fmaf(t, t, xs);
                    xf[at] = apply_norm<RMS>(p.norm, t, i);
                } else if (i < kc) {
                    xf[at] = 0.f;
                }
            }
        }
        if (RMS) {
            xs = warp_sum(xs);
            if (lane == 0) s_ss[warp] = xs;  // (read after the last barrier)
        }
    }
    partial_sync(DMV_CONSUMERS);

    {
        const int grp = warp / DMV_GROUP_WARPS, wg = warp % DMV_GROUP_WARPS;
        int ug[2], uc[2];  // this warp's units of a stage: row group and chunk
        bool mine[2];
        int s = grp;       // ring slot of this group's next stage
        uint32_t par = 0;
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            const int u = wg + t * DMV_GROUP_WARPS;
            ug[t] = u / p.cs;
            uc[t] = u - ug[t] * p.cs;
            mine[t] = ug[t] < p.gs;
        }
#pragma unroll 1
        for (int rs = grp; rs < nrs; rs += DMV_GROUPS) {
            const bool paired = (rs | 1) < nrs;  // both row stages of the pair exist
            f32x2 acc[2][DMV_ROWS];
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int i = 0; i < DMV_ROWS; ++i) acc[t][i] = 0ull;
#pragma unroll 1
            for (int seg = 0; seg < p.nseg; ++seg) {
                if (!dead && !mbar_wait_bounded(s_full + s, par)) dead = true;
#pragma unroll
                for (int t = 0; t < 2; ++t) {
                    const int c = seg * p.cs + uc[t];
                    if (mine[t] && !dead && c * 256 + lane * 8 < p.kp) {
                        const uint8_t* src = dmv_smem + s * DMV_STAGE + (ug[t] * DMV_ROWS * pitch + uc[t] * 256 + lane * 8) * 2;
                        uint4 w[DMV_ROWS];
#pragma unroll
                        for (int i = 0; i < DMV_ROWS; ++i) w[i] = *reinterpret_cast<const uint4*>(src + i * pitch * 2);
                        const Pairs8 x = read_lane_major(xf, c, lane);
#pragma unroll
                        for (int i = 0; i < DMV_ROWS; ++i) {
                            acc[t][i] = fma2(widen2(w[i].x), x.p[0], acc[t][i]);
                            acc[t][i] = fma2(widen2(w[i].y), x.p[1], acc[t][i]);
                            acc[t][i] = fma2(widen2(w[i].z), x.p[2], acc[t][i]);
                            acc[t][i] = fma2(widen2(w[i].w), x.p[3], acc[t][i]);
                        }
                    }
                }
                __syncwarp();
                if (lane == 0) mbar_arrive(s_empty + s);
                s += paired ? 2 : 1;  // the other group's stage of the pair lies between
                if (s >= p.stages) s -= p.stages, par ^= 1u;
            }
            float a[2 * DMV_ROWS];
#pragma unroll
            for (int i = 0; i < 2 * DMV_ROWS; ++i) a[i] = sum2(acc[i / DMV_ROWS][i % DMV_ROWS]);
            const float v = warp_sums_spread<2 * DMV_ROWS>(a);  // lanes 4i .. 4i+3 hold sum i
            const int i = lane >> 2, t = i / DMV_ROWS;
            if ((lane & 3) == 0 && (t ? mine[1] : mine[0]))
                part[(rs * per_stage + (t ? ug[1] : ug[0]) * DMV_ROWS + i % DMV_ROWS) * p.cs + (t ? uc[1] : uc[0])] = v;
        }
        if (dead && lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
    }
    __syncthreads();

    float rms_scale = 1.f;
    if (RMS) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < DMV_WARPS; ++i) ss += s_ss[i];
        rms_scale = 1.f / sqrtf(ss / (float)p.k + p.norm.eps);
    }
    float best = -INFINITY;
    int best_i = 0x7fffffff;
    for (int u = threadIdx.x; u < nu; u += DMV_CONSUMERS) {
        float v = 0.f, v2 = 0.f;
        const float* pr = part + u * p.unit * p.cs;
        for (int s = 0; s < p.cs; ++s) v += pr[s];
        if (p.unit == 2)
            for (int s = 0; s < p.cs; ++s) v2 += pr[p.cs + s];
        if (RMS) v *= rms_scale, v2 *= rms_scale;
        dense_epilogue<float, KINDS>(p.epi, 0, u0 + u, v, v2);
        if ((KINDS >> DE_AFFINE_LOGITS & 1) && p.epi.kind == DE_AFFINE_LOGITS) v = affine(p.epi, u0 + u, v);
        if (v > best) {
            best = v;
            best_i = u0 + u;
        }
    }
    if (!logits) return;
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
