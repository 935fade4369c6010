// Matrix memory with exponential gating (mLSTM), token by token: per head a matrix S [dim][vdim], a vector n [dim] and a running
// maximum m, all f32,
//     m' = max(f + m, i),   S' = exp(f + m - m') S + exp(i - m') k v^T,   n' likewise with k alone,
//     o = S'^T q / (max(|n' . q|, exp(-m')) + 1e-6),
// where i and f are the logs of the gates.  o is brought to unit rms per head, weighted and gated.  The state before position 0 is
// zero whatever the memory holds, so a sequence that starts in a used slot needs no clearing.
//
// mlstm_step_kernel serves decode steps (one position; or one per sequence of a batch) and short portions (a loop over their tokens).
// A cluster of blocks shares a head, each with its own columns of S and its own copies of n and m.  In a decode step the
// state, which the token before wrote, is fetched before the wait on the previous kernel.
#pragma once
#include "dense_ops.cuh"

namespace l2b {

constexpr int ML_WARPS = 8, ML_THREADS = ML_WARPS * 32, ML_MAX_CLUSTER = 8, ML_MAX_DIM = 1024, ML_MAX_COLS = 4;

struct MlstmShape {
    int heads, dim, vdim;
    int cl, cpl;        // blocks per head (1, 2, 4, 8); columns per lane: a block has 32 * cpl columns
    float cap, qscale, eps;
    // state of a sequence: S [heads][dim][vdim], then n [heads][cl][dim], then m [heads][cl]
    __host__ __device__ size_t n_at() const { return (size_t)heads * dim * vdim; }
    __host__ __device__ size_t m_at() const { return n_at() + (size_t)heads * cl * dim; }
    __host__ __device__ size_t size() const { return m_at() + (size_t)heads * cl; }
};
struct MlstmParams {
    MlstmShape s;
    const float* in;    // [tokens][ld]: q [heads][dim], at off_k k, at off_v v [heads][vdim], at off_g the output gate, at off_i / off_f the gates [heads]
    int ld, off_k, off_v, off_g, off_i, off_f;
    const float* norm;  // [heads * vdim]
    float* state;
    size_t state_stride;  // elements between the states of consecutive rows (batched decode), else 0
    const int* pos;       // decode: device scalar
    const int* pos_list;  // batched decode: position of every row
    int pos0;
    int tokens;           // tokens of a portion, one after the other (1 in a decode step)
    void* out;            // [tokens or rows][ldo]
    int ldo;
};

struct MlstmGates {
    float i, f;  // logs
};
__device__ __forceinline__ MlstmGates mlstm_gates(const MlstmParams& p, const float* in, int h) {
    MlstmGates g;
    g.i = p.s.cap * tanhf(__ldcg(in + p.off_i + h) / p.s.cap);
    g.f = log_sigmoid(p.s.cap * tanhf(__ldcg(in + p.off_f + h) / p.s.cap));
    return g;
}

// Grid (heads * cl, rows), clusters of cl.  Warp w has rows w, w + 8, ... of S, lane l columns l, l + 32, ... of the block's.  RPT: rows
// a thread holds in registers; when that is all of them (dim <= 8 RPT) they stay there over the tokens of a portion.
template <int RPT, int CPL, typename OT>
__global__ void __launch_bounds__(ML_THREADS) mlstm_step_kernel(const __grid_constant__ MlstmParams p) {
    __shared__ float s_q[ML_MAX_DIM], s_k[ML_MAX_DIM], s_n[ML_MAX_DIM];
    __shared__ float s_acc[ML_WARPS][32 * CPL], s_nq[ML_WARPS], s_red[ML_WARPS];
    __shared__ float s_ss[2][ML_MAX_CLUSTER];  // [token parity][block of the cluster]
    const MlstmShape& S = p.s;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = (int)blockIdx.y;
    const int h = (int)blockIdx.x / S.cl, rank = (int)blockIdx.x % S.cl, c0 = rank * 32 * CPL;
    pdl_launch_dependents();
    if (S.cl > 1) cluster_arrive();  // (waited for before the first store into another block's shared memory)
    float* const base = p.state + (size_t)row * p.state_stride;
    float* const gs = base + (size_t)h * S.dim * S.vdim + c0;
    float* const gn = base + S.n_at() + ((size_t)h * S.cl + rank) * S.dim;
    float* const gm = base + S.m_at() + (size_t)h * S.cl + rank;
    const bool fresh = (p.pos ? __ldcg(p.pos) : p.pos_list ? __ldcg(p.pos_list + row) : p.pos0) == 0;
    const bool resident = S.dim <= ML_WARPS * RPT;
    bool col[CPL];
#pragma unroll
    for (int j = 0; j < CPL; ++j) col[j] = c0 + lane + 32 * j < S.vdim;
    float st[RPT][CPL];
    auto load = [&](int d0, bool zero) {
#pragma unroll
        for (int r = 0; r < RPT; ++r)
#pragma unroll
            for (int j = 0; j < CPL; ++j) {
                const int d = d0 + warp + ML_WARPS * r;
                st[r][j] = !zero && d < S.dim && col[j] ? gs[(size_t)d * S.vdim + lane + 32 * j] : 0.f;
            }
    };
    auto store = [&](int d0) {
#pragma unroll
        for (int r = 0; r < RPT; ++r)
#pragma unroll
            for (int j = 0; j < CPL; ++j) {
                const int d = d0 + warp + ML_WARPS * r;
                if (d < S.dim && col[j]) gs[(size_t)d * S.vdim + lane + 32 * j] = st[r][j];
            }
    };
    load(0, fresh);
    for (int d = tid; d < S.dim; d += ML_THREADS) s_n[d] = fresh ? 0.f : gn[d];  // (a thread reads and writes its own elements only)
    float m = fresh ? 0.f : *gm;
    pdl_wait();
    for (int t = 0; t < p.tokens; ++t) {
        const float* const in = p.in + (size_t)(row + t) * p.ld;
        const MlstmGates g = mlstm_gates(p, in, h);
        const float mn = fmaxf(g.f + m, g.i), keep = expf(g.f + m - mn), add = expf(g.i - mn);
        m = mn;
        float nq = 0.f;
        for (int d = tid; d < S.dim; d += ML_THREADS) {
            const float q = __ldcg(in + (size_t)h * S.dim + d) * S.qscale, k = __ldcg(in + p.off_k + (size_t)h * S.dim + d);
            s_q[d] = q;
            s_k[d] = add * k;
            const float n = fmaf(keep, s_n[d], add * k);
            s_n[d] = n;
            nq = fmaf(n, q, nq);
        }
        float v[CPL], acc[CPL];
#pragma unroll
        for (int j = 0; j < CPL; ++j) {
            v[j] = col[j] ? __ldcg(in + p.off_v + (size_t)h * S.vdim + c0 + lane + 32 * j) : 0.f;
            acc[j] = 0.f;
        }
        nq = warp_sum(nq);
        if (lane == 0) s_nq[warp] = nq;
        __syncthreads();
        for (int d0 = 0; d0 < S.dim; d0 += ML_WARPS * RPT) {
            if (!resident && (t > 0 || d0 > 0)) load(d0, fresh && t == 0);
#pragma unroll
            for (int r = 0; r < RPT; ++r) {
                const int d = d0 + warp + ML_WARPS * r;
                if (d < S.dim) {
                    const float k = s_k[d], q = s_q[d];
#pragma unroll
                    for (int j = 0; j < CPL; ++j) {
                        st[r][j] = fmaf(keep, st[r][j], k * v[j]);
                        acc[j] = fmaf(st[r][j], q, acc[j]);
                    }
                }
            }
            if (!resident || t == p.tokens - 1) store(d0);
        }
#pragma unroll
        for (int j = 0; j < CPL; ++j) s_acc[warp][lane + 32 * j] = acc[j];
        __syncthreads();
        float o = 0.f;
        const int c = c0 + tid;
        const bool mine = tid < 32 * CPL && c < S.vdim;
        if (mine) {
            float dot = 0.f;
#pragma unroll
            for (int w = 0; w < ML_WARPS; ++w) {
                o += s_acc[w][tid];
                dot += s_nq[w];
            }
            o /= fmaxf(fabsf(dot), expf(-m)) + 1e-6f;
        }
        float ss = block_sum_all<ML_WARPS>(o * o, s_red);
        if (S.cl > 1) {
            if (t == 0) cluster_wait();
            if (tid < S.cl) st_cluster_f32(cluster_map(&s_ss[t & 1][rank], (uint32_t)tid), ss);
            cluster_sync_all();
            ss = 0.f;
            for (int r = 0; r < S.cl; ++r) ss += s_ss[t & 1][r];
        }
        if (mine) {
            const size_t at = (size_t)h * S.vdim + c;
            const float scale = 1.f / sqrtf(ss / (float)S.vdim + S.eps);
            put(static_cast<OT*>(p.out) + (size_t)(row + t) * p.ldo + at, o * scale * __ldg(p.norm + at) * sigmoid(__ldcg(in + p.off_g + at)));
        }
        // (the shared arrays are written again only after the barrier of block_sum_all, which every read above precedes)
    }
    for (int d = tid; d < S.dim; d += ML_THREADS) gn[d] = s_n[d];
    if (tid == 0) *gm = m;
}

}  // namespace l2b
