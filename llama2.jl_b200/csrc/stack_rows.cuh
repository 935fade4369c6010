// Row-wise kernels of layer-stack models: embedding rows, and the step between two dense products of a many-token pass
// (pending changes of the residual stream, norm, conversion to the operand type), which the decode path does in the prologue of
// dense_matvec_kernel.
#pragma once
#include "dense_ops.cuh"

namespace l2b {

// x[t] = scale * table[tokens[t]]; a token id outside [0, vocab) gives a row of zeros (the table is never read out of bounds).
// Grid (blocks per row, rows).
__global__ void scaled_embed_kernel(const bf16* __restrict__ table, const int* tokens, int width, int vocab, float scale, float* __restrict__ x) {
    pdl_launch_dependents();
    pdl_wait();
    const int tok = __ldcg(tokens + blockIdx.y);
    const bool valid = tok >= 0 && tok < vocab;
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < width; i += gridDim.x * blockDim.x)
        x[(size_t)blockIdx.y * width + i] = valid ? scale * __bfloat162float(table[(size_t)tok * width + i]) : 0.f;
}

struct RowsParams {
    float* x;              // residual stream [rows][width]
    int width;
    const int* index;      // rows to take (null: all, in order); the result of index[t] goes to act row t
    ResidualUpdate upd;    // y is [rows][width]
    int store_x;           // write the changed residual stream back
    NormParams norm;
    void* act;             // [rows][lda] operand of the next product (null: none)
    int lda;
};
// V: values a thread takes at a time (4 when width and lda allow 16-byte accesses, else 1)
template <typename AT, int V>
__global__ void __launch_bounds__(256) residual_rows_kernel(const __grid_constant__ RowsParams p) {
    __shared__ float s_red[8];
    struct alignas(4 * V) F { float v[V]; };
    struct alignas(sizeof(AT) * V) A { AT v[V]; };
    const int src = p.index ? __ldg(p.index + blockIdx.x) : (int)blockIdx.x;
    F* const x = reinterpret_cast<F*>(p.x + (size_t)src * p.width);
    const F* const y = p.upd.y ? reinterpret_cast<const F*>(p.upd.y + (size_t)src * p.width) : nullptr;
    const int n = p.width / V;
    float scale = 0.f;
    if (y) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < n; i += 256) {
            const F t = y[i];
#pragma unroll
            for (int k = 0; k < V; ++k) ss = fmaf(t.v[k], t.v[k], ss);
        }
        scale = 1.f / sqrtf(block_sum_all<8>(ss, s_red) / (float)p.width + p.upd.eps);
    }
    A* const act = p.act ? reinterpret_cast<A*>(static_cast<AT*>(p.act) + (size_t)blockIdx.x * p.lda) : nullptr;
    for (int i = threadIdx.x; i < n; i += 256) {
        F t = x[i];
        if (y) {
            const F b = y[i];
#pragma unroll
            for (int k = 0; k < V; ++k) t.v[k] = fmaf(b.v[k] * scale, __ldg(p.upd.side_w + i * V + k), t.v[k]);
        }
        if (p.upd.step)
#pragma unroll
            for (int k = 0; k < V; ++k) t.v[k] += __ldg(p.upd.step + i * V + k);
        if (p.store_x) x[i] = t;
        if (act) {
            A o;
#pragma unroll
            for (int k = 0; k < V; ++k) put(&o.v[k], apply_norm(p.norm, t.v[k], i * V + k));
            act[i] = o;
        }
    }
}

}  // namespace l2b
