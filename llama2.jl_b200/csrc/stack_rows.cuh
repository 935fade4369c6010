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
template <typename AT>
__global__ void __launch_bounds__(256) residual_rows_kernel(const __grid_constant__ RowsParams p) {
    __shared__ float s_red[8];
    const int src = p.index ? __ldg(p.index + blockIdx.x) : (int)blockIdx.x;
    float* x = p.x + (size_t)src * p.width;
    const float* y = p.upd.y ? p.upd.y + (size_t)src * p.width : nullptr;
    float scale = 0.f;
    if (y) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < p.width; i += 256) ss = fmaf(y[i], y[i], ss);
        scale = 1.f / sqrtf(block_sum_all<8>(ss, s_red) / (float)p.width + p.upd.eps);
    }
    AT* act = p.act ? static_cast<AT*>(p.act) + (size_t)blockIdx.x * p.lda : nullptr;
    for (int i = threadIdx.x; i < p.width; i += 256) {
        float t = x[i];
        if (y) t = fmaf(y[i] * scale, __ldg(p.upd.side_w + i), t);
        if (p.upd.step) t += __ldg(p.upd.step + i);
        if (p.store_x) x[i] = t;
        if (act) put(act + i, apply_norm(p.norm, t, i));
    }
}

}  // namespace l2b
