// Row-wise kernels of layer-stack models: embedding rows, and the step between two dense products of a many-token pass
// (pending changes of the residual stream, norm, conversion to the operand type), which the decode path does in the prologue of
// dense_matvec_kernel.
#pragma once
#include "dense_ops.cuh"

namespace l2b {

// x[t] = scale * table[tokens[t]] + pos_table[position of t]; a token id outside [0, vocab) gives a table row of zeros (no table is
// read out of bounds).  Grid (blocks per row, rows).
struct EmbedParams {
    const bf16* table;
    const int* tokens;
    int width, vocab;
    float scale;
    const bf16* pos_table;  // learned position vectors (null: none)
    int max_positions;
    const int* pos;         // decode: device scalar
    const int* pos_list;    // batched decode: position of every row
    int pos0;               // otherwise row r sits at pos0 + r
    float* x;
};
__global__ void embed_positions_kernel(const __grid_constant__ EmbedParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int row = (int)blockIdx.y, tok = __ldcg(p.tokens + row);
    const bool valid = tok >= 0 && tok < p.vocab;
    const int pos = p.pos ? __ldcg(p.pos) : p.pos_list ? __ldcg(p.pos_list + row) : p.pos0 + row;
    const bf16* const pv = p.pos_table && pos >= 0 && pos < p.max_positions ? p.pos_table + (size_t)pos * p.width : nullptr;
    const int first = blockIdx.x * blockDim.x + threadIdx.x, step = gridDim.x * blockDim.x;
    float* const x = p.x + (size_t)row * p.width;
    const bf16* const tv = p.table + (size_t)(valid ? tok : 0) * p.width;
    if ((p.width & 7) == 0) {  // eight values at a time
        const float scale = valid ? p.scale : 0.f;
        for (int i = first; i < p.width / 8; i += step) {
            const uint4 a = __ldg(reinterpret_cast<const uint4*>(tv) + i), b = pv ? __ldg(reinterpret_cast<const uint4*>(pv) + i) : make_uint4(0u, 0u, 0u, 0u);
            const uint32_t e[4] = {a.x, a.y, a.z, a.w}, q[4] = {b.x, b.y, b.z, b.w};
            float v[8];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                v[2 * k] = scale * __uint_as_float(e[k] << 16) + __uint_as_float(q[k] << 16);
                v[2 * k + 1] = scale * __uint_as_float(e[k] & 0xFFFF0000u) + __uint_as_float(q[k] & 0xFFFF0000u);
            }
            reinterpret_cast<float4*>(x)[2 * i] = make_float4(v[0], v[1], v[2], v[3]);
            reinterpret_cast<float4*>(x)[2 * i + 1] = make_float4(v[4], v[5], v[6], v[7]);
        }
        return;
    }
    for (int i = first; i < p.width; i += step) {
        const float e = valid ? p.scale * __bfloat162float(tv[i]) : 0.f;
        x[i] = pv ? e + __bfloat162float(pv[i]) : e;
    }
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
    __shared__ float s_red[8], s_red2[8];
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
    auto updated = [&](int i) {
        F t = x[i];
        if (y) {
            const F b = y[i];
#pragma unroll
            for (int k = 0; k < V; ++k) t.v[k] = fmaf(b.v[k] * scale, __ldg(p.upd.w + i * V + k), t.v[k]);
        }
        if (p.upd.step)
#pragma unroll
            for (int k = 0; k < V; ++k) t.v[k] += __ldg(p.upd.step + i * V + k);
        return t;
    };
    float rms_scale = 1.f;
    const bool rms = p.norm.kind == NORM_RMS;
    if (act && rms) {  // (the second pass finds its inputs in the first-level cache)
        float ss = 0.f;
        for (int i = threadIdx.x; i < n; i += 256) {
            const F t = updated(i);
#pragma unroll
            for (int k = 0; k < V; ++k) ss = fmaf(t.v[k], t.v[k], ss);
        }
        rms_scale = 1.f / sqrtf(block_sum_all<8>(ss, s_red2) / (float)p.width + p.norm.eps);
    }
    for (int i = threadIdx.x; i < n; i += 256) {
        const F t = updated(i);
        if (p.store_x) x[i] = t;
        if (act) {
            A o;
#pragma unroll
            for (int k = 0; k < V; ++k) put(&o.v[k], rms ? apply_norm<true>(p.norm, t.v[k], i * V + k) * rms_scale : apply_norm<false>(p.norm, t.v[k], i * V + k));
            act[i] = o;
        }
    }
}

}  // namespace l2b
