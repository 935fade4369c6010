// Differential attention over cached keys and values: every head has two softmax maps over the same values, and the second one's
// result is subtracted with a weight; queries and keys are normed per map and rotated in halves (dimensions i and i + rdims/2); the
// difference is brought to unit rms per head and passes an output gate.  A cache row of one key / value head is
//     [value, rounded up to 8 | key of map 1, rounded up to 8 | key of map 2, rounded up to 8],
// so that the two maps of the heads that share it are query vectors of cache_scan.cuh with zeros outside their own key.
//   head_rows_kernel    query vectors (for the scan, or as operands of head_prefill.cuh), new keys and values into the cache;
//   cache_scan_*_kernel scores and weighted sums;
//   head_output_kernel  merges the ranges, subtracts the maps, norms, gates.
#pragma once
#include "cache_scan.cuh"

namespace l2b {

struct HeadShape {
    int heads, kv_heads, dim, vdim, rdims;
    int dp, vp, row;    // stored key / value dimensions; cache row length vp + 2 dp
    float scale2;       // scale * log2(e)
    float eps;
    float lambda, out_scale;  // weight of the second map; factor after the norm
};
struct HeadAttnParams {
    HeadShape s;
    CacheScan c;            // heads: 2 per query head, map innermost; groups: key / value heads
    const float* in;        // [rows][ld]: q [heads][2][dim], then at off_k k [kv_heads][2][dim], at off_v v [kv_heads][vdim], at off_g the gate
    int ld, off_k, off_v, off_g;
    int own_kv;             // this layer has keys and values of its own
    const float* qnorm;     // [dim]
    const float* knorm;     // [dim]
    const float2* rope;     // [positions][rdims / 2]
    bf16* pq;               // queries as operands [rows][2 heads][dq] (null: query vectors of the scan)
    int dq;
    void* out;              // [rows][ldo]
    int ldo;
};

constexpr int HA_WARPS = 8;

// Element d of a vector of `dim` values at src after its norm (inv = 1 / rms) and the rotation.
__device__ __forceinline__ float normed_rotated(const float* src, float inv, const float* w, int d, int rdims, const float2* cs) {
    const float v = __ldcg(src + d) * inv * __ldg(w + d);
    const int half = rdims >> 1;
    if (d >= rdims) return v;
    const bool second = d >= half;
    const int i = second ? d - half : d, o = second ? i : i + half;
    const float2 t = __ldg(cs + i);
    const float u = __ldcg(src + o) * inv * __ldg(w + o);
    return second ? v * t.x + u * t.y : v * t.x - u * t.y;
}

// Grid (ceil(items / HA_WARPS), rows); a warp makes one item: the query of a (head, map), the key of a (kv head, map), a value.
template <typename CT>
__global__ void __launch_bounds__(HA_WARPS * 32) head_rows_kernel(const __grid_constant__ HeadAttnParams p) {
    const HeadShape& S = p.s;
    const int lane = threadIdx.x & 31, row = (int)blockIdx.y;
    int item = (int)blockIdx.x * HA_WARPS + ((int)threadIdx.x >> 5);
    pdl_launch_dependents();
    const int pos = scan_position(p.c, row);
    const float2* const cs = p.rope + (size_t)pos * (S.rdims >> 1);
    pdl_wait();
    const float* const in = p.in + (size_t)row * p.ld;
    const int nq = 2 * S.heads, nk = p.own_kv ? 2 * S.kv_heads : 0, nv = p.own_kv ? S.kv_heads : 0;
    if (item < nq + nk) {
        const bool query = item < nq;
        const int sub = query ? item : item - nq;
        const float* const src = in + (query ? 0 : p.off_k) + (size_t)sub * S.dim;
        const float* const w = query ? p.qnorm : p.knorm;
        float ss = 0.f;
        for (int d = lane; d < S.dim; d += 32) {
            const float v = __ldcg(src + d);
            ss = fmaf(v, v, ss);
        }
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)S.dim + S.eps);
        if (!query) {
            CT* const dst = static_cast<CT*>(p.c.cache) + (size_t)row * p.c.cache_stride + (size_t)(sub >> 1) * p.c.group_stride + (size_t)pos * S.row + S.vp + (sub & 1) * S.dp;
            for (int d = lane; d < S.dp; d += 32) put(dst + d, d < S.dim ? normed_rotated(src, inv, w, d, S.rdims, cs) : 0.f);
        } else if (p.pq) {
            bf16* const dst = p.pq + ((size_t)row * nq + sub) * p.dq;
            for (int d = lane; d < p.dq; d += 32) put(dst + d, d < S.dim ? normed_rotated(src, inv, w, d, S.rdims, cs) : 0.f);
        } else {
            float* const dst = p.c.qp + ((size_t)row * nq + sub) * S.row;
            const int k0 = S.vp + (sub & 1) * S.dp;
            for (int e = lane; e < S.row; e += 32) {
                const int d = e - k0;
                dst[e] = d >= 0 && d < S.dim ? S.scale2 * normed_rotated(src, inv, w, d, S.rdims, cs) : 0.f;
            }
        }
        return;
    }
    item -= nq + nk;
    if (item >= nv) return;
    const float* const src = in + p.off_v + (size_t)item * S.vdim;
    CT* const dst = static_cast<CT*>(p.c.cache) + (size_t)row * p.c.cache_stride + (size_t)item * p.c.group_stride + (size_t)pos * S.row;
    for (int d = lane; d < S.vp; d += 32) put(dst + d, d < S.vdim ? __ldcg(src + d) : 0.f);
}

// Grid (heads, rows).
template <typename OT>
__global__ void __launch_bounds__(HA_WARPS * 32) head_output_kernel(const __grid_constant__ HeadAttnParams p) {
    __shared__ float s_w[2 * CS_MAX_SPLIT];
    __shared__ float2 s_part[CS_MAX_ROW / 2];
    __shared__ float s_red[HA_WARPS];
    const HeadShape& S = p.s;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = (int)blockIdx.y, h = (int)blockIdx.x;
    pdl_launch_dependents();
    const int pos = scan_position(p.c, row), npos = pos + 1 - scan_first(p.c, pos), range = scan_range(npos, p.c.nsplit), ns = (npos + range - 1) / range;
    pdl_wait();
    const size_t slot = ((size_t)row * p.c.heads + 2 * h) * p.c.nsplit;  // the second map's slots follow the first one's
    if (warp < 2) {  // weights of the ranges of a map; ns <= 64
        const float2* const ml = p.c.part_ml + slot + (size_t)warp * p.c.nsplit;
        const float2 a = lane < ns ? __ldcg(ml + lane) : make_float2(-INFINITY, 0.f);
        const float2 b = lane + 32 < ns ? __ldcg(ml + 32 + lane) : make_float2(-INFINITY, 0.f);
        const float M = warp_max(fmaxf(a.x, b.x)), wa = exp2f(a.x - M), wb = exp2f(b.x - M);
        const float inv = (warp ? -S.lambda : 1.f) / warp_sum(fmaf(a.y, wa, b.y * wb));
        if (lane < ns) s_w[warp * ns + lane] = wa * inv;
        if (lane + 32 < ns) s_w[warp * ns + lane + 32] = wb * inv;
    }
    __syncthreads();
    constexpr int T = HA_WARPS * 32;
    const int np = S.vp >> 1, nsg = max(1, min(T / np, 8));  // column pairs; threads per pair
    for (int i = tid; i < np * nsg; i += T) {
        const int cp = i % np, sg = i / np;
        const float* const src = p.c.part_acc + slot * S.vp + 2 * cp;
        float2 a = make_float2(0.f, 0.f);
#pragma unroll 8
        for (int r = sg; r < 2 * ns; r += nsg) {
            const float2 x = __ldcg(reinterpret_cast<const float2*>(src + (size_t)(r < ns ? r : r - ns + p.c.nsplit) * S.vp));
            a.x = fmaf(x.x, s_w[r], a.x);
            a.y = fmaf(x.y, s_w[r], a.y);
        }
        s_part[i] = a;
    }
    __syncthreads();
    float ss = 0.f;
    for (int i = tid; i < np; i += T) {
        float2 a = s_part[i];
        for (int k = 1; k < nsg; ++k) {
            a.x += s_part[k * np + i].x;
            a.y += s_part[k * np + i].y;
        }
        s_part[i] = a;  // (read again by this thread only)
        ss += (2 * i < S.vdim ? a.x * a.x : 0.f) + (2 * i + 1 < S.vdim ? a.y * a.y : 0.f);
    }
    const float scale = S.out_scale / sqrtf(block_sum_all<HA_WARPS>(ss, s_red) / (float)S.vdim + S.eps);
    const float* const gate = p.in + (size_t)row * p.ld + p.off_g + (size_t)h * S.vdim;
    OT* const out = static_cast<OT*>(p.out) + (size_t)row * p.ldo + (size_t)h * S.vdim;
    for (int i = tid; i < np; i += T) {
        const float2 a = s_part[i];
        if (2 * i < S.vdim) put(out + 2 * i, a.x * scale * sigmoid(__ldcg(gate + 2 * i)));
        if (2 * i + 1 < S.vdim) put(out + 2 * i + 1, a.y * scale * sigmoid(__ldcg(gate + 2 * i + 1)));
    }
}

}  // namespace l2b
