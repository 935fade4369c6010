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
    bf16* pg;               // beside them: sigmoid of the gates [rows][heads * vp]
    void* out;              // [rows][ldo]
    int ldo;
};

constexpr int HA_WARPS = 8;

constexpr int HA_REGS = 4;  // values of a vector a lane holds (a longer vector is read again)

// A vector of `dim` values at src after its norm and the rotation, by a warp: lane l makes elements l, l + 32, ...; put_at(d, value) takes
// them, zeros from dim to `pad` included.
template <class PutAt>
__device__ __forceinline__ void normed_rotated(const float* src, const float* w, int dim, int rdims, float eps, const float2* cs, int pad, const PutAt& put_at) {
    const int lane = threadIdx.x & 31, half = rdims >> 1;
    float v[HA_REGS];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < HA_REGS; ++i) {
        v[i] = lane + 32 * i < dim ? __ldcg(src + lane + 32 * i) : 0.f;
        ss = fmaf(v[i], v[i], ss);
    }
    for (int d = lane + 32 * HA_REGS; d < dim; d += 32) {
        const float x = __ldcg(src + d);
        ss = fmaf(x, x, ss);
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dim + eps);
    auto partner = [&](int d) { return d >= rdims ? d : d >= half ? d - half : d + half; };
    auto turned = [&](int d, float x, float y) {  // x: element d, y: its partner, both without weight
        const float a = x * inv * __ldg(w + d);
        if (d >= rdims) return a;
        const bool second = d >= half;
        const float2 t = __ldg(cs + (second ? d - half : d));
        const float u = y * inv * __ldg(w + partner(d));
        return second ? a * t.x + u * t.y : a * t.x - u * t.y;
    };
#pragma unroll
    for (int i = 0; i < HA_REGS; ++i) {
        const int d = lane + 32 * i, o = partner(d);
        float y = 0.f;
        if (rdims <= 32 * HA_REGS) {
#pragma unroll
            for (int j = 0; j < HA_REGS; ++j) {
                if (32 * j < rdims && 32 * i < rdims) {  // (uniform)
                    const float x = __shfl_sync(0xffffffffu, v[j], o & 31);
                    if (o >> 5 == j) y = x;
                }
            }
        } else if (d < rdims) {
            y = __ldcg(src + o);
        }
        if (d < pad) put_at(d, d < dim ? turned(d, v[i], y) : 0.f);
    }
    for (int d = lane + 32 * HA_REGS; d < pad; d += 32) put_at(d, d < dim ? turned(d, __ldcg(src + d), __ldcg(src + partner(d))) : 0.f);
}

// The same by half / 4 lanes (a power of two) that hold both values of their pairs, four pairs each and four values at a time of the
// unrotated rest; for the portions of a prompt.  Everything is aligned to four values.
__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(bf16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w)); }
template <typename T>
__device__ __forceinline__ void normed_rotated_quads(const float* src, const float* w, int dim, int rdims, float eps, const float2* cs, int lanes, T* dst) {
    const int l = (threadIdx.x & 31) & (lanes - 1), half = rdims >> 1;
    const float4 a = __ldcg(reinterpret_cast<const float4*>(src) + l), b = __ldcg(reinterpret_cast<const float4*>(src + half) + l);
    float ss = a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w + b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w;
    for (int d = rdims + 4 * l; d < dim; d += 4 * lanes) {
        const float4 c = __ldcg(reinterpret_cast<const float4*>(src + d));
        ss += c.x * c.x + c.y * c.y + c.z * c.z + c.w * c.w;
    }
    for (int o = 1; o < lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = 1.f / sqrtf(ss / (float)dim + eps);
    const float4 wa = __ldg(reinterpret_cast<const float4*>(w) + l), wb = __ldg(reinterpret_cast<const float4*>(w + half) + l);
    const float4 t = __ldg(reinterpret_cast<const float4*>(cs) + 2 * l), u = __ldg(reinterpret_cast<const float4*>(cs) + 2 * l + 1);
    const float4 p = make_float4(a.x * inv * wa.x, a.y * inv * wa.y, a.z * inv * wa.z, a.w * inv * wa.w);
    const float4 q = make_float4(b.x * inv * wb.x, b.y * inv * wb.y, b.z * inv * wb.z, b.w * inv * wb.w);
    put4(dst + 4 * l, make_float4(p.x * t.x - q.x * t.y, p.y * t.z - q.y * t.w, p.z * u.x - q.z * u.y, p.w * u.z - q.w * u.w));
    put4(dst + half + 4 * l, make_float4(q.x * t.x + p.x * t.y, q.y * t.z + p.y * t.w, q.z * u.x + p.z * u.y, q.w * u.z + p.w * u.w));
    for (int d = rdims + 4 * l; d < dim; d += 4 * lanes) {
        const float4 c = __ldcg(reinterpret_cast<const float4*>(src + d)), wc = __ldg(reinterpret_cast<const float4*>(w + d));
        put4(dst + d, make_float4(c.x * inv * wc.x, c.y * inv * wc.y, c.z * inv * wc.z, c.w * inv * wc.w));
    }
}
// Grid (parts of the items, rows): the operands of a prompt portion.  Needs dim a multiple of 8 that is its own stored size, vdim a
// multiple of 8, `lanes` = rdims / 8 a power of two up to 32, ld and offsets multiples of 4.
__global__ void __launch_bounds__(HA_WARPS * 32) head_rows_quads_kernel(const __grid_constant__ HeadAttnParams p, int lanes) {
    const HeadShape& S = p.s;
    const int row = (int)blockIdx.y, pos = scan_position(p.c, row), per = HA_WARPS * 32 / lanes;  // vectors at a time
    const float2* const cs = p.rope + (size_t)pos * (S.rdims >> 1);
    const float* const in = p.in + (size_t)row * p.ld;
    bf16* const cache = static_cast<bf16*>(p.c.cache) + (size_t)pos * S.row;
    const int nq = 2 * S.heads, n = nq + (p.own_kv ? 2 * S.kv_heads : 0);
    for (int i0 = (int)blockIdx.x * per; i0 < n; i0 += (int)gridDim.x * per) {
        const int i = min(i0 + (int)threadIdx.x / lanes, n - 1);  // (the last ones may do the same work twice: shuffles need whole warps)
        if (i < nq) normed_rotated_quads(in + (size_t)i * S.dim, p.qnorm, S.dim, S.rdims, S.eps, cs, lanes, p.pq + ((size_t)row * nq + i) * p.dq);
        else normed_rotated_quads(in + p.off_k + (size_t)(i - nq) * S.dim, p.knorm, S.dim, S.rdims, S.eps, cs, lanes,
                                  cache + (size_t)((i - nq) >> 1) * p.c.group_stride + S.vp + ((i - nq) & 1) * S.dp);
    }
    for (int i = ((int)blockIdx.x * HA_WARPS * 32 + (int)threadIdx.x) * 4; i < S.heads * S.vdim; i += (int)gridDim.x * HA_WARPS * 128) {
        const float4 g = __ldcg(reinterpret_cast<const float4*>(in + p.off_g + i));
        put4(p.pg + (size_t)row * S.heads * S.vdim + i, make_float4(fast_sigmoid(g.x), fast_sigmoid(g.y), fast_sigmoid(g.z), fast_sigmoid(g.w)));
    }
    if (!p.own_kv) return;
    for (int i = ((int)blockIdx.x * HA_WARPS * 32 + (int)threadIdx.x) * 4; i < S.kv_heads * S.vdim; i += (int)gridDim.x * HA_WARPS * 128)
        put4(cache + (size_t)(i / S.vdim) * p.c.group_stride + i % S.vdim, __ldcg(reinterpret_cast<const float4*>(in + p.off_v + i)));
}

// Grid (ceil(items / HA_WARPS), rows); a warp makes one item: the query of a (head, map), the key of a (kv head, map), a value, a head's
// gates (operands only).
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
        if (!query) {
            CT* const dst = static_cast<CT*>(p.c.cache) + (size_t)row * p.c.cache_stride + (size_t)(sub >> 1) * p.c.group_stride + (size_t)pos * S.row + S.vp + (sub & 1) * S.dp;
            normed_rotated(src, w, S.dim, S.rdims, S.eps, cs, S.dp, [&](int d, float v) { put(dst + d, v); });
        } else if (p.pq) {
            bf16* const dst = p.pq + ((size_t)row * nq + sub) * p.dq;
            normed_rotated(src, w, S.dim, S.rdims, S.eps, cs, p.dq, [&](int d, float v) { put(dst + d, v); });
        } else {
            float* const dst = p.c.qp + ((size_t)row * nq + sub) * S.row;
            const int k0 = S.vp + (sub & 1) * S.dp, k1 = k0 + S.dp;
            for (int e = lane; e < S.row; e += 32)
                if (e < k0 || e >= k1) dst[e] = 0.f;
            normed_rotated(src, w, S.dim, S.rdims, S.eps, cs, S.dp, [&](int d, float v) { dst[k0 + d] = S.scale2 * v; });
        }
        return;
    }
    item -= nq + nk;
    if (item >= nv) {
        item -= nv;
        if (!p.pq || item >= S.heads) return;
        for (int d = lane; d < S.vp; d += 32)
            put(p.pg + ((size_t)row * S.heads + item) * S.vp + d, d < S.vdim ? fast_sigmoid(__ldcg(in + p.off_g + (size_t)item * S.vdim + d)) : 0.f);
        return;
    }
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
