// Latent attention (one cached latent and one shared rotated key part per position, a sink in the softmax, a sigmoid output gate)
// in its absorbed form: with q' = W_uk^T q_unrotated the score of a head against position t is
//     (q' . c_t + q_rotated . kr_t) * scale,
// and W_uv is applied once, to the weighted sum of the latents.  So a head reads one row [c | kr] per position for keys and values
// alike, and nothing per head is cached.  Three kernels, chained with programmatic dependent launch in a decode step:
//   latent_query_kernel   q' and the rotated query part of every (row, head); in a decode step one more block normalises and
//                         rotates the new position's latent and key and writes them to the cache;
//   cache_scan_*_kernel   scores and weighted sums (cache_scan.cuh);
//   latent_output_kernel  merges the ranges and the sink, applies W_uv and the gate.
// (One kernel with clusters that exchange q' and the partial results through distributed shared memory was about twice as slow: its
// code is several times as long and runs once per launch, so that fetching instructions bounds it.)
// Weights are fetched before the wait on the previous kernel.
// Many-token passes run the same kernels over rows with their own positions (batched decode: also their own caches), the new
// positions written by latent_rows_kernel.
#pragma once
#include "cache_scan.cuh"

namespace l2b {

constexpr int LA_WARPS = CS_WARPS, LA_CONSUMERS = CS_CONSUMERS;

struct LatentShape {
    int heads, dim, rot, rdims, vdim, rank;  // rdims: rotated dimensions of the rot part
    int rp, row;    // rank rounded up to 8; cache row length: rp + rot rounded up to 8
    int dp, vp;     // stored rows per head of W_uk / W_uv
    float scale2;   // scale * log2(e)
    float eps;
};
struct LatentAttnParams {
    LatentShape s;
    CacheScan c;            // heads in one group; q' and the rotated part are its query vectors
    const float* qdg;       // [rows][ld]: q, down projection, gate
    int ld, off_d, off_g;
    const bf16* uk;         // [heads * dp][rp]
    const bf16* uv;         // [heads * vp][rp]
    const float* sink;      // [heads]
    const float* dnorm;     // [rank]
    const float2* rope;     // [positions][rdims / 2]
    int csplit, vsplit;     // blocks per head (query), blocks per head (output)
    void* out;              // [rows][ldo]
    int ldo;
};

// Latent (normalised) and rotated key of one position into its cache row; NW warps.
template <typename CT, int NW>
__device__ __forceinline__ void store_latent_row(const LatentAttnParams& p, int row, int pos, float* s_red) {
    const LatentShape& S = p.s;
    const int tid = threadIdx.x;
    CT* const dst = static_cast<CT*>(p.c.cache) + (size_t)row * p.c.cache_stride + (size_t)pos * S.row;
    const float* const down = p.qdg + (size_t)row * p.ld + p.off_d;
    float ss = 0.f;
    for (int i = tid; i < S.rank; i += NW * 32) {
        const float v = __ldcg(down + i);
        ss = fmaf(v, v, ss);
    }
    const float scale = 1.f / sqrtf(block_sum_all<NW>(ss, s_red) / (float)S.rank + S.eps);
    for (int i = tid; i < S.rp; i += NW * 32) put(dst + i, i < S.rank ? __ldcg(down + i) * scale * __ldg(p.dnorm + i) : 0.f);
    const float2* const rope = p.rope + (size_t)pos * (S.rdims >> 1);
    for (int i = tid; i < S.row - S.rp; i += NW * 32)
        put(dst + S.rp + i, i < S.rot ? rotary_element(i, S.rdims, rope, [&](int j) { return __ldcg(down + S.rank + j); }) : 0.f);
}
template <typename CT>
__global__ void __launch_bounds__(128) latent_rows_kernel(const __grid_constant__ LatentAttnParams p) {
    __shared__ float s_red[4];
    store_latent_row<CT, 4>(p, (int)blockIdx.x, scan_position(p.c, (int)blockIdx.x), s_red);
}

// Grid (heads * csplit, plus one block in a decode step; rows).  A block makes the columns of a range of 8-column chunks; thread =
// (chunk, group of W_uk rows), the groups summed through shared memory.
template <typename CT>
__global__ void __launch_bounds__(LA_CONSUMERS) latent_query_kernel(const __grid_constant__ LatentAttnParams p) {
    __shared__ float s_red[LA_WARPS];
    __shared__ __align__(16) float s_part[LA_CONSUMERS * 8];
    constexpr int PRE = 8;  // rows of W_uk a thread fetches before the wait
    const LatentShape& S = p.s;
    const int tid = threadIdx.x, row = (int)blockIdx.y;
    pdl_launch_dependents();
    const int pos = scan_position(p.c, row);
    if (p.c.fused && (int)blockIdx.x == S.heads * p.csplit) {
        pdl_wait();
        store_latent_row<CT, LA_WARPS>(p, row, pos, s_red);
        return;
    }
    const int h = (int)blockIdx.x / p.csplit, part = (int)blockIdx.x % p.csplit;
    const int nchunk = S.rp >> 3, cpc = (nchunk + p.csplit - 1) / p.csplit;
    const int c0 = min(nchunk, part * cpc), nc = min(nchunk, c0 + cpc) - c0;  // (rp <= 1024: at most 128 chunks)
    const int ndg = nc > 0 ? LA_CONSUMERS / nc : 0, cc = nc > 0 ? tid % nc : 0, dg = nc > 0 ? tid / nc : 0;
    const bool active = nc > 0 && dg < ndg;
    const bf16* const w = p.uk + (size_t)h * S.dp * S.rp + (size_t)(c0 + cc) * 8;
    Raw8<bf16> pre[PRE];
#pragma unroll
    for (int i = 0; i < PRE; ++i) {
        pre[i].zero();
        if (active && dg + i * ndg < S.dim) pre[i].load(w + (size_t)(dg + i * ndg) * S.rp);
    }
    pdl_wait();
    const float* const q = p.qdg + (size_t)row * p.ld + h * (S.dim + S.rot);
    float* const out = p.c.qp + ((size_t)row * S.heads + h) * S.row;
    if (active) {
        f32x2 a[4] = {0ull, 0ull, 0ull, 0ull};
        float v[PRE];
#pragma unroll
        for (int i = 0; i < PRE; ++i) v[i] = dg + i * ndg < S.dim ? __ldcg(q + dg + i * ndg) : 0.f;
#pragma unroll
        for (int i = 0; i < PRE; ++i) {
            const Pairs8 x = pre[i].pairs();
#pragma unroll
            for (int k = 0; k < 4; ++k) a[k] = fma2(x.p[k], pack2(v[i], v[i]), a[k]);
        }
#pragma unroll 1
        for (int d = dg + PRE * ndg; d < S.dim; d += ndg) {
            Raw8<bf16> r;
            r.load(w + (size_t)d * S.rp);
            const float qd = __ldcg(q + d);
            const Pairs8 x = r.pairs();
#pragma unroll
            for (int k = 0; k < 4; ++k) a[k] = fma2(x.p[k], pack2(qd, qd), a[k]);
        }
        ulonglong2* dst = reinterpret_cast<ulonglong2*>(s_part + ((size_t)dg * nc + cc) * 8);
        dst[0] = make_ulonglong2(a[0], a[1]);
        dst[1] = make_ulonglong2(a[2], a[3]);
    }
    __syncthreads();
    const int n = min(ndg, S.dim);
    for (int i = tid; i < nc * 8; i += LA_CONSUMERS) {
        float v = 0.f;
#pragma unroll 4
        for (int d = 0; d < n; ++d) v += s_part[(size_t)d * nc * 8 + i];
        out[c0 * 8 + i] = v * S.scale2;
    }
    if (part == 0) {
        const float2* const rope = p.rope + (size_t)pos * (S.rdims >> 1);
        for (int i = tid; i < S.row - S.rp; i += LA_CONSUMERS)
            out[S.rp + i] = i < S.rot ? S.scale2 * rotary_element(i, S.rdims, rope, [&](int j) { return __ldcg(q + S.dim + j); }) : 0.f;
    }
}

// Grid (heads * vsplit, rows), clusters of the vsplit blocks of a head: each merges the ranges for its part of the latent and hands
// that part to the others through distributed shared memory, then applies its rows of W_uv (four at a time per warp) and the gate.
template <typename OT>
__global__ void __launch_bounds__(LA_CONSUMERS) latent_output_kernel(const __grid_constant__ LatentAttnParams p) {
    __shared__ float s_w[CS_MAX_SPLIT];
    __shared__ __align__(16) float s_c[1024];
    __shared__ float2 s_part[512];
    constexpr int UR = 4, PRE = 2;  // rows per warp at a time; 256-value pieces of the first rows fetched before the wait
    const LatentShape& S = p.s;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = (int)blockIdx.y, cl = p.vsplit;
    const int h = (int)blockIdx.x / cl, part = (int)blockIdx.x % cl;
    pdl_launch_dependents();
    if (cl > 1) cluster_arrive();  // (waited for before the first store into another block's shared memory)
    const int vpc = (S.vdim + cl - 1) / cl, v0 = min(S.vdim, part * vpc), v1 = min(S.vdim, v0 + vpc);
    const bf16* const uv = p.uv + (size_t)h * S.vp * S.rp;
    const int rw = v0 + warp * UR;
    Raw8<bf16> pre[PRE][UR];
#pragma unroll
    for (int i = 0; i < PRE; ++i)
#pragma unroll
        for (int u = 0; u < UR; ++u) {
            const int e = (i * 32 + lane) * 8;
            pre[i][u].zero();
            if (rw < v1 && e < S.rp) pre[i][u].load(uv + (size_t)min(rw + u, v1 - 1) * S.rp + e);
        }
    const int npos = scan_position(p.c, row) + 1, range = scan_range(npos, p.c.nsplit), ns = (npos + range - 1) / range;
    pdl_wait();
    const size_t slot = ((size_t)row * S.heads + h) * p.c.nsplit;
    if (warp == 0) {  // weights of the ranges; ns <= 64
        const float sink2 = __ldg(p.sink + h) * 1.4426950408889634f;
        const float2 a = lane < ns ? __ldcg(p.c.part_ml + slot + lane) : make_float2(-INFINITY, 0.f);
        const float2 b = lane + 32 < ns ? __ldcg(p.c.part_ml + slot + 32 + lane) : make_float2(-INFINITY, 0.f);
        const float M = warp_max(fmaxf(sink2, fmaxf(a.x, b.x)));
        const float wa = exp2f(a.x - M), wb = exp2f(b.x - M);
        const float inv = 1.f / (warp_sum(fmaf(a.y, wa, b.y * wb)) + exp2f(sink2 - M));  // the sink: a term of the denominator only
        s_w[lane] = wa * inv;
        s_w[lane + 32] = wb * inv;
    }
    const float* const gate = p.qdg + (size_t)row * p.ld + p.off_g + h * S.vdim;
    const float g0 = lane < UR && rw + lane < v1 ? __ldcg(gate + rw + lane) : 0.f;
    __syncthreads();
    {
        const int cs = (S.rp / 8 + cl - 1) / cl * 8, c0 = min(S.rp, part * cs), np = (min(S.rp, c0 + cs) - c0) / 2;  // this block's column pairs
        const int nsg = np > 0 ? max(1, min(LA_CONSUMERS / np, 8)) : 0;                                              // threads per pair
        for (int i = tid; i < np * nsg; i += LA_CONSUMERS) {
            const int cp = i % np, sg = i / np;
            float2 a = make_float2(0.f, 0.f);
            const float* const src = p.c.part_acc + slot * S.rp + c0 + 2 * cp;
#pragma unroll 8
            for (int r = sg; r < ns; r += nsg) {
                const float2 x = __ldcg(reinterpret_cast<const float2*>(src + (size_t)r * S.rp));
                a.x = fmaf(x.x, s_w[r], a.x);
                a.y = fmaf(x.y, s_w[r], a.y);
            }
            s_part[i] = a;
        }
        __syncthreads();
        if (cl > 1) cluster_wait();
        for (int i = tid; i < np; i += LA_CONSUMERS) {
            float2 a = s_part[i];
            for (int k = 1; k < nsg; ++k) {
                const float2 x = s_part[k * np + i];
                a.x += x.x;
                a.y += x.y;
            }
            float* const at = s_c + c0 + 2 * i;
            if (cl == 1) *reinterpret_cast<float2*>(at) = a;
            else
                for (int r = 0; r < cl; ++r) {
                    st_cluster_f32(cluster_map(at, (uint32_t)r), a.x);
                    st_cluster_f32(cluster_map(at + 1, (uint32_t)r), a.y);
                }
        }
        if (cl > 1) cluster_sync_all();
        else __syncthreads();
    }
    OT* const out = static_cast<OT*>(p.out) + (size_t)row * p.ldo + h * S.vdim;
#pragma unroll 1
    for (int r0 = rw; r0 < v1; r0 += LA_WARPS * UR) {
        float d[UR];
#pragma unroll
        for (int u = 0; u < UR; ++u) d[u] = 0.f;
        auto piece = [&](const Raw8<bf16>(&w)[UR], int e) {
            const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(s_c + e), b = *reinterpret_cast<const ulonglong2*>(s_c + e + 4);
#pragma unroll
            for (int u = 0; u < UR; ++u) {
                const Pairs8 x = w[u].pairs();
                d[u] += sum2(fma2(x.p[0], a.x, fma2(x.p[1], a.y, fma2(x.p[2], b.x, mul2(x.p[3], b.y)))));
            }
        };
        int e = lane * 8;
        if (r0 == rw) {
#pragma unroll
            for (int i = 0; i < PRE; ++i, e += 256)
                if (e < S.rp) piece(pre[i], e);
        }
#pragma unroll 1
        for (; e < S.rp; e += 256) {
            Raw8<bf16> w[UR];
#pragma unroll
            for (int u = 0; u < UR; ++u) w[u].load(uv + (size_t)min(r0 + u, v1 - 1) * S.rp + e);
            piece(w, e);
        }
        __syncwarp();
        warp_sums<UR>(d);
        const float v = lane == 0 ? d[0] : lane == 1 ? d[1] : lane == 2 ? d[2] : d[3];
        if (lane < UR && r0 + lane < v1) put(out + r0 + lane, v * sigmoid(r0 == rw ? g0 : __ldcg(gate + r0 + lane)));
    }
}

}  // namespace l2b
