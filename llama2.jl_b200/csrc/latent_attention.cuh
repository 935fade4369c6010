// Latent attention (one cached latent and one shared rotated key part per position, a sink in the softmax, a sigmoid output gate)
// in its absorbed form: with q' = W_uk^T q_unrotated the score of a head against position t is
//     (q' . c_t + q_rotated . kr_t) * scale,
// and W_uv is applied once, to the weighted sum of the latents.  So a head reads one row [c | kr] per position for keys and values
// alike, and nothing per head is cached.
//
// One thread-block cluster of `cl` blocks serves one (row, head).  The blocks
//   1. split the columns of W_uk^T q and hand their part to the others through distributed shared memory,
//   2. split the positions: a warp scores a batch of LA_BATCH positions (their lane reductions interleaved) and folds them into
//      its running softmax, exp2 domain, all in f32,
//   3. exchange (maximum, sum, unnormalised latent) -- one cluster barrier -- and
//   4. split the rows of W_uv; the result is gated and stored.
// In a decode step (fused = 1) the blocks normalise and rotate the new position's latent and key themselves and one of them
// writes it to the cache; the weights and the cached rows of the first batch are fetched before the wait on the previous kernel.
// Many-token passes (fused = 0) read the new positions from the cache (latent_rows_kernel has written them); every row has
// its own position, and in batched decode its own cache.
#pragma once
#include "dense_ops.cuh"

namespace l2b {

constexpr int LA_WARPS = 8, LA_THREADS = LA_WARPS * 32, LA_MAX_CL = 8;

struct LatentShape {
    int heads, dim, rot, rdims, vdim, rank;  // rdims: rotated dimensions of the rot part
    int rp, row;    // rank rounded up to 8; cache row length: rp + rot rounded up to 8
    int dp, vp;     // stored rows per head of W_uk / W_uv
    float scale2;   // scale * log2(e)
    float eps;
};
struct LatentAttnParams {
    LatentShape s;
    const float* qdg;       // [rows][ld]: q, down projection, gate
    int ld, off_d, off_g;
    const bf16* uk;         // [heads * dp][rp]
    const bf16* uv;         // [heads * vp][rp]
    const float* sink;      // [heads]
    const float* dnorm;     // [rank]
    const float2* rope;     // [positions][rdims / 2]
    void* cache;            // [positions][row]
    size_t cache_stride;    // elements between the caches of consecutive rows (batched decode), else 0
    const int* pos;         // decode: device scalar
    const int* pos_list;    // batched decode: position of every row
    int pos0;               // otherwise row r sits at pos0 + r
    void* out;              // [rows][ldo]
    int ldo;
    int fused, cl;
};
// shared memory in floats
struct LaSmem {
    int q, qf, kn, oc, scr, wml, rx_ml, rx_a, total;
};
__host__ __device__ inline LaSmem la_smem_layout(const LatentShape& s) {
    LaSmem o;
    int n = 0;
    auto take = [&](int k) { const int at = n; n += (k + 3) & ~3; return at; };
    o.q = take(s.dim + s.rot);
    o.qf = take(s.row);
    o.kn = take(s.row);
    o.oc = take(s.rp);
    o.wml = take(2 * LA_WARPS);
    o.rx_ml = take(2 * LA_MAX_CL);
    o.rx_a = take(LA_MAX_CL * s.rp);
    // the absorb stage's partial columns and the warps' partial latents share a region
    const int absorb = LA_THREADS * 8, warps = LA_WARPS * s.row;
    o.scr = take(absorb > warps ? absorb : warps);
    o.total = n;
    return o;
}

__device__ __forceinline__ uint32_t cluster_ctarank() {
    uint32_t r;
    asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
    return r;
}
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

// NI: 256-value pieces a cache row is spread over (32 lanes x 8 values each)
template <typename CT, typename OT, int NI>
__global__ void __launch_bounds__(LA_THREADS) latent_attention_kernel(const __grid_constant__ LatentAttnParams p) {
    extern __shared__ __align__(16) float la_smem[];
    __shared__ float s_red[LA_WARPS];
    constexpr int BATCH = NI <= 2 ? 4 : 2;
    constexpr int PRE = 4;  // rows of W_uk a thread fetches before the wait
    const LatentShape& S = p.s;
    const LaSmem L = la_smem_layout(S);
    float *const q = la_smem + L.q, *const qf = la_smem + L.qf, *const kn = la_smem + L.kn, *const oc = la_smem + L.oc, *const scr = la_smem + L.scr,
                 *const wml = la_smem + L.wml, *const rx_ml = la_smem + L.rx_ml, *const rx_a = la_smem + L.rx_a;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int cl = p.cl, rank = cl > 1 ? (int)cluster_ctarank() : 0;
    const int h = (int)blockIdx.x / cl, row = (int)blockIdx.y;
    pdl_launch_dependents();
    if (cl > 1) cluster_arrive();  // (waited for before the first store into another block's shared memory)
    const int pos = p.pos ? __ldcg(p.pos) : p.pos_list ? __ldcg(p.pos_list + row) : p.pos0 + row;
    const int npos = pos + 1;
    CT* const cache = static_cast<CT*>(p.cache) + (size_t)row * p.cache_stride;
    const float2* const rope = p.rope + (size_t)pos * (S.rdims >> 1);

    // ---- this block's columns of W_uk^T: 8-column chunks [c0, c0 + nc); thread = (chunk, group of rows d)
    const int nchunk = S.rp >> 3, cpc = (nchunk + cl - 1) / cl;
    const int c0 = min(nchunk, rank * cpc), nc = min(nchunk, c0 + cpc) - c0;
    const int ndg = nc > 0 ? LA_THREADS / nc : 0;  // (rp <= 1024: at most 128 chunks)
    const int cc = nc > 0 ? tid % nc : 0, dg = nc > 0 ? tid / nc : 0;
    const bool absorbing = nc > 0 && dg < ndg;
    const bf16* const ukp = p.uk + (size_t)h * S.dp * S.rp + (size_t)(c0 + cc) * 8;
    Raw8<bf16> pre[PRE];
#pragma unroll
    for (int i = 0; i < PRE; ++i) {
        pre[i].zero();
        if (absorbing && dg + i * ndg < S.dim) pre[i].load(ukp + (size_t)(dg + i * ndg) * S.rp);
    }
    // ---- this block's rows of W_uv into L2, this warp's first positions into registers
    const int vpc = (S.vdim + cl - 1) / cl, v0 = min(S.vdim, rank * vpc), v1 = min(S.vdim, v0 + vpc);
    const bf16* const uvp = p.uv + ((size_t)h * S.vp + v0) * S.rp;
    {
        const size_t bytes = (size_t)(v1 - v0) * S.rp * 2;
        for (size_t o = (size_t)tid * 128; o < bytes; o += (size_t)LA_THREADS * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(uvp) + o));
    }
    const int chunk = (npos + cl - 1) / cl;
    const int t0 = min(npos, rank * chunk), t1 = min(npos, t0 + chunk);
    const int known = p.fused ? npos - 1 : npos;  // positions below this are in the cache
    Raw8<CT> kr[BATCH][NI];
    auto fetch = [&](int tb) {
#pragma unroll
        for (int u = 0; u < BATCH; ++u)
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                kr[u][i].zero();
                const int e = (i * 32 + lane) * 8;
                if (tb + u < t1 && tb + u < known && e < S.row) kr[u][i].load(cache + (size_t)(tb + u) * S.row + e);
            }
    };
    const int tb0 = t0 + warp * BATCH;
    if (p.fused) fetch(tb0);  // earlier tokens wrote these

    pdl_wait();
    const float* const in = p.qdg + (size_t)row * p.ld;
    const float* const qh = in + h * (S.dim + S.rot);
    if (!p.fused) fetch(tb0);
    for (int i = tid; i < S.dim + S.rot; i += LA_THREADS) q[i] = __ldcg(qh + i);
    if (p.fused) {
        const float* down = in + p.off_d;
        float ss = 0.f;
        for (int i = tid; i < S.rank; i += LA_THREADS) {
            const float v = __ldcg(down + i);
            oc[i] = v;
            ss = fmaf(v, v, ss);
        }
        const float scale = 1.f / sqrtf(block_sum_all<LA_WARPS>(ss, s_red) / (float)S.rank + S.eps);
        for (int i = tid; i < S.rp; i += LA_THREADS) kn[i] = as_stored(cache, i < S.rank ? oc[i] * scale * __ldg(p.dnorm + i) : 0.f);
        for (int i = tid; i < S.row - S.rp; i += LA_THREADS)
            kn[S.rp + i] = as_stored(cache, i < S.rot ? rotary_element(i, S.rdims, rope, [&](int j) { return __ldcg(down + S.rank + j); }) : 0.f);
    }
    __syncthreads();
    if (p.fused && h == 0 && rank == 0)
        for (int i = tid; i < S.row; i += LA_THREADS) put(cache + (size_t)pos * S.row + i, kn[i]);

    // ---- q' (this block's columns)
    {
        float a[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) a[k] = 0.f;
        if (absorbing) {
#pragma unroll
            for (int i = 0; i < PRE; ++i) {
                const int d = dg + i * ndg;
                const float qd = d < S.dim ? q[d] : 0.f;
                const Vec8 w = pre[i].get();
#pragma unroll
                for (int k = 0; k < 8; ++k) a[k] = fmaf(w.v[k], qd, a[k]);
            }
            for (int d = dg + PRE * ndg; d < S.dim; d += ndg) {
                Raw8<bf16> r;
                r.load(ukp + (size_t)d * S.rp);
                const Vec8 w = r.get();
#pragma unroll
                for (int k = 0; k < 8; ++k) a[k] = fmaf(w.v[k], q[d], a[k]);
            }
            float4* dst = reinterpret_cast<float4*>(scr + ((size_t)dg * nc + cc) * 8);
            dst[0] = make_float4(a[0], a[1], a[2], a[3]);
            dst[1] = make_float4(a[4], a[5], a[6], a[7]);
        }
        for (int i = tid; i < S.row - S.rp; i += LA_THREADS) qf[S.rp + i] = i < S.rot ? S.scale2 * rotary_element(i, S.rdims, rope, [&](int j) { return q[S.dim + j]; }) : 0.f;
        __syncthreads();
        if (cl > 1) cluster_wait();
        for (int i = tid; i < nc * 8; i += LA_THREADS) {
            float v = 0.f;
            const int n = min(ndg, S.dim);
            for (int g = 0; g < n; ++g) v += scr[(size_t)g * nc * 8 + i];
            v *= S.scale2;
            if (cl == 1) qf[c0 * 8 + i] = v;
            else
                for (int r = 0; r < cl; ++r) st_cluster_f32(cluster_map(qf + c0 * 8 + i, (uint32_t)r), v);
        }
        if (cl > 1) cluster_sync_all();
        else __syncthreads();
    }

    // ---- positions t0 .. t1-1
    float m = -INFINITY, l = 0.f;
    {
        Vec8 qv[NI], acc[NI];
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int e = (i * 32 + lane) * 8;
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                qv[i].v[k] = e < S.row ? qf[e + k] : 0.f;
                acc[i].v[k] = 0.f;
            }
        }
        for (int tb = tb0; tb < t1; tb += LA_WARPS * BATCH) {
            if (tb != tb0) fetch(tb);
            float s[BATCH];
            Vec8 kv[BATCH][NI];
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                const bool own = tb + u >= known && tb + u < t1;  // the position of this decode step: not from the cache
                float d = 0.f;
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    kv[u][i] = kr[u][i].get();
                    const int e = (i * 32 + lane) * 8;
                    if (own && e < S.row)
#pragma unroll
                        for (int k = 0; k < 8; ++k) kv[u][i].v[k] = kn[e + k];
#pragma unroll
                    for (int k = 0; k < 8; ++k) d = fmaf(qv[i].v[k], kv[u][i].v[k], d);
                }
                s[u] = d;
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int u = 0; u < BATCH; ++u) s[u] += __shfl_xor_sync(0xffffffffu, s[u], o);
            float mx = m;
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                if (tb + u >= t1) s[u] = -INFINITY;
                mx = fmaxf(mx, s[u]);
            }
            const float corr = exp2f(m - mx);  // 0 for the first batch
            float ps = 0.f;
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                s[u] = exp2f(s[u] - mx);
                ps += s[u];
            }
            l = fmaf(l, corr, ps);
            m = mx;
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int k = 0; k < 8; ++k) {
                    float a = acc[i].v[k] * corr;
#pragma unroll
                    for (int u = 0; u < BATCH; ++u) a = fmaf(s[u], kv[u][i].v[k], a);
                    acc[i].v[k] = a;
                }
        }
        if (lane == 0) wml[warp] = m, wml[LA_WARPS + warp] = l;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int e = (i * 32 + lane) * 8;
            if (e < S.rp) {
                float4* dst = reinterpret_cast<float4*>(scr + (size_t)warp * S.row + e);
                dst[0] = make_float4(acc[i].v[0], acc[i].v[1], acc[i].v[2], acc[i].v[3]);
                dst[1] = make_float4(acc[i].v[4], acc[i].v[5], acc[i].v[6], acc[i].v[7]);
            }
        }
    }
    __syncthreads();

    // ---- the warps of this block, then the blocks of the cluster
    {
        float M = -INFINITY, wgt[LA_WARPS], Ls = 0.f;
#pragma unroll
        for (int w = 0; w < LA_WARPS; ++w) M = fmaxf(M, wml[w]);
#pragma unroll
        for (int w = 0; w < LA_WARPS; ++w) {
            wgt[w] = wml[w] == -INFINITY ? 0.f : exp2f(wml[w] - M);
            Ls = fmaf(wml[LA_WARPS + w], wgt[w], Ls);
        }
        for (int i = tid; i < S.rp; i += LA_THREADS) {
            float a = 0.f;
#pragma unroll
            for (int w = 0; w < LA_WARPS; ++w) a = fmaf(scr[(size_t)w * S.row + i], wgt[w], a);
            if (cl == 1) rx_a[i] = a;
            else
                for (int r = 0; r < cl; ++r) st_cluster_f32(cluster_map(rx_a + rank * S.rp + i, (uint32_t)r), a);
        }
        if (tid < cl) {
            if (cl == 1) rx_ml[0] = M, rx_ml[LA_MAX_CL] = Ls;
            else {
                st_cluster_f32(cluster_map(rx_ml + rank, (uint32_t)tid), M);
                st_cluster_f32(cluster_map(rx_ml + LA_MAX_CL + rank, (uint32_t)tid), Ls);
            }
        }
        if (cl > 1) cluster_sync_all();
        else __syncthreads();
        const float sink2 = __ldg(p.sink + h) * 1.4426950408889634f;
        M = sink2;
        for (int r = 0; r < cl; ++r) M = fmaxf(M, rx_ml[r]);
        Ls = exp2f(sink2 - M);  // the sink: a term of the denominator only
        for (int r = 0; r < cl; ++r) Ls = fmaf(rx_ml[LA_MAX_CL + r], rx_ml[r] == -INFINITY ? 0.f : exp2f(rx_ml[r] - M), Ls);
        const float inv = 1.f / Ls;
        for (int i = tid; i < S.rp; i += LA_THREADS) {
            float a = 0.f;
            for (int r = 0; r < cl; ++r) a = fmaf(rx_a[r * S.rp + i], rx_ml[r] == -INFINITY ? 0.f : exp2f(rx_ml[r] - M), a);
            oc[i] = a * inv;
        }
        __syncthreads();
    }

    // ---- this block's rows of W_uv, gated
    OT* const out = static_cast<OT*>(p.out) + (size_t)row * p.ldo + h * S.vdim;
    const float* const gate = in + p.off_g + h * S.vdim;
    for (int v = v0 + warp; v < v1; v += LA_WARPS) {
        const bf16* w = uvp + (size_t)(v - v0) * S.rp;
        float d = 0.f;
        for (int e = lane * 8; e < S.rp; e += 256) {
            Raw8<bf16> r;
            r.load(w + e);
            const Vec8 x = r.get();
#pragma unroll
            for (int k = 0; k < 8; ++k) d = fmaf(x.v[k], oc[e + k], d);
        }
        d = warp_sum(d);
        if (lane == 0) put(out + v, d * sigmoid(__ldcg(gate + v)));
    }
}

// Many-token passes: latent (normalised) and rotated key of every row into the cache.  One block per row.
template <typename CT>
__global__ void __launch_bounds__(128) latent_rows_kernel(const __grid_constant__ LatentAttnParams p) {
    __shared__ float s_red[4];
    const LatentShape& S = p.s;
    const int row = (int)blockIdx.x, tid = threadIdx.x;
    const int pos = p.pos_list ? __ldcg(p.pos_list + row) : p.pos0 + row;
    CT* const dst = static_cast<CT*>(p.cache) + (size_t)row * p.cache_stride + (size_t)pos * S.row;
    const float* down = p.qdg + (size_t)row * p.ld + p.off_d;
    float ss = 0.f;
    for (int i = tid; i < S.rank; i += 128) ss = fmaf(down[i], down[i], ss);
    const float scale = 1.f / sqrtf(block_sum_all<4>(ss, s_red) / (float)S.rank + S.eps);
    for (int i = tid; i < S.rp; i += 128) put(dst + i, i < S.rank ? down[i] * scale * __ldg(p.dnorm + i) : 0.f);
    const float2* rope = p.rope + (size_t)pos * (S.rdims >> 1);
    for (int i = tid; i < S.row - S.rp; i += 128)
        put(dst + S.rp + i, i < S.rot ? rotary_element(i, S.rdims, rope, [&](int j) { return down[S.rank + j]; }) : 0.f);
}

}  // namespace l2b
