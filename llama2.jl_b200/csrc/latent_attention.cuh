// Latent attention (one cached latent and one shared rotated key part per position, a sink in the softmax, a sigmoid output gate)
// in its absorbed form: with q' = W_uk^T q_unrotated the score of a head against position t is
//     (q' . c_t + q_rotated . kr_t) * scale,
// and W_uv is applied once, to the weighted sum of the latents.  So a head reads one row [c | kr] per position for keys and values
// alike, and nothing per head is cached.
//
// One thread-block cluster of `cl` blocks serves GH heads of one row.  The blocks
//   1. split the columns of W_uk^T q and hand their part to the others through distributed shared memory,
//   2. split the positions: a producer warp brings the block's cache rows (contiguous) into a ring of shared-memory stages with bulk
//      asynchronous copies; a warp scores a batch of positions of a stage for all GH heads (their lane sums taken together)
//      and folds them into its running softmax, exp2 domain, all in f32,
//   3. exchange (maximum, sum, unnormalised latent) -- one cluster barrier -- and
//   4. split the rows of W_uv; the result is gated and stored.
// In a decode step (fused = 1) the blocks normalise and rotate the new position's latent and key themselves and one of them
// writes it to the cache; the weights of step 1 and the ring's first stages are fetched before the wait on the previous kernel.
// Many-token passes (fused = 0) read the new positions from the cache (latent_rows_kernel has written them); every row has
// its own position, and in batched decode its own cache.
#pragma once
#include "dense_ops.cuh"

namespace l2b {

constexpr int LA_WARPS = 8, LA_CONSUMERS = LA_WARPS * 32, LA_THREADS = LA_CONSUMERS + 32, LA_MAX_CL = 8, LA_MAX_STAGES = 4;

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
    int fused, cl, stages;
    int* status;
};
template <typename CT>
__host__ __device__ constexpr int la_batch() { return sizeof(CT) == 2 ? 4 : 2; }  // positions of a stage per warp
template <typename CT>
__host__ __device__ constexpr int la_stage_rows() { return LA_WARPS * la_batch<CT>(); }

// shared memory, offsets in floats
struct LaSmem {
    int ring, q, qf, kn, oc, scr, wml, rx_ml, rx_a, total;
};
__host__ __device__ inline LaSmem la_smem_layout(const LatentShape& s, int gh, int stage_floats, int stages) {
    LaSmem o;
    int n = 0;
    auto take = [&](int k) { const int at = n; n += (k + 3) & ~3; return at; };
    const int pieces = (s.row + 255) / 256;
    o.ring = take(stage_floats * stages);
    o.q = take(gh * (s.dim + s.rot));
    o.qf = take(gh * pieces * 256);
    o.kn = take(s.row);
    o.oc = take(gh * s.rp);
    o.wml = take(gh * 2 * LA_WARPS);
    o.rx_ml = take(gh * 2 * LA_MAX_CL);
    o.rx_a = take(gh * LA_MAX_CL * s.rp);
    // the absorb stage's partial columns and the warps' partial latents share a region
    const int absorb = LA_CONSUMERS * 8, warps = gh * LA_WARPS * s.rp;
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

// NI: 256-value pieces a cache row is spread over (32 lanes x 8 values each); GH: heads per cluster
template <typename CT, typename OT, int NI, int GH>
__global__ void __launch_bounds__(LA_THREADS) latent_attention_kernel(const __grid_constant__ LatentAttnParams p) {
    extern __shared__ __align__(128) float la_smem[];
    __shared__ __align__(8) uint64_t s_full[LA_MAX_STAGES], s_empty[LA_MAX_STAGES];
    __shared__ float s_red[LA_WARPS];
    constexpr int BATCH = la_batch<CT>(), SP = la_stage_rows<CT>();
    constexpr int PRE = 4;  // rows of W_uk per head a thread fetches before the wait
    const LatentShape& S = p.s;
    const int stage_bytes = SP * S.row * (int)sizeof(CT);
    const LaSmem L = la_smem_layout(S, GH, stage_bytes / 4, p.stages);
    uint8_t* const ring = reinterpret_cast<uint8_t*>(la_smem + L.ring);
    float *const q = la_smem + L.q, *const qf = la_smem + L.qf, *const kn = la_smem + L.kn, *const oc = la_smem + L.oc, *const scr = la_smem + L.scr,
                 *const wml = la_smem + L.wml, *const rx_ml = la_smem + L.rx_ml, *const rx_a = la_smem + L.rx_a;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int cl = p.cl, rank = cl > 1 ? (int)cluster_ctarank() : 0;
    const int h0 = (int)blockIdx.x / cl * GH, row = (int)blockIdx.y;
    pdl_launch_dependents();
    if (cl > 1) cluster_arrive();  // (waited for before the first store into another block's shared memory)
    const int pos = p.pos ? __ldcg(p.pos) : p.pos_list ? __ldcg(p.pos_list + row) : p.pos0 + row;
    const int npos = pos + 1, qd = S.dim + S.rot;
    CT* const cache = static_cast<CT*>(p.cache) + (size_t)row * p.cache_stride;
    const float2* const rope = p.rope + (size_t)pos * (S.rdims >> 1);
    const int chunk = (npos + cl - 1) / cl;
    const int t0 = min(npos, rank * chunk), t1 = min(npos, t0 + chunk);
    const int tc = p.fused ? min(t1, npos - 1) : t1;  // positions t0 .. tc-1 are read from the cache
    const int nstage = tc > t0 ? (tc - t0 + SP - 1) / SP : 0;
    const int vpc = (S.vdim + cl - 1) / cl, v0 = min(S.vdim, rank * vpc), nv = min(S.vdim, v0 + vpc) - v0;  // this block's rows of W_uv
    if (tid == 0) {
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(s_full + i, 1);
            mbar_init(s_empty + i, LA_WARPS);
        }
        fence_barrier_init();
        fence_proxy_async();
    }
    __syncthreads();
    bool dead = false;
    auto bring = [&](int j) {  // stage j of the producer (one lane)
        const int s = j % p.stages, use = j / p.stages;
        if (use > 0 && !mbar_wait_bounded(s_empty + s, (uint32_t)((use - 1) & 1))) return false;
        const int t = t0 + j * SP;
        const uint32_t bytes = (uint32_t)(min(SP, tc - t) * S.row * (int)sizeof(CT));
        mbar_arrive_expect_tx(s_full + s, bytes);
        bulk_g2s_plain(ring + (size_t)s * stage_bytes, cache + (size_t)t * S.row, bytes, s_full + s);
        return true;
    };

    // ---- this block's columns of W_uk^T: 8-column chunks [c0, c0 + nc); thread = (chunk, group of rows d)
    const int nchunk = S.rp >> 3, cpc = (nchunk + cl - 1) / cl;
    const int c0 = min(nchunk, rank * cpc), nc = min(nchunk, c0 + cpc) - c0;
    const int ndg = nc > 0 ? LA_CONSUMERS / nc : 0;  // (rp <= 1024: at most 128 chunks)
    const int cc = nc > 0 ? tid % nc : 0, dg = nc > 0 ? tid / nc : 0;
    const bool absorbing = nc > 0 && dg < ndg && tid < LA_CONSUMERS;
    const bf16* const ukp = p.uk + (size_t)h0 * S.dp * S.rp + (size_t)(c0 + cc) * 8;
    Raw8<bf16> pre[GH][PRE];
#pragma unroll
    for (int g = 0; g < GH; ++g)
#pragma unroll
        for (int i = 0; i < PRE; ++i) {
            pre[g][i].zero();
            if (absorbing && dg + i * ndg < S.dim) pre[g][i].load(ukp + ((size_t)g * S.dp + dg + i * ndg) * S.rp);
        }
    int brought = 0;
    if (warp == LA_WARPS) {
        if (lane == 0 && p.fused)  // earlier tokens wrote these rows
            for (; brought < min(nstage, p.stages); ++brought) bring(brought);
        for (int g = 0; g < GH; ++g) {  // this block's rows of W_uv into L2
            const char* w = reinterpret_cast<const char*>(p.uv + ((size_t)(h0 + g) * S.vp + v0) * S.rp);
            for (size_t o = (size_t)lane * 128; o < (size_t)nv * S.rp * 2; o += 32 * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(w + o));
        }
    }

    pdl_wait();
    const float* const in = p.qdg + (size_t)row * p.ld;
    if (warp == LA_WARPS) {
        if (lane == 0) {
            while (brought < nstage && brought < p.stages) bring(brought++);  // (a whole ring needs no waiting)
        }
    } else {
        for (int i = tid; i < GH * qd; i += LA_CONSUMERS) q[i] = __ldcg(in + h0 * qd + i);
        if (p.fused) {
            const float* down = in + p.off_d;
            float ss = 0.f;
            for (int i = tid; i < S.rank; i += LA_CONSUMERS) {
                const float v = __ldcg(down + i);
                oc[i] = v;
                ss = fmaf(v, v, ss);
            }
            const float scale = 1.f / sqrtf(block_sum_all<LA_WARPS>(ss, s_red) / (float)S.rank + S.eps);
            for (int i = tid; i < S.rp; i += LA_CONSUMERS) kn[i] = as_stored(cache, i < S.rank ? oc[i] * scale * __ldg(p.dnorm + i) : 0.f);
            for (int i = tid; i < S.row - S.rp; i += LA_CONSUMERS)
                kn[S.rp + i] = as_stored(cache, i < S.rot ? rotary_element(i, S.rdims, rope, [&](int j) { return __ldcg(down + S.rank + j); }) : 0.f);
        }
        partial_sync(LA_CONSUMERS);
        if (p.fused && h0 == 0 && rank == 0)
            for (int i = tid; i < S.row; i += LA_CONSUMERS) put(cache + (size_t)pos * S.row + i, kn[i]);
        // rotated part of the queries, and zeros behind the row
        for (int i = tid; i < GH * (NI * 256 - S.rp); i += LA_CONSUMERS) {
            const int g = i / (NI * 256 - S.rp), d = i - g * (NI * 256 - S.rp);
            qf[g * NI * 256 + lane_major(S.rp + d)] = d < S.rot ? S.scale2 * rotary_element(d, S.rdims, rope, [&](int j) { return q[g * qd + S.dim + j]; }) : 0.f;
        }
    }
    // ---- q' (this block's columns), a head at a time
    if (cl > 1) cluster_wait();
    if (warp < LA_WARPS)
#pragma unroll
        for (int g = 0; g < GH; ++g) {
            const float* const qg = q + g * qd;
            if (absorbing) {
                f32x2 a[4];
#pragma unroll
                for (int k = 0; k < 4; ++k) a[k] = 0ull;
#pragma unroll
                for (int i = 0; i < PRE; ++i) {
                    const int d = dg + i * ndg;
                    const float v = d < S.dim ? qg[d] : 0.f;
                    const Pairs8 w = pre[g][i].pairs();
#pragma unroll
                    for (int k = 0; k < 4; ++k) a[k] = fma2(w.p[k], pack2(v, v), a[k]);
                }
                for (int d = dg + PRE * ndg; d < S.dim; d += ndg) {
                    Raw8<bf16> r;
                    r.load(ukp + ((size_t)g * S.dp + d) * S.rp);
                    const Pairs8 w = r.pairs();
#pragma unroll
                    for (int k = 0; k < 4; ++k) a[k] = fma2(w.p[k], pack2(qg[d], qg[d]), a[k]);
                }
                ulonglong2* dst = reinterpret_cast<ulonglong2*>(scr + ((size_t)dg * nc + cc) * 8);
                dst[0] = make_ulonglong2(a[0], a[1]);
                dst[1] = make_ulonglong2(a[2], a[3]);
            }
            partial_sync(LA_CONSUMERS);
            const int n = min(ndg, S.dim);
            for (int i = tid; i < nc * 8; i += LA_CONSUMERS) {
                float v4[4] = {0.f, 0.f, 0.f, 0.f};
                int d = 0;
                for (; d + 4 <= n; d += 4)
#pragma unroll
                    for (int k = 0; k < 4; ++k) v4[k] += scr[(size_t)(d + k) * nc * 8 + i];
                for (; d < n; ++d) v4[0] += scr[(size_t)d * nc * 8 + i];
                const float v = ((v4[0] + v4[1]) + (v4[2] + v4[3])) * S.scale2;
                float* const at = qf + g * NI * 256 + lane_major(c0 * 8 + i);
                if (cl == 1) *at = v;
                else
                    for (int r = 0; r < cl; ++r) st_cluster_f32(cluster_map(at, (uint32_t)r), v);
            }
            if (g + 1 < GH) partial_sync(LA_CONSUMERS);
        }
    if (cl > 1) cluster_sync_all();
    else __syncthreads();

    // ---- positions t0 .. t1-1
    if (warp == LA_WARPS) {
        if (lane == 0)
            while (brought < nstage && !dead) dead = !bring(brought++);
        if (dead) {
            atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
            for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
        }
        __syncwarp();
    } else {
        float m[GH], l[GH];
        f32x2 acc[GH][NI][4];
#pragma unroll
        for (int g = 0; g < GH; ++g) {
            m[g] = -INFINITY;
            l[g] = 0.f;
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int k = 0; k < 4; ++k) acc[g][i][k] = 0ull;
        }
        for (int j = 0; j < nstage; ++j) {
            const int s = j % p.stages, tb = t0 + j * SP + warp * BATCH;
            if (!dead && !mbar_wait_bounded(s_full + s, (uint32_t)((j / p.stages) & 1))) dead = true;
            __syncwarp();
            if (!dead && tb < tc) {
                const CT* src = reinterpret_cast<const CT*>(ring + (size_t)s * stage_bytes) + (size_t)warp * BATCH * S.row;
                Raw8<CT> kr[BATCH][NI];
                f32x2 d2[BATCH * GH];
#pragma unroll
                for (int u = 0; u < BATCH * GH; ++u) d2[u] = 0ull;
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const int e = (i * 32 + lane) * 8;
#pragma unroll
                    for (int u = 0; u < BATCH; ++u) {
                        kr[u][i].zero();
                        if (tb + u < tc && e < S.row) kr[u][i].read(src + (size_t)u * S.row + e);
                    }
                    Pairs8 qv[GH];
#pragma unroll
                    for (int g = 0; g < GH; ++g) qv[g] = read_lane_major(qf + g * NI * 256, i, lane);
#pragma unroll
                    for (int u = 0; u < BATCH; ++u) {
                        const Pairs8 kv = kr[u][i].pairs();
#pragma unroll
                        for (int g = 0; g < GH; ++g)
#pragma unroll
                            for (int k = 0; k < 4; ++k) d2[u * GH + g] = fma2(qv[g].p[k], kv.p[k], d2[u * GH + g]);
                    }
                }
                float sc[BATCH * GH];
#pragma unroll
                for (int u = 0; u < BATCH * GH; ++u) sc[u] = sum2(d2[u]);
                warp_sums<BATCH * GH>(sc);
#pragma unroll
                for (int g = 0; g < GH; ++g) {
                    float mx = m[g];
#pragma unroll
                    for (int u = 0; u < BATCH; ++u) {
                        if (tb + u >= tc) sc[u * GH + g] = -INFINITY;
                        mx = fmaxf(mx, sc[u * GH + g]);
                    }
                    const float corr = exp2f(m[g] - mx);  // 0 for the first batch (its first position is always in range)
                    float ps = 0.f;
#pragma unroll
                    for (int u = 0; u < BATCH; ++u) {
                        sc[u * GH + g] = exp2f(sc[u * GH + g] - mx);
                        ps += sc[u * GH + g];
                    }
                    l[g] = fmaf(l[g], corr, ps);
                    m[g] = mx;
                    const f32x2 c2 = pack2(corr, corr);
#pragma unroll
                    for (int i = 0; i < NI; ++i)
#pragma unroll
                        for (int k = 0; k < 4; ++k) acc[g][i][k] = mul2(acc[g][i][k], c2);
                }
#pragma unroll
                for (int i = 0; i < NI; ++i)
#pragma unroll
                    for (int u = 0; u < BATCH; ++u) {
                        const Pairs8 kv = kr[u][i].pairs();
#pragma unroll
                        for (int g = 0; g < GH; ++g) {
                            const f32x2 w2 = pack2(sc[u * GH + g], sc[u * GH + g]);
#pragma unroll
                            for (int k = 0; k < 4; ++k) acc[g][i][k] = fma2(w2, kv.p[k], acc[g][i][k]);
                        }
                    }
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(s_empty + s);
        }
        if (p.fused && t1 == npos && t0 < t1 && warp == 0) {  // the position of this decode step
            float sc[GH];
            Pairs8 kv[NI];
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int e = (i * 32 + lane) * 8;
#pragma unroll
                for (int k = 0; k < 4; ++k) kv[i].p[k] = e < S.row ? *reinterpret_cast<const f32x2*>(kn + e + 2 * k) : 0ull;
            }
#pragma unroll
            for (int g = 0; g < GH; ++g) {
                f32x2 d = 0ull;
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const Pairs8 qv = read_lane_major(qf + g * NI * 256, i, lane);
#pragma unroll
                    for (int k = 0; k < 4; ++k) d = fma2(qv.p[k], kv[i].p[k], d);
                }
                sc[g] = warp_sum(sum2(d));
                const float mx = fmaxf(m[g], sc[g]), corr = exp2f(m[g] - mx), w = exp2f(sc[g] - mx);
                l[g] = fmaf(l[g], corr, w);
                m[g] = mx;
#pragma unroll
                for (int i = 0; i < NI; ++i)
#pragma unroll
                    for (int k = 0; k < 4; ++k) acc[g][i][k] = fma2(pack2(w, w), kv[i].p[k], mul2(acc[g][i][k], pack2(corr, corr)));
            }
        }
        if (dead && lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
#pragma unroll
        for (int g = 0; g < GH; ++g) {
            if (lane == 0) wml[g * 2 * LA_WARPS + warp] = m[g], wml[g * 2 * LA_WARPS + LA_WARPS + warp] = l[g];
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int e = (i * 32 + lane) * 8;
                if (e < S.rp) {
                    ulonglong2* dst = reinterpret_cast<ulonglong2*>(scr + (size_t)(g * LA_WARPS + warp) * S.rp + e);
                    dst[0] = make_ulonglong2(acc[g][i][0], acc[g][i][1]);
                    dst[1] = make_ulonglong2(acc[g][i][2], acc[g][i][3]);
                }
            }
        }
        partial_sync(LA_CONSUMERS);
        // ---- the warps of this block; the result goes to every block of the cluster
#pragma unroll
        for (int g = 0; g < GH; ++g) {
            const float* const ml = wml + g * 2 * LA_WARPS;
            float M = -INFINITY, wgt[LA_WARPS], Ls = 0.f;
#pragma unroll
            for (int w = 0; w < LA_WARPS; ++w) M = fmaxf(M, ml[w]);
#pragma unroll
            for (int w = 0; w < LA_WARPS; ++w) {
                wgt[w] = ml[w] == -INFINITY ? 0.f : exp2f(ml[w] - M);
                Ls = fmaf(ml[LA_WARPS + w], wgt[w], Ls);
            }
            for (int i = tid * 4; i < S.rp; i += LA_CONSUMERS * 4) {
                float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int w = 0; w < LA_WARPS; ++w) {
                    const float4 x = *reinterpret_cast<const float4*>(scr + (size_t)(g * LA_WARPS + w) * S.rp + i);
                    a.x = fmaf(x.x, wgt[w], a.x); a.y = fmaf(x.y, wgt[w], a.y); a.z = fmaf(x.z, wgt[w], a.z); a.w = fmaf(x.w, wgt[w], a.w);
                }
                float* const at = rx_a + (size_t)(g * LA_MAX_CL + rank) * S.rp + i;
                if (cl == 1) *reinterpret_cast<float4*>(at) = a;
                else
                    for (int r = 0; r < cl; ++r) st_cluster_f32x4(cluster_map(at, (uint32_t)r), a);
            }
            if (tid < cl) {
                float* const at = rx_ml + g * 2 * LA_MAX_CL + rank;
                if (cl == 1) at[0] = M, at[LA_MAX_CL] = Ls;
                else {
                    st_cluster_f32(cluster_map(at, (uint32_t)tid), M);
                    st_cluster_f32(cluster_map(at + LA_MAX_CL, (uint32_t)tid), Ls);
                }
            }
        }
    }
    if (cl > 1) cluster_sync_all();
    else __syncthreads();
    if (warp == LA_WARPS) return;

    // ---- the blocks of the cluster
#pragma unroll
    for (int g = 0; g < GH; ++g) {
        const float* const ml = rx_ml + g * 2 * LA_MAX_CL;
        const float sink2 = __ldg(p.sink + h0 + g) * 1.4426950408889634f;
        float M = sink2, wgt[LA_MAX_CL];
        for (int r = 0; r < cl; ++r) M = fmaxf(M, ml[r]);
        float Ls = exp2f(sink2 - M);  // the sink: a term of the denominator only
#pragma unroll
        for (int r = 0; r < LA_MAX_CL; ++r) {
            wgt[r] = r < cl && ml[r] != -INFINITY ? exp2f(ml[r] - M) : 0.f;
            if (r < cl) Ls = fmaf(ml[LA_MAX_CL + r], wgt[r], Ls);
        }
        const float inv = 1.f / Ls;
        for (int i = tid; i < S.rp; i += LA_CONSUMERS) {
            float a = 0.f;
#pragma unroll
            for (int r = 0; r < LA_MAX_CL; ++r)
                if (r < cl) a = fmaf(rx_a[(size_t)(g * LA_MAX_CL + r) * S.rp + i], wgt[r], a);
            oc[g * S.rp + i] = a * inv;
        }
    }
    partial_sync(LA_CONSUMERS);

    // ---- this block's rows of W_uv, four at a time per warp, gated
    OT* const out = static_cast<OT*>(p.out) + (size_t)row * p.ldo;
    constexpr int UR = 4;
#pragma unroll 1
    for (int r0 = warp * UR; r0 < GH * nv; r0 += LA_WARPS * UR) {
        float d[UR], gate[UR];
        Raw8<bf16> w[UR][NI];
#pragma unroll
        for (int u = 0; u < UR; ++u) {
            const int r = min(r0 + u, GH * nv - 1), g = GH == 1 ? 0 : r / nv, v = v0 + r - g * nv;
            const bf16* src = p.uv + ((size_t)(h0 + g) * S.vp + v) * S.rp;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int e = (i * 32 + lane) * 8;
                w[u][i].zero();
                if (e < S.rp) w[u][i].load(src + e);
            }
            gate[u] = __ldcg(in + p.off_g + (h0 + g) * S.vdim + v);
        }
#pragma unroll
        for (int u = 0; u < UR; ++u) {
            const int r = min(r0 + u, GH * nv - 1), g = GH == 1 ? 0 : r / nv;
            f32x2 a = 0ull;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int e = (i * 32 + lane) * 8;
                if (e < S.rp) {
                    const Pairs8 x = w[u][i].pairs();
                    const ulonglong2 o0 = *reinterpret_cast<const ulonglong2*>(oc + g * S.rp + e), o1 = *reinterpret_cast<const ulonglong2*>(oc + g * S.rp + e + 4);
                    a = fma2(x.p[0], o0.x, a); a = fma2(x.p[1], o0.y, a); a = fma2(x.p[2], o1.x, a); a = fma2(x.p[3], o1.y, a);
                }
            }
            d[u] = sum2(a);
        }
        warp_sums<UR>(d);
        if (lane == 0)
#pragma unroll
            for (int u = 0; u < UR; ++u)
                if (r0 + u < GH * nv) {
                    const int r = r0 + u, g = GH == 1 ? 0 : r / nv, v = v0 + r - g * nv;
                    put(out + (h0 + g) * S.vdim + v, d[u] * sigmoid(gate[u]));
                }
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
