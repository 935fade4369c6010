// Latent attention (one cached latent and one shared rotated key part per position, a sink in the softmax, a sigmoid output gate)
// in its absorbed form: with q' = W_uk^T q_unrotated the score of a head against position t is
//     (q' . c_t + q_rotated . kr_t) * scale,
// and W_uv is applied once, to the weighted sum of the latents.  So a head reads one row [c | kr] per position for keys and values
// alike, and nothing per head is cached.  Three kernels, chained with programmatic dependent launch in a decode step:
//   latent_query_kernel   q' and the rotated query part of every (row, head); in a decode step one more block normalises and
//                         rotates the new position's latent and key and writes them to the cache;
//   latent_scan_mma_kernel (bf16 cache)  a block takes 16 heads and a range of positions, whose cache rows a producer warp brings into
//                         shared memory with bulk asynchronous copies; scores and weighted sums on the tensor cores with q' and
//                         the weights as two bf16 terms (high and low part: 16 significant bits), running softmax in the
//                         exp2 domain in f32; one partial result (maximum, sum, unnormalised latent) per head and range;
//   latent_scan_kernel    (f32 cache)  the same on the CUDA cores, 8 heads per block, one per warp;
//   latent_output_kernel  merges the ranges and the sink, applies W_uv and the gate.
// (One kernel with clusters that exchange q' and the partial results through distributed shared memory was about twice as slow: its
// code is several times as long and runs once per launch, so that fetching instructions bounds it.)
// Weights, and the cache rows that earlier tokens wrote, are fetched before the wait on the previous kernel.
// Many-token passes run the same kernels over rows with their own positions (batched decode: also their own caches), the new
// positions written by latent_rows_kernel.
#pragma once
#include "dense_ops.cuh"

namespace l2b {

constexpr int LA_WARPS = 8, LA_CONSUMERS = LA_WARPS * 32, LA_SCAN_THREADS = LA_CONSUMERS + 32;
constexpr int LA_STAGE_ROWS = 16, LA_MAX_STAGES = 4, LA_MAX_SPLIT = 64, LA_MIN_RANGE = 32;

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
    float* qp;              // [rows][heads][row]: q' and rotated part, times scale2
    float2* part_ml;        // [rows][heads][nsplit]
    float* part_acc;        // [rows][heads][nsplit][rp]
    int csplit, nsplit, vsplit;  // blocks per head (query), ranges of positions (scan), blocks per head (output)
    int stages;             // ring of the scan kernel
    void* out;              // [rows][ldo]
    int ldo;
    int fused;              // decode step: the new position's row is written by latent_query_kernel
    int* status;
};
__device__ __forceinline__ int latent_position(const LatentAttnParams& p, int row) {
    return p.pos ? __ldcg(p.pos) : p.pos_list ? __ldcg(p.pos_list + row) : p.pos0 + row;
}
// positions per range
__device__ __forceinline__ int latent_range(int npos, int nsplit) { return max(LA_MIN_RANGE, (npos + nsplit - 1) / nsplit); }

__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

// Latent (normalised) and rotated key of one position into its cache row; NW warps.
template <typename CT, int NW>
__device__ __forceinline__ void store_latent_row(const LatentAttnParams& p, int row, int pos, float* s_red) {
    const LatentShape& S = p.s;
    const int tid = threadIdx.x;
    CT* const dst = static_cast<CT*>(p.cache) + (size_t)row * p.cache_stride + (size_t)pos * S.row;
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
    store_latent_row<CT, 4>(p, (int)blockIdx.x, latent_position(p, (int)blockIdx.x), s_red);
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
    const int pos = latent_position(p, row);
    if (p.fused && (int)blockIdx.x == S.heads * p.csplit) {
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
    float* const out = p.qp + ((size_t)row * S.heads + h) * S.row;
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

// ---- scan on the tensor cores -----------------------------------------------------------------------------------
constexpr int LM_HEADS = 16;  // heads per block = M of mma.m16n8k16

// Bytes between cache rows in shared memory: 16 mod 128, so that eight rows of a fragment load fall in different banks; at least
// 16 bytes of zeros follow the row (the last K = 16 step may reach 8 values beyond it).
__host__ __device__ inline int lm_pitch(int row) { return (row * 2 + 127) / 128 * 128 + 16; }
__host__ __device__ inline int lm_stage_bytes(int row) { return LA_STAGE_ROWS * lm_pitch(row); }

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// x = hi + lo with both bf16: two values -> two packed words
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// Grid (nsplit * groups of 16 heads, rows).  N: K = 16 steps of a cache row, and pairs of 8-column tiles of the latent, per warp at most.
template <int N>
__global__ void __launch_bounds__(LA_SCAN_THREADS) latent_scan_mma_kernel(const __grid_constant__ LatentAttnParams p) {
    extern __shared__ __align__(128) uint8_t la_ring[];  // [stages][LA_STAGE_ROWS][pitch]
    __shared__ __align__(8) uint64_t s_full[LA_MAX_STAGES], s_empty[LA_MAX_STAGES];
    __shared__ float s_s[LA_WARPS][LM_HEADS][LA_STAGE_ROWS + 1];             // the warps' shares of the scores
    __shared__ __align__(16) uint32_t s_hi[LM_HEADS][12], s_lo[LM_HEADS][12];  // weights of a stage: 16 bf16 per head (rows padded)
    __shared__ float s_corr[LM_HEADS];
    constexpr int KS = N, NT = N;
    const LatentShape& S = p.s;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = (int)blockIdx.y;
    const int split = (int)blockIdx.x % p.nsplit, h0 = (int)blockIdx.x / p.nsplit * LM_HEADS;
    const int pitch = lm_pitch(S.row), stage_bytes = lm_stage_bytes(S.row);
    pdl_launch_dependents();
    if (tid == 0) {
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(s_full + i, 1);
            mbar_init(s_empty + i, LA_WARPS);
        }
        fence_barrier_init();
        fence_proxy_async();
    }
    for (int i = tid; i < p.stages * LA_STAGE_ROWS; i += LA_SCAN_THREADS)  // zeros behind every row
        for (int k = S.row * 2; k < pitch; k += 16) *reinterpret_cast<uint4*>(la_ring + (size_t)i * pitch + k) = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
    const int npos = latent_position(p, row) + 1, range = latent_range(npos, p.nsplit);
    const int t0 = min(npos, split * range), t1 = min(npos, t0 + range);
    const int nstage = (t1 - t0 + LA_STAGE_ROWS - 1) / LA_STAGE_ROWS;

    if (warp == LA_WARPS) {
        const bf16* const cache = static_cast<const bf16*>(p.cache) + (size_t)row * p.cache_stride;
        bool waited = false;
        for (int j = 0; j < nstage; ++j) {
            const int s = j % p.stages, use = j / p.stages, t = t0 + j * LA_STAGE_ROWS, te = min(t1, t + LA_STAGE_ROWS);
            if (!waited && (!p.fused || te == npos)) {  // rows of earlier tokens need not be waited for
                pdl_wait();
                waited = true;
            }
            if (!__all_sync(0xffffffffu, use == 0 || mbar_wait_bounded(s_empty + s, (uint32_t)((use - 1) & 1)))) {
                if (lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
                for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
                break;
            }
            if (lane == 0) mbar_arrive_expect_tx(s_full + s, (uint32_t)((te - t) * S.row * 2));
            __syncwarp();
            if (lane < te - t) bulk_g2s_plain(la_ring + (size_t)s * stage_bytes + lane * pitch, cache + (size_t)(t + lane) * S.row, (uint32_t)(S.row * 2), s_full + s);
        }
        return;
    }
    pdl_wait();
    const int g = lane >> 2, t4 = lane & 3;
    // this warp's K steps (warp, warp + 8, ...) of q', as A fragments in two terms
    uint32_t qhi[KS][4], qlo[KS][4];
#pragma unroll
    for (int i = 0; i < KS; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const int h = h0 + g + 8 * (k & 1), e = (warp + LA_WARPS * i) * 16 + 8 * (k >> 1) + 2 * t4;
            float2 v = make_float2(0.f, 0.f);
            if (h < S.heads && e < S.row) v = __ldcg(reinterpret_cast<const float2*>(p.qp + ((size_t)row * S.heads + h) * S.row + e));
            split2(v.x, v.y, qhi[i][k], qlo[i][k]);
        }
    float acc[NT][2][4];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int k = 0; k < 8; ++k) acc[i][k >> 2][k & 3] = 0.f;
    const int sh = tid >> 4, sp = tid & 15;  // softmax: this thread's head and position of a stage
    float m = -INFINITY, l = 0.f;
    bool dead = false;
#pragma unroll 1
    for (int j = 0; j < nstage; ++j) {
        const int s = j % p.stages, n = min(LA_STAGE_ROWS, t1 - t0 - j * LA_STAGE_ROWS);
        if (!dead && !__all_sync(0xffffffffu, mbar_wait_bounded(s_full + s, (uint32_t)((j / p.stages) & 1)))) dead = true;
        __syncwarp();
        const uint8_t* const st = la_ring + (size_t)s * stage_bytes;
        {
            float d[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
            for (int i = 0; i < KS; ++i) {
                const int k0 = (warp + LA_WARPS * i) * 16;
                if (k0 < S.row)
#pragma unroll
                    for (int t = 0; t < 2; ++t) {  // positions 8t .. 8t+7 of the stage
                        const uint8_t* at = st + (8 * t + g) * pitch + (k0 + 2 * t4) * 2;
                        const uint32_t b0 = *reinterpret_cast<const uint32_t*>(at), b1 = *reinterpret_cast<const uint32_t*>(at + 16);
                        mma_bf16(d[t], qhi[i], b0, b1);
                        mma_bf16(d[t], qlo[i], b0, b1);
                    }
            }
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int k = 0; k < 4; ++k) s_s[warp][g + 8 * (k >> 1)][8 * t + 2 * t4 + (k & 1)] = d[t][k];
        }
        // rows that were not copied (a last, partial stage) weigh nothing, but must hold numbers
        for (int i = n * (pitch / 16) + tid; i < LA_STAGE_ROWS * (pitch / 16); i += LA_CONSUMERS)
            *reinterpret_cast<uint4*>(la_ring + (size_t)s * stage_bytes + (size_t)i * 16) = make_uint4(0u, 0u, 0u, 0u);
        partial_sync(LA_CONSUMERS);
        {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < LA_WARPS; ++w) v += s_s[w][sh][sp];
            if (sp >= n) v = -INFINITY;  // (positions beyond the range: stale rows)
            float mx = v;
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            mx = fmaxf(m, mx);
            const float corr = exp2f(m - mx), w = exp2f(v - mx);
            float sum = w;
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l = fmaf(l, corr, sum);
            m = mx;
            const float w1 = __shfl_down_sync(0xffffffffu, w, 1);
            if ((sp & 1) == 0) split2(w, w1, s_hi[sh][sp >> 1], s_lo[sh][sp >> 1]);
            if (sp == 0) s_corr[sh] = corr;
        }
        partial_sync(LA_CONSUMERS);
        {
            const float ca = s_corr[g], cb = s_corr[g + 8];
            const uint32_t ahi[4] = {s_hi[g][t4], s_hi[g + 8][t4], s_hi[g][t4 + 4], s_hi[g + 8][t4 + 4]};
            const uint32_t alo[4] = {s_lo[g][t4], s_lo[g + 8][t4], s_lo[g][t4 + 4], s_lo[g + 8][t4 + 4]};
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int c0 = (warp + LA_WARPS * i) * 16;  // columns c0 .. c0+15: two tiles
                if (c0 >= S.rp) continue;                   // (uniform over the warp)
#pragma unroll
                for (int k = 0; k < 8; ++k) acc[i][k >> 2][k & 3] *= (k & 2) ? cb : ca;
                uint32_t b[4];
                // lanes 0-7: positions 0-7, columns c0..; 8-15: positions 8-15; 16-31: the same for columns c0+8..
                ldmatrix4_trans(b, smem_u32(st + (lane & 15) * pitch + (c0 + 8 * (lane >> 4)) * 2));
                mma_bf16(acc[i][0], ahi, b[0], b[1]);
                mma_bf16(acc[i][0], alo, b[0], b[1]);
                mma_bf16(acc[i][1], ahi, b[2], b[3]);
                mma_bf16(acc[i][1], alo, b[2], b[3]);
            }
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(s_empty + s);
    }
    if (dead && lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
    if (t0 >= t1) return;  // (a range without positions is not read by the merge)
    if (sp == 0 && h0 + sh < S.heads) p.part_ml[((size_t)row * S.heads + h0 + sh) * p.nsplit + split] = make_float2(m, l);
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) {  // tile k & 1, row half k >> 1
            const int h = h0 + g + 8 * (k >> 1), c = (warp + LA_WARPS * i) * 16 + 8 * (k & 1) + 2 * t4;
            if (h < S.heads && c < S.rp)
                *reinterpret_cast<float2*>(p.part_acc + (((size_t)row * S.heads + h) * p.nsplit + split) * S.rp + c) =
                    make_float2(acc[i][k & 1][2 * (k >> 1)], acc[i][k & 1][2 * (k >> 1) + 1]);
        }
}

// ---- scan on the CUDA cores ---------------------------------------------------------------------------------------
// Grid (nsplit * groups of 8 heads, rows).  NI: 256-value pieces a cache row is spread over (32 lanes x 8 values each).
template <typename CT, int NI>
__global__ void __launch_bounds__(LA_SCAN_THREADS) latent_scan_kernel(const __grid_constant__ LatentAttnParams p) {
    extern __shared__ __align__(128) uint8_t la_ring[];  // [stages][LA_STAGE_ROWS][row] of CT
    __shared__ __align__(8) uint64_t s_full[LA_MAX_STAGES], s_empty[LA_MAX_STAGES];
    constexpr int BATCH = NI <= 3 ? 4 : 2;
    const LatentShape& S = p.s;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = (int)blockIdx.y;
    const int split = (int)blockIdx.x % p.nsplit, h = (int)blockIdx.x / p.nsplit * LA_WARPS + warp;
    pdl_launch_dependents();
    if (tid == 0) {
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(s_full + i, 1);
            mbar_init(s_empty + i, LA_WARPS);
        }
        fence_barrier_init();
        fence_proxy_async();
    }
    __syncthreads();
    const int npos = latent_position(p, row) + 1, range = latent_range(npos, p.nsplit);
    const int t0 = min(npos, split * range), t1 = min(npos, t0 + range);
    const int nstage = (t1 - t0 + LA_STAGE_ROWS - 1) / LA_STAGE_ROWS;
    const int stage_bytes = LA_STAGE_ROWS * S.row * (int)sizeof(CT);

    if (warp == LA_WARPS) {
        if (lane == 0) {
            const CT* const cache = static_cast<const CT*>(p.cache) + (size_t)row * p.cache_stride;
            bool waited = false;
            for (int j = 0; j < nstage; ++j) {
                const int s = j % p.stages, use = j / p.stages, t = t0 + j * LA_STAGE_ROWS, te = min(t1, t + LA_STAGE_ROWS);
                if (!waited && (!p.fused || te == npos)) {  // rows of earlier tokens need not be waited for
                    pdl_wait();
                    waited = true;
                }
                if (use > 0 && !mbar_wait_bounded(s_empty + s, (uint32_t)((use - 1) & 1))) {
                    atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
                    for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
                    break;
                }
                const uint32_t bytes = (uint32_t)((te - t) * S.row * (int)sizeof(CT));
                mbar_arrive_expect_tx(s_full + s, bytes);
                bulk_g2s_plain(la_ring + (size_t)s * stage_bytes, cache + (size_t)t * S.row, bytes, s_full + s);
            }
        }
        return;
    }
    pdl_wait();
    const bool active = h < S.heads;
    f32x2 q[NI][4], acc[NI][4];
    const float* const qh = p.qp + ((size_t)row * S.heads + (active ? h : 0)) * S.row;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int e = (i * 32 + lane) * 8;
        ulonglong2 a = make_ulonglong2(0ull, 0ull), b = a;
        if (e < S.row) {
            a = __ldcg(reinterpret_cast<const ulonglong2*>(qh + e));
            b = __ldcg(reinterpret_cast<const ulonglong2*>(qh + e) + 1);
        }
        q[i][0] = a.x; q[i][1] = a.y; q[i][2] = b.x; q[i][3] = b.y;
#pragma unroll
        for (int k = 0; k < 4; ++k) acc[i][k] = 0ull;
    }
    float m = -INFINITY, l = 0.f;
    bool dead = false;
#pragma unroll 1
    for (int j = 0; j < nstage; ++j) {
        const int s = j % p.stages;
        if (!dead && !mbar_wait_bounded(s_full + s, (uint32_t)((j / p.stages) & 1))) dead = true;
        __syncwarp();
        const CT* src = reinterpret_cast<const CT*>(la_ring + (size_t)s * stage_bytes);
        const int n = __any_sync(0xffffffffu, dead) || !active ? 0 : min(LA_STAGE_ROWS, t1 - t0 - j * LA_STAGE_ROWS);
#pragma unroll 1
        for (int u0 = 0; u0 < n; u0 += BATCH, src += BATCH * S.row) {
            Pairs8 kv[BATCH][NI];
            float sc[BATCH];
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                f32x2 d = 0ull;
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const int e = (i * 32 + lane) * 8;
                    Raw8<CT> r;
                    r.zero();
                    if (u0 + u < n && e < S.row) r.read(src + u * S.row + e);
                    kv[u][i] = r.pairs();
#pragma unroll
                    for (int k = 0; k < 4; ++k) d = fma2(q[i][k], kv[u][i].p[k], d);
                }
                sc[u] = sum2(d);
            }
            warp_sums<BATCH>(sc);
            float mx = m;
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                if (u0 + u >= n) sc[u] = -INFINITY;
                mx = fmaxf(mx, sc[u]);
            }
            const float corr = exp2f(m - mx);  // 0 for the first batch (its first position is always in range)
            m = mx;
            l *= corr;
            const f32x2 c2 = pack2(corr, corr);
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int k = 0; k < 4; ++k) acc[i][k] = mul2(acc[i][k], c2);
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                const float w = exp2f(sc[u] - mx);
                const f32x2 w2 = pack2(w, w);
                l += w;
#pragma unroll
                for (int i = 0; i < NI; ++i)
#pragma unroll
                    for (int k = 0; k < 4; ++k) acc[i][k] = fma2(w2, kv[u][i].p[k], acc[i][k]);
            }
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(s_empty + s);
    }
    if (dead && lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
    if (!active || t0 >= t1) return;  // (a range without positions is not read by the merge)
    const size_t slot = ((size_t)row * S.heads + h) * p.nsplit + split;
    if (lane == 0) p.part_ml[slot] = make_float2(m, l);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int e = (i * 32 + lane) * 8;
        if (e < S.rp) {
            ulonglong2* dst = reinterpret_cast<ulonglong2*>(p.part_acc + slot * S.rp + e);
            dst[0] = make_ulonglong2(acc[i][0], acc[i][1]);
            dst[1] = make_ulonglong2(acc[i][2], acc[i][3]);
        }
    }
}

// Grid (heads * vsplit, rows), clusters of the vsplit blocks of a head: each merges the ranges for its part of the latent and hands
// that part to the others through distributed shared memory, then applies its rows of W_uv (four at a time per warp) and the gate.
template <typename OT>
__global__ void __launch_bounds__(LA_CONSUMERS) latent_output_kernel(const __grid_constant__ LatentAttnParams p) {
    __shared__ float s_w[LA_MAX_SPLIT];
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
    const int npos = latent_position(p, row) + 1, range = latent_range(npos, p.nsplit), ns = (npos + range - 1) / range;
    pdl_wait();
    const size_t slot = ((size_t)row * S.heads + h) * p.nsplit;
    if (warp == 0) {  // weights of the ranges; ns <= 64
        const float sink2 = __ldg(p.sink + h) * 1.4426950408889634f;
        const float2 a = lane < ns ? __ldcg(p.part_ml + slot + lane) : make_float2(-INFINITY, 0.f);
        const float2 b = lane + 32 < ns ? __ldcg(p.part_ml + slot + 32 + lane) : make_float2(-INFINITY, 0.f);
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
            const float* const src = p.part_acc + slot * S.rp + c0 + 2 * cp;
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
