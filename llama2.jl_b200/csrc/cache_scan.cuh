// Attention of a few query vectors over cached rows: one pass that scores the rows and sums their leading columns.  A position is one
// row of `row` values; a query vector has `row` values too (zeros where a part of the row is not a key of its own), its score against
// a position is their product, and what is summed with the softmax weights are the row's first `vcols` values.  Latent attention
// [latent | rotated key] and grouped attention with several maps per head [value | key of map 1 | key of map 2] are both of this kind.
// Consecutive query vectors ("heads") share a cache in groups of per_group.  Positions may be seen by chunks: only those of the
// query's own chunk.
//   cache_scan_mma_kernel (bf16 cache)  a block takes 16 heads of a group and a range of positions, whose rows a producer warp brings
//                         into shared memory with bulk asynchronous copies; scores and weighted sums on the tensor cores with the
//                         query vectors and the weights as two bf16 terms (high and low part: 16 significant bits), running softmax
//                         in the exp2 domain in f32; one partial result (maximum, sum, unnormalised vector) per head and range;
//   cache_scan_kernel     (f32 cache)  the same on the CUDA cores, 8 heads per block, one per warp.
// The mechanism's own kernels make the query vectors before and merge the ranges afterwards.  Rows that earlier tokens wrote are
// fetched before the wait on the previous kernel.
#pragma once
#include "dense_ops.cuh"

namespace l2b {

constexpr int CS_WARPS = 8, CS_CONSUMERS = CS_WARPS * 32, CS_SCAN_THREADS = CS_CONSUMERS + 32;
constexpr int CS_STAGE_ROWS = 16, CS_MAX_STAGES = 4, CS_MAX_SPLIT = 64, CS_MIN_RANGE = 32, CS_MAX_ROW = 1024;

struct CacheScan {
    int heads, per_group;   // query vectors of a position; of them per_group at a time share a cache
    int row, vcols;         // values of a row (a multiple of 8); leading ones that are summed (a multiple of 8)
    int chunk;              // positions of earlier chunks of this size are not seen (0: no chunks)
    size_t group_stride;    // elements between the caches of consecutive groups
    void* cache;            // [groups][positions][row]
    size_t cache_stride;    // elements between the caches of consecutive rows (batched decode), else 0
    const int* pos;         // decode: device scalar
    const int* pos_list;    // batched decode: position of every row
    int pos0;               // otherwise row r sits at pos0 + r
    float* qp;              // [rows][heads][row]: query vectors, times scale * log2(e)
    float2* part_ml;        // [rows][heads][nsplit]
    float* part_acc;        // [rows][heads][nsplit][vcols]
    int nsplit;             // ranges of positions
    int stages;             // ring slots
    int fused;              // decode step: only the newest position's row comes from the kernel before
    int* status;
};
__device__ __forceinline__ int scan_position(const CacheScan& p, int row) {
    return p.pos ? __ldcg(p.pos) : p.pos_list ? __ldcg(p.pos_list + row) : p.pos0 + row;
}
__device__ __forceinline__ int scan_first(const CacheScan& p, int pos) { return p.chunk ? pos / p.chunk * p.chunk : 0; }
// positions per range of `npos` visible ones
__device__ __forceinline__ int scan_range(int npos, int nsplit) { return max(CS_MIN_RANGE, (npos + nsplit - 1) / nsplit); }

// ---- scan on the tensor cores -----------------------------------------------------------------------------------
constexpr int CS_MMA_HEADS = 16;  // heads per block = M of mma.m16n8k16

// Bytes between cache rows in shared memory: 16 mod 128, so that eight rows of a fragment load fall in different banks; at least
// 16 bytes of zeros follow the row (the last K = 16 step may reach 8 values beyond it).
__host__ __device__ inline int cs_pitch(int row) { return (row * 2 + 127) / 128 * 128 + 16; }
__host__ __device__ inline int cs_mma_stage_bytes(int row) { return CS_STAGE_ROWS * cs_pitch(row); }

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// Grid (nsplit, blocks of 16 heads, rows).  N: K = 16 steps of a cache row, and pairs of 8-column tiles of the summed columns, per warp at most.
template <int N>
__global__ void __launch_bounds__(CS_SCAN_THREADS) cache_scan_mma_kernel(const __grid_constant__ CacheScan p) {
    extern __shared__ __align__(128) uint8_t cs_ring[];  // [stages][CS_STAGE_ROWS][pitch]
    __shared__ __align__(8) uint64_t s_full[CS_MAX_STAGES], s_empty[CS_MAX_STAGES];
    __shared__ float s_s[CS_WARPS][CS_MMA_HEADS][CS_STAGE_ROWS + 1];             // the warps' shares of the scores
    __shared__ __align__(16) uint32_t s_hi[CS_MMA_HEADS][12], s_lo[CS_MMA_HEADS][12];  // weights of a stage: 16 bf16 per head (rows padded)
    __shared__ float s_corr[CS_MMA_HEADS];
    constexpr int KS = N, NT = N;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = (int)blockIdx.z;
    const int split = (int)blockIdx.x, per = (p.per_group + CS_MMA_HEADS - 1) / CS_MMA_HEADS, group = per == 1 ? (int)blockIdx.y : (int)blockIdx.y / per;
    const int h0 = group * p.per_group + ((int)blockIdx.y - group * per) * CS_MMA_HEADS, h1 = (group + 1) * p.per_group;  // heads h0 .. of this group
    const int pitch = cs_pitch(p.row), stage_bytes = cs_mma_stage_bytes(p.row);
    pdl_launch_dependents();
    if (tid == 0) {
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(s_full + i, 1);
            mbar_init(s_empty + i, CS_WARPS);
        }
        fence_barrier_init();
        fence_proxy_async();
    }
    for (int i = tid; i < p.stages * CS_STAGE_ROWS; i += CS_SCAN_THREADS)  // zeros behind every row
        for (int k = p.row * 2; k < pitch; k += 16) *reinterpret_cast<uint4*>(cs_ring + (size_t)i * pitch + k) = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
    const int pos = scan_position(p, row), npos = pos + 1, first = scan_first(p, pos), range = scan_range(npos - first, p.nsplit);
    const int t0 = min(npos, first + split * range), t1 = min(npos, t0 + range);
    const int nstage = (t1 - t0 + CS_STAGE_ROWS - 1) / CS_STAGE_ROWS;

    if (warp == CS_WARPS) {
        const bf16* const cache = static_cast<const bf16*>(p.cache) + (size_t)row * p.cache_stride + (size_t)group * p.group_stride;
        bool waited = false;
        for (int j = 0; j < nstage; ++j) {
            const int s = j % p.stages, use = j / p.stages, t = t0 + j * CS_STAGE_ROWS, te = min(t1, t + CS_STAGE_ROWS);
            if (!waited && (!p.fused || te == npos)) {  // rows of earlier tokens need not be waited for
                pdl_wait();
                waited = true;
            }
            if (!__all_sync(0xffffffffu, use == 0 || mbar_wait_bounded(s_empty + s, (uint32_t)((use - 1) & 1)))) {
                if (lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
                for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
                break;
            }
            if (lane == 0) mbar_arrive_expect_tx(s_full + s, (uint32_t)((te - t) * p.row * 2));
            __syncwarp();
            if (lane < te - t) bulk_g2s_plain(cs_ring + (size_t)s * stage_bytes + lane * pitch, cache + (size_t)(t + lane) * p.row, (uint32_t)(p.row * 2), s_full + s);
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
            const int h = h0 + g + 8 * (k & 1), e = (warp + CS_WARPS * i) * 16 + 8 * (k >> 1) + 2 * t4;
            float2 v = make_float2(0.f, 0.f);
            if (h < h1 && e < p.row) v = __ldcg(reinterpret_cast<const float2*>(p.qp + ((size_t)row * p.heads + h) * p.row + e));
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
        const int s = j % p.stages, n = min(CS_STAGE_ROWS, t1 - t0 - j * CS_STAGE_ROWS);
        if (!dead && !__all_sync(0xffffffffu, mbar_wait_bounded(s_full + s, (uint32_t)((j / p.stages) & 1)))) dead = true;
        __syncwarp();
        const uint8_t* const st = cs_ring + (size_t)s * stage_bytes;
        {
            float d[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
            for (int i = 0; i < KS; ++i) {
                const int k0 = (warp + CS_WARPS * i) * 16;
                if (k0 < p.row)
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
        for (int i = n * (pitch / 16) + tid; i < CS_STAGE_ROWS * (pitch / 16); i += CS_CONSUMERS)
            *reinterpret_cast<uint4*>(cs_ring + (size_t)s * stage_bytes + (size_t)i * 16) = make_uint4(0u, 0u, 0u, 0u);
        partial_sync(CS_CONSUMERS);
        {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < CS_WARPS; ++w) v += s_s[w][sh][sp];
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
        partial_sync(CS_CONSUMERS);
        {
            const float ca = s_corr[g], cb = s_corr[g + 8];
            const uint32_t ahi[4] = {s_hi[g][t4], s_hi[g + 8][t4], s_hi[g][t4 + 4], s_hi[g + 8][t4 + 4]};
            const uint32_t alo[4] = {s_lo[g][t4], s_lo[g + 8][t4], s_lo[g][t4 + 4], s_lo[g + 8][t4 + 4]};
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int c0 = (warp + CS_WARPS * i) * 16;  // columns c0 .. c0+15: two tiles
                if (c0 >= p.vcols) continue;                   // (uniform over the warp)
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
    if (sp == 0 && h0 + sh < h1) p.part_ml[((size_t)row * p.heads + h0 + sh) * p.nsplit + split] = make_float2(m, l);
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) {  // tile k & 1, row half k >> 1
            const int h = h0 + g + 8 * (k >> 1), c = (warp + CS_WARPS * i) * 16 + 8 * (k & 1) + 2 * t4;
            if (h < h1 && c < p.vcols)
                *reinterpret_cast<float2*>(p.part_acc + (((size_t)row * p.heads + h) * p.nsplit + split) * p.vcols + c) =
                    make_float2(acc[i][k & 1][2 * (k >> 1)], acc[i][k & 1][2 * (k >> 1) + 1]);
        }
}

// ---- scan on the CUDA cores ---------------------------------------------------------------------------------------
// Grid (nsplit, blocks of 8 heads, rows).  NI: 256-value pieces a cache row is spread over (32 lanes x 8 values each).
template <typename CT, int NI>
__global__ void __launch_bounds__(CS_SCAN_THREADS) cache_scan_kernel(const __grid_constant__ CacheScan p) {
    extern __shared__ __align__(128) uint8_t cs_ring[];  // [stages][CS_STAGE_ROWS][row] of CT
    __shared__ __align__(8) uint64_t s_full[CS_MAX_STAGES], s_empty[CS_MAX_STAGES];
    constexpr int BATCH = NI <= 3 ? 4 : 2;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = (int)blockIdx.z;
    const int split = (int)blockIdx.x, per = (p.per_group + CS_WARPS - 1) / CS_WARPS, group = per == 1 ? (int)blockIdx.y : (int)blockIdx.y / per;
    const int hg = ((int)blockIdx.y - group * per) * CS_WARPS + warp, h = group * p.per_group + hg;
    pdl_launch_dependents();
    if (tid == 0) {
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(s_full + i, 1);
            mbar_init(s_empty + i, CS_WARPS);
        }
        fence_barrier_init();
        fence_proxy_async();
    }
    __syncthreads();
    const int pos = scan_position(p, row), npos = pos + 1, first = scan_first(p, pos), range = scan_range(npos - first, p.nsplit);
    const int t0 = min(npos, first + split * range), t1 = min(npos, t0 + range);
    const int nstage = (t1 - t0 + CS_STAGE_ROWS - 1) / CS_STAGE_ROWS;
    const int stage_bytes = CS_STAGE_ROWS * p.row * (int)sizeof(CT);

    if (warp == CS_WARPS) {
        if (lane == 0) {
            const CT* const cache = static_cast<const CT*>(p.cache) + (size_t)row * p.cache_stride + (size_t)group * p.group_stride;
            bool waited = false;
            for (int j = 0; j < nstage; ++j) {
                const int s = j % p.stages, use = j / p.stages, t = t0 + j * CS_STAGE_ROWS, te = min(t1, t + CS_STAGE_ROWS);
                if (!waited && (!p.fused || te == npos)) {  // rows of earlier tokens need not be waited for
                    pdl_wait();
                    waited = true;
                }
                if (use > 0 && !mbar_wait_bounded(s_empty + s, (uint32_t)((use - 1) & 1))) {
                    atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
                    for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
                    break;
                }
                const uint32_t bytes = (uint32_t)((te - t) * p.row * (int)sizeof(CT));
                mbar_arrive_expect_tx(s_full + s, bytes);
                bulk_g2s_plain(cs_ring + (size_t)s * stage_bytes, cache + (size_t)t * p.row, bytes, s_full + s);
            }
        }
        return;
    }
    pdl_wait();
    const bool active = hg < p.per_group;
    f32x2 q[NI][4], acc[NI][4];
    const float* const qh = p.qp + ((size_t)row * p.heads + (active ? h : 0)) * p.row;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int e = (i * 32 + lane) * 8;
        ulonglong2 a = make_ulonglong2(0ull, 0ull), b = a;
        if (e < p.row) {
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
        const CT* src = reinterpret_cast<const CT*>(cs_ring + (size_t)s * stage_bytes);
        const int n = __any_sync(0xffffffffu, dead) || !active ? 0 : min(CS_STAGE_ROWS, t1 - t0 - j * CS_STAGE_ROWS);
#pragma unroll 1
        for (int u0 = 0; u0 < n; u0 += BATCH, src += BATCH * p.row) {
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
                    if (u0 + u < n && e < p.row) r.read(src + u * p.row + e);
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
    const size_t slot = ((size_t)row * p.heads + h) * p.nsplit + split;
    if (lane == 0) p.part_ml[slot] = make_float2(m, l);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int e = (i * 32 + lane) * 8;
        if (e < p.vcols) {
            ulonglong2* dst = reinterpret_cast<ulonglong2*>(p.part_acc + slot * p.vcols + e);
            dst[0] = make_ulonglong2(acc[i][0], acc[i][1]);
            dst[1] = make_ulonglong2(acc[i][2], acc[i][3]);
        }
    }
}

}  // namespace l2b
