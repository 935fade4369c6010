// Differential attention of a long portion of a prompt, on the 5th-generation tensor cores, over 128-query x 128-key tiles of the
// cached keys and values (head_attention.cuh).  Grid (128-query tiles * heads); the two maps one after the other:
//   warp 0     producer: TMA tiled copies of Q (per map), of K and V per key tile, straight from the cache rows
//   warp 1     MMA issue: S_t = Q K_t^T into tensor memory, one tile ahead of O += P_t V_t; V is an operand whose rows run along K, as the
//              cache has it
//   warps 2-9  two threads per query, each with half of the tile's keys: scores from tensor memory, scale, causal and chunk mask,
//              running maximum (shared between the two) and sum in f32 (exp2 domain); P_t as bf16 into shared memory in operand
//              layout.  O is rescaled in tensor memory only when a row's maximum has grown by more than 2^8 since it was last taken.
//              The first map's result is put aside (f32); at the end the maps are subtracted, brought to unit rms and gated.
// Up to 128 value dimensions a block takes 256 columns of tensor memory (one buffer of scores), so that two blocks share an SM when
// their shared memory allows, one's softmax beside the other's products; beyond that 512 columns and two buffers.
// Key tiles start at the first chunk that a query of the block sees.  Every mbarrier wait is bounded, as in the GEMM.
#pragma once
#include "head_attention.cuh"
#include "tcgen05.cuh"

namespace l2b {

constexpr int HP_TILE = 128, HP_WARPS = 8, HP_THREADS = 64 + HP_WARPS * 32, HP_SUB = 128 * 128;  // bytes of a 128-row x 64-value operand tile
constexpr int HP_HALF_COLS = 128;  // value dimensions up to which half of the tensor memory is enough

struct HeadPrefillParams {
    HeadShape s;
    int n, pos0;      // queries at positions pos0 .. pos0 + n - 1
    int chunk;        // as in CacheScan
    int dq;           // stored dims per query and map: dim rounded up to 16
    int vn;           // vdim rounded up to 16
    int kstages;
    int paired;       // number of SMs when all blocks run at once, two per SM; else 0
    float* aside;     // [heads][128-query tiles][vdim][128]: the first map's result
    bf16* out;        // [n][ldo]
    int ldo;
    int* status;
};
struct HpSmem {
    int q, k, v, p, total, kbytes, vbytes;
};
__host__ __device__ inline HpSmem hp_smem_layout(int dim, int vn, int kstages) {
    HpSmem s;
    s.kbytes = (dim + 63) / 64 * HP_SUB;
    s.vbytes = (vn + 63) / 64 * HP_SUB;
    s.q = 0;
    s.k = s.q + s.kbytes;
    s.v = s.k + kstages * s.kbytes;
    s.p = s.v + s.vbytes;
    s.total = s.p + 2 * HP_SUB;
    return s;
}

__global__ void __launch_bounds__(HP_THREADS, 2) head_prefill_kernel(const __grid_constant__ HeadPrefillParams p, const __grid_constant__ CUtensorMap map_q,
                                                                  const __grid_constant__ CUtensorMap map_kv, const __grid_constant__ CUtensorMap map_g) {
    extern __shared__ __align__(1024) uint8_t hp_raw[];
    __shared__ __align__(8) uint64_t s_q, s_qfree, s_gate, s_k[2], s_kfree[2], s_v, s_s[2], s_sfree[2], s_p, s_o;
    __shared__ uint32_t s_tmem;
    __shared__ float s_row[2][2][HP_TILE];  // [tile parity][half][query]: the halves' maxima (at the ends: sums)
    __shared__ float s_ss[2][HP_TILE];
    uint8_t* smem = hp_raw + ((1024u - (smem_u32(hp_raw) & 1023u)) & 1023u);
    const HpSmem L = hp_smem_layout(p.s.dim, p.vn, p.kstages);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // longest first; when all blocks run at once, two per SM, the second of an SM is as short as the first is long
    const int blocks = (int)gridDim.x, rank = p.paired && (int)blockIdx.x >= p.paired ? blocks - 1 - ((int)blockIdx.x - p.paired) : (int)blockIdx.x;
    const int h = rank % p.s.heads, g = h / (p.s.heads / p.s.kv_heads), q0 = (blocks / p.s.heads - 1 - rank / p.s.heads) * HP_TILE;
    const int first = p.chunk ? (p.pos0 + q0) / p.chunk * p.chunk : 0;           // first key of the first tile
    const int last = p.pos0 + min(p.n, q0 + HP_TILE) - 1;                        // position of the last query
    const int nt = (last - first) / HP_TILE + 1, nt2 = 2 * nt;                   // key tiles per map, of both maps
    const int late = p.chunk ? last / p.chunk * p.chunk : 0;                     // where the last query's chunk begins
    const int nd = (p.s.dim + 63) / 64, nv = (p.vn + 63) / 64;
    const int nsb = p.vn <= HP_HALF_COLS ? 1 : 2;                                // buffers of scores
    if (threadIdx.x == 0) {
        mbar_init(&s_q, 1);
        mbar_init(&s_qfree, 1);
        mbar_init(&s_gate, 1);
        mbar_init(&s_v, 1);
        mbar_init(&s_p, HP_WARPS);
        mbar_init(&s_o, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(s_k + i, 1);
            mbar_init(s_kfree + i, 1);
            mbar_init(s_s + i, 1);
            mbar_init(s_sfree + i, HP_WARPS);
        }
        fence_barrier_init();
        fence_proxy_async();
    }
    if (warp == 1) tmem_alloc(&s_tmem, nsb * 256);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem, tmem_o = tmem + (uint32_t)(nsb * 128);

    if (warp == 0) {
        if (lane == 0) {
            bool ok = true;
            for (int t = 0; t < nt2 && ok; ++t) {
                const int map = t >= nt, pos = first + (t - map * nt) * HP_TILE;
                if (t == map * nt) {
                    if (map && !mbar_wait_bounded(&s_qfree, 0u)) {
                        ok = false;
                        break;
                    }
                    mbar_arrive_expect_tx(&s_q, (uint32_t)L.kbytes);
                    for (int i = 0; i < nd; ++i) tma_load_2d(smem + L.q + i * HP_SUB, &map_q, (2 * h + map) * p.dq + 64 * i, q0, &s_q);
                }
                const int s = p.kstages == 2 ? (t & 1) : 0, use = p.kstages == 2 ? t >> 1 : t;
                if (use > 0 && !mbar_wait_bounded(s_kfree + s, (uint32_t)((use - 1) & 1))) {
                    ok = false;
                    break;
                }
                mbar_arrive_expect_tx(s_k + s, (uint32_t)L.kbytes);
                for (int i = 0; i < nd; ++i) tma_load_3d(smem + L.k + s * L.kbytes + i * HP_SUB, &map_kv, p.s.vp + map * p.s.dp + 64 * i, pos, g, s_k + s);
                if (t > 0 && !mbar_wait_bounded(&s_o, (uint32_t)((t - 1) & 1))) {  // P V of the tile before has read V
                    ok = false;
                    break;
                }
                mbar_arrive_expect_tx(&s_v, (uint32_t)L.vbytes);
                for (int i = 0; i < nv; ++i) tma_load_3d(smem + L.v + i * HP_SUB, &map_kv, 64 * i, pos, g, &s_v);
            }
            if (ok && mbar_wait_bounded(&s_o, (uint32_t)((nt2 - 1) & 1))) {  // all products are done: the gates take the operands' place
                mbar_arrive_expect_tx(&s_gate, (uint32_t)L.vbytes);
                for (int i = 0; i < nv; ++i) tma_load_2d(smem + L.q + i * HP_SUB, &map_g, h * p.s.vp + 64 * i, q0, &s_gate);
            } else {
                ok = false;
            }
            if (!ok) {
                atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
                for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_s = umma_idesc_bf16(128, 128), idesc_o = umma_idesc_bf16(128, p.vn, 0, 1);
            bool ok = true;
            auto pv = [&](int t) {
                if (!mbar_wait_bounded(&s_v, (uint32_t)(t & 1)) || !mbar_wait_bounded(&s_p, (uint32_t)(t & 1))) {
                    ok = false;
                    return;
                }
                tc_fence_after();
                const int map = t >= nt;
                for (int kk = 0; kk < 8; ++kk)
                    umma_bf16(tmem_o, umma_desc_sw128(smem + L.p + (kk >> 2) * HP_SUB, (kk & 3) * 32), umma_desc_sw128_mn(smem + L.v, kk * 2048, HP_SUB), idesc_o,
                              (t - map * nt) | kk ? 1u : 0u);
                umma_commit(&s_o);
            };
            for (int t = 0; t < nt2 && ok; ++t) {
                const int map = t >= nt, s = p.kstages == 2 ? (t & 1) : 0, use = p.kstages == 2 ? t >> 1 : t, b = t & (nsb - 1), sb = t / nsb;
                if ((t == map * nt && !mbar_wait_bounded(&s_q, (uint32_t)map)) || !mbar_wait_bounded(s_k + s, (uint32_t)(use & 1)) ||
                    (sb > 0 && !mbar_wait_bounded(s_sfree + b, (uint32_t)((sb - 1) & 1)))) {
                    ok = false;
                    break;
                }
                tc_fence_after();
                for (int kk = 0; 16 * kk < p.s.dim; ++kk)
                    umma_bf16(tmem + (uint32_t)(b * 128), umma_desc_sw128(smem + L.q + (kk >> 2) * HP_SUB, (kk & 3) * 32),
                              umma_desc_sw128(smem + L.k + s * L.kbytes + (kk >> 2) * HP_SUB, (kk & 3) * 32), idesc_s, kk ? 1u : 0u);
                umma_commit(s_s + b);
                umma_commit(s_kfree + s);
                if (t == nt - 1) umma_commit(&s_qfree);
                if (t > 0) pv(t - 1);
            }
            if (ok) pv(nt2 - 1);
            if (!ok) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
        }
    } else {
        const int qd = warp & 3, half = (warp - 2) >> 2, r = 32 * qd + lane;
        const uint32_t lane_off = (uint32_t)(32 * qd) << 16;
        const int qi = q0 + r, qpos = p.pos0 + qi, qfirst = p.chunk ? qpos / p.chunk * p.chunk : 0;
        float* const aside = p.aside + ((size_t)h * (blocks / p.s.heads) + q0 / HP_TILE) * p.s.vdim * HP_TILE + r;
        float m = 0.f, l = 0.f;
        bool ok = true;
        for (int t = 0; t < nt2; ++t) {
            const int b = t & (nsb - 1), tp = t & 1, map = t >= nt, j = t - map * nt;
            if (ok && !__all_sync(0xffffffffu, mbar_wait_bounded(s_s + b, (uint32_t)((t / nsb) & 1)))) ok = false;
            tc_fence_after();
            const uint32_t ts = tmem + lane_off + (uint32_t)(b * 128 + half * 64);
            const int tile = first + j * HP_TILE, k0 = tile + half * 64, lo = qfirst - k0, hi = qpos - k0;  // keys lo .. hi of this half are seen
            const bool masked = tile + HP_TILE - 1 > p.pos0 + q0 || tile < late;
            float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll 1
            for (int c = 0; c < 64; c += 32) {
                float s[32];
                tmem_ld32f(ts + (uint32_t)c, s);
                if (masked) {
#pragma unroll
                    for (int k = 0; k < 32; ++k)
                        if (c + k > hi || c + k < lo) s[k] = -INFINITY;
                }
#pragma unroll
                for (int k = 0; k < 32; ++k) m4[k & 3] = fmaxf(m4[k & 3], s[k]);
            }
            s_row[tp][half][r] = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
            partial_sync_2(HP_WARPS * 32);
            const float mx = fmaxf(s_row[tp][0][r], s_row[tp][1][r]) * p.s.scale2;  // (scale2 > 0)
            if (ok && t > 0 && !__all_sync(0xffffffffu, mbar_wait_bounded(&s_o, (uint32_t)((t - 1) & 1)))) ok = false;  // P and O are free
            tc_fence_after();
            if (map && j == 0) {  // put the first map's result aside
                s_ss[half][r] = l;
                partial_sync_2(HP_WARPS * 32);
                const float inv = 1.f / (s_ss[0][r] + s_ss[1][r]);
                l = 0.f;
#pragma unroll 1
                for (int c = 32 * half; c < p.s.vdim; c += 64) {
                    float o[32];
                    tmem_ld32f(tmem_o + lane_off + (uint32_t)c, o);
#pragma unroll
                    for (int k = 0; k < 32; ++k)
                        if (c + k < p.s.vdim) aside[(c + k) * HP_TILE] = o[k] * inv;
                }
            }
            if (j == 0) {
                m = fmaxf(mx, -1e30f);  // (a tile may hold no key of this query's chunk)
            } else if (__any_sync(0xffffffffu, mx > m + 8.f)) {  // (the same decision in both halves)
                const float mn = mx > m + 8.f ? mx : m, corr = fast_exp2(m - mn);
                l *= corr;
                m = mn;
#pragma unroll 1
                for (int c = 32 * half; c < p.vn; c += 64) {
                    float o[32];
                    tmem_ld32f(tmem_o + lane_off + (uint32_t)c, o);
#pragma unroll
                    for (int k = 0; k < 32; ++k) o[k] *= corr;
                    tmem_st32f(tmem_o + lane_off + (uint32_t)c, o);
                }
            }
            float l4[4] = {0.f, 0.f, 0.f, 0.f};
            uint8_t* const pr = smem + L.p + half * HP_SUB;
#pragma unroll 1
            for (int c = 0; c < 64; c += 32) {
                float s[32];
                tmem_ld32f(ts + (uint32_t)c, s);
#pragma unroll
                for (int k = 0; k < 32; ++k) s[k] = fast_exp2(fmaf(s[k], p.s.scale2, -m));
                if (masked) {
#pragma unroll
                    for (int k = 0; k < 32; ++k)
                        if (c + k > hi || c + k < lo) s[k] = 0.f;
                }
#pragma unroll
                for (int k = 0; k < 32; ++k) l4[k & 3] += s[k];
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    *reinterpret_cast<uint4*>(pr + sw128_chunk(r, (c >> 3) + i)) = make_uint4(pack_bf16(s[8 * i], s[8 * i + 1]), pack_bf16(s[8 * i + 2], s[8 * i + 3]),
                                                                                              pack_bf16(s[8 * i + 4], s[8 * i + 5]), pack_bf16(s[8 * i + 6], s[8 * i + 7]));
            }
            l += (l4[0] + l4[1]) + (l4[2] + l4[3]);
            fence_proxy_async();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) {
                mbar_arrive(s_sfree + b);
                mbar_arrive(&s_p);
            }
        }
        if (ok && !__all_sync(0xffffffffu, mbar_wait_bounded(&s_o, (uint32_t)((nt2 - 1) & 1)))) ok = false;
        s_row[nt2 & 1][half][r] = l;
        partial_sync_2(HP_WARPS * 32);
        tc_fence_after();
        const float w2 = -p.s.lambda / (s_row[nt2 & 1][0][r] + s_row[nt2 & 1][1][r]);
        auto difference = [&](int c, float (&o)[32]) {  // (rows beyond n: any numbers, not stored)
            tmem_ld32f(tmem_o + lane_off + (uint32_t)c, o);
#pragma unroll
            for (int k = 0; k < 32; ++k)
                if (c + k < p.s.vdim) o[k] = fmaf(w2, o[k], aside[(c + k) * HP_TILE]);
        };
        float ss = 0.f;
#pragma unroll 1
        for (int c = 32 * half; c < p.s.vdim; c += 64) {
            float o[32];
            difference(c, o);
#pragma unroll
            for (int k = 0; k < 32; ++k) ss = c + k < p.s.vdim ? fmaf(o[k], o[k], ss) : ss;
        }
        s_ss[half][r] = ss;
        partial_sync_2(HP_WARPS * 32);
        if (ok && !__all_sync(0xffffffffu, mbar_wait_bounded(&s_gate, 0u))) ok = false;
        if (!ok) {
            if (lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
        } else {
            const float scale = p.s.out_scale / sqrtf((s_ss[0][r] + s_ss[1][r]) / (float)p.s.vdim + p.s.eps);
            bf16* out = p.out + (size_t)qi * p.ldo + (size_t)h * p.s.vdim;
            const bool wide = ((p.s.vdim | p.ldo) & 7) == 0;
#pragma unroll 1
            for (int c = 32 * half; c < p.s.vdim; c += 64) {
                float o[32];
                difference(c, o);
                const int n = qi < p.n ? p.s.vdim - c : 0;  // values of this query to store
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const uint4 g8 = *reinterpret_cast<const uint4*>(smem + L.q + (c >> 6) * HP_SUB + sw128_chunk(r, 4 * half + i));
                    const uint4 v = make_uint4(mul_pack_bf16(g8.x, o[8 * i] * scale, o[8 * i + 1] * scale), mul_pack_bf16(g8.y, o[8 * i + 2] * scale, o[8 * i + 3] * scale),
                                               mul_pack_bf16(g8.z, o[8 * i + 4] * scale, o[8 * i + 5] * scale), mul_pack_bf16(g8.w, o[8 * i + 6] * scale, o[8 * i + 7] * scale));
                    if (wide) {
                        if (8 * i < n) *reinterpret_cast<uint4*>(out + c + 8 * i) = v;
                    } else {
                        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                        for (int k = 0; k < 8; ++k)
                            if (8 * i + k < n) out[c + 8 * i + k] = __ushort_as_bfloat16((unsigned short)(w[k >> 1] >> (16 * (k & 1))));
                    }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, nsb * 256);
}

}  // namespace l2b
