// mLSTM over a long portion of a prompt, in chunks of 128 tokens on the 5th-generation tensor cores.  With F the running sum of the log
// forget gates within a chunk, a_s = i_s - F_s, and M_t = max(m_0, max_{s <= t} a_s) (so that the running maximum is m_t = F_t + M_t),
//     S_t = exp(m_0 - M_t) S_0 + sum_{s <= t} exp(a_s - M_t) k_s v_s^T        (both sides scaled by exp(-m_t)),
// every exponent at most zero.  So a chunk is two products with weights in between, and the state goes from chunk to chunk by one more:
//   mlstm_operands_kernel  q (times dim^-1/2), k, v, and the output gate times the norm's weight, as bf16;
//   mlstm_gates_kernel     a, M and the factors of every token and chunk, the running maximum after the portion;
//   mlstm_state_kernel     a block has 128 x 64 values of a head's S in tensor memory, f32, and goes through the chunks: hands S out as
//                          two bf16 terms (16 significant bits) for the kernel below, decays it, adds K^T (u V), where u V is split
//                          into two terms as well and u itself is one more column, which gives n;
//   mlstm_chunk_kernel     a block has a chunk and 128 columns of a head: A = (Q K^T) weighted and masked (f32, then two bf16 terms),
//                          O = A V, R = Q S_0; the columns of a head meet in a cluster for the unit rms; weight and gate.
// Every mbarrier wait is bounded, as in the GEMM.
#pragma once
#include "mlstm.cuh"
#include "tcgen05.cuh"

namespace l2b {

constexpr int MP_L = 128, MP_MAX_CHUNKS = 32, MP_SUB = 128 * 128;  // tokens of a chunk; bytes of a 128-row x 64-value operand tile
constexpr int MP_WARPS = 8, MP_THREADS = 64 + MP_WARPS * 32;
constexpr int MP_STATE_COLS = 64, MP_COLS = 128;                   // columns of a block: state kernel, chunk kernel

struct MlstmPrefillParams {
    MlstmParams m;       // one sequence; out: bf16
    int n, nchunk;
    int dp, vp, vs;      // dim rounded up to 16; vdim rounded up to 8 (operands), and of the states' rows
    bf16 *q, *k, *v, *g;  // [n][heads * dp] twice, [n][heads * vp] twice
    float *a, *mx, *w, *floor, *u;  // [heads][nchunk * MP_L]: a_t, M_t, exp(m_0 - M_t), exp(-m_t), exp(a_t - M of the chunk's end)
    float* decay;        // [heads][nchunk]: exp(m_0 - M of the chunk's end)
    bf16 *sh, *sl;       // [nchunk][heads][dp][vs]: S before the chunk, high and low terms
    float* sn;           // [nchunk][heads][dp]: n before the chunk
    int vt, sstages;     // chunk kernel: blocks per head (1, 2, 4, 8); ring slots of S
    int* status;
};

// Grid (n): one token's operands.
__global__ void __launch_bounds__(256) mlstm_operands_kernel(const __grid_constant__ MlstmPrefillParams p) {
    const MlstmShape& S = p.m.s;
    const int t = (int)blockIdx.x;
    const float* const in = p.m.in + (size_t)t * p.m.ld;
    auto part = [&](bf16* out, int dim, int pad, auto value) {  // value(index among heads * dim)
        bf16* const dst = out + (size_t)t * S.heads * pad;
        for (int i = 2 * threadIdx.x; i < S.heads * pad; i += 512) {
            const int h = i / pad, d = i - h * pad;  // (pad is even)
            *reinterpret_cast<uint32_t*>(dst + i) = pack_bf16(d < dim ? value(h * dim + d) : 0.f, d + 1 < dim ? value(h * dim + d + 1) : 0.f);
        }
    };
    part(p.q, S.dim, p.dp, [&](int i) { return __ldcg(in + i) * S.qscale; });
    part(p.k, S.dim, p.dp, [&](int i) { return __ldcg(in + p.m.off_k + i); });
    part(p.v, S.vdim, p.vp, [&](int i) { return __ldcg(in + p.m.off_v + i); });
    part(p.g, S.vdim, p.vp, [&](int i) { return __ldg(p.m.norm + i) * fast_sigmoid(__ldcg(in + p.m.off_g + i)); });
}

// Grid (heads), a warp per chunk, a lane four consecutive tokens.
__global__ void __launch_bounds__(MP_MAX_CHUNKS * 32) mlstm_gates_kernel(const __grid_constant__ MlstmPrefillParams p) {
    __shared__ float s_f[MP_MAX_CHUNKS], s_a[MP_MAX_CHUNKS];
    const MlstmShape& S = p.m.s;
    const int h = (int)blockIdx.x, c = (int)threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* const gm = p.m.state + S.m_at() + (size_t)h * S.cl;
    float m0 = p.m.pos0 == 0 ? 0.f : gm[0];
    float f[4], a[4], A[4];
    float sum = 0.f, top = -INFINITY;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const int t = c * MP_L + lane * 4 + k;
        f[k] = 0.f;
        a[k] = -INFINITY;  // (the log input gate until F is known)
        if (t < p.n) {
            const MlstmGates g = mlstm_gates(p.m, p.m.in + (size_t)t * p.m.ld, h);
            f[k] = g.f;
            a[k] = g.i;
        }
        sum += f[k];
    }
    float before = sum;  // sum of f over the lanes up to this one
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, before, o);
        if (lane >= o) before += x;
    }
    const float total = __shfl_sync(0xffffffffu, before, 31);
    float F = __shfl_up_sync(0xffffffffu, before, 1);
    if (lane == 0) F = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        F += f[k];
        f[k] = F;
        a[k] -= F;
        top = fmaxf(top, a[k]);
        A[k] = top;
    }
    float upto = top;  // maximum of a over the lanes up to this one
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, upto, o);
        if (lane >= o) upto = fmaxf(upto, x);
    }
    const float end_a = __shfl_sync(0xffffffffu, upto, 31);
    float pre = __shfl_up_sync(0xffffffffu, upto, 1);
    if (lane == 0) pre = -INFINITY;
    if (lane == 31) {
        s_f[c] = total;
        s_a[c] = end_a;
    }
    __syncthreads();
    for (int i = 0; i < c; ++i) m0 = s_f[i] + fmaxf(m0, s_a[i]);
    if (c < p.nchunk) {
        const float end = fmaxf(m0, end_a);
        const size_t at = ((size_t)h * p.nchunk + c) * MP_L + lane * 4;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float M = fmaxf(m0, fmaxf(pre, A[k]));
            p.a[at + k] = a[k];
            p.mx[at + k] = M;
            p.w[at + k] = expf(m0 - M);
            p.floor[at + k] = expf(-f[k] - M);
            p.u[at + k] = expf(a[k] - end);
        }
        if (lane == 0) p.decay[(size_t)h * p.nchunk + c] = expf(m0 - end);
        if (c == p.nchunk - 1) {
            __syncwarp();
            for (int r = lane; r < S.cl; r += 32) gm[r] = total + end;
        }
    }
}

// Grid (blocks of 64 columns, blocks of 128 rows, heads).
struct MsSmem {  // K [2 stages][2 pieces of 64 dims], u V [2 stages] high and low [2 pieces each: 64 columns; u]
    static constexpr int k = 0, w = 4 * MP_SUB, wbytes = 4 * MP_SUB, total = 12 * MP_SUB;
};
__global__ void __launch_bounds__(MP_THREADS, 1) mlstm_state_kernel(const __grid_constant__ MlstmPrefillParams p, const __grid_constant__ CUtensorMap map_k) {
    extern __shared__ __align__(1024) uint8_t ms_raw[];
    __shared__ __align__(8) uint64_t s_k[2], s_kfree[2], s_w, s_mma;
    __shared__ uint32_t s_tmem;
    uint8_t* smem = ms_raw + ((1024u - (smem_u32(ms_raw) & 1023u)) & 1023u);
    const MlstmShape& S = p.m.s;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c0 = (int)blockIdx.x * MP_STATE_COLS, d0 = (int)blockIdx.y * 128, h = (int)blockIdx.z;
    if (threadIdx.x == 0) {
        mbar_init(&s_w, MP_WARPS);
        mbar_init(&s_mma, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(s_k + i, 1);
            mbar_init(s_kfree + i, 1);
        }
        fence_barrier_init();
        fence_proxy_async();
    }
    if (warp == 1) tmem_alloc(&s_tmem, 128);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;

    if (warp == 0) {
        if (lane == 0) {
            for (int c = 0; c < p.nchunk; ++c) {
                const int s = c & 1;
                if (c >= 2 && !mbar_wait_bounded(s_kfree + s, (uint32_t)(((c >> 1) - 1) & 1))) {
                    atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
                    for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
                    break;
                }
                mbar_arrive_expect_tx(s_k + s, 2 * MP_SUB);
                for (int i = 0; i < 2; ++i) tma_load_2d(smem + MsSmem::k + (2 * s + i) * MP_SUB, &map_k, h * p.dp + d0 + 64 * i, c * MP_L, s_k + s);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = umma_idesc_bf16(128, MP_STATE_COLS + 16, 1, 1);
            for (int c = 0; c < p.nchunk; ++c) {
                const int s = c & 1;
                if (!mbar_wait_bounded(s_k + s, (uint32_t)((c >> 1) & 1)) || !mbar_wait_bounded(&s_w, (uint32_t)(c & 1))) {
                    atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
                    break;
                }
                tc_fence_after();
                for (int term = 0; term < 2; ++term)
                    for (int kk = 0; kk < 8; ++kk)
                        umma_bf16(tmem, umma_desc_sw128_mn(smem + MsSmem::k + 2 * s * MP_SUB, kk * 2048, MP_SUB),
                                  umma_desc_sw128_mn(smem + MsSmem::w + s * MsSmem::wbytes + 2 * term * MP_SUB, kk * 2048, MP_SUB), idesc, 1u);
                umma_commit(s_kfree + s);
                umma_commit(&s_mma);
            }
        }
    } else {
        const int qd = warp & 3, half = (warp - 2) >> 2, r = 32 * qd + lane;  // this thread's row of S (lane of tensor memory), 32 columns
        const uint32_t at = tmem + ((uint32_t)(32 * qd) << 16) + (uint32_t)(32 * half), at_n = tmem + ((uint32_t)(32 * qd) << 16) + MP_STATE_COLS;
        const int d = d0 + r, cc = c0 + 32 * half;                            // first column
        const bool row_in = d < S.dim, has_n = half == 0 && blockIdx.x == 0;
        float* const gs = p.m.state + ((size_t)h * S.dim + d) * S.vdim + cc;
        float* const gn = p.m.state + S.n_at() + (size_t)h * S.cl * S.dim + d;  // + copy * dim
        const bool fresh = p.m.pos0 == 0;
        // u V: this thread's token of a chunk and its 32 columns
        const int tok = r;
        uint4 v[4];
        float u = 0.f, decay = 0.f;
        auto fetch = [&](int c) {
            const bf16* src = p.v + (size_t)(c * MP_L + tok) * S.heads * p.vp + (size_t)h * p.vp + cc;
#pragma unroll
            for (int i = 0; i < 4; ++i)
                v[i] = c < p.nchunk && c * MP_L + tok < p.n && cc + 8 * i < p.vp ? __ldg(reinterpret_cast<const uint4*>(src) + i) : make_uint4(0u, 0u, 0u, 0u);
            u = c < p.nchunk ? __ldg(p.u + ((size_t)h * p.nchunk + c) * MP_L + tok) : 0.f;
        };
        auto weigh = [&](int c) {  // u V of chunk c in two terms; rows are tokens
            uint8_t* const wh = smem + MsSmem::w + (c & 1) * MsSmem::wbytes;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const uint32_t x[4] = {v[i].x, v[i].y, v[i].z, v[i].w};
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int k = 0; k < 4; ++k) split2(u * __uint_as_float(x[k] << 16), u * __uint_as_float(x[k] & 0xFFFF0000u), hi[k], lo[k]);
                const int off = sw128_chunk(tok, 4 * half + i);
                *reinterpret_cast<uint4*>(wh + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                *reinterpret_cast<uint4*>(wh + 2 * MP_SUB + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
            // column 64: u; columns 65 .. 79: zeros
            uint32_t hi, lo;
            split2(u, 0.f, hi, lo);
            const int off = MP_SUB + sw128_chunk(tok, half);
            *reinterpret_cast<uint4*>(wh + off) = make_uint4(half ? 0u : hi, 0u, 0u, 0u);
            *reinterpret_cast<uint4*>(wh + 2 * MP_SUB + off) = make_uint4(half ? 0u : lo, 0u, 0u, 0u);
        };
        fetch(0);
        weigh(0);
        fetch(1);
        bool ok = true;
        for (int c = 0; c <= p.nchunk; ++c) {
            float st[32], n = 0.f;
            if (c < p.nchunk) decay = __ldg(p.decay + (size_t)h * p.nchunk + c);
            if (c == 0) {
#pragma unroll
                for (int k = 0; k < 32; ++k) st[k] = !fresh && row_in && cc + k < S.vdim ? gs[k] : 0.f;
                if (!fresh && row_in && half == 0) n = gn[0];
            } else {
                if (ok && !__all_sync(0xffffffffu, mbar_wait_bounded(&s_mma, (uint32_t)((c - 1) & 1)))) ok = false;
                tc_fence_after();
                tmem_ld32f(at, st);
                n = tmem_ld1f(at_n);
            }
            if (c == p.nchunk) {
                if (ok && row_in) {
#pragma unroll
                    for (int k = 0; k < 32; ++k)
                        if (cc + k < S.vdim) gs[k] = st[k];
                    if (has_n)
                        for (int i = 0; i < S.cl; ++i) gn[(size_t)i * S.dim] = n;
                }
                break;
            }
            float kept[32];
#pragma unroll
            for (int k = 0; k < 32; ++k) kept[k] = st[k] * decay;
            tmem_st32f(at, kept);
            if (half == 0) tmem_st1f(at_n, n * decay);
            fence_proxy_async();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&s_w);
            // beside the products: the state before this chunk, for the chunk kernel, and the next chunk's operand (its place is free, as
            // the products before these are done)
            if (d < p.dp) {
                const size_t row = ((size_t)c * S.heads + h) * p.dp + d;
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    uint32_t hi[4], lo[4];
#pragma unroll
                    for (int k = 0; k < 4; ++k) split2(row_in ? st[8 * i + 2 * k] : 0.f, row_in ? st[8 * i + 2 * k + 1] : 0.f, hi[k], lo[k]);
                    if (cc + 8 * i < p.vs) {
                        *reinterpret_cast<uint4*>(p.sh + row * p.vs + cc + 8 * i) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                        *reinterpret_cast<uint4*>(p.sl + row * p.vs + cc + 8 * i) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
                    }
                }
                if (has_n) p.sn[row] = row_in ? n : 0.f;
            }
            if (c + 1 < p.nchunk) weigh(c + 1);
            fetch(c + 2);
        }
        if (!ok && lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, 128);
}

// Grid (vt, chunks, heads), clusters of vt blocks.
constexpr int MC_MAX_DP = 320, MC_ROWS = 32, MC_BOX = MC_ROWS * 128, MC_SLOT = 4 * MC_BOX, MC_MAX_SLOTS = 4;  // a ring slot: 32 rows of S x 128 columns, both terms
struct McSmem {  // Q, K (later A high and low), V, ring of S
    int q, k, v, s, total, qbytes;
};
__host__ __device__ inline McSmem mc_smem_layout(int dp, int sstages) {
    McSmem L;
    L.qbytes = (dp + 63) / 64 * MP_SUB;
    L.q = 0;
    L.k = L.qbytes;
    L.v = L.k + (L.qbytes > 4 * MP_SUB ? L.qbytes : 4 * MP_SUB);
    L.s = L.v + 2 * MP_SUB;
    L.total = L.s + sstages * MC_SLOT;
    return L;
}
__global__ void __launch_bounds__(MP_THREADS, 1) mlstm_chunk_kernel(const __grid_constant__ MlstmPrefillParams p, const __grid_constant__ CUtensorMap map_q,
                                                                 const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                                                                 const __grid_constant__ CUtensorMap map_sh, const __grid_constant__ CUtensorMap map_sl,
                                                                 const __grid_constant__ CUtensorMap map_g) {
    extern __shared__ __align__(1024) uint8_t mc_raw[];
    __shared__ __align__(8) uint64_t s_qk, s_v, s_s[MC_MAX_SLOTS], s_sfree[MC_MAX_SLOTS], s_a, s_p, s_o, s_gate;
    __shared__ uint32_t s_tmem;
    __shared__ float s_g[MP_L];                     // a of the chunk's tokens
    __shared__ __align__(16) float s_n[MC_MAX_DP];  // n before the chunk
    __shared__ float s_den[2][MP_L];                // halves' shares of n . q
    __shared__ float s_part[2][MP_L];               // halves' sums of squares
    __shared__ float s_ss[ML_MAX_CLUSTER][MP_L];    // blocks' sums of squares
    uint8_t* smem = mc_raw + ((1024u - (smem_u32(mc_raw) & 1023u)) & 1023u);
    const MlstmShape& S = p.m.s;
    const McSmem L = mc_smem_layout(p.dp, p.sstages);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rank = (int)blockIdx.x, c0 = rank * MP_COLS, c = (int)blockIdx.y, h = (int)blockIdx.z;
    const int nd = (p.dp + 63) / 64, ns = (p.dp + MC_ROWS - 1) / MC_ROWS, t0 = c * MP_L;
    const bool state = c > 0 || p.m.pos0 > 0;       // (a sequence's first chunk has none)
    if (threadIdx.x == 0) {
        mbar_init(&s_qk, 1);
        mbar_init(&s_v, 1);
        mbar_init(&s_a, 1);
        mbar_init(&s_p, MP_WARPS);
        mbar_init(&s_o, 1);
        mbar_init(&s_gate, 1);
        for (int i = 0; i < p.sstages; ++i) {
            mbar_init(s_s + i, 1);
            mbar_init(s_sfree + i, 1);
        }
        fence_barrier_init();
        fence_proxy_async();
    }
    if (warp == 1) tmem_alloc(&s_tmem, 512);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem, tmem_a = tmem, tmem_o = tmem + 128, tmem_r = tmem + 256;
    if (p.vt > 1) cluster_arrive();  // (waited for before the first store into another block's shared memory)
    float o[2][32];                  // this thread's results (columns 32 half + 64 i ..)

    if (warp == 0) {
        if (lane == 0) {
            bool ok = true;
            mbar_arrive_expect_tx(&s_qk, (uint32_t)(2 * L.qbytes));
            for (int i = 0; i < nd; ++i) {
                tma_load_2d(smem + L.q + i * MP_SUB, &map_q, h * p.dp + 64 * i, t0, &s_qk);
                tma_load_2d(smem + L.k + i * MP_SUB, &map_k, h * p.dp + 64 * i, t0, &s_qk);
            }
            mbar_arrive_expect_tx(&s_v, 2 * MP_SUB);
            for (int i = 0; i < 2; ++i) tma_load_2d(smem + L.v + i * MP_SUB, &map_v, h * p.vp + c0 + 64 * i, t0, &s_v);
            for (int j = 0; state && j < ns && ok; ++j) {
                const int s = j % p.sstages, use = j / p.sstages;
                if (use > 0 && !mbar_wait_bounded(s_sfree + s, (uint32_t)((use - 1) & 1))) {
                    ok = false;
                    break;
                }
                uint8_t* const dst = smem + L.s + s * MC_SLOT;  // high: 2 x [32 rows][64 columns], then low
                mbar_arrive_expect_tx(s_s + s, MC_SLOT);
                const int row = (c * S.heads + h) * p.dp + MC_ROWS * j;
                for (int i = 0; i < 2; ++i) {
                    tma_load_2d(dst + i * MC_BOX, &map_sh, c0 + 64 * i, row, s_s + s);
                    tma_load_2d(dst + (2 + i) * MC_BOX, &map_sl, c0 + 64 * i, row, s_s + s);
                }
            }
            if (ok && mbar_wait_bounded(&s_o, 0u)) {  // all products are done: the gates take the operands' place
                mbar_arrive_expect_tx(&s_gate, 2 * MP_SUB);
                for (int i = 0; i < 2; ++i) tma_load_2d(smem + L.q + i * MP_SUB, &map_g, h * p.vp + c0 + 64 * i, t0, &s_gate);
            } else {
                ok = false;
            }
            if (!ok) {
                atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
                for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land within microseconds
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc_a = umma_idesc_bf16(128, 128), idesc_v = umma_idesc_bf16(128, MP_COLS, 0, 1);
            bool ok = mbar_wait_bounded(&s_qk, 0u);
            if (ok) {
                tc_fence_after();
                for (int kk = 0; 16 * kk < p.dp; ++kk)
                    umma_bf16(tmem_a, umma_desc_sw128(smem + L.q + (kk >> 2) * MP_SUB, (kk & 3) * 32), umma_desc_sw128(smem + L.k + (kk >> 2) * MP_SUB, (kk & 3) * 32), idesc_a,
                              kk ? 1u : 0u);
                umma_commit(&s_a);
            }
            for (int j = 0; state && j < ns && ok; ++j) {
                const int s = j % p.sstages, use = j / p.sstages;
                if (!mbar_wait_bounded(s_s + s, (uint32_t)(use & 1))) {
                    ok = false;
                    break;
                }
                tc_fence_after();
                const uint8_t* const src = smem + L.s + s * MC_SLOT;
                for (int term = 0; term < 2; ++term)
                    for (int kk = 0; kk < MC_ROWS / 16 && MC_ROWS * j + 16 * kk < p.dp; ++kk)
                        umma_bf16(tmem_r, umma_desc_sw128(smem + L.q + (j >> 1) * MP_SUB, (j & 1) * 64 + kk * 32), umma_desc_sw128_mn(src + 2 * term * MC_BOX, kk * 2048, MC_BOX),
                                  idesc_v, j | term | kk ? 1u : 0u);
                umma_commit(s_sfree + s);
            }
            if (ok && (!mbar_wait_bounded(&s_v, 0u) || !mbar_wait_bounded(&s_p, 0u))) ok = false;
            if (ok) {
                tc_fence_after();
                for (int term = 0; term < 2; ++term)
                    for (int kk = 0; kk < 8; ++kk)
                        umma_bf16(tmem_o, umma_desc_sw128(smem + L.k + (2 * term + (kk >> 2)) * MP_SUB, (kk & 3) * 32), umma_desc_sw128_mn(smem + L.v, kk * 2048, MP_SUB), idesc_v,
                                  term | kk ? 1u : 0u);
                umma_commit(&s_o);
            }
            if (!ok) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
        }
        __syncwarp();
    } else {
        const int qd = warp & 3, half = (warp - 2) >> 2, r = 32 * qd + lane, tid = (int)threadIdx.x - 64;
        const uint32_t lane_off = (uint32_t)(32 * qd) << 16;
        const size_t at = ((size_t)h * p.nchunk + c) * MP_L;
        if (tid < MP_L) s_g[tid] = __ldg(p.a + at + tid);
        if (state)
            for (int i = tid; i < p.dp; i += MP_WARPS * 32) s_n[i] = __ldg(p.sn + ((size_t)c * S.heads + h) * p.dp + i);
        const float M = __ldg(p.mx + at + r), w = __ldg(p.w + at + r), floor = __ldg(p.floor + at + r);
        bool ok = true;
        float den = 0.f;
        partial_sync_2(MP_WARPS * 32);
        if (!__all_sync(0xffffffffu, mbar_wait_bounded(&s_qk, 0u))) ok = false;
        if (state && ok) {  // n . q of this token: the halves take alternate 64-value pieces
            for (int j = half; j < nd; j += 2)
#pragma unroll 2
                for (int i = 0; i < 8 && 64 * j + 8 * i < p.dp; ++i) {
                    const uint4 x = *reinterpret_cast<const uint4*>(smem + L.q + j * MP_SUB + sw128_chunk(r, i));
                    const float4 a = *reinterpret_cast<const float4*>(s_n + 64 * j + 8 * i), b = *reinterpret_cast<const float4*>(s_n + 64 * j + 8 * i + 4);
                    den += __uint_as_float(x.x << 16) * a.x + __uint_as_float(x.x & 0xFFFF0000u) * a.y + __uint_as_float(x.y << 16) * a.z + __uint_as_float(x.y & 0xFFFF0000u) * a.w +
                           __uint_as_float(x.z << 16) * b.x + __uint_as_float(x.z & 0xFFFF0000u) * b.y + __uint_as_float(x.w << 16) * b.z + __uint_as_float(x.w & 0xFFFF0000u) * b.w;
                }
            den *= w;
        }
        if (ok && !__all_sync(0xffffffffu, mbar_wait_bounded(&s_a, 0u))) ok = false;
        tc_fence_after();
        // weights: this thread's row, keys 64 half .. ; A takes the place of K
#pragma unroll 1
        for (int i = 0; i < 64; i += 32) {
            float s[32];
            tmem_ld32f(tmem_a + lane_off + (uint32_t)(64 * half + i), s);
            const int k0 = 64 * half + i;
#pragma unroll
            for (int k = 0; k < 32; ++k) {
                s[k] = k0 + k <= r ? s[k] * fast_exp2((s_g[k0 + k] - M) * 1.4426950408889634f) : 0.f;
                den += s[k];
            }
            uint8_t* const hi_at = smem + L.k + half * MP_SUB;
#pragma unroll
            for (int g = 0; g < 4; ++g) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int k = 0; k < 4; ++k) split2(s[8 * g + 2 * k], s[8 * g + 2 * k + 1], hi[k], lo[k]);
                const int off = sw128_chunk(r, (i >> 3) + g);
                *reinterpret_cast<uint4*>(hi_at + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                *reinterpret_cast<uint4*>(hi_at + 2 * MP_SUB + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
        }
        s_den[half][r] = den;
        fence_proxy_async();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&s_p);
        partial_sync_2(MP_WARPS * 32);
        den = 1.f / (fmaxf(fabsf(s_den[0][r] + s_den[1][r]), floor) + 1e-6f);
        if (ok && !__all_sync(0xffffffffu, mbar_wait_bounded(&s_o, 0u))) ok = false;
        tc_fence_after();
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int col = 32 * half + 64 * i;
            tmem_ld32f(tmem_o + lane_off + (uint32_t)col, o[i]);
            if (state) {
                float x[32];
                tmem_ld32f(tmem_r + lane_off + (uint32_t)col, x);
#pragma unroll
                for (int k = 0; k < 32; ++k) o[i][k] = fmaf(w, x[k], o[i][k]);
            }
#pragma unroll
            for (int k = 0; k < 32; ++k) {
                o[i][k] = c0 + col + k < S.vdim ? o[i][k] * den : 0.f;
                ss = fmaf(o[i][k], o[i][k], ss);
            }
        }
        s_part[half][r] = ss;
        if (ok && !__all_sync(0xffffffffu, mbar_wait_bounded(&s_gate, 0u))) ok = false;
        if (!ok && lane == 0) atomicExch(p.status, DEV_ERR_TMA_TIMEOUT);
        partial_sync_2(MP_WARPS * 32);
    }
    // (the threads of every warp come here: the cluster's barriers count all of them)
    const int row = 32 * (warp & 3) + lane, half = (warp - 2) >> 2;
    if (p.vt > 1) {
        cluster_wait();
        if (warp >= 2) {
            const float ss = s_part[0][row] + s_part[1][row];
            for (int i = half; i < p.vt; i += 2) st_cluster_f32(cluster_map(&s_ss[rank][row], (uint32_t)i), ss);
        }
        cluster_sync_all();
    } else if (warp >= 2) {
        if (half == 0) s_ss[0][row] = s_part[0][row] + s_part[1][row];
        partial_sync_2(MP_WARPS * 32);
    }
    if (warp >= 2) {
        float ss = 0.f;
        for (int i = 0; i < p.vt; ++i) ss += s_ss[i][row];
        const float scale = 1.f / sqrtf(ss / (float)S.vdim + S.eps);
        bf16* const out = static_cast<bf16*>(p.m.out);
        const bool wide = ((S.vdim | p.m.ldo) & 7) == 0;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int cc = c0 + 32 * half + 64 * i;           // first column within the head
            const int nv = t0 + row < p.n ? S.vdim - cc : 0;  // values of this token to store
            bf16* const dst = out + (size_t)(t0 + row) * p.m.ldo + (size_t)h * S.vdim + cc;
#pragma unroll
            for (int g = 0; g < 4; ++g) {
                const uint4 g8 = *reinterpret_cast<const uint4*>(smem + L.q + i * MP_SUB + sw128_chunk(row, 4 * half + g));
                const float* const x = o[i] + 8 * g;
                const uint4 v = make_uint4(mul_pack_bf16(g8.x, x[0] * scale, x[1] * scale), mul_pack_bf16(g8.y, x[2] * scale, x[3] * scale),
                                           mul_pack_bf16(g8.z, x[4] * scale, x[5] * scale), mul_pack_bf16(g8.w, x[6] * scale, x[7] * scale));
                if (wide) {
                    if (8 * g < nv) *reinterpret_cast<uint4*>(dst + 8 * g) = v;
                } else {
                    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                    for (int k = 0; k < 8; ++k)
                        if (8 * g + k < nv) dst[8 * g + k] = __ushort_as_bfloat16((unsigned short)(w[k >> 1] >> (16 * (k & 1))));
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, 512);
}

}  // namespace l2b
