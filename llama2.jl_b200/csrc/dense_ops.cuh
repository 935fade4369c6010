// Arithmetic shared by the kernels of the layer-stack models (stack.cu): 8 stored values at a time as f32, activations, rotary
// pairs, and the epilogues of the dense matrix products.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace l2b {

typedef __nv_bfloat16 bf16;

// Two f32 values in one register pair: one instruction does both multiply-adds, each rounded as fmaf rounds.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ float sum2(f32x2 v) {
    float lo, hi;
    unpack2(v, lo, hi);
    return lo + hi;
}
// two stored bf16 (one word) as two f32
__device__ __forceinline__ f32x2 widen2(uint32_t w) { return pack2(__uint_as_float(w << 16), __uint_as_float(w & 0xFFFF0000u)); }

// An f32 vector that warps read 8 consecutive values per lane (value e = 256 c + 8 lane + j) lies in shared memory as two float4
// halves per 256 values, so that the 16-byte reads of a warp are free of bank conflicts.
__device__ __forceinline__ int lane_major(int e) { return (e & ~255) + ((e >> 2) & 1) * 128 + ((e >> 3) & 31) * 4 + (e & 3); }
struct Pairs8 {
    f32x2 p[4];
};
__device__ __forceinline__ Pairs8 read_lane_major(const float* x, int c, int lane) {
    const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(x + c * 256 + lane * 4), b = *reinterpret_cast<const ulonglong2*>(x + c * 256 + 128 + lane * 4);
    Pairs8 o;
    o.p[0] = a.x; o.p[1] = a.y; o.p[2] = b.x; o.p[3] = b.y;
    return o;
}

// N sums over the lanes of a warp at once.  While more than one value is left, a step exchanges half of the values across a lane bit
// and halves their number; the remaining bits are reduced as usual.  Lanes i * 32/N .. end up with sum i.
template <int N>
__device__ __forceinline__ float warp_sums_spread(const float (&v)[N]) {
    static_assert(N == 1 || N == 2 || N == 4 || N == 8, "number of sums");
    const int lane = threadIdx.x & 31;
    float t[N];
#pragma unroll
    for (int i = 0; i < N; ++i) t[i] = v[i];
    int o = 16;
#pragma unroll
    for (int n = N; n > 1; n >>= 1, o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int i = 0; i < n / 2; ++i) {
            const float keep = up ? t[i + n / 2] : t[i], send = up ? t[i] : t[i + n / 2];
            t[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
    }
#pragma unroll
    for (; o > 0; o >>= 1) t[0] += __shfl_xor_sync(0xffffffffu, t[0], o);
    return t[0];
}
// The same with every lane getting all sums.
template <int N>
__device__ __forceinline__ void warp_sums(float (&v)[N]) {
    const float t = warp_sums_spread<N>(v);
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = N > 1 ? __shfl_sync(0xffffffffu, t, i * (32 / N)) : t;
}

template <typename T>
struct Raw8;  // eight consecutive values (16-byte aligned bf16 or f32) as loaded, before conversion
template <>
struct Raw8<bf16> {
    uint4 r;
    __device__ __forceinline__ void zero() { r = make_uint4(0u, 0u, 0u, 0u); }
    __device__ __forceinline__ void load(const bf16* p) { r = __ldcg(reinterpret_cast<const uint4*>(p)); }
    __device__ __forceinline__ void read(const void* smem) { r = *static_cast<const uint4*>(smem); }
    __device__ __forceinline__ Pairs8 pairs() const {
        Pairs8 o;
        o.p[0] = widen2(r.x); o.p[1] = widen2(r.y); o.p[2] = widen2(r.z); o.p[3] = widen2(r.w);
        return o;
    }
};
template <>
struct Raw8<float> {
    float4 a, b;
    __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
    __device__ __forceinline__ void read(const void* smem) {
        a = static_cast<const float4*>(smem)[0];
        b = static_cast<const float4*>(smem)[1];
    }
    __device__ __forceinline__ Pairs8 pairs() const {
        Pairs8 o;
        o.p[0] = pack2(a.x, a.y); o.p[1] = pack2(a.z, a.w); o.p[2] = pack2(b.x, b.y); o.p[3] = pack2(b.z, b.w);
        return o;
    }
};

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float gelu_tanh(float z) {
    const float t = tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z));  // sqrt(2 / pi)
    return 0.5f * z * (1.f + t);
}
__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float dynamic_tanh(float x, float alpha, float w, float b) { return fmaf(tanhf(alpha * x), w, b); }

// element d of a vector whose first rdims elements are interleaved rotary pairs; get(i) reads element i, cs = this position's row
template <class Get>
__device__ __forceinline__ float rotary_element(int d, int rdims, const float2* cs, Get get) {
    if (d >= rdims) return get(d);
    const float2 t = __ldg(cs + (d >> 1));
    return (d & 1) ? get(d) * t.x + get(d - 1) * t.y : get(d) * t.x - get(d + 1) * t.y;
}

// What happens to a result of a dense product W x before it is stored.
enum : int {
    DE_STORE = 0,     // y[t][f] f32
    DE_RESIDUAL = 1,  // y[t][f] += f32
    DE_GEGLU = 2,     // act[t][f] = gelu_tanh(gate) * up (two weight rows per result)
    DE_SIDE = 3,      // act[t][f] = gelu_tanh(v) * e, e = element e_off + f of the token's row of an embedding table
    DE_LOGITS = 4,    // as DE_STORE, and the block's first maximum
    DE_STORE_ACT = 5, // act[t][f]
    DE_STORE_T = 6,   // act[f][t] (transposed)
    DE_SWIGLU = 7,    // act[t][f] = silu(gate) * up (two weight rows per result)
    DE_AFFINE = 8,    // y[t][f] = mul * v + bias[f]
    DE_AFFINE_LOGITS = 9  // as DE_AFFINE, and the block's first maximum
};
struct DenseEpilogue {
    int kind;
    float mul;            // DE_AFFINE, DE_AFFINE_LOGITS
    const float* bias;    // the same (null: nothing)
    float* y;
    void* act;
    int ld;               // elements between rows of y / act
    const bf16* etab;     // DE_SIDE
    int e_ld, e_off;
    const int* tokens;    // DE_SIDE: token of result row t
    int vocab;            // DE_SIDE: rows of the table (an id outside it contributes zero)
};
inline DenseEpilogue dense_epilogue_of(int kind, float* y, void* act, int ld) {
    DenseEpilogue e = {};
    e.kind = kind;
    e.y = y;
    e.act = act;
    e.ld = ld;
    return e;
}
inline DenseEpilogue affine_epilogue(int kind, float mul, const float* bias, float* y, int ld) {
    DenseEpilogue e = dense_epilogue_of(kind, y, nullptr, ld);
    e.mul = mul;
    e.bias = bias;
    return e;
}
__device__ __forceinline__ float affine(const DenseEpilogue& e, int f, float v) { return e.bias ? fmaf(v, e.mul, __ldg(e.bias + f)) : v * e.mul; }
__device__ __forceinline__ float side_value(const DenseEpilogue& e, int t, int f) {
    const int tok = __ldg(e.tokens + t);
    const bool valid = tok >= 0 && tok < e.vocab;  // (the load does not depend on it: several are in flight together)
    const float v = __bfloat162float(e.etab[(size_t)(valid ? tok : 0) * e.e_ld + e.e_off + f]);
    return valid ? v : 0.f;
}
// KINDS: bits of the kinds a kernel may meet (code for kinds that a short kernel never meets costs it time).
constexpr unsigned DE_EVERY = ~0u;
template <typename AT, unsigned KINDS = DE_EVERY>
__device__ __forceinline__ void dense_epilogue(const DenseEpilogue& e, int t, int f, float v, float v2) {
    const size_t o = (size_t)t * e.ld + f;
    AT* act = static_cast<AT*>(e.act);
    switch (e.kind) {
        case DE_STORE: case DE_LOGITS: e.y[o] = v; break;
        case DE_RESIDUAL: e.y[o] += v; break;
        case DE_GEGLU: if (KINDS >> DE_GEGLU & 1) put(act + o, gelu_tanh(v) * v2); break;
        case DE_SIDE: if (KINDS >> DE_SIDE & 1) put(act + o, gelu_tanh(v) * side_value(e, t, f)); break;
        case DE_STORE_ACT: if (KINDS >> DE_STORE_ACT & 1) put(act + o, v); break;
        case DE_STORE_T: if (KINDS >> DE_STORE_T & 1) put(act + (size_t)f * e.ld + t, v); break;
        case DE_SWIGLU: if (KINDS >> DE_SWIGLU & 1) put(act + o, silu(v) * v2); break;
        case DE_AFFINE: case DE_AFFINE_LOGITS: if (KINDS >> DE_AFFINE & 1) e.y[o] = affine(e, f, v); break;
    }
}

// Pending changes of the residual stream that the next reader applies: x' = x + y / rms(y) * w + step.
struct ResidualUpdate {
    const float* y;       // result whose norm comes before it is added: a sublayer's, or the per-layer token input's (null: none)
    const float* w;       // that norm's weight
    float eps;
    const float* step;    // vector added at the beginning of a loop pass (null: none)
};
// The norm in front of a dense product.
enum : int { NORM_NONE = 0, NORM_DYNAMIC_TANH = 1, NORM_RMS = 2 };
struct NormParams {
    int kind;
    float alpha;          // dynamic tanh
    float eps;            // rms
    const float* w;
    const float* b;       // dynamic tanh
};
// One value; rms: without the factor 1 / rms(x).
template <bool RMS>
__device__ __forceinline__ float apply_norm(const NormParams& n, float x, int i) {
    if (RMS) return x * __ldg(n.w + i);
    return n.kind ? dynamic_tanh(x, n.alpha, __ldg(n.w + i), __ldg(n.b + i)) : x;
}

// Barrier over the first `threads` threads of the block.
__device__ __forceinline__ void partial_sync(int threads) { asm volatile("bar.sync 1, %0;" ::"r"(threads) : "memory"); }

__device__ __forceinline__ void partial_sync_2(int threads) { asm volatile("bar.sync 2, %0;" ::"r"(threads) : "memory"); }  // any `threads` threads

// 2^x as one special-function instruction (about 2 ulp; results below the normal range become 0)
__device__ __forceinline__ float fast_exp2(float x) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}

__device__ __forceinline__ uint32_t pack_bf16(float x, float y) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    return *reinterpret_cast<const uint32_t*>(&h);
}
// x = hi + lo with both bf16: two values -> two packed words
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x, y);
    lo = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
}

// sigmoid for results that are rounded to bf16 next
__device__ __forceinline__ float fast_sigmoid(float z) { return __fdividef(1.f, 1.f + fast_exp2(z * -1.4426950408889634f)); }

// two packed bf16 times two f32
__device__ __forceinline__ uint32_t mul_pack_bf16(uint32_t g, float x, float y) { return pack_bf16(__uint_as_float(g << 16) * x, __uint_as_float(g & 0xFFFF0000u) * y); }

// Sum over the first NW warps of a block; each of their threads gets it.  s holds NW floats and may be reused after the next barrier.
template <int NW>
__device__ __forceinline__ float block_sum_all(float v, float* s) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) s[threadIdx.x >> 5] = v;
    partial_sync(NW * 32);
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < NW; ++i) t += s[i];
    return t;
}

}  // namespace l2b
