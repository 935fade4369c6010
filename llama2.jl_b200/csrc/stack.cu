// Layer-stack models: weights, caches and the kernel sequences of one position and of many (see stack.h).
#include "stack.h"

#include <algorithm>
#include <cmath>
#include <map>
#include <memory>
#include <mutex>

#include "dense_gemm.cuh"
#include "dense_matvec.cuh"
#include "latent_attention.cuh"
#include "latent_prefill.cuh"
#include "stack_rows.cuh"

using namespace l2b;

namespace {

int up(int v, int m) { return (v + m - 1) / m * m; }

// A weight matrix in bf16, rows padded to a multiple of 8 values.  Several tensors may be row ranges of one matrix; `pair` = 2:
// rows 2u and 2u + 1 belong to result u (gate and up).
struct StackMatrix {
    bf16* w = nullptr;
    int rows = 0, k = 0, kp = 0, pair = 1;
    int64_t bytes() const { return (int64_t)rows * kp * 2; }
    const bf16* second() const { return w + kp; }
    size_t stride() const { return (size_t)kp * pair; }
    int results() const { return rows / pair; }
};
struct StackNorm {
    float* w = nullptr;
    float* b = nullptr;
    float alpha = 1.f;
};
struct StackLayerW {
    StackNorm norm1, norm2;
    StackMatrix qdg;  // query, down and gate projections, one below the other
    StackMatrix uk, uv, o, gu, down, side_gate, side_proj;
    float *dkv_norm = nullptr, *sink = nullptr, *side_norm = nullptr;
    LatentShape shape;
    int off_d = 0, off_g = 0;
};

// Where a tensor of the file goes.
struct TensorSlot {
    std::vector<int64_t> shape;
    StackMatrix* mat = nullptr;    // matrix rows row0, row0 + row_step, ...; heads > 0: rows of a head are head_pad apart
    int row0 = 0, row_step = 1, head_rows = 0, head_pad = 0;
    float** vec = nullptr;         // f32 vector (any shape, flattened)
    float* scalar = nullptr;       // host scalar
    bool loaded = false;
};

}  // namespace

struct StackModel {
    StackConfig cfg;
    bool f32 = false;
    std::vector<StackLayerW> layers;
    std::vector<LayerRun> runs;
    StackMatrix embed, head, side_embed;
    StackNorm final_norm;
    float* loop_step = nullptr;  // [times][width]
    std::map<std::string, TensorSlot> slots;
    std::vector<void*> owned;
};

static int32_t alloc_owned(std::vector<void*>& owned, void** p, size_t bytes) {
    CU(cudaMalloc(p, bytes));
    owned.push_back(*p);
    CU(cudaMemset(*p, 0, bytes));
    return L2B_OK;
}

static int32_t make_matrix(StackModel* m, StackMatrix& w, int rows, int k, int pair = 1) {
    w.rows = rows;
    w.k = k;
    w.kp = up(k, 8);
    w.pair = pair;
    return alloc_owned(m->owned, (void**)&w.w, (size_t)w.bytes());
}

static void add_matrix(StackModel* m, const std::string& name, StackMatrix& w, int rows, int row0 = 0, int row_step = 1, int head_rows = 0, int head_pad = 0) {
    TensorSlot s;
    s.shape = {rows, w.k};
    s.mat = &w;
    s.row0 = row0;
    s.row_step = row_step;
    s.head_rows = head_rows;
    s.head_pad = head_pad;
    m->slots[name] = s;
}
static void add_vector(StackModel* m, const std::string& name, float** v, std::vector<int64_t> shape) {
    TensorSlot s;
    s.shape = std::move(shape);
    s.vec = v;
    m->slots[name] = s;
}
static void add_norm(StackModel* m, const std::string& name, StackNorm& n) {
    add_vector(m, name, &n.w, {m->cfg.width});
    switch (m->cfg.norm) {
        case NormKind::DynamicTanh:
            add_vector(m, name + ".b", &n.b, {m->cfg.width});
            TensorSlot s;
            s.scalar = &n.alpha;
            m->slots[name + ".alpha"] = s;
            break;
    }
}
static NormParams norm_params(const StackModel* m, const StackNorm& n) {
    NormParams p = {0, 0.f, nullptr, nullptr};
    switch (m->cfg.norm) {
        case NormKind::DynamicTanh: p = {1, n.alpha, n.w, n.b}; break;
    }
    return p;
}

static int32_t build_latent_attention(StackModel* m, StackLayerW& w, const MixerConfig& c, const std::string& p) {
    const int width = m->cfg.width;
    LatentShape& s = w.shape;
    s.heads = c.heads; s.dim = c.dim; s.rot = c.rot_dim; s.rdims = c.rot.dims; s.vdim = c.vdim; s.rank = c.kv_rank;
    s.rp = up(c.kv_rank, 8);
    s.row = s.rp + up(c.rot_dim, 8);
    s.dp = up(c.dim, 16);
    s.vp = up(c.vdim, 16);
    s.scale2 = (float)((double)c.scale * 1.4426950408889634);
    s.eps = m->cfg.eps;
    if (s.row > 1024) return fail(L2B_ERR_UNSUPPORTED_TYPE, "latent attention takes kv_rank + rot_dim up to 1024");
    const int nq = c.heads * (c.dim + c.rot_dim), nd = c.kv_rank + c.rot_dim, ng = c.heads * c.vdim;
    w.off_d = nq;
    w.off_g = nq + nd;
    L2B_TRY(make_matrix(m, w.qdg, nq + nd + ng, width));
    add_matrix(m, p + "q", w.qdg, nq, 0);
    add_matrix(m, p + "dkv", w.qdg, nd, nq);
    add_matrix(m, p + "g", w.qdg, ng, nq + nd);
    L2B_TRY(make_matrix(m, w.uk, c.heads * s.dp, c.kv_rank));
    add_matrix(m, p + "uk", w.uk, c.heads * c.dim, 0, 1, c.dim, s.dp);
    L2B_TRY(make_matrix(m, w.uv, c.heads * s.vp, c.kv_rank));
    add_matrix(m, p + "uv", w.uv, c.heads * c.vdim, 0, 1, c.vdim, s.vp);
    L2B_TRY(make_matrix(m, w.o, width, ng));
    add_matrix(m, p + "o", w.o, width);
    add_vector(m, p + "dkv.norm", &w.dkv_norm, {c.kv_rank});
    add_vector(m, p + "sink", &w.sink, {c.heads});
    return L2B_OK;
}

int32_t stack_model_create(const char* json, size_t n, bool f32, StackModel** out) {
    *out = nullptr;
    std::unique_ptr<StackModel, void (*)(StackModel*)> m(new StackModel(), stack_model_free);
    std::string err;
    if (!parse_stack_config(json, n, m->cfg, err)) return fail(L2B_ERR_BAD_ARG, err);
    const StackConfig& c = m->cfg;
    m->f32 = f32;
    m->runs = c.runs();
    m->layers.resize(c.layers.size());
    L2B_TRY(make_matrix(m.get(), m->head, c.vocab, c.width));
    add_matrix(m.get(), "head", m->head, c.vocab);
    m->embed.rows = c.vocab; m->embed.k = m->embed.kp = c.width;  // read row by row: not padded
    L2B_TRY(alloc_owned(m->owned, (void**)&m->embed.w, (size_t)m->embed.bytes()));
    add_matrix(m.get(), "embed", m->embed, c.vocab);
    add_norm(m.get(), "final.norm", m->final_norm);
    if (c.has_loop()) add_vector(m.get(), "loop.step", &m->loop_step, {c.loop_times, c.width});
    if (c.side_dim) {
        m->side_embed.rows = c.vocab; m->side_embed.k = m->side_embed.kp = c.side_dim * (int)c.layers.size();
        L2B_TRY(alloc_owned(m->owned, (void**)&m->side_embed.w, (size_t)m->side_embed.bytes()));
        add_matrix(m.get(), "side.embed", m->side_embed, c.vocab);
    }
    for (size_t i = 0; i < c.layers.size(); ++i) {
        const StackLayerConfig& l = c.layers[i];
        StackLayerW& w = m->layers[i];
        const std::string p = "l" + std::to_string(i) + ".";
        add_norm(m.get(), p + "norm1", w.norm1);
        switch (l.mix.kind) {
            case MixerKind::LatentAttention: L2B_TRY(build_latent_attention(m.get(), w, l.mix, p + "mix.")); break;
        }
        switch (l.mlp) {
            case MlpKind::None: break;
            case MlpKind::GatedGeluTanh:
                add_norm(m.get(), p + "norm2", w.norm2);
                L2B_TRY(make_matrix(m.get(), w.gu, 2 * l.ff, c.width, 2));
                add_matrix(m.get(), p + "mlp.gate", w.gu, l.ff, 0, 2);
                add_matrix(m.get(), p + "mlp.up", w.gu, l.ff, 1, 2);
                L2B_TRY(make_matrix(m.get(), w.down, c.width, l.ff));
                add_matrix(m.get(), p + "mlp.down", w.down, c.width);
                break;
        }
        if (c.side_dim) {
            L2B_TRY(make_matrix(m.get(), w.side_gate, c.side_dim, c.width));
            add_matrix(m.get(), p + "side.gate", w.side_gate, c.side_dim);
            L2B_TRY(make_matrix(m.get(), w.side_proj, c.width, c.side_dim));
            add_matrix(m.get(), p + "side.proj", w.side_proj, c.width);
            add_vector(m.get(), p + "side.norm", &w.side_norm, {c.width});
        }
    }
    *out = m.release();
    return L2B_OK;
}

const StackConfig& stack_model_config(const StackModel* m) { return m->cfg; }
bool stack_model_has(const StackModel* m, const std::string& name) { return m->slots.count(name) != 0; }

int32_t stack_model_upload(StackModel* m, const char* name, int dtype, const void* host, const int64_t* shape, int ndim) {
    auto it = m->slots.find(name);
    if (it == m->slots.end()) return fail(L2B_ERR_BAD_ARG, std::string("the design has no tensor ") + name);
    TensorSlot& s = it->second;
    int64_t count = 1;
    for (int i = 0; i < ndim; ++i) count *= shape[i];
    if (s.scalar ? count != 1 : std::vector<int64_t>(shape, shape + ndim) != s.shape) return fail(L2B_ERR_BAD_ARG, std::string("tensor ") + name + " has an unexpected shape");
    if (dtype != L2B_TYPE_BF16 && !(dtype == L2B_TYPE_F32 && !s.mat))
        return fail(L2B_ERR_UNSUPPORTED_TYPE, std::string("tensor ") + name + ": matrices must be bf16, vectors bf16 or f32");
    if (s.mat) {
        const StackMatrix& w = *s.mat;
        const size_t src_pitch = (size_t)w.k * 2, dst_pitch = (size_t)w.kp * 2;
        const int rows = (int)s.shape[0], per = s.head_rows ? s.head_rows : rows, pad = s.head_rows ? s.head_pad : 0;
        for (int g = 0; g * per < rows; ++g)
            CU(cudaMemcpy2D(w.w + (size_t)(s.row0 + (size_t)g * pad) * w.kp, dst_pitch * s.row_step, static_cast<const uint8_t*>(host) + (size_t)g * per * src_pitch, src_pitch,
                            src_pitch, per, cudaMemcpyHostToDevice));
    } else {
        std::vector<float> v((size_t)count);
        for (int64_t i = 0; i < count; ++i) {
            if (dtype == L2B_TYPE_F32) v[i] = static_cast<const float*>(host)[i];
            else {
                const uint32_t u = (uint32_t) static_cast<const uint16_t*>(host)[i] << 16;
                memcpy(&v[i], &u, 4);
            }
        }
        if (s.scalar) *s.scalar = v[0];
        else {
            if (!*s.vec) L2B_TRY(alloc_owned(m->owned, (void**)s.vec, (size_t)count * 4));
            CU(cudaMemcpy(*s.vec, v.data(), (size_t)count * 4, cudaMemcpyHostToDevice));
        }
    }
    s.loaded = true;
    return L2B_OK;
}

int32_t stack_model_finalize(StackModel* m) {
    for (const auto& s : m->slots)
        if (!s.second.loaded) return fail(L2B_ERR_STATE, "tensor " + s.first + " is missing");
    return L2B_OK;
}

void stack_model_free(StackModel* m) {
    if (!m) return;
    for (void* p : m->owned) cudaFree(p);
    delete m;
}

int64_t stack_model_bytes_per_token(const StackModel* m) {
    int64_t b = m->head.bytes() + (int64_t)m->cfg.width * 2;
    for (const LayerRun& r : m->runs) {
        const StackLayerW& w = m->layers[r.layer];
        b += w.qdg.bytes() + w.uk.bytes() + w.uv.bytes() + w.o.bytes() + w.gu.bytes() + w.down.bytes() + w.side_gate.bytes() + w.side_proj.bytes();
    }
    return b;
}

// ---------------------------------------------------------------------------------------------
// session
// ---------------------------------------------------------------------------------------------
struct StackSession {
    const StackModel* m = nullptr;
    StackSessionInfo info;
    DeviceInfo di;
    std::vector<void*> owned;
    std::vector<void*> cache;                    // per run: [n_seq][seq_len][row] of bf16 or f32
    std::vector<size_t> cache_bytes;
    std::vector<const float2*> rope;             // per layer
    // one position
    float *x[2] = {nullptr, nullptr}, *qdg1 = nullptr, *att1 = nullptr, *hid1 = nullptr, *y1 = nullptr;
    int x_last = 0;
    // absorbed attention: queries and partial results of up to ABSORB_ROWS rows
    float *qp = nullptr, *part_acc = nullptr;
    float2* part_ml = nullptr;
    // many positions
    float *xr = nullptr, *qdg = nullptr, *y = nullptr;
    void *act = nullptr, *act2 = nullptr;        // operands of the products, [max_rows][k rounded up to 8]
    bf16 *pq = nullptr, *pk = nullptr, *pv = nullptr;  // expanded attention: queries, keys, transposed values
    int pv_ld = 0;
};

static size_t act_bytes(const StackModel* m) { return m->f32 ? 4 : 2; }

constexpr int ABSORB_ROWS = 64;  // rows per pass of the absorbed form of the attention (bounds its scratch)
// The expanded form of the attention (latent_prefill.cuh) is for portions of at least this many rows.
constexpr int EXPAND_MIN_ROWS = 48;

// Groups of heads and ranges of positions of the scan kernel: about one block per SM in a decode step, two for several rows.
static int latent_groups(const LatentShape& s, bool f32) { return f32 ? (s.heads + LA_WARPS - 1) / LA_WARPS : (s.heads + LM_HEADS - 1) / LM_HEADS; }
static int latent_splits(const LatentShape& s, bool f32, int rows, const DeviceInfo& di) {
    return std::max(1, std::min(LA_MAX_SPLIT, (rows == 1 ? 1 : 2) * di.sms / (latent_groups(s, f32) * rows)));
}

static int prefill_kstages(const LatentShape& s, const DeviceInfo& di) {
    if (s.vp > 256) return 0;
    for (int k = 2; k >= 1; --k)
        if (lp_smem_layout(s.dim, s.rot, s.vp, k).total + 1024 <= di.max_smem_optin - 1024) return k;
    return 0;
}

static std::once_flag g_stack_attr_once;
static cudaError_t g_stack_attr_err = cudaSuccess;
static int32_t set_stack_kernel_attrs() {
    std::call_once(g_stack_attr_once, [] {
        int dev = 0, optin = 0;
        cudaGetDevice(&dev);
        cudaDeviceGetAttribute(&optin, cudaDevAttrMaxSharedMemoryPerBlockOptin, dev);
        auto set = [&](const void* f) {
            cudaFuncAttributes fa;
            cudaError_t e = cudaFuncGetAttributes(&fa, f);
            if (e == cudaSuccess) e = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, optin - (int)fa.sharedSizeBytes);
            if (e != cudaSuccess) g_stack_attr_err = e;
        };
        set((const void*)dense_matvec_kernel);
        set((const void*)latent_prefill_kernel);
        set((const void*)bf16_gemm_kernel<32, 1>); set((const void*)bf16_gemm_kernel<32, 2>);
        set((const void*)bf16_gemm_kernel<64, 1>); set((const void*)bf16_gemm_kernel<64, 2>);
        set((const void*)bf16_gemm_kernel<128, 1>); set((const void*)bf16_gemm_kernel<128, 2>);
        set((const void*)latent_scan_kernel<float, 1>); set((const void*)latent_scan_kernel<float, 2>);
        set((const void*)latent_scan_kernel<float, 3>); set((const void*)latent_scan_kernel<float, 4>);
        set((const void*)latent_scan_mma_kernel<1>); set((const void*)latent_scan_mma_kernel<2>); set((const void*)latent_scan_mma_kernel<3>);
        set((const void*)latent_scan_mma_kernel<5>); set((const void*)latent_scan_mma_kernel<8>);
    });
    if (g_stack_attr_err != cudaSuccess) return fail(L2B_ERR_CUDA, std::string("cudaFuncSetAttribute: ") + cudaGetErrorString(g_stack_attr_err));
    return L2B_OK;
}

static int32_t build_rope(StackSession* s) {
    std::map<std::pair<double, int>, const float2*> made;
    for (const StackLayerConfig& l : s->m->cfg.layers) {
        const RotaryConfig& r = l.mix.rot;
        const float2*& t = made[{r.base, r.dims}];
        if (!t) {
            const int h = r.dims / 2;
            std::vector<float2> cs((size_t)s->info.seq_len * h);
            for (int i = 0; i < h; ++i) {
                const double f = std::pow(r.base, -2.0 * i / r.dims);
                for (int p = 0; p < s->info.seq_len; ++p) cs[(size_t)p * h + i] = make_float2((float)std::cos(p * f), (float)std::sin(p * f));
            }
            void* d = nullptr;
            L2B_TRY(alloc_owned(s->owned, &d, cs.size() * sizeof(float2)));
            CU(cudaMemcpy(d, cs.data(), cs.size() * sizeof(float2), cudaMemcpyHostToDevice));
            t = static_cast<const float2*>(d);
        }
        s->rope.push_back(t);
    }
    return L2B_OK;
}

int32_t stack_session_create(const StackModel* m, const StackSessionInfo& info, const DeviceInfo& di, cudaStream_t st, StackSession** out) {
    *out = nullptr;
    L2B_TRY(set_stack_kernel_attrs());
    std::unique_ptr<StackSession, void (*)(StackSession*)> s(new StackSession(), stack_session_free);
    s->m = m;
    s->info = info;
    s->di = di;
    const StackConfig& c = m->cfg;
    int max_qdg = 1, max_k = c.width, max_k2 = 1;
    size_t pq = 0, pk = 0, pv = 0;
    s->pv_ld = up(info.seq_len, 8);
    for (const StackLayerW& w : m->layers) {
        max_qdg = std::max(max_qdg, w.qdg.rows);
        max_k2 = std::max(std::max(max_k2, w.o.k), std::max(w.down.k, w.side_proj.k));
        pq = std::max(pq, (size_t)w.shape.heads * (w.shape.dp + up(w.shape.rot, 16)));
        pk = std::max(pk, (size_t)w.shape.heads * w.shape.dp);
        pv = std::max(pv, (size_t)w.shape.heads * w.shape.vp);
    }
    auto alloc = [&](auto*& p, size_t bytes) { return alloc_owned(s->owned, (void**)&p, bytes); };
    for (const LayerRun& r : m->runs) {
        const size_t b = (size_t)info.n_seq * info.seq_len * m->layers[r.layer].shape.row * act_bytes(m);
        void* p = nullptr;
        L2B_TRY(alloc_owned(s->owned, &p, b));
        s->cache.push_back(p);
        s->cache_bytes.push_back(b);
    }
    L2B_TRY(build_rope(s.get()));
    if (info.decode) {
        for (float*& x : s->x) L2B_TRY(alloc(x, (size_t)c.width * 4));
        L2B_TRY(alloc(s->qdg1, (size_t)max_qdg * 4));
        L2B_TRY(alloc(s->att1, (size_t)max_k2 * 4));
        L2B_TRY(alloc(s->hid1, (size_t)max_k2 * 4));
        L2B_TRY(alloc(s->y1, (size_t)c.width * 4));
    }
    size_t qp = 0, pml = 0, pacc = 0;
    for (const StackLayerW& w : m->layers)
        for (int rows = 1; rows <= std::max(1, std::min(ABSORB_ROWS, info.max_rows)); ++rows) {
            const size_t pairs = (size_t)w.shape.heads * rows, slots = pairs * latent_splits(w.shape, m->f32, rows, di);
            qp = std::max(qp, pairs * w.shape.row);
            pml = std::max(pml, slots);
            pacc = std::max(pacc, slots * w.shape.rp);
        }
    L2B_TRY(alloc(s->qp, qp * 4));
    L2B_TRY(alloc(s->part_ml, pml * sizeof(float2)));
    L2B_TRY(alloc(s->part_acc, pacc * 4));
    const size_t T = (size_t)info.max_rows;
    L2B_TRY(alloc(s->xr, T * c.width * 4));
    L2B_TRY(alloc(s->qdg, T * max_qdg * 4));
    L2B_TRY(alloc(s->y, T * c.width * 4));
    L2B_TRY(alloc(s->act, T * up(max_k, 8) * act_bytes(m)));
    L2B_TRY(alloc(s->act2, T * up(max_k2, 8) * act_bytes(m)));
    if (!m->f32 && info.n_seq == 1 && info.max_rows >= EXPAND_MIN_ROWS) {
        L2B_TRY(alloc(s->pq, T * pq * 2));
        L2B_TRY(alloc(s->pk, (size_t)info.seq_len * pk * 2));
        L2B_TRY(alloc(s->pv, pv * s->pv_ld * 2));
    }
    CU(cudaStreamSynchronize(st));
    CU(cudaDeviceSynchronize());
    *out = s.release();
    return L2B_OK;
}

void stack_session_free(StackSession* s) {
    if (!s) return;
    for (void* p : s->owned) cudaFree(p);
    delete s;
}

int32_t stack_session_reset(StackSession* s, cudaStream_t st) {
    for (size_t i = 0; i < s->cache.size(); ++i) CU(cudaMemsetAsync(s->cache[i], 0, s->cache_bytes[i], st));
    return L2B_OK;
}
int stack_session_max_rows(const StackSession* s) { return s->info.max_rows; }
const float* stack_session_residual(const StackSession* s) { return s->x[s->x_last]; }

// ---- latent attention launch -------------------------------------------------------------------
static LatentAttnParams latent_params(const StackSession* s, int run, const float* qdg) {
    const StackModel* m = s->m;
    const int l = m->runs[run].layer;
    const StackLayerW& w = m->layers[l];
    LatentAttnParams a;
    memset(&a, 0, sizeof(a));
    a.s = w.shape;
    a.qdg = qdg; a.ld = w.qdg.rows; a.off_d = w.off_d; a.off_g = w.off_g;
    a.uk = w.uk.w; a.uv = w.uv.w; a.sink = w.sink; a.dnorm = w.dkv_norm; a.rope = s->rope[l];
    a.cache = s->cache[run];
    a.qp = s->qp; a.part_ml = s->part_ml; a.part_acc = s->part_acc;
    return a;
}
// The absorbed form for `rows` rows (row pointers already in `a`): query, scan, output.  chained: the first launch depends
// programmatically on the kernel before it (decode).
template <typename CT, typename OT>
static cudaError_t launch_latent_attention(LatentAttnParams a, int rows, bool chained, const DeviceInfo& di, cudaStream_t st) {
    const LatentShape& s = a.s;
    const long pairs = (long)s.heads * rows;
    for (a.csplit = 1; a.csplit < 8 && pairs * a.csplit < di.sms;) a.csplit *= 2;
    for (a.vsplit = 1; a.vsplit < 4 && pairs * a.vsplit < di.sms;) a.vsplit *= 2;
    constexpr bool f32 = sizeof(CT) == 4;
    a.nsplit = latent_splits(s, f32, rows, di);
    const int stage = f32 ? LA_STAGE_ROWS * s.row * 4 : lm_stage_bytes(s.row);
    a.stages = std::max(1, std::min(LA_MAX_STAGES, (di.max_smem_optin - 16 * 1024) / stage));
    cudaError_t e = launch_kernel(latent_query_kernel<CT>, dim3(s.heads * a.csplit + (a.fused ? 1 : 0), rows), dim3(LA_CONSUMERS), 0, st, chained, a);
    if (e != cudaSuccess) return e;
    const dim3 grid(latent_groups(s, f32) * a.nsplit, rows), block(LA_SCAN_THREADS);
    const size_t smem = (size_t)a.stages * stage;
    auto go = [&](auto k) { return launch_kernel(k, grid, block, smem, st, true, a); };
    if (f32) {
        const int pieces = (s.row + 255) / 256;
        e = pieces == 1 ? go(latent_scan_kernel<float, 1>) : pieces == 2 ? go(latent_scan_kernel<float, 2>) : pieces == 3 ? go(latent_scan_kernel<float, 3>) : go(latent_scan_kernel<float, 4>);
    } else {
        e = s.row <= 128 ? go(latent_scan_mma_kernel<1>) : s.row <= 256 ? go(latent_scan_mma_kernel<2>) : s.row <= 384 ? go(latent_scan_mma_kernel<3>)
            : s.row <= 640 ? go(latent_scan_mma_kernel<5>) : go(latent_scan_mma_kernel<8>);
    }
    if (e != cudaSuccess) return e;
    return launch_kernel(latent_output_kernel<OT>, dim3(s.heads * a.vsplit, rows), dim3(LA_CONSUMERS), 0, st, true, a, a.vsplit);
}

// ---- one position ------------------------------------------------------------------------------
static int32_t launch_dense_matvec(const StackSession* s, const StackMatrix& w, DmvParams& p, int* status, cudaStream_t st, int* nblocks = nullptr) {
    p.status = status;
    p.w = w.w; p.kp = w.kp; p.k = w.k; p.unit = w.pair;
    const int results = w.results(), grid = std::min(s->di.sms, results);
    p.per_lo = results / grid;
    p.per_rem = results % grid;
    p.nchunk = (w.k + 255) / 256;
    p.nseg = (p.nchunk + DMV_WARPS - 1) / DMV_WARPS;
    p.cs = (p.nchunk + p.nseg - 1) / p.nseg;
    p.nseg = (p.nchunk + p.cs - 1) / p.cs;
    p.gs = p.nseg == 1 ? DMV_WARPS / p.cs : 1;
    p.stages = dmv_choose_stages(p, (size_t)s->di.max_smem_optin - 2048);
    if (p.stages < 2) return fail(L2B_ERR_BAD_ARG, "input vector too long for shared memory");
    const size_t smem = (size_t)p.stages * DMV_STAGE + dmv_fixed_bytes(p);
    CU(launch_kernel(dense_matvec_kernel, dim3(grid), dim3(DMV_THREADS), smem, st, true, p));
    if (nblocks) *nblocks = grid;
    return L2B_OK;
}

int32_t stack_enqueue_token(StackSession* s, const int* token, const int* pos, float* logits, float* amax_val, int* amax_idx, int* status, cudaStream_t st,
                            int* nlaunch, int* nparts) {
    const StackModel* m = s->m;
    const StackConfig& c = m->cfg;
    int count = 0, cur = 0;
    CU(launch_kernel_args(scaled_embed_kernel, dim3(std::max(1, std::min(32, c.width / 256))), dim3(256), 0, st, false, 1, (const bf16*)m->embed.w, token, c.width, c.vocab,
                          c.embed_scale, s->x[0]));
    ++count;
    const float* side_w = nullptr;  // non-null: y1 awaits its norm and its place in the residual stream
    const float* step = nullptr;
    // the residual stream as input of a product, with whatever is pending applied on the way
    auto from_residual = [&](DmvParams& p, const StackNorm* norm) {
        memset(&p, 0, sizeof(p));
        p.x = s->x[cur];
        if (norm) p.norm = norm_params(m, *norm);
        p.upd.eps = c.eps;
        p.upd.step = step;
        if (side_w) {
            p.upd.y = s->y1;
            p.upd.side_w = side_w;
        }
        if (step || side_w) {
            cur ^= 1;
            p.x_out = s->x[cur];
        }
        step = side_w = nullptr;
    };
    auto from_vector = [&](DmvParams& p, const float* x) {
        memset(&p, 0, sizeof(p));
        p.x = x;
    };
    auto mv = [&](const StackMatrix& w, DmvParams& p, int kind, float* out, int* nb = nullptr) -> int32_t {
        p.epi.kind = kind;
        p.epi.y = out;
        p.epi.act = out;
        ++count;
        return launch_dense_matvec(s, w, p, status, st, nb);
    };
    DmvParams p;
    for (size_t r = 0; r < m->runs.size(); ++r) {
        const int l = m->runs[r].layer;
        const StackLayerW& w = m->layers[l];
        if (m->runs[r].pass >= 0) step = m->loop_step + (size_t)m->runs[r].pass * c.width;
        from_residual(p, &w.norm1);
        L2B_TRY(mv(w.qdg, p, DE_STORE, s->qdg1));
        {
            LatentAttnParams a = latent_params(s, (int)r, s->qdg1);
            a.pos = pos;
            a.out = s->att1;
            a.ldo = w.o.k;
            a.fused = 1;
            a.status = status;
            CU(m->f32 ? (launch_latent_attention<float, float>(a, 1, true, s->di, st)) : (launch_latent_attention<bf16, float>(a, 1, true, s->di, st)));
            count += 3;
        }
        from_vector(p, s->att1);
        L2B_TRY(mv(w.o, p, DE_RESIDUAL, s->x[cur]));
        if (w.gu.w) {
            from_residual(p, &w.norm2);
            L2B_TRY(mv(w.gu, p, DE_GEGLU, s->hid1));
            from_vector(p, s->hid1);
            L2B_TRY(mv(w.down, p, DE_RESIDUAL, s->x[cur]));
        }
        if (c.side_dim) {
            from_residual(p, nullptr);
            p.epi.etab = m->side_embed.w;
            p.epi.e_ld = m->side_embed.kp;
            p.epi.e_off = l * c.side_dim;
            p.epi.tokens = token;
            p.epi.vocab = c.vocab;
            L2B_TRY(mv(w.side_gate, p, DE_SIDE, s->hid1));
            from_vector(p, s->hid1);
            L2B_TRY(mv(w.side_proj, p, DE_STORE, s->y1));
            side_w = w.side_norm;
        }
    }
    from_residual(p, &m->final_norm);
    s->x_last = cur;
    p.amax_val = amax_val;
    p.amax_idx = amax_idx;
    L2B_TRY(mv(m->head, p, DE_LOGITS, logits, nparts));
    if (nlaunch) *nlaunch = count;
    return L2B_OK;
}

// ---- many positions ----------------------------------------------------------------------------
static int32_t bf16_map(CUtensorMap& map, const bf16* base, int64_t inner, int64_t rows, int64_t stride_elems, int box_rows) {
    EncodeTiledFn enc = encode_tiled_fn();
    if (!enc) return fail(L2B_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
    const cuuint64_t dims[2] = {(cuuint64_t)inner, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)stride_elems * 2};
    const cuuint32_t box[2] = {64u, (cuuint32_t)box_rows}, estr[2] = {1u, 1u};
    const CUresult r = enc(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<bf16*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                           CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(L2B_ERR_CUDA, "cuTensorMapEncodeTiled failed with code " + std::to_string((int)r));
    return L2B_OK;
}

// W x for n rows of x ([n][ldx], bf16 or f32 by the model's compute type), then `epi`.
static int32_t launch_gemm(const StackSession* s, const StackMatrix& w, const void* x, int ldx, int n, const DenseEpilogue& epi, int* status, cudaStream_t st) {
    const int rows = w.results();
    if (s->m->f32) {
        GemmF32Params g;
        memset(&g, 0, sizeof(g));
        g.w = w.w; g.w2 = w.second(); g.wstride = w.stride(); g.x = static_cast<const float*>(x); g.ldx = ldx;
        g.rows = rows; g.n_tok = n; g.k = w.k; g.epi = epi;
        const dim3 grid((rows + 63) / 64, (n + 63) / 64);
        if (w.pair == 2) f32_gemm_kernel<true><<<grid, 256, 0, st>>>(g);
        else f32_gemm_kernel<false><<<grid, 256, 0, st>>>(g);
        CU(cudaGetLastError());
        return L2B_OK;
    }
    // Token tile: as wide as the rows there are, narrower while the tiles do not fill the GPU.  Weight tiles per block: what takes fewer
    // rounds of the GPU, a round of two weight tiles costing about 1.55 rounds of one (2 when short products leave the epilogue exposed).
    auto up_div = [](long a, long b) { return (a + b - 1) / b; };
    const long sms = s->di.sms;
    int bn = n <= 32 ? 32 : n <= 64 ? 64 : 128;
    while (bn > 32 && up_div(rows, 128) * up_div(n, bn) < sms) bn /= 2;
    const double one = (double)up_div(up_div(rows, 128) * up_div(n, bn), sms), two = (w.k < 1024 ? 2.0 : 1.55) * (double)up_div(up_div(rows, 256) * up_div(n, bn), sms);
    const int na = w.pair == 2 || two < one ? 2 : 1;
    GemmDenseParams g;
    memset(&g, 0, sizeof(g));
    g.rows = rows; g.n_tok = n; g.k = w.k; g.epi = epi; g.status = status;
    g.row2 = w.pair == 2 || na == 1 ? 0 : 128;
    const int stage = bg_stage_bytes(bn, na);
    g.stages = std::min(BG_MAX_STAGES, (s->di.max_smem_optin - 4096) / stage);
    CUtensorMap ma, ma2, mb;
    L2B_TRY(bf16_map(ma, w.w, w.k, rows, (int64_t)w.stride(), 128));
    ma2 = ma;
    if (w.pair == 2) L2B_TRY(bf16_map(ma2, w.second(), w.k, rows, (int64_t)w.stride(), 128));
    L2B_TRY(bf16_map(mb, static_cast<const bf16*>(x), w.k, n, ldx, bn));
    const int per = w.pair == 2 ? 128 : 128 * na;
    g.mtiles = (rows + per - 1) / per;
    g.ntiles = (n + bn - 1) / bn;
    const dim3 grid((unsigned)std::min<long>((long)g.mtiles * g.ntiles, s->di.sms)), block(BG_THREADS);
    const size_t smem = (size_t)g.stages * stage + 1024;
    auto go = [&](auto k) { return launch_kernel_args(k, grid, block, smem, st, false, 1, g, ma, ma2, mb); };
    cudaError_t e;
    if (na == 1) e = bn == 32 ? go(bf16_gemm_kernel<32, 1>) : bn == 64 ? go(bf16_gemm_kernel<64, 1>) : go(bf16_gemm_kernel<128, 1>);
    else e = bn == 32 ? go(bf16_gemm_kernel<32, 2>) : bn == 64 ? go(bf16_gemm_kernel<64, 2>) : go(bf16_gemm_kernel<128, 2>);
    CU(e);
    return L2B_OK;
}

static int32_t launch_residual_rows(const StackSession* s, const RowsParams& r, int n, cudaStream_t st) {
    const bool wide = r.width % 4 == 0;
    if (s->m->f32) wide ? residual_rows_kernel<float, 4><<<n, 256, 0, st>>>(r) : residual_rows_kernel<float, 1><<<n, 256, 0, st>>>(r);
    else wide ? residual_rows_kernel<bf16, 4><<<n, 256, 0, st>>>(r) : residual_rows_kernel<bf16, 1><<<n, 256, 0, st>>>(r);
    CU(cudaGetLastError());
    return L2B_OK;
}

// Attention of n rows: latents and rotated keys into the cache, then the expanded form (long portions of one sequence, bf16) or the
// absorbed form.  Result (gated) in act2 [n][ldo].
static int32_t enqueue_latent_rows(StackSession* s, int run, int n, int pos0, const int* pos_list, int ldo, int* status, cudaStream_t st, long long* launches) {
    const StackModel* m = s->m;
    const StackLayerW& w = m->layers[m->runs[run].layer];
    const LatentShape& sh = w.shape;
    LatentAttnParams a = latent_params(s, run, s->qdg);
    a.pos0 = pos0;
    a.pos_list = pos_list;
    a.cache_stride = pos_list ? (size_t)s->info.seq_len * sh.row : 0;
    a.out = s->act2;
    a.ldo = ldo;
    if (m->f32) latent_rows_kernel<float><<<n, 128, 0, st>>>(a);
    else latent_rows_kernel<bf16><<<n, 128, 0, st>>>(a);
    CU(cudaGetLastError());
    ++*launches;
    const int kstages = prefill_kstages(sh, s->di);
    if (!s->pq || pos_list || n < EXPAND_MIN_ROWS || kstages == 0 || !(sh.scale2 > 0.f)) {
        a.status = status;
        for (int r = 0; r < n; r += ABSORB_ROWS) {
            const int k = std::min(ABSORB_ROWS, n - r);
            LatentAttnParams b = a;
            b.qdg += (size_t)r * a.ld;
            b.pos0 += r;
            if (pos_list) b.pos_list += r;
            b.cache = static_cast<uint8_t*>(a.cache) + (size_t)r * a.cache_stride * act_bytes(m);
            b.out = static_cast<uint8_t*>(a.out) + (size_t)r * ldo * act_bytes(m);
            CU(m->f32 ? (launch_latent_attention<float, float>(b, k, false, s->di, st)) : (launch_latent_attention<bf16, bf16>(b, k, false, s->di, st)));
            *launches += 3;
        }
        return L2B_OK;
    }
    const int npos = pos0 + n, dq = sh.dp + up(sh.rot, 16);
    const bf16* cache = static_cast<const bf16*>(a.cache);
    DenseEpilogue e;
    memset(&e, 0, sizeof(e));
    e.kind = DE_STORE_ACT;
    e.act = s->pk;
    e.ld = sh.heads * sh.dp;
    L2B_TRY(launch_gemm(s, w.uk, cache, sh.row, npos, e, status, st));
    e.kind = DE_STORE_T;
    e.act = s->pv;
    e.ld = s->pv_ld;
    L2B_TRY(launch_gemm(s, w.uv, cache, sh.row, npos, e, status, st));
    latent_queries_kernel<<<dim3(n, sh.heads), 128, 0, st>>>(s->qdg, a.ld, a.rope, pos0, sh, dq, s->pq);
    CU(cudaGetLastError());
    LatentPrefillParams f;
    memset(&f, 0, sizeof(f));
    f.n = n; f.pos0 = pos0; f.dim = sh.dim; f.rot = sh.rot; f.vdim = sh.vdim; f.dp = sh.dp; f.dq = dq; f.vp = sh.vp; f.kstages = kstages;
    f.scale2 = sh.scale2; f.sink = w.sink; f.gate = s->qdg + w.off_g; f.ld = a.ld; f.out = static_cast<bf16*>(s->act2); f.ldo = ldo; f.status = status;
    CUtensorMap mq, mk, mkr, mv;
    L2B_TRY(bf16_map(mq, s->pq, (int64_t)sh.heads * dq, n, (int64_t)sh.heads * dq, LP_TILE));
    L2B_TRY(bf16_map(mk, s->pk, (int64_t)sh.heads * sh.dp, npos, (int64_t)sh.heads * sh.dp, LP_TILE));
    L2B_TRY(bf16_map(mkr, cache + sh.rp, sh.rot, npos, sh.row, LP_TILE));
    L2B_TRY(bf16_map(mv, s->pv, npos, (int64_t)sh.heads * sh.vp, s->pv_ld, sh.vp));
    const size_t smem = (size_t)lp_smem_layout(sh.dim, sh.rot, sh.vp, kstages).total + 1024;
    CU(launch_kernel_args(latent_prefill_kernel, dim3((n + LP_TILE - 1) / LP_TILE, sh.heads), dim3(LP_THREADS), smem, st, false, 1, f, mq, mk, mkr, mv));
    *launches += 4;
    return L2B_OK;
}

int32_t stack_enqueue_rows(StackSession* s, const int* dev_tokens, int n, int pos0, const int* pos_list, int* status, cudaStream_t st, long long* launches) {
    const StackModel* m = s->m;
    const StackConfig& c = m->cfg;
    if (n < 1 || n > s->info.max_rows) return fail(L2B_ERR_BAD_ARG, "too many rows for one pass");
    long long count = 0;
    CU(launch_kernel_args(scaled_embed_kernel, dim3(std::max(1, std::min(16, c.width / 256)), n), dim3(256), 0, st, false, 1, (const bf16*)m->embed.w, dev_tokens, c.width,
                          c.vocab, c.embed_scale, s->xr));
    ++count;
    const int lda = up(c.width, 8);
    const float* side_w = nullptr;
    const float* step = nullptr;
    // the residual stream, with whatever is pending applied, normed into the operand buffer
    auto from_residual = [&](const StackNorm* norm, bool operand) -> int32_t {
        RowsParams r;
        memset(&r, 0, sizeof(r));
        r.x = s->xr;
        r.width = c.width;
        r.upd.eps = c.eps;
        r.upd.step = step;
        if (side_w) {
            r.upd.y = s->y;
            r.upd.side_w = side_w;
        }
        r.store_x = step || side_w;
        if (norm) r.norm = norm_params(m, *norm);
        if (operand) r.act = s->act;
        r.lda = lda;
        step = side_w = nullptr;
        ++count;
        return launch_residual_rows(s, r, n, st);
    };
    auto gemm = [&](const StackMatrix& w, const void* x, int kind, float* y, void* act, int ld) -> int32_t {
        DenseEpilogue e;
        memset(&e, 0, sizeof(e));
        e.kind = kind;
        e.y = y;
        e.act = act;
        e.ld = ld;
        ++count;
        return launch_gemm(s, w, x, up(w.k, 8), n, e, status, st);
    };
    for (size_t r = 0; r < m->runs.size(); ++r) {
        const int l = m->runs[r].layer;
        const StackLayerW& w = m->layers[l];
        if (m->runs[r].pass >= 0) step = m->loop_step + (size_t)m->runs[r].pass * c.width;
        L2B_TRY(from_residual(&w.norm1, true));
        L2B_TRY(gemm(w.qdg, s->act, DE_STORE, s->qdg, nullptr, w.qdg.rows));
        L2B_TRY(enqueue_latent_rows(s, (int)r, n, pos0, pos_list, up(w.o.k, 8), status, st, &count));
        L2B_TRY(gemm(w.o, s->act2, DE_RESIDUAL, s->xr, nullptr, c.width));
        if (w.gu.w) {
            L2B_TRY(from_residual(&w.norm2, true));
            L2B_TRY(gemm(w.gu, s->act, DE_GEGLU, nullptr, s->act2, up(w.down.k, 8)));
            L2B_TRY(gemm(w.down, s->act2, DE_RESIDUAL, s->xr, nullptr, c.width));
        }
        if (c.side_dim) {
            L2B_TRY(from_residual(nullptr, true));
            DenseEpilogue e;
            memset(&e, 0, sizeof(e));
            e.kind = DE_SIDE;
            e.act = s->act2;
            e.ld = up(c.side_dim, 8);
            e.etab = m->side_embed.w;
            e.e_ld = m->side_embed.kp;
            e.e_off = l * c.side_dim;
            e.tokens = dev_tokens;
            e.vocab = c.vocab;
            L2B_TRY(launch_gemm(s, w.side_gate, s->act, lda, n, e, status, st));
            ++count;
            L2B_TRY(gemm(w.side_proj, s->act2, DE_STORE, s->y, nullptr, c.width));
            side_w = w.side_norm;
        }
    }
    if (side_w) L2B_TRY(from_residual(nullptr, false));
    if (launches) *launches += count;
    return L2B_OK;
}

int32_t stack_enqueue_logits(StackSession* s, const int* dev_index, int n, float* logits, int* status, cudaStream_t st, long long* launches) {
    const StackModel* m = s->m;
    RowsParams r;
    memset(&r, 0, sizeof(r));
    r.x = s->xr;
    r.width = m->cfg.width;
    r.index = dev_index;
    r.norm = norm_params(m, m->final_norm);
    r.act = s->act;
    r.lda = up(m->cfg.width, 8);
    L2B_TRY(launch_residual_rows(s, r, n, st));
    DenseEpilogue e;
    memset(&e, 0, sizeof(e));
    e.kind = DE_STORE;
    e.y = logits;
    e.ld = m->cfg.vocab;
    L2B_TRY(launch_gemm(s, m->head, s->act, r.lda, n, e, status, st));
    if (launches) *launches += 2;
    return L2B_OK;
}
