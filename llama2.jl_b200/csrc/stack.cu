// Layer-stack models: weights, caches and the kernel sequences of one position and of many (see stack.h).
#include "stack.h"

#include <algorithm>
#include <cmath>
#include <map>
#include <memory>
#include <mutex>

#include "dense_gemm.cuh"
#include "dense_matvec.cuh"
#include "head_prefill.cuh"
#include "latent_attention.cuh"
#include "latent_prefill.cuh"
#include "mlstm_prefill.cuh"
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
    StackNorm norm1, norm2, norm1b, norm2b;
    StackMatrix in;               // what the mixer projects its input to, one below the other: latent attention q, down, gate;
    float* in_bias = nullptr;     // differential attention q, k, v, gate; mLSTM q, k, v, gate, input gate, forget gate
    StackMatrix o, gu, down, side_gate, side_proj;
    float* side_norm = nullptr;
    int off_k = 0, off_v = 0, off_g = 0, off_d = 0, off_i = 0, off_f = 0;  // first rows of the parts of `in`
    CacheScan scan = {};          // attention: its shape
    // latent attention
    StackMatrix uk, uv;
    float *dkv_norm = nullptr, *sink = nullptr;
    LatentShape latent;
    // differential attention
    float *q_norm = nullptr, *k_norm = nullptr;
    std::vector<float> lq1, lk1, lq2, lk2;
    HeadShape head;
    // mLSTM
    float* out_norm = nullptr;
    MlstmShape mlstm;
};

// Where a tensor of the file goes.
struct TensorSlot {
    std::vector<int64_t> shape;
    StackMatrix* mat = nullptr;    // matrix rows row0, row0 + row_step, ...; heads > 0: rows of a head are head_pad apart
    int row0 = 0, row_step = 1, head_rows = 0, head_pad = 0;
    float** vec = nullptr;         // f32 vector (any shape, flattened), vec_at values into its allocation
    size_t vec_at = 0;
    float* scalar = nullptr;       // host scalar
    std::vector<float>* host = nullptr;  // vector that stays on the host
    bool loaded = false;
};

}  // namespace

struct StackModel {
    StackConfig cfg;
    bool f32 = false;
    std::vector<StackLayerW> layers;
    std::vector<LayerRun> runs;
    StackMatrix embed, head, side_embed, positions;
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
static void add_vector(StackModel* m, const std::string& name, float** v, std::vector<int64_t> shape, size_t at = 0) {
    TensorSlot s;
    s.shape = std::move(shape);
    s.vec = v;
    s.vec_at = at;
    m->slots[name] = s;
}
static void add_host_vector(StackModel* m, const std::string& name, std::vector<float>& v, int n) {
    TensorSlot s;
    s.shape = {n};
    s.host = &v;
    m->slots[name] = s;
}
// A table that is read row by row (not padded).
static int32_t add_table(StackModel* m, const std::string& name, StackMatrix& t, int rows, int width) {
    t.rows = rows; t.k = t.kp = width;
    L2B_TRY(alloc_owned(m->owned, (void**)&t.w, (size_t)t.bytes()));
    add_matrix(m, name, t, rows);
    return L2B_OK;
}
static void add_norm(StackModel* m, const std::string& name, StackNorm& n) {
    add_vector(m, name, &n.w, {m->cfg.width});
    switch (m->cfg.norm) {
        case NormKind::DynamicTanh: {
            add_vector(m, name + ".b", &n.b, {m->cfg.width});
            TensorSlot s;
            s.scalar = &n.alpha;
            m->slots[name + ".alpha"] = s;
            break;
        }
        case NormKind::Rms: break;
    }
}
static NormParams norm_params(const StackModel* m, const StackNorm& n) {
    NormParams p = {NORM_NONE, 0.f, 0.f, nullptr, nullptr};
    switch (m->cfg.norm) {
        case NormKind::DynamicTanh: p = {NORM_DYNAMIC_TANH, n.alpha, 0.f, n.w, n.b}; break;
        case NormKind::Rms: p = {NORM_RMS, 0.f, m->cfg.eps, n.w, nullptr}; break;
    }
    return p;
}

static int32_t build_latent_attention(StackModel* m, StackLayerW& w, const MixerConfig& c, const std::string& p) {
    const int width = m->cfg.width;
    LatentShape& s = w.latent;
    s.heads = c.heads; s.dim = c.dim; s.rot = c.rot_dim; s.rdims = c.rot.dims; s.vdim = c.vdim; s.rank = c.kv_rank;
    s.rp = up(c.kv_rank, 8);
    s.row = s.rp + up(c.rot_dim, 8);
    s.dp = up(c.dim, 16);
    s.vp = up(c.vdim, 16);
    s.scale2 = (float)((double)c.scale * 1.4426950408889634);
    s.eps = m->cfg.eps;
    if (s.row > CS_MAX_ROW) return fail(L2B_ERR_UNSUPPORTED_TYPE, "latent attention takes kv_rank + rot_dim up to " + std::to_string(CS_MAX_ROW));
    w.scan.heads = w.scan.per_group = s.heads;
    w.scan.row = s.row;
    w.scan.vcols = s.rp;
    const int nq = c.heads * (c.dim + c.rot_dim), nd = c.kv_rank + c.rot_dim, ng = c.heads * c.vdim;
    w.off_d = nq;
    w.off_g = nq + nd;
    L2B_TRY(make_matrix(m, w.in, nq + nd + ng, width));
    add_matrix(m, p + "q", w.in, nq, 0);
    add_matrix(m, p + "dkv", w.in, nd, nq);
    add_matrix(m, p + "g", w.in, ng, nq + nd);
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

static int32_t build_differential_attention(StackModel* m, StackLayerW& w, const MixerConfig& c, const std::string& p) {
    const int width = m->cfg.width;
    HeadShape& s = w.head;
    s.heads = c.heads; s.kv_heads = c.kv_heads; s.dim = c.dim; s.vdim = c.vdim; s.rdims = c.rot.dims;
    s.dp = up(c.dim, 8);
    s.vp = up(c.vdim, 8);
    s.row = s.vp + 2 * s.dp;
    s.scale2 = (float)((double)c.scale * 1.4426950408889634);
    s.eps = m->cfg.eps;
    s.lambda = c.diff;  // (completed by stack_model_finalize)
    s.out_scale = 1.f - c.diff;
    if (s.row > CS_MAX_ROW) return fail(L2B_ERR_UNSUPPORTED_TYPE, "differential attention takes vdim + 2 dim up to " + std::to_string(CS_MAX_ROW));
    w.scan.heads = 2 * s.heads;
    w.scan.per_group = 2 * (s.heads / s.kv_heads);
    w.scan.row = s.row;
    w.scan.vcols = s.vp;
    w.scan.chunk = c.chunk;
    const bool own = c.kv_from < 0;
    const int nq = 2 * c.heads * c.dim, nk = own ? 2 * c.kv_heads * c.dim : 0, nv = own ? c.kv_heads * c.vdim : 0, ng = c.heads * c.vdim;
    w.off_k = nq;
    w.off_v = nq + nk;
    w.off_g = nq + nk + nv;
    L2B_TRY(make_matrix(m, w.in, nq + nk + nv + ng, width));
    L2B_TRY(alloc_owned(m->owned, (void**)&w.in_bias, (size_t)w.in.rows * 4));
    add_matrix(m, p + "q", w.in, nq, 0);
    add_vector(m, p + "q.b", &w.in_bias, {nq}, 0);
    add_vector(m, p + "q.norm", &w.q_norm, {c.dim});
    if (own) {
        add_matrix(m, p + "k", w.in, nk, w.off_k);
        add_vector(m, p + "k.b", &w.in_bias, {nk}, w.off_k);
        add_vector(m, p + "k.norm", &w.k_norm, {c.dim});
        add_matrix(m, p + "v", w.in, nv, w.off_v);
        add_vector(m, p + "v.b", &w.in_bias, {nv}, w.off_v);
    }
    add_matrix(m, p + "g", w.in, ng, w.off_g);
    L2B_TRY(make_matrix(m, w.o, width, ng));
    add_matrix(m, p + "o", w.o, width);
    add_host_vector(m, p + "lq1", w.lq1, c.dim);
    add_host_vector(m, p + "lk1", w.lk1, c.dim);
    add_host_vector(m, p + "lq2", w.lq2, c.dim);
    add_host_vector(m, p + "lk2", w.lk2, c.dim);
    return L2B_OK;
}

static int32_t build_mlstm(StackModel* m, StackLayerW& w, const MixerConfig& c, const std::string& p) {
    const int width = m->cfg.width;
    MlstmShape& s = w.mlstm;
    s.heads = c.heads; s.dim = c.dim; s.vdim = c.vdim;
    s.cap = c.gate_cap;
    s.qscale = (float)(1.0 / std::sqrt((double)c.dim));
    s.eps = m->cfg.eps;
    for (s.cpl = 1; s.cpl < ML_MAX_COLS && 32 * s.cpl * ML_MAX_CLUSTER < c.vdim;) s.cpl *= 2;
    for (s.cl = 1; 32 * s.cpl * s.cl < c.vdim;) s.cl *= 2;
    if (s.cl > ML_MAX_CLUSTER || c.dim > ML_MAX_DIM)
        return fail(L2B_ERR_UNSUPPORTED_TYPE, "mLSTM takes dim up to " + std::to_string(ML_MAX_DIM) + " and vdim up to " + std::to_string(32 * ML_MAX_COLS * ML_MAX_CLUSTER));
    const int nk = c.heads * c.dim, nv = c.heads * c.vdim;
    w.off_k = nk;
    w.off_v = 2 * nk;
    w.off_g = w.off_v + nv;
    w.off_i = w.off_g + nv;
    w.off_f = w.off_i + c.heads;
    L2B_TRY(make_matrix(m, w.in, w.off_f + c.heads, width));
    L2B_TRY(alloc_owned(m->owned, (void**)&w.in_bias, (size_t)w.in.rows * 4));
    add_matrix(m, p + "q", w.in, nk, 0);
    add_matrix(m, p + "k", w.in, nk, w.off_k);
    add_matrix(m, p + "v", w.in, nv, w.off_v);
    add_matrix(m, p + "g", w.in, nv, w.off_g);
    add_matrix(m, p + "i", w.in, c.heads, w.off_i);
    add_vector(m, p + "i.b", &w.in_bias, {c.heads}, w.off_i);
    add_matrix(m, p + "f", w.in, c.heads, w.off_f);
    add_vector(m, p + "f.b", &w.in_bias, {c.heads}, w.off_f);
    add_vector(m, p + "norm", &w.out_norm, {nv});
    L2B_TRY(make_matrix(m, w.o, width, nv));
    add_matrix(m, p + "o", w.o, width);
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
    L2B_TRY(add_table(m.get(), "embed", m->embed, c.vocab, c.width));
    if (c.max_positions) L2B_TRY(add_table(m.get(), "pos", m->positions, c.max_positions, c.width));
    add_norm(m.get(), "final.norm", m->final_norm);
    if (c.has_loop()) add_vector(m.get(), "loop.step", &m->loop_step, {c.loop_times, c.width});
    if (c.side_dim) L2B_TRY(add_table(m.get(), "side.embed", m->side_embed, c.vocab, c.side_dim * (int)c.layers.size()));
    for (size_t i = 0; i < c.layers.size(); ++i) {
        const StackLayerConfig& l = c.layers[i];
        StackLayerW& w = m->layers[i];
        const std::string p = "l" + std::to_string(i) + ".";
        add_norm(m.get(), p + "norm1", w.norm1);
        if (c.post_norm) add_norm(m.get(), p + "norm1b", w.norm1b);
        switch (l.mix.kind) {
            case MixerKind::LatentAttention: L2B_TRY(build_latent_attention(m.get(), w, l.mix, p + "mix.")); break;
            case MixerKind::DifferentialAttention: L2B_TRY(build_differential_attention(m.get(), w, l.mix, p + "mix.")); break;
            case MixerKind::Mlstm: L2B_TRY(build_mlstm(m.get(), w, l.mix, p + "mix.")); break;
        }
        switch (l.mlp) {
            case MlpKind::None: break;
            case MlpKind::GatedGeluTanh:
            case MlpKind::GatedSilu:
                add_norm(m.get(), p + "norm2", w.norm2);
                if (c.post_norm) add_norm(m.get(), p + "norm2b", w.norm2b);
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
        else if (s.host) *s.host = std::move(v);
        else {
            if (!*s.vec) L2B_TRY(alloc_owned(m->owned, (void**)s.vec, (size_t)count * 4));
            CU(cudaMemcpy(*s.vec + s.vec_at, v.data(), (size_t)count * 4, cudaMemcpyHostToDevice));
        }
    }
    s.loaded = true;
    return L2B_OK;
}

int32_t stack_model_finalize(StackModel* m) {
    for (const auto& s : m->slots)
        if (!s.second.loaded) return fail(L2B_ERR_STATE, "tensor " + s.first + " is missing");
    for (size_t i = 0; i < m->layers.size(); ++i) {
        StackLayerW& w = m->layers[i];
        if (m->cfg.layers[i].mix.kind != MixerKind::DifferentialAttention) continue;
        auto dot = [](const std::vector<float>& a, const std::vector<float>& b) {
            double v = 0.0;
            for (size_t k = 0; k < a.size(); ++k) v += (double)a[k] * b[k];
            return v;
        };
        w.head.lambda = (float)(std::exp(dot(w.lq1, w.lk1)) - std::exp(dot(w.lq2, w.lk2)) + (double)m->cfg.layers[i].mix.diff);
    }
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
        b += w.in.bytes() + w.uk.bytes() + w.uv.bytes() + w.o.bytes() + w.gu.bytes() + w.down.bytes() + w.side_gate.bytes() + w.side_proj.bytes();
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
    // per run, attention: rows of every position in bf16 or f32, [n_seq][groups][seq_len][row] (null: another run's are used)
    // mLSTM: the f32 states [n_seq][size]
    std::vector<void*> cache;
    std::vector<size_t> cache_bytes;
    std::vector<int> cache_run;                  // per run: the run whose cache it uses
    std::vector<const float2*> rope;             // per layer
    // one position
    float *x[2] = {nullptr, nullptr}, *in1 = nullptr, *att1 = nullptr, *hid1 = nullptr, *y1 = nullptr;
    int x_last = 0;
    // absorbed attention: queries and partial results of up to ABSORB_ROWS rows
    float *qp = nullptr, *part_acc = nullptr;
    float2* part_ml = nullptr;
    // many positions
    float *xr = nullptr, *in = nullptr, *y = nullptr;
    void *act = nullptr, *act2 = nullptr;        // operands of the products, [max_rows][k rounded up to 8]
    // prompt attention: queries; latent attention: expanded keys, transposed values; differential attention: gates
    bf16 *pq = nullptr, *pk = nullptr, *pv = nullptr, *pg = nullptr;
    int pv_ld = 0;
    float* aside = nullptr;                      // differential attention: the first map's result
    MlstmPrefillParams mp = {};                  // mLSTM in chunks: buffers (q null: there are none)
};

static size_t act_bytes(const StackModel* m) { return m->f32 ? 4 : 2; }

constexpr int ABSORB_ROWS = 64;  // rows per pass of the absorbed form of the attention (bounds its scratch)
// The tiled forms of the attention (latent_prefill.cuh, head_prefill.cuh) and the chunked form of the recurrence (mlstm_prefill.cuh)
// are for portions of at least this many rows.
constexpr int EXPAND_MIN_ROWS = 48, MLSTM_MIN_ROWS = 32;

// Blocks of query vectors and ranges of positions of the scan kernel: about one block per SM in a decode step, two for several rows.
static int scan_blocks(const CacheScan& c, bool f32) {
    const int per = f32 ? CS_WARPS : CS_MMA_HEADS;
    return c.heads / c.per_group * ((c.per_group + per - 1) / per);
}
static int scan_splits(const CacheScan& c, bool f32, int rows, const DeviceInfo& di) {
    return std::max(1, std::min(CS_MAX_SPLIT, (rows == 1 ? 1 : 2) * di.sms / (scan_blocks(c, f32) * rows)));
}

static int prefill_kstages(const LatentShape& s, const DeviceInfo& di) {
    if (s.vp > 256) return 0;
    for (int k = 2; k >= 1; --k)
        if (lp_smem_layout(s.dim, s.rot, s.vp, k).total + 1024 <= di.max_smem_optin - 1024) return k;
    return 0;
}

// Key stages of the tiled differential attention (0: the heads do not fit it), and whether two of its blocks share an SM.
static int head_prefill_kstages(const HeadShape& s, const DeviceInfo& di, bool* two = nullptr) {
    const int vn = up(s.vdim, 16), sm_bytes = di.max_smem_optin + 1024;                       // (1 KiB of an SM's shared memory goes to every block)
    auto bytes = [&](int k) { return hp_smem_layout(s.dim, vn, k).total + 1024 + 5 * 1024; };  // (static shared memory included)
    if (two) *two = false;
    if (vn > 256 || !(s.scale2 > 0.f)) return 0;
    if (vn <= HP_HALF_COLS && 2 * (bytes(1) + 1024) <= sm_bytes) {
        if (two) *two = true;
        return 2 * (bytes(2) + 1024) <= sm_bytes ? 2 : 1;
    }
    for (int k = 2; k >= 1; --k)
        if (bytes(k) <= di.max_smem_optin) return k;
    return 0;
}
// Ring slots of the chunk kernel (0: the heads do not fit the chunked form).
static int mlstm_prefill_stages(const MlstmShape& s, const DeviceInfo& di) {
    for (int k = MC_MAX_SLOTS; k >= 1; --k)
        if (up(s.dim, 16) <= MC_MAX_DP && mc_smem_layout(up(s.dim, 16), k).total + 1024 <= di.max_smem_optin - 10 * 1024) return k;
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
        set((const void*)dense_matvec_kernel<false, DMV_KINDS_GELU>); set((const void*)dense_matvec_kernel<true, DMV_KINDS_GELU>);
        set((const void*)dense_matvec_kernel<false, DMV_KINDS_SILU>); set((const void*)dense_matvec_kernel<true, DMV_KINDS_SILU>);
        set((const void*)latent_prefill_kernel);
        set((const void*)head_prefill_kernel);
        set((const void*)mlstm_state_kernel);
        set((const void*)mlstm_chunk_kernel);
        set((const void*)bf16_gemm_kernel<32, 1>); set((const void*)bf16_gemm_kernel<32, 2>);
        set((const void*)bf16_gemm_kernel<64, 1>); set((const void*)bf16_gemm_kernel<64, 2>);
        set((const void*)bf16_gemm_kernel<128, 1>); set((const void*)bf16_gemm_kernel<128, 2>);
        set((const void*)cache_scan_kernel<float, 1>); set((const void*)cache_scan_kernel<float, 2>);
        set((const void*)cache_scan_kernel<float, 3>); set((const void*)cache_scan_kernel<float, 4>);
        set((const void*)cache_scan_mma_kernel<1>); set((const void*)cache_scan_mma_kernel<2>); set((const void*)cache_scan_mma_kernel<3>);
        set((const void*)cache_scan_mma_kernel<5>); set((const void*)cache_scan_mma_kernel<8>);
    });
    if (g_stack_attr_err != cudaSuccess) return fail(L2B_ERR_CUDA, std::string("cudaFuncSetAttribute: ") + cudaGetErrorString(g_stack_attr_err));
    return L2B_OK;
}

static int32_t build_rope(StackSession* s) {
    std::map<std::pair<double, int>, const float2*> made;
    for (const StackLayerConfig& l : s->m->cfg.layers) {
        const RotaryConfig& r = l.mix.rot;
        if (r.dims == 0) {
            s->rope.push_back(nullptr);
            continue;
        }
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
    int max_in = 1, max_k = c.width, max_k2 = 1;
    size_t pq = 0, pk = 0, pv = 0, pg = 0, aside = 0, mh = 0, mk = 0, mv = 0, ms = 0;
    s->pv_ld = up(info.seq_len, 8);
    for (size_t i = 0; i < m->layers.size(); ++i) {
        const StackLayerW& w = m->layers[i];
        max_in = std::max(max_in, w.in.rows);
        max_k2 = std::max(std::max(max_k2, w.o.k), std::max(w.down.k, w.side_proj.k));
        if (w.head.heads && head_prefill_kstages(w.head, di)) {
            pq = std::max(pq, (size_t)2 * w.head.heads * up(w.head.dim, 16));
            aside = std::max(aside, (size_t)w.head.heads * w.head.vdim);
            pg = std::max(pg, (size_t)w.head.heads * w.head.vp);
        }
        if (w.mlstm.heads && mlstm_prefill_stages(w.mlstm, di)) {
            const MlstmShape& sh = w.mlstm;
            mh = std::max(mh, (size_t)sh.heads);
            mk = std::max(mk, (size_t)sh.heads * up(sh.dim, 16));
            mv = std::max(mv, (size_t)sh.heads * up(sh.vdim, 8));
            ms = std::max(ms, (size_t)sh.heads * up(sh.dim, 16) * up(sh.vdim, 8));
        }
        if (c.layers[i].mix.kind != MixerKind::LatentAttention) continue;
        pq = std::max(pq, (size_t)w.latent.heads * (w.latent.dp + up(w.latent.rot, 16)));
        pk = std::max(pk, (size_t)w.latent.heads * w.latent.dp);
        pv = std::max(pv, (size_t)w.latent.heads * w.latent.vp);
    }
    auto alloc = [&](auto*& p, size_t bytes) { return alloc_owned(s->owned, (void**)&p, bytes); };
    std::map<int, int> last_run;  // of a layer
    for (size_t r = 0; r < m->runs.size(); ++r) {
        const int l = m->runs[r].layer;
        const MixerConfig& mix = c.layers[l].mix;
        const StackLayerW& w = m->layers[l];
        last_run[l] = (int)r;
        size_t b = 0;
        if (mix.kind == MixerKind::Mlstm) b = (size_t)info.n_seq * w.mlstm.size() * 4;
        else if (mix.kv_from < 0) b = (size_t)info.n_seq * (w.scan.heads / w.scan.per_group) * info.seq_len * w.scan.row * act_bytes(m);
        void* p = nullptr;
        if (b) L2B_TRY(alloc_owned(s->owned, &p, b));
        s->cache.push_back(p);
        s->cache_bytes.push_back(b);
        s->cache_run.push_back(mix.kv_from < 0 ? (int)r : last_run[mix.kv_from]);
    }
    L2B_TRY(build_rope(s.get()));
    if (info.decode) {
        for (float*& x : s->x) L2B_TRY(alloc(x, (size_t)c.width * 4));
        L2B_TRY(alloc(s->in1, (size_t)max_in * 4));
        L2B_TRY(alloc(s->att1, (size_t)max_k2 * 4));
        L2B_TRY(alloc(s->hid1, (size_t)max_k2 * 4));
        L2B_TRY(alloc(s->y1, (size_t)c.width * 4));
    }
    size_t qp = 0, pml = 0, pacc = 0;
    for (const StackLayerW& w : m->layers) {
        if (!w.scan.heads) continue;
        for (int rows = 1; rows <= std::max(1, std::min(ABSORB_ROWS, info.max_rows)); ++rows) {
            const size_t pairs = (size_t)w.scan.heads * rows, slots = pairs * scan_splits(w.scan, m->f32, rows, di);
            qp = std::max(qp, pairs * w.scan.row);
            pml = std::max(pml, slots);
            pacc = std::max(pacc, slots * w.scan.vcols);
        }
    }
    L2B_TRY(alloc(s->qp, std::max<size_t>(qp, 1) * 4));
    L2B_TRY(alloc(s->part_ml, std::max<size_t>(pml, 1) * sizeof(float2)));
    L2B_TRY(alloc(s->part_acc, std::max<size_t>(pacc, 1) * 4));
    const size_t T = (size_t)info.max_rows;
    L2B_TRY(alloc(s->xr, T * c.width * 4));
    L2B_TRY(alloc(s->in, T * max_in * 4));
    L2B_TRY(alloc(s->y, T * c.width * 4));
    L2B_TRY(alloc(s->act, T * up(max_k, 8) * act_bytes(m)));
    L2B_TRY(alloc(s->act2, T * up(max_k2, 8) * act_bytes(m)));
    if (!m->f32 && info.n_seq == 1 && info.max_rows >= EXPAND_MIN_ROWS && pq) {
        L2B_TRY(alloc(s->pq, T * pq * 2));
        if (pk) L2B_TRY(alloc(s->pk, (size_t)info.seq_len * pk * 2));
        if (pv) L2B_TRY(alloc(s->pv, pv * s->pv_ld * 2));
        if (aside) L2B_TRY(alloc(s->aside, (size_t)up((int)T, HP_TILE) * aside * 4));
        if (pg) L2B_TRY(alloc(s->pg, T * pg * 2));
    }
    const size_t nchunk = (T + MP_L - 1) / MP_L;
    if (!m->f32 && info.n_seq == 1 && info.max_rows >= MLSTM_MIN_ROWS && mh && nchunk <= MP_MAX_CHUNKS) {
        MlstmPrefillParams& p = s->mp;
        for (bf16** b : {&p.q, &p.k}) L2B_TRY(alloc(*b, T * mk * 2));
        for (bf16** b : {&p.v, &p.g}) L2B_TRY(alloc(*b, T * mv * 2));
        for (float** f : {&p.a, &p.mx, &p.w, &p.floor, &p.u}) L2B_TRY(alloc(*f, mh * nchunk * MP_L * 4));
        L2B_TRY(alloc(p.decay, mh * nchunk * 4));
        for (bf16** b : {&p.sh, &p.sl}) L2B_TRY(alloc(*b, nchunk * ms * 2));
        L2B_TRY(alloc(p.sn, nchunk * mk * 4));
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
    for (size_t i = 0; i < s->cache.size(); ++i)
        if (s->cache[i]) CU(cudaMemsetAsync(s->cache[i], 0, s->cache_bytes[i], st));
    return L2B_OK;
}
int stack_session_max_rows(const StackSession* s) { return s->info.max_rows; }
const float* stack_session_residual(const StackSession* s) { return s->x[s->x_last]; }

// ---- attention launches ------------------------------------------------------------------------
// The scan of a run with everything but the rows' positions.
static CacheScan scan_params(const StackSession* s, int run) {
    const StackLayerW& w = s->m->layers[s->m->runs[run].layer];
    CacheScan c = w.scan;
    c.group_stride = (size_t)s->info.seq_len * c.row;
    c.cache = s->cache[s->cache_run[run]];
    c.qp = s->qp; c.part_ml = s->part_ml; c.part_acc = s->part_acc;
    return c;
}
static void plan_scan(CacheScan& c, bool f32, int rows, const DeviceInfo& di) {
    c.nsplit = scan_splits(c, f32, rows, di);
    const int stage = f32 ? CS_STAGE_ROWS * c.row * 4 : cs_mma_stage_bytes(c.row);
    c.stages = std::max(1, std::min(CS_MAX_STAGES, (di.max_smem_optin - 16 * 1024) / stage));
}
static cudaError_t launch_scan(const CacheScan& c, bool f32, int rows, cudaStream_t st) {
    const dim3 grid(c.nsplit, scan_blocks(c, f32), rows), block(CS_SCAN_THREADS);
    const size_t smem = (size_t)c.stages * (f32 ? CS_STAGE_ROWS * c.row * 4 : cs_mma_stage_bytes(c.row));
    auto go = [&](auto k) { return launch_kernel(k, grid, block, smem, st, true, c); };
    if (f32) {
        const int pieces = (c.row + 255) / 256;
        return pieces == 1 ? go(cache_scan_kernel<float, 1>) : pieces == 2 ? go(cache_scan_kernel<float, 2>) : pieces == 3 ? go(cache_scan_kernel<float, 3>) : go(cache_scan_kernel<float, 4>);
    }
    return c.row <= 128 ? go(cache_scan_mma_kernel<1>) : c.row <= 256 ? go(cache_scan_mma_kernel<2>) : c.row <= 384 ? go(cache_scan_mma_kernel<3>)
           : c.row <= 640 ? go(cache_scan_mma_kernel<5>) : go(cache_scan_mma_kernel<8>);
}

static LatentAttnParams latent_params(const StackSession* s, int run, const float* in) {
    const int l = s->m->runs[run].layer;
    const StackLayerW& w = s->m->layers[l];
    LatentAttnParams a;
    memset(&a, 0, sizeof(a));
    a.s = w.latent;
    a.c = scan_params(s, run);
    a.qdg = in; a.ld = w.in.rows; a.off_d = w.off_d; a.off_g = w.off_g;
    a.uk = w.uk.w; a.uv = w.uv.w; a.sink = w.sink; a.dnorm = w.dkv_norm; a.rope = s->rope[l];
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
    plan_scan(a.c, f32, rows, di);
    cudaError_t e = launch_kernel(latent_query_kernel<CT>, dim3(s.heads * a.csplit + (a.c.fused ? 1 : 0), rows), dim3(LA_CONSUMERS), 0, st, chained, a);
    if (e != cudaSuccess) return e;
    e = launch_scan(a.c, f32, rows, st);
    if (e != cudaSuccess) return e;
    return launch_kernel(latent_output_kernel<OT>, dim3(s.heads * a.vsplit, rows), dim3(LA_CONSUMERS), 0, st, true, a, a.vsplit);
}

static HeadAttnParams head_params(const StackSession* s, int run, const float* in) {
    const int l = s->m->runs[run].layer;
    const StackLayerW& w = s->m->layers[l];
    HeadAttnParams a;
    memset(&a, 0, sizeof(a));
    a.s = w.head;
    a.c = scan_params(s, run);
    a.in = in; a.ld = w.in.rows; a.off_k = w.off_k; a.off_v = w.off_v; a.off_g = w.off_g;
    a.own_kv = s->cache_run[run] == run;
    a.qnorm = w.q_norm; a.knorm = w.k_norm; a.rope = s->rope[l];
    return a;
}
template <typename CT>
static cudaError_t launch_head_rows(const HeadAttnParams& a, int rows, bool chained, cudaStream_t st) {
    const int items = 2 * a.s.heads + (a.own_kv ? 3 * a.s.kv_heads : 0) + (a.pq ? a.s.heads : 0);
    return launch_kernel(head_rows_kernel<CT>, dim3((items + HA_WARPS - 1) / HA_WARPS, rows), dim3(HA_WARPS * 32), 0, st, chained, a);
}
// Differential attention of `rows` rows: query vectors and new cache rows, scan, output.
template <typename CT, typename OT>
static cudaError_t launch_head_attention(HeadAttnParams a, int rows, bool chained, const DeviceInfo& di, cudaStream_t st) {
    constexpr bool f32 = sizeof(CT) == 4;
    plan_scan(a.c, f32, rows, di);
    cudaError_t e = launch_head_rows<CT>(a, rows, chained, st);
    if (e != cudaSuccess) return e;
    e = launch_scan(a.c, f32, rows, st);
    if (e != cudaSuccess) return e;
    return launch_kernel(head_output_kernel<OT>, dim3(a.s.heads, rows), dim3(HA_WARPS * 32), 0, st, true, a);
}

// ---- mLSTM launches ----------------------------------------------------------------------------
static MlstmParams mlstm_params(const StackSession* s, int run, const float* in) {
    const StackLayerW& w = s->m->layers[s->m->runs[run].layer];
    MlstmParams a;
    memset(&a, 0, sizeof(a));
    a.s = w.mlstm;
    a.in = in; a.ld = w.in.rows; a.off_k = w.off_k; a.off_v = w.off_v; a.off_g = w.off_g; a.off_i = w.off_i; a.off_f = w.off_f;
    a.norm = w.out_norm;
    a.state = static_cast<float*>(s->cache[run]);
    a.tokens = 1;
    return a;
}
// `rows` sequences by one token each, or (rows = 1) a.tokens tokens of one sequence.
template <typename OT>
static cudaError_t launch_mlstm_step(const MlstmParams& a, int rows, bool chained, cudaStream_t st) {
    const dim3 grid(a.s.heads * a.s.cl, rows);
    auto go = [&](auto k) { return launch_kernel(k, grid, dim3(ML_THREADS), 0, st, chained, a, a.s.cl); };
    if (a.s.dim <= ML_WARPS * 16)
        return a.s.cpl == 1 ? go(mlstm_step_kernel<16, 1, OT>) : a.s.cpl == 2 ? go(mlstm_step_kernel<16, 2, OT>) : go(mlstm_step_kernel<16, 4, OT>);
    return a.s.cpl == 1 ? go(mlstm_step_kernel<32, 1, OT>) : a.s.cpl == 2 ? go(mlstm_step_kernel<32, 2, OT>) : go(mlstm_step_kernel<32, 4, OT>);
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
    const bool rms = p.norm.kind == NORM_RMS;
    if (!(DMV_KINDS_GELU >> p.epi.kind & 1) && !(DMV_KINDS_SILU >> p.epi.kind & 1)) return fail(L2B_ERR_BAD_ARG, "the matrix-vector kernel has no such epilogue");
    CU(launch_kernel(DMV_KINDS_GELU >> p.epi.kind & 1 ? (rms ? dense_matvec_kernel<true, DMV_KINDS_GELU> : dense_matvec_kernel<false, DMV_KINDS_GELU>)
                                                      : (rms ? dense_matvec_kernel<true, DMV_KINDS_SILU> : dense_matvec_kernel<false, DMV_KINDS_SILU>),
                     dim3(grid), dim3(DMV_THREADS), smem, st, true, p));
    if (nblocks) *nblocks = grid;
    return L2B_OK;
}

static EmbedParams embed_params(const StackModel* m, const int* tokens, float* x) {
    EmbedParams e;
    memset(&e, 0, sizeof(e));
    e.table = m->embed.w; e.tokens = tokens; e.width = m->cfg.width; e.vocab = m->cfg.vocab; e.scale = m->cfg.embed_scale;
    e.pos_table = m->positions.w; e.max_positions = m->cfg.max_positions;
    e.x = x;
    return e;
}
static int embed_blocks(int width) { return std::max(1, std::min(16, width % 8 == 0 ? (width + 2047) / 2048 : width / 256)); }
static int mlp_epilogue(MlpKind k) { return k == MlpKind::GatedSilu ? DE_SWIGLU : DE_GEGLU; }

int32_t stack_enqueue_token(StackSession* s, const int* token, const int* pos, float* logits, float* amax_val, int* amax_idx, int* status, cudaStream_t st,
                            int* nlaunch, int* nparts) {
    const StackModel* m = s->m;
    const StackConfig& c = m->cfg;
    int count = 0, cur = 0;
    EmbedParams ep = embed_params(m, token, s->x[0]);
    ep.pos = pos;
    CU(launch_kernel(embed_positions_kernel, dim3(std::max(1, std::min(32, c.width / 256)), 1), dim3(32), 0, st, false, ep));
    ++count;
    const float* add_w = nullptr;  // non-null: y1 awaits its norm (this is its weight) and its place in the residual stream
    const float* step = nullptr;
    // the residual stream as input of a product, with whatever is pending applied on the way
    auto from_residual = [&](DmvParams& p, const StackNorm* norm) {
        memset(&p, 0, sizeof(p));
        p.x = s->x[cur];
        if (norm) p.norm = norm_params(m, *norm);
        p.upd.eps = c.eps;
        p.upd.step = step;
        if (add_w) {
            p.upd.y = s->y1;
            p.upd.w = add_w;
        }
        if (step || add_w) {
            cur ^= 1;
            p.x_out = s->x[cur];
        }
        step = add_w = nullptr;
    };
    auto from_vector = [&](DmvParams& p, const float* x) {
        memset(&p, 0, sizeof(p));
        p.x = x;
    };
    auto mv_epi = [&](const StackMatrix& w, DmvParams& p, const DenseEpilogue& e, int* nb = nullptr) -> int32_t {
        p.epi = e;
        ++count;
        return launch_dense_matvec(s, w, p, status, st, nb);
    };
    auto mv = [&](const StackMatrix& w, DmvParams& p, int kind, float* out) -> int32_t { return mv_epi(w, p, dense_epilogue_of(kind, out, out, 0)); };
    // a sublayer's result: added to the residual stream, or kept for its norm
    auto result = [&](const StackMatrix& w, DmvParams& p, const StackNorm& post) -> int32_t {
        if (!c.post_norm) return mv(w, p, DE_RESIDUAL, s->x[cur]);
        add_w = post.w;
        return mv(w, p, DE_STORE, s->y1);
    };
    DmvParams p;
    for (size_t r = 0; r < m->runs.size(); ++r) {
        const int l = m->runs[r].layer;
        const StackLayerW& w = m->layers[l];
        if (m->runs[r].pass >= 0) step = m->loop_step + (size_t)m->runs[r].pass * c.width;
        from_residual(p, &w.norm1);
        L2B_TRY(mv_epi(w.in, p, w.in_bias ? affine_epilogue(DE_AFFINE, 1.f, w.in_bias, s->in1, 0) : dense_epilogue_of(DE_STORE, s->in1, nullptr, 0)));
        switch (c.layers[l].mix.kind) {
            case MixerKind::LatentAttention: {
                LatentAttnParams a = latent_params(s, (int)r, s->in1);
                a.c.pos = pos;
                a.c.fused = 1;
                a.c.status = status;
                a.out = s->att1;
                a.ldo = w.o.k;
                CU(m->f32 ? (launch_latent_attention<float, float>(a, 1, true, s->di, st)) : (launch_latent_attention<bf16, float>(a, 1, true, s->di, st)));
                count += 3;
                break;
            }
            case MixerKind::DifferentialAttention: {
                HeadAttnParams a = head_params(s, (int)r, s->in1);
                a.c.pos = pos;
                a.c.fused = 1;
                a.c.status = status;
                a.out = s->att1;
                a.ldo = w.o.k;
                CU(m->f32 ? (launch_head_attention<float, float>(a, 1, true, s->di, st)) : (launch_head_attention<bf16, float>(a, 1, true, s->di, st)));
                count += 3;
                break;
            }
            case MixerKind::Mlstm: {
                MlstmParams a = mlstm_params(s, (int)r, s->in1);
                a.pos = pos;
                a.out = s->att1;
                a.ldo = w.o.k;
                CU(launch_mlstm_step<float>(a, 1, true, st));
                ++count;
                break;
            }
        }
        from_vector(p, s->att1);
        L2B_TRY(result(w.o, p, w.norm1b));
        if (w.gu.w) {
            from_residual(p, &w.norm2);
            L2B_TRY(mv(w.gu, p, mlp_epilogue(c.layers[l].mlp), s->hid1));
            from_vector(p, s->hid1);
            L2B_TRY(result(w.down, p, w.norm2b));
        }
        if (c.side_dim) {
            from_residual(p, nullptr);
            DenseEpilogue e = dense_epilogue_of(DE_SIDE, nullptr, s->hid1, 0);
            e.etab = m->side_embed.w;
            e.e_ld = m->side_embed.kp;
            e.e_off = l * c.side_dim;
            e.tokens = token;
            e.vocab = c.vocab;
            L2B_TRY(mv_epi(w.side_gate, p, e));
            from_vector(p, s->hid1);
            L2B_TRY(mv(w.side_proj, p, DE_STORE, s->y1));
            add_w = w.side_norm;
        }
    }
    from_residual(p, &m->final_norm);
    s->x_last = cur;
    p.amax_val = amax_val;
    p.amax_idx = amax_idx;
    L2B_TRY(mv_epi(m->head, p, c.logit_scale == 1.f ? dense_epilogue_of(DE_LOGITS, logits, nullptr, 0) : affine_epilogue(DE_AFFINE_LOGITS, c.logit_scale, nullptr, logits, 0), nparts));
    if (nlaunch) *nlaunch = count;
    return L2B_OK;
}

// ---- many positions ----------------------------------------------------------------------------
// A tile of 64 values x box_rows rows; depth > 1: of one of `depth` matrices (the tile does not reach into the next one).
static int32_t bf16_map(CUtensorMap& map, const bf16* base, int64_t inner, int64_t rows, int64_t stride_elems, int box_rows, int64_t depth = 1, int64_t depth_stride = 0) {
    EncodeTiledFn enc = encode_tiled_fn();
    if (!enc) return fail(L2B_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
    const int rank = depth_stride ? 3 : 2;
    const cuuint64_t dims[3] = {(cuuint64_t)inner, (cuuint64_t)rows, (cuuint64_t)depth}, strides[2] = {(cuuint64_t)stride_elems * 2, (cuuint64_t)depth_stride * 2};
    const cuuint32_t box[3] = {64u, (cuuint32_t)box_rows, 1u}, estr[3] = {1u, 1u, 1u};
    const CUresult r = enc(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<bf16*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
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

// A pass over rows in parts of at most ABSORB_ROWS: go(parameters of the part, its rows).
template <class P, class Go>
static int32_t rows_in_parts(const StackSession* s, const P& a, int n, const Go& go) {
    for (int r = 0; r < n; r += ABSORB_ROWS) {
        P b = a;
        b.c.pos0 += r;
        if (b.c.pos_list) b.c.pos_list += r;
        b.c.cache = static_cast<uint8_t*>(a.c.cache) + (size_t)r * a.c.cache_stride * act_bytes(s->m);
        b.out = static_cast<uint8_t*>(a.out) + (size_t)r * a.ldo * act_bytes(s->m);
        CU(go(b, r, std::min(ABSORB_ROWS, n - r)));
    }
    return L2B_OK;
}

// Latent attention of n rows: latents and rotated keys into the cache, then the expanded form (long portions of one sequence, bf16) or
// the absorbed form.  Result (gated) in act2 [n][ldo].
static int32_t enqueue_latent_rows(StackSession* s, int run, int n, int pos0, const int* pos_list, int ldo, int* status, cudaStream_t st, long long* launches) {
    const StackModel* m = s->m;
    const StackLayerW& w = m->layers[m->runs[run].layer];
    const LatentShape& sh = w.latent;
    LatentAttnParams a = latent_params(s, run, s->in);
    a.c.pos0 = pos0;
    a.c.pos_list = pos_list;
    a.c.cache_stride = pos_list ? (size_t)s->info.seq_len * sh.row : 0;
    a.c.status = status;
    a.out = s->act2;
    a.ldo = ldo;
    if (m->f32) latent_rows_kernel<float><<<n, 128, 0, st>>>(a);
    else latent_rows_kernel<bf16><<<n, 128, 0, st>>>(a);
    CU(cudaGetLastError());
    ++*launches;
    const int kstages = prefill_kstages(sh, s->di);
    if (!s->pq || pos_list || n < EXPAND_MIN_ROWS || kstages == 0 || !(sh.scale2 > 0.f))
        return rows_in_parts(s, a, n, [&](LatentAttnParams& b, int r, int k) {
            b.qdg += (size_t)r * a.ld;
            *launches += 3;
            return m->f32 ? (launch_latent_attention<float, float>(b, k, false, s->di, st)) : (launch_latent_attention<bf16, bf16>(b, k, false, s->di, st));
        });
    const int npos = pos0 + n, dq = sh.dp + up(sh.rot, 16);
    const bf16* cache = static_cast<const bf16*>(a.c.cache);
    L2B_TRY(launch_gemm(s, w.uk, cache, sh.row, npos, dense_epilogue_of(DE_STORE_ACT, nullptr, s->pk, sh.heads * sh.dp), status, st));
    L2B_TRY(launch_gemm(s, w.uv, cache, sh.row, npos, dense_epilogue_of(DE_STORE_T, nullptr, s->pv, s->pv_ld), status, st));
    latent_queries_kernel<<<dim3(n, sh.heads), 128, 0, st>>>(s->in, a.ld, a.rope, pos0, sh, dq, s->pq);
    CU(cudaGetLastError());
    LatentPrefillParams f;
    memset(&f, 0, sizeof(f));
    f.n = n; f.pos0 = pos0; f.dim = sh.dim; f.rot = sh.rot; f.vdim = sh.vdim; f.dp = sh.dp; f.dq = dq; f.vp = sh.vp; f.kstages = kstages;
    f.scale2 = sh.scale2; f.sink = w.sink; f.gate = s->in + w.off_g; f.ld = a.ld; f.out = static_cast<bf16*>(s->act2); f.ldo = ldo; f.status = status;
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

// Differential attention of n rows: the tiled form (long portions of one sequence, bf16), or the scan over rows.  Result (gated) in
// act2 [n][ldo].
static int32_t enqueue_head_rows(StackSession* s, int run, int n, int pos0, const int* pos_list, int ldo, int* status, cudaStream_t st, long long* launches) {
    const StackModel* m = s->m;
    HeadAttnParams a = head_params(s, run, s->in);
    a.c.pos0 = pos0;
    a.c.pos_list = pos_list;
    a.c.cache_stride = pos_list ? (size_t)a.s.kv_heads * a.c.group_stride : 0;
    a.c.status = status;
    a.out = s->act2;
    a.ldo = ldo;
    const HeadShape& sh = a.s;
    bool two;
    const int kstages = head_prefill_kstages(sh, s->di, &two), blocks = (n + HP_TILE - 1) / HP_TILE * sh.heads;
    if (!s->pq || pos_list || n < EXPAND_MIN_ROWS || kstages == 0)
        return rows_in_parts(s, a, n, [&](HeadAttnParams& b, int r, int k) {
            b.in += (size_t)r * a.ld;
            *launches += 3;
            return m->f32 ? (launch_head_attention<float, float>(b, k, false, s->di, st)) : (launch_head_attention<bf16, bf16>(b, k, false, s->di, st));
        });
    a.pq = s->pq;
    a.dq = up(sh.dim, 16);
    a.pg = s->pg;
    const int lanes = sh.rdims / 8, vectors = 2 * sh.heads + (a.own_kv ? 2 * sh.kv_heads : 0), per = lanes ? HA_WARPS * 32 / lanes : 1;
    if (sh.rdims % 8 == 0 && lanes && (lanes & (lanes - 1)) == 0 && lanes <= 32 && sh.dim % 16 == 0 && sh.vdim % 8 == 0)
        head_rows_quads_kernel<<<dim3((vectors + per - 1) / per, n), HA_WARPS * 32, 0, st>>>(a, lanes);
    else launch_head_rows<bf16>(a, n, false, st);
    CU(cudaGetLastError());
    HeadPrefillParams f;
    memset(&f, 0, sizeof(f));
    f.s = sh; f.n = n; f.pos0 = pos0; f.chunk = a.c.chunk; f.dq = a.dq; f.vn = up(sh.vdim, 16); f.kstages = kstages;
    f.paired = two && blocks > s->di.sms && blocks <= 2 * s->di.sms ? s->di.sms : 0;
    f.aside = s->aside; f.out = static_cast<bf16*>(s->act2); f.ldo = ldo; f.status = status;
    CUtensorMap mq, mkv, mg;
    L2B_TRY(bf16_map(mq, s->pq, (int64_t)2 * sh.heads * a.dq, n, (int64_t)2 * sh.heads * a.dq, HP_TILE));
    L2B_TRY(bf16_map(mkv, static_cast<const bf16*>(a.c.cache), sh.row, pos0 + n, sh.row, HP_TILE, sh.kv_heads, (int64_t)a.c.group_stride));
    L2B_TRY(bf16_map(mg, s->pg, (int64_t)sh.heads * sh.vp, n, (int64_t)sh.heads * sh.vp, HP_TILE));
    const size_t smem = (size_t)hp_smem_layout(sh.dim, f.vn, kstages).total + 1024;
    CU(launch_kernel_args(head_prefill_kernel, dim3(blocks), dim3(HP_THREADS), smem, st, false, 1, f, mq, mkv, mg));
    *launches += 2;
    return L2B_OK;
}

// mLSTM of n rows: n tokens of one sequence (in chunks, when there are many; bf16), or one of every sequence.  Result (gated) in act2
// [n][ldo].
static int32_t enqueue_mlstm_rows(StackSession* s, int run, int n, int pos0, const int* pos_list, int ldo, int* status, cudaStream_t st, long long* launches) {
    const StackModel* m = s->m;
    MlstmParams a = mlstm_params(s, run, s->in);
    a.pos0 = pos0;
    a.pos_list = pos_list;
    a.state_stride = pos_list ? a.s.size() : 0;
    a.tokens = pos_list ? 1 : n;
    a.out = s->act2;
    a.ldo = ldo;
    const MlstmShape& sh = a.s;
    const int stages = mlstm_prefill_stages(sh, s->di);
    if (s->mp.q && !pos_list && n >= MLSTM_MIN_ROWS && stages) {
        MlstmPrefillParams p = s->mp;
        p.m = a;
        p.n = n;
        p.nchunk = (n + MP_L - 1) / MP_L;
        p.dp = up(sh.dim, 16);
        p.vp = p.vs = up(sh.vdim, 8);
        p.sstages = stages;
        p.status = status;
        for (p.vt = 1; p.vt * MP_COLS < sh.vdim;) p.vt *= 2;
        CUtensorMap mq, mk, mv, msh, msl, mg;
        const int64_t nk = (int64_t)sh.heads * p.dp, nv = (int64_t)sh.heads * p.vp, rows = (int64_t)p.nchunk * sh.heads * p.dp;
        L2B_TRY(bf16_map(mq, p.q, nk, n, nk, MP_L));
        L2B_TRY(bf16_map(mk, p.k, nk, n, nk, MP_L));
        L2B_TRY(bf16_map(mv, p.v, nv, n, nv, MP_L));
        L2B_TRY(bf16_map(mg, p.g, nv, n, nv, MP_L));
        L2B_TRY(bf16_map(msh, p.sh, p.vs, rows, p.vs, MC_ROWS));
        L2B_TRY(bf16_map(msl, p.sl, p.vs, rows, p.vs, MC_ROWS));
        mlstm_operands_kernel<<<n, 256, 0, st>>>(p);
        CU(cudaGetLastError());
        mlstm_gates_kernel<<<sh.heads, 32 * p.nchunk, 0, st>>>(p);
        CU(cudaGetLastError());
        const dim3 sgrid((sh.vdim + MP_STATE_COLS - 1) / MP_STATE_COLS, (sh.dim + 127) / 128, sh.heads), cgrid(p.vt, p.nchunk, sh.heads);
        CU(launch_kernel_args(mlstm_state_kernel, sgrid, dim3(MP_THREADS), (size_t)MsSmem::total + 1024, st, false, 1, p, mk));
        CU(launch_kernel_args(mlstm_chunk_kernel, cgrid, dim3(MP_THREADS), (size_t)mc_smem_layout(p.dp, stages).total + 1024, st, false, p.vt, p, mq, mk, mv, msh, msl, mg));
        *launches += 4;
        return L2B_OK;
    }
    const int rows = pos_list ? n : 1;
    CU(m->f32 ? launch_mlstm_step<float>(a, rows, false, st) : launch_mlstm_step<bf16>(a, rows, false, st));
    ++*launches;
    return L2B_OK;
}

int32_t stack_enqueue_rows(StackSession* s, const int* dev_tokens, int n, int pos0, const int* pos_list, int* status, cudaStream_t st, long long* launches) {
    const StackModel* m = s->m;
    const StackConfig& c = m->cfg;
    if (n < 1 || n > s->info.max_rows) return fail(L2B_ERR_BAD_ARG, "too many rows for one pass");
    long long count = 0;
    EmbedParams ep = embed_params(m, dev_tokens, s->xr);
    ep.pos0 = pos0;
    ep.pos_list = pos_list;
    CU(launch_kernel(embed_positions_kernel, dim3(embed_blocks(c.width), n), dim3(256), 0, st, false, ep));
    ++count;
    const int lda = up(c.width, 8);
    const float* add_w = nullptr;  // non-null: y awaits its norm (this is its weight) and its place in the residual stream
    const float* step = nullptr;
    // the residual stream, with whatever is pending applied, normed into the operand buffer
    auto from_residual = [&](const StackNorm* norm, bool operand) -> int32_t {
        RowsParams r;
        memset(&r, 0, sizeof(r));
        r.x = s->xr;
        r.width = c.width;
        r.upd.eps = c.eps;
        r.upd.step = step;
        if (add_w) {
            r.upd.y = s->y;
            r.upd.w = add_w;
        }
        r.store_x = step || add_w;
        if (norm) r.norm = norm_params(m, *norm);
        if (operand) r.act = s->act;
        r.lda = lda;
        step = add_w = nullptr;
        ++count;
        return launch_residual_rows(s, r, n, st);
    };
    auto gemm_epi = [&](const StackMatrix& w, const void* x, const DenseEpilogue& e) -> int32_t {
        ++count;
        return launch_gemm(s, w, x, up(w.k, 8), n, e, status, st);
    };
    auto gemm = [&](const StackMatrix& w, const void* x, int kind, float* y, void* act, int ld) -> int32_t { return gemm_epi(w, x, dense_epilogue_of(kind, y, act, ld)); };
    // a sublayer's result: added to the residual stream, or kept for its norm
    auto result = [&](const StackMatrix& w, const StackNorm& post) -> int32_t {
        if (!c.post_norm) return gemm(w, s->act2, DE_RESIDUAL, s->xr, nullptr, c.width);
        add_w = post.w;
        return gemm(w, s->act2, DE_STORE, s->y, nullptr, c.width);
    };
    for (size_t r = 0; r < m->runs.size(); ++r) {
        const int l = m->runs[r].layer;
        const StackLayerW& w = m->layers[l];
        if (m->runs[r].pass >= 0) step = m->loop_step + (size_t)m->runs[r].pass * c.width;
        L2B_TRY(from_residual(&w.norm1, true));
        L2B_TRY(gemm_epi(w.in, s->act, w.in_bias ? affine_epilogue(DE_AFFINE, 1.f, w.in_bias, s->in, w.in.rows) : dense_epilogue_of(DE_STORE, s->in, nullptr, w.in.rows)));
        switch (c.layers[l].mix.kind) {
            case MixerKind::LatentAttention: L2B_TRY(enqueue_latent_rows(s, (int)r, n, pos0, pos_list, up(w.o.k, 8), status, st, &count)); break;
            case MixerKind::DifferentialAttention: L2B_TRY(enqueue_head_rows(s, (int)r, n, pos0, pos_list, up(w.o.k, 8), status, st, &count)); break;
            case MixerKind::Mlstm: L2B_TRY(enqueue_mlstm_rows(s, (int)r, n, pos0, pos_list, up(w.o.k, 8), status, st, &count)); break;
        }
        L2B_TRY(result(w.o, w.norm1b));
        if (w.gu.w) {
            L2B_TRY(from_residual(&w.norm2, true));
            L2B_TRY(gemm(w.gu, s->act, mlp_epilogue(c.layers[l].mlp), nullptr, s->act2, up(w.down.k, 8)));
            L2B_TRY(result(w.down, w.norm2b));
        }
        if (c.side_dim) {
            L2B_TRY(from_residual(nullptr, true));
            DenseEpilogue e = dense_epilogue_of(DE_SIDE, nullptr, s->act2, up(c.side_dim, 8));
            e.etab = m->side_embed.w;
            e.e_ld = m->side_embed.kp;
            e.e_off = l * c.side_dim;
            e.tokens = dev_tokens;
            e.vocab = c.vocab;
            L2B_TRY(gemm_epi(w.side_gate, s->act, e));
            L2B_TRY(gemm(w.side_proj, s->act2, DE_STORE, s->y, nullptr, c.width));
            add_w = w.side_norm;
        }
    }
    if (add_w) L2B_TRY(from_residual(nullptr, false));
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
    const DenseEpilogue e = m->cfg.logit_scale == 1.f ? dense_epilogue_of(DE_STORE, logits, nullptr, m->cfg.vocab) : affine_epilogue(DE_AFFINE, m->cfg.logit_scale, nullptr, logits, m->cfg.vocab);
    L2B_TRY(launch_gemm(s, m->head, s->act, r.lda, n, e, status, st));
    if (launches) *launches += 2;
    return L2B_OK;
}
