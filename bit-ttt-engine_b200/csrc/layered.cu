// Layer-list models: dense 16-bit projections, a mixer per layer (attention over an unquantised cache, latent attention,
// state-space, wkv and gated linear recurrences), dense or mixture feed-forwards, norms on the sublayers' outputs and, by
// design, on their inputs, looped runs of layers.  The model object, its step loop (graph per batch size), prefill loop, head,
// pick, positions and trace are those of model.cu; this file owns the layers.
#include <math.h>
#include <string.h>

#include <algorithm>
#include <new>
#include <vector>

#include "bt_model_impl.cuh"

namespace bt {

namespace {

template <typename T>
cudaError_t dev_alloc(T** p, size_t count) { return cudaMalloc(reinterpret_cast<void**>(p), (count ? count : 1) * sizeof(T)); }

constexpr int kTensorKinds = BT_LT_S_DOWN + 1;
static_assert(kTensorKinds <= 64, "the set of tensors received is a 64-bit mask");
inline int pad8(int n) { return (n + 7) / 8 * 8; }

// Floats (tiles: columns) per row that the sublayers need on the way; the largest of any layer.
struct RowNeeds {
    int proj = 0, mix = 0, ff = 0, conv = 0, v = 0, q = 0;
    int a = 0, b = 0, c = 0;    // f32 rows inside a mixer
    int mt = 0, ft = 0, t1 = 0, t2 = 0;  // bf16 tiles: mixer output, feed-forward, inside a mixer
    int logits = 0, top = 0, experts = 0, e_ff = 0, e_ff_pad = 0;
    bool moe = false;
};

// What the sublayers of `rows` tokens write on the way.
struct RowBuffers {
    int rows = 0;
    float* proj = nullptr;     // a mixer's input projection
    float* mix = nullptr;      // attention output / gated recurrence output, f32 rows
    float* y = nullptr;        // a sublayer's output before its norm
    float* ff = nullptr;       // feed-forward activations, f32 rows
    float* conv = nullptr;     // recurrence: channels after convolution and silu
    float* v_first = nullptr;
    float* hn = nullptr;       // a sublayer's normed input, f32 rows
    float* cat = nullptr;      // loops: stream and embedding side by side (fused step: the embedding)
    float* a = nullptr;        // latent: absorbed queries; rglru: convolution outputs; wkv: low-rank decay inputs
    float* b = nullptr;        // latent: weighted latents; rglru: gates; wkv: decays
    float* c = nullptr;        // latent: rotated queries; wkv: mixed inputs, finished rows
    float* wkv_pre = nullptr;  // wkv: decays up to each block of tokens
    void* q = nullptr;         // prepared queries
    uint8_t* xt = nullptr;     // bf16 models: tiled activations (sublayer input, mixer output, feed-forward, inside a mixer)
    uint8_t* mt = nullptr;
    uint8_t* ft = nullptr;
    uint8_t* t1 = nullptr;
    uint8_t* t2 = nullptr;
    float* scratch = nullptr;  // partial sums of the tcgen05 product
    // mixture of experts
    float* logits = nullptr;
    int* choice = nullptr;     // chosen expert, place, destination per row; counts, starts, tiles
    float* wt = nullptr;
    uint8_t* xe = nullptr;     // inputs and activations grouped by expert: tiles or f32 rows
    uint8_t* fe = nullptr;
    float* ye = nullptr;
    int64_t grouped = 0;
    void release() {
        for (void* p : {(void*)proj, (void*)mix, (void*)y, (void*)ff, (void*)conv, (void*)v_first, (void*)hn, (void*)cat, (void*)a, (void*)b, (void*)c, (void*)wkv_pre, q,
                        (void*)xt, (void*)mt, (void*)ft, (void*)t1, (void*)t2, (void*)scratch, (void*)logits, (void*)choice, (void*)wt, (void*)xe, (void*)fe, (void*)ye})
            cudaFree(p);
        *this = RowBuffers();
    }
};

struct LayLayer {
    bt_layer_config c{};
    // in: q|k|v, z|x|B|C|dt, q|latent|gates, y|x, or r, k, v, gate as blocks; mid, mid2: products inside the mixer (latent:
    // keys' and values' matrices per head; rglru: gates; wkv: decay's low rank); expand: keys and values of all heads
    DenseLin in, o, up, down, mid, mid2, expand, router, e_up, e_down, s_up, s_down;
    float* vec[kTensorKinds] = {nullptr};  // the small tensors, f32 on the device
    float* in_bias = nullptr;
    float* mid_bias = nullptr;
    float vmix = 0.f;
    bool v_source = false, v_target = false;  // gives / takes the mixed-in values
    uint64_t set = 0;                          // tensors received
    std::vector<uint8_t> experts_set;          // per expert: gate, up, down
    int table = -1;                            // rotation table
    int inner() const {  // outputs of the mixer
        if (c.mixer == BT_MIX_RGLRU) return c.channels;
        return c.heads * (c.mixer == BT_MIX_WKV ? c.dim : c.vdim);
    }
    int channels() const { return c.mixer == BT_MIX_RGLRU ? c.channels : inner() + 2 * c.groups * c.state; }
    int state_pad() const { return ssm_state_pad(c.state); }
    int v_width() const { return c.kv_heads * c.vdim; }
    int64_t state_floats() const {  // per sequence
        switch (c.mixer) {
            case BT_MIX_SSM: return (int64_t)inner() * state_pad();
            case BT_MIX_WKV: return (int64_t)inner() * c.dim;
            case BT_MIX_RGLRU: return c.channels;
        }
        return 0;
    }
    int64_t ring_floats(int width) const {
        switch (c.mixer) {
            case BT_MIX_SSM: case BT_MIX_RGLRU: return (int64_t)c.conv_taps * channels();
            case BT_MIX_WKV: return 2ll * width;
        }
        return 0;
    }
    const DenseLin* const* lins(size_t* n) const {
        all[0] = &in; all[1] = &o; all[2] = &up; all[3] = &down; all[4] = &mid; all[5] = &mid2; all[6] = &expand; all[7] = &router;
        all[8] = &e_up; all[9] = &e_down; all[10] = &s_up; all[11] = &s_down;
        *n = 12;
        return all;
    }
    mutable const DenseLin* all[12];
};

// One run of a layer: its own cache or state.
struct LayRun {
    int layer = 0, pass = -1;  // pass: a loop's pass begins here
    bt_kv_cache* kv = nullptr;
    float* state = nullptr;
    float* ring = nullptr;
};
struct RotTable {
    double base;
    int dims;
    float* cos_t;
    float* sin_t;
};

}  // namespace

struct Layered {
    bt_layers_config c{};
    std::vector<LayLayer> layers;
    std::vector<LayRun> runs;
    std::vector<RotTable> tables;
    DenseLin loop_in;
    float* loop_step = nullptr;
    unsigned loop_set = 0;
    __nv_bfloat16* pos_table = nullptr;
    float* h2 = nullptr;  // second residual-stream buffer of the fused decode step
    RowBuffers dec, pf;
    bool f32 = false;
    RowNeeds need;
    int fused_rows = 0;
    __nv_bfloat16* kv16 = nullptr;  // prefill: keys and values expanded from latents
    size_t kv16_elems = 0;
    float* wkv_seg = nullptr;       // prefill: states of the segments of a wkv recurrence
    bool loops() const { return c.loop_times > 0; }
};

namespace {

bt_status alloc_lin(DenseLin& l, int n, int k, int blocks = 1) {
    l.n = n; l.k = k; l.n_pad = (n + 127) / 128 * 128; l.k_pad = dense_kpad(k); l.blocks = blocks;
    BT_CUDA_TRY(dev_alloc(&l.tiles, l.bytes()));
    BT_CUDA_TRY(cudaMemset(l.tiles, 0, l.bytes()));
    return BT_OK;
}

// elements a tensor of this layer must have (experts: one expert's); 0: the layer has no such tensor
int64_t tensor_elems(const Layered* L, const LayLayer& l, int kind) {
    const bt_layer_config& c = l.c;
    const int64_t W = L->c.width, H = c.heads, inner = l.inner(), C = c.channels;
    const bool att = c.mixer == BT_MIX_ATTENTION, ssm = c.mixer == BT_MIX_SSM, lat = c.mixer == BT_MIX_LATENT, wkv = c.mixer == BT_MIX_WKV,
               rg = c.mixer == BT_MIX_RGLRU, mlp = c.mlp != BT_MLP_NONE, dense = c.mlp == BT_MLP_DENSE_RELU2, moe = c.mlp == BT_MLP_MOE_SWIGLU;
    switch (kind) {
        case BT_LT_NORM1: return W;
        case BT_LT_NORM2: return mlp ? W : 0;
        case BT_LT_PRE1: return L->c.pre_norm ? W : 0;
        case BT_LT_PRE2: return L->c.pre_norm && mlp ? W : 0;
        case BT_LT_Q: return att ? H * c.dim * W : (lat ? H * (c.dim + c.rot_dim) * W : 0);
        case BT_LT_K: return att ? (int64_t)c.kv_heads * c.dim * W : 0;
        case BT_LT_V: return att ? (int64_t)c.kv_heads * c.vdim * W : 0;
        case BT_LT_O: return !ssm ? inner * W : 0;
        case BT_LT_Q_NORM: return att && c.qk_norm ? H * c.dim : 0;
        case BT_LT_K_NORM: return att && c.qk_norm ? (int64_t)c.kv_heads * c.dim : 0;
        case BT_LT_SINK: return att && c.sink ? H : 0;
        case BT_LT_VMIX: return att && c.v_mix ? 1 : 0;
        case BT_LT_SSM_IN: return ssm ? (int64_t)(inner + l.channels() + H) * W : 0;
        case BT_LT_SSM_CONV: return ssm ? (int64_t)l.channels() * c.conv_taps : 0;
        case BT_LT_SSM_CONV_B: return ssm ? l.channels() : 0;
        case BT_LT_SSM_DT_BIAS: case BT_LT_SSM_A_LOG: case BT_LT_SSM_D: return ssm ? H : 0;
        case BT_LT_SSM_NORM: return ssm ? inner : 0;
        case BT_LT_SSM_O: return ssm ? inner * W : 0;
        case BT_LT_MLP_UP: case BT_LT_MLP_DOWN: return dense ? (int64_t)c.ff * W : 0;
        case BT_LT_DKV: return lat ? (int64_t)(c.kv_rank + c.rot_dim) * W : 0;
        case BT_LT_DKV_NORM: return lat ? c.kv_rank : 0;
        case BT_LT_UK: return lat ? H * c.dim * c.kv_rank : 0;
        case BT_LT_UV: return lat ? inner * c.kv_rank : 0;
        case BT_LT_GATE: return lat && c.out_gate ? H * W : 0;
        case BT_LT_MU_R: case BT_LT_MU_K: case BT_LT_MU_V: case BT_LT_MU_G: case BT_LT_MU_W: return wkv ? W : 0;
        case BT_LT_WKV_R: case BT_LT_WKV_K: case BT_LT_WKV_V: case BT_LT_WKV_G: return wkv ? inner * W : 0;
        case BT_LT_WKV_W1: return wkv ? c.decay_rank * W : 0;
        case BT_LT_WKV_W2: return wkv ? inner * c.decay_rank : 0;
        case BT_LT_WKV_W0: case BT_LT_WKV_U: case BT_LT_WKV_NORM: return wkv ? inner : 0;
        case BT_LT_RG_Y: case BT_LT_RG_X: return rg ? C * W : 0;
        case BT_LT_RG_CONV: return rg ? C * c.conv_taps : 0;
        case BT_LT_RG_RA: case BT_LT_RG_RI: return rg ? C * (C / c.blocks) : 0;
        case BT_LT_RG_Y_B: case BT_LT_RG_X_B: case BT_LT_RG_CONV_B: case BT_LT_RG_RA_B: case BT_LT_RG_RI_B: case BT_LT_RG_LAM: return rg ? C : 0;
        case BT_LT_ROUTER: return moe ? c.experts * W : 0;
        case BT_LT_ROUTER_B: return moe ? c.experts : 0;
        case BT_LT_E_GATE: case BT_LT_E_UP: case BT_LT_E_DOWN: return moe ? c.ff * W : 0;
        case BT_LT_S_GATE: case BT_LT_S_UP: case BT_LT_S_DOWN: return moe && c.shared_ff ? c.shared_ff * W : 0;
    }
    return 0;
}
bool is_expert_kind(int kind) { return kind == BT_LT_E_GATE || kind == BT_LT_E_UP || kind == BT_LT_E_DOWN; }

bt_status upload_rows(const DenseLin& lin, const float* host, int rows, int row0, int row_step = 1, int block = 0) {
    const int step = (int)std::max<int64_t>(1, (16 << 20) / lin.k);
    float* tmp = nullptr;
    BT_CUDA_TRY(dev_alloc(&tmp, (size_t)std::min(step, rows) * lin.k));
    cudaError_t e = cudaSuccess;
    for (int r = 0; r < rows && e == cudaSuccess; r += step) {
        const int n = std::min(step, rows - r);
        e = cudaMemcpy(tmp, host + (size_t)r * lin.k, (size_t)n * lin.k * sizeof(float), cudaMemcpyHostToDevice);
        if (e == cudaSuccess) e = launch_dense_tile(tmp, n, lin.k, row0 + r * row_step, lin, 0, row_step, block);
        if (e == cudaSuccess) e = cudaDeviceSynchronize();
    }
    cudaFree(tmp);
    BT_CUDA_TRY(e);
    return BT_OK;
}

bt_status upload_vec(float** dst, const float* host, int64_t n, float add) {
    std::vector<float> v(host, host + n);
    if (add != 0.0f) for (float& x : v) x += add;
    if (!*dst) BT_CUDA_TRY(dev_alloc(dst, (size_t)n));
    BT_CUDA_TRY(cudaMemcpy(*dst, v.data(), (size_t)n * sizeof(float), cudaMemcpyHostToDevice));
    return BT_OK;
}

// wide: the buffers of the unfused paths (prefill, steps of many sequences) as well
bt_status alloc_rows(const bt_model* m, RowBuffers& r, int rows, bool wide) {
    const Layered* L = m->lay;
    const RowNeeds& q = L->need;
    r.release();
    const size_t n = (size_t)rows, mp = (size_t)dense_mpad(rows);
    const int W = L->c.width, kpw = dense_kpad(W);
    struct { float** p; size_t count; } floats[] = {
        {&r.proj, n * q.proj}, {&r.mix, n * q.mix}, {&r.y, n * W}, {&r.ff, n * q.ff}, {&r.v_first, n * q.v}, {&r.hn, n * W},
        {&r.cat, L->loops() ? n * 2 * kpw : 0}, {&r.a, n * q.a}, {&r.b, n * q.b}, {&r.logits, n * q.logits}};
    for (auto& f : floats) {
        BT_CUDA_TRY(dev_alloc(f.p, f.count));
        BT_CUDA_TRY(cudaMemset(*f.p, 0, std::max<size_t>(f.count, 1) * sizeof(float)));
    }
    if (wide) {
        BT_CUDA_TRY(dev_alloc(&r.conv, n * q.conv));
        BT_CUDA_TRY(dev_alloc(&r.c, n * q.c));
        BT_CUDA_TRY(cudaMalloc(&r.q, std::max<size_t>(16, n * q.q * sizeof(float))));
        if (!L->f32) {
            int64_t pre = 0;
            for (const LayLayer& l : L->layers)
                if (l.c.mixer == BT_MIX_WKV) pre = std::max(pre, wkv_prefix_floats(l.c.heads, l.c.dim, rows, L->c.max_batch));
            BT_CUDA_TRY(dev_alloc(&r.wkv_pre, (size_t)pre));
            size_t scratch = 0;
            for (const LayLayer& l : L->layers) {
                size_t count;
                const DenseLin* const* all = l.lins(&count);
                for (size_t i = 0; i < count; ++i)
                    if (all[i]->tiles) scratch = std::max(scratch, dense_tc_scratch(*all[i], std::min(rows, 128), m->sm_count));
            }
            if (L->loops()) scratch = std::max(scratch, dense_tc_scratch(L->loop_in, std::min(rows, 128), m->sm_count));
            BT_CUDA_TRY(dev_alloc(&r.scratch, scratch));
            struct { uint8_t** p; int k; } tiles[] = {{&r.xt, L->loops() ? 2 * kpw : W}, {&r.mt, q.mt}, {&r.ft, q.ft}, {&r.t1, q.t1}, {&r.t2, q.t2}};
            for (auto& t : tiles) {  // zeroed once: rows and columns of the padding stay finite
                const size_t bytes = mp * dense_kpad(std::max(t.k, 1)) * 2;
                BT_CUDA_TRY(dev_alloc(t.p, bytes));
                BT_CUDA_TRY(cudaMemset(*t.p, 0, bytes));
            }
        }
        if (q.moe) {
            r.grouped = 0;
            for (const LayLayer& l : L->layers)
                if (l.c.mlp == BT_MLP_MOE_SWIGLU) r.grouped = std::max(r.grouped, moe_grouped_rows(rows, l.c.top, l.c.experts));
            const size_t g = (size_t)r.grouped, es = L->f32 ? 4 : 2;
            const size_t xe = g * (L->f32 ? W : kpw) * es, fe = g * (L->f32 ? q.e_ff : q.e_ff_pad) * es;
            const size_t ints = n * 3 * q.top + 2 * (size_t)q.experts + (q.experts + 1) + 4 + 4 * (n * q.top / 64 + q.experts + 1);
            BT_CUDA_TRY(dev_alloc(&r.choice, ints));
            BT_CUDA_TRY(cudaMemset(r.choice, 0, ints * sizeof(int)));
            BT_CUDA_TRY(dev_alloc(&r.wt, n * q.top));
            BT_CUDA_TRY(dev_alloc(&r.xe, xe));
            BT_CUDA_TRY(cudaMemset(r.xe, 0, xe));
            BT_CUDA_TRY(dev_alloc(&r.fe, fe));
            BT_CUDA_TRY(cudaMemset(r.fe, 0, fe));
            BT_CUDA_TRY(dev_alloc(&r.ye, g * W));
        }
    }
    BT_CUDA_TRY(cudaDeviceSynchronize());
    r.rows = rows;
    return BT_OK;
}

DenseAttn attn_args(const bt_model* m, const LayLayer& l, const LayRun& run, const RowBuffers& r, int batch, int n) {
    const bt_layer_config& c = l.c;
    DenseAttn a;
    a.qkv = r.proj;
    a.ld = l.in.n;
    a.q_norm = l.vec[BT_LT_Q_NORM];
    a.k_norm = l.vec[BT_LT_K_NORM];
    a.eps = m->lay->c.norm_eps;
    a.temp_coef = c.q_temp_coef;
    a.temp_every = c.q_temp_every;
    a.temp_every_int = c.q_temp_every >= 1.0 && c.q_temp_every < 1e9 && c.q_temp_every == floor(c.q_temp_every) ? (int)c.q_temp_every : 0;
    a.v_lambda = l.vmix;
    a.v_first_in = l.v_target ? r.v_first : nullptr;
    a.v_first_out = l.v_source ? r.v_first : nullptr;
    a.scale = c.scale;
    a.softcap = c.softcap;
    a.sink = l.vec[BT_LT_SINK];
    a.kv = run.kv->dense;
    a.pos = m->pos;
    a.batch = batch; a.q_rows = n; a.heads = c.heads; a.n_kv = c.kv_heads; a.dk = c.dim; a.dv = c.vdim;
    a.sm_count = m->sm_count;
    a.q_buf = r.q;
    return a;
}
SsmArgs ssm_args(const bt_model* m, const LayLayer& l, const LayRun& run, const RowBuffers& r, int batch, int n) {
    const bt_layer_config& c = l.c;
    SsmArgs a;
    a.proj = r.proj;
    a.ld = l.in.n;
    a.conv_w = l.vec[BT_LT_SSM_CONV]; a.conv_b = l.vec[BT_LT_SSM_CONV_B];
    a.dt_bias = l.vec[BT_LT_SSM_DT_BIAS]; a.a_log = l.vec[BT_LT_SSM_A_LOG]; a.d = l.vec[BT_LT_SSM_D];
    a.heads = c.heads; a.vdim = c.vdim; a.state = c.state; a.groups = c.groups; a.taps = c.conv_taps;
    a.ring = run.ring; a.s = run.state; a.state_pad = l.state_pad();
    a.pos = m->pos;
    a.batch = batch; a.q_rows = n;
    a.conv_out = r.conv;
    a.y = r.mix;
    a.sm_count = m->sm_count;
    return a;
}

LatentAttn latent_args(const bt_model* m, const LayLayer& l, const LayRun& run, const RowBuffers& r, int batch, int n) {
    const Layered* L = m->lay;
    const bt_layer_config& c = l.c;
    LatentAttn a;
    a.proj = r.proj; a.ld = l.in.n;
    a.c_norm = l.vec[BT_LT_DKV_NORM]; a.eps = L->c.norm_eps; a.scale = c.scale; a.gate = c.out_gate != 0;
    if (l.table >= 0) { a.cos_t = L->tables[(size_t)l.table].cos_t; a.sin_t = L->tables[(size_t)l.table].sin_t; }
    a.heads = c.heads; a.dim = c.dim; a.rot = c.rot_dim; a.rot_dims = c.rot_dims; a.vdim = c.vdim; a.rank = c.kv_rank;
    a.kv = run.kv->latent;
    a.pos = m->pos; a.batch = batch; a.q_rows = n; a.sm_count = m->sm_count;
    a.q_abs = r.a;
    a.m_pad = dense_mpad((int64_t)batch * n);
    return a;
}
WkvArgs wkv_args(const bt_model* m, const LayLayer& l, const LayRun& run, const RowBuffers& r, int batch, int n) {
    const bt_layer_config& c = l.c;
    WkvArgs a;
    a.proj = r.proj; a.ld = 4ll * l.inner();
    a.u = l.vec[BT_LT_WKV_U]; a.norm = l.vec[BT_LT_WKV_NORM]; a.w0 = l.vec[BT_LT_WKV_W0]; a.eps = m->lay->c.norm_eps;
    a.heads = c.heads; a.dim = c.dim; a.s = run.state; a.pos = m->pos; a.batch = batch; a.q_rows = n;
    a.y = r.mix;
    a.low = r.a; a.rank = c.decay_rank;
    a.w = r.b; a.hn = r.hn; a.shift = run.ring; a.shift_slot = (int64_t)m->cfg.max_batch * m->lay->c.width; a.width = m->lay->c.width;
    a.sm_count = m->sm_count;
    a.split16 = !m->lay->f32;
    a.seg_s = m->lay->f32 ? nullptr : m->lay->wkv_seg;
    a.seg_w = r.wkv_pre;
    return a;
}
RgluArgs rglru_args(const bt_model* m, const LayLayer& l, const LayRun& run, const RowBuffers& r, int batch, int n) {
    const bt_layer_config& c = l.c;
    RgluArgs a;
    a.proj = r.proj; a.ld = l.in.n;
    a.conv_w = l.vec[BT_LT_RG_CONV]; a.conv_b = l.vec[BT_LT_RG_CONV_B];
    a.channels = c.channels; a.blocks = c.blocks; a.taps = c.conv_taps; a.ring = run.ring;
    a.lam = l.vec[BT_LT_RG_LAM]; a.state = run.state; a.pos = m->pos; a.batch = batch; a.q_rows = n;
    a.u = r.a; a.gates = r.b;
    a.u_tiles = m->lay->f32 ? nullptr : r.t1;
    a.m_pad = dense_mpad((int64_t)batch * n);
    return a;
}

cudaError_t trace_stream(const bt_model* m, int run, const float* h, int rows, cudaStream_t s) {
    if (!m->trace) return cudaSuccess;
    if (rows > m->trace_rows) return cudaErrorInvalidValue;
    const size_t W = (size_t)m->cfg.hidden_dim;
    return cudaMemcpyAsync(m->trace + (size_t)run * m->trace_rows * W, h, (size_t)rows * W * sizeof(float), cudaMemcpyDeviceToDevice, s);
}

// The launches of a pass by what they do; a pass can be asked for some of them only (measurement aid).
enum Part : int { PART_IN = 1, PART_CORE = 2, PART_O = 4, PART_UP = 8, PART_DOWN = 16, PART_ROWS = 32, PART_MID = 64, PART_ROUTE = 128, PART_LOOP = 256, PART_ALL = 511 };

// norm weight of a sublayer's input (null: it reads the stream as it is)
const float* input_norm(const Layered* L, const LayLayer& l, bool mlp) {
    return L->c.pre_norm ? l.vec[mlp ? BT_LT_PRE2 : BT_LT_PRE1] : nullptr;
}

// One decode step for a few sequences: three to five dependent launches per mixer, two or three per feed-forward.
// A sublayer's output norm, the residual sum and the next sublayer's input norm are the prologue of the next projection,
// which reads the old stream and the un-normed output and leaves the new stream in the other buffer.
bt_status step_fused(bt_model* m, int batch, cudaStream_t s, int parts = PART_ALL) {
    Layered* L = m->lay;
    RowBuffers& r = L->dec;
    const int W = L->c.width, sm = m->sm_count;
    const float eps = L->c.norm_eps;
    float* cur = m->h;
    float* other = L->h2;
    const float* pending = nullptr;  // norm weight of the sublayer whose output waits in r.y
    ActOut emb;
    if (L->loops()) { emb.rows = r.cat; emb.ld = W; }
    if (parts & PART_ROWS)
        BT_CUDA_TRY(launch_embed_pos(m->tokens, m->embed, L->pos_table, m->pos, batch, 1, W, m->cfg.vocab_size, L->c.max_positions, cur, ActOut(), s, true, emb));
    auto stream_in = [&](const float* next_w) {
        DenseIn in;
        in.ld = W; in.eps = eps; in.pos = m->pos;
        if (pending) {
            in.kind = DPRO_RESNORM; in.x = r.y; in.w = pending; in.h = cur; in.h_out = other; in.next_w = next_w;
            std::swap(cur, other);
            pending = nullptr;
        } else if (next_w) {
            in.kind = DPRO_GROUPNORM; in.x = cur; in.w = next_w;
        } else {
            in.x = cur;
        }
        return in;
    };
    auto product = [&](int part, const DenseLin& lin, const DenseIn& in, float* out, int64_t ld, int act, const float* bias = nullptr, int64_t out_block = 0) -> cudaError_t {
        if (!(parts & part)) return cudaSuccess;
        DenseSeg seg;
        seg.lin = &lin; seg.out = out; seg.ld = ld; seg.act = act; seg.bias = bias; seg.out_block = out_block;
        return launch_dense_stream_segs(&seg, 1, in, batch, sm, s, true);
    };
    RowArgs res;  // the residual sum on its own
    res.op = ROW_RESNORM; res.y = r.y; res.ld = W; res.eps = eps; res.rows = batch; res.k = W;
    for (size_t ri = 0; ri < L->runs.size(); ++ri) {
        LayRun& run = L->runs[ri];
        LayLayer& l = L->layers[(size_t)run.layer];
        const bt_layer_config& c = l.c;
        if (run.pass >= 0) {
            DenseIn in = stream_in(nullptr);
            in.kx = W; in.cat = r.cat;
            if (in.kind == DPRO_RESNORM) { in.h_out = nullptr; std::swap(cur, other); }  // the sum itself is not needed again
            BT_CUDA_TRY(product(PART_LOOP, L->loop_in, in, other, W, DACT_NONE, L->loop_step + (size_t)run.pass * W));
            std::swap(cur, other);
        }
        DenseIn in = stream_in(input_norm(L, l, false)), o;
        o.x = r.mix; o.ld = l.inner();
        if (c.mixer == BT_MIX_WKV) {
            in.shift = run.ring; in.shift_slot = (int64_t)m->cfg.max_batch * W;
            DenseLin part[4];
            DenseSeg seg[5];
            for (int i = 0; i < 4; ++i) {
                part[i] = l.in;
                part[i].blocks = 1;
                part[i].tiles += i * l.in.block_bytes();
                seg[i].lin = &part[i]; seg[i].out = r.proj + (size_t)i * l.inner(); seg[i].ld = 4 * l.inner(); seg[i].mu = l.vec[BT_LT_MU_R + i];
            }
            seg[4].lin = &l.mid; seg[4].out = r.a; seg[4].ld = c.decay_rank; seg[4].act = DACT_TANH; seg[4].mu = l.vec[BT_LT_MU_W];
            if (parts & PART_IN) BT_CUDA_TRY(launch_dense_stream_segs(seg, 5, in, batch, sm, s, true));
            WkvArgs a = wkv_args(m, l, run, r, batch, 1);
            a.w2_tiles = l.mid2.tiles; a.w2_pad = l.mid2.n_pad;
            if (parts & PART_CORE) BT_CUDA_TRY(launch_wkv_step(a, s, true));
        } else {
            BT_CUDA_TRY(product(PART_IN, l.in, in, r.proj, l.in.n, DACT_NONE, l.in_bias));
            if (c.mixer == BT_MIX_ATTENTION) {
                ActOut att;
                att.rows = r.mix; att.ld = l.inner();
                if (parts & PART_CORE) BT_CUDA_TRY(launch_attn_span(attn_args(m, l, run, r, batch, 1), false, att, s, true));
            } else if (c.mixer == BT_MIX_SSM) {
                if (parts & PART_CORE) BT_CUDA_TRY(launch_ssm_step(ssm_args(m, l, run, r, batch, 1), s, true));
                o.kind = DPRO_GROUPNORM; o.w = l.vec[BT_LT_SSM_NORM]; o.eps = eps; o.groups = c.norm_groups;
            } else if (c.mixer == BT_MIX_LATENT) {
                DenseIn q, v;
                q.x = r.proj; q.ld = l.in.n; q.x_block = c.dim + c.rot_dim;
                BT_CUDA_TRY(product(PART_MID, l.mid, q, r.a, (int64_t)c.heads * c.kv_rank, DACT_NONE, nullptr, c.kv_rank));
                ActOut lat;
                lat.rows = r.b; lat.ld = (int64_t)c.heads * c.kv_rank;
                if (parts & PART_CORE) BT_CUDA_TRY(launch_latent_span(latent_args(m, l, run, r, batch, 1), false, lat, s, true));
                v.x = r.b; v.ld = (int64_t)c.heads * c.kv_rank; v.x_block = c.kv_rank;
                BT_CUDA_TRY(product(PART_MID, l.mid2, v, r.mix, l.inner(), DACT_NONE, nullptr, c.vdim));
            } else {  // rglru: convolution in the prologue, recurrence in the epilogue of the gates' product
                DenseIn g;
                g.kind = DPRO_CONV; g.x = r.proj + c.channels; g.ld = l.in.n; g.x_block = l.mid.k;
                g.ring = run.ring; g.conv_w = l.vec[BT_LT_RG_CONV]; g.conv_b = l.vec[BT_LT_RG_CONV_B]; g.taps = c.conv_taps; g.channels = c.channels;
                g.pos = m->pos; g.rg.y = r.proj; g.rg.lam = l.vec[BT_LT_RG_LAM]; g.rg.state = run.state;
                BT_CUDA_TRY(product(PART_CORE, l.mid, g, r.mix, l.inner(), DACT_RGLRU, l.mid_bias, l.mid.k));
            }
        }
        BT_CUDA_TRY(product(PART_O, l.o, o, r.y, W, DACT_NONE));
        pending = l.vec[BT_LT_NORM1];
        if (c.mlp == BT_MLP_DENSE_RELU2) {
            BT_CUDA_TRY(product(PART_UP, l.up, stream_in(input_norm(L, l, true)), r.ff, c.ff, DACT_RELU2));
            DenseIn d;
            d.x = r.ff; d.ld = c.ff;
            BT_CUDA_TRY(product(PART_DOWN, l.down, d, r.y, W, DACT_NONE));
            pending = l.vec[BT_LT_NORM2];
        } else if (c.mlp == BT_MLP_MOE_SWIGLU) {
            // the router's logits and the shared expert's activations in one launch, then the chosen experts
            const int fp = dense_kpad(c.ff);
            DenseIn x = stream_in(input_norm(L, l, true));
            if (L->c.pre_norm) x.n_out = r.hn;
            MoeStep a;
            a.up = &l.e_up; a.down = &l.e_down; a.shared_down = c.shared_ff ? &l.s_down : nullptr;
            a.logits = r.logits; a.experts = c.experts; a.top = c.top; a.rows = batch; a.x = L->c.pre_norm ? r.hn : cur;
            a.ff = r.ff; a.ff_ld = (int64_t)c.top * fp + (c.shared_ff ? dense_kpad(c.shared_ff) : 0); a.y = r.y; a.sm_count = sm;
            DenseSeg seg[2];
            seg[0].lin = &l.router; seg[0].out = r.logits; seg[0].ld = c.experts; seg[0].bias = l.vec[BT_LT_ROUTER_B];
            if (c.shared_ff) { seg[1].lin = &l.s_up; seg[1].out = r.ff + (size_t)c.top * fp; seg[1].ld = a.ff_ld; seg[1].act = DACT_SWIGLU; }
            if (parts & PART_ROUTE) BT_CUDA_TRY(launch_dense_stream_segs(seg, c.shared_ff ? 2 : 1, x, batch, sm, s, true));
            if (parts & PART_UP) BT_CUDA_TRY(launch_moe_up(a, s, true));
            if (parts & PART_DOWN) BT_CUDA_TRY(launch_moe_down(a, s, true));
            pending = l.vec[BT_LT_NORM2];
        }
        if (m->trace) {  // the stream after the layer, into the trace only
            if (batch > m->trace_rows) return set_error(BT_ERR_NOMEM, "the trace buffer holds fewer rows than sequences");
            res.w = pending; res.h_in = cur; res.h_out = m->trace + ri * (size_t)m->trace_rows * W;
            BT_CUDA_TRY(launch_row_op(res, s, true));
        }
    }
    res.w = pending; res.h_in = cur; res.h_out = m->h;  // in place when the stream is there already
    if (parts & PART_ROWS) BT_CUDA_TRY(launch_row_op(res, s, true));
    return BT_OK;
}

// Room for the expanded keys and values of `seqs` sequences.
bt_status expand_room(Layered* L, size_t elems) {
    if (elems <= L->kv16_elems) return BT_OK;
    BT_CUDA_TRY(cudaDeviceSynchronize());
    cudaFree(L->kv16);
    L->kv16 = nullptr;
    L->kv16_elems = 0;
    BT_CUDA_TRY(dev_alloc(&L->kv16, elems));
    L->kv16_elems = elems;
    return BT_OK;
}
constexpr size_t kExpandElems = (size_t)512 << 20;  // a group of sequences is expanded at a time: 1 GB

// `n` new tokens for each of `batch` sequences, every stage its own kernel over all rows: tcgen05 products of bf16
// activations (f32 models: f32 products), attention by tiles of query positions.  The stream ends in h.
constexpr int kTileRowsMin = 16;  // new tokens per sequence from which the tile kernel pays
struct RowPass {
    bt_model* m;
    Layered* L;
    RowBuffers& r;
    float* h;
    int batch, n, M, past, parts;
    cudaStream_t s;
    int W, sm, kpw;
    float eps;
    bool f32;
    unsigned int* err;
    int64_t mp;

    RowPass(bt_model* model, RowBuffers& buffers, float* stream, int b, int tokens, int before, cudaStream_t st, int which)
        : m(model), L(model->lay), r(buffers), h(stream), batch(b), n(tokens), M(b * tokens), past(before), parts(which), s(st) {
        W = L->c.width; sm = m->sm_count; kpw = dense_kpad(W); eps = L->c.norm_eps; f32 = L->f32;
        err = device_error_word(m->device);
        mp = dense_mpad(M);
    }
    ActOut tiled(uint8_t* t) const { ActOut o; o.tiles = t; o.m_pad = mp; return o; }
    ActOut plain(float* p, int64_t ld) const { ActOut o; o.rows = p; o.ld = ld; return o; }
    static DenseOut rows_out(float* p, int64_t ld, int act = DACT_NONE, const float* bias = nullptr, int64_t out_block = 0) {
        DenseOut o;
        o.out = p; o.ld = ld; o.act = act; o.bias = bias; o.out_block = out_block;
        return o;
    }
    cudaError_t product(int part, const DenseLin& lin, const uint8_t* xt, const float* x, int64_t ldx, const DenseOut& o, int64_t x_block = 0) {
        if (!(parts & part)) return cudaSuccess;
        return f32 ? launch_dense_f32(lin, x, ldx, x_block, M, o, s) : launch_dense_tc(lin, xt, M, o, r.scratch, err, sm, s);
    }
    // f32 rows a sublayer reads (f32 models)
    const float* in_rows() const { return L->c.pre_norm ? r.hn : h; }
    // Where the residual sum leaves the input of what comes next: a feed-forward (mlp), run `ri`'s mixer, or nothing.
    void next_input(size_t ri, bool mlp, RowArgs& a) const {
        a.act = ActOut();
        a.next_w = nullptr;
        if (ri >= L->runs.size()) return;
        const LayLayer& l = L->layers[(size_t)L->runs[ri].layer];
        if (!mlp && L->runs[ri].pass >= 0) {  // the stream itself, in front of the embedding
            a.act = f32 ? plain(r.cat, 2 * kpw) : tiled(r.xt);
            return;
        }
        a.next_w = input_norm(L, l, mlp);
        const bool rows = l.c.mixer == BT_MIX_WKV && !mlp;
        if (f32 || rows) { if (a.next_w || rows) a.act = plain(r.hn, W); }
        else a.act = tiled(r.xt);
    }
    // the input of run `ri` from the stream alone
    bt_status first_input(size_t ri) {
        const LayRun& run = L->runs[ri];
        const float* w = input_norm(L, L->layers[(size_t)run.layer], false);
        if (w) {
            RowArgs a;
            a.op = ROW_GROUPNORM; a.y = h; a.ld = W; a.w = w; a.eps = eps; a.rows = M; a.k = W;
            const bool rows = f32 || L->layers[(size_t)run.layer].c.mixer == BT_MIX_WKV;
            a.act = rows ? plain(r.hn, W) : tiled(r.xt);
            if (parts & PART_ROWS) BT_CUDA_TRY(launch_row_op(a, s, false));
        } else if (L->layers[(size_t)run.layer].c.mixer == BT_MIX_WKV) {
            BT_CUDA_TRY(cudaMemcpyAsync(r.hn, h, (size_t)M * W * sizeof(float), cudaMemcpyDeviceToDevice, s));
        } else if (!f32) {
            BT_CUDA_TRY(launch_rows_tile(h, W, 0, 1, W, 1, DACT_NONE, M, r.xt, mp, s));
        }
        return BT_OK;
    }

    bt_status attention(LayLayer& l, LayRun& run) {
        BT_CUDA_TRY(product(PART_IN, l.in, r.xt, in_rows(), W, rows_out(r.proj, l.in.n)));
        if (!(parts & PART_CORE)) return BT_OK;
        DenseAttn a = attn_args(m, l, run, r, batch, n);
        const ActOut out = f32 ? plain(r.mix, l.inner()) : tiled(r.mt);
        if (n >= kTileRowsMin && attn_tile_fits(a)) {
            a.q_bf16 = true;
            BT_CUDA_TRY(launch_attn_prep(a, s));
            BT_CUDA_TRY(launch_attn_tile(a, out, s));
        } else if (n == 1) {
            BT_CUDA_TRY(launch_attn_span(a, false, out, s, false));
        } else {
            BT_CUDA_TRY(launch_attn_prep(a, s));
            BT_CUDA_TRY(launch_attn_span(a, true, out, s, false));
        }
        return BT_OK;
    }
    bt_status ssm(LayLayer& l, LayRun& run) {
        BT_CUDA_TRY(product(PART_IN, l.in, r.xt, in_rows(), W, rows_out(r.proj, l.in.n)));
        SsmArgs a = ssm_args(m, l, run, r, batch, n);
        if (parts & PART_CORE) BT_CUDA_TRY(n == 1 ? launch_ssm_step(a, s, false) : launch_ssm_prefill(a, !f32, s));
        RowArgs g;
        g.op = ROW_GROUPNORM; g.y = r.mix; g.ld = l.inner(); g.w = l.vec[BT_LT_SSM_NORM]; g.eps = eps; g.groups = l.c.norm_groups;
        g.rows = M; g.k = l.inner();
        g.act = f32 ? plain(r.proj, l.inner()) : tiled(r.mt);  // the projection rows are used up
        if (parts & PART_ROWS) BT_CUDA_TRY(launch_row_op(g, s, false));
        return BT_OK;
    }
    bt_status latent(LayLayer& l, LayRun& run) {
        const bt_layer_config& c = l.c;
        BT_CUDA_TRY(product(PART_IN, l.in, r.xt, in_rows(), W, rows_out(r.proj, l.in.n)));
        LatentAttn a = latent_args(m, l, run, r, batch, n);
        if (n >= kTileRowsMin && latent_tile_fits(a)) {
            // keys and values of every position so far, a group of sequences at a time
            a.q_buf = reinterpret_cast<__nv_bfloat16*>(r.q);
            if (parts & PART_CORE) BT_CUDA_TRY(launch_latent_prep(a, s));
            const int64_t rows = ((int64_t)past + n + 63) / 64 * 64, tile_rows = dense_mpad(past + n), tile_bytes = tile_rows * l.expand.k_pad * 2;
            const int64_t seq = rows * l.expand.n;
            const int group = (int)std::max<int64_t>(1, std::min<int64_t>(batch, (int64_t)kExpandElems / seq));
            bt_status st = expand_room(L, (size_t)(group * (seq + tile_bytes / 2)));
            uint8_t* tiles = reinterpret_cast<uint8_t*>(L->kv16 + group * seq);  // the latents as the product reads them
            if (st != BT_OK) return st;
            for (int b0 = 0; b0 < batch; b0 += group) {
                const int nb = std::min(group, batch - b0);
                DenseOut o;
                o.out_rows16 = L->kv16; o.ld = l.expand.n; o.out_block = seq; o.shared_weights = true; o.blocks = nb; o.x_block = tile_bytes; o.m_pad = tile_rows;
                if (parts & PART_MID) {
                    BT_CUDA_TRY(launch_latent_tiles(a.kv, b0, nb, past + n, tiles, tile_rows, s));
                    BT_CUDA_TRY(launch_dense_tc(l.expand, tiles, past + n, o, nullptr, err, sm, s));
                }
                if (parts & PART_CORE) BT_CUDA_TRY(launch_latent_tile(a, L->kv16, rows, b0, nb, tiled(r.mt), s));
            }
            return BT_OK;
        }
        if (f32) { a.q_rows32 = r.c; a.q_rot = r.c + (size_t)M * c.heads * c.dim; }
        else { a.q_tiles = r.t1; a.q_rot = r.c; }
        const int64_t lat = (int64_t)c.heads * c.kv_rank;
        if (parts & PART_CORE) BT_CUDA_TRY(launch_latent_prep(a, s));
        DenseOut qa = rows_out(r.a, lat, DACT_NONE, nullptr, c.kv_rank);
        qa.halves = 2;
        BT_CUDA_TRY(product(PART_MID, l.mid, r.t1, r.c, (int64_t)c.heads * c.dim, qa, c.dim));
        if (parts & PART_CORE) BT_CUDA_TRY(launch_latent_span(a, true, f32 ? plain(r.b, lat) : tiled(r.t2), s, false));
        DenseOut v = rows_out(r.mix, l.inner(), DACT_NONE, nullptr, c.vdim);
        const bool direct = !f32 && c.vdim % 8 == 0;
        if (direct) { v.out = nullptr; v.out_tiles = r.mt; }
        BT_CUDA_TRY(product(PART_MID, l.mid2, r.t2, r.b, lat, v, c.kv_rank));
        if (!f32 && !direct && (parts & PART_MID)) BT_CUDA_TRY(launch_rows_tile(r.mix, l.inner(), 0, 1, l.inner(), 1, DACT_NONE, M, r.mt, mp, s));
        return BT_OK;
    }
    bt_status wkv(LayLayer& l, LayRun& run) {
        const int HD = l.inner(), rank = l.c.decay_rank;
        WkvMix x;
        x.hn = r.hn;
        for (int i = 0; i < 5; ++i) x.mu[i] = l.vec[BT_LT_MU_R + i];
        x.shift = run.ring; x.shift_slot = (int64_t)m->cfg.max_batch * W; x.pos = m->pos; x.batch = batch; x.q_rows = n; x.width = W;
        x.m_pad = mp;
        if (f32) x.rows5 = r.c; else { x.tiles4 = r.t1; x.tiles_w = r.t2; }
        if (parts & PART_ROWS) BT_CUDA_TRY(launch_wkv_mix(x, s));
        BT_CUDA_TRY(product(PART_IN, l.in, r.t1, r.c, 5ll * W, rows_out(r.proj, 4ll * HD, DACT_NONE, nullptr, HD), W));
        DenseOut low = rows_out(r.a, rank, f32 ? DACT_TANH : DACT_NONE);
        low.halves = 2;
        BT_CUDA_TRY(product(PART_MID, l.mid, r.t2, r.c + 4ll * W, 5ll * W, low));
        if (!f32 && (parts & PART_MID)) BT_CUDA_TRY(launch_rows_tile(r.a, rank, 0, 1, rank, 2, DACT_TANH, M, r.t2, mp, s));
        DenseOut z = rows_out(r.b, HD, DACT_DECAY, l.vec[BT_LT_WKV_W0]);
        z.halves = 2;
        BT_CUDA_TRY(product(PART_MID, l.mid2, r.t2, r.a, rank, z));
        if (parts & PART_CORE) BT_CUDA_TRY(launch_wkv_prefill(wkv_args(m, l, run, r, batch, n), s));
        RowArgs g;
        g.op = ROW_GROUPNORM; g.y = r.mix; g.ld = HD; g.w = l.vec[BT_LT_WKV_NORM]; g.eps = eps; g.groups = l.c.heads; g.rows = M; g.k = HD;
        g.gate = r.proj + 3ll * HD; g.gate_ld = 4ll * HD;
        g.act = f32 ? plain(r.c, HD) : tiled(r.mt);
        if (parts & PART_ROWS) BT_CUDA_TRY(launch_row_op(g, s, false));
        return BT_OK;
    }
    bt_status rglru(LayLayer& l, LayRun& run) {
        const int C = l.c.channels;
        BT_CUDA_TRY(product(PART_IN, l.in, r.xt, in_rows(), W, rows_out(r.proj, l.in.n, DACT_NONE, l.in_bias)));
        RgluArgs a = rglru_args(m, l, run, r, batch, n);
        if (parts & PART_CORE) BT_CUDA_TRY(launch_rglru_conv(a, s));
        DenseOut g = rows_out(r.b, 2ll * C, DACT_NONE, l.mid_bias, l.mid.n);
        g.halves = 2;
        BT_CUDA_TRY(product(PART_MID, l.mid, r.t1, r.a, C, g, l.mid.k));
        if (parts & PART_CORE) BT_CUDA_TRY(launch_rglru_scan(a, f32 ? plain(r.mix, C) : tiled(r.mt), s));
        return BT_OK;
    }
    // the chosen experts' outputs stay in r.ye; `res` adds them up
    bt_status moe(LayLayer& l, RowArgs& res) {
        const bt_layer_config& c = l.c;
        const RowNeeds& q = L->need;
        BT_CUDA_TRY(product(PART_ROUTE, l.router, r.xt, in_rows(), W, rows_out(r.logits, c.experts, DACT_NONE, l.vec[BT_LT_ROUTER_B])));
        MoeRoute a;
        a.logits = r.logits; a.ld = c.experts; a.rows = M; a.experts = c.experts; a.top = c.top;
        a.tile = f32 ? 64 : moe_tile_rows(M, c.top, c.experts);
        a.max_tiles = moe_max_tiles(M, c.top, c.experts, a.tile);
        int* p = r.choice;
        a.tiles = reinterpret_cast<ExpertTile*>(p); p += 4 * ((size_t)r.rows * q.top / 64 + q.experts + 1);
        a.sel = p; p += (size_t)r.rows * q.top;
        a.rank = p; p += (size_t)r.rows * q.top;
        a.dst = p; p += (size_t)r.rows * q.top;
        a.counts = p; p += q.experts;
        a.counts_done = p; p += q.experts;
        a.row_start = p; p += q.experts + 1;
        a.n_tiles = p;
        a.wt = r.wt; a.k = W; a.x_tiles = r.xt; a.m_pad = mp; a.me_pad = r.grouped; a.x = in_rows();
        if (f32) a.xe = reinterpret_cast<float*>(r.xe); else a.xe_tiles = r.xe;
        if (parts & PART_ROUTE) BT_CUDA_TRY(launch_moe_route(a, s));
        ExpertPlan plan;
        plan.tiles = a.tiles; plan.n_tiles = a.n_tiles; plan.row_start = a.row_start; plan.counts = a.counts_done; plan.tile = a.tile;
        plan.max_tiles = a.max_tiles; plan.max_rows = M;
        float* fe = reinterpret_cast<float*>(r.fe);
        DenseOut up = rows_out(f32 ? fe : nullptr, c.ff, DACT_SWIGLU), down = rows_out(r.ye, W);
        up.out_tiles = f32 ? nullptr : r.fe;
        up.plan = down.plan = &plan;
        up.m_pad = down.m_pad = r.grouped;
        BT_CUDA_TRY(product(PART_UP, l.e_up, r.xe, a.xe, W, up));
        BT_CUDA_TRY(product(PART_DOWN, l.e_down, r.fe, fe, c.ff, down));
        if (c.shared_ff) {
            DenseOut su = rows_out(f32 ? r.ff : nullptr, c.shared_ff, DACT_SWIGLU);
            su.out_tiles = f32 ? nullptr : r.ft;
            BT_CUDA_TRY(product(PART_UP, l.s_up, r.xt, in_rows(), W, su));
            BT_CUDA_TRY(product(PART_DOWN, l.s_down, r.ft, r.ff, c.shared_ff, rows_out(r.y, W)));
        } else {
            res.y = nullptr;
        }
        res.ye = r.ye; res.ye_ld = W; res.dst = a.dst; res.wt = a.wt; res.top = c.top;
        return BT_OK;
    }

    bt_status run(const int32_t* tokens) {
        bt_status st;
        const LayRun& run0 = L->runs[0];
        const bool plain_start = run0.pass >= 0 || !L->c.pre_norm;
        ActOut x0, front;
        if (L->loops()) x0 = f32 ? plain(r.cat + kpw, 2 * kpw) : tiled(r.xt + (size_t)(kpw / 64) * mp * 128);
        if (plain_start && !f32) front = tiled(r.xt);
        if (run0.pass >= 0 && f32) front = plain(r.cat, 2 * kpw);
        if (parts & PART_ROWS)
            BT_CUDA_TRY(launch_embed_pos(tokens, m->embed, L->pos_table, m->pos, batch, n, W, m->cfg.vocab_size, L->c.max_positions, h, front, s, false, x0));
        if (run0.pass < 0 && (L->c.pre_norm || L->layers[0].c.mixer == BT_MIX_WKV) && (st = first_input(0)) != BT_OK) return st;
        for (size_t ri = 0; ri < L->runs.size(); ++ri) {
            LayRun& run = L->runs[ri];
            LayLayer& l = L->layers[(size_t)run.layer];
            if (run.pass >= 0) {
                BT_CUDA_TRY(product(PART_LOOP, L->loop_in, r.xt, r.cat, 2 * kpw, rows_out(h, W, DACT_NONE, L->loop_step + (size_t)run.pass * W)));
                if ((st = first_input(ri)) != BT_OK) return st;
            }
            const float* mixed = r.mix;
            switch (l.c.mixer) {
                case BT_MIX_ATTENTION: st = attention(l, run); break;
                case BT_MIX_SSM: st = ssm(l, run); mixed = r.proj; break;
                case BT_MIX_LATENT: st = latent(l, run); break;
                case BT_MIX_WKV: st = wkv(l, run); mixed = r.c; break;
                default: st = rglru(l, run);
            }
            if (st != BT_OK) return st;
            BT_CUDA_TRY(product(PART_O, l.o, r.mt, mixed, l.inner(), rows_out(r.y, W)));
            RowArgs res;
            res.op = ROW_RESNORM; res.y = r.y; res.ld = W; res.eps = eps; res.rows = M; res.k = W; res.h_in = h; res.h_out = h;
            res.w = l.vec[BT_LT_NORM1];
            const bool mlp = l.c.mlp != BT_MLP_NONE;
            next_input(mlp ? ri : ri + 1, mlp, res);
            if (parts & PART_ROWS) BT_CUDA_TRY(launch_row_op(res, s, false));
            if (mlp) {
                if (l.c.mlp == BT_MLP_DENSE_RELU2) {
                    DenseOut up = rows_out(f32 ? r.ff : nullptr, l.c.ff, DACT_RELU2);
                    up.out_tiles = f32 ? nullptr : r.ft;
                    BT_CUDA_TRY(product(PART_UP, l.up, r.xt, in_rows(), W, up));
                    BT_CUDA_TRY(product(PART_DOWN, l.down, r.ft, r.ff, l.c.ff, rows_out(r.y, W)));
                } else if ((st = moe(l, res)) != BT_OK) {
                    return st;
                }
                res.w = l.vec[BT_LT_NORM2];
                next_input(ri + 1, false, res);
                if (parts & PART_ROWS) BT_CUDA_TRY(launch_row_op(res, s, false));
            }
            BT_CUDA_TRY(trace_stream(m, (int)ri, h, M, s));
        }
        return BT_OK;
    }
};
bt_status forward_rows(bt_model* m, const int32_t* tokens, float* h, RowBuffers& r, int batch, int n, int past, cudaStream_t s, int parts = PART_ALL) {
    return RowPass(m, r, h, batch, n, past, s, parts).run(tokens);
}

bool step_is_fused(const bt_model* m, int batch) { return batch <= m->lay->fused_rows; }

}  // namespace

bt_status layered_step(bt_model* m, int batch, cudaStream_t s) {
    return step_is_fused(m, batch) ? step_fused(m, batch, s) : forward_rows(m, m->tokens, m->h, m->lay->dec, batch, 1, m->host_pos, s);
}

bt_status layered_prefill(bt_model* m, int batch, int n, int past, cudaStream_t s) {
    return forward_rows(m, m->pf_tokens, m->pf_h, m->lay->pf, batch, n, past, s);
}

bt_status layered_prefill_buffers(bt_model* m, int rows) {
    if (rows <= m->pf_rows) return BT_OK;
    BT_CUDA_TRY(cudaDeviceSynchronize());
    cudaFree(m->pf_tokens); cudaFree(m->pf_h);
    m->pf_tokens = nullptr; m->pf_h = nullptr;
    m->pf_rows = 0;
    BT_CUDA_TRY(dev_alloc(&m->pf_tokens, (size_t)rows));
    BT_CUDA_TRY(dev_alloc(&m->pf_h, (size_t)rows * m->cfg.hidden_dim));
    bt_status st = alloc_rows(m, m->lay->pf, rows, true);
    if (st != BT_OK) return st;
    m->pf_rows = rows;
    return BT_OK;
}

bt_status layered_set_tensor(bt_model* m, bt_tensor_kind kind, const float* data, int64_t n_elem, bt_dtype storage) {
    Layered* L = m->lay;
    DeviceGuard guard(m->device);
    const int64_t W = L->c.width, VW = (int64_t)L->c.vocab_size * W;
    if (kind == BT_T_NORM_F) {
        if (n_elem != W) return set_error(BT_ERR_SHAPE, "bt_model_set_tensor: norm weight has %lld elements, %lld expected", (long long)n_elem, (long long)W);
        return upload_vec(&m->norm_f, data, W, L->c.norm_one_plus ? 1.0f : 0.0f);
    }
    if (storage != BT_BF16) return set_error(BT_ERR_ARG, "bt_model_set_tensor: layer-list models keep their tables in bf16");
    int64_t expect = VW;
    if (kind == BT_T_POS) expect = (int64_t)L->c.max_positions * W;
    if (kind == BT_T_LOOP_IN) expect = L->loops() ? 2 * W * W : 0;
    if (kind == BT_T_LOOP_STEP) expect = (int64_t)L->c.loop_times * W;
    const bool known = kind == BT_T_EMBED || kind == BT_T_LM_HEAD || kind == BT_T_POS || kind == BT_T_LOOP_IN || kind == BT_T_LOOP_STEP;
    if (!known || n_elem != expect || expect == 0)
        return set_error(BT_ERR_SHAPE, "bt_model_set_tensor: tensor %d with %lld elements, %lld expected", (int)kind, (long long)n_elem, (long long)expect);
    if (kind == BT_T_LOOP_STEP) {
        L->loop_set |= 1u;
        return upload_vec(&L->loop_step, data, n_elem, 0.0f);
    }
    if (kind == BT_T_LOOP_IN) {  // each half at a multiple of 64 inputs
        const int64_t kp = dense_kpad((int)W);
        std::vector<float> padded((size_t)(W * 2 * kp), 0.0f);
        for (int64_t r = 0; r < W; ++r)
            for (int half = 0; half < 2; ++half) memcpy(padded.data() + (r * 2 + half) * kp, data + (r * 2 + half) * W, (size_t)W * sizeof(float));
        L->loop_set |= 2u;
        return upload_rows(L->loop_in, padded.data(), (int)W, 0);
    }
    __nv_bfloat16** dst = kind == BT_T_EMBED ? &m->embed : (kind == BT_T_POS ? &L->pos_table : &m->lm_head);
    if (kind == BT_T_LM_HEAD && m->head_ld != W) {  // rows padded to whole 16-byte pieces
        std::vector<float> padded((size_t)L->c.vocab_size * m->head_ld, 0.0f);
        for (int64_t v = 0; v < L->c.vocab_size; ++v) memcpy(padded.data() + v * m->head_ld, data + v * W, (size_t)W * sizeof(float));
        if (!*dst) BT_CUDA_TRY(dev_alloc(dst, padded.size()));
        return upload_16bit(padded.data(), (int64_t)padded.size(), *dst, false);
    }
    if (!*dst) BT_CUDA_TRY(dev_alloc(dst, (size_t)n_elem));
    return upload_16bit(data, n_elem, *dst, false);
}

namespace {

// rotation angles position * base^(-2i / dims), their cosines and sines in f64, kept in f32
bt_status rot_table(Layered* L, double base, int dims, int* index) {
    for (size_t i = 0; i < L->tables.size(); ++i)
        if (L->tables[i].base == base && L->tables[i].dims == dims) { *index = (int)i; return BT_OK; }
    const int half = dims / 2;
    const size_t count = (size_t)L->c.max_seq_len * half;
    std::vector<float> c(count), s(count);
    std::vector<double> f((size_t)half);
    for (int i = 0; i < half; ++i) f[(size_t)i] = pow(base, -2.0 * i / dims);
    for (int p = 0; p < L->c.max_seq_len; ++p)
        for (int i = 0; i < half; ++i) {
            c[(size_t)p * half + i] = (float)cos(p * f[(size_t)i]);
            s[(size_t)p * half + i] = (float)sin(p * f[(size_t)i]);
        }
    RotTable t{base, dims, nullptr, nullptr};
    bt_status st = upload_vec(&t.cos_t, c.data(), (int64_t)count, 0.0f);
    if (st == BT_OK) st = upload_vec(&t.sin_t, s.data(), (int64_t)count, 0.0f);
    L->tables.push_back(t);
    *index = (int)L->tables.size() - 1;
    return st;
}

void grow(int& a, int64_t b) { a = std::max<int>(a, (int)b); }

void add_needs(const Layered* L, const LayLayer& l, RowNeeds& q) {
    const bt_layer_config& c = l.c;
    const int W = L->c.width, kpw = dense_kpad(W);
    grow(q.proj, c.mixer == BT_MIX_WKV ? 4 * l.inner() : l.in.n);
    grow(q.mix, l.inner());
    grow(q.mt, l.inner());
    switch (c.mixer) {
        case BT_MIX_ATTENTION:
            grow(q.q, (int64_t)c.heads * pad8(c.dim));
            grow(q.v, l.v_width());
            break;
        case BT_MIX_LATENT: {
            const int64_t lat = (int64_t)c.heads * c.kv_rank;
            grow(q.a, lat);
            grow(q.b, lat);
            grow(q.c, (int64_t)c.heads * (c.rot_dim + (L->f32 ? c.dim : 0)));
            grow(q.q, (int64_t)c.heads * (pad8(c.dim) + pad8(c.rot_dim)) / 2);
            grow(q.t1, (int64_t)c.heads * 2 * dense_kpad(c.dim));
            grow(q.t2, (int64_t)c.heads * dense_kpad(c.kv_rank));
            break;
        }
        case BT_MIX_WKV:
            grow(q.a, c.decay_rank);
            grow(q.b, l.inner());
            if (L->f32) grow(q.c, std::max(5 * W, l.inner()));
            grow(q.t1, 4 * kpw);
            grow(q.t2, 2 * std::max(kpw, dense_kpad(c.decay_rank)));
            break;
        case BT_MIX_RGLRU:
            grow(q.a, c.channels);
            grow(q.b, 2 * c.channels);
            grow(q.t1, (int64_t)c.blocks * 2 * dense_kpad(c.channels / c.blocks));
            break;
    }
    if (c.mlp == BT_MLP_DENSE_RELU2) {
        grow(q.ff, c.ff);
        grow(q.ft, c.ff);
    } else if (c.mlp == BT_MLP_MOE_SWIGLU) {
        q.moe = true;
        grow(q.ff, (int64_t)c.top * dense_kpad(c.ff) + dense_kpad(std::max(c.shared_ff, 1)));
        grow(q.ft, std::max(c.shared_ff, 1));
        grow(q.logits, c.experts);
        grow(q.experts, c.experts);
        grow(q.top, c.top);
        grow(q.e_ff, c.ff);
        grow(q.e_ff_pad, dense_kpad(c.ff));
    }
}

}  // namespace

bt_status layered_finalize(bt_model* m) {
    Layered* L = m->lay;
    if (!m->embed || !m->lm_head || !m->norm_f || (L->c.max_positions > 0 && !L->pos_table) || (L->loops() && L->loop_set != 3u))
        return set_error(BT_ERR_ARG, "bt_model_finalize: embedding, positions, loop tensors, lm_head or final norm missing");
    for (size_t i = 0; i < L->layers.size(); ++i) {
        const LayLayer& l = L->layers[i];
        for (int k = 0; k < kTensorKinds; ++k)
            if (tensor_elems(L, l, k) > 0 && !is_expert_kind(k) && !(l.set >> k & 1u))
                return set_error(BT_ERR_ARG, "bt_model_finalize: tensor %d of layer %d was never set", k, (int)i);
        for (size_t e = 0; e < l.experts_set.size(); ++e)
            if (l.experts_set[e] != 7) return set_error(BT_ERR_ARG, "bt_model_finalize: expert %d of layer %d is incomplete", (int)e, (int)i);
    }
    const int B = L->c.max_batch, W = L->c.width;
    bt_status st;
    L->fused_rows = std::min(8, B);
    auto fit = [&](const DenseLin& d) {
        while (d.tiles && L->fused_rows > 0 && !dense_stream_fits(d, L->fused_rows)) --L->fused_rows;
    };
    if (L->loops()) fit(L->loop_in);
    for (LayLayer& l : L->layers) {
        add_needs(L, l, L->need);
        for (const DenseLin* d : {&l.in, &l.o, &l.up, &l.down, &l.mid, &l.mid2, &l.router, &l.s_up}) fit(*d);
        if (l.c.mlp == BT_MLP_MOE_SWIGLU) {
            MoeStep a;
            a.up = &l.e_up; a.down = &l.e_down; a.shared_down = l.c.shared_ff ? &l.s_down : nullptr;
            a.experts = l.c.experts; a.top = l.c.top;
            while (L->fused_rows > 0 && (a.rows = L->fused_rows, !moe_step_fits(a))) --L->fused_rows;
        }
        if (l.c.mixer == BT_MIX_LATENT && l.c.rot_dims > 0 && (st = rot_table(L, l.c.rot_base, l.c.rot_dims, &l.table)) != BT_OK) return st;
        if (l.c.mixer == BT_MIX_SSM) {
            const LayRun none;
            grow(L->need.conv, ssm_conv_floats(ssm_args(m, l, none, L->dec, 1, 1)));
        }
    }
    for (LayRun& run : L->runs) {
        const LayLayer& l = L->layers[(size_t)run.layer];
        const bt_dtype dt = L->f32 ? BT_F32 : BT_BF16;
        if (l.c.mixer == BT_MIX_ATTENTION) {
            if ((st = bt_kv_create_dense(&run.kv, B, l.c.kv_heads, l.c.dim, l.c.vdim, L->c.max_seq_len, dt, m->device)) != BT_OK) return st;
        } else if (l.c.mixer == BT_MIX_LATENT) {
            if ((st = bt_kv_create_latent(&run.kv, B, l.c.kv_rank, l.c.rot_dim, L->c.max_seq_len, dt, m->device)) != BT_OK) return st;
        } else {
            BT_CUDA_TRY(dev_alloc(&run.state, (size_t)(B * l.state_floats())));
            BT_CUDA_TRY(dev_alloc(&run.ring, (size_t)(B * l.ring_floats(W))));
        }
    }
    if (!L->f32) {
        int64_t most = 0;
        for (const LayLayer& l : L->layers)
            if (l.c.mixer == BT_MIX_WKV) most = std::max(most, wkv_segment_floats(l.c.heads, l.c.dim));
        if (most) BT_CUDA_TRY(dev_alloc(&L->wkv_seg, (size_t)(most * B)));
    }
    m->rms_eps = L->c.norm_eps;
    m->logit_cap = L->c.logit_softcap;
    m->head_rows = std::max(B, 64);
    const size_t R = (size_t)m->head_rows;
    BT_CUDA_TRY(dev_alloc(&m->tokens, (size_t)B));
    BT_CUDA_TRY(dev_alloc(&m->pos, (size_t)B));
    BT_CUDA_TRY(dev_alloc(&m->h, R * W));
    BT_CUDA_TRY(dev_alloc(&L->h2, (size_t)B * W));
    BT_CUDA_TRY(dev_alloc(&m->logits, R * L->c.vocab_size));
    BT_CUDA_TRY(dev_alloc(&m->next, R));
    BT_CUDA_TRY(dev_alloc(&m->cand_val, R * lm_head_max_candidates(m->sm_count)));
    BT_CUDA_TRY(dev_alloc(&m->cand_idx, R * lm_head_max_candidates(m->sm_count)));
    if (!L->f32) {  // the head on tensor cores for more than 8 rows
        BT_CUDA_TRY(cudaMalloc(&m->lm_tiles, lm_head_tc_weight_bytes(L->c.vocab_size, W)));
        BT_CUDA_TRY(cudaMalloc(&m->lm_btiles, lm_head_tc_act_bytes(W)));
        BT_CUDA_TRY(launch_lm_retile(m->lm_head, L->c.vocab_size, W, m->lm_tiles, 0, m->head_ld));
        BT_CUDA_TRY(cudaDeviceSynchronize());
    }
    if ((st = alloc_rows(m, L->dec, B, B > L->fused_rows)) != BT_OK) return st;
    BT_CUDA_TRY(cudaMallocHost(reinterpret_cast<void**>(&m->tokens_pinned), (size_t)B * sizeof(int32_t)));
    BT_CUDA_TRY(cudaMallocHost(reinterpret_cast<void**>(&m->next_pinned), (size_t)B * sizeof(int32_t)));
    BT_CUDA_TRY(cudaMallocHost(reinterpret_cast<void**>(&m->err_pinned), sizeof(unsigned int)));
    *m->err_pinned = 0;
    BT_CUDA_TRY(cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking));
    return BT_OK;
}

void layered_destroy(bt_model* m) {
    Layered* L = m->lay;
    for (LayLayer& l : L->layers) {
        size_t count;
        const DenseLin* const* all = l.lins(&count);
        for (size_t i = 0; i < count; ++i) cudaFree(all[i]->tiles);
        for (float* v : l.vec) cudaFree(v);
        cudaFree(l.in_bias); cudaFree(l.mid_bias);
    }
    for (LayRun& run : L->runs) {
        bt_kv_destroy(run.kv);
        cudaFree(run.state); cudaFree(run.ring);
    }
    for (RotTable& t : L->tables) { cudaFree(t.cos_t); cudaFree(t.sin_t); }
    L->dec.release();
    L->pf.release();
    cudaFree(L->pos_table); cudaFree(L->h2); cudaFree(L->loop_in.tiles); cudaFree(L->loop_step); cudaFree(L->kv16); cudaFree(L->wkv_seg);
    delete L;
    m->lay = nullptr;
}

bt_status layered_reset(bt_model* m) {
    for (LayRun& run : m->lay->runs) {
        if (run.kv) { bt_status st = bt_kv_reset(run.kv); if (st != BT_OK) return st; }
        const LayLayer& l = m->lay->layers[(size_t)run.layer];
        const size_t B = (size_t)m->cfg.max_batch;
        if (run.state) BT_CUDA_TRY(cudaMemset(run.state, 0, B * l.state_floats() * sizeof(float)));
        if (run.ring) BT_CUDA_TRY(cudaMemset(run.ring, 0, B * l.ring_floats(m->lay->c.width) * sizeof(float)));
    }
    return BT_OK;
}

int layered_launches(const bt_model* m, int batch) {
    const Layered* L = m->lay;
    const bool fused = step_is_fused(m, batch);
    int n = 1 + (fused ? 1 : 0);  // embedding; fused: the last residual sum
    auto product = [&](const DenseLin& d, int act = DACT_NONE) { return fused || L->f32 ? 1 : dense_tc_kernels(d, batch, m->sm_count, act); };
    if (!fused && L->c.pre_norm && L->runs[0].pass < 0) ++n;
    for (const LayRun& run : L->runs) {
        const LayLayer& l = L->layers[(size_t)run.layer];
        const bool b16 = !L->f32;
        if (run.pass >= 0) n += product(L->loop_in) + (fused ? 0 : 1);
        n += product(l.in) + 1 + product(l.o);  // with attention or recurrence
        switch (l.c.mixer) {
            case BT_MIX_SSM: n += fused ? 0 : 1; break;
            case BT_MIX_LATENT: n += product(l.mid) + product(l.mid2) + (fused ? 0 : 1 + (b16 && l.c.vdim % 8 ? 1 : 0)); break;
            case BT_MIX_WKV: n += fused ? 0 : 2 + product(l.mid) + product(l.mid2) + (b16 ? 1 : 0); break;
            case BT_MIX_RGLRU: n += fused ? 0 : 1 + product(l.mid); break;
        }
        if (l.c.mlp == BT_MLP_DENSE_RELU2) n += product(l.up) + product(l.down);
        if (l.c.mlp == BT_MLP_MOE_SWIGLU)
            n += fused ? 3 : product(l.router) + 3 + 2 + (l.c.shared_ff ? product(l.s_up, DACT_SWIGLU) + product(l.s_down) : 0);
        if (!fused) n += 1 + (l.c.mlp != BT_MLP_NONE ? 1 : 0);
    }
    if (m->lm_tiles && batch > 8) return n + 4;  // prepare, product, arg-max, position advance
    return n + (batch <= 4 ? 1 : (batch + 7) / 8) + 1;
}

int layered_runs(const bt_model* m) { return (int)m->lay->runs.size(); }

bt_kv_cache* layered_kv(bt_model* m, int run) {
    return run < 0 || run >= (int)m->lay->runs.size() ? nullptr : m->lay->runs[(size_t)run].kv;
}

}  // namespace bt

using namespace bt;

extern "C" int bt_model_layer_runs(const bt_model* m) { return m ? (m->lay ? layered_runs(m) : m->cfg.num_layers) : 0; }

extern "C" bt_status bt_model_enqueue_parts(bt_model* m, int batch, int n_tokens, int parts, void* stream) {
    if (!m || !m->lay || !m->finalized) return set_error(BT_ERR_ARG, "bt_model_enqueue_parts: not a finalized layer-list model");
    if (batch < 1 || batch > m->cfg.max_batch || n_tokens < 1 || (n_tokens > 1 && (int64_t)batch * n_tokens > m->pf_rows) ||
        m->host_pos + n_tokens > m->cfg.max_position_embeddings)
        return set_error(BT_ERR_SHAPE, "bt_model_enqueue_parts: %d sequences of %d tokens (prefill that many first)", batch, n_tokens);
    DeviceGuard guard(m->device);
    cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
    if (n_tokens > 1) return forward_rows(m, m->pf_tokens, m->pf_h, m->lay->pf, batch, n_tokens, m->host_pos, s, parts);
    return step_is_fused(m, batch) ? step_fused(m, batch, s, parts) : forward_rows(m, m->tokens, m->h, m->lay->dec, batch, 1, m->host_pos, s, parts);
}

namespace {

bt_status check_layer(const bt_layer_config& l, int i, int width, int* v_width) {
    const bool heads = l.mixer != BT_MIX_RGLRU;
    if (heads && (l.heads < 1 || (l.mixer != BT_MIX_WKV && l.vdim < 1))) return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: no heads", i);
    switch (l.mixer) {
        case BT_MIX_ATTENTION:
            if (l.kv_heads < 1 || l.heads % l.kv_heads != 0 || l.dim < 1)
                return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: %d query heads over %d KV heads of size %d", i, l.heads, l.kv_heads, l.dim);
            if (l.vdim > attn_max_dim() || l.dim > attn_max_dim())
                return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: key and value heads of %d and %d, at most %d", i, l.dim, l.vdim, attn_max_dim());
            if (l.q_temp_coef != 0.0f && !(l.q_temp_every > 0.0)) return set_error(BT_ERR_ARG, "bt_model_create_layers: layer %d: q_temp_every must be positive", i);
            if (l.v_mix) {
                if (*v_width && *v_width != l.kv_heads * l.vdim) return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: value mixing between layers of different value size", i);
                *v_width = l.kv_heads * l.vdim;
            }
            break;
        case BT_MIX_SSM:
            if (l.groups < 1 || l.heads % l.groups != 0 || !ssm_state_pad(l.state) || l.conv_taps < 1 || l.norm_groups < 1 ||
                (l.heads * l.vdim) % l.norm_groups != 0)
                return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: %d heads, %d groups, state %d, %d taps, %d norm groups", i, l.heads, l.groups, l.state, l.conv_taps, l.norm_groups);
            break;
        case BT_MIX_LATENT:
            if (l.dim < 1 || l.kv_rank < 1 || l.kv_rank > latent_max_rank() || l.rot_dim < 1 || l.rot_dim > latent_max_rot() || l.rot_dims < 0 ||
                l.rot_dims % 2 || l.rot_dims > l.rot_dim || (l.rot_dims && !(l.rot_base > 0.0)))
                return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: heads of %d, latent rank %d (at most %d), %d of %d rotated (at most %d)", i, l.dim, l.kv_rank, latent_max_rank(), l.rot_dims, l.rot_dim, latent_max_rot());
            break;
        case BT_MIX_WKV:
            if (l.dim < 1 || l.dim > wkv_max_dim() || l.decay_rank < 1 || l.decay_rank > 512)
                return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: wkv heads of %d (at most %d), decay rank %d (at most 512)", i, l.dim, wkv_max_dim(), l.decay_rank);
            break;
        case BT_MIX_RGLRU:
            if (l.channels < 1 || l.blocks < 1 || l.channels % l.blocks != 0 || l.conv_taps < 1)
                return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: %d channels in %d blocks, %d taps", i, l.channels, l.blocks, l.conv_taps);
            break;
        default:
            return set_error(BT_ERR_ARG, "bt_model_create_layers: layer %d: unknown mixer %d", i, l.mixer);
    }
    if (l.mlp == BT_MLP_MOE_SWIGLU) {
        if (l.ff < 1 || l.experts < 1 || l.experts > moe_max_experts() || l.top < 1 || l.top > l.experts || l.top > 64 || l.shared_ff < 0)
            return set_error(BT_ERR_ARG, "bt_model_create_layers: layer %d: the best %d of %d experts of width %d (shared %d)", i, l.top, l.experts, l.ff, l.shared_ff);
    } else if (l.mlp != BT_MLP_NONE && (l.mlp != BT_MLP_DENSE_RELU2 || l.ff < 1)) {
        return set_error(BT_ERR_ARG, "bt_model_create_layers: layer %d: unknown feed-forward %d of width %d", i, l.mlp, l.ff);
    }
    (void)width;
    return BT_OK;
}

bt_status alloc_layer(LayLayer& l, int W, bool f32) {
    const bt_layer_config& c = l.c;
    bt_status st = BT_OK;
    auto lin = [&](DenseLin& d, int n, int k, int blocks = 1) { if (st == BT_OK) st = alloc_lin(d, n, k, blocks); };
    switch (c.mixer) {
        case BT_MIX_ATTENTION: lin(l.in, c.heads * c.dim + c.kv_heads * (c.dim + c.vdim), W); break;
        case BT_MIX_SSM: lin(l.in, l.inner() + l.channels() + c.heads, W); break;
        case BT_MIX_LATENT:
            lin(l.in, c.heads * (c.dim + c.rot_dim) + c.kv_rank + c.rot_dim + (c.out_gate ? c.heads : 0), W);
            lin(l.mid, c.kv_rank, c.dim, c.heads);
            lin(l.mid2, c.vdim, c.kv_rank, c.heads);
            if (!f32) lin(l.expand, c.heads * (pad8(c.dim) + pad8(c.vdim)), c.kv_rank);
            break;
        case BT_MIX_WKV:
            lin(l.in, l.inner(), W, 4);
            lin(l.mid, c.decay_rank, W);
            lin(l.mid2, l.inner(), c.decay_rank);
            break;
        default:
            lin(l.in, 2 * c.channels, W);
            lin(l.mid, 2 * (c.channels / c.blocks), c.channels / c.blocks, c.blocks);
    }
    lin(l.o, W, l.inner());
    if (c.mlp == BT_MLP_DENSE_RELU2) { lin(l.up, c.ff, W); lin(l.down, W, c.ff); }
    if (c.mlp == BT_MLP_MOE_SWIGLU) {
        lin(l.router, c.experts, W);
        lin(l.e_up, 2 * c.ff, W, c.experts);
        lin(l.e_down, W, c.ff, c.experts);
        if (c.shared_ff) { lin(l.s_up, 2 * c.shared_ff, W); lin(l.s_down, W, c.shared_ff); }
        l.experts_set.assign((size_t)c.experts, 0);
    }
    return st;
}

// part of a vector that several tensors share
bt_status upload_part(float** dst, int64_t total, const float* host, int64_t n, int64_t first, int64_t step) {
    if (!*dst) {
        BT_CUDA_TRY(dev_alloc(dst, (size_t)total));
        BT_CUDA_TRY(cudaMemset(*dst, 0, (size_t)total * sizeof(float)));
    }
    BT_CUDA_TRY(cudaMemcpy2D(*dst + first, (size_t)step * sizeof(float), host, sizeof(float), sizeof(float), (size_t)n, cudaMemcpyHostToDevice));
    return BT_OK;
}

}  // namespace

extern "C" bt_status bt_model_create_layers(bt_model** out, const bt_layers_config* cfg, const bt_layer_config* layers, int device) {
    if (!out || !cfg || !layers) return set_error(BT_ERR_ARG, "bt_model_create_layers: null pointer");
    *out = nullptr;
    const bt_layers_config& c = *cfg;
    if (c.vocab_size < 1 || c.width < 1 || c.num_layers < 1 || c.max_positions < 0)
        return set_error(BT_ERR_SHAPE, "bt_model_create_layers: bad dimensions");
    if (c.max_seq_len < 1 || (c.max_positions > 0 && c.max_seq_len > c.max_positions))
        return set_error(BT_ERR_SHAPE, "bt_model_create_layers: max_seq_len %d outside 1..%d", c.max_seq_len, c.max_positions);
    if (c.max_batch < 1 || c.max_batch > 64) return set_error(BT_ERR_ARG, "bt_model_create_layers: max_batch must be 1..64");
    if (c.dtype != BT_BF16 && c.dtype != BT_F32) return set_error(BT_ERR_ARG, "bt_model_create_layers: dtype must be BT_BF16 or BT_F32");
    if (c.loop_times < 0 || (c.loop_times > 0 && (c.loop_start < 0 || c.loop_start >= c.loop_stop || c.loop_stop > c.num_layers)))
        return set_error(BT_ERR_SHAPE, "bt_model_create_layers: loop over layers %d .. %d of %d, %d times", c.loop_start, c.loop_stop, c.num_layers, c.loop_times);
    int v_width = 0;
    for (int i = 0; i < c.num_layers; ++i) {
        bt_status st = check_layer(layers[i], i, c.width, &v_width);
        if (st != BT_OK) return st;
    }
    if (bt_device_count() <= device || device < 0) return set_error(BT_ERR_DEVICE, "bt_model_create_layers: no CUDA device %d", device);
    DeviceGuard guard(device);
    if (!guard.ok || !device_error_word(device)) return set_error(BT_ERR_DEVICE, "bt_model_create_layers: cannot use device %d", device);
    bt_model* m = new (std::nothrow) bt_model();
    Layered* L = new (std::nothrow) Layered();
    if (!m || !L) { delete m; delete L; return set_error(BT_ERR_NOMEM, "host allocation failed"); }
    m->lay = L;
    m->device = device;
    m->sm_count = device_sm_count(device);
    m->cfg.arch = 2;
    m->cfg.vocab_size = c.vocab_size;
    m->cfg.hidden_dim = c.width;
    m->cfg.num_layers = c.num_layers;
    m->cfg.max_position_embeddings = c.max_seq_len;
    m->cfg.max_batch = c.max_batch;
    m->head_ld = (c.width + 7) / 8 * 8;
    L->c = c;
    L->f32 = c.dtype == BT_F32;
    L->layers.resize((size_t)c.num_layers);
    bool source = false;
    for (int i = 0; i < c.num_layers; ++i) {
        LayLayer& l = L->layers[(size_t)i];
        l.c = layers[i];
        if (l.c.mixer == BT_MIX_ATTENTION) {
            l.v_source = l.c.v_mix && !source;
            l.v_target = l.c.v_mix && source;
            source |= l.c.v_mix != 0;
        }
        bt_status st = alloc_layer(l, c.width, L->f32);
        if (st != BT_OK) { bt_model_destroy(m); return st; }
    }
    auto add_run = [&](int layer, int pass) {
        LayRun run;
        run.layer = layer; run.pass = pass;
        L->runs.push_back(run);
    };
    const int start = L->loops() ? c.loop_start : 0, stop = L->loops() ? c.loop_stop : 0;
    for (int i = 0; i < start; ++i) add_run(i, -1);
    for (int t = 0; t < c.loop_times; ++t)
        for (int i = start; i < stop; ++i) add_run(i, i == start ? t : -1);
    for (int i = stop; i < c.num_layers; ++i) add_run(i, -1);
    if (L->loops()) {
        bt_status st = alloc_lin(L->loop_in, c.width, 2 * dense_kpad(c.width));
        if (st != BT_OK) { bt_model_destroy(m); return st; }
    }
    *out = m;
    return BT_OK;
}

extern "C" bt_status bt_model_set_layer_tensor(bt_model* m, int layer, bt_layer_tensor kind, const float* data, int64_t n_elem) {
    if (!m || !data || !m->lay) return set_error(BT_ERR_ARG, "bt_model_set_layer_tensor: null pointer or not a layer-list model");
    if (m->finalized) return set_error(BT_ERR_ARG, "bt_model_set_layer_tensor: model already finalized");
    if (layer < 0 || layer >= m->cfg.num_layers || (int)kind < 0 || (int)kind >= kTensorKinds || is_expert_kind(kind))
        return set_error(BT_ERR_ARG, "bt_model_set_layer_tensor: layer %d / tensor %d out of range", layer, (int)kind);
    Layered* L = m->lay;
    LayLayer& l = L->layers[(size_t)layer];
    const int64_t expect = tensor_elems(L, l, kind);
    if (expect == 0 || n_elem != expect)
        return set_error(BT_ERR_SHAPE, "bt_model_set_layer_tensor: layer %d tensor %d has %lld elements, %lld expected", layer, (int)kind, (long long)n_elem, (long long)expect);
    DeviceGuard guard(m->device);
    const bt_layer_config& c = l.c;
    const bool lat = c.mixer == BT_MIX_LATENT;
    const int nq = c.heads * (c.dim + (lat ? c.rot_dim : 0)), nk = c.kv_heads * c.dim;
    const int kb = c.mixer == BT_MIX_RGLRU ? c.channels / c.blocks : 0;
    bt_status st = BT_OK;
    auto rows = [&](const DenseLin& lin, int n, int row0 = 0, int step = 1, int block = 0, const float* from = nullptr) {
        if (st == BT_OK) st = upload_rows(lin, from ? from : data, n, row0, step, block);
    };
    switch (kind) {
        case BT_LT_Q: rows(l.in, nq); break;
        case BT_LT_K: rows(l.in, nk, nq); break;
        case BT_LT_V: rows(l.in, c.kv_heads * c.vdim, nq + nk); break;
        case BT_LT_SSM_IN: rows(l.in, l.in.n); break;
        case BT_LT_O: case BT_LT_SSM_O: rows(l.o, l.o.n); break;
        case BT_LT_MLP_UP: rows(l.up, l.up.n); break;
        case BT_LT_MLP_DOWN: rows(l.down, l.down.n); break;
        case BT_LT_DKV: rows(l.in, c.kv_rank + c.rot_dim, nq); break;
        case BT_LT_GATE: rows(l.in, c.heads, nq + c.kv_rank + c.rot_dim); break;
        case BT_LT_UK: {  // per head: transposed for the absorbed queries, as it is for the expanded keys
            std::vector<float> t((size_t)c.kv_rank * c.dim);
            for (int h = 0; h < c.heads && st == BT_OK; ++h) {
                const float* w = data + (size_t)h * c.dim * c.kv_rank;
                for (int d = 0; d < c.dim; ++d)
                    for (int r = 0; r < c.kv_rank; ++r) t[(size_t)r * c.dim + d] = w[(size_t)d * c.kv_rank + r];
                rows(l.mid, c.kv_rank, 0, 1, h, t.data());
                if (l.expand.tiles) rows(l.expand, c.dim, h * pad8(c.dim), 1, 0, w);
            }
            break;
        }
        case BT_LT_UV:
            for (int h = 0; h < c.heads && st == BT_OK; ++h) {
                const float* w = data + (size_t)h * c.vdim * c.kv_rank;
                rows(l.mid2, c.vdim, 0, 1, h, w);
                if (l.expand.tiles) rows(l.expand, c.vdim, c.heads * pad8(c.dim) + h * pad8(c.vdim), 1, 0, w);
            }
            break;
        case BT_LT_WKV_R: case BT_LT_WKV_K: case BT_LT_WKV_V: case BT_LT_WKV_G: rows(l.in, l.in.n, 0, 1, (int)kind - (int)BT_LT_WKV_R); break;
        case BT_LT_WKV_W1: rows(l.mid, l.mid.n); break;
        case BT_LT_WKV_W2: rows(l.mid2, l.mid2.n); break;
        case BT_LT_RG_Y: rows(l.in, c.channels); break;
        case BT_LT_RG_X: rows(l.in, c.channels, c.channels); break;
        case BT_LT_RG_Y_B: st = upload_part(&l.in_bias, 2ll * c.channels, data, c.channels, 0, 1); break;
        case BT_LT_RG_X_B: st = upload_part(&l.in_bias, 2ll * c.channels, data, c.channels, c.channels, 1); break;
        case BT_LT_RG_RA: case BT_LT_RG_RI:  // the two gates of a channel in neighbouring rows
            for (int b = 0; b < c.blocks; ++b) rows(l.mid, kb, kind == BT_LT_RG_RA ? 0 : 1, 2, b, data + (size_t)b * kb * kb);
            break;
        case BT_LT_RG_RA_B: st = upload_part(&l.mid_bias, 2ll * c.channels, data, c.channels, 0, 2); break;
        case BT_LT_RG_RI_B: st = upload_part(&l.mid_bias, 2ll * c.channels, data, c.channels, 1, 2); break;
        case BT_LT_ROUTER: rows(l.router, c.experts); break;
        case BT_LT_S_GATE: rows(l.s_up, c.shared_ff, 0, 2); break;
        case BT_LT_S_UP: rows(l.s_up, c.shared_ff, 1, 2); break;
        case BT_LT_S_DOWN: rows(l.s_down, l.s_down.n); break;
        case BT_LT_VMIX: l.vmix = data[0]; break;
        case BT_LT_NORM1: case BT_LT_NORM2: case BT_LT_PRE1: case BT_LT_PRE2:
            st = upload_vec(&l.vec[kind], data, n_elem, L->c.norm_one_plus ? 1.0f : 0.0f);
            break;
        default: st = upload_vec(&l.vec[kind], data, n_elem, 0.0f); break;
    }
    if (st == BT_OK) l.set |= 1ull << (int)kind;
    return st;
}

extern "C" bt_status bt_model_set_expert_tensor(bt_model* m, int layer, int expert, bt_layer_tensor kind, const float* data, int64_t n_elem) {
    if (!m || !data || !m->lay) return set_error(BT_ERR_ARG, "bt_model_set_expert_tensor: null pointer or not a layer-list model");
    if (m->finalized) return set_error(BT_ERR_ARG, "bt_model_set_expert_tensor: model already finalized");
    if (layer < 0 || layer >= m->cfg.num_layers || !is_expert_kind(kind) || expert < 0 || expert >= (int)m->lay->layers[(size_t)layer].experts_set.size())
        return set_error(BT_ERR_ARG, "bt_model_set_expert_tensor: layer %d / expert %d / tensor %d out of range", layer, expert, (int)kind);
    LayLayer& l = m->lay->layers[(size_t)layer];
    if (n_elem != tensor_elems(m->lay, l, kind))
        return set_error(BT_ERR_SHAPE, "bt_model_set_expert_tensor: layer %d tensor %d has %lld elements, %lld expected", layer, (int)kind, (long long)n_elem, (long long)tensor_elems(m->lay, l, kind));
    DeviceGuard guard(m->device);
    const int part = kind == BT_LT_E_GATE ? 0 : (kind == BT_LT_E_UP ? 1 : 2);
    bt_status st = part < 2 ? upload_rows(l.e_up, data, l.c.ff, part, 2, expert) : upload_rows(l.e_down, data, l.e_down.n, 0, 1, expert);
    if (st == BT_OK) l.experts_set[(size_t)expert] |= (uint8_t)(1u << part);
    return st;
}

extern "C" float* bt_model_recurrent_state(bt_model* m, int run, int64_t* n_floats) {
    if (n_floats) *n_floats = 0;
    if (!m || !m->lay || run < 0 || run >= layered_runs(m)) return nullptr;
    const LayRun& r = m->lay->runs[(size_t)run];
    if (n_floats && r.state) *n_floats = (int64_t)m->cfg.max_batch * m->lay->layers[(size_t)r.layer].state_floats();
    return r.state;
}
extern "C" float* bt_model_conv_ring(bt_model* m, int run, int64_t* n_floats) {
    if (n_floats) *n_floats = 0;
    if (!m || !m->lay || run < 0 || run >= layered_runs(m)) return nullptr;
    const LayRun& r = m->lay->runs[(size_t)run];
    if (n_floats && r.ring) *n_floats = (int64_t)m->cfg.max_batch * m->lay->layers[(size_t)r.layer].ring_floats(m->lay->c.width);
    return r.ring;
}
