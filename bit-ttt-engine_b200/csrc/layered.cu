// Layer-list models: dense 16-bit projections, a mixer per layer (attention over an unquantised cache, state-space
// recurrence), learned positions, norms on the sublayers' outputs.  The model object, its step loop (graph per batch
// size), prefill loop, head, pick, positions and trace are those of model.cu; this file owns the layers.
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

constexpr int kTensorKinds = BT_LT_MLP_DOWN + 1;

// What the sublayers of `rows` tokens write on the way.
struct RowBuffers {
    int rows = 0;
    float* proj = nullptr;     // a mixer's input projection
    float* mix = nullptr;      // attention output / gated recurrence output, f32 rows
    float* y = nullptr;        // a sublayer's output before its norm
    float* ff = nullptr;       // feed-forward activations, f32 rows
    float* conv = nullptr;     // recurrence: channels after convolution and silu
    float* v_first = nullptr;
    void* q = nullptr;         // prepared queries
    uint8_t* xt = nullptr;     // bf16 models: tiled activations (residual stream, mixer output, feed-forward)
    uint8_t* mt = nullptr;
    uint8_t* ft = nullptr;
    float* scratch = nullptr;  // partial sums of the tcgen05 product
    void release() {
        for (void* p : {(void*)proj, (void*)mix, (void*)y, (void*)ff, (void*)conv, (void*)v_first, q, (void*)xt, (void*)mt, (void*)ft, (void*)scratch}) cudaFree(p);
        *this = RowBuffers();
    }
};

struct LayLayer {
    bt_layer_config c{};
    DenseLin in, o, up, down;  // in: q|k|v, or z|x|B|C|dt
    float* vec[kTensorKinds] = {nullptr};  // the small tensors, f32 on the device
    float vmix = 0.f;
    bool v_source = false, v_target = false;  // gives / takes the mixed-in values
    unsigned set = 0;                          // tensors received
    bt_kv_cache* kv = nullptr;
    float* state = nullptr;
    float* ring = nullptr;
    int inner() const { return c.heads * c.vdim; }
    int channels() const { return inner() + 2 * c.groups * c.state; }
    int state_pad() const { return ssm_state_pad(c.state); }
    int v_width() const { return c.kv_heads * c.vdim; }
};

}  // namespace

struct Layered {
    bt_layers_config c{};
    std::vector<LayLayer> layers;
    __nv_bfloat16* pos_table = nullptr;
    float* h2 = nullptr;  // second residual-stream buffer of the fused decode step
    RowBuffers dec, pf;
    bool f32 = false;
    int max_in = 0, max_mix = 0, max_ff = 0, max_channels = 0, max_q = 0, max_v = 0, fused_rows = 0;
};

namespace {

bt_status alloc_lin(DenseLin& l, int n, int k) {
    l.n = n; l.k = k; l.n_pad = (n + 127) / 128 * 128; l.k_pad = dense_kpad(k);
    BT_CUDA_TRY(dev_alloc(&l.tiles, l.bytes()));
    BT_CUDA_TRY(cudaMemset(l.tiles, 0, l.bytes()));
    return BT_OK;
}

// elements a tensor of this layer must have; 0: the layer has no such tensor
int64_t tensor_elems(const Layered* L, const LayLayer& l, int kind) {
    const bt_layer_config& c = l.c;
    const int64_t W = L->c.width;
    const bool att = c.mixer == BT_MIX_ATTENTION, ssm = c.mixer == BT_MIX_SSM, mlp = c.mlp != BT_MLP_NONE;
    switch (kind) {
        case BT_LT_NORM1: return W;
        case BT_LT_NORM2: return mlp ? W : 0;
        case BT_LT_Q: return att ? (int64_t)c.heads * c.dim * W : 0;
        case BT_LT_K: return att ? (int64_t)c.kv_heads * c.dim * W : 0;
        case BT_LT_V: return att ? (int64_t)c.kv_heads * c.vdim * W : 0;
        case BT_LT_O: return att ? (int64_t)l.inner() * W : 0;
        case BT_LT_Q_NORM: return att && c.qk_norm ? (int64_t)c.heads * c.dim : 0;
        case BT_LT_K_NORM: return att && c.qk_norm ? (int64_t)c.kv_heads * c.dim : 0;
        case BT_LT_SINK: return att && c.sink ? c.heads : 0;
        case BT_LT_VMIX: return att && c.v_mix ? 1 : 0;
        case BT_LT_SSM_IN: return ssm ? (int64_t)(l.inner() + l.channels() + c.heads) * W : 0;
        case BT_LT_SSM_CONV: return ssm ? (int64_t)l.channels() * c.conv_taps : 0;
        case BT_LT_SSM_CONV_B: return ssm ? l.channels() : 0;
        case BT_LT_SSM_DT_BIAS: case BT_LT_SSM_A_LOG: case BT_LT_SSM_D: return ssm ? c.heads : 0;
        case BT_LT_SSM_NORM: return ssm ? l.inner() : 0;
        case BT_LT_SSM_O: return ssm ? (int64_t)l.inner() * W : 0;
        case BT_LT_MLP_UP: case BT_LT_MLP_DOWN: return mlp ? (int64_t)c.ff * W : 0;
    }
    return 0;
}

bt_status upload_rows(const DenseLin& lin, const float* host, int rows, int row0) {
    const int step = (int)std::max<int64_t>(1, (16 << 20) / lin.k);
    float* tmp = nullptr;
    BT_CUDA_TRY(dev_alloc(&tmp, (size_t)std::min(step, rows) * lin.k));
    cudaError_t e = cudaSuccess;
    for (int r = 0; r < rows && e == cudaSuccess; r += step) {
        const int n = std::min(step, rows - r);
        e = cudaMemcpy(tmp, host + (size_t)r * lin.k, (size_t)n * lin.k * sizeof(float), cudaMemcpyHostToDevice);
        if (e == cudaSuccess) e = launch_dense_tile(tmp, n, lin.k, row0 + r, lin, 0);
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
    r.release();
    const size_t n = (size_t)rows, mp = (size_t)dense_mpad(rows);
    BT_CUDA_TRY(dev_alloc(&r.proj, n * L->max_in));
    BT_CUDA_TRY(dev_alloc(&r.mix, n * L->max_mix));
    BT_CUDA_TRY(dev_alloc(&r.y, n * L->c.width));
    BT_CUDA_TRY(dev_alloc(&r.ff, n * L->max_ff));
    BT_CUDA_TRY(dev_alloc(&r.v_first, n * L->max_v));
    if (wide) {
        BT_CUDA_TRY(dev_alloc(&r.conv, n * L->max_channels));
        BT_CUDA_TRY(cudaMalloc(&r.q, std::max<size_t>(16, n * L->max_q * sizeof(float))));
        if (!L->f32) {
            size_t scratch = 0;
            for (const LayLayer& l : L->layers)
                for (const DenseLin* d : {&l.in, &l.o, &l.up, &l.down})
                    if (d->tiles) scratch = std::max(scratch, dense_tc_scratch(*d, std::min(rows, 128), m->sm_count));
            BT_CUDA_TRY(dev_alloc(&r.scratch, scratch));
            struct { uint8_t** p; int k; } tiles[] = {{&r.xt, L->c.width}, {&r.mt, L->max_mix}, {&r.ft, L->max_ff}};
            for (auto& t : tiles) {  // zeroed once: rows and columns of the padding stay finite
                const size_t bytes = mp * dense_kpad(std::max(t.k, 1)) * 2;
                BT_CUDA_TRY(dev_alloc(t.p, bytes));
                BT_CUDA_TRY(cudaMemset(*t.p, 0, bytes));
            }
            BT_CUDA_TRY(cudaDeviceSynchronize());
        }
    }
    r.rows = rows;
    return BT_OK;
}

DenseAttn attn_args(const bt_model* m, const LayLayer& l, const RowBuffers& r, int batch, int n) {
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
    a.kv = l.kv->dense;
    a.pos = m->pos;
    a.batch = batch; a.q_rows = n; a.heads = c.heads; a.n_kv = c.kv_heads; a.dk = c.dim; a.dv = c.vdim;
    a.sm_count = m->sm_count;
    a.q_buf = r.q;
    return a;
}
SsmArgs ssm_args(const bt_model* m, const LayLayer& l, const RowBuffers& r, int batch, int n) {
    const bt_layer_config& c = l.c;
    SsmArgs a;
    a.proj = r.proj;
    a.ld = l.in.n;
    a.conv_w = l.vec[BT_LT_SSM_CONV]; a.conv_b = l.vec[BT_LT_SSM_CONV_B];
    a.dt_bias = l.vec[BT_LT_SSM_DT_BIAS]; a.a_log = l.vec[BT_LT_SSM_A_LOG]; a.d = l.vec[BT_LT_SSM_D];
    a.heads = c.heads; a.vdim = c.vdim; a.state = c.state; a.groups = c.groups; a.taps = c.conv_taps;
    a.ring = l.ring; a.s = l.state; a.state_pad = l.state_pad();
    a.pos = m->pos;
    a.batch = batch; a.q_rows = n;
    a.conv_out = r.conv;
    a.y = r.mix;
    a.sm_count = m->sm_count;
    return a;
}

cudaError_t trace_stream(const bt_model* m, int layer, const float* h, int rows, cudaStream_t s) {
    if (!m->trace) return cudaSuccess;
    if (rows > m->trace_rows) return cudaErrorInvalidValue;
    const size_t W = (size_t)m->cfg.hidden_dim;
    return cudaMemcpyAsync(m->trace + (size_t)layer * m->trace_rows * W, h, (size_t)rows * W * sizeof(float), cudaMemcpyDeviceToDevice, s);
}

// The launches of a pass by what they do; a pass can be asked for some of them only (measurement aid).
enum Part : int { PART_IN = 1, PART_CORE = 2, PART_O = 4, PART_UP = 8, PART_DOWN = 16, PART_ROWS = 32, PART_ALL = 63 };

// One decode step for a few sequences: four or five dependent launches per attention layer, three per recurrent one.
// A sublayer's output norm and the residual sum are the prologue of the next projection, which reads the old stream
// and the un-normed output and leaves the new stream in the other buffer.
bt_status step_fused(bt_model* m, int batch, cudaStream_t s, int parts = PART_ALL) {
    Layered* L = m->lay;
    RowBuffers& r = L->dec;
    const int W = L->c.width, sm = m->sm_count;
    const float eps = L->c.norm_eps;
    float* cur = m->h;
    float* other = L->h2;
    const float* pending = nullptr;  // norm weight of the sublayer whose output waits in r.y
    if (parts & PART_ROWS)
        BT_CUDA_TRY(launch_embed_pos(m->tokens, m->embed, L->pos_table, m->pos, batch, 1, W, m->cfg.vocab_size, L->c.max_positions, cur, ActOut(), s, true));
    auto from_stream = [&](int part, const DenseLin& lin, float* out, int act) -> cudaError_t {
        DenseIn in;
        if (pending) {
            in.kind = DPRO_RESNORM; in.x = r.y; in.ld = W; in.w = pending; in.eps = eps; in.h = cur; in.h_out = other;
            std::swap(cur, other);
            pending = nullptr;
        } else {
            in.x = cur; in.ld = W;
        }
        if (!(parts & part)) return cudaSuccess;
        return launch_dense_stream(lin, in, batch, out, lin.n, act, sm, s, true);
    };
    RowArgs res;  // the residual sum on its own
    res.op = ROW_RESNORM; res.y = r.y; res.ld = W; res.eps = eps; res.rows = batch; res.k = W;
    for (size_t li = 0; li < L->layers.size(); ++li) {
        LayLayer& l = L->layers[li];
        BT_CUDA_TRY(from_stream(PART_IN, l.in, r.proj, DACT_NONE));
        DenseIn o;
        o.x = r.mix; o.ld = l.inner();
        if (l.c.mixer == BT_MIX_ATTENTION) {
            ActOut att;
            att.rows = r.mix; att.ld = l.inner();
            if (parts & PART_CORE) BT_CUDA_TRY(launch_attn_span(attn_args(m, l, r, batch, 1), false, att, s, true));
        } else {
            if (parts & PART_CORE) BT_CUDA_TRY(launch_ssm_step(ssm_args(m, l, r, batch, 1), s, true));
            o.kind = DPRO_GROUPNORM; o.w = l.vec[BT_LT_SSM_NORM]; o.eps = eps; o.groups = l.c.norm_groups;
        }
        if (parts & PART_O) BT_CUDA_TRY(launch_dense_stream(l.o, o, batch, r.y, W, DACT_NONE, sm, s, true));
        pending = l.vec[BT_LT_NORM1];
        if (l.c.mlp != BT_MLP_NONE) {
            BT_CUDA_TRY(from_stream(PART_UP, l.up, r.ff, DACT_RELU2));
            DenseIn d;
            d.x = r.ff; d.ld = l.c.ff;
            if (parts & PART_DOWN) BT_CUDA_TRY(launch_dense_stream(l.down, d, batch, r.y, W, DACT_NONE, sm, s, true));
            pending = l.vec[BT_LT_NORM2];
        }
        if (m->trace) {  // the stream after the layer, into the trace only
            if (batch > m->trace_rows) return set_error(BT_ERR_NOMEM, "the trace buffer holds fewer rows than sequences");
            res.w = pending; res.h_in = cur; res.h_out = m->trace + li * (size_t)m->trace_rows * W;
            BT_CUDA_TRY(launch_row_op(res, s, true));
        }
    }
    res.w = pending; res.h_in = cur; res.h_out = m->h;  // in place when the stream is there already
    if (parts & PART_ROWS) BT_CUDA_TRY(launch_row_op(res, s, true));
    return BT_OK;
}

// `n` new tokens for each of `batch` sequences, every stage its own kernel over all rows: tcgen05 products of bf16
// activations (f32 models: f32 products), attention by tiles of query positions.  The stream ends in h.
constexpr int kTileRowsMin = 16;  // new tokens per sequence from which the tile kernel pays
bt_status forward_rows(bt_model* m, const int32_t* tokens, float* h, RowBuffers& r, int batch, int n, cudaStream_t s,
                       int parts = PART_ALL) {
    Layered* L = m->lay;
    const int W = L->c.width, sm = m->sm_count, M = batch * n;
    const float eps = L->c.norm_eps;
    const bool f32 = L->f32;
    unsigned int* err = device_error_word(m->device);
    const int64_t mp = dense_mpad(M);
    auto tiled = [&](uint8_t* t) { ActOut o; o.tiles = t; o.m_pad = mp; return o; };
    auto plain = [&](float* p, int64_t ld) { ActOut o; o.rows = p; o.ld = ld; return o; };
    const ActOut xa = f32 ? ActOut() : tiled(r.xt);
    auto product = [&](int part, const DenseLin& lin, const uint8_t* xt, const float* x, float* out, uint8_t* ot, int act) -> cudaError_t {
        if (!(parts & part)) return cudaSuccess;
        return f32 ? launch_dense_f32(lin, x, lin.k, M, out, lin.n, act, s)
                   : launch_dense_tc(lin, xt, M, out, lin.n, ot, act, r.scratch, err, sm, s);
    };
    RowArgs res;
    res.op = ROW_RESNORM; res.y = r.y; res.ld = W; res.eps = eps; res.rows = M; res.k = W; res.h_in = h; res.h_out = h; res.act = xa;
    if (parts & PART_ROWS)
        BT_CUDA_TRY(launch_embed_pos(tokens, m->embed, L->pos_table, m->pos, batch, n, W, m->cfg.vocab_size, L->c.max_positions, h, xa, s, false));
    for (size_t li = 0; li < L->layers.size(); ++li) {
        LayLayer& l = L->layers[li];
        BT_CUDA_TRY(product(PART_IN, l.in, r.xt, h, r.proj, nullptr, DACT_NONE));
        const float* mixed = r.mix;
        if (l.c.mixer == BT_MIX_ATTENTION) {
            DenseAttn a = attn_args(m, l, r, batch, n);
            const ActOut out = f32 ? plain(r.mix, l.inner()) : tiled(r.mt);
            if (!(parts & PART_CORE)) {
            } else if (n >= kTileRowsMin && attn_tile_fits(a)) {
                a.q_bf16 = true;
                BT_CUDA_TRY(launch_attn_prep(a, s));
                BT_CUDA_TRY(launch_attn_tile(a, out, s));
            } else if (n == 1) {
                BT_CUDA_TRY(launch_attn_span(a, false, out, s, false));
            } else {
                BT_CUDA_TRY(launch_attn_prep(a, s));
                BT_CUDA_TRY(launch_attn_span(a, true, out, s, false));
            }
        } else {
            SsmArgs a = ssm_args(m, l, r, batch, n);
            if (parts & PART_CORE) BT_CUDA_TRY(n == 1 ? launch_ssm_step(a, s, false) : launch_ssm_prefill(a, !f32, s));
            RowArgs g;
            g.op = ROW_GROUPNORM; g.y = r.mix; g.ld = l.inner(); g.w = l.vec[BT_LT_SSM_NORM]; g.eps = eps; g.groups = l.c.norm_groups;
            g.rows = M; g.k = l.inner();
            g.act = f32 ? plain(r.proj, l.inner()) : tiled(r.mt);  // the projection rows are used up
            if (parts & PART_ROWS) BT_CUDA_TRY(launch_row_op(g, s, false));
            mixed = r.proj;
        }
        BT_CUDA_TRY(product(PART_O, l.o, r.mt, mixed, r.y, nullptr, DACT_NONE));
        res.w = l.vec[BT_LT_NORM1];
        if (parts & PART_ROWS) BT_CUDA_TRY(launch_row_op(res, s, false));
        if (l.c.mlp != BT_MLP_NONE) {
            BT_CUDA_TRY(product(PART_UP, l.up, r.xt, h, r.ff, f32 ? nullptr : r.ft, DACT_RELU2));
            BT_CUDA_TRY(product(PART_DOWN, l.down, r.ft, r.ff, r.y, nullptr, DACT_NONE));
            res.w = l.vec[BT_LT_NORM2];
            if (parts & PART_ROWS) BT_CUDA_TRY(launch_row_op(res, s, false));
        }
        BT_CUDA_TRY(trace_stream(m, (int)li, h, M, s));
    }
    return BT_OK;
}

bool step_is_fused(const bt_model* m, int batch) { return batch <= m->lay->fused_rows; }

}  // namespace

bt_status layered_step(bt_model* m, int batch, cudaStream_t s) {
    return step_is_fused(m, batch) ? step_fused(m, batch, s) : forward_rows(m, m->tokens, m->h, m->lay->dec, batch, 1, s);
}

bt_status layered_prefill(bt_model* m, int batch, int n, cudaStream_t s) {
    return forward_rows(m, m->pf_tokens, m->pf_h, m->lay->pf, batch, n, s);
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
    const int64_t expect = kind == BT_T_POS ? (int64_t)L->c.max_positions * W : VW;
    if ((kind != BT_T_EMBED && kind != BT_T_LM_HEAD && kind != BT_T_POS) || n_elem != expect || expect == 0)
        return set_error(BT_ERR_SHAPE, "bt_model_set_tensor: tensor %d with %lld elements, %lld expected", (int)kind, (long long)n_elem, (long long)expect);
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

bt_status layered_finalize(bt_model* m) {
    Layered* L = m->lay;
    if (!m->embed || !m->lm_head || !m->norm_f || (L->c.max_positions > 0 && !L->pos_table))
        return set_error(BT_ERR_ARG, "bt_model_finalize: embedding, positions, lm_head or final norm missing");
    for (size_t i = 0; i < L->layers.size(); ++i)
        for (int k = 0; k < kTensorKinds; ++k)
            if (tensor_elems(L, L->layers[i], k) > 0 && !(L->layers[i].set >> k & 1u))
                return set_error(BT_ERR_ARG, "bt_model_finalize: tensor %d of layer %d was never set", k, (int)i);
    const int B = L->c.max_batch, W = L->c.width;
    bt_status st;
    L->fused_rows = std::min(8, B);
    for (LayLayer& l : L->layers) {
        L->max_in = std::max(L->max_in, l.in.n);
        L->max_mix = std::max(L->max_mix, l.inner());
        L->max_ff = std::max(L->max_ff, l.up.n);
        for (const DenseLin* d : {&l.in, &l.o, &l.up, &l.down})
            while (d->tiles && L->fused_rows > 0 && !dense_stream_fits(*d, L->fused_rows)) --L->fused_rows;
        if (l.c.mixer == BT_MIX_ATTENTION) {
            if ((st = bt_kv_create_dense(&l.kv, B, l.c.kv_heads, l.c.dim, l.c.vdim, L->c.max_seq_len, L->f32 ? BT_F32 : BT_BF16, m->device)) != BT_OK) return st;
            L->max_q = std::max(L->max_q, l.c.heads * l.kv->dense.k_stride);
            L->max_v = std::max(L->max_v, l.v_width());
        } else {
            L->max_channels = std::max(L->max_channels, (int)ssm_conv_floats(ssm_args(m, l, L->dec, 1, 1)));
            BT_CUDA_TRY(dev_alloc(&l.state, (size_t)B * l.inner() * l.state_pad()));
            BT_CUDA_TRY(dev_alloc(&l.ring, (size_t)B * l.c.conv_taps * l.channels()));
        }
    }
    m->rms_eps = L->c.norm_eps;
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
        for (DenseLin* d : {&l.in, &l.o, &l.up, &l.down}) cudaFree(d->tiles);
        for (float* v : l.vec) cudaFree(v);
        bt_kv_destroy(l.kv);
        cudaFree(l.state); cudaFree(l.ring);
    }
    L->dec.release();
    L->pf.release();
    cudaFree(L->pos_table); cudaFree(L->h2);
    delete L;
    m->lay = nullptr;
}

bt_status layered_reset(bt_model* m) {
    for (LayLayer& l : m->lay->layers) {
        if (l.kv) { bt_status st = bt_kv_reset(l.kv); if (st != BT_OK) return st; }
        const size_t B = (size_t)m->cfg.max_batch;
        if (l.state) BT_CUDA_TRY(cudaMemset(l.state, 0, B * l.inner() * l.state_pad() * sizeof(float)));
        if (l.ring) BT_CUDA_TRY(cudaMemset(l.ring, 0, B * l.c.conv_taps * l.channels() * sizeof(float)));
    }
    return BT_OK;
}

int layered_launches(const bt_model* m, int batch) {
    const Layered* L = m->lay;
    const bool fused = step_is_fused(m, batch);
    int n = 1 + (fused ? 1 : 0);  // embedding; fused: the last residual sum
    auto product = [&](const DenseLin& d) { return fused || L->f32 ? 1 : dense_tc_kernels(d, batch, m->sm_count); };
    for (const LayLayer& l : L->layers) {
        n += product(l.in) + 1 + product(l.o);
        if (l.c.mlp != BT_MLP_NONE) n += product(l.up) + product(l.down);
        if (!fused) n += 1 + (l.c.mixer == BT_MIX_SSM ? 1 : 0) + (l.c.mlp != BT_MLP_NONE ? 1 : 0);
    }
    if (m->lm_tiles && batch > 8) return n + 4;  // prepare, product, arg-max, position advance
    return n + (batch <= 4 ? 1 : (batch + 7) / 8) + 1;
}

bt_kv_cache* layered_kv(bt_model* m, int layer) {
    return layer < 0 || layer >= (int)m->lay->layers.size() ? nullptr : m->lay->layers[(size_t)layer].kv;
}

}  // namespace bt

using namespace bt;

extern "C" bt_status bt_model_enqueue_parts(bt_model* m, int batch, int n_tokens, int parts, void* stream) {
    if (!m || !m->lay || !m->finalized) return set_error(BT_ERR_ARG, "bt_model_enqueue_parts: not a finalized layer-list model");
    if (batch < 1 || batch > m->cfg.max_batch || n_tokens < 1 || (n_tokens > 1 && (int64_t)batch * n_tokens > m->pf_rows))
        return set_error(BT_ERR_SHAPE, "bt_model_enqueue_parts: %d sequences of %d tokens (prefill that many first)", batch, n_tokens);
    DeviceGuard guard(m->device);
    cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
    if (n_tokens > 1) return forward_rows(m, m->pf_tokens, m->pf_h, m->lay->pf, batch, n_tokens, s, parts);
    return step_is_fused(m, batch) ? step_fused(m, batch, s, parts) : forward_rows(m, m->tokens, m->h, m->lay->dec, batch, 1, s, parts);
}

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
    int v_width = 0;
    for (int i = 0; i < c.num_layers; ++i) {
        const bt_layer_config& l = layers[i];
        if (l.heads < 1 || l.vdim < 1) return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: no heads", i);
        if (l.mixer == BT_MIX_ATTENTION) {
            if (l.kv_heads < 1 || l.heads % l.kv_heads != 0 || l.dim < 1)
                return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: %d query heads over %d KV heads of size %d", i, l.heads, l.kv_heads, l.dim);
            if (l.vdim > attn_max_dim() || l.dim > attn_max_dim())
                return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: key and value heads of %d and %d, at most %d", i, l.dim, l.vdim, attn_max_dim());
            if (l.q_temp_coef != 0.0f && !(l.q_temp_every > 0.0)) return set_error(BT_ERR_ARG, "bt_model_create_layers: layer %d: q_temp_every must be positive", i);
            if (l.v_mix) {
                if (v_width && v_width != l.kv_heads * l.vdim) return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: value mixing between layers of different value size", i);
                v_width = l.kv_heads * l.vdim;
            }
        } else if (l.mixer == BT_MIX_SSM) {
            if (l.groups < 1 || l.heads % l.groups != 0 || !ssm_state_pad(l.state) || l.conv_taps < 1 || l.norm_groups < 1 ||
                (l.heads * l.vdim) % l.norm_groups != 0)
                return set_error(BT_ERR_SHAPE, "bt_model_create_layers: layer %d: %d heads, %d groups, state %d, %d taps, %d norm groups", i, l.heads, l.groups, l.state, l.conv_taps, l.norm_groups);
        } else {
            return set_error(BT_ERR_ARG, "bt_model_create_layers: layer %d: unknown mixer %d", i, l.mixer);
        }
        if (l.mlp != BT_MLP_NONE && (l.mlp != BT_MLP_DENSE_RELU2 || l.ff < 1))
            return set_error(BT_ERR_ARG, "bt_model_create_layers: layer %d: unknown feed-forward %d of width %d", i, l.mlp, l.ff);
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
        bt_status st;
        if (l.c.mixer == BT_MIX_ATTENTION) {
            l.v_source = l.c.v_mix && !source;
            l.v_target = l.c.v_mix && source;
            source |= l.c.v_mix != 0;
            st = alloc_lin(l.in, l.c.heads * l.c.dim + l.c.kv_heads * (l.c.dim + l.c.vdim), c.width);
        } else {
            st = alloc_lin(l.in, l.inner() + l.channels() + l.c.heads, c.width);
        }
        if (st == BT_OK) st = alloc_lin(l.o, c.width, l.inner());
        if (st == BT_OK && l.c.mlp != BT_MLP_NONE) st = alloc_lin(l.up, l.c.ff, c.width);
        if (st == BT_OK && l.c.mlp != BT_MLP_NONE) st = alloc_lin(l.down, c.width, l.c.ff);
        if (st != BT_OK) { bt_model_destroy(m); return st; }
    }
    *out = m;
    return BT_OK;
}

extern "C" bt_status bt_model_set_layer_tensor(bt_model* m, int layer, bt_layer_tensor kind, const float* data, int64_t n_elem) {
    if (!m || !data || !m->lay) return set_error(BT_ERR_ARG, "bt_model_set_layer_tensor: null pointer or not a layer-list model");
    if (m->finalized) return set_error(BT_ERR_ARG, "bt_model_set_layer_tensor: model already finalized");
    if (layer < 0 || layer >= m->cfg.num_layers || (int)kind < 0 || (int)kind >= kTensorKinds)
        return set_error(BT_ERR_ARG, "bt_model_set_layer_tensor: layer %d / tensor %d out of range", layer, (int)kind);
    Layered* L = m->lay;
    LayLayer& l = L->layers[(size_t)layer];
    const int64_t expect = tensor_elems(L, l, kind);
    if (expect == 0 || n_elem != expect)
        return set_error(BT_ERR_SHAPE, "bt_model_set_layer_tensor: layer %d tensor %d has %lld elements, %lld expected", layer, (int)kind, (long long)n_elem, (long long)expect);
    DeviceGuard guard(m->device);
    const bt_layer_config& c = l.c;
    const int nq = c.heads * c.dim, nk = c.kv_heads * c.dim;
    bt_status st = BT_OK;
    switch (kind) {
        case BT_LT_Q: st = upload_rows(l.in, data, nq, 0); break;
        case BT_LT_K: st = upload_rows(l.in, data, nk, nq); break;
        case BT_LT_V: st = upload_rows(l.in, data, c.kv_heads * c.vdim, nq + nk); break;
        case BT_LT_SSM_IN: st = upload_rows(l.in, data, l.in.n, 0); break;
        case BT_LT_O: case BT_LT_SSM_O: st = upload_rows(l.o, data, l.o.n, 0); break;
        case BT_LT_MLP_UP: st = upload_rows(l.up, data, l.up.n, 0); break;
        case BT_LT_MLP_DOWN: st = upload_rows(l.down, data, l.down.n, 0); break;
        case BT_LT_VMIX: l.vmix = data[0]; break;
        case BT_LT_NORM1: case BT_LT_NORM2: st = upload_vec(&l.vec[kind], data, n_elem, L->c.norm_one_plus ? 1.0f : 0.0f); break;
        default: st = upload_vec(&l.vec[kind], data, n_elem, 0.0f); break;
    }
    if (st == BT_OK) l.set |= 1u << (int)kind;
    return st;
}

extern "C" float* bt_model_recurrent_state(bt_model* m, int layer, int64_t* n_floats) {
    if (n_floats) *n_floats = 0;
    if (!m || !m->lay || layer < 0 || layer >= m->cfg.num_layers) return nullptr;
    LayLayer& l = m->lay->layers[(size_t)layer];
    if (n_floats && l.state) *n_floats = (int64_t)m->cfg.max_batch * l.inner() * l.state_pad();
    return l.state;
}
extern "C" float* bt_model_conv_ring(bt_model* m, int layer, int64_t* n_floats) {
    if (n_floats) *n_floats = 0;
    if (!m || !m->lay || layer < 0 || layer >= m->cfg.num_layers) return nullptr;
    LayLayer& l = m->lay->layers[(size_t)layer];
    if (n_floats && l.ring) *n_floats = (int64_t)m->cfg.max_batch * l.c.conv_taps * l.channels();
    return l.ring;
}
