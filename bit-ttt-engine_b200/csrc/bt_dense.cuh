// Building blocks of decoders with dense 16-bit projections and a per-layer choice of mixer (softmax attention with
// capped scores and a sink, state-space recurrence): weight and activation layouts, launchers.
#pragma once

#include "bt_common.cuh"

namespace bt {

// ---------------------------------------------------------------------------------------
// Dense matrices [rows, k] in bf16, "tiled": blocks of 64 inputs, inside a block groups of 8 rows (1024 bytes each),
// inside a group 8 core matrices of 8 rows x 16 bytes.  Any run of row groups of one block is contiguous, so that
//  - a warp of the streaming product reads 1024 consecutive bytes = 8 rows x 64 inputs with two 16-byte loads per lane,
//  - an operand tile of the tcgen05 product (128 rows or up to 256 tokens, K-major, no swizzle) is one bulk copy.
// Weights and activations share the layout; rows are padded to rows_pad, inputs to a multiple of 64 (weights: zeros).
// ---------------------------------------------------------------------------------------
constexpr int kDenseK = 64;
__host__ __device__ inline int64_t dense_off(int64_t row, int c, int64_t rows_pad) {  // byte offset
    return (int64_t)(c >> 6) * rows_pad * 128 + (row >> 3) * 1024 + ((c & 63) >> 3) * 128 + (row & 7) * 16 + (c & 7) * 2;
}
__host__ __device__ inline int dense_kpad(int k) { return (k + kDenseK - 1) / kDenseK * kDenseK; }

struct DenseLin {
    uint8_t* tiles = nullptr;  // device
    int n = 0, k = 0;
    int n_pad = 0, k_pad = 0;  // multiples of 128 and 64
    size_t bytes() const { return (size_t)n_pad * k_pad * 2; }
};

// f32 rows [rows, k] on the device -> rows [row0, row0 + rows) of the tiled matrix
cudaError_t launch_dense_tile(const float* src, int rows, int k, int row0, const DenseLin& lin, cudaStream_t s);

// Where a kernel leaves activations for the next projection: f32 rows, or bf16 in the tiled layout.
struct ActOut {
    float* rows = nullptr;
    int64_t ld = 0;
    uint8_t* tiles = nullptr;
    int64_t m_pad = 0;
};
inline int64_t dense_mpad(int64_t m) { return m <= 64 ? 64 : (m <= 128 ? 128 : (m + 255) / 256 * 256); }

enum DenseAct : int { DACT_NONE = 0, DACT_RELU2 = 1 };

// How the streaming product (<= 8 rows) obtains its input rows.
enum DensePro : int {
    DPRO_ROWS = 0,      // x[b, c] as it is
    DPRO_RESNORM = 1,   // h[b, c] + (x[b, :] / rms(x[b, :]))[c] * w[c]; block 0 also writes the sum to h_out
    DPRO_GROUPNORM = 2  // x / rms (per equal part of the row) * w
};
struct DenseIn {
    int kind = DPRO_ROWS;
    const float* x = nullptr;
    int64_t ld = 0;
    const float* w = nullptr;
    float eps = 0.f;
    int groups = 1;
    const float* h = nullptr;  // DPRO_RESNORM: the residual stream, rows of k floats
    float* h_out = nullptr;
};
// out[b, n] = act(W x), all arithmetic in f32 on the bf16 weights; rows <= 8 and rows * k_pad * 4 within shared memory.
bool dense_stream_fits(const DenseLin& lin, int rows);
cudaError_t launch_dense_stream(const DenseLin& lin, const DenseIn& in, int rows, float* out, int64_t ld, int act,
                                int sm_count, cudaStream_t s, bool pdl);

// tcgen05 product of tiled bf16 activations; f32 accumulation.  Output: act(.) as f32 rows (out) or as tiled bf16
// activations (out_tiles).  With few row tiles the inputs are cut over several CTAs, whose partial sums go through
// `scratch` (dense_tc_scratch floats) and are added in a fixed order.
size_t dense_tc_scratch(const DenseLin& lin, int64_t m, int sm_count);
int dense_tc_kernels(const DenseLin& lin, int64_t m, int sm_count);
cudaError_t launch_dense_tc(const DenseLin& lin, const uint8_t* x_tiles, int64_t m, float* out, int64_t ld,
                            uint8_t* out_tiles, int act, float* scratch, unsigned int* err, int sm_count, cudaStream_t s);

// f32 product of f32 rows (no tensor cores), for 32-bit models
cudaError_t launch_dense_f32(const DenseLin& lin, const float* x, int64_t ldx, int64_t m, float* out, int64_t ld, int act,
                             cudaStream_t s);

// ---------------------------------------------------------------------------------------
// Row kernels
// ---------------------------------------------------------------------------------------
// h = table[token] (+ pos_table[pos[b] + i]); rows ordered [sequence][token], q_rows tokens per sequence
cudaError_t launch_embed_pos(const int32_t* tokens, const __nv_bfloat16* table, const __nv_bfloat16* pos_table,
                             const int32_t* pos, int batch, int q_rows, int hidden, int vocab, int max_pos, float* h,
                             const ActOut& act, cudaStream_t s, bool pdl);

// RESNORM: h_out = h_in + y / rms(y) * w (in place allowed), act = h_out;
// GROUPNORM: act = y / rms per part * w.
enum RowOp : int { ROW_RESNORM = 0, ROW_GROUPNORM = 1 };
struct RowArgs {
    int op = ROW_RESNORM;
    const float* y = nullptr;
    int64_t ld = 0;
    const float* w = nullptr;
    float eps = 0.f;
    int groups = 1;
    const float* h_in = nullptr;
    float* h_out = nullptr;
    int64_t rows = 0;
    int k = 0;
    ActOut act;
};
cudaError_t launch_row_op(const RowArgs& a, cudaStream_t s, bool pdl);

// ---------------------------------------------------------------------------------------
// Attention over a 16- or 32-bit cache
// ---------------------------------------------------------------------------------------
struct DenseKvView {
    void* k = nullptr;  // [batch, n_kv, max_seq, k_stride] bf16 or f32, zero beyond k_dim
    void* v = nullptr;  // [batch, n_kv, max_seq, v_stride]
    int max_seq = 0, k_stride = 0, v_stride = 0;
    bool f32 = false;
};

struct DenseAttn {
    // the projections q | k | v of the new tokens: rows of (H dk + G dk + G dv) floats
    const float* qkv = nullptr;
    int64_t ld = 0;
    const float* q_norm = nullptr;  // [H dk] norm over the whole query row (null: none); likewise k_norm [G dk]
    const float* k_norm = nullptr;
    float eps = 0.f;
    float temp_coef = 0.f;          // q *= 1 + coef * ln(floor((pos + 1) / every) + 1)
    double temp_every = 1.0;
    int temp_every_int = 0;         // the same where it is a whole number, else 0
    float v_lambda = 0.f;           // v = (1 - lambda) v + lambda v_first, when v_first_in is set
    const float* v_first_in = nullptr;
    float* v_first_out = nullptr;   // the projected v of the new tokens is kept here for later layers
    float scale = 1.f, softcap = 0.f;  // softcap 0: none
    const float* sink = nullptr;    // [H], null: none
    DenseKvView kv;
    const int32_t* pos = nullptr;   // [batch] position of the first new token
    int batch = 1, q_rows = 1, heads = 1, n_kv = 1, dk = 0, dv = 0;
    int sm_count = 0;
    void* q_buf = nullptr;          // prefill: prepared queries [rows, H, k_stride], bf16 (tile kernel) or f32
    bool q_bf16 = false;
};
// Query and key norm, temperature, value mixing; keys and values go to the cache, queries to q_buf.
cudaError_t launch_attn_prep(const DenseAttn& a, cudaStream_t s);
// One new token per CTA group.  prepared = false (q_rows == 1): the preparation runs inside the kernel.
cudaError_t launch_attn_span(const DenseAttn& a, bool prepared, const ActOut& out, cudaStream_t s, bool pdl);
// Tiles of query positions on the tensor cores (bf16 cache, prepared bf16 queries)
bool attn_tile_fits(const DenseAttn& a);
cudaError_t launch_attn_tile(const DenseAttn& a, const ActOut& out, cudaStream_t s);
int attn_max_dim();  // of query/key and of value heads

// ---------------------------------------------------------------------------------------
// State-space recurrence (per head: S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x)
// ---------------------------------------------------------------------------------------
struct SsmArgs {
    const float* proj = nullptr;   // rows z | x | B | C | dt
    int64_t ld = 0;
    const float* conv_w = nullptr; // [channels, taps], channels = inner + 2 groups state
    const float* conv_b = nullptr;
    const float* dt_bias = nullptr;
    const float* a_log = nullptr;
    const float* d = nullptr;
    int heads = 1, vdim = 1, state = 1, groups = 1, taps = 1;
    float* ring = nullptr;         // [batch, taps, channels] last inputs of the convolution, slot = position % taps
    float* s = nullptr;            // [batch, heads, vdim, state_pad] f32
    int state_pad = 0;
    const int32_t* pos = nullptr;
    int batch = 1, q_rows = 1;
    float* conv_out = nullptr;     // prefill: x | B | C of the rows after convolution and silu
    float* y = nullptr;            // [rows, inner] (S^T C + D x) * silu(z)
    int sm_count = 0;
};
int ssm_state_pad(int state);     // 0: not supported
cudaError_t launch_ssm_step(const SsmArgs& a, cudaStream_t s, bool pdl);     // q_rows == 1
int64_t ssm_conv_floats(const SsmArgs& a);  // floats per row that conv_out needs
// bf16: 64 tokens at a time on the tensor cores, convolution outputs in bf16; else token by token in f32
cudaError_t launch_ssm_prefill(const SsmArgs& a, bool bf16, cudaStream_t s);

}  // namespace bt
