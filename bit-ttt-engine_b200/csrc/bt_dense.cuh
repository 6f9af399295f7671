// Building blocks of decoders with dense 16-bit projections and a per-layer choice of mixer (softmax attention with
// capped scores and a sink, latent attention, three recurrences) and feed-forward (dense, mixture of experts): weight and
// activation layouts, launchers.
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

// One matrix, or `blocks` matrices of one shape behind one another: the diagonal blocks of a block-diagonal matrix, the
// experts of a mixture.
struct DenseLin {
    uint8_t* tiles = nullptr;  // device
    int n = 0, k = 0;          // of one block
    int n_pad = 0, k_pad = 0;  // multiples of 128 and 64
    int blocks = 1;
    size_t block_bytes() const { return (size_t)n_pad * k_pad * 2; }
    size_t bytes() const { return (size_t)blocks * block_bytes(); }
    int chunks() const { return k_pad / kDenseK; }
};

// f32 rows [rows, k] on the device -> rows row0, row0 + row_step, ... of a block of the tiled matrix
cudaError_t launch_dense_tile(const float* src, int rows, int k, int row0, const DenseLin& lin, cudaStream_t s, int row_step = 1,
                              int block = 0);

// Where a kernel leaves activations for the next projection: f32 rows, or bf16 in the tiled layout.
struct ActOut {
    float* rows = nullptr;
    int64_t ld = 0;
    uint8_t* tiles = nullptr;
    int64_t m_pad = 0;
};
inline int64_t dense_mpad(int64_t m) { return m <= 64 ? 64 : (m <= 128 ? 128 : (m + 255) / 256 * 256); }

// SWIGLU: rows 2j and 2j + 1 of the matrix are gate j and up j, the product has n / 2 outputs silu(gate) * up.
// RGLRU: rows 2j and 2j + 1 are the two gates of channel j (streaming product only, behind DPRO_CONV).  DECAY: exp(-exp(v)).
enum DenseAct : int { DACT_NONE = 0, DACT_RELU2 = 1, DACT_TANH = 2, DACT_DECAY = 3, DACT_SWIGLU = 4, DACT_RGLRU = 5 };
inline int dense_outputs(const DenseLin& lin, int act) { return act >= DACT_SWIGLU ? lin.n / 2 : lin.n; }

// The gated linear recurrence of one token per sequence:
// S <- a S + sqrt(1 - a^2) i u, a = exp(-8 r softplus(lam)), output S * gelu_tanh(y); r, i sigmoids of the gates
struct RgluStep {
    const float* y = nullptr;   // rows of stride ld
    const float* lam = nullptr;
    float* state = nullptr;     // [batch, channels]
};

// How the streaming product (<= 8 rows) obtains its input rows.
enum DensePro : int {
    DPRO_ROWS = 0,       // x[b, c] as it is
    DPRO_RESNORM = 1,    // h[b, c] + (x[b, :] / rms(x[b, :]))[c] * w[c]; block 0 also writes the sum to h_out
    DPRO_GROUPNORM = 2,  // x / rms (per equal part of the row) * w
    DPRO_CONV = 3        // causal convolution per channel over x and the ring of earlier inputs; the first CTA of a block of
                         // channels also stores the new inputs
};
struct DenseIn {
    int kind = DPRO_ROWS;
    const float* x = nullptr;
    int64_t ld = 0;
    int64_t x_block = 0;       // block-diagonal products: columns from one block's input to the next
    const float* w = nullptr;
    float eps = 0.f;
    int groups = 1;
    const float* h = nullptr;  // DPRO_RESNORM: the residual stream, rows of k floats
    float* h_out = nullptr;
    const float* next_w = nullptr;  // DPRO_RESNORM: the sum goes through another norm before the product
    float* n_out = nullptr;    // block 0 writes the product's input rows here
    int kx = 0;                // columns of x where it is only the front part of the input; `cat` rows of as many columns follow
    const float* cat = nullptr;  // at the next multiple of 64
    float* shift = nullptr;    // token shift (segments with mu): [2][max_batch][k] inputs by parity of the position
    int64_t shift_slot = 0;
    const int32_t* pos = nullptr;
    float* ring = nullptr;     // DPRO_CONV: [batch, taps, channels], slot = position % taps
    const float* conv_w = nullptr;
    const float* conv_b = nullptr;
    int taps = 1, channels = 0;
    RgluStep rg;               // DACT_RGLRU
};
// Rows of a streaming product that belong together; up to kMaxSegs products of one input run as one launch.
constexpr int kMaxSegs = 5;
struct DenseSeg {
    const DenseLin* lin = nullptr;
    float* out = nullptr;
    int64_t ld = 0;
    int act = DACT_NONE;
    const float* bias = nullptr;  // [blocks, n]
    const float* mu = nullptr;    // [k]: the segment reads x + (x of the token before - x) * mu
    int64_t out_block = 0;        // block-diagonal products: columns from one block's outputs to the next
};
// out[b, n] = act(W x + bias), all arithmetic in f32 on the bf16 weights; rows <= 8 and rows * k_pad * 4 within shared memory.
bool dense_stream_fits(const DenseLin& lin, int rows);
cudaError_t launch_dense_stream(const DenseLin& lin, const DenseIn& in, int rows, float* out, int64_t ld, int act,
                                int sm_count, cudaStream_t s, bool pdl);
cudaError_t launch_dense_stream_segs(const DenseSeg* segs, int nseg, const DenseIn& in, int rows, int sm_count, cudaStream_t s, bool pdl);

// Rows of a mixture of experts, grouped by expert: blocks of up to `tile` rows of one expert each, made on the device.
struct ExpertTile {
    int expert, row0, row_end, pad;
};
struct ExpertPlan {
    const ExpertTile* tiles = nullptr;  // device
    const int* n_tiles = nullptr;       // device
    const int* row_start = nullptr;     // device [experts + 1]
    const int* counts = nullptr;        // device [experts]
    int tile = 0;                       // rows per tile: 64, 128 or 256
    int max_tiles = 0;                  // upper bound, for launch shapes
    int max_rows = 0;                   // rows one expert can have
};

// What a product over many rows does besides W x: every field but `out` / `out_tiles` / `out_rows16` is optional.
struct DenseOut {
    float* out = nullptr;              // f32 rows
    int64_t ld = 0;
    uint8_t* out_tiles = nullptr;      // or bf16 in the tiled layout
    __nv_bfloat16* out_rows16 = nullptr;  // or bf16 rows of stride ld (a multiple of 8)
    int act = DACT_NONE;
    const float* bias = nullptr;       // [blocks, n]
    int64_t out_block = 0;             // columns (out, out_tiles) or elements (out_rows16) from one block's outputs to the next
    bool shared_weights = false;       // every block has its own input and output, the matrix is one
    int blocks = 0;                    // with shared_weights: their number
    int64_t x_block = 0;               // with shared_weights: bytes from one block's input tiles to the next
    int64_t m_pad = 0;                 // rows the input tiles are padded to (0: dense_mpad(m))
    int halves = 1;                    // 2: the input is hi | lo bf16, kpad(k) columns each (per block)
    const ExpertPlan* plan = nullptr;  // blocks are experts; rows by the plan
};
// tcgen05 product of tiled bf16 activations; f32 accumulation.  With few row tiles the inputs of a plain product are cut
// over several CTAs, whose partial sums go through `scratch` (dense_tc_scratch floats) and are added in a fixed order.
// Block-diagonal products: block b reads the columns b * halves * kpad(k) .. of the input.
size_t dense_tc_scratch(const DenseLin& lin, int64_t m, int sm_count);
int dense_tc_kernels(const DenseLin& lin, int64_t m, int sm_count, int act = DACT_NONE);
cudaError_t launch_dense_tc(const DenseLin& lin, const uint8_t* x_tiles, int64_t m, const DenseOut& o, float* scratch,
                            unsigned int* err, int sm_count, cudaStream_t s);

// f32 product of f32 rows (no tensor cores), for 32-bit models; block b reads the columns b * x_block ..
cudaError_t launch_dense_f32(const DenseLin& lin, const float* x, int64_t ldx, int64_t x_block, int64_t m, const DenseOut& o,
                             cudaStream_t s);

// ---------------------------------------------------------------------------------------
// Row kernels
// ---------------------------------------------------------------------------------------
// h = table[token] (+ pos_table[pos[b] + i]); rows ordered [sequence][token], q_rows tokens per sequence
cudaError_t launch_embed_pos(const int32_t* tokens, const __nv_bfloat16* table, const __nv_bfloat16* pos_table,
                             const int32_t* pos, int batch, int q_rows, int hidden, int vocab, int max_pos, float* h,
                             const ActOut& act, cudaStream_t s, bool pdl, const ActOut& act2 = ActOut());

// RESNORM: h_out = h_in + y / rms(y) * w (in place allowed), act = h_out, or h_out / rms(h_out) * next_w;
//          y may be a mixture: y + sum_j wt[row, j] * ye[dst[row, j]]
// GROUPNORM: act = y / rms per part * w (* silu(gate)).
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
    const float* next_w = nullptr;
    const float* ye = nullptr;    // rows of ye_ld floats
    int64_t ye_ld = 0;
    const int* dst = nullptr;     // [rows, top]
    const float* wt = nullptr;
    int top = 0;
    const float* gate = nullptr;  // rows of gate_ld floats
    int64_t gate_ld = 0;
    int64_t rows = 0;
    int k = 0;
    ActOut act;
};
cudaError_t launch_row_op(const RowArgs& a, cudaStream_t s, bool pdl);
// f32 rows of `blocks` parts of k columns (part stride x_block) -> tiled bf16, every part padded to a multiple of 64 columns;
// halves = 2: hi | lo
cudaError_t launch_rows_tile(const float* x, int64_t ld, int64_t x_block, int blocks, int k, int halves, int act, int64_t rows,
                             uint8_t* tiles, int64_t m_pad, cudaStream_t s);

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
// Latent attention: keys and values of all heads are products of one latent row per position, one rotated key part is
// shared by the heads
// ---------------------------------------------------------------------------------------
// f32 models: rows of `stride` floats.  bf16: groups of 8 positions, inside a group core matrices of 8 positions x 16 bytes over
// the columns, latent [rank padded to 16] | rotated part [rot padded to 16]; a run of groups is contiguous.
struct LatentView {
    void* rows = nullptr;
    int max_seq = 0, seq_pad = 0, rank = 0, rot = 0, stride = 0;
    bool f32 = false;
    __host__ __device__ int rot_col() const { return (rank + 15) / 16 * 16; }
    __host__ __device__ int cols() const { return rot_col() + (rot + 15) / 16 * 16; }
    __host__ __device__ int64_t seq_bytes() const { return f32 ? (int64_t)max_seq * stride * 4 : (int64_t)seq_pad * cols() * 2; }
    __host__ __device__ int64_t off(int64_t pos, int c) const { return (pos >> 3) * cols() * 16 + (c >> 3) * 128 + (pos & 7) * 16 + (c & 7) * 2; }  // bytes
};
struct LatentAttn {
    const float* proj = nullptr;   // rows q [heads][dim | rot] | latent [rank] | rotated key part [rot] | output gates [heads]
    int64_t ld = 0;
    const float* c_norm = nullptr; // [rank]
    float eps = 0.f, scale = 1.f;
    bool gate = false;
    const float* cos_t = nullptr;  // [max_seq, rot_dims / 2]
    const float* sin_t = nullptr;
    int heads = 1, dim = 0, rot = 0, rot_dims = 0, vdim = 0, rank = 0;
    LatentView kv;
    const int32_t* pos = nullptr;
    int batch = 1, q_rows = 1, sm_count = 0;
    float* q_abs = nullptr;        // [rows][heads][rank]: the queries' unrotated part times the key matrix
    float* q_rot = nullptr;        // prepared: rotated parts [rows][heads][rot]
    uint8_t* q_tiles = nullptr;    // prepared: unrotated parts as tiled hi | lo blocks (bf16) ...
    float* q_rows32 = nullptr;     // ... or f32 rows [rows][heads][dim]
    __nv_bfloat16* q_buf = nullptr;  // tile kernel: [rows][heads][pad8(dim) + pad8(rot)]
    int64_t m_pad = 0;
};
// latents of positions [0, n) of `nb` sequences -> tiled activations [nb][kpad(rank) / 64][m_pad][64]
cudaError_t launch_latent_tiles(const LatentView& v, int b0, int nb, int64_t n, uint8_t* tiles, int64_t m_pad, cudaStream_t s);
// New tokens: latents normed, key parts rotated, both into the cache; queries to q_buf, or to q_rot and q_tiles / q_rows32
cudaError_t launch_latent_prep(const LatentAttn& a, cudaStream_t s);
// Attention over the latents (absorbed queries), one query position per CTA group; output rows [heads][rank], weighted by
// sigmoid(gate).  out.tiles: blocks of kpad(rank) columns per head.  prepared = false (q_rows == 1): the kernel rotates and
// appends itself.
cudaError_t launch_latent_span(const LatentAttn& a, bool prepared, const ActOut& out, cudaStream_t s, bool pdl);
// Tiles of query positions over expanded keys and values of `nb` sequences from b0: kv16 [nb][kv_rows][heads pad8(dim) |
// heads pad8(vdim)] bf16 rows; the rotated key parts come from the cache.
bool latent_tile_fits(const LatentAttn& a);
cudaError_t launch_latent_tile(const LatentAttn& a, const __nv_bfloat16* kv16, int64_t kv_rows, int b0, int nb, const ActOut& out, cudaStream_t s);
int latent_max_rank();
int latent_max_rot();

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


// ---------------------------------------------------------------------------------------
// Recurrence with a decay per key channel and a bonus for the current token (the RWKV-6 form), per head:
//   o = (S + diag(u) k v^T)^T r,  S <- diag(exp(-exp(z))) S + k v^T;  o / rms(o) * norm * silu(gate)
// ---------------------------------------------------------------------------------------
struct WkvArgs {
    const float* proj = nullptr;   // rows r | k | v | gate, each [heads dim]
    int64_t ld = 0;
    const float* u = nullptr;      // [heads, dim]
    const float* norm = nullptr;   // [heads dim]
    float eps = 0.f;
    int heads = 1, dim = 1;
    float* s = nullptr;            // [batch, heads, dim (key), dim (value)] f32
    const int32_t* pos = nullptr;
    int batch = 1, q_rows = 1;
    float* y = nullptr;            // rows [heads dim]: step: the finished rows; prefill: o as it is
    // step: the low-rank input of the decays and their matrix
    const float* low = nullptr;    // rows of `rank` floats
    int rank = 0;
    const uint8_t* w2_tiles = nullptr;  // tiled [heads dim, rank], rows padded to w2_pad
    int w2_pad = 0;
    const float* w0 = nullptr;     // [heads dim]
    // prefill: the decays, and the token shift's state
    const float* w = nullptr;      // rows [heads dim]
    const float* hn = nullptr;     // rows [width]
    float* shift = nullptr;        // [2][max_batch][width], slot = parity of the position
    int64_t shift_slot = 0;
    int width = 0;
    int sm_count = 0;
    bool split16 = false;          // prefill: the factors of the products with states and values as bf16 hi + lo
    // prefill in segments of the tokens, side by side (null: one after the other)
    float* seg_s = nullptr;        // wkv_segment_floats per sequence: states and decays of the segments
    float* seg_w = nullptr;        // wkv_prefix_floats: decays up to each block of 64 tokens
};
int64_t wkv_segment_floats(int heads, int dim);  // 0: the head size has no such form
int64_t wkv_prefix_floats(int heads, int dim, int64_t rows, int batch);
int wkv_max_dim();
cudaError_t launch_wkv_step(const WkvArgs& a, cudaStream_t s, bool pdl);
cudaError_t launch_wkv_prefill(const WkvArgs& a, cudaStream_t s);
// Token shift of the new rows: x + (x before - x) * mu for the inputs r, k, v, gate (four blocks of tiles or rows) and the
// decay (tiles: hi | lo).
struct WkvMix {
    const float* hn = nullptr;
    const float* mu[5] = {nullptr, nullptr, nullptr, nullptr, nullptr};  // r, k, v, gate, decay
    const float* shift = nullptr;
    int64_t shift_slot = 0;
    const int32_t* pos = nullptr;
    int batch = 1, q_rows = 1, width = 0;
    uint8_t* tiles4 = nullptr;   // bf16
    uint8_t* tiles_w = nullptr;
    int64_t m_pad = 0;
    float* rows5 = nullptr;      // f32: [rows][5][width]
};
cudaError_t launch_wkv_mix(const WkvMix& a, cudaStream_t s);

// ---------------------------------------------------------------------------------------
// Gated linear recurrence per channel over many tokens (see RgluStep)
// ---------------------------------------------------------------------------------------
struct RgluArgs {
    const float* proj = nullptr;   // rows y | x, each [channels]
    int64_t ld = 0;
    const float* conv_w = nullptr; // [channels, taps]
    const float* conv_b = nullptr;
    int channels = 1, blocks = 1, taps = 1;
    float* ring = nullptr;         // [batch, taps, channels], slot = position % taps
    const float* lam = nullptr;
    float* state = nullptr;        // [batch, channels]
    const int32_t* pos = nullptr;
    int batch = 1, q_rows = 1;
    float* u = nullptr;            // rows [channels]: convolution outputs
    uint8_t* u_tiles = nullptr;    // the same as tiled hi | lo blocks (bf16 models)
    int64_t m_pad = 0;
    const float* gates = nullptr;  // rows [channels][2]
};
cudaError_t launch_rglru_conv(const RgluArgs& a, cudaStream_t s);
cudaError_t launch_rglru_scan(const RgluArgs& a, const ActOut& out, cudaStream_t s);

// ---------------------------------------------------------------------------------------
// Mixture of experts
// ---------------------------------------------------------------------------------------
int moe_max_experts();
// <= 8 rows: the chosen experts of each row, streamed.  logits [rows, experts]; ff rows of ff_ld floats: [top][kpad(ff)] and,
// at shared_at, the shared expert's activations.
struct MoeStep {
    const DenseLin* up = nullptr;      // gate and up rows in turn
    const DenseLin* down = nullptr;
    const DenseLin* shared_down = nullptr;  // null: no shared expert
    const float* logits = nullptr;
    int experts = 1, top = 1, rows = 1;
    const float* x = nullptr;          // [rows, k]
    float* ff = nullptr;
    int64_t ff_ld = 0;
    float* y = nullptr;                // [rows, n of down]
    int sm_count = 0;
};
bool moe_step_fits(const MoeStep& a);
cudaError_t launch_moe_up(const MoeStep& a, cudaStream_t s, bool pdl);
cudaError_t launch_moe_down(const MoeStep& a, cudaStream_t s, bool pdl);
// Many rows: choice and weights per row, plan of the expert products, the rows copied behind one another by expert.
struct MoeRoute {
    const float* logits = nullptr;  // rows of ld floats
    int64_t ld = 0;
    int64_t rows = 0;
    int experts = 1, top = 1, tile = 64, max_tiles = 0;
    int* sel = nullptr;             // [rows, top] expert
    int* rank = nullptr;            // [rows, top] place among the expert's rows
    float* wt = nullptr;            // [rows, top]
    int* dst = nullptr;             // [rows, top] row of the grouped activations
    int* counts = nullptr;          // [experts] zero before the first call
    int* counts_done = nullptr;     // [experts] the counts of this call
    int* row_start = nullptr;       // [experts + 1]
    ExpertTile* tiles = nullptr;
    int* n_tiles = nullptr;
    // rows to group: tiled bf16 or f32
    const uint8_t* x_tiles = nullptr;
    int64_t m_pad = 0;
    uint8_t* xe_tiles = nullptr;
    int64_t me_pad = 0;
    const float* x = nullptr;
    float* xe = nullptr;
    int k = 0;
};
int moe_tile_rows(int64_t rows, int top, int experts);
int moe_max_tiles(int64_t rows, int top, int experts, int tile);
int64_t moe_grouped_rows(int64_t rows, int top, int experts);  // rows of the grouped activations, padding included
cudaError_t launch_moe_route(const MoeRoute& a, cudaStream_t s);

}  // namespace bt
