// The model object behind bt_model: what every architecture shares (tokens, positions, residual stream, head, graphs,
// prefill staging) and the ternary Llama / TTT layers.  Layer-list models hang their own layers under `lay`.
#pragma once

#include <vector>

#include "bt_handles.cuh"

namespace bt {

constexpr float kRmsEps = 1e-5f;  // model/block.rs:10, model/llama.rs:13

struct Layered;  // layered.cu

struct HostLinear {
    std::vector<uint8_t> packed;  // [n_out, k_in/4, n_bases]
    int64_t n_out = 0, k_in = 0;
    int n_bases = 1;
    float scales[8] = {0};
    bool set = false;
};

struct Layer {
    HostLinear host[9];
    bt_linear* qkv = nullptr;
    bt_linear* o = nullptr;
    bt_linear* gate_up_il = nullptr;   // gate/up interleaved by 8 rows (fused SwiGLU epilogue; SwiGLU row kernel)
    bt_linear* down = nullptr;
    bt_linear* ttt_down = nullptr;
    bt_linear* ttt_up = nullptr;
    float* norm1 = nullptr;
    float* norm2 = nullptr;
    bt_kv_cache* kv = nullptr;
    float* w_state = nullptr;  // [max_batch, d, d]
};

}  // namespace bt

using bt::HostLinear;
using bt::Layer;
using bt::kRmsEps;

struct bt_model {
    bt_model_config cfg{};
    int device = 0;
    int sm_count = 0;
    int head_dim = 0, d_small = 0, qkv_dim = 0;
    int tp = 1;                      // tensor-parallel degree
    int nh_l = 0, nkv_l = 0, i_l = 0;  // this rank's query heads, KV heads, MLP columns
    void* comm = nullptr;            // NCCL communicator when tp > 1
    void* peer = nullptr;            // peer-memory exchange (CUDA IPC inboxes) when the ranks have set it up
    int32_t* acc_i32 = nullptr;      // [max_batch, hidden] accumulators of a row-parallel projection
    bool finalized = false;
    bool multi_basis = false;        // a projection has several bases: the step runs quantiser and product kernels separately
    std::vector<Layer> layers;
    __nv_bfloat16* embed = nullptr;   // 16-bit storage: bf16, or IEEE half when embed_f16
    __nv_bfloat16* lm_head = nullptr;
    bool embed_f16 = false, head_f16 = false;
    float* norm_f = nullptr;
    float rms_eps = kRmsEps;
    float logit_cap = 0.f;           // logits <- cap * tanh(logits / cap); 0: none
    int head_ld = 0;                 // row stride of lm_head (0: hidden)
    int head_rows = 0;               // rows the head's buffers (h, logits, next) hold; >= max_batch
    bt::Layered* lay = nullptr;      // arch 2: per-layer mixers with dense projections (layered.cu)
    float* inv_freq = nullptr;
    float* rope_cos = nullptr;   // [max_pos, head_dim/2]
    float* rope_sin = nullptr;
    // activations
    int32_t* tokens = nullptr;
    int32_t* pos = nullptr;
    float* h = nullptr;
    int8_t* q = nullptr;
    int64_t q_stride = 0;
    float* sx = nullptr;
    int32_t* qsum = nullptr;
    float* qkv = nullptr;
    float* att = nullptr;
    float* gu = nullptr;
    float* feat = nullptr;
    float* z = nullptr;
    float* xn = nullptr;
    float* logits = nullptr;
    int32_t* next = nullptr;
    float* act = nullptr;            // [max_batch, intermediate] silu(gate)*up
    float* xt = nullptr;             // [max_batch, max(hidden, intermediate)] transformed rows (batches above 8)
    int8_t* qtc = nullptr;           // activations in the tensor-core product's layout (batches above 8)
    void* lm_tiles = nullptr;        // lm_head in tensor-core tile order (batches above 8, hidden % 64 == 0)
    void* lm_btiles = nullptr;       // normalised hidden states as bf16 hi|lo tiles
    float* lm_gather = nullptr;      // tensor parallelism: the ranks' vocabulary slices of the logits, [tp][batch][vl]
    int64_t vl = 0;                  // rows of the head per rank (multiple of 128)
    unsigned int* absmax = nullptr;  // [num_layers][2][max_batch] max|x| cells of the fused path
    float* cand_val = nullptr;
    int32_t* cand_idx = nullptr;
    int32_t* tokens_pinned = nullptr;
    int32_t* next_pinned = nullptr;
    float* trace = nullptr;          // inspection aid: per-layer intermediate tensors of a step (caller's device buffer)
    int trace_rows = 0;              // rows per tensor the trace buffer was sized for
    // prefill scratch (allocated at the first bt_model_prefill, for pf_rows = sequences x tokens of a chunk)
    int pf_rows = 0;
    int32_t* pf_tokens = nullptr;
    float* pf_h = nullptr;
    float* pf_qkv = nullptr;
    float* pf_att = nullptr;
    float* pf_gu = nullptr;
    float* pf_act = nullptr;         // silu(gate)*up rows, only while a trace is recorded
    int pf_act_rows = 0;
    int8_t* pf_qtc = nullptr;
    float* pf_sx = nullptr;
    int32_t* pf_qsum = nullptr;
    std::vector<int32_t> pf_host;
    unsigned int* err_pinned = nullptr;  // tensor parallel: the device error word as read after a step
    int host_pos = 0;
    int64_t ternary_bytes = 0;
    cudaStream_t stream = nullptr;
    cudaGraphExec_t graphs[65] = {nullptr};
};

namespace bt {
// arch 2 (layered.cu); each is called by the entry point of the same name in model.cu
bt_status layered_finalize(bt_model* m);
void layered_destroy(bt_model* m);
bt_status layered_reset(bt_model* m);
bt_status layered_set_tensor(bt_model* m, bt_tensor_kind kind, const float* data, int64_t n_elem, bt_dtype storage);
bt_status layered_step(bt_model* m, int batch, cudaStream_t s);          // up to the residual stream in m->h
bt_status layered_prefill_buffers(bt_model* m, int rows);
bt_status layered_prefill(bt_model* m, int batch, int n, int past, cudaStream_t s);  // up to the residual stream in m->pf_h
int layered_launches(const bt_model* m, int batch);
int layered_runs(const bt_model* m);
bt_kv_cache* layered_kv(bt_model* m, int run);
// f32 host values -> 16-bit device storage (model.cu)
bt_status upload_16bit(const float* host, int64_t n, __nv_bfloat16* dst, bool f16);
}  // namespace bt
