// Latent attention: per position the cache holds one normed latent row and one rotated key part for all heads.  A query's
// unrotated part meets the latents through the key matrix (absorbed by the product in front of these kernels), the weighted
// latents leave for the value matrix (the product behind them).  Scores, softmax and running sums are f32.
#include <cooperative_groups.h>

#include "bt_dense.cuh"
#include "bt_ptx.cuh"

namespace cg = cooperative_groups;

namespace bt {

namespace {

constexpr int kMaxRank = 512, kMaxRot = 128, kMaxSplits = 16;
constexpr unsigned kErrLatentTimeout = 0x4c41544eu;  // 'LATN'

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }

// element j of a vector whose first rot_dims dimensions are turned in neighbouring pairs
__device__ __forceinline__ float rotated(const LatentAttn& a, const float* x, int j, int p) {
    if (j >= a.rot_dims) return x[j];
    const int64_t at = (int64_t)p * (a.rot_dims >> 1) + (j >> 1);
    const float c = a.cos_t[at], s = a.sin_t[at];
    return (j & 1) ? fmaf(x[j], c, x[j - 1] * s) : fmaf(x[j], c, -x[j + 1] * s);
}
// 1 / rms of the latent columns of a row; `red` holds 32 floats
__device__ __forceinline__ float latent_inv(const LatentAttn& a, const float* c, float* red) {
    float ss = 0.0f;
    for (int i = threadIdx.x; i < a.rank; i += blockDim.x) ss = fmaf(c[i], c[i], ss);
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.0f;
    for (int i = 0; i < (int)(blockDim.x >> 5); ++i) ss += red[i];
    return 1.0f / sqrtf(ss / (float)a.rank + a.eps);
}

// ---------------------------------------------------------------------------------------
// new tokens of a prefill: one CTA per row
// ---------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentAttn a) {
    __shared__ float red[32];
    const int64_t r = blockIdx.x;
    const int b = (int)(r / a.q_rows), p = a.pos[b] + (int)(r % a.q_rows);
    const float* row = a.proj + r * a.ld;
    const int H = a.heads, hd = a.dim + a.rot, kr = a.kv.rot_col();
    const float* c = row + H * hd;
    const float inv = latent_inv(a, c, red);
    if (p < 0 || p >= a.kv.max_seq) return;
    uint8_t* seq = reinterpret_cast<uint8_t*>(a.kv.rows) + b * a.kv.seq_bytes();
    if (a.kv.f32) {
        float* dst = reinterpret_cast<float*>(seq) + (int64_t)p * a.kv.stride;
        for (int i = threadIdx.x; i < a.rank; i += 256) dst[i] = c[i] * inv * a.c_norm[i];
        for (int i = threadIdx.x; i < a.rot; i += 256) dst[a.rank + i] = rotated(a, c + a.rank, i, p);
    } else {
        for (int i = threadIdx.x; i < a.rank; i += 256)
            *reinterpret_cast<__nv_bfloat16*>(seq + a.kv.off(p, i)) = __float2bfloat16_rn(c[i] * inv * a.c_norm[i]);
        for (int i = threadIdx.x; i < a.rot; i += 256)
            *reinterpret_cast<__nv_bfloat16*>(seq + a.kv.off(p, kr + i)) = __float2bfloat16_rn(rotated(a, c + a.rank, i, p));
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (a.q_buf) {  // the sizes padded to whole 16-byte pieces
        const int d8 = (a.dim + 7) / 8 * 8, w = d8 + (a.rot + 7) / 8 * 8;
        for (int h = warp; h < H; h += 8) {
            const float* q = row + h * hd;
            __nv_bfloat16* dst = a.q_buf + (r * H + h) * w;
            for (int i = lane; i < w; i += 32)
                dst[i] = __float2bfloat16_rn(i < d8 ? (i < a.dim ? q[i] : 0.0f) : (i - d8 < a.rot ? rotated(a, q + a.dim, i - d8, p) : 0.0f));
        }
        return;
    }
    const int kd = dense_kpad(a.dim);
    for (int h = warp; h < H; h += 8) {
        const float* q = row + h * hd;
        for (int i = lane; i < a.rot; i += 32) a.q_rot[(r * H + h) * a.rot + i] = rotated(a, q + a.dim, i, p);
        if (a.q_rows32)
            for (int i = lane; i < a.dim; i += 32) a.q_rows32[(r * H + h) * a.dim + i] = q[i];
        if (a.q_tiles)
            for (int i = lane; i < kd; i += 32) {
                const float v = i < a.dim ? q[i] : 0.0f;
                const __nv_bfloat16 hi = __float2bfloat16_rn(v);
                *reinterpret_cast<__nv_bfloat16*>(a.q_tiles + dense_off(r, h * 2 * kd + i, a.m_pad)) = hi;
                *reinterpret_cast<__nv_bfloat16*>(a.q_tiles + dense_off(r, (h * 2 + 1) * kd + i, a.m_pad)) = __float2bfloat16_rn(v - __bfloat162float(hi));
            }
    }
}

__global__ void __launch_bounds__(256) latent_tiles_kernel(const LatentView v, int b0, int64_t n, uint8_t* __restrict__ tiles, int64_t m_pad) {
    const int per = dense_kpad(v.rank) / 8;  // pieces per position
    const int64_t groups = (n + 7) / 8, total = groups * per * 8;
    const uint8_t* src = reinterpret_cast<const uint8_t*>(v.rows) + (b0 + (int64_t)blockIdx.y) * v.seq_bytes();
    uint8_t* dst = tiles + blockIdx.y * m_pad * per * 16;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t pos = i / (per * 8) * 8 + (i & 7);
        const int c = (int)(i / 8 % per) * 8;
        *reinterpret_cast<uint4*>(dst + dense_off(pos, c, m_pad)) = c < v.rot_col() ? *reinterpret_cast<const uint4*>(src + v.off(pos, c)) : make_uint4(0, 0, 0, 0);
    }
}

// The end of a span kernel: every CTA of the cluster holds maxima, sums and un-normed outputs [head][W] of its span; each
// finishes an equal share of the outputs.  LOG2: the maxima are in units of ln 2.  fac: [heads][kMaxSplits] floats.
template <bool LOG2>
__device__ __forceinline__ void merge_spans(const LatentAttn& a, float* m_s, float* l_s, float* o_s, float* fac, int W, int nh, int head0,
                                            int64_t r, int split, int splits, const ActOut& out) {
    cg::cluster_group cluster = cg::this_cluster();
    if (splits > 1) cluster.sync(); else __syncthreads();
    const float* gates = a.gate ? a.proj + r * a.ld + a.heads * (a.dim + a.rot) + a.rank + a.rot : nullptr;
    // a span's factor per head: its share of the softmax over all spans, times the output gate
    for (int h = threadIdx.x; h < nh; h += blockDim.x) {
        float ms[kMaxSplits], ls[kMaxSplits], m = -INFINITY, den = 0.0f;
#pragma unroll
        for (int s = 0; s < kMaxSplits; ++s) {  // all remote reads in flight together
            ms[s] = s < splits ? *(splits > 1 ? cluster.map_shared_rank(m_s, s) + h : m_s + h) : -INFINITY;
            ls[s] = s < splits ? *(splits > 1 ? cluster.map_shared_rank(l_s, s) + h : l_s + h) : 0.0f;
        }
#pragma unroll
        for (int s = 0; s < kMaxSplits; ++s) m = fmaxf(m, ms[s]);
#pragma unroll
        for (int s = 0; s < kMaxSplits; ++s) {
            ms[s] = LOG2 ? ex2(ms[s] - m) : expf(ms[s] - m);  // an empty span: 0
            den = fmaf(ls[s], ms[s], den);
        }
        const float f = (gates ? sigmoid_f(gates[head0 + h]) : 1.0f) / den;
#pragma unroll
        for (int s = 0; s < kMaxSplits; ++s)
            if (s < splits) fac[h * kMaxSplits + s] = ms[s] * f;
    }
    __syncthreads();
    const int kr = dense_kpad(a.rank), quads = (a.rank + 3) / 4, total = nh * quads;  // W is a multiple of 4
    const int i1 = (int)((int64_t)total * (split + 1) / splits);
    for (int i = (int)((int64_t)total * split / splits) + threadIdx.x; i < i1; i += blockDim.x) {
        const int h = i / quads, c = (i - h * quads) * 4, head = head0 + h;
        float v[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll 8
        for (int s = 0; s < splits; ++s) {
            const float4 o = *reinterpret_cast<const float4*>((splits > 1 ? cluster.map_shared_rank(o_s, s) : o_s) + h * W + c);
            const float f = fac[h * kMaxSplits + s];
            v[0] = fmaf(o.x, f, v[0]); v[1] = fmaf(o.y, f, v[1]); v[2] = fmaf(o.z, f, v[2]); v[3] = fmaf(o.w, f, v[3]);
        }
        if (out.tiles && c + 4 <= a.rank) {
            *reinterpret_cast<uint2*>(out.tiles + dense_off(r, head * kr + c, out.m_pad)) = make_uint2(ptx::pack2(v[0], v[1]), ptx::pack2(v[2], v[3]));
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (c + j >= a.rank) break;
                if (out.tiles) *reinterpret_cast<__nv_bfloat16*>(out.tiles + dense_off(r, head * kr + c + j, out.m_pad)) = __float2bfloat16_rn(v[j]);
                else out.rows[r * out.ld + head * a.rank + c + j] = v[j];
            }
        }
    }
    if (splits > 1) cluster.sync();  // no CTA leaves while its sums are being read
}

// ---------------------------------------------------------------------------------------
// one query position, HG heads, on the tensor cores (bf16 cache)
// ---------------------------------------------------------------------------------------
// The cache is laid out in core matrices (8 positions x 16 bytes), per group of 8 positions all columns one after the other, so
// that a block of 128 positions is a few bulk copies.  In shared memory it is the K-major A operand of the scores (positions x
// columns) and, read the other way, the MN-major A operand of the values (latent columns x positions).
//   scores^T [128 positions][HG]  = block . queries^T            (tcgen05, accumulators in TMEM)
//   softmax: scores through shared memory, a warp per HG / 16 heads; weights leave as bf16 hi and lo
//   outputs^T [rank][2 HG]       += block^T . [hi | lo]^T        (tiles of 128 latent columns, accumulators in TMEM)
// The outputs are rescaled only when a maximum has grown by more than 2^8.
constexpr int kSpanThreads = 512, kSpanWarps = kSpanThreads / 32, kKeys = 128, kMaxStages = 3;
constexpr float kLazy = 8.0f;

template <int HG>
struct SpanCfg {
    static constexpr int kP = HG * kKeys * 2;                                   // bytes of the weights' hi (lo) part
    static constexpr int kTmem = HG == 32 ? 512 : 256;                           // columns: scores, outputs of up to four tiles
    static constexpr size_t kFixed = (size_t)2 * kP + HG * kKeys * 4 + (3 + kMaxSplits) * HG * 4 + 32 * 4 + 128;
    __host__ __device__ static size_t q(int cols) { return (size_t)HG * cols * 2; }
    static size_t fixed(int cols) { return q(cols) + kFixed + (size_t)cols * 2; }
};
__device__ __forceinline__ uint32_t span_idesc(int n, bool a_mn) {  // f32 += bf16 . bf16, M = 128
    return (1u << 4) | (1u << 7) | (1u << 10) | ((a_mn ? 1u : 0u) << 15) | ((uint32_t)(n >> 3) << 17) | (8u << 24);
}

template <int HG>
__global__ void __launch_bounds__(kSpanThreads, 1) latent_span_tc_kernel(const LatentAttn a, bool prepared, int splits, int stages,
                                                                         unsigned int* err, const ActOut out) {
    using Cfg = SpanCfg<HG>;
    constexpr int NS = HG / kSpanWarps;  // heads of a warp in the softmax
    extern __shared__ __align__(128) uint8_t sm[];
    const int kl = a.kv.rot_col(), cols = a.kv.cols(), pieces = cols / 8;
    const uint32_t group = (uint32_t)cols * 16;          // bytes of 8 positions (heads)
    const uint32_t stage_bytes = group * (kKeys / 8);
    uint8_t* q_s = sm + (size_t)stages * stage_bytes;    // queries [HG / 8][pieces][8 heads][16 bytes]
    uint8_t* p_hi = q_s + Cfg::q(cols);                // softmax weights [HG / 8][16 pieces][8 heads][16 bytes]
    uint8_t* p_lo = p_hi + Cfg::kP;
    float* s_s = reinterpret_cast<float*>(p_lo + Cfg::kP);  // scores [HG][128]
    float* m_s = s_s + HG * kKeys;
    float* l_s = m_s + HG;
    float* al_s = l_s + HG;
    float* fac = al_s + HG;                              // [HG][kMaxSplits]
    float* red = fac + HG * kMaxSplits;
    uint64_t* full = reinterpret_cast<uint64_t*>(red + 32);
    uint64_t* s_done = full + kMaxStages;
    uint64_t* o_done = s_done + 1;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 1);
    __nv_bfloat16* new_s = reinterpret_cast<__nv_bfloat16*>(full + 16);  // the new token's row [cols]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int H = a.heads, hd = a.dim + a.rot;
    const int head0 = blockIdx.y * HG, nh = min(HG, H - head0);
    const int64_t r = blockIdx.z;
    const int b = (int)(r / a.q_rows), split = blockIdx.x;
    const int p = a.pos[b] + (int)(r % a.q_rows);
    const int total = min(p + 1, a.kv.max_seq);
    const int span = ((total + splits - 1) / splits + 7) / 8 * 8;
    const int t0 = min(split * span, total), t1 = min(t0 + span, total);
    const int blocks = (t1 - t0 + kKeys - 1) / kKeys;
    const bool owner = !prepared && t1 == p + 1 && t0 < t1;
    uint8_t* seq = reinterpret_cast<uint8_t*>(a.kv.rows) + b * a.kv.seq_bytes();
    bool ok = true;
    if (threadIdx.x == 0) {
        for (int s = 0; s < kMaxStages; ++s) ptx::mbar_init(&full[s], 1);
        ptx::mbar_init(s_done, 1);
        ptx::mbar_init(o_done, 1);
        ptx::mbar_fence_init();
    }
    if (warp == 1) { ptx::tmem_alloc(tmem_slot, Cfg::kTmem); ptx::tmem_relinquish(); }
    ptx::tc_fence_before();
    __syncthreads();
    ptx::tc_fence_after();
    const uint32_t tmem = *tmem_slot, tmem_o = tmem + HG;
    auto load = [&](int i) {  // warp 0: the i-th block of the span
        if (i >= blocks) return;
        const int slot = i % stages, live = (min(kKeys, t1 - t0 - i * kKeys) + 7) / 8;  // groups with a position of the span
        if (lane == 0) ptx::mbar_arrive_expect_tx(&full[slot], live * group);
        __syncwarp();
        const int g0 = lane * 2, n = min(2, live - g0);  // two groups a lane
        if (n > 0) ptx::bulk_g2s(sm + (size_t)slot * stage_bytes + g0 * group, seq + ((int64_t)t0 / 8 + i * (kKeys / 8) + g0) * group, n * group, &full[slot]);
    };
    if (prepared) ptx::pdl_wait();  // the cache rows come from the kernel in front
    if (blocks > 0 && blocks <= stages) {  // groups of the last block that no copy fills
        uint8_t* st = sm + (size_t)(blocks - 1) * stage_bytes;
        const uint32_t o = (uint32_t)((t1 - t0 - (blocks - 1) * kKeys + 7) / 8) * group;
        for (uint32_t e = o + threadIdx.x * 16; e < stage_bytes; e += kSpanThreads * 16) *reinterpret_cast<uint4*>(st + e) = make_uint4(0, 0, 0, 0);
    }
    if (warp == 0)
        for (int i = 0; i < stages; ++i) load(i);
    if (!prepared) ptx::pdl_wait();
    ptx::pdl_launch_dependents();

    // ---- queries: [absorbed | rotated] ----
    const float* row = a.proj + r * a.ld;
    for (int i = threadIdx.x; i < HG * pieces; i += kSpanThreads) {  // eight columns at a time
        const int h = i / pieces, piece = i - h * pieces, c = piece * 8;
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = 0.0f;
        if (h < nh) {
            if (c < kl) {
                const float* src = a.q_abs + (r * H + head0 + h) * a.rank + c;
                if (c + 8 <= a.rank && (a.rank & 3) == 0) {
                    const float4 x = *reinterpret_cast<const float4*>(src), y = *reinterpret_cast<const float4*>(src + 4);
                    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; v[4] = y.x; v[5] = y.y; v[6] = y.z; v[7] = y.w;
                } else {
#pragma unroll
                    for (int j = 0; j < 8; ++j) if (c + j < a.rank) v[j] = src[j];
                }
            } else {
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    if (c + j - kl < a.rot)
                        v[j] = prepared ? a.q_rot[(r * H + head0 + h) * a.rot + c + j - kl] : rotated(a, row + (head0 + h) * hd + a.dim, c + j - kl, p);
            }
        }
        *reinterpret_cast<uint4*>(q_s + (h >> 3) * group + piece * 128 + (h & 7) * 16) =
            make_uint4(ptx::pack2(v[0], v[1]), ptx::pack2(v[2], v[3]), ptx::pack2(v[4], v[5]), ptx::pack2(v[6], v[7]));
    }
    if (owner) {
        const float* c = row + H * hd;
        const float inv = latent_inv(a, c, red);
        for (int i = threadIdx.x; i < cols; i += kSpanThreads) {
            float v = 0.0f;
            if (i < kl) { if (i < a.rank) v = c[i] * inv * a.c_norm[i]; }
            else if (i - kl < a.rot) v = rotated(a, c + a.rank, i - kl, p);
            const __nv_bfloat16 w = __float2bfloat16_rn(v);
            new_s[i] = w;
            if (blockIdx.y == 0) *reinterpret_cast<__nv_bfloat16*>(seq + a.kv.off(p, i)) = w;
        }
    }
    ptx::fence_async_smem();
    __syncthreads();

    float m_run[NS], l_run[NS];  // heads NS warp ..: reference maximum; this lane's share of the sum
#pragma unroll
    for (int j = 0; j < NS; ++j) { m_run[j] = -INFINITY; l_run[j] = 0.0f; }
    const float unit = a.scale * 1.4426950408889634f;
    const int steps = cols / 16, m_tiles = (a.rank + 127) / 128;
    for (int i = 0; i < blocks; ++i) {
        const int slot = i % stages;
        uint8_t* st = sm + (size_t)slot * stage_bytes;
        const uint32_t kv = ptx::smem_u32(st);
        const int base = t0 + i * kKeys;
        if (warp == 0 && i > 0) {  // the block before this one is used up: its slot takes the next one to come
            ok &= ptx::mbar_wait_bounded(o_done, (uint32_t)((i - 1) & 1));
            load(i + stages - 1);
        }
        if (owner && i == blocks - 1) {  // the new row has not been in the copy
            ok &= ptx::mbar_wait_bounded(&full[slot], (uint32_t)((i / stages) & 1));
            const int at = p - base;
            for (int c = threadIdx.x; c < pieces; c += kSpanThreads)
                *reinterpret_cast<uint4*>(st + (at >> 3) * group + c * 128 + (at & 7) * 16) = *reinterpret_cast<const uint4*>(new_s + c * 8);
            ptx::fence_async_smem();
            __syncthreads();
        }
        if (warp == 1 && lane == 0) {
            ok &= ptx::mbar_wait_bounded(&full[slot], (uint32_t)((i / stages) & 1));
            ptx::tc_fence_after();
            uint64_t ad = ptx::smem_desc(kv, 128, group), qd = ptx::smem_desc(ptx::smem_u32(q_s), 128, group);
            ptx::umma_f16(tmem, ad, qd, span_idesc(HG, false), 0u);
#pragma unroll 4
            for (int k = 1; k < steps; ++k) {  // 256 bytes further in units of 16
                ad += 16;
                qd += 16;
                ptx::umma_f16(tmem, ad, qd, span_idesc(HG, false), 1u);
            }
            ptx::umma_commit(s_done);
        }
        __syncwarp();
        if (warp == 15 && i + stages < blocks && lane < 8) {  // the block that will take this one's slot comes into L2 meanwhile
            const int g0 = lane * 2, n = min(2, (min(kKeys, t1 - t0 - (i + stages) * kKeys) + 7) / 8 - g0);
            if (n > 0) ptx::prefetch_l2(seq + ((int64_t)t0 / 8 + (i + stages) * (kKeys / 8) + g0) * group, n * group);
        }
        if (warp < 4) {  // lane = position
            ok &= ptx::mbar_wait_bounded(s_done, (uint32_t)(i & 1));
            ptx::tc_fence_after();
            const int key = warp * 32 + lane;
            const bool live = base + key < t1;
#pragma unroll
            for (int c = 0; c < HG; c += 16) {
                uint32_t v[16];
                ptx::tmem_ld16(tmem + ((uint32_t)(warp * 32) << 16) + c, v);
                ptx::tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 16; ++j) s_s[(c + j) * kKeys + key] = live ? __uint_as_float(v[j]) * unit : -INFINITY;
            }
            ptx::tc_fence_before();
        }
        __syncthreads();
        if (i > 0) {  // the weights' buffers and the outputs are free
            ok &= ptx::mbar_wait_bounded(o_done, (uint32_t)((i - 1) & 1));
            ptx::tc_fence_after();
        }
        bool grown = false;
        {
            float4 x[NS];
            float mx[NS];
#pragma unroll
            for (int j = 0; j < NS; ++j) {
                x[j] = *reinterpret_cast<const float4*>(s_s + (warp * NS + j) * kKeys + lane * 4);
                mx[j] = fmaxf(fmaxf(x[j].x, x[j].y), fmaxf(x[j].z, x[j].w));
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int j = 0; j < NS; ++j) mx[j] = fmaxf(mx[j], __shfl_xor_sync(0xffffffffu, mx[j], o));
#pragma unroll
            for (int j = 0; j < NS; ++j) {
                const int h = warp * NS + j;
                float al = 1.0f;
                if (mx[j] > m_run[j] + kLazy) {  // the first block always
                    al = ex2(m_run[j] - mx[j]);
                    m_run[j] = mx[j];
                    grown = true;
                }
                const float e0 = ex2(x[j].x - m_run[j]), e1 = ex2(x[j].y - m_run[j]), e2 = ex2(x[j].z - m_run[j]), e3 = ex2(x[j].w - m_run[j]);
                l_run[j] = fmaf(l_run[j], al, (e0 + e1) + (e2 + e3));
                const uint32_t h0 = ptx::pack2(e0, e1), h1 = ptx::pack2(e2, e3);
                const int o = (h >> 3) * 2048 + (lane >> 1) * 128 + (h & 7) * 16 + (lane & 1) * 8;
                *reinterpret_cast<uint2*>(p_hi + o) = make_uint2(h0, h1);
                *reinterpret_cast<uint2*>(p_lo + o) = make_uint2(ptx::pack2(e0 - __uint_as_float(h0 << 16), e1 - __uint_as_float(h0 & 0xffff0000u)),
                                                                 ptx::pack2(e2 - __uint_as_float(h1 << 16), e3 - __uint_as_float(h1 & 0xffff0000u)));
                if (lane == 0) al_s[h] = al;
            }
        }
        ptx::fence_async_smem();
        const int rescale = __syncthreads_or(grown && i > 0);
        if (rescale) {  // warps w, w + 4, ... take the same lanes and different tiles
            for (int mt = warp >> 2; mt < m_tiles; mt += 4) {
                const uint32_t at = tmem_o + mt * 2 * HG + ((uint32_t)((warp & 3) * 32) << 16);
#pragma unroll
                for (int c = 0; c < 2 * HG; c += 16) {
                    uint32_t v[16];
                    ptx::tmem_ld16(at + c, v);
                    ptx::tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 16; ++j) v[j] = __float_as_uint(__uint_as_float(v[j]) * al_s[(c + j) % HG]);
                    ptx::tmem_st16(at + c, v);
                }
            }
            ptx::tmem_st_wait();
            ptx::tc_fence_before();
            __syncthreads();
        }
        if (warp == 1 && lane == 0) {
            ptx::tc_fence_after();
            const uint64_t pd = ptx::smem_desc(ptx::smem_u32(p_hi), 128, 2048);  // hi and lo rows behind one another
            uint64_t at = ptx::smem_desc(kv, group, 128);
            for (int mt = 0; mt < m_tiles; ++mt, at += 2048 / 16) {
                uint64_t ad = at;
#pragma unroll
                for (int k = 0; k < kKeys / 16; ++k, ad += group / 8)  // two groups of positions further
                    ptx::umma_f16(tmem_o + mt * 2 * HG, ad, pd + k * 16, span_idesc(2 * HG, true), i > 0 || k > 0 ? 1u : 0u);
            }
            ptx::umma_commit(o_done);
        }
    }
#pragma unroll
    for (int j = 0; j < NS; ++j) {
        const float l = warp_sum(l_run[j]);
        if (lane == 0) { m_s[warp * NS + j] = m_run[j]; l_s[warp * NS + j] = l; }
    }
    const int W = m_tiles * 128;
    float* o_s = reinterpret_cast<float*>(sm);  // [heads][W], in the ring's place
    if (blocks > 0) {
        ok &= ptx::mbar_wait_bounded(o_done, (uint32_t)((blocks - 1) & 1));
        ptx::tc_fence_after();
    }
    __syncthreads();
    for (int mt = warp >> 2; mt < m_tiles; mt += 4)
#pragma unroll
        for (int c = 0; c < HG; c += 16) {
            uint32_t v[16], l[16];
            const uint32_t at = tmem_o + mt * 2 * HG + c + ((uint32_t)((warp & 3) * 32) << 16);
            ptx::tmem_ld16(at, v);
            ptx::tmem_ld16(at + HG, l);
            ptx::tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j)
                o_s[(c + j) * W + mt * 128 + (warp & 3) * 32 + lane] = blocks > 0 ? __uint_as_float(v[j]) + __uint_as_float(l[j]) : 0.0f;
        }
    if (!ok) atomicExch(err, kErrLatentTimeout);
    ptx::tc_fence_before();
    __syncthreads();
    if (warp == 1) ptx::tmem_dealloc(tmem, Cfg::kTmem);
    merge_spans<true>(a, m_s, l_s, o_s, fac, W, nh, head0, r, split, splits, out);
}

// ---------------------------------------------------------------------------------------
// the same in f32 on the FMA units (32-bit models): 8 heads per CTA, tiles of 32 positions
// ---------------------------------------------------------------------------------------
constexpr int kF32Heads = 8, kF32Keys = 32, kF32Threads = 256;
__global__ void __launch_bounds__(kF32Threads) latent_span_f32_kernel(const LatentAttn a, bool prepared, int splits, const ActOut out) {
    extern __shared__ __align__(16) float fs[];
    const int D = a.rank + a.rot, W = (a.rank + 3) / 4 * 4;
    float* o_s = fs;                          // [8][W]
    float* q_s = o_s + kF32Heads * W;         // [8][D]
    float* p_s = q_s + kF32Heads * D;         // [8][32]
    float* m_s = p_s + kF32Heads * kF32Keys;
    float* l_s = m_s + kF32Heads;
    float* al_s = l_s + kF32Heads;
    float* fac = al_s + kF32Heads;            // [8][kMaxSplits]
    float* red = fac + kF32Heads * kMaxSplits;  // 32
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int H = a.heads, hd = a.dim + a.rot;
    const int head0 = blockIdx.y * kF32Heads, nh = min(kF32Heads, H - head0);
    const int64_t r = blockIdx.z;
    const int b = (int)(r / a.q_rows), split = blockIdx.x;
    ptx::pdl_wait();
    ptx::pdl_launch_dependents();
    const int p = a.pos[b] + (int)(r % a.q_rows);
    const int total = min(p + 1, a.kv.max_seq);
    const int span = ((total + splits - 1) / splits + 7) / 8 * 8;
    const int t0 = min(split * span, total), t1 = min(t0 + span, total);
    float* cache = reinterpret_cast<float*>(a.kv.rows) + (int64_t)b * a.kv.max_seq * a.kv.stride;
    const float* row = a.proj + r * a.ld;
    for (int i = threadIdx.x; i < kF32Heads * D; i += kF32Threads) {
        const int h = i / D, c = i - h * D;
        float v = 0.0f;
        if (h < nh)
            v = c < a.rank ? a.q_abs[(r * H + head0 + h) * a.rank + c]
                           : (prepared ? a.q_rot[(r * H + head0 + h) * a.rot + c - a.rank] : rotated(a, row + (head0 + h) * hd + a.dim, c - a.rank, p));
        q_s[i] = v;
    }
    if (!prepared && t1 == p + 1 && t0 < t1) {  // (head chunks write the same values)
        const float* c = row + H * hd;
        const float inv = latent_inv(a, c, red);
        float* dst = cache + (int64_t)p * a.kv.stride;
        for (int i = threadIdx.x; i < D; i += kF32Threads) dst[i] = i < a.rank ? c[i] * inv * a.c_norm[i] : rotated(a, c + a.rank, i - a.rank, p);
    }
    if (threadIdx.x < kF32Heads) { m_s[threadIdx.x] = -INFINITY; l_s[threadIdx.x] = 0.0f; }
    __syncthreads();
    float acc[kF32Heads][kMaxRank / kF32Threads] = {};
    for (int base = t0; base < t1; base += kF32Keys) {
        for (int k = warp; k < kF32Keys; k += 8) {
            const int t = base + k;
            float s[kF32Heads] = {};
            if (t < t1)
                for (int c = lane; c < D; c += 32) {
                    const float x = cache[(int64_t)t * a.kv.stride + c];
#pragma unroll
                    for (int h = 0; h < kF32Heads; ++h) s[h] = fmaf(x, q_s[h * D + c], s[h]);
                }
#pragma unroll
            for (int h = 0; h < kF32Heads; ++h) {
                s[h] = warp_sum(s[h]);
                if (lane == h) p_s[h * kF32Keys + k] = t < t1 ? s[h] * a.scale : -INFINITY;
            }
        }
        __syncthreads();
        {   // a warp per head
            const float x = p_s[warp * kF32Keys + lane];
            const float m_old = m_s[warp], m_new = fmaxf(m_old, warp_max(x));
            const float e = expf(x - m_new), sum = warp_sum(e);
            p_s[warp * kF32Keys + lane] = e;
            if (lane == 0) {
                const float al = expf(m_old - m_new);
                al_s[warp] = al;
                m_s[warp] = m_new;
                l_s[warp] = l_s[warp] * al + sum;
            }
        }
        __syncthreads();
#pragma unroll
        for (int h = 0; h < kF32Heads; ++h)
#pragma unroll
            for (int j = 0; j < kMaxRank / kF32Threads; ++j) acc[h][j] *= al_s[h];
        const int n = min(kF32Keys, t1 - base);
        for (int k = 0; k < n; ++k)
#pragma unroll
            for (int j = 0; j < kMaxRank / kF32Threads; ++j) {
                const int c = threadIdx.x + j * kF32Threads;
                if (c < a.rank) {
                    const float x = cache[(int64_t)(base + k) * a.kv.stride + c];
#pragma unroll
                    for (int h = 0; h < kF32Heads; ++h) acc[h][j] = fmaf(p_s[h * kF32Keys + k], x, acc[h][j]);
                }
            }
        __syncthreads();
    }
#pragma unroll
    for (int h = 0; h < kF32Heads; ++h)
#pragma unroll
        for (int j = 0; j < kMaxRank / kF32Threads; ++j) {
            const int c = threadIdx.x + j * kF32Threads;
            if (c < a.rank) o_s[h * W + c] = acc[h][j];
        }
    merge_spans<false>(a, m_s, l_s, o_s, fac, W, nh, head0, r, split, splits, out);
}

template <typename... KArgs, typename... Args>
cudaError_t launch_cluster(void (*kernel)(KArgs...), dim3 grid, int threads, size_t smem, cudaStream_t s, bool pdl, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3((unsigned)threads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = grid.x; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}
// active: for 1, 2, 4, ... CTAs the clusters that can be resident at once (a cluster sits in one GPC); null: as many as there are SMs
int span_splits(const LatentAttn& a, int64_t groups, const int* active = nullptr) {
    int splits = 1;
    for (int i = 1; splits < kMaxSplits && groups * splits * 2 <= a.sm_count && splits * kKeys < a.kv.max_seq && (!active || groups <= active[i]); ++i) splits *= 2;
    return splits;
}

constexpr size_t kSpanSmem = 224 * 1024;
template <int HG>
cudaError_t span_launch(const LatentAttn& a, bool prepared, const ActOut& out, unsigned int* err, cudaStream_t s, bool pdl) {
    static PerDeviceOnce once;
    static int active[5];  // every device of a process is the same GPU model
    cudaError_t e = once.run([] {
        cudaError_t x = cudaFuncSetAttribute(latent_span_tc_kernel<HG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSpanSmem);
        if (x == cudaSuccess) x = cudaFuncSetAttribute(latent_span_tc_kernel<HG>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
        for (int i = 0; i < 5 && x == cudaSuccess; ++i) {
            cudaLaunchConfig_t cfg = {};
            cudaLaunchAttribute attr;
            attr.id = cudaLaunchAttributeClusterDimension;
            attr.val.clusterDim.x = 1u << i; attr.val.clusterDim.y = 1; attr.val.clusterDim.z = 1;
            cfg.gridDim = dim3(1u << i); cfg.blockDim = dim3(kSpanThreads); cfg.dynamicSmemBytes = kSpanSmem; cfg.attrs = &attr; cfg.numAttrs = 1;
            x = cudaOccupancyMaxActiveClusters(&active[i], latent_span_tc_kernel<HG>, &cfg);
        }
        return x;
    });
    if (e != cudaSuccess) return e;
    const int cols = a.kv.cols(), hg = (a.heads + HG - 1) / HG;
    const size_t stage = (size_t)cols * kKeys * 2, fixed = SpanCfg<HG>::fixed(cols), outs = (size_t)HG * ((a.rank + 127) / 128 * 128) * sizeof(float);
    // (the values are read in whole tiles of 128 latent columns: up to 2 KB behind a stage, which is shared memory in use)
    int stages = (int)((kSpanSmem - fixed) / stage);
    stages = stages > kMaxStages ? kMaxStages : stages;
    if (stages < 1 || stages * stage < outs) return cudaErrorInvalidConfiguration;
    const int64_t rows = (int64_t)a.batch * a.q_rows;
    const int splits = span_splits(a, rows * hg, active);
    // one CTA per SM, whatever its registers: none waits for tensor memory while its cluster holds some elsewhere
    const size_t smem = stages * stage + fixed, least = (size_t)116 * 1024;
    return launch_cluster(latent_span_tc_kernel<HG>, dim3((unsigned)splits, (unsigned)hg, (unsigned)rows), kSpanThreads, smem > least ? smem : least, s, pdl,
                          a, prepared, splits, stages, err, out);
}

}  // namespace

int latent_max_rank() { return kMaxRank; }
int latent_max_rot() { return kMaxRot; }

cudaError_t launch_latent_tiles(const LatentView& v, int b0, int nb, int64_t n, uint8_t* tiles, int64_t m_pad, cudaStream_t s) {
    if (v.f32) return cudaErrorInvalidValue;
    const int64_t total = (n + 7) / 8 * dense_kpad(v.rank);
    latent_tiles_kernel<<<dim3((unsigned)((total + 255) / 256 < 592 ? (total + 255) / 256 : 592), (unsigned)nb), 256, 0, s>>>(v, b0, n, tiles, m_pad);
    return cudaGetLastError();
}

cudaError_t launch_latent_prep(const LatentAttn& a, cudaStream_t s) {
    latent_prep_kernel<<<(unsigned)(a.batch * a.q_rows), 256, 0, s>>>(a);
    return cudaGetLastError();
}

cudaError_t launch_latent_span(const LatentAttn& a, bool prepared, const ActOut& out, cudaStream_t s, bool pdl) {
    if (a.rank > kMaxRank || a.rot > kMaxRot || (!prepared && a.q_rows != 1)) return cudaErrorInvalidValue;
    if (a.kv.f32) {
        static PerDeviceOnce once;
        cudaError_t e = once.run([] {
            cudaError_t x = cudaFuncSetAttribute(latent_span_f32_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
            return x != cudaSuccess ? x : cudaFuncSetAttribute(latent_span_f32_kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
        });
        if (e != cudaSuccess) return e;
        const int hg = (a.heads + kF32Heads - 1) / kF32Heads;
        const int64_t rows = (int64_t)a.batch * a.q_rows;
        const int splits = span_splits(a, rows * hg);
        const size_t smem = ((size_t)kF32Heads * (2 * a.rank + 3 + a.rot) + kF32Heads * kF32Keys + (3 + kMaxSplits) * kF32Heads + 32) * sizeof(float);
        return launch_cluster(latent_span_f32_kernel, dim3((unsigned)splits, (unsigned)hg, (unsigned)rows), kF32Threads, smem, s, pdl, a, prepared, splits, out);
    }
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    unsigned int* err = device_error_word(dev);
    // 32 heads share the cache rows once that leaves no SM idle
    const int cols = a.kv.cols();
    const bool wide = a.heads > 16 && (int64_t)a.batch * a.q_rows * ((a.heads + 31) / 32) * 4 >= a.sm_count &&
                      (size_t)cols * kKeys * 2 + SpanCfg<32>::fixed(cols) <= kSpanSmem;
    return wide ? span_launch<32>(a, prepared, out, err, s, pdl) : span_launch<16>(a, prepared, out, err, s, pdl);
}

}  // namespace bt
