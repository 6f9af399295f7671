// Latent attention: per position the cache holds one normed latent row and one rotated key part for all heads.  A query's
// unrotated part meets the latents through the key matrix (absorbed by the product in front of these kernels), the weighted
// latents leave for the value matrix (the product behind them).  Scores, softmax and running sums are f32.
#include <cooperative_groups.h>

#include "bt_dense.cuh"
#include "bt_ptx.cuh"

namespace cg = cooperative_groups;

namespace bt {

namespace {

constexpr int kMaxRank = 512, kMaxRot = 128;
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
    const int H = a.heads, hd = a.dim + a.rot, kr = dense_kpad(a.rank);
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
            *reinterpret_cast<__nv_bfloat16*>(seq + dense_off(p, i, a.kv.seq_pad)) = __float2bfloat16_rn(c[i] * inv * a.c_norm[i]);
        for (int i = threadIdx.x; i < a.rot; i += 256)
            *reinterpret_cast<__nv_bfloat16*>(seq + dense_off(p, kr + i, a.kv.seq_pad)) = __float2bfloat16_rn(rotated(a, c + a.rank, i, p));
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

// The end of a span kernel: every CTA of the cluster holds maxima, sums and un-normed outputs [head][W] of its span; each
// finishes an equal share of the outputs.  LOG2: the maxima are in units of ln 2.
template <bool LOG2>
__device__ __forceinline__ void merge_spans(const LatentAttn& a, float* m_s, float* l_s, float* o_s, int W, int nh, int head0,
                                            int64_t r, int split, int splits, const ActOut& out) {
    cg::cluster_group cluster = cg::this_cluster();
    if (splits > 1) cluster.sync(); else __syncthreads();
    const float* gates = a.gate ? a.proj + r * a.ld + a.heads * (a.dim + a.rot) + a.rank + a.rot : nullptr;
    const int kr = dense_kpad(a.rank), total = nh * a.rank;
    const int i1 = (int)((int64_t)total * (split + 1) / splits);
    for (int i = (int)((int64_t)total * split / splits) + threadIdx.x; i < i1; i += blockDim.x) {
        const int h = i / a.rank, c = i - h * a.rank, head = head0 + h;
        float ms[8], ls[8], os[8], m = -INFINITY;
#pragma unroll
        for (int s = 0; s < 8; ++s) {  // all remote reads in flight together
            ms[s] = -INFINITY; ls[s] = os[s] = 0.0f;
            if (s < splits) {
                ms[s] = *(splits > 1 ? cluster.map_shared_rank(m_s, s) + h : m_s + h);
                ls[s] = *(splits > 1 ? cluster.map_shared_rank(l_s, s) + h : l_s + h);
                os[s] = *(splits > 1 ? cluster.map_shared_rank(o_s, s) + h * W + c : o_s + h * W + c);
            }
            m = fmaxf(m, ms[s]);
        }
        float den = 0.0f, num = 0.0f;
#pragma unroll
        for (int s = 0; s < 8; ++s) {
            const float f = LOG2 ? ex2(ms[s] - m) : expf(ms[s] - m);  // an empty span: 0
            den = fmaf(ls[s], f, den);
            num = fmaf(os[s], f, num);
        }
        float v = num / den;
        if (gates) v *= sigmoid_f(gates[head]);
        if (out.tiles) *reinterpret_cast<__nv_bfloat16*>(out.tiles + dense_off(r, head * kr + c, out.m_pad)) = __float2bfloat16_rn(v);
        else out.rows[r * out.ld + head * a.rank + c] = v;
    }
    if (splits > 1) cluster.sync();  // no CTA leaves while its sums are being read
}

// ---------------------------------------------------------------------------------------
// one query position, 16 heads, on the tensor cores (bf16 cache)
// ---------------------------------------------------------------------------------------
// The cache is laid out in core matrices (8 positions x 16 bytes), so blocks of 64 positions arrive as one bulk copy per 64
// columns and every ldmatrix reads 128 consecutive bytes.  Per block: eight warps make the scores of 8 positions each, then
// the softmax of two heads each, then 8 NT latent columns each.  Queries and softmax weights enter as bf16 hi + lo.
constexpr int kSpanThreads = 256, kKeys = 64, kHeads = 16;

struct SpanShape {
    int chunks, kc, kr;  // 64-column blocks; 16-column steps of the latent part and of all columns in use
    int stages;
};
__host__ __device__ inline size_t span_fixed_bytes(int chunks) {
    return (size_t)2 * chunks * 2048 + 2 * 2048 + (size_t)kHeads * kKeys * 4 + 3 * kHeads * 4 + 32 * 4 + (size_t)chunks * 128 + 64;
}

template <int NT>
__global__ void __launch_bounds__(kSpanThreads) latent_span_mma_kernel(const LatentAttn a, bool prepared, int splits, int stages,
                                                                       unsigned int* err, const ActOut out) {
    extern __shared__ __align__(128) uint8_t sm[];
    const int kcl = dense_kpad(a.rank) / 64, chunks = kcl + dense_kpad(a.rot) / 64;
    const int stage_bytes = chunks * kKeys * 128;
    uint8_t* q_hi = sm + (size_t)stages * stage_bytes;   // [chunk][2 groups of 8 heads][8 pieces][8 heads][16 bytes]
    uint8_t* q_lo = q_hi + chunks * 2048;
    uint8_t* p_hi = q_lo + chunks * 2048;                // softmax weights [16 heads][64 positions], core matrices
    uint8_t* p_lo = p_hi + 2048;
    float* s_s = reinterpret_cast<float*>(p_lo + 2048);  // scores [16][64]
    float* m_s = s_s + kHeads * kKeys;
    float* l_s = m_s + kHeads;
    float* al_s = l_s + kHeads;
    float* red = al_s + kHeads;
    __nv_bfloat16* new_s = reinterpret_cast<__nv_bfloat16*>(red + 32);  // the new token's row [chunks * 64]
    uint64_t* full = reinterpret_cast<uint64_t*>(new_s + chunks * 64);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int H = a.heads, hd = a.dim + a.rot;
    const int head0 = blockIdx.y * kHeads, nh = min(kHeads, H - head0);
    const int64_t r = blockIdx.z;
    const int b = (int)(r / a.q_rows), split = blockIdx.x;
    const int p = a.pos[b] + (int)(r % a.q_rows);
    const int total = min(p + 1, a.kv.max_seq);
    const int span = ((total + splits - 1) / splits + kKeys - 1) / kKeys * kKeys;
    const int t0 = min(split * span, total), t1 = min(t0 + span, total);
    const int blocks = (t1 - t0 + kKeys - 1) / kKeys;
    const bool owner = !prepared && t1 == p + 1 && t0 < t1;
    uint8_t* seq = reinterpret_cast<uint8_t*>(a.kv.rows) + b * a.kv.seq_bytes();
    bool ok = true;
    if (threadIdx.x == 0) {
        for (int s = 0; s < stages; ++s) ptx::mbar_init(&full[s], 1);
        ptx::mbar_fence_init();
    }
    __syncthreads();
    auto load = [&](int i) {  // thread 0: the i-th block of the span
        if (i >= blocks) return;
        uint8_t* st = sm + (size_t)(i % stages) * stage_bytes;
        ptx::mbar_arrive_expect_tx(&full[i % stages], stage_bytes);
        for (int c = 0; c < chunks; ++c)
            ptx::bulk_g2s(st + c * kKeys * 128, seq + ((int64_t)c * a.kv.seq_pad + t0 + i * kKeys) * 128, kKeys * 128, &full[i % stages]);
    };
    if (prepared) ptx::pdl_wait();  // the cache rows come from the kernel in front
    if (threadIdx.x == 0)
        for (int i = 0; i < stages - 1; ++i) load(i);
    if (!prepared) ptx::pdl_wait();
    ptx::pdl_launch_dependents();

    // ---- queries: [absorbed | rotated] as hi and lo ----
    const float* row = a.proj + r * a.ld;
    const int kl = kcl * 64;
    for (int i = threadIdx.x; i < kHeads * chunks * 64; i += kSpanThreads) {
        const int h = i / (chunks * 64), c = i - h * chunks * 64;
        float v = 0.0f;
        if (h < nh) {
            if (c < kl) { if (c < a.rank) v = a.q_abs[(r * H + head0 + h) * a.rank + c]; }
            else if (c - kl < a.rot) v = prepared ? a.q_rot[(r * H + head0 + h) * a.rot + c - kl] : rotated(a, row + (head0 + h) * hd + a.dim, c - kl, p);
        }
        const int o = (c >> 6) * 2048 + (h >> 3) * 1024 + ((c & 63) >> 3) * 128 + (h & 7) * 16 + (c & 7) * 2;
        const __nv_bfloat16 hi = __float2bfloat16_rn(v);
        *reinterpret_cast<__nv_bfloat16*>(q_hi + o) = hi;
        *reinterpret_cast<__nv_bfloat16*>(q_lo + o) = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
    if (owner) {
        const float* c = row + H * hd;
        const float inv = latent_inv(a, c, red);
        for (int i = threadIdx.x; i < chunks * 64; i += kSpanThreads) {
            float v = 0.0f;
            if (i < kl) { if (i < a.rank) v = c[i] * inv * a.c_norm[i]; }
            else if (i - kl < a.rot) v = rotated(a, c + a.rank, i - kl, p);
            const __nv_bfloat16 w = __float2bfloat16_rn(v);
            new_s[i] = w;
            if (blockIdx.y == 0) *reinterpret_cast<__nv_bfloat16*>(seq + dense_off(p, i, a.kv.seq_pad)) = w;
        }
    }
    if (threadIdx.x < kHeads) { m_s[threadIdx.x] = -INFINITY; l_s[threadIdx.x] = 0.0f; }
    __syncthreads();

    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;
    const float unit = a.scale * 1.4426950408889634f;
    const int steps_l = (a.rank + 15) / 16, steps_r = (a.rot + 15) / 16;
    const uint32_t q_off = ((lane >> 3) & 1) * 1024 + (lane >> 4) * 128 + (lane & 7) * 16;
    const uint32_t qh = ptx::smem_u32(q_hi) + q_off, ql = ptx::smem_u32(q_lo) + q_off;
    const uint32_t ph = ptx::smem_u32(p_hi) + q_off, pl = ptx::smem_u32(p_lo) + q_off;
    const uint32_t core = (lane >> 3) * 128 + (lane & 7) * 16;  // four pieces of eight positions

    for (int i = 0; i < blocks; ++i) {
        uint8_t* st = sm + (size_t)(i % stages) * stage_bytes;
        ok &= ptx::mbar_wait_bounded(&full[i % stages], (uint32_t)((i / stages) & 1));
        const int base = t0 + i * kKeys;
        if (owner && i == blocks - 1) {  // the new row has not been in the copy
            const int at = p - base;
            for (int c = threadIdx.x; c < chunks * 8; c += kSpanThreads)
                *reinterpret_cast<uint4*>(st + (c >> 3) * kKeys * 128 + (at >> 3) * 1024 + (c & 7) * 128 + (at & 7) * 16) = *reinterpret_cast<const uint4*>(new_s + c * 8);
            __syncthreads();
        }
        const uint32_t kv = ptx::smem_u32(st);
        float s[4][4] = {};  // hi and lo, even and odd steps
        auto score_steps = [&](int chunk0, int steps) {
            for (int k = 0; k < steps; k += 2) {
                const uint32_t q0 = (uint32_t)((chunk0 + (k >> 2)) * 2048 + (k & 3) * 256);
                uint32_t kf[4], qa[4];
                ptx::ldsm4(kf, kv + (chunk0 + (k >> 2)) * kKeys * 128 + warp * 1024 + (k & 3) * 256 + core);
                ptx::ldsm4(qa, qh + q0);
                ptx::mma_bf16(s[0], qa, kf[0], kf[1]);
                ptx::ldsm4(qa, ql + q0);
                ptx::mma_bf16(s[1], qa, kf[0], kf[1]);
                ptx::ldsm4(qa, qh + q0 + 256);
                ptx::mma_bf16(s[2], qa, kf[2], kf[3]);
                ptx::ldsm4(qa, ql + q0 + 256);
                ptx::mma_bf16(s[3], qa, kf[2], kf[3]);
            }
        };
        score_steps(0, steps_l);     // an odd last step meets zeros of the padding
        score_steps(kcl, steps_r);
        {
            const int k0 = warp * 8 + (lane & 3) * 2;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int key = k0 + (j & 1), h = (lane >> 2) + (j >> 1) * 8;
                s_s[h * kKeys + key] = base + key < t1 ? (s[0][j] + s[1][j] + s[2][j] + s[3][j]) * unit : -INFINITY;
            }
        }
        __syncthreads();
        if (threadIdx.x == 0) load(i + stages - 1);  // into the slot of the block before this one
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int h = warp * 2 + j;
            const float2 x = *reinterpret_cast<const float2*>(s_s + h * kKeys + lane * 2);
            const float m_old = m_s[h], m_new = fmaxf(m_old, warp_max(fmaxf(x.x, x.y)));
            const float e0 = ex2(x.x - m_new), e1 = ex2(x.y - m_new);
            const float sum = warp_sum(e0 + e1);
            const uint32_t hi = ptx::pack2(e0, e1);
            const int o = (h >> 3) * 1024 + (lane >> 2) * 128 + (h & 7) * 16 + (lane & 3) * 4;
            *reinterpret_cast<uint32_t*>(p_hi + o) = hi;
            *reinterpret_cast<uint32_t*>(p_lo + o) = ptx::pack2(e0 - __uint_as_float(hi << 16), e1 - __uint_as_float(hi & 0xffff0000u));
            __syncwarp();
            if (lane == 0) {
                const float al = ex2(m_old - m_new);  // 0 for the first block
                al_s[h] = al;
                m_s[h] = m_new;
                l_s[h] = l_s[h] * al + sum;
            }
        }
        __syncthreads();
        const float al0 = al_s[lane >> 2], al1 = al_s[(lane >> 2) + 8];
#pragma unroll
        for (int n = 0; n < NT; ++n) { acc[n][0] *= al0; acc[n][1] *= al0; acc[n][2] *= al1; acc[n][3] *= al1; }
#pragma unroll
        for (int k = 0; k < kKeys / 16; ++k) {
            uint32_t hi[4], lo[4];
            ptx::ldsm4(hi, ph + k * 256);
            ptx::ldsm4(lo, pl + k * 256);
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                const int col = (warp * NT + n) * 8;
                if (col < a.rank) {
                    uint32_t vf[4];  // (positions 0-7, 8-15) x (columns 0-7, 8-15)
                    ptx::ldsm4t(vf, kv + (col >> 6) * kKeys * 128 + (2 * k + ((lane >> 3) & 1)) * 1024 + (((col & 63) >> 3) + (lane >> 4)) * 128 + (lane & 7) * 16);
                    ptx::mma_bf16(acc[n], hi, vf[0], vf[1]);
                    ptx::mma_bf16(acc[n + 1], hi, vf[2], vf[3]);
                    ptx::mma_bf16(acc[n], lo, vf[0], vf[1]);
                    ptx::mma_bf16(acc[n + 1], lo, vf[2], vf[3]);
                }
            }
        }
    }
    __syncthreads();  // the ring is free
    constexpr int W = 64 * NT;
    float* o_s = reinterpret_cast<float*>(sm);  // [16][W], in the ring's place
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int j = 0; j < 4; ++j) o_s[((lane >> 2) + (j >> 1) * 8) * W + (warp * NT + n) * 8 + (lane & 3) * 2 + (j & 1)] = acc[n][j];
    if (!ok) atomicExch(err, kErrLatentTimeout);
    merge_spans<true>(a, m_s, l_s, o_s, W, nh, head0, r, split, splits, out);
}

// ---------------------------------------------------------------------------------------
// the same in f32 on the FMA units (32-bit models): 8 heads per CTA, tiles of 32 positions
// ---------------------------------------------------------------------------------------
constexpr int kF32Heads = 8, kF32Keys = 32;
__global__ void __launch_bounds__(kSpanThreads) latent_span_f32_kernel(const LatentAttn a, bool prepared, int splits, const ActOut out) {
    extern __shared__ __align__(16) float fs[];
    const int D = a.rank + a.rot, W = a.rank;
    float* q_s = fs;                          // [8][D]
    float* o_s = q_s + kF32Heads * D;         // [8][rank]
    float* p_s = o_s + kF32Heads * W;         // [8][32]
    float* m_s = p_s + kF32Heads * kF32Keys;
    float* l_s = m_s + kF32Heads;
    float* al_s = l_s + kF32Heads;
    float* red = al_s + kF32Heads;            // 32
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
    for (int i = threadIdx.x; i < kF32Heads * D; i += kSpanThreads) {
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
        for (int i = threadIdx.x; i < D; i += kSpanThreads) dst[i] = i < a.rank ? c[i] * inv * a.c_norm[i] : rotated(a, c + a.rank, i - a.rank, p);
    }
    if (threadIdx.x < kF32Heads) { m_s[threadIdx.x] = -INFINITY; l_s[threadIdx.x] = 0.0f; }
    __syncthreads();
    float acc[kF32Heads][kMaxRank / kSpanThreads] = {};
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
            for (int j = 0; j < kMaxRank / kSpanThreads; ++j) acc[h][j] *= al_s[h];
        const int n = min(kF32Keys, t1 - base);
        for (int k = 0; k < n; ++k)
#pragma unroll
            for (int j = 0; j < kMaxRank / kSpanThreads; ++j) {
                const int c = threadIdx.x + j * kSpanThreads;
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
        for (int j = 0; j < kMaxRank / kSpanThreads; ++j) {
            const int c = threadIdx.x + j * kSpanThreads;
            if (c < a.rank) o_s[h * W + c] = acc[h][j];
        }
    merge_spans<false>(a, m_s, l_s, o_s, W, nh, head0, r, split, splits, out);
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
int span_splits(const LatentAttn& a, int64_t groups) {
    int splits = 1;
    while (splits < 8 && groups * splits * 2 <= a.sm_count && splits * 64 < a.kv.max_seq) splits *= 2;
    return splits;
}

constexpr size_t kSpanSmem = 220 * 1024;
template <int NT>
cudaError_t span_launch(const LatentAttn& a, bool prepared, const ActOut& out, unsigned int* err, cudaStream_t s, bool pdl) {
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(latent_span_mma_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSpanSmem); });
    if (e != cudaSuccess) return e;
    const int chunks = (dense_kpad(a.rank) + dense_kpad(a.rot)) / 64, hg = (a.heads + kHeads - 1) / kHeads;
    const size_t stage = (size_t)chunks * kKeys * 128, fixed = span_fixed_bytes(chunks);
    int stages = (int)((kSpanSmem - fixed) / stage);
    if (stages < 2) return cudaErrorInvalidConfiguration;
    // up to 110 KB: two CTAs share an SM; the ring must also take the outputs
    const int small = (int)((110 * 1024 - fixed) / stage);
    stages = small >= 2 && 110 * 1024 > fixed ? small : stages;
    if (stages > 4) stages = 4;
    size_t ring = stages * stage;
    const size_t outs = (size_t)kHeads * 64 * NT * sizeof(float);
    while (ring < outs) { ++stages; ring += stage; }
    const int64_t rows = (int64_t)a.batch * a.q_rows;
    const int splits = span_splits(a, rows * hg);
    return launch_cluster(latent_span_mma_kernel<NT>, dim3((unsigned)splits, (unsigned)hg, (unsigned)rows), kSpanThreads, ring + fixed, s, pdl,
                          a, prepared, splits, stages, err, out);
}

}  // namespace

int latent_max_rank() { return kMaxRank; }
int latent_max_rot() { return kMaxRot; }

cudaError_t launch_latent_prep(const LatentAttn& a, cudaStream_t s) {
    latent_prep_kernel<<<(unsigned)(a.batch * a.q_rows), 256, 0, s>>>(a);
    return cudaGetLastError();
}

cudaError_t launch_latent_span(const LatentAttn& a, bool prepared, const ActOut& out, cudaStream_t s, bool pdl) {
    if (a.rank > kMaxRank || a.rot > kMaxRot || (!prepared && a.q_rows != 1)) return cudaErrorInvalidValue;
    if (a.kv.f32) {
        static PerDeviceOnce once;
        cudaError_t e = once.run([] { return cudaFuncSetAttribute(latent_span_f32_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024); });
        if (e != cudaSuccess) return e;
        const int hg = (a.heads + kF32Heads - 1) / kF32Heads;
        const int64_t rows = (int64_t)a.batch * a.q_rows;
        const int splits = span_splits(a, rows * hg);
        const size_t smem = ((size_t)kF32Heads * (2 * a.rank + a.rot) + kF32Heads * kF32Keys + 3 * kF32Heads + 32) * sizeof(float);
        return launch_cluster(latent_span_f32_kernel, dim3((unsigned)splits, (unsigned)hg, (unsigned)rows), kSpanThreads, smem, s, pdl, a, prepared, splits, out);
    }
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    unsigned int* err = device_error_word(dev);
    if (a.rank <= 128) return span_launch<2>(a, prepared, out, err, s, pdl);
    if (a.rank <= 256) return span_launch<4>(a, prepared, out, err, s, pdl);
    return span_launch<8>(a, prepared, out, err, s, pdl);
}

}  // namespace bt
