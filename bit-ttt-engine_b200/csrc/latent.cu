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
        float ms[kMaxSplits], ls[kMaxSplits], os[kMaxSplits], m = -INFINITY;
#pragma unroll
        for (int s = 0; s < kMaxSplits; ++s) {  // all remote reads in flight together
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
        for (int s = 0; s < kMaxSplits; ++s) {
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
// one query position, 16 MT heads, on the tensor cores (bf16 cache)
// ---------------------------------------------------------------------------------------
// The cache is laid out in core matrices (8 positions x 16 bytes), so blocks of 32 positions arrive as one bulk copy per 64
// columns and every ldmatrix reads 128 consecutive bytes.  Per block: sixteen warps share the scores' product, eight parts of
// the columns (each warp has its part of the queries in registers) x 16 positions, and leave partial scores; then each makes
// the softmax of MT heads and multiplies its 8 NT latent columns.  Softmax weights enter their product as bf16 hi + lo.
constexpr int kSpanThreads = 512, kSpanWarps = kSpanThreads / 32, kKeys = 32, kMaxSteps = (kMaxRank + kMaxRot) / 16 / 8;
constexpr int kScoreLd = 40;  // floats per row of partial scores

template <int MT>
struct SpanCfg {
    static constexpr int H = 16 * MT;
    static constexpr size_t kPart = (size_t)8 * H * kScoreLd * 4;  // partial scores; first the queries
    static size_t part(int chunks) { const size_t q = (size_t)chunks * MT * 2048; return q > kPart ? q : kPart; }
    static size_t fixed(int chunks) { return part(chunks) + (size_t)MT * 2 * 1024 + 3 * H * 4 + 32 * 4 + (size_t)chunks * 128 + 64; }
};

template <int NT, int MT>
__global__ void __launch_bounds__(kSpanThreads, 1) latent_span_mma_kernel(const LatentAttn a, bool prepared, int splits, int stages,
                                                                       int part_bytes, unsigned int* err, const ActOut out) {
    constexpr int NH = 16 * MT, NS = MT;  // heads of the CTA; of a warp in the softmax
    extern __shared__ __align__(128) uint8_t sm[];
    const int kcl = dense_kpad(a.rank) / 64, chunks = kcl + dense_kpad(a.rot) / 64;
    const int stage_bytes = chunks * kKeys * 128;
    uint8_t* q_s = sm + (size_t)stages * stage_bytes;    // [chunk][MT][2 groups of 8 heads][8 pieces][8 heads][16 bytes]
    float* s_s = reinterpret_cast<float*>(q_s);          // [8 warps][heads][kScoreLd]
    uint8_t* p_hi = q_s + part_bytes;                    // softmax weights [MT][16 heads][32 positions], core matrices
    uint8_t* p_lo = p_hi + MT * 1024;
    float* m_s = reinterpret_cast<float*>(p_lo + MT * 1024);
    float* l_s = m_s + NH;
    float* al_s = l_s + NH;
    float* red = al_s + NH;
    __nv_bfloat16* new_s = reinterpret_cast<__nv_bfloat16*>(red + 32);  // the new token's row [chunks * 64]
    uint64_t* full = reinterpret_cast<uint64_t*>(new_s + chunks * 64);  // up to eight
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int H = a.heads, hd = a.dim + a.rot;
    const int head0 = blockIdx.y * NH, nh = min(NH, H - head0);
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
    auto load = [&](int i, int slot) {  // warp 0: the i-th block of the span, a lane per 64 columns
        if (i >= blocks) return;
        if (lane == 0) ptx::mbar_arrive_expect_tx(&full[slot], stage_bytes);
        __syncwarp();
        if (lane < chunks)
            ptx::bulk_g2s(sm + (size_t)slot * stage_bytes + lane * kKeys * 128, seq + ((int64_t)lane * a.kv.seq_pad + t0 + i * kKeys) * 128, kKeys * 128, &full[slot]);
    };
    if (prepared) ptx::pdl_wait();  // the cache rows come from the kernel in front
    if (warp == 0)
        for (int i = 0; i < stages - 1; ++i) load(i, i);
    if (!prepared) ptx::pdl_wait();
    ptx::pdl_launch_dependents();

    // ---- queries: [absorbed | rotated] ----
    const float* row = a.proj + r * a.ld;
    const int kl = kcl * 64;
    for (int i = threadIdx.x; i < NH * chunks * 32; i += kSpanThreads) {  // two columns at a time
        const int h = i / (chunks * 32), c = (i - h * chunks * 32) * 2;
        float v[2] = {0.0f, 0.0f};
        if (h < nh)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                if (c < kl) { if (c + j < a.rank) v[j] = a.q_abs[(r * H + head0 + h) * a.rank + c + j]; }
                else if (c + j - kl < a.rot) v[j] = prepared ? a.q_rot[(r * H + head0 + h) * a.rot + c + j - kl] : rotated(a, row + (head0 + h) * hd + a.dim, c + j - kl, p);
            }
        *reinterpret_cast<uint32_t*>(q_s + (c >> 6) * MT * 2048 + (h >> 3) * 1024 + ((c & 63) >> 3) * 128 + (h & 7) * 16 + (c & 7) * 2) = ptx::pack2(v[0], v[1]);
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
    __syncthreads();
    // this warp's 16-column steps: part, part + 8, ... of the latent part's and the rotated part's
    const int part = warp & 7, half = warp >> 3;
    const int steps_l = (a.rank + 15) / 16, steps = steps_l + (a.rot + 15) / 16;
    uint32_t qf[kMaxSteps][MT][4];
    uint32_t k_off[kMaxSteps];
#pragma unroll
    for (int i = 0; i < kMaxSteps; ++i) {
        const int ks = part + 8 * i, kk = ks < steps_l ? ks : ks - steps_l + kcl * 4;
        k_off[i] = (uint32_t)((kk >> 2) * kKeys * 128 + (kk & 3) * 256 + half * 2048);
        if (ks < steps)
#pragma unroll
            for (int m = 0; m < MT; ++m)
                ptx::ldsm4(qf[i][m], ptx::smem_u32(q_s) + ((kk >> 2) * MT + m) * 2048 + (kk & 3) * 256 + ((lane >> 3) & 1) * 1024 + (lane >> 4) * 128 + (lane & 7) * 16);
    }
    __syncthreads();  // the partial scores take the queries' place

    float acc[MT][NT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[m][i][j] = 0.0f;
    float m_run[NS], l_run[NS];  // heads NS warp ..: maximum; this lane's share of the sum
#pragma unroll
    for (int j = 0; j < NS; ++j) { m_run[j] = -INFINITY; l_run[j] = 0.0f; }
    const float unit = a.scale * 1.4426950408889634f;
    const uint32_t p_off = ((lane >> 3) & 1) * 512 + (lane >> 4) * 128 + (lane & 7) * 16;
    const uint32_t ph = ptx::smem_u32(p_hi) + p_off, pl = ptx::smem_u32(p_lo) + p_off;
    const uint32_t k_core = (lane >> 4) * 1024 + ((lane >> 3) & 1) * 128 + (lane & 7) * 16;  // two groups of positions x two pieces

    int slot = 0, before = stages - 1;  // ring slots of this block and of the one before it
    uint32_t parity = 0;
    for (int i = 0; i < blocks; ++i) {
        uint8_t* st = sm + (size_t)slot * stage_bytes;
        ok &= ptx::mbar_wait_bounded(&full[slot], parity);
        const int base = t0 + i * kKeys;
        if (owner && i == blocks - 1) {  // the new row has not been in the copy
            const int at = p - base;
            for (int c = threadIdx.x; c < chunks * 8; c += kSpanThreads)
                *reinterpret_cast<uint4*>(st + (c >> 3) * kKeys * 128 + (at >> 3) * 1024 + (c & 7) * 128 + (at & 7) * 16) = *reinterpret_cast<const uint4*>(new_s + c * 8);
            __syncthreads();
        }
        const uint32_t kv = ptx::smem_u32(st);
        {
            float s[MT][2][4] = {};
#pragma unroll
            for (int k = 0; k < kMaxSteps; ++k)
                if (part + 8 * k < steps) {
                    uint32_t kf[4];
                    ptx::ldsm4(kf, kv + k_off[k] + k_core);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        ptx::mma_bf16(s[m][0], qf[k][m], kf[0], kf[1]);
                        ptx::mma_bf16(s[m][1], qf[k][m], kf[2], kf[3]);
                    }
                }
            float* sp = s_s + (part * NH + (lane >> 2)) * kScoreLd + half * 16 + (lane & 3) * 2;
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int g = 0; g < 2; ++g) {
                    *reinterpret_cast<float2*>(sp + m * 16 * kScoreLd + g * 8) = make_float2(s[m][g][0], s[m][g][1]);
                    *reinterpret_cast<float2*>(sp + (m * 16 + 8) * kScoreLd + g * 8) = make_float2(s[m][g][2], s[m][g][3]);
                }
        }
        __syncthreads();
        if (warp == 0) load(i + stages - 1, before);  // into the slot of the block before this one
        {
            float x[NS], mx[NS];
#pragma unroll
            for (int j = 0; j < NS; ++j) {
                const float* sp = s_s + (warp * NS + j) * kScoreLd + lane;
                float v = 0.0f;
#pragma unroll
                for (int w = 0; w < 8; ++w) v += sp[w * NH * kScoreLd];
                x[j] = base + lane < t1 ? v * unit : -INFINITY;
                mx[j] = x[j];
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int j = 0; j < NS; ++j) mx[j] = fmaxf(mx[j], __shfl_xor_sync(0xffffffffu, mx[j], o));
#pragma unroll
            for (int j = 0; j < NS; ++j) {
                const int h = warp * NS + j;
                const float m_new = fmaxf(m_run[j], mx[j]), al = ex2(m_run[j] - m_new), e = ex2(x[j] - m_new);  // al: 0 for the first block
                m_run[j] = m_new;
                l_run[j] = fmaf(l_run[j], al, e);
                const __nv_bfloat16 hi = __float2bfloat16_rn(e);
                const int o = (h >> 4) * 1024 + ((h >> 3) & 1) * 512 + (lane >> 3) * 128 + (h & 7) * 16 + (lane & 7) * 2;
                *reinterpret_cast<__nv_bfloat16*>(p_hi + o) = hi;
                *reinterpret_cast<__nv_bfloat16*>(p_lo + o) = __float2bfloat16_rn(e - __bfloat162float(hi));
                if (lane == 0) al_s[h] = al;
            }
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float al0 = al_s[m * 16 + (lane >> 2)], al1 = al_s[m * 16 + (lane >> 2) + 8];
            if (__any_sync(0xffffffffu, al0 != 1.0f || al1 != 1.0f))
#pragma unroll
                for (int n = 0; n < NT; ++n) { acc[m][n][0] *= al0; acc[m][n][1] *= al0; acc[m][n][2] *= al1; acc[m][n][3] *= al1; }
        }
        const int col0 = warp * NT * 8;
        if (col0 < a.rank) {
            uint32_t hi[2][MT][4], lo[2][MT][4];
#pragma unroll
            for (int k = 0; k < 2; ++k)
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    ptx::ldsm4(hi[k][m], ph + m * 1024 + k * 256);
                    ptx::ldsm4(lo[k][m], pl + m * 1024 + k * 256);
                }
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                const int col = col0 + n * 8;
                uint32_t vf[4];  // 8 columns of the four groups of positions
                ptx::ldsm4t(vf, kv + (col >> 6) * kKeys * 128 + ((col & 63) >> 3) * 128 + (lane >> 3) * 1024 + (lane & 7) * 16);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    ptx::mma_bf16(acc[m][n], hi[0][m], vf[0], vf[1]);
                    ptx::mma_bf16(acc[m][n], lo[0][m], vf[0], vf[1]);
                    ptx::mma_bf16(acc[m][n], hi[1][m], vf[2], vf[3]);
                    ptx::mma_bf16(acc[m][n], lo[1][m], vf[2], vf[3]);
                }
            }
        }
        before = slot;
        if (++slot == stages) { slot = 0; parity ^= 1; }
    }
#pragma unroll
    for (int j = 0; j < NS; ++j) {
        const float l = warp_sum(l_run[j]);
        if (lane == 0) { m_s[warp * NS + j] = m_run[j]; l_s[warp * NS + j] = l; }
    }
    __syncthreads();  // the ring is free
    constexpr int W = 8 * kSpanWarps * NT;
    float* o_s = reinterpret_cast<float*>(sm);  // [heads][W], in the ring's place
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int j = 0; j < 4; ++j) o_s[(m * 16 + (lane >> 2) + (j >> 1) * 8) * W + (warp * NT + n) * 8 + (lane & 3) * 2 + (j & 1)] = acc[m][n][j];
    if (!ok) atomicExch(err, kErrLatentTimeout);
    merge_spans<true>(a, m_s, l_s, o_s, W, nh, head0, r, split, splits, out);
}

// ---------------------------------------------------------------------------------------
// the same in f32 on the FMA units (32-bit models): 8 heads per CTA, tiles of 32 positions
// ---------------------------------------------------------------------------------------
constexpr int kF32Heads = 8, kF32Keys = 32, kF32Threads = 256;
__global__ void __launch_bounds__(kF32Threads) latent_span_f32_kernel(const LatentAttn a, bool prepared, int splits, const ActOut out) {
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
    while (splits < kMaxSplits && groups * splits * 2 <= a.sm_count && splits * 64 < a.kv.max_seq) splits *= 2;
    return splits;
}

constexpr size_t kSpanSmem = 220 * 1024;
template <int NT, int MT>
cudaError_t span_launch(const LatentAttn& a, bool prepared, const ActOut& out, unsigned int* err, cudaStream_t s, bool pdl) {
    static PerDeviceOnce once;
    cudaError_t e = once.run([] {
        cudaError_t x = cudaFuncSetAttribute(latent_span_mma_kernel<NT, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSpanSmem);
        return x != cudaSuccess ? x : cudaFuncSetAttribute(latent_span_mma_kernel<NT, MT>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    });
    if (e != cudaSuccess) return e;
    const int chunks = (dense_kpad(a.rank) + dense_kpad(a.rot)) / 64, hg = (a.heads + 16 * MT - 1) / (16 * MT);
    const size_t stage = (size_t)chunks * kKeys * 128, fixed = SpanCfg<MT>::fixed(chunks), outs = (size_t)16 * MT * 8 * kSpanWarps * NT * sizeof(float);
    // six blocks in flight where two CTAs then share an SM, else as many as fit; the ring must also take the outputs
    int stages = 6;
    if (stages * stage + fixed > 110 * 1024) stages = (int)((kSpanSmem - fixed) / stage) < 6 ? (int)((kSpanSmem - fixed) / stage) : 6;
    while (stages * stage < outs) ++stages;
    if (stages < 2 || stages > 8 || stages * stage + fixed > kSpanSmem) return cudaErrorInvalidConfiguration;
    const int64_t rows = (int64_t)a.batch * a.q_rows;
    const int splits = span_splits(a, rows * hg);
    return launch_cluster(latent_span_mma_kernel<NT, MT>, dim3((unsigned)splits, (unsigned)hg, (unsigned)rows), kSpanThreads, stages * stage + fixed, s, pdl,
                          a, prepared, splits, stages, (int)SpanCfg<MT>::part(chunks), err, out);
}
template <int NT>
cudaError_t span_launch_m(const LatentAttn& a, bool prepared, const ActOut& out, unsigned int* err, cudaStream_t s, bool pdl) {
    // 32 heads share the cache rows once that leaves no SM idle
    const bool wide = a.heads > 16 && (int64_t)a.batch * a.q_rows * ((a.heads + 31) / 32) * 4 >= a.sm_count;
    return wide ? span_launch<NT, 2>(a, prepared, out, err, s, pdl) : span_launch<NT, 1>(a, prepared, out, err, s, pdl);
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
        cudaError_t e = once.run([] {
            cudaError_t x = cudaFuncSetAttribute(latent_span_f32_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
            return x != cudaSuccess ? x : cudaFuncSetAttribute(latent_span_f32_kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
        });
        if (e != cudaSuccess) return e;
        const int hg = (a.heads + kF32Heads - 1) / kF32Heads;
        const int64_t rows = (int64_t)a.batch * a.q_rows;
        const int splits = span_splits(a, rows * hg);
        const size_t smem = ((size_t)kF32Heads * (2 * a.rank + a.rot) + kF32Heads * kF32Keys + 3 * kF32Heads + 32) * sizeof(float);
        return launch_cluster(latent_span_f32_kernel, dim3((unsigned)splits, (unsigned)hg, (unsigned)rows), kF32Threads, smem, s, pdl, a, prepared, splits, out);
    }
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    unsigned int* err = device_error_word(dev);
    if (a.rank <= 128) return span_launch_m<1>(a, prepared, out, err, s, pdl);
    if (a.rank <= 256) return span_launch_m<2>(a, prepared, out, err, s, pdl);
    return span_launch_m<4>(a, prepared, out, err, s, pdl);
}

}  // namespace bt
