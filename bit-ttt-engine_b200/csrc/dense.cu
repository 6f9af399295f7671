// Dense bf16 projections: streaming product for up to 8 rows (f32 activations), tcgen05 product for more (bf16
// activations), f32 product for 32-bit models; each also block-diagonal, the last two also over rows grouped by expert.  And
// the row kernels around them (embedding with learned positions, output norm + residual + next norm, norm in equal parts).
#include "bt_dense.cuh"
#include "bt_ptx.cuh"

namespace bt {

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Sum over the block (multiple of 32 threads); `red` holds 33 floats and is reused by the next call.
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
    if (l == 0) red[w] = v;
    __syncthreads();
    float r = l < nw ? red[l] : 0.0f;
    r = warp_sum(r);
    __syncthreads();
    return r;
}

__device__ __forceinline__ float act_fn(int act, float v) {
    if (act == DACT_RELU2) { v = fmaxf(v, 0.0f); v *= v; }
    else if (act == DACT_TANH) v = tanhf(v);
    else if (act == DACT_DECAY) v = expf(-expf(v));
    return v;
}
__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float silu_fast(float v) { return __fdividef(v, 1.0f + __expf(-v)); }  // where the result is rounded to bf16
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float gelu_tanh_f(float v) { return 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v))); }

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    __nv_bfloat162 p = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&p);
}

// ---------------------------------------------------------------------------------------
// weights: f32 rows -> tiled bf16
// ---------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) dense_tile_kernel(const float* __restrict__ src, int rows, int k, int row0, int row_step,
                                                         uint8_t* __restrict__ tiles, int n_pad, int k_pad) {
    const int64_t total = (int64_t)rows * (k_pad / 8);
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int r = (int)(i / (k_pad / 8)), c0 = (int)(i % (k_pad / 8)) * 8;
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = c0 + j < k ? src[(int64_t)r * k + c0 + j] : 0.0f;
        uint4 u = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
        *reinterpret_cast<uint4*>(tiles + dense_off(row0 + r * row_step, c0, n_pad)) = u;
    }
}

// ---------------------------------------------------------------------------------------
// streaming product, up to 8 rows
// ---------------------------------------------------------------------------------------
// A warp works on 8 weight rows at a time: lane = row (lane & 7) x one of four 8-input pieces (lane >> 3), two loads
// of 16 bytes per block of 64 inputs.  `wk` warps of the CTA share a row group and take its input blocks in turn, the
// 16 / wk slots work on neighbouring row groups; partial sums meet in shared memory (double-buffered, one barrier per
// row group).  The loads of the next batch of blocks are in flight while a batch is multiplied, and the first batch is
// requested before the wait on the kernel in front.
constexpr int kStreamThreads = 512, kStreamWarps = 16, kBatch = 4;

struct StreamSeg {
    const uint8_t* w;
    int n, n_pad, ctas;
    float* out;
    int64_t ld, out_block;
    const float* bias;
    const float* mu;
    int act;
};
struct StreamArgs {
    StreamSeg seg[kMaxSegs];
    int nseg, blocks;  // blocks > 1: one segment, its CTAs once per block
    int k, k_pad;
    int wk;            // warps per row group: 1, 2, 4, 8, 16
    DenseIn in;
};

// out row `b` of the inputs: xs[0 .. kxp)
template <int B>
__device__ __forceinline__ void stream_input(const StreamArgs& a, const float* mu, int blk, bool first, float* xs, float* red) {
    const DenseIn& in = a.in;
    const int kp = a.k_pad, k = in.cat ? in.kx : a.k;  // columns of x
    const int kxp = in.cat ? dense_kpad(k) : kp;
    const float* x0 = in.x + (int64_t)blk * in.x_block;
    if (in.kind == DPRO_ROWS) {
#pragma unroll
        for (int b = 0; b < B; ++b)
            for (int c = threadIdx.x; c < kxp; c += kStreamThreads) xs[b * kp + c] = c < k ? x0[b * in.ld + c] : 0.0f;
    } else if (in.kind == DPRO_RESNORM) {
        for (int b = 0; b < B; ++b) {
            float ss = 0.0f;
            for (int c = threadIdx.x; c < kxp; c += kStreamThreads) {
                const float y = c < k ? x0[b * in.ld + c] : 0.0f;
                xs[b * kp + c] = y;
                ss = fmaf(y, y, ss);
            }
            ss = block_sum(ss, red);
            float inv = 1.0f / sqrtf(ss / (float)k + in.eps);
            float s2 = 0.0f;
            for (int c = threadIdx.x; c < k; c += kStreamThreads) {
                const float v = fmaf(xs[b * kp + c] * inv, in.w[c], in.h[(int64_t)b * k + c]);
                xs[b * kp + c] = v;
                s2 = fmaf(v, v, s2);
                if (blockIdx.x == 0 && in.h_out) in.h_out[(int64_t)b * k + c] = v;
            }
            if (in.next_w) {
                s2 = block_sum(s2, red);
                inv = 1.0f / sqrtf(s2 / (float)k + in.eps);
                for (int c = threadIdx.x; c < k; c += kStreamThreads) {
                    const float v = xs[b * kp + c] * inv * in.next_w[c];
                    xs[b * kp + c] = v;
                    if (blockIdx.x == 0 && in.n_out) in.n_out[(int64_t)b * k + c] = v;
                }
            }
        }
    } else if (in.kind == DPRO_CONV) {
        const int ch0 = blk * k;
        for (int b = 0; b < B; ++b) {
            const int p = in.pos[b];
            float* ring = in.ring + (int64_t)b * in.taps * in.channels;
            for (int c = threadIdx.x; c < kxp; c += kStreamThreads) {
                float v = 0.0f;
                if (c < k) {
                    const int ch = ch0 + c;
                    const float x = x0[b * in.ld + c];
                    v = in.conv_b[ch];
                    for (int back = in.taps - 1; back > 0; --back)
                        if (p >= back) v = fmaf(in.conv_w[(int64_t)ch * in.taps + in.taps - 1 - back], ring[(int64_t)((p - back) % in.taps) * in.channels + ch], v);
                    v = fmaf(in.conv_w[(int64_t)ch * in.taps + in.taps - 1], x, v);
                    if (first) ring[(int64_t)(p % in.taps) * in.channels + ch] = x;  // no CTA reads this slot at this position
                }
                xs[b * kp + c] = v;
            }
        }
    } else {
        const int part = k / in.groups;
        for (int b = 0; b < B; ++b) {
            if (in.groups == 1) {
                float ss = 0.0f;
                for (int c = threadIdx.x; c < kxp; c += kStreamThreads) {
                    const float y = c < k ? x0[b * in.ld + c] : 0.0f;
                    xs[b * kp + c] = y;
                    ss = fmaf(y, y, ss);
                }
                ss = block_sum(ss, red);
                const float inv = 1.0f / sqrtf(ss / (float)k + in.eps);
                for (int c = threadIdx.x; c < k; c += kStreamThreads) {
                    const float v = xs[b * kp + c] * inv * in.w[c];
                    xs[b * kp + c] = v;
                    if (blockIdx.x == 0 && in.n_out) in.n_out[(int64_t)b * k + c] = v;
                }
            } else {
                // a warp per part
                for (int c = k + threadIdx.x; c < kp; c += kStreamThreads) xs[b * kp + c] = 0.0f;
                for (int g = threadIdx.x >> 5; g < in.groups; g += kStreamWarps) {
                    const float* x = x0 + b * in.ld + (int64_t)g * part;
                    float ss = 0.0f;
                    for (int c = threadIdx.x & 31; c < part; c += 32) ss = fmaf(x[c], x[c], ss);
                    ss = warp_sum(ss);
                    const float inv = 1.0f / sqrtf(ss / (float)part + in.eps);
                    for (int c = threadIdx.x & 31; c < part; c += 32)
                        xs[b * kp + g * part + c] = x[c] * inv * in.w[g * part + c];
                }
            }
        }
    }
    if (mu)  // token shift; every thread finds its own columns as it left them above
        for (int b = 0; b < B; ++b) {
            const int p = in.pos[b];
            float* keep = in.shift + (int64_t)(p & 1) * in.shift_slot + (int64_t)b * k;
            const float* before = in.shift + (int64_t)((p + 1) & 1) * in.shift_slot + (int64_t)b * k;
            for (int c = threadIdx.x; c < k; c += kStreamThreads) {
                const float v = xs[b * kp + c], prev = p > 0 ? before[c] : 0.0f;
                if (blockIdx.x == 0) keep[c] = v;
                xs[b * kp + c] = fmaf(prev - v, mu[c], v);
            }
        }
    if (in.cat)
        for (int b = 0; b < B; ++b)
            for (int c = threadIdx.x; c < kp - kxp; c += kStreamThreads) xs[b * kp + kxp + c] = c < k ? in.cat[(int64_t)b * k + c] : 0.0f;
    __syncthreads();
}

// rows 2j and 2j + 1 as the two gates of a channel
__device__ __forceinline__ float rglru_step(const RgluStep& rg, float zr, float zi, float u, int ch, int b, int channels, int64_t ld, int p) {
    const float la = -8.0f * sigmoid_f(zr) * softplus_f(rg.lam[ch]);
    float* st = rg.state + (int64_t)b * channels + ch;
    const float s = fmaf(expf(la), p > 0 ? *st : 0.0f, sqrtf(-expm1f(2.0f * la)) * sigmoid_f(zi) * u);
    *st = s;
    return s * gelu_tanh_f(rg.y[b * ld + ch]);
}

template <int B>
__global__ void __launch_bounds__(kStreamThreads, 1) dense_stream_kernel(const __grid_constant__ StreamArgs a) {
    extern __shared__ __align__(16) float xs[];  // [B][k_pad], then 2 x [16 warps][8 rows][B]
    __shared__ float red[33];
    float* part = xs + (size_t)B * a.k_pad;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int wk = a.wk, slots = kStreamWarps / wk;
    const int slot = warp / wk, kw = warp - slot * wk;
    int cta = blockIdx.x, blk = 0, si = 0;
    if (a.blocks > 1) {
        blk = cta / a.seg[0].ctas;
        cta -= blk * a.seg[0].ctas;
    } else {
        while (si + 1 < a.nseg && cta >= a.seg[si].ctas) cta -= a.seg[si++].ctas;
    }
    const StreamSeg& g = a.seg[si];
    const int groups = (g.n + 7) >> 3, chunks = a.k_pad / kDenseK;
    const int step = g.ctas * slots;
    const int64_t block_stride = (int64_t)g.n_pad * 128;
    const uint8_t* lane_base = g.w + (int64_t)blk * block_stride * chunks + lane * 16;

    uint4 buf[2][2 * kBatch];
    // batch `i` of row group rg: the input blocks kw + (i * kBatch + j) * wk
    auto fetch = [&](uint4 (&d)[2 * kBatch], int rg, int i) {
        const bool live = rg < groups;
        const uint8_t* p = lane_base + (int64_t)rg * 1024;
#pragma unroll
        for (int j = 0; j < kBatch; ++j) {
            const int kc = kw + (i * kBatch + j) * wk;
            if (live && kc < chunks) {
                d[2 * j] = __ldg(reinterpret_cast<const uint4*>(p + kc * block_stride));
                d[2 * j + 1] = __ldg(reinterpret_cast<const uint4*>(p + kc * block_stride + 512));
            } else {
                d[2 * j] = d[2 * j + 1] = make_uint4(0, 0, 0, 0);
            }
        }
    };
    const int per_rg = (chunks + wk * kBatch - 1) / (wk * kBatch);  // batches per row group (the same for every warp)
    int rg = cta * slots + slot;
    fetch(buf[0], rg, 0);
    ptx::pdl_wait();
    ptx::pdl_launch_dependents();
    stream_input<B>(a, g.mu, blk, cta == 0, xs, red);

    float acc[B];
#pragma unroll
    for (int b = 0; b < B; ++b) acc[b] = 0.0f;
    const float* xl = xs + (lane >> 3) * 8;
    auto multiply = [&](const uint4 (&d)[2 * kBatch], int i) {
#pragma unroll
        for (int j = 0; j < kBatch; ++j) {
            const int kc = kw + (i * kBatch + j) * wk;
            if (kc < chunks) {
#pragma unroll
                for (int hlf = 0; hlf < 2; ++hlf) {
                    const uint4 u = d[2 * j + hlf];
                    const float w0 = __uint_as_float(u.x << 16), w1 = __uint_as_float(u.x & 0xffff0000u);
                    const float w2 = __uint_as_float(u.y << 16), w3 = __uint_as_float(u.y & 0xffff0000u);
                    const float w4 = __uint_as_float(u.z << 16), w5 = __uint_as_float(u.z & 0xffff0000u);
                    const float w6 = __uint_as_float(u.w << 16), w7 = __uint_as_float(u.w & 0xffff0000u);
#pragma unroll
                    for (int b = 0; b < B; ++b) {
                        const float* x = xl + b * a.k_pad + kc * kDenseK + hlf * 32;
                        const float4 x0 = *reinterpret_cast<const float4*>(x), x1 = *reinterpret_cast<const float4*>(x + 4);
                        float r = acc[b];
                        r = fmaf(w0, x0.x, r); r = fmaf(w1, x0.y, r); r = fmaf(w2, x0.z, r); r = fmaf(w3, x0.w, r);
                        r = fmaf(w4, x1.x, r); r = fmaf(w5, x1.y, r); r = fmaf(w6, x1.z, r); r = fmaf(w7, x1.w, r);
                        acc[b] = r;
                    }
                }
            }
        }
    };
    int pb = 0;
    const int base_step = step;
    const bool pairs = g.act >= DACT_SWIGLU;
    for (int base = cta * slots; base < groups; base += base_step, rg += base_step, pb ^= 1) {
        // two batches per turn, so that the register buffers are indexed by constants
        for (int i = 0; i < per_rg; i += 2) {
            if (i + 1 < per_rg) fetch(buf[1], rg, i + 1);
            multiply(buf[0], i);
            if (i + 1 < per_rg) {
                if (i + 2 < per_rg) fetch(buf[0], rg, i + 2); else fetch(buf[0], rg + base_step, 0);
                multiply(buf[1], i + 1);
            } else {
                fetch(buf[0], rg + base_step, 0);
            }
        }
        float* pw = part + (size_t)pb * kStreamWarps * 8 * B;
#pragma unroll
        for (int b = 0; b < B; ++b) {
            float r = acc[b];
            r += __shfl_xor_sync(0xffffffffu, r, 8);
            r += __shfl_xor_sync(0xffffffffu, r, 16);
            if (lane < 8) pw[(warp * 8 + lane) * B + b] = r;
            acc[b] = 0.0f;
        }
        __syncthreads();
        for (int o = threadIdx.x; o < slots * 8 * B; o += kStreamThreads) {
            const int sl = o / (8 * B), e = o - sl * 8 * B, row = e / B, b = e - row * B;
            float v = 0.0f;
            for (int w = 0; w < wk; ++w) v += pw[(size_t)(sl * wk + w) * 8 * B + e];
            const int n = (base + sl) * 8 + row;
            if (n >= g.n) continue;
            if (g.bias) v += g.bias[(int64_t)blk * g.n + n];
            if (!pairs) {
                g.out[b * g.ld + blk * g.out_block + n] = act_fn(g.act, v);
            } else if ((row & 1) == 0) {
                float v2 = 0.0f;
                for (int w = 0; w < wk; ++w) v2 += pw[(size_t)(sl * wk + w) * 8 * B + e + B];
                if (g.bias) v2 += g.bias[(int64_t)blk * g.n + n + 1];
                const int f = n >> 1;
                if (g.act == DACT_SWIGLU) v = silu_f(v) * v2;
                else v = rglru_step(a.in.rg, v, v2, xs[b * a.k_pad + f], blk * a.k + f, b, a.in.channels, a.in.ld, a.in.pos[b]);
                g.out[b * g.ld + blk * g.out_block + f] = v;
            }
        }
    }
}

template <int B>
cudaError_t stream_launch(const StreamArgs& a, int grid, size_t smem, cudaStream_t s, bool pdl) {
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(dense_stream_kernel<B>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024); });
    if (e != cudaSuccess) return e;
    return launch_pdl(dense_stream_kernel<B>, dim3(grid), dim3(kStreamThreads), smem, s, pdl, a);
}
size_t stream_smem(const DenseLin& lin, int rows) {
    return ((size_t)rows * lin.k_pad + 2 * kStreamWarps * 8 * rows) * sizeof(float);
}

// ---------------------------------------------------------------------------------------
// tcgen05 product: A = 128 weight rows, B = NT token rows, K = 64 per stage, accumulators in TMEM (two sets)
// ---------------------------------------------------------------------------------------
constexpr int kTcRows = 128, kTcThreads = 6 * 32;
constexpr unsigned kErrDenseTimeout = 0x444e5354u;  // 'DNST'

__device__ __forceinline__ uint32_t tc_idesc(int n) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(kTcRows >> 4) << 24);  // f32 += bf16 . bf16
}

struct TcArgs {
    const uint8_t* w;
    const uint8_t* x;
    int n, n_pad, w_chunks, chunks;  // chunks: 64-input blocks of the input, hi and lo halves counted
    int64_t m, m_pad;
    int splits, blocks;
    int64_t w_block, x_block;        // bytes from one block to the next
    float* out;
    int64_t ld, part_stride, out_block;
    const float* bias;
    uint8_t* out_tiles;
    __nv_bfloat16* out_rows16;
    int n_out, act;                  // outputs of a block
    const ExpertTile* plan;          // rows grouped by expert (null: all rows in every block)
    const int* n_plan;
    unsigned int* err;
};

template <int NT>
struct TcCfg {
    static constexpr int kStageBytes = (kTcRows + NT) * 128;
    static constexpr int kStages = NT >= 256 ? 4 : (NT >= 128 ? 6 : 8);
    static constexpr int kEpi = 4 * 32 * (8 * 16 + 16);  // per epilogue warp: 32 tokens x 32 features of bf16, padded
    static constexpr size_t kSmem = (size_t)kStages * kStageBytes + kEpi + 256;
};

// What the epilogue does is a constant of the kernel: f32 rows as they are, f32 rows with bias and activation, tiled bf16
// (squared relu), gate and up pairs to tiled bf16, bf16 rows.
enum TcEpi : int { TC_ROWS, TC_ROWS_ACT, TC_TILES, TC_PAIRS, TC_ROWS16 };

template <int NT, int EPI>
__global__ void __launch_bounds__(kTcThreads, 1) dense_tc_kernel(const TcArgs a) {
    using Cfg = TcCfg<NT>;
    constexpr int S = Cfg::kStages;
    extern __shared__ __align__(128) uint8_t smem[];
    uint8_t* epi = smem + (size_t)S * Cfg::kStageBytes;
    uint64_t* full = reinterpret_cast<uint64_t*>(epi + Cfg::kEpi);
    uint64_t* empty = full + S;
    uint64_t* acc_full = empty + S;   // two accumulator sets
    uint64_t* acc_empty = acc_full + 2;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row_sets = a.n_pad / kTcRows;
    const int tok_blocks = a.plan ? *a.n_plan : (int)((a.m + NT - 1) / NT);
    const int tiles = row_sets * tok_blocks * a.splits * a.blocks;

    if (threadIdx.x == 0) {
        for (int s = 0; s < S; ++s) { ptx::mbar_init(&full[s], 1); ptx::mbar_init(&empty[s], 1); }
        for (int s = 0; s < 2; ++s) { ptx::mbar_init(&acc_full[s], 1); ptx::mbar_init(&acc_empty[s], 128); }
        ptx::mbar_fence_init();
    }
    if (warp == 1) { ptx::tmem_alloc(tmem_slot, 2 * NT); ptx::tmem_relinquish(); }
    ptx::tc_fence_before();
    __syncthreads();
    ptx::tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    bool ok = true;
    // tile -> (block, split, token block, row set): neighbouring CTAs share the activations of a token block
    struct Tile { int blk, rs, c0, c1, sp; int64_t tok0, tok_end; };
    auto decode = [&](int t) {
        Tile d;
        const int per = row_sets * tok_blocks, q = t / per, u = t - q * per, tb = u / row_sets;
        d.rs = u - tb * row_sets;
        if (a.plan) {
            const ExpertTile e = a.plan[tb];
            d.blk = e.expert; d.tok0 = e.row0; d.tok_end = e.row_end; d.sp = 0; d.c0 = 0; d.c1 = a.chunks;
            return d;
        }
        d.blk = a.splits > 1 ? 0 : q;
        d.sp = a.splits > 1 ? q : 0;
        d.c0 = (int)((int64_t)a.chunks * d.sp / a.splits);
        d.c1 = (int)((int64_t)a.chunks * (d.sp + 1) / a.splits);
        d.tok0 = (int64_t)tb * NT;
        d.tok_end = a.m;
        return d;
    };
    // an expert's tile is as wide as its rows need
    auto tile_rows = [&](const Tile& d) -> uint32_t { return a.plan ? (uint32_t)((d.tok_end - d.tok0 + 15) / 16 * 16) : (uint32_t)NT; };

    if (warp == 0) {
        if (lane == 0) {
            int slot = 0, issued = 0; uint32_t par = 1; bool first = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
                const Tile d = decode(t);
                const uint8_t* wp = a.w + (int64_t)d.blk * a.w_block + (int64_t)d.rs * kTcRows * 128;
                const uint8_t* xp = a.x + (a.plan ? 0 : (int64_t)d.blk * a.x_block) + d.tok0 * 128;
                const uint32_t x_bytes = tile_rows(d) * 128;
                for (int kc = d.c0; kc < d.c1; ++kc) {
                    const int wc = kc >= a.w_chunks ? kc - a.w_chunks : kc;  // hi and lo halves meet the same weights
                    if (!first) { if (!ptx::mbar_wait_bounded(&empty[slot], par)) { ok = false; break; } }
                    uint8_t* st = smem + (size_t)slot * Cfg::kStageBytes;
                    ptx::mbar_arrive_expect_tx(&full[slot], kTcRows * 128 + x_bytes);
                    ptx::bulk_g2s(st, wp + (int64_t)wc * a.n_pad * 128, kTcRows * 128, &full[slot]);
                    ptx::bulk_g2s(st + kTcRows * 128, xp + (int64_t)kc * a.m_pad * 128, x_bytes, &full[slot]);
                    ++issued;
                    if (++slot == S) { slot = 0; first = false; par ^= 1; }
                }
            }
            if (!ok)  // copies in flight land before the CTA gives up its shared memory
                for (int s = 0; s < S; ++s) {
                    const int fills = issued / S + (s < issued % S ? 1 : 0);
                    if (fills) ptx::mbar_wait_bounded(&full[s], (uint32_t)((fills - 1) & 1));
                }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            int slot = 0, set = 0; uint32_t par = 0, acc_par = 1; int done = 0;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, ++done) {
                const Tile d = decode(t);
                const uint32_t idesc = tc_idesc((int)tile_rows(d));
                if (done >= 2) ok &= ptx::mbar_spin_relaxed(&acc_empty[set], acc_par);
                ptx::tc_fence_after();
                for (int kc = d.c0; kc < d.c1 && ok; ++kc) {
                    ok &= ptx::mbar_spin_relaxed(&full[slot], par);
                    ptx::tc_fence_after();
                    const uint32_t a_addr = ptx::smem_u32(smem + (size_t)slot * Cfg::kStageBytes);
                    const uint32_t b_addr = a_addr + kTcRows * 128;
#pragma unroll
                    for (int ks = 0; ks < kDenseK / 16; ++ks)
                        ptx::umma_f16(tmem_base + set * NT, ptx::smem_desc(a_addr + ks * 256, 128, 1024),
                                      ptx::smem_desc(b_addr + ks * 256, 128, 1024), idesc, (kc > d.c0 || ks > 0) ? 1u : 0u);
                    ptx::umma_commit(&empty[slot]);
                    if (++slot == S) { slot = 0; par ^= 1; }
                }
                ptx::umma_commit(&acc_full[set]);
                set ^= 1;
                if (set == 0) acc_par ^= 1;
            }
        }
    } else {
        const int sub = warp & 3;
        uint8_t* stage = epi + (size_t)sub * 32 * (8 * 16 + 16);
        int set = 0; uint32_t acc_par = 0;
        for (int t = blockIdx.x; t < tiles; t += gridDim.x) {
            const Tile d = decode(t);
            ok &= ptx::mbar_wait_bounded(&acc_full[set], acc_par);
            ptx::tc_fence_after();
            const int f = d.rs * kTcRows + sub * 32 + lane;  // row of the block
            const int64_t tok0 = d.tok0, tok_end = d.tok_end;
            const float bias = EPI == TC_ROWS_ACT && a.bias && f < a.n ? a.bias[(int64_t)d.blk * a.n + f] : 0.0f;
            auto finish = [&](float x) { return EPI == TC_ROWS_ACT ? act_fn(a.act, x + bias) : x; };
#pragma unroll 1
            for (int q = 0; q < NT; q += 32) {
                if (tok0 + q >= tok_end) break;
                uint32_t v[32];
                ptx::tmem_ld32(tmem_base + ((uint32_t)(sub * 32) << 16) + set * NT + q, v);
                ptx::tmem_ld_wait();
                if (EPI == TC_PAIRS) {
                    // neighbouring lanes hold gate and up: the even one finishes the first 16 tokens, the odd one the others;
                    // pieces of (one token, 8 features) through shared memory, [token group][8 features][token]
#pragma unroll
                    for (int j = 0; j < 16; ++j) {
                        const uint32_t got = __shfl_xor_sync(0xffffffffu, (lane & 1) ? v[j] : v[j + 16], 1);
                        const float gate = __uint_as_float((lane & 1) ? got : v[j]), up = __uint_as_float((lane & 1) ? v[j + 16] : got);
                        const int tk = j + (lane & 1) * 16, ft = lane >> 1;
                        *reinterpret_cast<__nv_bfloat16*>(stage + ((tk >> 3) * 2 + (ft >> 3)) * 144 + (tk & 7) * 16 + (ft & 7) * 2) = __float2bfloat16_rn(silu_fast(gate) * up);
                    }
                    __syncwarp();
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        const int piece = i * 32 + lane, core = piece >> 3, tk = piece & 7;
                        const int64_t token = tok0 + q + (core >> 1) * 8 + tk;
                        const int feat = d.rs * (kTcRows / 2) + sub * 16 + (core & 1) * 8;
                        if (token < tok_end && feat < dense_kpad(a.n_out))
                            *reinterpret_cast<uint4*>(a.out_tiles + dense_off(token, feat, a.m_pad)) =
                                *reinterpret_cast<const uint4*>(stage + core * 144 + tk * 16);
                    }
                    __syncwarp();
                } else if (EPI == TC_TILES || EPI == TC_ROWS16) {
                    // through shared memory into 16-byte pieces (one token, 8 features): [token group][8 features][token]
#pragma unroll
                    for (int j = 0; j < 32; ++j) {
                        float r = __uint_as_float(v[j]);
                        if (EPI == TC_TILES && a.act == DACT_RELU2) { r = fmaxf(r, 0.0f); r *= r; }
                        *reinterpret_cast<__nv_bfloat16*>(stage + ((j >> 3) * 4 + (lane >> 3)) * 144 + (j & 7) * 16 + (lane & 7) * 2) = __float2bfloat16_rn(r);
                    }
                    __syncwarp();
                    const int col0 = EPI == TC_TILES ? (int)(d.blk * a.out_block) : 0;
                    const int limit = EPI == TC_TILES && col0 + a.n_out == a.blocks * a.n_out ? dense_kpad(col0 + a.n_out) - col0 : a.n_out;
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int piece = i * 32 + lane, core = piece >> 3, tk = piece & 7;  // core = token group * 4 + feature group
                        const int64_t token = tok0 + q + (core >> 2) * 8 + tk;
                        const int feat = d.rs * kTcRows + sub * 32 + (core & 3) * 8;
                        if (token < tok_end && feat < limit) {
                            void* dst = EPI == TC_TILES ? (void*)(a.out_tiles + dense_off(token, col0 + feat, a.m_pad))
                                                    : (void*)(a.out_rows16 + d.blk * a.out_block + token * a.ld + feat);
                            *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(stage + core * 144 + tk * 16);
                        }
                    }
                    __syncwarp();
                } else if (f < a.n) {
                    float* o = a.out + (int64_t)d.sp * a.part_stride + (a.plan ? 0 : d.blk * a.out_block) + (tok0 + q) * a.ld + f;
                    if (tok0 + q + 32 <= tok_end) {
#pragma unroll
                        for (int j = 0; j < 32; ++j) o[j * a.ld] = finish(__uint_as_float(v[j]));
                    } else {
#pragma unroll
                        for (int j = 0; j < 32; ++j)
                            if (tok0 + q + j < tok_end) o[j * a.ld] = finish(__uint_as_float(v[j]));
                    }
                }
            }
            ptx::tc_fence_before();
            ptx::mbar_arrive(&acc_empty[set]);
            set ^= 1;
            if (set == 0) acc_par ^= 1;
        }
    }
    if (!ok) atomicExch(a.err, kErrDenseTimeout);
    ptx::tc_fence_before();
    __syncthreads();
    if (warp == 1) ptx::tmem_dealloc(tmem_base, 2 * NT);
}

// sum of the partial products in the order of the splits, activation, f32 rows or tiled bf16
__global__ void __launch_bounds__(256) dense_reduce_kernel(const float* __restrict__ parts, int splits, int64_t part_stride,
                                                           int64_t pld, int64_t m, int n, int n_out, int act, float* __restrict__ out,
                                                           int64_t ld, uint8_t* __restrict__ tiles, int64_t m_pad, const float* __restrict__ bias) {
    const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
    const int64_t r = blockIdx.y;
    if (c0 >= n_out) return;
    float v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = 0.0f;
    for (int s = 0; s < splits; ++s) {
        const float* p = parts + s * part_stride + r * pld + c0;  // pld: multiple of 128, rows 16-byte aligned
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        v[0] += a.x; v[1] += a.y; v[2] += a.z; v[3] += a.w;
        v[4] += b.x; v[5] += b.y; v[6] += b.z; v[7] += b.w;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = c0 + j < n ? act_fn(act, v[j] + (bias ? bias[c0 + j] : 0.0f)) : 0.0f;
    if (tiles)
        *reinterpret_cast<uint4*>(tiles + dense_off(r, c0, m_pad)) =
            make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
    else
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (c0 + j < n) out[r * ld + c0 + j] = v[j];
}

template <int NT, int EPI>
cudaError_t tc_launch_e(const TcArgs& a, int sm_count, cudaStream_t s) {
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(dense_tc_kernel<NT, EPI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TcCfg<NT>::kSmem); });
    if (e != cudaSuccess) return e;
    const int64_t tiles = (int64_t)(a.n_pad / kTcRows) * ((a.m + NT - 1) / NT) * a.splits * a.blocks;  // a.m: the plan's upper bound
    dense_tc_kernel<NT, EPI><<<(unsigned)(tiles < sm_count ? tiles : sm_count), kTcThreads, TcCfg<NT>::kSmem, s>>>(a);
    return cudaGetLastError();
}
template <int NT>
cudaError_t tc_launch(const TcArgs& a, int sm_count, cudaStream_t s) {
    if (a.act == DACT_SWIGLU) return tc_launch_e<NT, TC_PAIRS>(a, sm_count, s);
    if (a.out_tiles) return tc_launch_e<NT, TC_TILES>(a, sm_count, s);
    if (a.out_rows16) return tc_launch_e<NT, TC_ROWS16>(a, sm_count, s);
    return a.bias || a.act != DACT_NONE ? tc_launch_e<NT, TC_ROWS_ACT>(a, sm_count, s) : tc_launch_e<NT, TC_ROWS>(a, sm_count, s);
}

// token rows per tile: 64 and 128 while one block covers them; above, 256 unless that leaves SMs idle
int tc_tokens(const DenseLin& lin, int64_t m, int sm_count, int blocks = 1) {
    if (m <= 64) return 64;
    if (m <= 128) return 128;
    const int64_t rs = (int64_t)blocks * lin.n_pad / kTcRows;
    const int64_t w256 = (rs * ((m + 255) / 256) + sm_count - 1) / sm_count * 2, w128 = (rs * ((m + 127) / 128) + sm_count - 1) / sm_count;
    return 4 * w128 < 3 * w256 ? 128 : 256;  // the smaller tile reads its operands twice as often
}
int tc_splits(const DenseLin& lin, int64_t m, int sm_count) {
    if (m > 128 || lin.blocks > 1) return 1;
    const int tiles = lin.n_pad / kTcRows, chunks = lin.k_pad / kDenseK;
    int s = sm_count / tiles;
    if (s > chunks / 4) s = chunks / 4;
    return s < 1 ? 1 : (s > 8 ? 8 : s);
}

// ---------------------------------------------------------------------------------------
// f32 product for 32-bit models: 64 x 64 outputs per CTA, 4 x 4 per thread
// ---------------------------------------------------------------------------------------
struct F32Args {
    const uint8_t* w;
    int n, n_pad, k, k_pad;
    int64_t w_block;
    const float* x;
    int64_t ldx, x_block, m;
    float* out;
    int64_t ld, out_block;
    const float* bias;
    int act;
    const int* row_start;  // rows grouped by expert: block z has counts[z] rows from row_start[z]
    const int* counts;
};
__global__ void __launch_bounds__(256) dense_f32_kernel(const F32Args a) {
    __shared__ float ws[32][68], xs[32][68];
    const int n0 = blockIdx.x * 64, blk = blockIdx.z;
    int64_t m0 = (int64_t)blockIdx.y * 64, m_end = a.m;
    if (a.row_start) {
        if (m0 >= a.counts[blk]) return;
        m0 += a.row_start[blk];
        m_end = (int64_t)a.row_start[blk] + a.counts[blk];
    }
    const uint8_t* w = a.w + blk * a.w_block;
    const float* x = a.x + (a.row_start ? 0 : blk * a.x_block);
    float* out = a.out + (a.row_start ? 0 : blk * a.out_block);
    const int tn = threadIdx.x & 15, tm = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < a.k_pad; k0 += 32) {
        __syncthreads();
        {   // weights: 64 rows x 32 inputs, one 16-byte piece per thread
            const int row = threadIdx.x & 63, c = (threadIdx.x >> 6) * 8;
            const uint4 u = *reinterpret_cast<const uint4*>(w + dense_off(n0 + row, k0 + c, a.n_pad));
            const uint32_t q[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                ws[c + 2 * j][row] = __uint_as_float(q[j] << 16);
                ws[c + 2 * j + 1][row] = __uint_as_float(q[j] & 0xffff0000u);
            }
        }
        for (int i = threadIdx.x; i < 64 * 32; i += 256) {
            const int row = i >> 5, c = i & 31;
            xs[c][row] = (m0 + row < m_end && k0 + c < a.k) ? x[(m0 + row) * a.ldx + k0 + c] : 0.0f;
        }
        __syncthreads();
#pragma unroll 8
        for (int c = 0; c < 32; ++c) {
            const float4 wv = *reinterpret_cast<const float4*>(&ws[c][tn * 4]);
            const float4 xv = *reinterpret_cast<const float4*>(&xs[c][tm * 4]);
            const float wr[4] = {wv.x, wv.y, wv.z, wv.w}, xr[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xr[i], wr[j], acc[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int64_t r = m0 + tm * 4 + i;
        if (r >= m_end) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int c = n0 + tn * 4 + j;
            if (c >= a.n) continue;
            if (a.bias) acc[i][j] += a.bias[(int64_t)blk * a.n + c];
            if (a.act != DACT_SWIGLU) out[r * a.ld + c] = act_fn(a.act, acc[i][j]);
            else if (j & 1) out[r * a.ld + (c >> 1)] = silu_f(acc[i][j - 1]) * acc[i][j];
        }
    }
}

// ---------------------------------------------------------------------------------------
// row kernels
// ---------------------------------------------------------------------------------------
// Eight consecutive columns of a row to the next projection's input (tiled: zero from k to the padded width).
__device__ __forceinline__ void put8(const ActOut& o, int64_t row, int c0, int k, const float (&v)[8]) {
    if (o.tiles)
        *reinterpret_cast<uint4*>(o.tiles + dense_off(row, c0, o.m_pad)) =
            make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
    if (o.rows)
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (c0 + j < k) o.rows[row * o.ld + c0 + j] = v[j];
}
__device__ __forceinline__ void get8(const float* p, int c0, int k, bool vec, float (&v)[8]) {
    if (vec && c0 + 8 <= k) {
        const float4 a = *reinterpret_cast<const float4*>(p + c0), b = *reinterpret_cast<const float4*>(p + c0 + 4);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = c0 + j < k ? p[c0 + j] : 0.0f;
    }
}

__global__ void __launch_bounds__(512) embed_pos_kernel(const int32_t* __restrict__ tokens, const __nv_bfloat16* __restrict__ table,
                                                        const __nv_bfloat16* __restrict__ pos_table, const int32_t* __restrict__ pos,
                                                        int q_rows, int hidden, int vocab, int max_pos, float* __restrict__ h,
                                                        const ActOut act, const ActOut act2) {
    ptx::pdl_wait();
    ptx::pdl_launch_dependents();
    const int64_t row = blockIdx.x;
    int tok = tokens[row];
    tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
    const __nv_bfloat16* e = table + (int64_t)tok * hidden;
    const __nv_bfloat16* pe = nullptr;
    if (pos_table) {
        int p = pos[row / q_rows] + (int)(row % q_rows);
        p = p < 0 ? 0 : (p >= max_pos ? max_pos - 1 : p);
        pe = pos_table + (int64_t)p * hidden;
    }
    for (int c0 = threadIdx.x * 8; c0 < dense_kpad(hidden); c0 += blockDim.x * 8) {
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int c = c0 + j;
            v[j] = c < hidden ? __bfloat162float(e[c]) + (pe ? __bfloat162float(pe[c]) : 0.0f) : 0.0f;
            if (c < hidden) h[row * hidden + c] = v[j];
        }
        put8(act, row, c0, hidden, v);
        put8(act2, row, c0, hidden, v);
    }
}

// Norm in equal parts of a multiple of eight columns: a warp per part and turn, the part in registers.
template <int NI>
__global__ void __launch_bounds__(256) group_norm_kernel(const RowArgs a, int part) {
    const int64_t row = blockIdx.x;
    const int k = a.k, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    ptx::pdl_wait();
    ptx::pdl_launch_dependents();
    const float* y = a.y + row * a.ld;
    const bool vec = (reinterpret_cast<uintptr_t>(y) & 15) == 0;
    for (int g = warp; g < a.groups; g += 8) {
        float v[NI][8];
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < NI; ++i) get8(y + g * part, (i * 32 + lane) * 8, part, vec, v[i]);
#pragma unroll
        for (int i = 0; i < NI; ++i)
#pragma unroll
            for (int j = 0; j < 8; ++j) ss = fmaf(v[i][j], v[i][j], ss);
        const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)part + a.eps);
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int c0 = (i * 32 + lane) * 8;
            if (c0 >= part) break;
            float w[8];
            get8(a.w + g * part, c0, part, true, w);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[i][j] = v[i][j] * inv * w[j];
            if (a.gate) {
                get8(a.gate + row * a.gate_ld + g * part, c0, part, false, w);
#pragma unroll
                for (int j = 0; j < 8; ++j) v[i][j] *= silu_f(w[j]);
            }
            put8(a.act, row, g * part + c0, k, v[i]);
        }
    }
    const float zero[8] = {};
    for (int c0 = k + (int)threadIdx.x * 8; c0 < dense_kpad(k); c0 += 256 * 8) put8(a.act, row, c0, k, zero);
}

// NC: groups of eight columns per thread; the whole row is requested before anything is computed.
template <int NC>
__global__ void __launch_bounds__(512) row_op_kernel(const RowArgs a) {
    __shared__ float red[33];
    extern __shared__ float inv_g[];
    const int64_t row = blockIdx.x;
    const int k = a.k, kp = dense_kpad(k);
    float v[NC][8], w[NC][8], h[NC][8];
#pragma unroll
    for (int i = 0; i < NC; ++i) get8(a.w, (i * blockDim.x + threadIdx.x) * 8, k, true, w[i]);
    ptx::pdl_wait();
    ptx::pdl_launch_dependents();
    const float* y = a.y + row * a.ld;
    const bool vec = (reinterpret_cast<uintptr_t>(y) & 15) == 0;
    const bool parts = a.op == ROW_GROUPNORM && a.groups > 1;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
        const int c0 = (i * blockDim.x + threadIdx.x) * 8;
        if (a.y) get8(y, c0, k, vec, v[i]);
        else
#pragma unroll
            for (int j = 0; j < 8; ++j) v[i][j] = 0.0f;
        if (a.op == ROW_RESNORM) get8(a.h_in + row * k, c0, k, (k & 3) == 0, h[i]);
    }
    for (int e = 0; e < a.top; ++e) {
        const float f = a.wt[row * a.top + e];
        const float* ye = a.ye + (int64_t)a.dst[row * a.top + e] * a.ye_ld;
        const bool evec = (reinterpret_cast<uintptr_t>(ye) & 15) == 0;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            float q[8];
            get8(ye, (i * blockDim.x + threadIdx.x) * 8, k, evec, q);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[i][j] = fmaf(f, q[j], v[i][j]);
        }
    }
    float inv = 0.0f;
    if (!parts) {
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < NC; ++i)
#pragma unroll
            for (int j = 0; j < 8; ++j) ss = fmaf(v[i][j], v[i][j], ss);
        ss = block_sum(ss, red);
        inv = 1.0f / sqrtf(ss / (float)k + a.eps);
    } else {
        // equal parts, a warp per part for the sums
        const int part = k / a.groups, nw = blockDim.x >> 5;
        for (int g = threadIdx.x >> 5; g < a.groups; g += nw) {
            float ss = 0.0f;
            for (int c = threadIdx.x & 31; c < part; c += 32) { const float x = y[g * part + c]; ss = fmaf(x, x, ss); }
            ss = warp_sum(ss);
            if ((threadIdx.x & 31) == 0) inv_g[g] = 1.0f / sqrtf(ss / (float)part + a.eps);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < NC; ++i) {
        const int c0 = (i * blockDim.x + threadIdx.x) * 8;
        if (c0 >= kp) break;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (parts) {
                v[i][j] = c0 + j < k ? v[i][j] * inv_g[(c0 + j) / (k / a.groups)] * w[i][j] : 0.0f;
                if (a.gate && c0 + j < k) v[i][j] *= silu_f(a.gate[row * a.gate_ld + c0 + j]);
            } else {
                v[i][j] = a.op == ROW_RESNORM ? fmaf(v[i][j] * inv, w[i][j], h[i][j]) : v[i][j] * inv * w[i][j];
                if (a.gate && c0 + j < k) v[i][j] *= silu_f(a.gate[row * a.gate_ld + c0 + j]);
            }
        }
        if (a.op == ROW_RESNORM) {
            float* o = a.h_out + row * k;
            if ((k & 3) == 0 && c0 + 8 <= k) {
                *reinterpret_cast<float4*>(o + c0) = make_float4(v[i][0], v[i][1], v[i][2], v[i][3]);
                *reinterpret_cast<float4*>(o + c0 + 4) = make_float4(v[i][4], v[i][5], v[i][6], v[i][7]);
            } else {
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    if (c0 + j < k) o[c0 + j] = v[i][j];
            }
        }
        if (!a.next_w) put8(a.act, row, c0, k, v[i]);
    }
    if (a.next_w) {
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            const int c0 = (i * blockDim.x + threadIdx.x) * 8;
#pragma unroll
            for (int j = 0; j < 8; ++j) ss = c0 + j < k ? fmaf(v[i][j], v[i][j], ss) : ss;
            get8(a.next_w, c0, k, true, w[i]);
        }
        ss = block_sum(ss, red);
        inv = 1.0f / sqrtf(ss / (float)k + a.eps);
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            const int c0 = (i * blockDim.x + threadIdx.x) * 8;
            if (c0 >= kp) break;
#pragma unroll
            for (int j = 0; j < 8; ++j) v[i][j] = c0 + j < k ? v[i][j] * inv * w[i][j] : 0.0f;
            put8(a.act, row, c0, k, v[i]);
        }
    }
}

// f32 rows in parts -> tiled bf16 (hi | lo): a thread per 8 columns of one row
__global__ void __launch_bounds__(256) rows_tile_kernel(const float* __restrict__ x, int64_t ld, int64_t x_block, int blocks, int k, int halves,
                                                        int act, int64_t rows, uint8_t* __restrict__ tiles, int64_t m_pad) {
    const int kp = dense_kpad(k), per = kp / 8;
    const int64_t total = rows * blocks * per;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int c0 = (int)(i % per) * 8, blk = (int)(i / per % blocks);
        const int64_t row = i / per / blocks;
        const float* p = x + row * ld + blk * x_block;
        float v[8], lo[8];
        get8(p, c0, k, (reinterpret_cast<uintptr_t>(p) & 15) == 0, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            v[j] = act_fn(act, v[j]);
            lo[j] = v[j] - __bfloat162float(__float2bfloat16_rn(v[j]));
        }
        ActOut o;
        o.tiles = tiles; o.m_pad = m_pad;
        put8(o, row, blk * halves * kp + c0, 0, v);
        if (halves == 2) put8(o, row, (blk * 2 + 1) * kp + c0, 0, lo);
    }
}

unsigned row_threads(int k) {
    const int t = (dense_kpad(k) / 8 + 31) / 32 * 32;
    return (unsigned)(t < 64 ? 64 : (t > 512 ? 512 : t));
}

}  // namespace

cudaError_t launch_dense_tile(const float* src, int rows, int k, int row0, const DenseLin& lin, cudaStream_t s, int row_step, int block) {
    if (k != lin.k || row0 < 0 || row_step < 1 || rows < 1 || row0 + (int64_t)(rows - 1) * row_step >= lin.n || block < 0 || block >= lin.blocks)
        return cudaErrorInvalidValue;
    dense_tile_kernel<<<1184, 256, 0, s>>>(src, rows, k, row0, row_step, lin.tiles + block * lin.block_bytes(), lin.n_pad, lin.k_pad);
    return cudaGetLastError();
}

bool dense_stream_fits(const DenseLin& lin, int rows) { return rows >= 1 && rows <= 8 && stream_smem(lin, rows) <= 220 * 1024; }

cudaError_t launch_dense_stream(const DenseLin& lin, const DenseIn& in, int rows, float* out, int64_t ld, int act,
                                int sm_count, cudaStream_t s, bool pdl) {
    DenseSeg seg;
    seg.lin = &lin; seg.out = out; seg.ld = ld; seg.act = act;
    return launch_dense_stream_segs(&seg, 1, in, rows, sm_count, s, pdl);
}

cudaError_t launch_dense_stream_segs(const DenseSeg* segs, int nseg, const DenseIn& in, int rows, int sm_count, cudaStream_t s, bool pdl) {
    if (nseg < 1 || nseg > kMaxSegs) return cudaErrorInvalidValue;
    const DenseLin& lin = *segs[0].lin;
    if (!dense_stream_fits(lin, rows) || (in.cat && lin.k != 2 * dense_kpad(in.kx))) return cudaErrorInvalidValue;
    StreamArgs a;
    a.nseg = nseg; a.blocks = lin.blocks; a.k = lin.k; a.k_pad = lin.k_pad; a.in = in;
    const int chunks = lin.k_pad / kDenseK;
    // as many warps per row group as there are input blocks: the finest spread of row groups over the SMs
    int wk = kStreamWarps;
    while (wk > chunks) wk >>= 1;
    a.wk = wk;
    const int slots = kStreamWarps / wk;
    int64_t groups = 0;
    for (int i = 0; i < nseg; ++i) {
        const DenseLin& l = *segs[i].lin;
        if (l.k != lin.k || (nseg > 1 && l.blocks != 1) || (segs[i].act >= DACT_SWIGLU && l.n % 2)) return cudaErrorInvalidValue;
        StreamSeg& g = a.seg[i];
        g.w = l.tiles; g.n = l.n; g.n_pad = l.n_pad; g.out = segs[i].out; g.ld = segs[i].ld; g.out_block = segs[i].out_block;
        g.bias = segs[i].bias; g.mu = segs[i].mu; g.act = segs[i].act;
        groups += (l.n + 7) / 8;
    }
    // the SMs in proportion to the segments' rows, or an equal share for every block
    int grid = 0;
    for (int i = 0; i < nseg; ++i) {
        const int g8 = (segs[i].lin->n + 7) / 8, blocks = (g8 + slots - 1) / slots;
        int share = lin.blocks > 1 ? sm_count / lin.blocks : (nseg > 1 ? (int)((int64_t)(sm_count - nseg) * g8 / groups) + 1 : sm_count);
        if (share < 1) share = 1;
        a.seg[i].ctas = blocks < share ? blocks : share;
        grid += a.seg[i].ctas;
    }
    grid *= lin.blocks;
    const size_t smem = stream_smem(lin, rows);
    switch (rows) {
        case 1: return stream_launch<1>(a, grid, smem, s, pdl);
        case 2: return stream_launch<2>(a, grid, smem, s, pdl);
        case 3: return stream_launch<3>(a, grid, smem, s, pdl);
        case 4: return stream_launch<4>(a, grid, smem, s, pdl);
        case 5: return stream_launch<5>(a, grid, smem, s, pdl);
        case 6: return stream_launch<6>(a, grid, smem, s, pdl);
        case 7: return stream_launch<7>(a, grid, smem, s, pdl);
        default: return stream_launch<8>(a, grid, smem, s, pdl);
    }
}

size_t dense_tc_scratch(const DenseLin& lin, int64_t m, int sm_count) {
    const int sp = tc_splits(lin, m, sm_count);
    return sp > 1 ? (size_t)sp * (size_t)m * lin.n_pad : 0;
}
int dense_tc_kernels(const DenseLin& lin, int64_t m, int sm_count, int act) { return act < DACT_SWIGLU && tc_splits(lin, m, sm_count) > 1 ? 2 : 1; }

cudaError_t launch_dense_tc(const DenseLin& lin, const uint8_t* x_tiles, int64_t m, const DenseOut& o, float* scratch,
                            unsigned int* err, int sm_count, cudaStream_t s) {
    const int blocks = o.shared_weights ? o.blocks : lin.blocks, n_out = dense_outputs(lin, o.act);
    const bool whole = o.act == DACT_SWIGLU || o.out_rows16 || o.plan || blocks > 1;  // never cut
    const int sp = whole ? 1 : tc_splits(lin, m, sm_count);
    const int nt = o.plan ? o.plan->tile : tc_tokens(lin, m, sm_count, blocks);
    if ((o.act == DACT_SWIGLU && (!o.out_tiles || lin.n % 2 || o.bias)) || o.act == DACT_RGLRU ||
        (sp == 1 && o.out_tiles && (o.bias || (o.act != DACT_NONE && o.act != DACT_RELU2 && o.act != DACT_SWIGLU))) || (o.out_rows16 && (o.bias || o.act != DACT_NONE)) || o.halves < 1 || o.halves > 2 ||
        (o.out_rows16 && (o.ld % 8 || o.out_block % 8 || n_out % 8)) || (o.out_tiles && blocks > 1 && !o.plan && (o.out_block % 8 || n_out % 8)))
        return cudaErrorInvalidValue;
    TcArgs a;
    a.w = lin.tiles; a.x = x_tiles; a.n = lin.n; a.n_pad = lin.n_pad; a.w_chunks = lin.chunks(); a.chunks = o.halves * lin.chunks();
    a.m = m; a.m_pad = o.m_pad ? o.m_pad : dense_mpad(m); a.splits = sp; a.err = err; a.n_out = n_out;
    a.blocks = o.plan ? 1 : blocks; a.w_block = o.shared_weights ? 0 : (int64_t)lin.block_bytes();
    a.x_block = o.shared_weights ? o.x_block : (int64_t)a.chunks * a.m_pad * 128;
    a.out_block = o.out_block; a.bias = o.bias; a.plan = nullptr; a.n_plan = nullptr; a.out_rows16 = nullptr;
    if (sp > 1) {
        a.out = scratch; a.ld = lin.n_pad; a.part_stride = m * (int64_t)lin.n_pad; a.out_tiles = nullptr; a.act = DACT_NONE;
        a.bias = nullptr;
        a.n = lin.n_pad;  // the padded rows are zero weights: the reduction may read whole vectors
    } else {
        a.out = o.out; a.ld = o.ld; a.part_stride = 0; a.out_tiles = o.out_tiles; a.out_rows16 = o.out_rows16; a.act = o.act;
    }
    if (o.plan) {
        a.plan = o.plan->tiles; a.n_plan = o.plan->n_tiles;
        a.m = (int64_t)o.plan->max_tiles * nt;
    }
    cudaError_t e = nt == 64 ? tc_launch<64>(a, sm_count, s) : (nt == 128 ? tc_launch<128>(a, sm_count, s) : tc_launch<256>(a, sm_count, s));
    if (e != cudaSuccess || sp == 1) return e;
    const int cols = o.out_tiles ? dense_kpad(lin.n) : lin.n;
    dense_reduce_kernel<<<dim3((unsigned)((cols + 2047) / 2048), (unsigned)m), 256, 0, s>>>(
        scratch, sp, a.part_stride, a.ld, m, lin.n, cols, o.act, o.out, o.ld, o.out_tiles, a.m_pad, o.bias);
    return cudaGetLastError();
}

cudaError_t launch_dense_f32(const DenseLin& lin, const float* x, int64_t ldx, int64_t x_block, int64_t m, const DenseOut& o, cudaStream_t s) {
    if (o.act == DACT_RGLRU || (o.act == DACT_SWIGLU && lin.n % 2) || !o.out) return cudaErrorInvalidValue;
    F32Args a;
    a.w = lin.tiles; a.n = lin.n; a.n_pad = lin.n_pad; a.k = lin.k; a.k_pad = lin.k_pad; a.w_block = (int64_t)lin.block_bytes();
    a.x = x; a.ldx = ldx; a.x_block = x_block; a.m = m; a.out = o.out; a.ld = o.ld; a.out_block = o.out_block; a.bias = o.bias; a.act = o.act;
    a.row_start = o.plan ? o.plan->row_start : nullptr;
    a.counts = o.plan ? o.plan->counts : nullptr;
    const int64_t rows = o.plan ? o.plan->max_rows : m;
    dense_f32_kernel<<<dim3((unsigned)((lin.n + 63) / 64), (unsigned)((rows + 63) / 64), (unsigned)lin.blocks), 256, 0, s>>>(a);
    return cudaGetLastError();
}

cudaError_t launch_rows_tile(const float* x, int64_t ld, int64_t x_block, int blocks, int k, int halves, int act, int64_t rows,
                             uint8_t* tiles, int64_t m_pad, cudaStream_t s) {
    if (halves < 1 || halves > 2 || act >= DACT_SWIGLU) return cudaErrorInvalidValue;
    const int64_t total = rows * blocks * (dense_kpad(k) / 8);
    rows_tile_kernel<<<(unsigned)((total + 255) / 256 < 4736 ? (total + 255) / 256 : 4736), 256, 0, s>>>(x, ld, x_block, blocks, k, halves, act, rows, tiles, m_pad);
    return cudaGetLastError();
}

cudaError_t launch_embed_pos(const int32_t* tokens, const __nv_bfloat16* table, const __nv_bfloat16* pos_table,
                             const int32_t* pos, int batch, int q_rows, int hidden, int vocab, int max_pos, float* h,
                             const ActOut& act, cudaStream_t s, bool pdl, const ActOut& act2) {
    return launch_pdl(embed_pos_kernel, dim3((unsigned)(batch * q_rows)), dim3(row_threads(hidden)), 0, s, pdl, tokens, table,
                      pos_table, pos, q_rows, hidden, vocab, max_pos, h, act, act2);
}

cudaError_t launch_row_op(const RowArgs& a, cudaStream_t s, bool pdl) {
    const size_t smem = a.op == ROW_GROUPNORM && a.groups > 1 ? (size_t)a.groups * sizeof(float) : 0;
    if (smem > 40 * 1024) return cudaErrorInvalidConfiguration;
    if (a.op == ROW_GROUPNORM && a.groups > 1) {
        const int part = a.k / a.groups;
        if (part % 8 == 0 && part <= 2048) {
            const dim3 grid((unsigned)a.rows);
            if (part <= 256) return launch_pdl(group_norm_kernel<1>, grid, dim3(256), 0, s, pdl, a, part);
            if (part <= 1024) return launch_pdl(group_norm_kernel<4>, grid, dim3(256), 0, s, pdl, a, part);
            return launch_pdl(group_norm_kernel<8>, grid, dim3(256), 0, s, pdl, a, part);
        }
    }
    // many rows: fewer threads with more of the row each, so that more rows share an SM
    unsigned threads = row_threads(a.k);
    if (a.rows > 64) threads = threads > 256 ? (threads / 4 + 31) / 32 * 32 : (threads > 128 ? (threads / 2 + 31) / 32 * 32 : threads);
    const dim3 grid((unsigned)a.rows), block(threads);
    const int nc = (dense_kpad(a.k) / 8 + (int)block.x - 1) / (int)block.x;
    if (nc <= 1) return launch_pdl(row_op_kernel<1>, grid, block, smem, s, pdl, a);
    if (nc <= 2) return launch_pdl(row_op_kernel<2>, grid, block, smem, s, pdl, a);
    if (nc <= 4) return launch_pdl(row_op_kernel<4>, grid, block, smem, s, pdl, a);
    return nc <= 8 ? launch_pdl(row_op_kernel<8>, grid, block, smem, s, pdl, a) : cudaErrorInvalidConfiguration;
}

}  // namespace bt
