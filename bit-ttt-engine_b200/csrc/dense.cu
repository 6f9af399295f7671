// Dense bf16 projections: streaming product for up to 8 rows (f32 activations), tcgen05 product for more (bf16
// activations), f32 product for 32-bit models; and the row kernels around them (embedding with learned positions,
// output norm + residual, norm in equal parts).
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
    return v;
}

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    __nv_bfloat162 p = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&p);
}

// ---------------------------------------------------------------------------------------
// weights: f32 rows -> tiled bf16
// ---------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) dense_tile_kernel(const float* __restrict__ src, int rows, int k, int row0,
                                                         uint8_t* __restrict__ tiles, int n_pad, int k_pad) {
    const int64_t total = (int64_t)rows * (k_pad / 8);
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int r = (int)(i / (k_pad / 8)), c0 = (int)(i % (k_pad / 8)) * 8;
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = c0 + j < k ? src[(int64_t)r * k + c0 + j] : 0.0f;
        uint4 u = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
        *reinterpret_cast<uint4*>(tiles + dense_off(row0 + r, c0, n_pad)) = u;
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

struct StreamArgs {
    const uint8_t* w;
    int n, n_pad, k, k_pad;
    int wk;  // warps per row group: 1, 2, 4, 8, 16
    DenseIn in;
    float* out;
    int64_t ld;
    int act;
};

template <int B>
__device__ __forceinline__ void stream_input(const StreamArgs& a, float* xs, float* red) {
    const int k = a.k, kp = a.k_pad;
    const DenseIn& in = a.in;
    if (in.kind == DPRO_ROWS) {
#pragma unroll
        for (int b = 0; b < B; ++b)
            for (int c = threadIdx.x; c < kp; c += kStreamThreads) xs[b * kp + c] = c < k ? in.x[b * in.ld + c] : 0.0f;
    } else if (in.kind == DPRO_RESNORM) {
        for (int b = 0; b < B; ++b) {
            float ss = 0.0f;
            for (int c = threadIdx.x; c < kp; c += kStreamThreads) {
                const float y = c < k ? in.x[b * in.ld + c] : 0.0f;
                xs[b * kp + c] = y;
                ss = fmaf(y, y, ss);
            }
            ss = block_sum(ss, red);
            const float inv = 1.0f / sqrtf(ss / (float)k + in.eps);
            for (int c = threadIdx.x; c < k; c += kStreamThreads) {
                const float v = fmaf(xs[b * kp + c] * inv, in.w[c], in.h[(int64_t)b * k + c]);
                xs[b * kp + c] = v;
                if (blockIdx.x == 0) in.h_out[(int64_t)b * k + c] = v;
            }
        }
    } else {
        const int part = k / in.groups;
        for (int b = 0; b < B; ++b) {
            if (in.groups == 1) {
                float ss = 0.0f;
                for (int c = threadIdx.x; c < kp; c += kStreamThreads) {
                    const float y = c < k ? in.x[b * in.ld + c] : 0.0f;
                    xs[b * kp + c] = y;
                    ss = fmaf(y, y, ss);
                }
                ss = block_sum(ss, red);
                const float inv = 1.0f / sqrtf(ss / (float)k + in.eps);
                for (int c = threadIdx.x; c < k; c += kStreamThreads) xs[b * kp + c] = xs[b * kp + c] * inv * in.w[c];
            } else {
                // a warp per part
                for (int c = k + threadIdx.x; c < kp; c += kStreamThreads) xs[b * kp + c] = 0.0f;
                for (int g = threadIdx.x >> 5; g < in.groups; g += kStreamWarps) {
                    const float* x = in.x + b * in.ld + (int64_t)g * part;
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
    __syncthreads();
}

template <int B>
__global__ void __launch_bounds__(kStreamThreads, 1) dense_stream_kernel(const StreamArgs a) {
    extern __shared__ __align__(16) float xs[];  // [B][k_pad], then 2 x [16 warps][8 rows][B]
    __shared__ float red[33];
    float* part = xs + (size_t)B * a.k_pad;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int wk = a.wk, slots = kStreamWarps / wk;
    const int slot = warp / wk, kw = warp - slot * wk;
    const int groups = (a.n + 7) >> 3, chunks = a.k_pad / kDenseK;
    const int step = gridDim.x * slots;
    const int64_t block_stride = (int64_t)a.n_pad * 128;
    const uint8_t* lane_base = a.w + lane * 16;

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
    int rg = blockIdx.x * slots + slot;
    fetch(buf[0], rg, 0);
    ptx::pdl_wait();
    ptx::pdl_launch_dependents();
    stream_input<B>(a, xs, red);

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
    for (int base = blockIdx.x * slots; base < groups; base += base_step, rg += base_step, pb ^= 1) {
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
            if (n < a.n) a.out[b * a.ld + n] = act_fn(a.act, v);
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
    int n, n_pad, chunks;
    int64_t m, m_pad;
    int splits;
    float* out;
    int64_t ld, part_stride;
    uint8_t* out_tiles;
    int out_kpad, act;
    unsigned int* err;
};

template <int NT>
struct TcCfg {
    static constexpr int kStageBytes = (kTcRows + NT) * 128;
    static constexpr int kStages = NT >= 256 ? 4 : (NT >= 128 ? 6 : 8);
    static constexpr int kEpi = 4 * 32 * (8 * 16 + 16);  // per epilogue warp: 32 tokens x 32 features of bf16, padded
    static constexpr size_t kSmem = (size_t)kStages * kStageBytes + kEpi + 256;
};

template <int NT>
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
    const int tok_blocks = (int)((a.m + NT - 1) / NT);
    const int tiles = row_sets * tok_blocks * a.splits;

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
    // tile -> (split, token block, row set): neighbouring CTAs share the activations of a token block
    auto decode = [&](int t, int& rs, int& tb, int& c0, int& c1, int& sp) {
        sp = t / (row_sets * tok_blocks);
        const int u = t - sp * row_sets * tok_blocks;
        tb = u / row_sets;
        rs = u - tb * row_sets;
        c0 = (int)((int64_t)a.chunks * sp / a.splits);
        c1 = (int)((int64_t)a.chunks * (sp + 1) / a.splits);
    };

    if (warp == 0) {
        if (lane == 0) {
            int slot = 0, issued = 0; uint32_t par = 1; bool first = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
                int rs, tb, c0, c1, sp;
                decode(t, rs, tb, c0, c1, sp);
                const uint8_t* wp = a.w + (int64_t)rs * kTcRows * 128;
                const uint8_t* xp = a.x + (int64_t)tb * NT * 128;
                for (int kc = c0; kc < c1; ++kc) {
                    if (!first) { if (!ptx::mbar_wait_bounded(&empty[slot], par)) { ok = false; break; } }
                    uint8_t* st = smem + (size_t)slot * Cfg::kStageBytes;
                    ptx::mbar_arrive_expect_tx(&full[slot], Cfg::kStageBytes);
                    ptx::bulk_g2s(st, wp + (int64_t)kc * a.n_pad * 128, kTcRows * 128, &full[slot]);
                    ptx::bulk_g2s(st + kTcRows * 128, xp + (int64_t)kc * a.m_pad * 128, NT * 128, &full[slot]);
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
            const uint32_t idesc = tc_idesc(NT);
            int slot = 0, set = 0; uint32_t par = 0, acc_par = 1; int done = 0;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, ++done) {
                int rs, tb, c0, c1, sp;
                decode(t, rs, tb, c0, c1, sp);
                if (done >= 2) ok &= ptx::mbar_spin_relaxed(&acc_empty[set], acc_par);
                ptx::tc_fence_after();
                for (int kc = c0; kc < c1 && ok; ++kc) {
                    ok &= ptx::mbar_spin_relaxed(&full[slot], par);
                    ptx::tc_fence_after();
                    const uint32_t a_addr = ptx::smem_u32(smem + (size_t)slot * Cfg::kStageBytes);
                    const uint32_t b_addr = a_addr + kTcRows * 128;
#pragma unroll
                    for (int ks = 0; ks < kDenseK / 16; ++ks)
                        ptx::umma_f16(tmem_base + set * NT, ptx::smem_desc(a_addr + ks * 256, 128, 1024),
                                      ptx::smem_desc(b_addr + ks * 256, 128, 1024), idesc, (kc > c0 || ks > 0) ? 1u : 0u);
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
            int rs, tb, c0, c1, sp;
            decode(t, rs, tb, c0, c1, sp);
            ok &= ptx::mbar_wait_bounded(&acc_full[set], acc_par);
            ptx::tc_fence_after();
            const int f = rs * kTcRows + sub * 32 + lane;
            const int64_t tok0 = (int64_t)tb * NT;
#pragma unroll 1
            for (int q = 0; q < NT; q += 32) {
                if (tok0 + q >= a.m) break;
                uint32_t v[32];
                ptx::tmem_ld32(tmem_base + ((uint32_t)(sub * 32) << 16) + set * NT + q, v);
                ptx::tmem_ld_wait();
                if (a.out_tiles) {
                    // through shared memory into 16-byte pieces (one token, 8 features): [token group][8 features][token]
#pragma unroll
                    for (int j = 0; j < 32; ++j) {
                        const float r = act_fn(a.act, __uint_as_float(v[j]));
                        *reinterpret_cast<__nv_bfloat16*>(stage + ((j >> 3) * 4 + (lane >> 3)) * 144 + (j & 7) * 16 + (lane & 7) * 2) = __float2bfloat16_rn(r);
                    }
                    __syncwarp();
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int piece = i * 32 + lane, core = piece >> 3, tk = piece & 7;  // core = token group * 4 + feature group
                        const int64_t token = tok0 + q + (core >> 2) * 8 + tk;
                        const int feat = rs * kTcRows + sub * 32 + (core & 3) * 8;
                        if (token < a.m && feat < a.out_kpad)
                            *reinterpret_cast<uint4*>(a.out_tiles + dense_off(token, feat, a.m_pad)) =
                                *reinterpret_cast<const uint4*>(stage + core * 144 + tk * 16);
                    }
                    __syncwarp();
                } else if (f < a.n) {
                    float* o = a.out + (int64_t)sp * a.part_stride + (tok0 + q) * a.ld + f;
                    if (tok0 + q + 32 <= a.m) {
#pragma unroll
                        for (int j = 0; j < 32; ++j) o[j * a.ld] = act_fn(a.act, __uint_as_float(v[j]));
                    } else {
#pragma unroll
                        for (int j = 0; j < 32; ++j)
                            if (tok0 + q + j < a.m) o[j * a.ld] = act_fn(a.act, __uint_as_float(v[j]));
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
                                                           int64_t ld, uint8_t* __restrict__ tiles, int64_t m_pad) {
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
    for (int j = 0; j < 8; ++j) v[j] = c0 + j < n ? act_fn(act, v[j]) : 0.0f;
    if (tiles)
        *reinterpret_cast<uint4*>(tiles + dense_off(r, c0, m_pad)) =
            make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
    else
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (c0 + j < n) out[r * ld + c0 + j] = v[j];
}

template <int NT>
cudaError_t tc_launch(const TcArgs& a, int sm_count, cudaStream_t s) {
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(dense_tc_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TcCfg<NT>::kSmem); });
    if (e != cudaSuccess) return e;
    const int64_t tiles = (int64_t)(a.n_pad / kTcRows) * ((a.m + NT - 1) / NT) * a.splits;
    dense_tc_kernel<NT><<<(unsigned)(tiles < sm_count ? tiles : sm_count), kTcThreads, TcCfg<NT>::kSmem, s>>>(a);
    return cudaGetLastError();
}

// token rows per tile: 64 and 128 while one block covers them; above, 256 unless that leaves SMs idle
int tc_tokens(const DenseLin& lin, int64_t m, int sm_count) {
    if (m <= 64) return 64;
    if (m <= 128) return 128;
    const int64_t rs = lin.n_pad / kTcRows;
    const int64_t w256 = (rs * ((m + 255) / 256) + sm_count - 1) / sm_count * 2, w128 = (rs * ((m + 127) / 128) + sm_count - 1) / sm_count;
    return 4 * w128 < 3 * w256 ? 128 : 256;  // the smaller tile reads its operands twice as often
}
int tc_splits(const DenseLin& lin, int64_t m, int sm_count) {
    if (m > 128) return 1;
    const int tiles = lin.n_pad / kTcRows, chunks = lin.k_pad / kDenseK;
    int s = sm_count / tiles;
    if (s > chunks / 4) s = chunks / 4;
    return s < 1 ? 1 : (s > 8 ? 8 : s);
}

// ---------------------------------------------------------------------------------------
// f32 product for 32-bit models: 64 x 64 outputs per CTA, 4 x 4 per thread
// ---------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) dense_f32_kernel(const uint8_t* __restrict__ w, int n, int n_pad, int k, int k_pad,
                                                        const float* __restrict__ x, int64_t ldx, int64_t m,
                                                        float* __restrict__ out, int64_t ld, int act) {
    __shared__ float ws[32][68], xs[32][68];
    const int n0 = blockIdx.x * 64;
    const int64_t m0 = (int64_t)blockIdx.y * 64;
    const int tn = threadIdx.x & 15, tm = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < k_pad; k0 += 32) {
        __syncthreads();
        {   // weights: 64 rows x 32 inputs, one 16-byte piece per thread
            const int row = threadIdx.x & 63, c = (threadIdx.x >> 6) * 8;
            const uint4 u = *reinterpret_cast<const uint4*>(w + dense_off(n0 + row, k0 + c, n_pad));
            const uint32_t q[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                ws[c + 2 * j][row] = __uint_as_float(q[j] << 16);
                ws[c + 2 * j + 1][row] = __uint_as_float(q[j] & 0xffff0000u);
            }
        }
        for (int i = threadIdx.x; i < 64 * 32; i += 256) {
            const int row = i >> 5, c = i & 31;
            xs[c][row] = (m0 + row < m && k0 + c < k) ? x[(m0 + row) * ldx + k0 + c] : 0.0f;
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
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int64_t r = m0 + tm * 4 + i;
            const int c = n0 + tn * 4 + j;
            if (r < m && c < n) out[r * ld + c] = act_fn(act, acc[i][j]);
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
                                                        const ActOut act) {
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
        get8(y, c0, k, vec, v[i]);
        if (a.op == ROW_RESNORM) get8(a.h_in + row * k, c0, k, (k & 3) == 0, h[i]);
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
            if (parts) v[i][j] = c0 + j < k ? v[i][j] * inv_g[(c0 + j) / (k / a.groups)] * w[i][j] : 0.0f;
            else v[i][j] = a.op == ROW_RESNORM ? fmaf(v[i][j] * inv, w[i][j], h[i][j]) : v[i][j] * inv * w[i][j];
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
        put8(a.act, row, c0, k, v[i]);
    }
}

unsigned row_threads(int k) {
    const int t = (dense_kpad(k) / 8 + 31) / 32 * 32;
    return (unsigned)(t < 64 ? 64 : (t > 512 ? 512 : t));
}

}  // namespace

cudaError_t launch_dense_tile(const float* src, int rows, int k, int row0, const DenseLin& lin, cudaStream_t s) {
    if (k != lin.k || row0 < 0 || row0 + rows > lin.n) return cudaErrorInvalidValue;
    dense_tile_kernel<<<1184, 256, 0, s>>>(src, rows, k, row0, lin.tiles, lin.n_pad, lin.k_pad);
    return cudaGetLastError();
}

bool dense_stream_fits(const DenseLin& lin, int rows) { return rows >= 1 && rows <= 8 && stream_smem(lin, rows) <= 220 * 1024; }

cudaError_t launch_dense_stream(const DenseLin& lin, const DenseIn& in, int rows, float* out, int64_t ld, int act,
                                int sm_count, cudaStream_t s, bool pdl) {
    if (!dense_stream_fits(lin, rows)) return cudaErrorInvalidValue;
    StreamArgs a;
    a.w = lin.tiles; a.n = lin.n; a.n_pad = lin.n_pad; a.k = lin.k; a.k_pad = lin.k_pad;
    a.in = in; a.out = out; a.ld = ld; a.act = act;
    const int chunks = lin.k_pad / kDenseK, groups = (lin.n + 7) / 8;
    // as many warps per row group as there are input blocks: the finest spread of row groups over the SMs
    int wk = kStreamWarps;
    while (wk > chunks) wk >>= 1;
    a.wk = wk;
    const int slots = kStreamWarps / wk;
    const int blocks = (groups + slots - 1) / slots;
    const int grid = blocks < sm_count ? blocks : sm_count;
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
int dense_tc_kernels(const DenseLin& lin, int64_t m, int sm_count) { return tc_splits(lin, m, sm_count) > 1 ? 2 : 1; }

cudaError_t launch_dense_tc(const DenseLin& lin, const uint8_t* x_tiles, int64_t m, float* out, int64_t ld,
                            uint8_t* out_tiles, int act, float* scratch, unsigned int* err, int sm_count, cudaStream_t s) {
    const int nt = tc_tokens(lin, m, sm_count), sp = tc_splits(lin, m, sm_count);
    const int out_kpad = dense_kpad(lin.n);
    TcArgs a;
    a.w = lin.tiles; a.x = x_tiles; a.n = lin.n; a.n_pad = lin.n_pad; a.chunks = lin.k_pad / kDenseK;
    a.m = m; a.m_pad = dense_mpad(m); a.splits = sp; a.err = err; a.out_kpad = out_kpad;
    if (sp > 1) {
        a.out = scratch; a.ld = lin.n_pad; a.part_stride = m * (int64_t)lin.n_pad; a.out_tiles = nullptr; a.act = DACT_NONE;
        a.n = lin.n_pad;  // the padded rows are zero weights: the reduction may read whole vectors
    } else {
        a.out = out; a.ld = ld; a.part_stride = 0; a.out_tiles = out_tiles; a.act = act;
    }
    cudaError_t e = nt == 64 ? tc_launch<64>(a, sm_count, s) : (nt == 128 ? tc_launch<128>(a, sm_count, s) : tc_launch<256>(a, sm_count, s));
    if (e != cudaSuccess || sp == 1) return e;
    const int n_out = out_tiles ? out_kpad : lin.n;
    dense_reduce_kernel<<<dim3((unsigned)((n_out + 2047) / 2048), (unsigned)m), 256, 0, s>>>(
        scratch, sp, a.part_stride, a.ld, m, lin.n, n_out, act, out, ld, out_tiles, a.m_pad);
    return cudaGetLastError();
}

cudaError_t launch_dense_f32(const DenseLin& lin, const float* x, int64_t ldx, int64_t m, float* out, int64_t ld, int act,
                             cudaStream_t s) {
    dense_f32_kernel<<<dim3((unsigned)((lin.n + 63) / 64), (unsigned)((m + 63) / 64)), 256, 0, s>>>(
        lin.tiles, lin.n, lin.n_pad, lin.k, lin.k_pad, x, ldx, m, out, ld, act);
    return cudaGetLastError();
}

cudaError_t launch_embed_pos(const int32_t* tokens, const __nv_bfloat16* table, const __nv_bfloat16* pos_table,
                             const int32_t* pos, int batch, int q_rows, int hidden, int vocab, int max_pos, float* h,
                             const ActOut& act, cudaStream_t s, bool pdl) {
    return launch_pdl(embed_pos_kernel, dim3((unsigned)(batch * q_rows)), dim3(row_threads(hidden)), 0, s, pdl, tokens, table,
                      pos_table, pos, q_rows, hidden, vocab, max_pos, h, act);
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
