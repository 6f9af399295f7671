// Mixture of experts: the choice of experts (softmax over the chosen logits), the streamed experts of a decode step, and for
// many rows the plan of the grouped products and the copies of the rows by expert.  Logits, choice and weights are f32.
#include "bt_dense.cuh"
#include "bt_ptx.cuh"

namespace bt {

namespace {

constexpr int kMaxExperts = 1024, kMaxTop = 64;

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }

// The `top` largest of n logits by one warp, the lower index first among equals: sel / wt in order, weights a softmax over
// the chosen.  z (shared memory) is used up.
__device__ __forceinline__ void choose(float* z, int n, int top, int lane, int* sel, float* wt) {
    float first = 0.0f, sum = 0.0f;
    for (int j = 0; j < top; ++j) {
        float v = -INFINITY;
        int at = n;
        for (int e = lane; e < n; e += 32)
            if (z[e] > v) { v = z[e]; at = e; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, v, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (ov > v || (ov == v && oa < at)) { v = ov; at = oa; }
        }
        if (at >= n) at = 0;  // only if a logit is not a number
        if (j == 0) first = v;
        const float e = expf(v - first);
        sum += e;
        if (lane == 0) {
            sel[j] = at;
            wt[j] = e;
            z[at] = -INFINITY;
        }
        __syncwarp();
    }
    for (int j = lane; j < top; j += 32) wt[j] /= sum;
    __syncwarp();
}

// ---------------------------------------------------------------------------------------
// up to 8 rows: the chosen experts' matrices streamed as in the dense streaming product
// ---------------------------------------------------------------------------------------
// Units of work: UP: (row, choice, group of 8 matrix rows); DOWN: (row, group of 8 matrix rows) over the inputs of all chosen
// experts and of the shared one.  `wk` warps share a unit and take its blocks of 64 inputs in turn.
constexpr int kStepThreads = 512, kStepWarps = 16, kBatch = 4, kMaxRows = 8;

struct MoeStream {
    const uint8_t* w;        // experts
    const uint8_t* ws;       // DOWN: shared expert, or null
    int64_t block_bytes;
    int n_pad, ns_pad;
    int n, k, k_pad, chunks; // of one expert; chunks: of a unit
    int ks, ks_pad;          // DOWN: the shared expert's inputs
    int wk;
    const float* logits;
    int experts, top, rows;
    const float* x;
    int64_t x_ld;
    float* out;
    int64_t out_ld;
};

template <bool DOWN>
__global__ void __launch_bounds__(kStepThreads, 1) moe_stream_kernel(const __grid_constant__ MoeStream a) {
    extern __shared__ __align__(16) float xs[];
    __shared__ int sel[kMaxRows * kMaxTop];
    __shared__ float wt[kMaxRows * kMaxTop];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int slots = kStepWarps / a.wk, slot = warp / a.wk, kw = warp - slot * a.wk;
    const int xrow = DOWN ? a.top * a.k_pad + a.ks_pad : a.k_pad;  // inputs of a row
    float* part = xs + (size_t)a.rows * xrow;                      // [2][16 warps][8]
    const int groups = (a.n + 7) >> 3;
    const int units = groups * a.rows * (DOWN ? 1 : a.top);
    const int cpe = a.k_pad / kDenseK;
    ptx::pdl_wait();
    ptx::pdl_launch_dependents();
    // the choice; the logits wait where the inputs come next
    for (int i = threadIdx.x; i < a.rows * a.experts; i += kStepThreads) xs[i] = a.logits[i];
    __syncthreads();
    if (warp < a.rows) choose(xs + warp * a.experts, a.experts, a.top, lane, sel + warp * a.top, wt + warp * a.top);
    __syncthreads();
    for (int b = 0; b < a.rows; ++b) {
        const float* x = a.x + b * a.x_ld;
        for (int c = threadIdx.x; c < xrow; c += kStepThreads) {
            float v;
            if (!DOWN) {
                v = c < a.k ? x[c] : 0.0f;
            } else if (c < a.top * a.k_pad) {
                const int j = c / a.k_pad;
                v = c - j * a.k_pad < a.k ? x[c] * wt[b * a.top + j] : 0.0f;
            } else {
                v = c - a.top * a.k_pad < a.ks ? x[c] : 0.0f;
            }
            xs[(size_t)b * xrow + c] = v;
        }
    }
    __syncthreads();

    uint4 buf[2][2 * kBatch];
    auto fetch = [&](uint4 (&d)[2 * kBatch], int u, int i) {
        const bool live = u < units;
        const int q = live ? u / groups : 0, g = u - q * groups;  // UP: q = row * top + choice; DOWN: row
        const uint8_t* p = a.w + (int64_t)g * 1024 + lane * 16;
        if (!DOWN) p += sel[q] * a.block_bytes;
#pragma unroll
        for (int j = 0; j < kBatch; ++j) {
            const int kc = kw + (i * kBatch + j) * a.wk;
            if (live && kc < a.chunks) {
                const uint8_t* s;
                if (!DOWN) {
                    s = p + (int64_t)kc * a.n_pad * 128;
                } else {
                    const int e = kc / cpe;
                    s = e < a.top ? p + sel[q * a.top + e] * a.block_bytes + (int64_t)(kc - e * cpe) * a.n_pad * 128
                                  : a.ws + (int64_t)g * 1024 + lane * 16 + (int64_t)(kc - a.top * cpe) * a.ns_pad * 128;
                }
                d[2 * j] = __ldg(reinterpret_cast<const uint4*>(s));
                d[2 * j + 1] = __ldg(reinterpret_cast<const uint4*>(s + 512));
            } else {
                d[2 * j] = d[2 * j + 1] = make_uint4(0, 0, 0, 0);
            }
        }
    };
    float acc = 0.0f;
    auto multiply = [&](const uint4 (&d)[2 * kBatch], int u, int i) {
        const int row = u < units ? (DOWN ? u / groups : u / groups / a.top) : 0;
        const float* xl = xs + (size_t)row * xrow + (lane >> 3) * 8;
#pragma unroll
        for (int j = 0; j < kBatch; ++j) {
            const int kc = kw + (i * kBatch + j) * a.wk;
            if (kc < a.chunks) {
#pragma unroll
                for (int hlf = 0; hlf < 2; ++hlf) {
                    const uint4 w = d[2 * j + hlf];
                    const float* x = xl + kc * kDenseK + hlf * 32;
                    const float4 x0 = *reinterpret_cast<const float4*>(x), x1 = *reinterpret_cast<const float4*>(x + 4);
                    acc = fmaf(__uint_as_float(w.x << 16), x0.x, acc); acc = fmaf(__uint_as_float(w.x & 0xffff0000u), x0.y, acc);
                    acc = fmaf(__uint_as_float(w.y << 16), x0.z, acc); acc = fmaf(__uint_as_float(w.y & 0xffff0000u), x0.w, acc);
                    acc = fmaf(__uint_as_float(w.z << 16), x1.x, acc); acc = fmaf(__uint_as_float(w.z & 0xffff0000u), x1.y, acc);
                    acc = fmaf(__uint_as_float(w.w << 16), x1.z, acc); acc = fmaf(__uint_as_float(w.w & 0xffff0000u), x1.w, acc);
                }
            }
        }
    };
    const int per = (a.chunks + a.wk * kBatch - 1) / (a.wk * kBatch);
    const int step = gridDim.x * slots;
    int u = blockIdx.x * slots + slot, pb = 0;
    fetch(buf[0], u, 0);
    for (int base = blockIdx.x * slots; base < units; base += step, u += step, pb ^= 1) {
        for (int i = 0; i < per; i += 2) {
            if (i + 1 < per) fetch(buf[1], u, i + 1);
            multiply(buf[0], u, i);
            if (i + 1 < per) {
                if (i + 2 < per) fetch(buf[0], u, i + 2); else fetch(buf[0], u + step, 0);
                multiply(buf[1], u, i + 1);
            } else {
                fetch(buf[0], u + step, 0);
            }
        }
        float* pw = part + pb * kStepWarps * 8;
        acc += __shfl_xor_sync(0xffffffffu, acc, 8);
        acc += __shfl_xor_sync(0xffffffffu, acc, 16);
        if (lane < 8) pw[warp * 8 + lane] = acc;
        acc = 0.0f;
        __syncthreads();
        for (int o = threadIdx.x; o < slots * 8; o += kStepThreads) {
            const int un = base + (o >> 3), row = o & 7;
            if (un >= units) continue;
            const int q = un / groups, n = (un - q * groups) * 8 + row;
            if (n >= a.n) continue;
            const float* p = pw + (o >> 3) * a.wk * 8 + row;
            float v = 0.0f;
            for (int w = 0; w < a.wk; ++w) v += p[w * 8];
            if (DOWN) {
                a.out[q * a.out_ld + n] = v;
            } else if ((row & 1) == 0) {
                float v2 = 0.0f;
                for (int w = 0; w < a.wk; ++w) v2 += p[w * 8 + 1];
                a.out[(q / a.top) * a.out_ld + (q % a.top) * dense_kpad(a.n / 2) + (n >> 1)] = silu_f(v) * v2;
            }
        }
    }
}

size_t step_smem(int rows, int xrow, int experts) {
    const size_t x = (size_t)rows * xrow, z = (size_t)rows * experts;
    return ((x > z ? x : z) + 2 * kStepWarps * 8) * sizeof(float);
}
template <bool DOWN>
cudaError_t stream_launch(const MoeStream& a, int sm_count, cudaStream_t s, bool pdl) {
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(moe_stream_kernel<DOWN>, cudaFuncAttributeMaxDynamicSharedMemorySize, 216 * 1024); });
    if (e != cudaSuccess) return e;
    const int slots = kStepWarps / a.wk, units = (a.n + 7) / 8 * a.rows * (DOWN ? 1 : a.top), ctas = (units + slots - 1) / slots;
    return launch_pdl(moe_stream_kernel<DOWN>, dim3((unsigned)(ctas < sm_count ? ctas : sm_count)), dim3(kStepThreads),
                      step_smem(a.rows, DOWN ? a.top * a.k_pad + a.ks_pad : a.k_pad, a.experts), s, pdl, a);
}
int step_warps(int chunks) {
    int wk = kStepWarps;
    while (wk > chunks) wk >>= 1;
    return wk;
}

// ---------------------------------------------------------------------------------------
// many rows
// ---------------------------------------------------------------------------------------
// choice per row (a warp each), the row's place among its expert's rows
__global__ void __launch_bounds__(256) moe_choose_kernel(const MoeRoute a) {
    extern __shared__ float zs[];  // [8][experts], then choices and weights
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t r = (int64_t)blockIdx.x * 8 + warp;
    if (r >= a.rows) return;
    float* z = zs + warp * a.experts;
    int* sel = reinterpret_cast<int*>(zs + 8 * a.experts) + warp * a.top;
    float* wt = zs + 8 * a.experts + 8 * a.top + warp * a.top;
    for (int e = lane; e < a.experts; e += 32) z[e] = a.logits[r * a.ld + e];
    __syncwarp();
    choose(z, a.experts, a.top, lane, sel, wt);
    for (int j = lane; j < a.top; j += 32) {
        a.sel[r * a.top + j] = sel[j];
        a.wt[r * a.top + j] = wt[j];
        a.rank[r * a.top + j] = atomicAdd(a.counts + sel[j], 1);
    }
}

// one CTA: the experts' rows behind one another, each at a multiple of 8, in tiles of about equal size, at
// most `tile` rows; the counts start over
__global__ void __launch_bounds__(kMaxExperts) moe_plan_kernel(const MoeRoute a) {
    __shared__ int rows_s[32], tiles_s[32];
    const int e = threadIdx.x, lane = e & 31, warp = e >> 5;
    const int n = e < a.experts ? a.counts[e] : 0;
    const int padded = (n + 7) / 8 * 8, nt = (n + a.tile - 1) / a.tile;
    int rs = padded, ts = nt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const int r0 = __shfl_up_sync(0xffffffffu, rs, o), t0 = __shfl_up_sync(0xffffffffu, ts, o);
        if (lane >= o) { rs += r0; ts += t0; }
    }
    if (lane == 31) { rows_s[warp] = rs; tiles_s[warp] = ts; }
    __syncthreads();
    if (warp == 0) {
        int r = rows_s[lane], t = tiles_s[lane];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int r0 = __shfl_up_sync(0xffffffffu, r, o), t0 = __shfl_up_sync(0xffffffffu, t, o);
            if (lane >= o) { r += r0; t += t0; }
        }
        rows_s[lane] = r;
        tiles_s[lane] = t;
    }
    __syncthreads();
    const int r0 = (warp ? rows_s[warp - 1] : 0) + rs - padded, t0 = (warp ? tiles_s[warp - 1] : 0) + ts - nt;
    if (e < a.experts) {
        a.row_start[e] = r0;
        a.counts_done[e] = n;
        a.counts[e] = 0;
        const int each = nt ? ((n + nt - 1) / nt + 15) / 16 * 16 : 0;
        for (int i = 0; i < nt && t0 + i < a.max_tiles; ++i) {
            ExpertTile t;
            t.expert = e; t.row0 = r0 + i * each; t.row_end = r0 + min(n, (i + 1) * each); t.pad = 0;
            a.tiles[t0 + i] = t;
        }
    }
    if (e == 0) {
        a.row_start[a.experts] = rows_s[31];
        *a.n_tiles = min(tiles_s[31], a.max_tiles);
    }
}

// a CTA per row: its place in every chosen expert's rows, its inputs copied there
__global__ void __launch_bounds__(256) moe_group_kernel(const MoeRoute a) {
    __shared__ int dst[kMaxTop];
    const int64_t r = blockIdx.x;
    if ((int)threadIdx.x < a.top) {
        const int d = a.row_start[a.sel[r * a.top + threadIdx.x]] + a.rank[r * a.top + threadIdx.x];
        dst[threadIdx.x] = d;
        a.dst[r * a.top + threadIdx.x] = d;
    }
    __syncthreads();
    if (a.xe_tiles) {
        for (int c = threadIdx.x * 8; c < dense_kpad(a.k); c += 256 * 8) {
            const uint4 v = *reinterpret_cast<const uint4*>(a.x_tiles + dense_off(r, c, a.m_pad));
            for (int j = 0; j < a.top; ++j) *reinterpret_cast<uint4*>(a.xe_tiles + dense_off(dst[j], c, a.me_pad)) = v;
        }
    } else {
        for (int c = threadIdx.x; c < a.k; c += 256) {
            const float v = a.x[r * a.k + c];
            for (int j = 0; j < a.top; ++j) a.xe[(int64_t)dst[j] * a.k + c] = v;
        }
    }
}

}  // namespace

int moe_max_experts() { return kMaxExperts; }

bool moe_step_fits(const MoeStep& a) {
    const int ks_pad = a.shared_down ? a.shared_down->k_pad : 0;
    return a.rows <= kMaxRows && a.top <= kMaxTop && step_smem(a.rows, a.up->k_pad, a.experts) <= 216 * 1024 &&
           step_smem(a.rows, a.top * a.down->k_pad + ks_pad, a.experts) <= 216 * 1024;
}

cudaError_t launch_moe_up(const MoeStep& a, cudaStream_t s, bool pdl) {
    if (!moe_step_fits(a) || a.up->n % 2) return cudaErrorInvalidValue;
    MoeStream m = {};
    m.w = a.up->tiles; m.block_bytes = (int64_t)a.up->block_bytes(); m.n_pad = a.up->n_pad; m.n = a.up->n; m.k = a.up->k; m.k_pad = a.up->k_pad;
    m.chunks = a.up->chunks(); m.wk = step_warps(m.chunks);
    m.logits = a.logits; m.experts = a.experts; m.top = a.top; m.rows = a.rows; m.x = a.x; m.x_ld = a.up->k; m.out = a.ff; m.out_ld = a.ff_ld;
    return stream_launch<false>(m, a.sm_count, s, pdl);
}

cudaError_t launch_moe_down(const MoeStep& a, cudaStream_t s, bool pdl) {
    if (!moe_step_fits(a) || (a.shared_down && a.shared_down->n != a.down->n)) return cudaErrorInvalidValue;
    MoeStream m = {};
    m.w = a.down->tiles; m.block_bytes = (int64_t)a.down->block_bytes(); m.n_pad = a.down->n_pad; m.n = a.down->n; m.k = a.down->k; m.k_pad = a.down->k_pad;
    m.chunks = a.top * a.down->chunks();
    if (a.shared_down) {
        m.ws = a.shared_down->tiles; m.ns_pad = a.shared_down->n_pad; m.ks = a.shared_down->k; m.ks_pad = a.shared_down->k_pad;
        m.chunks += a.shared_down->chunks();
    }
    m.wk = step_warps(m.chunks);
    m.logits = a.logits; m.experts = a.experts; m.top = a.top; m.rows = a.rows; m.x = a.ff; m.x_ld = a.ff_ld; m.out = a.y; m.out_ld = a.down->n;
    return stream_launch<true>(m, a.sm_count, s, pdl);
}

// most rows per tile of the grouped products
int moe_tile_rows(int64_t rows, int top, int experts) {
    const int64_t each = rows * top / experts;
    return each <= 48 ? 64 : (each <= 112 ? 128 : 256);
}
int moe_max_tiles(int64_t rows, int top, int experts, int tile) {
    const int64_t all = rows * top, busy = all < experts ? all : experts;
    return (int)(all / tile + busy);
}
int64_t moe_grouped_rows(int64_t rows, int top, int experts) { return (rows * top + 7ll * experts + 7) / 8 * 8 + 256; }

cudaError_t launch_moe_route(const MoeRoute& a, cudaStream_t s) {
    if (a.experts > kMaxExperts || a.top > kMaxTop || a.top > a.experts) return cudaErrorInvalidValue;
    const size_t smem = (size_t)8 * (a.experts + 2 * a.top) * sizeof(float);
    moe_choose_kernel<<<(unsigned)((a.rows + 7) / 8), 256, smem, s>>>(a);
    moe_plan_kernel<<<1, kMaxExperts, 0, s>>>(a);
    moe_group_kernel<<<(unsigned)a.rows, 256, 0, s>>>(a);
    return cudaGetLastError();
}

}  // namespace bt
