// Recurrence with a decay per key channel and a bonus for the current token (the RWKV-6 form), per head:
//   o = (S + diag(u) k v^T)^T r,   S <- diag(exp(-exp(z))) S + k v^T.
// State, decays, exponents and every sum of the recurrence are f32.
#include "bt_dense.cuh"
#include "bt_ptx.cuh"

namespace bt {

namespace {

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// ---------------------------------------------------------------------------------------
// token shift of the new rows: one CTA per row
// ---------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) wkv_mix_kernel(const WkvMix a) {
    const int64_t r = blockIdx.x;
    const int b = (int)(r / a.q_rows), i = (int)(r % a.q_rows), W = a.width;
    const int p0 = a.pos[b];
    const float* h = a.hn + r * W;
    const float* before = i > 0 ? h - W : (p0 > 0 ? a.shift + (int64_t)((p0 + 1) & 1) * a.shift_slot + (int64_t)b * W : nullptr);
    for (int c = threadIdx.x; c < W; c += 256) {
        const float v = h[c], d = (before ? before[c] : 0.0f) - v;
#pragma unroll
        for (int s = 0; s < 5; ++s) a.rows5[(r * 5 + s) * W + c] = fmaf(d, a.mu[s][c], v);
    }
}
// the same into tiles: a CTA per 8 rows, eight lanes per piece of 8 columns, so that a piece of the rows is one run of 128 bytes
__global__ void __launch_bounds__(256) wkv_mix_tiles_kernel(const WkvMix a) {
    const int64_t r = (int64_t)blockIdx.x * 8 + (threadIdx.x & 7);
    if (r >= (int64_t)a.batch * a.q_rows) return;
    const int b = (int)(r / a.q_rows), i = (int)(r % a.q_rows), W = a.width, kp = dense_kpad(W);
    const int p0 = a.pos[b];
    const float* h = a.hn + r * W;
    const float* before = i > 0 ? h - W : (p0 > 0 ? a.shift + (int64_t)((p0 + 1) & 1) * a.shift_slot + (int64_t)b * W : nullptr);
    const bool vec = (W & 3) == 0;
    auto get = [&](const float* p, int c0, float (&v)[8]) {
        if (p && vec && c0 + 8 <= W) {
            const float4 x = *reinterpret_cast<const float4*>(p + c0), y = *reinterpret_cast<const float4*>(p + c0 + 4);
            v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; v[4] = y.x; v[5] = y.y; v[6] = y.z; v[7] = y.w;
        } else {
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] = p && c0 + j < W ? p[c0 + j] : 0.0f;
        }
    };
    for (int c0 = (threadIdx.x >> 3) * 8; c0 < kp; c0 += 32 * 8) {
        float v[8], d[8];
        get(h, c0, v);
        get(before, c0, d);
#pragma unroll
        for (int j = 0; j < 8; ++j) d[j] -= v[j];
#pragma unroll
        for (int s = 0; s < 5; ++s) {
            float m[8];
            get(a.mu[s], c0, m);
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                const float x = fmaf(d[j], m[j], v[j]), y = fmaf(d[j + 1], m[j + 1], v[j + 1]);
                hi[j / 2] = ptx::pack2(x, y);
                lo[j / 2] = ptx::pack2(x - __uint_as_float(hi[j / 2] << 16), y - __uint_as_float(hi[j / 2] & 0xffff0000u));
            }
            uint8_t* dst = s < 4 ? a.tiles4 + dense_off(r, s * kp + c0, a.m_pad) : a.tiles_w + dense_off(r, c0, a.m_pad);
            *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            if (s == 4) *reinterpret_cast<uint4*>(a.tiles_w + dense_off(r, kp + c0, a.m_pad)) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
    }
}

// ---------------------------------------------------------------------------------------
// one token per sequence: decays, recurrence, norm of the head's output and gate in one launch; or, with the decays given,
// the recurrence alone
// ---------------------------------------------------------------------------------------
// A CTA per (head, sequence); threads as key groups x value columns.
constexpr int kStepThreads = 512, kMaxRank = 512;

template <int CW>  // columns: 32, 64, 128, 256
__global__ void __launch_bounds__(kStepThreads) wkv_step_kernel(const WkvArgs a) {
    constexpr int G = kStepThreads / CW, KPT = CW / G > 0 ? CW / G : 1;  // key groups, keys per thread
    __shared__ float r_s[CW], k_s[CW], w_s[CW], ru_s[CW];
    __shared__ float low_s[kMaxRank];
    __shared__ float part[kStepThreads];
    __shared__ float red[CW / 32 + 1];
    const int head = blockIdx.x, b = blockIdx.y, D = a.dim, HD = a.heads * D;
    const int col = threadIdx.x % CW, g = threadIdx.x / CW;
    const int p = a.pos[b];
    float* state = a.s + ((int64_t)b * a.heads + head) * D * D;
    // the state is not written by the kernel in front
    float s[KPT];
#pragma unroll
    for (int j = 0; j < KPT; ++j) {
        const int k = g + j * G;
        s[j] = p > 0 && k < D && col < D ? state[(int64_t)k * D + col] : 0.0f;
    }
    ptx::pdl_wait();
    ptx::pdl_launch_dependents();
    const float* row = a.proj + b * a.ld + head * D;
    if (!a.w)
        for (int i = threadIdx.x; i < a.rank; i += kStepThreads) low_s[i] = a.low[(int64_t)b * a.rank + i];
    if (threadIdx.x < CW) {
        const bool live = threadIdx.x < D;
        const float rv = live ? row[threadIdx.x] : 0.0f, kv = live ? row[HD + threadIdx.x] : 0.0f;
        r_s[threadIdx.x] = rv;
        k_s[threadIdx.x] = kv;
        ru_s[threadIdx.x] = live ? rv * a.u[head * D + threadIdx.x] * kv : 0.0f;
    }
    const float v = col < D ? row[2 * HD + col] : 0.0f;
    __syncthreads();
    if (!a.w) {  // decays of the head's key channels: G threads share a channel
        float z = 0.0f;
        if (col < D)
            for (int c0 = g * 8; c0 < a.rank; c0 += G * 8) {
                const uint4 u = *reinterpret_cast<const uint4*>(a.w2_tiles + dense_off(head * D + col, c0, a.w2_pad));
                const uint32_t q[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
                for (int j = 0; j < 4; ++j) {  // beyond the rank the weights are zero
                    z = fmaf(__uint_as_float(q[j] << 16), c0 + 2 * j < a.rank ? low_s[c0 + 2 * j] : 0.0f, z);
                    z = fmaf(__uint_as_float(q[j] & 0xffff0000u), c0 + 2 * j + 1 < a.rank ? low_s[c0 + 2 * j + 1] : 0.0f, z);
                }
            }
        part[threadIdx.x] = z;
    }
    __syncthreads();
    if (threadIdx.x < CW) {
        float z = 0.0f;
        if (a.w) {
            if (threadIdx.x < D) z = a.w[(int64_t)b * HD + head * D + threadIdx.x];
        } else {
#pragma unroll
            for (int i = 0; i < G; ++i) z += part[i * CW + threadIdx.x];
            z = threadIdx.x < D ? expf(-expf(z + a.w0[head * D + threadIdx.x])) : 0.0f;
        }
        w_s[threadIdx.x] = z;
    }
    __syncthreads();
    float o = 0.0f;
#pragma unroll
    for (int j = 0; j < KPT; ++j) {
        const int k = g + j * G;
        o = fmaf(r_s[k], s[j], fmaf(ru_s[k], v, o));
        const float n = fmaf(w_s[k], s[j], k_s[k] * v);
        if (k < D && col < D) state[(int64_t)k * D + col] = n;
    }
    part[threadIdx.x] = o;
    __syncthreads();
    if (threadIdx.x < CW) {
        o = 0.0f;
#pragma unroll
        for (int i = 0; i < G; ++i) o += part[i * CW + threadIdx.x];
        if (a.w && threadIdx.x < D) a.y[(int64_t)b * HD + head * D + threadIdx.x] = o;
        const float ss = warp_sum(o * o);
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    }
    if (a.w) {
        if (head == 0) {  // the token shift's state
            float* keep = a.shift + (int64_t)(p & 1) * a.shift_slot + (int64_t)b * a.width;
            for (int c = threadIdx.x; c < a.width; c += kStepThreads) keep[c] = a.hn[(int64_t)b * a.width + c];
        }
        return;
    }
    __syncthreads();
    if (threadIdx.x < D) {
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < CW / 32; ++i) ss += red[i];
        const float gate = silu_f(row[3 * HD + threadIdx.x]);
        a.y[(int64_t)b * HD + head * D + threadIdx.x] = o / sqrtf(ss / (float)D + a.eps) * a.norm[head * D + threadIdx.x] * gate;
    }
}

// ---------------------------------------------------------------------------------------
// many tokens
// ---------------------------------------------------------------------------------------
// A CTA owns 64 value columns of one head.  Four warps compute, 16 columns each: eight lanes share
// four columns, each with 4 NJ of their state elements in registers (key channels 32 j + 4 lane .. + 3); tokens go by
// fours, whose sums over the lanes are folded together.  Two more warps bring r, k, the decays and v of a tile of tokens into
// shared memory, two tiles ahead, and make the current token's own weight, sum of r u k, one tile ahead.
constexpr int kScanCompute = 4, kScanThreads = 32 * kScanCompute + 64, kScanCols = 64, kScanBufs = 3;
template <int NJ>
struct ScanCfg {
    static constexpr int DP = 32 * NJ, TT = NJ <= 4 ? 16 : 8;
    static constexpr int kTile = TT * (3 * DP + kScanCols + 1);  // floats: r, k, w, v, bonus
    static constexpr size_t kSmem = (size_t)kScanBufs * kTile * sizeof(float);
};
template <int NJ>
__global__ void __launch_bounds__(kScanThreads, NJ <= 2 ? 2 : 1) wkv_scan_kernel(const WkvArgs a) {
    using Cfg = ScanCfg<NJ>;
    constexpr int DP = Cfg::DP, TT = Cfg::TT, Q = DP / 4;  // Q: 16-byte pieces per row
    extern __shared__ __align__(16) float sm[];
    const int head = blockIdx.x, v0 = blockIdx.y * kScanCols, b = blockIdx.z;
    const int D = a.dim, HD = a.heads * D, vc = min(kScanCols, D - v0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int p0 = a.pos[b], count = a.q_rows, tiles = (count + TT - 1) / TT;
    const int64_t row0 = (int64_t)b * count;
    float* state = a.s + ((int64_t)b * a.heads + head) * D * D;
    for (int i = threadIdx.x; i < kScanBufs * Cfg::kTile; i += kScanThreads) sm[i] = 0.0f;  // columns beyond the head's stay zero
    __syncthreads();
    auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };
    if (warp >= kScanCompute) {
        const int tid = threadIdx.x - 32 * kScanCompute;
        const float* rows = a.proj + row0 * a.ld + head * D;
        const float* wrows = a.w + row0 * HD + head * D;
        const bool vec = (D & 3) == 0 && (a.ld & 3) == 0;
        auto fetch = [&](int ti) {
            if (ti >= tiles) return;
            float* t = sm + (ti % kScanBufs) * Cfg::kTile;
            const int i0 = ti * TT, n = min(TT, count - i0);
            if (vec) {
#pragma unroll 4
                for (int e = tid; e < TT * Q; e += 64) {
                    const int i = e / Q, c = e % Q * 4;
                    if (i < n && c < D) {
                        const float* src = rows + (int64_t)(i0 + i) * a.ld + c;
                        const uint32_t dst = ptx::smem_u32(t + i * DP + c);
                        ptx::cp16(dst, src, true);
                        ptx::cp16(dst + TT * DP * 4, src + HD, true);
                        ptx::cp16(dst + 2 * TT * DP * 4, wrows + (int64_t)(i0 + i) * HD + c, true);
                    }
                }
                for (int e = tid; e < TT * (kScanCols / 4); e += 64) {
                    const int i = e / (kScanCols / 4), c = e % (kScanCols / 4) * 4;
                    if (i < n && c < vc) ptx::cp16(ptx::smem_u32(t + 3 * TT * DP + i * kScanCols + c), rows + (int64_t)(i0 + i) * a.ld + 2 * HD + v0 + c, true);
                }
            } else {
                for (int e = tid; e < n * DP; e += 64) {
                    const int i = e / DP, c = e % DP;
                    if (c >= D) continue;
                    const float* src = rows + (int64_t)(i0 + i) * a.ld + c;
                    t[i * DP + c] = src[0];
                    t[TT * DP + i * DP + c] = src[HD];
                    t[2 * TT * DP + i * DP + c] = wrows[(int64_t)(i0 + i) * HD + c];
                }
                for (int e = tid; e < n * kScanCols; e += 64) {
                    const int i = e / kScanCols, c = e % kScanCols;
                    if (c < vc) t[3 * TT * DP + i * kScanCols + c] = rows[(int64_t)(i0 + i) * a.ld + 2 * HD + v0 + c];
                }
            }
            for (int e = tid; e < (TT - n) * DP; e += 64) {  // behind the last token: nothing is added, nothing decays
                const int o = n * DP + e;
                t[o] = 0.0f;
                t[TT * DP + o] = 0.0f;
                t[2 * TT * DP + o] = 1.0f;
            }
        };
        float uu[NJ];  // the bonus
#pragma unroll
        for (int j = 0; j < NJ; ++j) uu[j] = j * 32 + lane < D ? a.u[head * D + j * 32 + lane] : 0.0f;
        auto bonus = [&](int ti) {  // each of the two warps half of the tile's tokens
            if (ti >= tiles) return;
            float* t = sm + (ti % kScanBufs) * Cfg::kTile;
            const int from = (warp - kScanCompute) * (TT / 2);
            float x[TT / 2];
#pragma unroll
            for (int i = 0; i < TT / 2; ++i) {
                x[i] = 0.0f;
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const int at = (from + i) * DP + j * 32 + lane;
                    x[i] = fmaf(t[at] * uu[j], t[TT * DP + at], x[i]);
                }
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int i = 0; i < TT / 2; ++i) x[i] += __shfl_xor_sync(0xffffffffu, x[i], o);
            if (lane == 0)
#pragma unroll
                for (int i = 0; i < TT / 2; ++i) t[TT * (3 * DP + kScanCols) + from + i] = x[i];
        };
        auto landed = [&] {  // the copies of both warps, all but the last tile asked for
            asm volatile("cp.async.wait_group 1;" ::: "memory");
            asm volatile("bar.sync 1, 64;" ::: "memory");
        };
        fetch(0);
        commit();
        fetch(1);
        commit();
        landed();
        bonus(0);
        __syncthreads();
        for (int ti = 0; ti < tiles; ++ti) {
            fetch(ti + 2);
            commit();
            landed();
            bonus(ti + 1);
            __syncthreads();
        }
        if (blockIdx.x == 0 && blockIdx.y == 0) {  // the token shift's state
            float* keep = a.shift + (int64_t)((p0 + a.q_rows - 1) & 1) * a.shift_slot + (int64_t)b * a.width;
            for (int c = tid; c < a.width; c += 64) keep[c] = a.hn[(row0 + count - 1) * a.width + c];
        }
        return;
    }
    const int col = warp * 16 + (lane >> 3) * 4, kg = lane & 7;
    float s[4 * NJ][4];  // key channels x columns
#pragma unroll
    for (int j = 0; j < 4 * NJ; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int k = 32 * (j >> 2) + 4 * kg + (j & 3);
            s[j][c] = col + c < vc && k < D && p0 > 0 ? state[(int64_t)k * D + v0 + col + c] : 0.0f;
        }
    __syncthreads();
    for (int ti = 0; ti < tiles; ++ti) {
        const float* rs = sm + (ti % kScanBufs) * Cfg::kTile;
        const float* ks = rs + TT * DP;
        const float* ws = ks + TT * DP;
        const float* vs = ws + TT * DP;
        const float* bonus_s = vs + TT * kScanCols;
        const int i0 = ti * TT;
#pragma unroll 1
        for (int g = 0; g < TT && i0 + g < count; g += 4) {
            float o[4][4];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float4 v = *reinterpret_cast<const float4*>(vs + (g + q) * kScanCols + col);
                const float vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                for (int c = 0; c < 4; ++c) o[q][c] = 0.0f;
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const int at = (g + q) * DP + 32 * j + 4 * kg;
                    const float4 x = *reinterpret_cast<const float4*>(rs + at), y = *reinterpret_cast<const float4*>(ks + at), z = *reinterpret_cast<const float4*>(ws + at);
                    const float r[4] = {x.x, x.y, x.z, x.w}, k[4] = {y.x, y.y, y.z, y.w}, w[4] = {z.x, z.y, z.z, z.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e)
#pragma unroll
                        for (int c = 0; c < 4; ++c) {
                            o[q][c] = fmaf(r[e], s[4 * j + e][c], o[q][c]);
                            s[4 * j + e][c] = fmaf(w[e], s[4 * j + e][c], k[e] * vv[c]);
                        }
                }
            }
            // fold over the eight lanes of the columns: lane kg ends with two columns of token g + kg / 2
#pragma unroll
            for (int st = 2; st > 0; st >>= 1) {
                const bool hi = kg & (2 * st);
#pragma unroll
                for (int q = 0; q < st; ++q)
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        const float give = hi ? o[q][c] : o[q + st][c], keep = hi ? o[q + st][c] : o[q][c];
                        o[q][c] = keep + __shfl_xor_sync(0xffffffffu, give, 2 * st);
                    }
            }
            const int c0 = (kg & 1) * 2, tk = g + (kg >> 1);
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                const float give = c0 ? o[0][c] : o[0][c + 2], keep = c0 ? o[0][c + 2] : o[0][c];
                o[0][c] = keep + __shfl_xor_sync(0xffffffffu, give, 1);
            }
            if (i0 + tk < count) {
                float* y = a.y + (row0 + i0 + tk) * HD + head * D + v0 + col + c0;
                const float bonus = bonus_s[tk];
#pragma unroll
                for (int c = 0; c < 2; ++c)
                    if (col + c0 + c < vc) y[c] = fmaf(bonus, vs[tk * kScanCols + col + c0 + c], o[0][c]);
            }
        }
        __syncthreads();  // the tile may be refilled, the next one is there
    }
#pragma unroll
    for (int j = 0; j < 4 * NJ; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int k = 32 * (j >> 2) + 4 * kg + (j & 3);
            if (col + c < vc && k < D) state[(int64_t)k * D + v0 + col + c] = s[j][c];
        }
}

// ---------------------------------------------------------------------------------------
// many tokens of a 16-bit model, heads of at most 64: sixteen tokens at a time on the tensor cores
// ---------------------------------------------------------------------------------------
// With P_t the product of the block's decays before token t and Q_t of those behind it, a block of tokens is
//   o_t = (r_t P_t)^T S + sum over s <= t of A_ts v_s,    S <- diag(all decays) S + sum over s of (k_s Q_s) v_s^T,
//   A_ts = sum over channels of r_t k_s (the decays between s and t) for s < t,    A_tt = sum of r_t u k_t.
// No quotient of decays appears, so nothing overflows.  A, P and Q are made in f32; the factors of the products go in as bf16
// hi + lo (16 significand bits), sums and the state stay f32.  A CTA owns a head and a segment of the tokens, a warp 16 value
// columns of it, whose state S^T stays in the warp's accumulators.
// Several segments: each but the first starts from zero; wkv_join_kernel carries the states over the segments, wkv_carry_kernel
// adds what a segment's incoming state means for its tokens.
constexpr int kSegments = 16, kBlock = 64;  // most segments; their length is a multiple of kBlock
constexpr int kTok = 16, kHead = 64, kLd = 72, kLdA = 24;  // tokens per step, padded head, bf16 elements per shared-memory row
struct BlockSmem {
    float raw[2][4][kTok][kHead];  // r, k, decays, v as they come
    float decay[2][kHead];         // a step's whole decay per channel
    __nv_bfloat16 rows[2][6][kTok][kLd];  // hi and lo of r P, k Q and v
    __nv_bfloat16 tri[2][2][kTok][kLdA];  // hi and lo of A
};
__device__ __forceinline__ void split16(float v, __nv_bfloat16& hi, __nv_bfloat16& lo) {
    hi = __float2bfloat16_rn(v);
    lo = __float2bfloat16_rn(v - __bfloat162float(hi));
}
// two values into bf16 pairs: hi parts and lo parts
__device__ __forceinline__ void split16x2(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = ptx::pack2(x, y);
    lo = ptx::pack2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}
__global__ void __launch_bounds__(128, 3) wkv_block_kernel(const WkvArgs a, int segs, int seg_tokens) {
    extern __shared__ __align__(16) uint8_t block_smem[];
    BlockSmem& m = *reinterpret_cast<BlockSmem*>(block_smem);
    const int D = a.dim, HD = a.heads * D;
    const int head = blockIdx.x, seg = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int first = seg * seg_tokens, count = min(seg_tokens, a.q_rows - first), steps = (count + kTok - 1) / kTok;
    const int p0 = a.pos[b];
    const int64_t row0 = (int64_t)b * a.q_rows + first;
    // where the segment's last state goes: the sequence's state, or its place among the segments
    float* state = a.s + ((int64_t)b * a.heads + head) * D * D;
    float* result = segs > 1 ? a.seg_s + (((int64_t)b * a.heads + head) * kSegments + seg) * (D * D + D) : state;
    const float* proj = a.proj + row0 * a.ld + head * D;
    const float* wrow = a.w + row0 * HD + head * D;
    auto fetch = [&](int i) {
        if (i < steps) {
#pragma unroll
            for (int e = tid; e < kTok * kHead / 4; e += 128) {
                const int t = e >> 4, c = (e & 15) * 4, at = i * kTok + t;
                const bool ok = at < count && c < D;
                const float* src = proj + (int64_t)(ok ? at : 0) * a.ld + (ok ? c : 0);
                ptx::cp16(ptx::smem_u32(&m.raw[i & 1][0][t][c]), src, ok);
                ptx::cp16(ptx::smem_u32(&m.raw[i & 1][1][t][c]), src + HD, ok);
                ptx::cp16(ptx::smem_u32(&m.raw[i & 1][3][t][c]), src + 2 * HD, ok);
                if (at < count) ptx::cp16(ptx::smem_u32(&m.raw[i & 1][2][t][c]), wrow + (int64_t)at * HD + (ok ? c : 0), ok);
                else *reinterpret_cast<float4*>(&m.raw[i & 1][2][t][c]) = make_float4(1.f, 1.f, 1.f, 1.f);  // behind the last token nothing decays
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0);
    fetch(1);
    for (int i = tid; i < (int)sizeof(m.tri) / 4; i += 128) reinterpret_cast<uint32_t*>(m.tri)[i] = 0;  // above A's diagonal
    float st[8][4];  // S^T: tiles of 8 key channels; this lane's rows (values) and columns (keys) as in an accumulator
    const int vr = warp * 16 + (lane >> 2), kc = (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int v = vr + (e >> 1) * 8, k = n * 8 + kc + (e & 1);
            st[n][e] = v < D && k < D && p0 > 0 && seg == 0 ? state[k * D + v] : 0.0f;
        }
    const int c4 = (lane & 15) * 4, s0 = 2 * warp + (lane >> 4), s1 = kTok - 1 - s0;  // A's columns of this lane's group
    float u[4], whole = 1.0f;  // whole: the decays of the segment so far, channel tid
#pragma unroll
    for (int e = 0; e < 4; ++e) u[e] = c4 + e < D ? a.u[head * D + c4 + e] : 0.0f;
    for (int i = 0; i < steps; ++i) {
        const int buf = i & 1;
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const float(*rs)[kHead] = m.raw[buf][0], (*ks)[kHead] = m.raw[buf][1], (*ws)[kHead] = m.raw[buf][2], (*vs)[kHead] = m.raw[buf][3];
        {   // r with the decays before it (threads 0-63), k with those behind it
            const int c = tid & 63;
            float run = 1.0f;
            if (tid < 64) {
#pragma unroll
                for (int t = 0; t < kTok; ++t) {
                    split16(rs[t][c] * run, m.rows[buf][0][t][c], m.rows[buf][1][t][c]);
                    run *= ws[t][c];
                }
                m.decay[buf][c] = run;
                if (segs > 1 && c < D) {
                    if (seg > 0 && i * kTok % kBlock == 0)
                        a.seg_w[(((int64_t)b * ((a.q_rows + kBlock - 1) / kBlock) + (first + i * kTok) / kBlock) * a.heads + head) * D + c] = whole;
                    whole *= run;
                }
            } else {
#pragma unroll
                for (int t = kTok - 1; t >= 0; --t) {
                    split16(ks[t][c] * run, m.rows[buf][2][t][c], m.rows[buf][3][t][c]);
                    run *= ws[t][c];
                }
            }
        }
        {   // v
            const int t = tid >> 3, c = (tid & 7) * 8;
            const float4 x = *reinterpret_cast<const float4*>(&vs[t][c]), y = *reinterpret_cast<const float4*>(&vs[t][c + 4]);
            uint4 hi, lo;
            split16x2(x.x, x.y, hi.x, lo.x);
            split16x2(x.z, x.w, hi.y, lo.y);
            split16x2(y.x, y.y, hi.z, lo.z);
            split16x2(y.z, y.w, hi.w, lo.w);
            *reinterpret_cast<uint4*>(&m.rows[buf][4][t][c]) = hi;
            *reinterpret_cast<uint4*>(&m.rows[buf][5][t][c]) = lo;
        }
        {   // A: sixteen lanes share columns s0 and 15 - s0, fifteen elements below the diagonal and two on it
            float x[16], last = 0.0f, kd[4];
            const int n0 = kTok - 1 - s0;  // elements of column s0
            const float4 ka = *reinterpret_cast<const float4*>(&ks[s0][c4]), kb = *reinterpret_cast<const float4*>(&ks[s1][c4]);
            const float4 ra = *reinterpret_cast<const float4*>(&rs[s0][c4]), rb = *reinterpret_cast<const float4*>(&rs[s1][c4]);
            x[15] = ra.x * u[0] * ka.x + ra.y * u[1] * ka.y + ra.z * u[2] * ka.z + ra.w * u[3] * ka.w;
            last = rb.x * u[0] * kb.x + rb.y * u[1] * kb.y + rb.z * u[2] * kb.z + rb.w * u[3] * kb.w;
            kd[0] = ka.x; kd[1] = ka.y; kd[2] = ka.z; kd[3] = ka.w;
#pragma unroll
            for (int j = 0; j < kTok - 1; ++j) {
                if (j == n0) { kd[0] = kb.x; kd[1] = kb.y; kd[2] = kb.z; kd[3] = kb.w; }
                const int t = j < n0 ? s0 + 1 + j : j + 1;
                const float4 r = *reinterpret_cast<const float4*>(&rs[t][c4]), w = *reinterpret_cast<const float4*>(&ws[t][c4]);
                x[j] = fmaf(r.x, kd[0], fmaf(r.y, kd[1], fmaf(r.z, kd[2], r.w * kd[3])));
                kd[0] *= w.x; kd[1] *= w.y; kd[2] *= w.z; kd[3] *= w.w;
            }
#pragma unroll
            for (int h = 8; h > 0; h >>= 1) {
                const bool up = lane & h;
#pragma unroll
                for (int q = 0; q < h; ++q) {
                    const float give = up ? x[q] : x[q + h], keep = up ? x[q + h] : x[q];
                    x[q] = keep + __shfl_xor_sync(0xffffffffu, give, h);
                }
                last += __shfl_xor_sync(0xffffffffu, last, h);
            }
            const int l = lane & 15, s = l < n0 || l == 15 ? s0 : s1, t = l == 15 ? s0 : (l < n0 ? s0 + 1 + l : l + 1);
            split16(x[0], m.tri[buf][0][t][s], m.tri[buf][1][t][s]);
            if (l == 0) split16(last, m.tri[buf][0][s1][s1], m.tri[buf][1][s1][s1]);
        }
        __syncthreads();
        fetch(i + 2);
        float o[2][4] = {};  // o^T: tiles of 8 tokens
        uint32_t vh[4], vl[4];
        {
            const uint32_t at = (((lane & 7) + (lane >> 4) * 8) * kLd + warp * 16 + ((lane >> 3) & 1) * 8) * 2;
            ptx::ldsm4t(vh, ptx::smem_u32(m.rows[buf][4]) + at);
            ptx::ldsm4t(vl, ptx::smem_u32(m.rows[buf][5]) + at);
            uint32_t th[4], tl[4];
            const uint32_t ta = (((lane & 7) + (lane >> 4) * 8) * kLdA + ((lane >> 3) & 1) * 8) * 2;
            ptx::ldsm4(th, ptx::smem_u32(m.tri[buf][0]) + ta);
            ptx::ldsm4(tl, ptx::smem_u32(m.tri[buf][1]) + ta);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                ptx::mma_bf16(o[n], vh, th[2 * n], th[2 * n + 1]);
                ptx::mma_bf16(o[n], vl, th[2 * n], th[2 * n + 1]);
                ptx::mma_bf16(o[n], vh, tl[2 * n], tl[2 * n + 1]);
            }
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) {  // sixteen key channels
            uint32_t sh[4], sl[4], bh[4], bl[4];
            split16x2(st[2 * k][0], st[2 * k][1], sh[0], sl[0]);
            split16x2(st[2 * k][2], st[2 * k][3], sh[1], sl[1]);
            split16x2(st[2 * k + 1][0], st[2 * k + 1][1], sh[2], sl[2]);
            split16x2(st[2 * k + 1][2], st[2 * k + 1][3], sh[3], sl[3]);
            const uint32_t ra = (((lane & 7) + (lane >> 4) * 8) * kLd + k * 16 + ((lane >> 3) & 1) * 8) * 2;
            ptx::ldsm4(bh, ptx::smem_u32(m.rows[buf][0]) + ra);
            ptx::ldsm4(bl, ptx::smem_u32(m.rows[buf][1]) + ra);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                ptx::mma_bf16(o[n], sh, bh[2 * n], bh[2 * n + 1]);
                ptx::mma_bf16(o[n], sl, bh[2 * n], bh[2 * n + 1]);
                ptx::mma_bf16(o[n], sh, bl[2 * n], bl[2 * n + 1]);
            }
            const uint32_t ka = (((lane & 7) + ((lane >> 3) & 1) * 8) * kLd + k * 16 + (lane >> 4) * 8) * 2;
            ptx::ldsm4t(bh, ptx::smem_u32(m.rows[buf][2]) + ka);
            ptx::ldsm4t(bl, ptx::smem_u32(m.rows[buf][3]) + ka);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                float(&x)[4] = st[2 * k + n];
                const float2 d = *reinterpret_cast<const float2*>(&m.decay[buf][k * 16 + n * 8 + kc]);
                x[0] *= d.x; x[1] *= d.y; x[2] *= d.x; x[3] *= d.y;
                ptx::mma_bf16(x, vh, bh[2 * n], bh[2 * n + 1]);
                ptx::mma_bf16(x, vl, bh[2 * n], bh[2 * n + 1]);
                ptx::mma_bf16(x, vh, bl[2 * n], bl[2 * n + 1]);
            }
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = i * kTok + n * 8 + kc + (e & 1), v = vr + (e >> 1) * 8;
                if (t < count && v < D) a.y[(row0 + t) * HD + head * D + v] = o[n][e];
            }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int v = vr + (e >> 1) * 8, k = n * 8 + kc + (e & 1);
            if (v < D && k < D) result[k * D + v] = st[n][e];
        }
    if (segs > 1 && tid < D) result[D * D + tid] = whole;  // heads of 64: threads 0-63
    if (head == 0 && seg == segs - 1) {  // the token shift's state
        float* keep = a.shift + (int64_t)((p0 + a.q_rows - 1) & 1) * a.shift_slot + (int64_t)b * a.width;
        for (int c = tid; c < a.width; c += 128) keep[c] = a.hn[(row0 + count - 1) * a.width + c];
    }
}

// The states over the segments: a segment's place gets its incoming state, the sequence the last one.
__global__ void __launch_bounds__(256) wkv_join_kernel(const WkvArgs a, int segs) {
    const int D = a.dim, e = blockIdx.x * 256 + threadIdx.x;
    if (e >= D * D) return;
    const int64_t head = blockIdx.y;  // of all sequences
    float* seg = a.seg_s + head * kSegments * (D * D + D);
    float own[kSegments], decay[kSegments];
#pragma unroll
    for (int i = 0; i < kSegments; ++i) {
        own[i] = i < segs ? seg[(int64_t)i * (D * D + D) + e] : 0.0f;
        decay[i] = i < segs ? seg[(int64_t)i * (D * D + D) + D * D + e / D] : 0.0f;
    }
    float s = own[0];
#pragma unroll
    for (int i = 1; i < kSegments; ++i)
        if (i < segs) {
            seg[(int64_t)i * (D * D + D) + e] = s;
            s = fmaf(decay[i], s, own[i]);
        }
    a.s[head * D * D + e] = s;
}

// o_t += (r_t times the decays since the segment's start)^T S for the segments behind the first: a CTA per head and 64 tokens,
// on the tensor cores, both factors as bf16 hi + lo (16 significand bits).  Head size 64.
constexpr int kCarryDim = 64, kCarryLd = 72;
__global__ void __launch_bounds__(256) wkv_carry_kernel(const WkvArgs a, int seg_tokens) {
    __shared__ __align__(16) __nv_bfloat16 rh[64][kCarryLd], rl[64][kCarryLd], sh[64][kCarryLd], sl[64][kCarryLd];
    __shared__ float part[4][64];
    __shared__ int any;
    const int D = kCarryDim, HD = a.heads * D;
    const int per = seg_tokens / kBlock;
    const int head = blockIdx.x, seg = blockIdx.y / per + 1, b = blockIdx.z, t0 = (blockIdx.y % per) * kBlock;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int first = seg * seg_tokens, count = min(seg_tokens, a.q_rows - first);
    if (t0 >= count) return;
    const int64_t row0 = (int64_t)b * a.q_rows + first;
    const float* S = a.seg_s + (((int64_t)b * a.heads + head) * kSegments + seg) * (D * D + D);
    const int ch = threadIdx.x & 63, quarter = threadIdx.x >> 6;  // a channel, 16 of the 64 tokens
    float r[16], w[16], p = 1.0f, run;                              // run: the decays before the token
    {
        run = a.seg_w[(((int64_t)b * ((a.q_rows + kBlock - 1) / kBlock) + (first + t0) / kBlock) * a.heads + head) * D + ch];
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const int t = t0 + quarter * 16 + i;
        const bool ok = t < count;
        r[i] = ok ? a.proj[(row0 + t) * a.ld + head * D + ch] : 0.0f;
        w[i] = ok ? a.w[(row0 + t) * HD + head * D + ch] : 1.0f;
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) p *= w[i];
    part[quarter][ch] = p;
    if (threadIdx.x == 0) any = 0;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 3; ++i)
        if (i < quarter) run *= part[i][ch];
    bool live = false;
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const float v = r[i] * run;
        live |= v != 0.0f;
        run *= w[i];
        const __nv_bfloat16 hi = __float2bfloat16_rn(v);
        rh[quarter * 16 + i][ch] = hi;
        rl[quarter * 16 + i][ch] = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
    if (live) any = 1;
    __syncthreads();
    if (any == 0) return;  // everything has decayed away
    for (int i = threadIdx.x; i < D * D; i += 256) {  // [key][value]
        const float v = S[i];
        const __nv_bfloat16 hi = __float2bfloat16_rn(v);
        sh[i >> 6][i & 63] = hi;
        sl[i >> 6][i & 63] = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
    __syncthreads();
    // warps as 4 (16 tokens) x 2 (32 values)
    const int tt = warp >> 1, vv = (warp & 1) * 32;
    float o[4][4] = {};
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        uint32_t ah[4], al[4];
        const uint32_t a_off = ((tt * 16 + (lane & 15)) * kCarryLd + k * 16 + (lane >> 4) * 8) * 2;
        ptx::ldsm4(ah, ptx::smem_u32(rh) + a_off);
        ptx::ldsm4(al, ptx::smem_u32(rl) + a_off);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            uint32_t bh[4], bl[4];
            const uint32_t b_off = ((k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kCarryLd + vv + n * 16 + (lane >> 4) * 8) * 2;
            ptx::ldsm4t(bh, ptx::smem_u32(sh) + b_off);
            ptx::ldsm4t(bl, ptx::smem_u32(sl) + b_off);
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                ptx::mma_bf16(o[2 * n + q], ah, bh[2 * q], bh[2 * q + 1]);
                ptx::mma_bf16(o[2 * n + q], al, bh[2 * q], bh[2 * q + 1]);
                ptx::mma_bf16(o[2 * n + q], ah, bl[2 * q], bl[2 * q + 1]);
            }
        }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int t = t0 + tt * 16 + (lane >> 2) + half * 8;
            if (t < count) {
                float2* y = reinterpret_cast<float2*>(a.y + (row0 + t) * HD + head * D + vv + n * 8 + (lane & 3) * 2);
                float2 x = *y;
                x.x += o[n][2 * half];
                x.y += o[n][2 * half + 1];
                *y = x;
            }
        }
}

// segments of the tokens: the fewest rounds of CTAs (three share an SM) times tokens, no segment below 128 tokens
int segments(const WkvArgs& a) {
    if (!a.seg_s || !a.seg_w || a.dim != kCarryDim) return 1;
    const int64_t ctas = (int64_t)a.heads * a.batch, slots = 3ll * a.sm_count;
    int best = 1;
    int64_t least = 0;
    for (int segs = 1; segs <= kSegments && (segs == 1 || a.q_rows / segs >= 128); ++segs) {
        const int64_t cost = (ctas * segs + slots - 1) / slots * (((a.q_rows + segs - 1) / segs + kBlock - 1) / kBlock);
        if (segs == 1 || cost < least) { best = segs; least = cost; }
    }
    return best;
}
template <int NJ>
cudaError_t scan_launch(const WkvArgs& a, cudaStream_t s) {
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(wkv_scan_kernel<NJ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ScanCfg<NJ>::kSmem); });
    if (e != cudaSuccess) return e;
    wkv_scan_kernel<NJ><<<dim3((unsigned)a.heads, (unsigned)((a.dim + kScanCols - 1) / kScanCols), (unsigned)a.batch), kScanThreads, ScanCfg<NJ>::kSmem, s>>>(a);
    return cudaGetLastError();
}
bool takes_blocks(const WkvArgs& a) { return a.split16 && a.dim <= kHead && a.dim % 4 == 0 && a.ld % 4 == 0 && a.q_rows >= kTok; }
cudaError_t block_launch(const WkvArgs& a, cudaStream_t s) {
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(wkv_block_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(BlockSmem)); });
    if (e != cudaSuccess) return e;
    int segs = segments(a);
    const int tokens = ((a.q_rows + segs - 1) / segs + kBlock - 1) / kBlock * kBlock;
    segs = (a.q_rows + tokens - 1) / tokens;
    wkv_block_kernel<<<dim3((unsigned)a.heads, (unsigned)segs, (unsigned)a.batch), 128, sizeof(BlockSmem), s>>>(a, segs, tokens);
    if (segs > 1) {
        wkv_join_kernel<<<dim3((unsigned)((a.dim * a.dim + 255) / 256), (unsigned)(a.heads * a.batch)), 256, 0, s>>>(a, segs);
        wkv_carry_kernel<<<dim3((unsigned)a.heads, (unsigned)((segs - 1) * (tokens / kBlock)), (unsigned)a.batch), 256, 0, s>>>(a, tokens);
    }
    return cudaGetLastError();
}
cudaError_t step_launch(const WkvArgs& a, cudaStream_t s, bool pdl) {
    const dim3 grid((unsigned)a.heads, (unsigned)a.batch), block(kStepThreads);
    if (a.dim <= 32) return launch_pdl(wkv_step_kernel<32>, grid, block, 0, s, pdl, a);
    if (a.dim <= 64) return launch_pdl(wkv_step_kernel<64>, grid, block, 0, s, pdl, a);
    if (a.dim <= 128) return launch_pdl(wkv_step_kernel<128>, grid, block, 0, s, pdl, a);
    return launch_pdl(wkv_step_kernel<256>, grid, block, 0, s, pdl, a);
}

}  // namespace

int wkv_max_dim() { return 256; }
int64_t wkv_segment_floats(int heads, int dim) { return dim == kCarryDim ? (int64_t)heads * kSegments * (dim * dim + dim) : 0; }
int64_t wkv_prefix_floats(int heads, int dim, int64_t rows, int batch) { return dim == kCarryDim ? (rows / kBlock + batch) * heads * dim : 0; }

cudaError_t launch_wkv_mix(const WkvMix& a, cudaStream_t s) {
    const unsigned rows = (unsigned)(a.batch * a.q_rows);
    if (a.rows5) wkv_mix_kernel<<<rows, 256, 0, s>>>(a);
    else wkv_mix_tiles_kernel<<<(rows + 7) / 8, 256, 0, s>>>(a);
    return cudaGetLastError();
}

cudaError_t launch_wkv_step(const WkvArgs& a, cudaStream_t s, bool pdl) {
    if (a.dim > wkv_max_dim() || a.rank > kMaxRank || a.q_rows != 1) return cudaErrorInvalidValue;
    WkvArgs x = a;
    x.w = nullptr;
    return step_launch(x, s, pdl);
}

cudaError_t launch_wkv_prefill(const WkvArgs& a, cudaStream_t s) {
    if (a.dim > wkv_max_dim() || !a.w) return cudaErrorInvalidValue;
    if (a.q_rows == 1) return step_launch(a, s, false);
    if (takes_blocks(a)) return block_launch(a, s);
    if (a.dim <= 32) return scan_launch<1>(a, s);
    if (a.dim <= 64) return scan_launch<2>(a, s);
    if (a.dim <= 128) return scan_launch<4>(a, s);
    return scan_launch<8>(a, s);
}

}  // namespace bt
