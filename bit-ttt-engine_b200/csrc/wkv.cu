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
    const int b = (int)(r / a.q_rows), i = (int)(r % a.q_rows), W = a.width, kp = dense_kpad(W);
    const int p0 = a.pos[b];
    const float* h = a.hn + r * W;
    const float* before = i > 0 ? h - W : (p0 > 0 ? a.shift + (int64_t)((p0 + 1) & 1) * a.shift_slot + (int64_t)b * W : nullptr);
    if (a.rows5) {
        for (int c = threadIdx.x; c < W; c += 256) {
            const float v = h[c], d = (before ? before[c] : 0.0f) - v;
#pragma unroll
            for (int s = 0; s < 5; ++s) a.rows5[(r * 5 + s) * W + c] = fmaf(d, a.mu[s][c], v);
        }
        return;
    }
    for (int c0 = threadIdx.x * 8; c0 < kp; c0 += 256 * 8) {
        float v[8], d[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const bool live = c0 + j < W;
            v[j] = live ? h[c0 + j] : 0.0f;
            d[j] = (live && before ? before[c0 + j] : 0.0f) - v[j];
        }
#pragma unroll
        for (int s = 0; s < 5; ++s) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                const float x = c0 + j < W ? fmaf(d[j], a.mu[s][c0 + j], v[j]) : 0.0f;
                const float y = c0 + j + 1 < W ? fmaf(d[j + 1], a.mu[s][c0 + j + 1], v[j + 1]) : 0.0f;
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
// many tokens, one after the other
// ---------------------------------------------------------------------------------------
// A CTA owns 16 value columns of one head.  Two warps compute, 8 columns each: eight lanes share two columns, each with 4 NJ
// of their state elements in registers as pairs (key channels 32 j + 4 lane .. + 3); tokens go by eights, whose sums over the
// lanes are folded together.  Two more warps bring r, k, the decays and v of a tile of tokens into shared memory, two tiles
// ahead, and make the current token's own weight, sum of r u k, one tile ahead.
constexpr int kScanThreads = 128, kScanCols = 16, kScanBufs = 3;
template <int NJ>
struct ScanCfg {
    static constexpr int DP = 32 * NJ, TT = NJ <= 4 ? 16 : 8;
    static constexpr int kTile = TT * (3 * DP + kScanCols + 1);  // floats: r, k, w, v, bonus
    static constexpr size_t kSmem = (size_t)kScanBufs * kTile * sizeof(float);
};
// two f32 values side by side
typedef unsigned long long f2;
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
    f2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
    f2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f2 pair2(float x, float y) {
    f2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
    return d;
}
__device__ __forceinline__ float2 split2(f2 a) {
    float2 d;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(a));
    return d;
}

template <int NJ>
__global__ void __launch_bounds__(kScanThreads) wkv_scan_kernel(const WkvArgs a) {
    using Cfg = ScanCfg<NJ>;
    constexpr int DP = Cfg::DP, TT = Cfg::TT, Q = DP / 4;  // Q: 16-byte pieces per row
    extern __shared__ __align__(16) float sm[];
    const int head = blockIdx.x, v0 = blockIdx.y * kScanCols, b = blockIdx.z;
    const int D = a.dim, HD = a.heads * D, vc = min(kScanCols, D - v0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int p0 = a.pos[b], tiles = (a.q_rows + TT - 1) / TT;
    for (int i = threadIdx.x; i < kScanBufs * Cfg::kTile; i += kScanThreads) sm[i] = 0.0f;  // columns beyond the head's stay zero
    __syncthreads();
    auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };
    if (warp >= 2) {
        const int tid = threadIdx.x - 64;
        const float* rows = a.proj + (int64_t)b * a.q_rows * a.ld + head * D;
        const float* wrows = a.w + (int64_t)b * a.q_rows * HD + head * D;
        const bool vec = (D & 3) == 0 && (a.ld & 3) == 0;
        auto fetch = [&](int ti) {
            if (ti >= tiles) return;
            float* t = sm + (ti % kScanBufs) * Cfg::kTile;
            const int i0 = ti * TT, n = min(TT, a.q_rows - i0);
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
                if (tid < TT * (kScanCols / 4)) {
                    const int i = tid / (kScanCols / 4), c = tid % (kScanCols / 4) * 4;
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
        float uu[NJ];
#pragma unroll
        for (int j = 0; j < NJ; ++j) uu[j] = j * 32 + lane < D ? a.u[head * D + j * 32 + lane] : 0.0f;
        auto bonus = [&](int ti) {  // each of the two warps half of the tile's tokens
            if (ti >= tiles) return;
            float* t = sm + (ti % kScanBufs) * Cfg::kTile;
            const int first = (warp - 2) * (TT / 2);
            float x[TT / 2];
#pragma unroll
            for (int i = 0; i < TT / 2; ++i) {
                x[i] = 0.0f;
#pragma unroll
                for (int j = 0; j < NJ; ++j) x[i] = fmaf(t[(first + i) * DP + j * 32 + lane] * uu[j], t[TT * DP + (first + i) * DP + j * 32 + lane], x[i]);
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int i = 0; i < TT / 2; ++i) x[i] += __shfl_xor_sync(0xffffffffu, x[i], o);
            if (lane == 0)
#pragma unroll
                for (int i = 0; i < TT / 2; ++i) t[TT * (3 * DP + kScanCols) + first + i] = x[i];
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
            const int64_t last = (int64_t)b * a.q_rows + a.q_rows - 1;
            float* keep = a.shift + (int64_t)((p0 + a.q_rows - 1) & 1) * a.shift_slot + (int64_t)b * a.width;
            for (int c = tid; c < a.width; c += 64) keep[c] = a.hn[last * a.width + c];
        }
        return;
    }
    const int col = warp * 8 + (lane >> 3) * 2, kg = lane & 7;
    float* state = a.s + ((int64_t)b * a.heads + head) * D * D + v0 + col;
    f2 s[2 * NJ][2];  // pairs of key channels x two columns
#pragma unroll
    for (int j = 0; j < 2 * NJ; ++j)
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            float x[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int k = 32 * (j >> 1) + 4 * kg + 2 * (j & 1) + e;
                x[e] = col + c < vc && k < D && p0 > 0 ? state[(int64_t)k * D + c] : 0.0f;
            }
            s[j][c] = pair2(x[0], x[1]);
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
        for (int g = 0; g < TT && i0 + g < a.q_rows; g += 8) {
            float o[8][2];
            // a token's values are loaded while the one before it is worked on
            ulonglong2 r4[2][NJ], k4[2][NJ], w4[2][NJ];
            float2 v2[2];
            auto take = [&](int which, int tk) {
                v2[which] = *reinterpret_cast<const float2*>(vs + tk * kScanCols + col);
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const int at = tk * DP + 32 * j + 4 * kg;
                    r4[which][j] = *reinterpret_cast<const ulonglong2*>(rs + at);
                    k4[which][j] = *reinterpret_cast<const ulonglong2*>(ks + at);
                    w4[which][j] = *reinterpret_cast<const ulonglong2*>(ws + at);
                }
            };
            take(0, g);
#pragma unroll
            for (int q = 0; q < 8; ++q) {
                if (q < 7) take((q + 1) & 1, g + q + 1);
                const f2 vv[2] = {pair2(v2[q & 1].x, v2[q & 1].x), pair2(v2[q & 1].y, v2[q & 1].y)};
                f2 sum[2][2];
#pragma unroll
                for (int j = 0; j < 2 * NJ; ++j) {
                    const ulonglong2 x = r4[q & 1][j >> 1], y = k4[q & 1][j >> 1], z = w4[q & 1][j >> 1];
                    const f2 r = j & 1 ? x.y : x.x, k = j & 1 ? y.y : y.x, w = j & 1 ? z.y : z.x;
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        sum[j & 1][c] = j < 2 ? mul2(r, s[j][c]) : fma2(r, s[j][c], sum[j & 1][c]);
                        s[j][c] = fma2(w, s[j][c], mul2(k, vv[c]));
                    }
                }
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    const float2 x = split2(sum[0][c]), y = split2(sum[1][c]);
                    o[q][c] = (x.x + y.x) + (x.y + y.y);
                }
            }
            // fold over the eight lanes of a column pair: lane kg ends with token g + kg
#pragma unroll
            for (int st = 4; st > 0; st >>= 1) {
                const bool hi = kg & st;
#pragma unroll
                for (int q = 0; q < st; ++q)
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        const float give = hi ? o[q][c] : o[q + st][c], keep = hi ? o[q + st][c] : o[q][c];
                        o[q][c] = keep + __shfl_xor_sync(0xffffffffu, give, st);
                    }
            }
            const int tk = g + kg;
            if (i0 + tk < a.q_rows) {
                float* y = a.y + ((int64_t)b * a.q_rows + i0 + tk) * HD + head * D + v0 + col;
                const float bonus = bonus_s[tk];
#pragma unroll
                for (int c = 0; c < 2; ++c)
                    if (col + c < vc) y[c] = fmaf(bonus, vs[tk * kScanCols + col + c], o[0][c]);
            }
        }
        __syncthreads();  // the tile may be refilled, the next one is there
    }
#pragma unroll
    for (int j = 0; j < 2 * NJ; ++j)
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            const float2 x = split2(s[j][c]);
            const int k = 32 * (j >> 1) + 4 * kg + 2 * (j & 1);
            if (col + c < vc) {
                if (k < D) state[(int64_t)k * D + c] = x.x;
                if (k + 1 < D) state[(int64_t)(k + 1) * D + c] = x.y;
            }
        }
}

template <int NJ>
cudaError_t scan_launch(const WkvArgs& a, cudaStream_t s) {
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(wkv_scan_kernel<NJ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ScanCfg<NJ>::kSmem); });
    if (e != cudaSuccess) return e;
    wkv_scan_kernel<NJ><<<dim3((unsigned)a.heads, (unsigned)((a.dim + kScanCols - 1) / kScanCols), (unsigned)a.batch), kScanThreads, ScanCfg<NJ>::kSmem, s>>>(a);
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

cudaError_t launch_wkv_mix(const WkvMix& a, cudaStream_t s) {
    wkv_mix_kernel<<<(unsigned)(a.batch * a.q_rows), 256, 0, s>>>(a);
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
    if (a.dim <= 32) return scan_launch<1>(a, s);
    if (a.dim <= 64) return scan_launch<2>(a, s);
    if (a.dim <= 128) return scan_launch<4>(a, s);
    return scan_launch<8>(a, s);
}

}  // namespace bt
