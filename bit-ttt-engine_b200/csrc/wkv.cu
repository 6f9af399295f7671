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
// one token per sequence: decays, recurrence, norm of the head's output and gate in one launch
// ---------------------------------------------------------------------------------------
// A CTA per (head, sequence); threads as key groups x value columns, 32 KEYS state rows per thread group and turn.
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
    {   // decays of the head's key channels: G threads share a channel
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
#pragma unroll
        for (int i = 0; i < G; ++i) z += part[i * CW + threadIdx.x];
        w_s[threadIdx.x] = threadIdx.x < D ? expf(-expf(z + a.w0[head * D + threadIdx.x])) : 0.0f;
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
        const float ss = warp_sum(o * o);
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
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
// A CTA owns 32 value columns of one head: eight lanes share a column, each with 4 NJ state elements in registers (key
// channels 32 j + 4 lane .. + 3).  r, k, the decays and v of a tile of tokens are staged in shared memory, the next tile's
// values wait in registers.
template <int NJ>
__global__ void __launch_bounds__(256) wkv_scan_kernel(const WkvArgs a) {
    constexpr int DP = 32 * NJ, TT = NJ <= 4 ? 16 : 8, NL = TT * DP / 256;
    __shared__ __align__(16) float r_s[TT * DP], k_s[TT * DP], w_s[TT * DP];
    __shared__ float v_s[TT * 32], bonus_s[TT];
    const int head = blockIdx.x, v0 = blockIdx.y * 32, b = blockIdx.z;
    const int D = a.dim, HD = a.heads * D, vc = min(32, D - v0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int col = warp * 4 + (lane >> 3), kg = lane & 7;
    const bool live = col < vc;
    const int p0 = a.pos[b];
    float* state = a.s + ((int64_t)b * a.heads + head) * D * D + v0 + (live ? col : 0);
    float s[4 * NJ];
#pragma unroll
    for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int k = 32 * j + 4 * kg + e;
            s[4 * j + e] = live && k < D && p0 > 0 ? state[(int64_t)k * D] : 0.0f;
        }
    const float* base = a.proj + (int64_t)b * a.q_rows * a.ld + head * D;
    const float* zb = a.z + (int64_t)b * a.q_rows * HD + head * D;
    float rr[NL], kr[NL], zr[NL], vr[TT * 32 / 256];
    auto fetch = [&](int i0) {
#pragma unroll
        for (int i = 0; i < NL; ++i) {
            const int e = threadIdx.x + i * 256, t = i0 + e / DP, c = e % DP;
            const bool ok = t < a.q_rows && c < D;
            rr[i] = ok ? base[(int64_t)t * a.ld + c] : 0.0f;
            kr[i] = ok ? base[(int64_t)t * a.ld + HD + c] : 0.0f;
            zr[i] = ok ? zb[(int64_t)t * HD + c] : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < TT * 32 / 256; ++i) {
            const int e = threadIdx.x + i * 256, t = i0 + e / 32, c = e % 32;
            vr[i] = t < a.q_rows && c < vc ? base[(int64_t)t * a.ld + 2 * HD + v0 + c] : 0.0f;
        }
    };
    fetch(0);
    for (int i0 = 0; i0 < a.q_rows; i0 += TT) {
        const int n = min(TT, a.q_rows - i0);
        __syncthreads();
#pragma unroll
        for (int i = 0; i < NL; ++i) {
            const int e = threadIdx.x + i * 256;
            r_s[e] = rr[i];
            k_s[e] = kr[i];
            w_s[e] = expf(-expf(zr[i]));
        }
#pragma unroll
        for (int i = 0; i < TT * 32 / 256; ++i) v_s[threadIdx.x + i * 256] = vr[i];
        fetch(i0 + TT);
        __syncthreads();
        for (int t = warp; t < n; t += 8) {
            float x = 0.0f;
            for (int c = lane; c < D; c += 32) x = fmaf(r_s[t * DP + c] * a.u[head * D + c], k_s[t * DP + c], x);
            x = warp_sum(x);
            if (lane == 0) bonus_s[t] = x;
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float v = v_s[t * 32 + col];
            float o0 = 0.0f, o1 = 0.0f;
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const int at = t * DP + 32 * j + 4 * kg;
                const float4 r = *reinterpret_cast<const float4*>(r_s + at), k = *reinterpret_cast<const float4*>(k_s + at), w = *reinterpret_cast<const float4*>(w_s + at);
                o0 = fmaf(r.x, s[4 * j], o0); o1 = fmaf(r.y, s[4 * j + 1], o1);
                o0 = fmaf(r.z, s[4 * j + 2], o0); o1 = fmaf(r.w, s[4 * j + 3], o1);
                s[4 * j] = fmaf(w.x, s[4 * j], k.x * v);
                s[4 * j + 1] = fmaf(w.y, s[4 * j + 1], k.y * v);
                s[4 * j + 2] = fmaf(w.z, s[4 * j + 2], k.z * v);
                s[4 * j + 3] = fmaf(w.w, s[4 * j + 3], k.w * v);
            }
            float o = o0 + o1;
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            o += __shfl_xor_sync(0xffffffffu, o, 4);
            if (live && kg == (t & 7)) a.y[((int64_t)b * a.q_rows + i0 + t) * HD + head * D + v0 + col] = fmaf(bonus_s[t], v, o);
        }
    }
    if (live)
#pragma unroll
        for (int j = 0; j < NJ; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int k = 32 * j + 4 * kg + e;
                if (k < D) state[(int64_t)k * D] = s[4 * j + e];
            }
    if (blockIdx.x == 0 && blockIdx.y == 0) {  // the token shift's state
        const int64_t last = (int64_t)b * a.q_rows + a.q_rows - 1;
        float* keep = a.shift + (int64_t)((p0 + a.q_rows - 1) & 1) * a.shift_slot + (int64_t)b * a.width;
        for (int c = threadIdx.x; c < a.width; c += 256) keep[c] = a.hn[last * a.width + c];
    }
}

template <int NJ>
cudaError_t scan_launch(const WkvArgs& a, cudaStream_t s) {
    wkv_scan_kernel<NJ><<<dim3((unsigned)a.heads, (unsigned)((a.dim + 31) / 32), (unsigned)a.batch), 256, 0, s>>>(a);
    return cudaGetLastError();
}

}  // namespace

int wkv_max_dim() { return 256; }

cudaError_t launch_wkv_mix(const WkvMix& a, cudaStream_t s) {
    wkv_mix_kernel<<<(unsigned)(a.batch * a.q_rows), 256, 0, s>>>(a);
    return cudaGetLastError();
}

cudaError_t launch_wkv_step(const WkvArgs& a, cudaStream_t s, bool pdl) {
    if (a.dim > wkv_max_dim() || a.rank > kMaxRank || a.q_rows != 1) return cudaErrorInvalidValue;
    const dim3 grid((unsigned)a.heads, (unsigned)a.batch), block(kStepThreads);
    if (a.dim <= 32) return launch_pdl(wkv_step_kernel<32>, grid, block, 0, s, pdl, a);
    if (a.dim <= 64) return launch_pdl(wkv_step_kernel<64>, grid, block, 0, s, pdl, a);
    if (a.dim <= 128) return launch_pdl(wkv_step_kernel<128>, grid, block, 0, s, pdl, a);
    return launch_pdl(wkv_step_kernel<256>, grid, block, 0, s, pdl, a);
}

cudaError_t launch_wkv_prefill(const WkvArgs& a, bool bf16, cudaStream_t s) {
    (void)bf16;
    if (a.dim <= 32) return scan_launch<1>(a, s);
    if (a.dim <= 64) return scan_launch<2>(a, s);
    if (a.dim <= 128) return scan_launch<4>(a, s);
    return a.dim <= wkv_max_dim() ? scan_launch<8>(a, s) : cudaErrorInvalidValue;
}

}  // namespace bt
