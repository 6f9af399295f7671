// Gated linear recurrence per channel over many tokens: S <- a S + sqrt(1 - a^2) i u with a = exp(-8 r softplus(lam)),
// output S * gelu_tanh(y); u a causal convolution.  One token per sequence runs inside the gates' product (dense.cu).
// Everything here is f32.
#include "bt_dense.cuh"
#include "bt_ptx.cuh"

namespace bt {

namespace {

__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float gelu_tanh_f(float v) { return 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v))); }

// Eight tokens x 32 values of bf16, one value per lane and token, as 16-byte pieces of the tiled layout: [8 values][token][16 bytes]
__device__ __forceinline__ void stage8(uint8_t* st, int lane, int j, __nv_bfloat16 v) {
    *reinterpret_cast<__nv_bfloat16*>(st + (lane >> 3) * 128 + j * 16 + (lane & 7) * 2) = v;
}

// ---------------------------------------------------------------------------------------
// convolution: a warp per 32 columns of a block (padded to a multiple of 64) and 8 tokens
// ---------------------------------------------------------------------------------------
constexpr int kConvTokens = 8;
template <int TAPS>  // 4: up to four taps, the inputs in registers; 0: any number
__global__ void __launch_bounds__(256) rglru_conv_kernel(const RgluArgs a) {
    __shared__ __align__(16) uint8_t st[8][512];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kb = a.channels / a.blocks, kp = dense_kpad(kb);
    const int cg = blockIdx.x * 8 + warp;  // group of 32 padded columns
    if (cg * 32 >= a.blocks * kp) return;
    const int blk = cg * 32 / kp, c = cg * 32 - blk * kp + lane, ch = blk * kb + c;
    const bool live = c < kb;
    const int b = blockIdx.z, i0 = blockIdx.y * kConvTokens, p0 = a.pos[b];
    const int n = min(kConvTokens, a.q_rows - i0);
    const int64_t row0 = (int64_t)b * a.q_rows;
    const float* x = a.proj + row0 * a.ld + a.channels + (live ? ch : 0);
    const float* ring = a.ring + (int64_t)b * a.taps * a.channels + (live ? ch : 0);
    float v[kConvTokens];
    if (live) {
        const float bias = a.conv_b[ch];
        if (TAPS == 4) {
            float w[4], in[kConvTokens + 3];
#pragma unroll
            for (int j = 0; j < 4; ++j) w[j] = j < a.taps ? a.conv_w[(int64_t)ch * a.taps + a.taps - 1 - j] : 0.0f;  // by distance back
#pragma unroll
            for (int j = 0; j < kConvTokens + 3; ++j) {
                const int i = i0 + j - 3, p = p0 + i;
                in[j] = 0.0f;
                if (i >= 0) { if (j - 3 < n) in[j] = x[(int64_t)i * a.ld]; }
                else if (p >= 0 && -i < a.taps) in[j] = ring[(int64_t)(p % a.taps) * a.channels];
            }
#pragma unroll
            for (int j = 0; j < kConvTokens; ++j) {
                v[j] = bias;
#pragma unroll
                for (int k = 3; k >= 0; --k) v[j] = fmaf(w[k], in[j + 3 - k], v[j]);
            }
        } else {
#pragma unroll 1
            for (int j = 0; j < n; ++j) {
                float s = bias;
                for (int t = 0; t < a.taps; ++t) {
                    const int back = a.taps - 1 - t, i = i0 + j - back, p = p0 + i;
                    if (p < 0) continue;  // zeros before the start
                    s = fmaf(a.conv_w[(int64_t)ch * a.taps + t], i >= 0 ? x[(int64_t)i * a.ld] : ring[(int64_t)(p % a.taps) * a.channels], s);
                }
#pragma unroll
                for (int q = 0; q < kConvTokens; ++q)
                    if (q == j) v[q] = s;
            }
        }
#pragma unroll
        for (int j = 0; j < kConvTokens; ++j)
            if (j < n) a.u[(row0 + i0 + j) * a.channels + ch] = v[j];
    }
    if (!a.u_tiles) return;
    float lo[kConvTokens];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
#pragma unroll
        for (int j = 0; j < kConvTokens; ++j) {
            const float f = half ? lo[j] : (live && j < n ? v[j] : 0.0f);
            const __nv_bfloat16 q = __float2bfloat16_rn(f);
            if (!half) lo[j] = f - __bfloat162float(q);
            stage8(st[warp], lane, j, q);
        }
        __syncwarp();
        if ((lane & 7) < n)
            *reinterpret_cast<uint4*>(a.u_tiles + dense_off(row0 + i0 + (lane & 7), (blk * 2 + half) * kp + cg * 32 - blk * kp + (lane >> 3) * 8, a.m_pad)) =
                *reinterpret_cast<const uint4*>(st[warp] + lane * 16);
        __syncwarp();
    }
}

// decay and input of one token: a = exp(la), sqrt(1 - a^2) i u, la = lam8 * r
__device__ __forceinline__ void gate_inputs(float zr, float zi, float u, float lam8, float& av, float& xv) {
    const float e = expm1f(lam8 * sigmoid_f(zr));     // a - 1
    av = 1.0f + e;
    xv = sqrtf(-e * (2.0f + e)) * sigmoid_f(zi) * u;  // 1 - a^2 = -(a - 1)(a + 1)
}

// ---------------------------------------------------------------------------------------
// recurrence over many tokens
// ---------------------------------------------------------------------------------------
// A CTA owns CH channels of one sequence; a tile of tokens is cut into 512 / CH pieces of 8.  Every thread folds its piece into
// (product of a, S from zero), a scan over the pieces of a channel gives each its incoming state.  The next tile's values are
// requested before the scan.
constexpr int kScanThreads = 512, kPer = 8;

template <int CH>  // 16 or 32
__global__ void __launch_bounds__(kScanThreads, 1) rglru_scan_kernel(const RgluArgs a, const ActOut out) {
    constexpr int NS = kScanThreads / CH, TW = 32 / CH, TT = NS * kPer;  // pieces, pieces per warp, tokens per tile
    __shared__ float pa[NS][CH + 1], ps[NS][CH + 1];
    __shared__ float carry[CH];
    __shared__ __align__(16) uint8_t stage[kScanThreads / 32][TW][CH * 16];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = lane % CH, seg = warp * TW + lane / CH;
    const int b = blockIdx.y, ch = blockIdx.x * CH + c, C = a.channels;
    const bool live = ch < C;
    const int p0 = a.pos[b];
    if (threadIdx.x < CH) carry[threadIdx.x] = blockIdx.x * CH + threadIdx.x < C && p0 > 0 ? a.state[(int64_t)b * C + blockIdx.x * CH + threadIdx.x] : 0.0f;
    const float lam8 = live ? -8.0f * softplus_f(a.lam[ch]) : 0.0f;
    const int64_t row0 = (int64_t)b * a.q_rows;
    float2 g[kPer];
    float u[kPer], y[kPer];
    auto fetch = [&](int i0) {
#pragma unroll
        for (int j = 0; j < kPer; ++j) {
            const int64_t r = row0 + i0 + j;
            const bool ok = live && i0 + j < a.q_rows;
            g[j] = ok ? *reinterpret_cast<const float2*>(a.gates + (r * C + ch) * 2) : make_float2(0.f, 0.f);
            u[j] = ok ? a.u[r * C + ch] : 0.0f;
            y[j] = ok ? a.proj[r * a.ld + ch] : 0.0f;
        }
    };
    fetch(seg * kPer);
    for (int t0 = 0; t0 < a.q_rows; t0 += TT) {
        const int i0 = t0 + seg * kPer;
        float av[kPer], xv[kPer], yv[kPer], fa = 1.0f, fs = 0.0f;
#pragma unroll
        for (int j = 0; j < kPer; ++j) {
            const bool ok = live && i0 + j < a.q_rows;
            gate_inputs(g[j].x, g[j].y, u[j], lam8, av[j], xv[j]);
            if (!ok) { av[j] = 1.0f; xv[j] = 0.0f; }  // beyond the end the state passes through
            yv[j] = y[j];
            fs = fmaf(av[j], fs, xv[j]);
            fa *= av[j];
        }
        fetch(i0 + TT);
        pa[seg][c] = fa;
        ps[seg][c] = fs;
        __syncthreads();
        {   // threads as channel x piece
            const int sc = threadIdx.x / NS, sg = threadIdx.x % NS;
            float A = pa[sg][sc], S = ps[sg][sc];
#pragma unroll
            for (int o = 1; o < NS; o <<= 1) {
                const float A0 = __shfl_up_sync(0xffffffffu, A, o, NS), S0 = __shfl_up_sync(0xffffffffu, S, o, NS);
                if (sg >= o) { S = fmaf(A, S0, S); A *= A0; }
            }
            const float in = carry[sc];
            const float after = fmaf(A, in, S);
            float before = __shfl_up_sync(0xffffffffu, after, 1, NS);
            if (sg == 0) before = in;
            ps[sg][sc] = before;
            __syncwarp();
            if (sg == NS - 1) carry[sc] = after;
        }
        __syncthreads();
        float s = ps[seg][c];
#pragma unroll
        for (int j = 0; j < kPer; ++j) {
            s = fmaf(av[j], s, xv[j]);
            yv[j] = s * gelu_tanh_f(yv[j]);
        }
        if (out.tiles) {
            uint8_t* st = stage[warp][lane / CH];
#pragma unroll
            for (int j = 0; j < kPer; ++j) stage8(st, c, j, __float2bfloat16_rn(yv[j]));
            __syncwarp();
            const int j = c & 7, c0 = blockIdx.x * CH + (c >> 3) * 8;
            if (i0 + j < a.q_rows && c0 < dense_kpad(C))
                *reinterpret_cast<uint4*>(out.tiles + dense_off(row0 + i0 + j, c0, out.m_pad)) = *reinterpret_cast<const uint4*>(st + c * 16);
            __syncwarp();
        } else if (live) {
#pragma unroll
            for (int j = 0; j < kPer; ++j)
                if (i0 + j < a.q_rows) out.rows[(row0 + i0 + j) * out.ld + ch] = yv[j];
        }
    }
    __syncthreads();
    if (threadIdx.x < CH && live) {
        a.state[(int64_t)b * C + ch] = carry[c];
        // the convolution's last inputs stay behind for the next tokens
        for (int i = max(0, a.q_rows - a.taps); i < a.q_rows; ++i)
            a.ring[((int64_t)b * a.taps + (p0 + i) % a.taps) * C + ch] = a.proj[(row0 + i) * a.ld + C + ch];
    }
}

// one token per sequence, gates and convolution done: a thread per channel and sequence
__global__ void __launch_bounds__(128) rglru_one_kernel(const RgluArgs a, const ActOut out) {
    const int ch = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y, C = a.channels;
    if (ch >= C) return;
    const int p = a.pos[b];
    const float2 g = *reinterpret_cast<const float2*>(a.gates + ((int64_t)b * C + ch) * 2);
    float av, xv;
    gate_inputs(g.x, g.y, a.u[(int64_t)b * C + ch], -8.0f * softplus_f(a.lam[ch]), av, xv);
    float* st = a.state + (int64_t)b * C + ch;
    const float s = fmaf(av, p > 0 ? *st : 0.0f, xv);
    *st = s;
    const float y = s * gelu_tanh_f(a.proj[b * a.ld + ch]);
    if (out.tiles) *reinterpret_cast<__nv_bfloat16*>(out.tiles + dense_off(b, ch, out.m_pad)) = __float2bfloat16_rn(y);
    else out.rows[b * out.ld + ch] = y;
    a.ring[((int64_t)b * a.taps + p % a.taps) * C + ch] = a.proj[b * a.ld + C + ch];
}

}  // namespace

cudaError_t launch_rglru_conv(const RgluArgs& a, cudaStream_t s) {
    const int groups = a.blocks * dense_kpad(a.channels / a.blocks) / 32;
    const dim3 grid((unsigned)((groups + 7) / 8), (unsigned)((a.q_rows + kConvTokens - 1) / kConvTokens), (unsigned)a.batch);
    if (a.taps <= 4) rglru_conv_kernel<4><<<grid, 256, 0, s>>>(a);
    else rglru_conv_kernel<0><<<grid, 256, 0, s>>>(a);
    return cudaGetLastError();
}

cudaError_t launch_rglru_scan(const RgluArgs& a, const ActOut& out, cudaStream_t s) {
    if (a.q_rows == 1)
        rglru_one_kernel<<<dim3((unsigned)((a.channels + 127) / 128), (unsigned)a.batch), 128, 0, s>>>(a, out);
    else if ((int64_t)a.channels * a.batch < 4096)
        rglru_scan_kernel<16><<<dim3((unsigned)((a.channels + 15) / 16), (unsigned)a.batch), kScanThreads, 0, s>>>(a, out);
    else
        rglru_scan_kernel<32><<<dim3((unsigned)((a.channels + 31) / 32), (unsigned)a.batch), kScanThreads, 0, s>>>(a, out);
    return cudaGetLastError();
}

}  // namespace bt
