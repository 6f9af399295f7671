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

// A thread per 8 channels (of one block of channels) and token.
__global__ void __launch_bounds__(256) rglru_conv_kernel(const RgluArgs a) {
    const int kb = a.channels / a.blocks, kp = dense_kpad(kb), per = kp / 8;
    const int64_t total = (int64_t)a.batch * a.q_rows * a.blocks * per;
    for (int64_t e = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (int64_t)gridDim.x * blockDim.x) {
        const int c0 = (int)(e % per) * 8, blk = (int)(e / per % a.blocks);
        const int64_t r = e / per / a.blocks;
        const int b = (int)(r / a.q_rows), i = (int)(r % a.q_rows), p = a.pos[b] + i;
        const int ch0 = blk * kb + c0;
        const float* x = a.proj + r * a.ld + a.channels + ch0;
        const float* ring = a.ring + (int64_t)b * a.taps * a.channels + ch0;
        const int n = min(8, kb - c0);
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = j < n ? a.conv_b[ch0 + j] : 0.0f;
        for (int t = 0; t < a.taps; ++t) {
            const int back = a.taps - 1 - t;
            if (back > p) continue;  // zeros before the start
            const float* src = back <= i ? x - (int64_t)back * a.ld : ring + (int64_t)((p - back) % a.taps) * a.channels;
#pragma unroll
            for (int j = 0; j < 8; ++j)
                if (j < n) v[j] = fmaf(a.conv_w[(int64_t)(ch0 + j) * a.taps + t], src[j], v[j]);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (j < n) a.u[r * a.channels + ch0 + j] = v[j];
        if (a.u_tiles) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                hi[j] = ptx::pack2(v[2 * j], v[2 * j + 1]);
                lo[j] = ptx::pack2(v[2 * j] - __uint_as_float(hi[j] << 16), v[2 * j + 1] - __uint_as_float(hi[j] & 0xffff0000u));
            }
            *reinterpret_cast<uint4*>(a.u_tiles + dense_off(r, blk * 2 * kp + c0, a.m_pad)) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(a.u_tiles + dense_off(r, (blk * 2 + 1) * kp + c0, a.m_pad)) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
    }
}

// A CTA owns 32 channels of one sequence; a tile of 256 tokens is cut over 32 warps, 8 tokens each.  Every warp folds its
// tokens into (product of a, S from zero), a scan over the 32 pairs per channel gives each warp its incoming state.
constexpr int kWarps = 32, kPer = 8, kTile = kWarps * kPer;

__global__ void __launch_bounds__(kWarps * 32, 1) rglru_scan_kernel(const RgluArgs a, const ActOut out) {
    __shared__ float pa[32][33], ps[32][33];       // [warp][channel]
    __shared__ float carry[32];
    __shared__ __align__(16) uint8_t stage[kWarps][512];  // 8 tokens x 32 channels of bf16: [8 channels][token][16 bytes]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int b = blockIdx.y, ch = blockIdx.x * 32 + lane, C = a.channels;
    const bool live = ch < C;
    const int p0 = a.pos[b];
    if (warp == 0) carry[lane] = live && p0 > 0 ? a.state[(int64_t)b * C + ch] : 0.0f;
    const float lam = live ? -8.0f * softplus_f(a.lam[ch]) : 0.0f;
    const int64_t row0 = (int64_t)b * a.q_rows;
    for (int t0 = 0; t0 < a.q_rows; t0 += kTile) {
        const int i0 = t0 + warp * kPer;
        float2 g[kPer];
        float u[kPer], y[kPer];
#pragma unroll
        for (int j = 0; j < kPer; ++j) {
            const int64_t r = row0 + i0 + j;
            const bool ok = live && i0 + j < a.q_rows;
            g[j] = ok ? *reinterpret_cast<const float2*>(a.gates + (r * C + ch) * 2) : make_float2(0.f, 0.f);
            u[j] = ok ? a.u[r * C + ch] : 0.0f;
            y[j] = ok ? a.proj[r * a.ld + ch] : 0.0f;
        }
        float av[kPer], xv[kPer], fa = 1.0f, fs = 0.0f;
#pragma unroll
        for (int j = 0; j < kPer; ++j) {
            const float la = lam * sigmoid_f(g[j].x);
            const bool ok = live && i0 + j < a.q_rows;
            av[j] = ok ? expf(la) : 1.0f;  // beyond the end the state passes through
            xv[j] = ok ? sqrtf(-expm1f(2.0f * la)) * sigmoid_f(g[j].y) * u[j] : 0.0f;
            fs = fmaf(av[j], fs, xv[j]);
            fa *= av[j];
        }
        pa[warp][lane] = fa;
        ps[warp][lane] = fs;
        __syncthreads();
        {   // warp = channel, lane = the tokens' warp
            float A = pa[lane][warp], S = ps[lane][warp];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float A0 = __shfl_up_sync(0xffffffffu, A, o), S0 = __shfl_up_sync(0xffffffffu, S, o);
                if (lane >= o) { S = fmaf(A, S0, S); A *= A0; }
            }
            const float in = carry[warp];
            const float after = fmaf(A, in, S);
            float before = __shfl_up_sync(0xffffffffu, after, 1);
            if (lane == 0) before = in;
            ps[lane][warp] = before;
            __syncwarp();
            if (lane == 31) carry[warp] = after;
        }
        __syncthreads();
        float s = ps[warp][lane];
#pragma unroll
        for (int j = 0; j < kPer; ++j) {
            s = fmaf(av[j], s, xv[j]);
            y[j] = s * gelu_tanh_f(y[j]);
        }
        if (out.tiles) {
#pragma unroll
            for (int j = 0; j < kPer; ++j)
                *reinterpret_cast<__nv_bfloat16*>(stage[warp] + (lane >> 3) * 128 + j * 16 + (lane & 7) * 2) = __float2bfloat16_rn(y[j]);
            __syncwarp();
            const int j = lane & 7, c0 = blockIdx.x * 32 + (lane >> 3) * 8;
            if (i0 + j < a.q_rows && c0 < dense_kpad(C))
                *reinterpret_cast<uint4*>(out.tiles + dense_off(row0 + i0 + j, c0, out.m_pad)) = *reinterpret_cast<const uint4*>(stage[warp] + lane * 16);
            __syncwarp();
        } else if (live) {
#pragma unroll
            for (int j = 0; j < kPer; ++j)
                if (i0 + j < a.q_rows) out.rows[(row0 + i0 + j) * out.ld + ch] = y[j];
        }
        __syncthreads();
    }
    if (warp == 0 && live) {
        a.state[(int64_t)b * C + ch] = carry[lane];
        // the convolution's last inputs stay behind for the next tokens
        for (int i = max(0, a.q_rows - a.taps); i < a.q_rows; ++i)
            a.ring[((int64_t)b * a.taps + (p0 + i) % a.taps) * C + ch] = a.proj[(row0 + i) * a.ld + C + ch];
    }
}

}  // namespace

cudaError_t launch_rglru_conv(const RgluArgs& a, cudaStream_t s) {
    const int64_t total = (int64_t)a.batch * a.q_rows * a.blocks * (dense_kpad(a.channels / a.blocks) / 8);
    rglru_conv_kernel<<<(unsigned)((total + 255) / 256 < 9472 ? (total + 255) / 256 : 9472), 256, 0, s>>>(a);
    return cudaGetLastError();
}

cudaError_t launch_rglru_scan(const RgluArgs& a, const ActOut& out, cudaStream_t s) {
    rglru_scan_kernel<<<dim3((unsigned)((a.channels + 31) / 32), (unsigned)a.batch), kWarps * 32, 0, s>>>(a, out);
    return cudaGetLastError();
}

}  // namespace bt
