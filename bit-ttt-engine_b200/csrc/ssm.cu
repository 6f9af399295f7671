// State-space recurrence with a scalar decay per head (the Mamba-2 form):
//   S <- exp(-exp(A_log) dt) S + dt B x^T,   y = S^T C + D x,
// x, B and C after a causal convolution per channel and silu, dt = softplus(dt + dt_bias).  The result leaves gated:
// y * silu(z).  State, decays, step sizes and every sum of the recurrence are f32.
#include "bt_dense.cuh"
#include "bt_ptx.cuh"

namespace bt {

namespace {

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }

// Input of the convolution at position p - back, for a token at row r (i-th new token, position p): from the projection
// rows while it is one of the new tokens, else from the ring of earlier inputs; zero before the start.
__device__ __forceinline__ float conv_tap(const SsmArgs& a, const float* x_row, int64_t ld, const float* ring, int channels,
                                          int ch, int i, int p, int back) {
    if (back <= i) return x_row[ch - (int64_t)back * ld];
    const int q = p - back;
    return q >= 0 ? ring[(int64_t)(q % a.taps) * channels + ch] : 0.0f;
}
__device__ __forceinline__ float conv_silu(const SsmArgs& a, const float* x_row, const float* ring, int channels, int ch,
                                           int i, int p) {
    float v = a.conv_b[ch];
    const float* w = a.conv_w + (int64_t)ch * a.taps;
    for (int j = 0; j < a.taps; ++j) v = fmaf(w[j], conv_tap(a, x_row, a.ld, ring, channels, ch, i, p, a.taps - 1 - j), v);
    return silu_f(v);
}

// ---------------------------------------------------------------------------------------
// convolution of the new tokens (prefill)
// ---------------------------------------------------------------------------------------
constexpr int kConvTokens = 8;
__global__ void __launch_bounds__(256) ssm_conv_kernel(const SsmArgs a, int channels) {
    const int ch = blockIdx.x * blockDim.x + threadIdx.x;
    if (ch >= channels) return;
    const int b = blockIdx.z, i0 = blockIdx.y * kConvTokens, i1 = min(i0 + kConvTokens, a.q_rows);
    const int inner = a.heads * a.vdim, p0 = a.pos[b];
    const float* ring = a.ring + (int64_t)b * a.taps * channels;
    for (int i = i0; i < i1; ++i) {
        const int64_t r = (int64_t)b * a.q_rows + i;
        a.conv_out[r * channels + ch] = conv_silu(a, a.proj + r * a.ld + inner, ring, channels, ch, i, p0 + i);
    }
}

// ---------------------------------------------------------------------------------------
// recurrence, token by token
// ---------------------------------------------------------------------------------------
// A CTA owns up to 64 columns of one head's state (vdim x state, columns = vdim): four lanes share a column, each with
// 4 NJ of its state elements in registers (elements 16 j + 4 lane .. + 3).  B, C, x and the step sizes of a tile of
// tokens are staged in shared memory.  STEP: one token, the convolution inside the kernel.
constexpr int kSsmTokens = 16;

template <int NJ, bool STEP>
__global__ void __launch_bounds__(256) ssm_scan_kernel(const SsmArgs a, int channels) {
    constexpr int NP = 16 * NJ;
    extern __shared__ __align__(16) float sm[];
    constexpr int TT = STEP ? 1 : kSsmTokens;
    float* b_s = sm;                    // [TT][NP]
    float* c_s = b_s + TT * NP;         // [TT][NP]
    float* x_s = c_s + TT * NP;         // [TT][64]
    float* z_s = x_s + TT * 64;         // [TT][64] silu(z)
    float* dt_s = z_s + TT * 64;        // [TT] step, [TT] decay
    float* dec_s = dt_s + TT;
    const int head = blockIdx.x, v0 = blockIdx.y * 64, b = blockIdx.z;
    const int vc = min(64, a.vdim - v0), N = a.state, inner = a.heads * a.vdim;
    const int g = head / (a.heads / a.groups);
    const int col = threadIdx.x >> 2, ln = threadIdx.x & 3;
    const bool live = col < vc;
    float* state = a.s + (((int64_t)b * a.heads + head) * a.vdim + v0 + (live ? col : 0)) * a.state_pad;
    const int xch = head * a.vdim + v0, bch = inner + g * N, cch = inner + (a.groups + g) * N;
    float* ring = a.ring + (int64_t)b * a.taps * channels;
    const float a_neg = -expf(a.a_log[head]), bias = a.dt_bias[head], dskip = a.d[head];
    if (STEP) ptx::pdl_wait();
    if (STEP) ptx::pdl_launch_dependents();
    const int p0 = a.pos[b];
    float4 s[NJ];
#pragma unroll
    for (int j = 0; j < NJ; ++j)
        s[j] = live && p0 > 0 ? *reinterpret_cast<const float4*>(state + 16 * j + 4 * ln) : make_float4(0.f, 0.f, 0.f, 0.f);

    for (int i0 = 0; i0 < a.q_rows; i0 += TT) {
        const int n = min(TT, a.q_rows - i0);
        const int64_t r0 = (int64_t)b * a.q_rows + i0;
        __syncthreads();
        for (int e = threadIdx.x; e < n * NP; e += 256) {
            const int t = e / NP, c = e - t * NP;
            float vb = 0.0f, vcx = 0.0f;
            if (c < N) {
                if (STEP) {
                    const float* xr = a.proj + r0 * a.ld + inner;
                    vb = conv_silu(a, xr, ring, channels, bch + c, 0, p0);
                    vcx = conv_silu(a, xr, ring, channels, cch + c, 0, p0);
                } else {
                    vb = a.conv_out[(r0 + t) * channels + bch + c];
                    vcx = a.conv_out[(r0 + t) * channels + cch + c];
                }
            }
            b_s[e] = vb;
            c_s[e] = vcx;
        }
        for (int e = threadIdx.x; e < n * 64; e += 256) {
            const int t = e >> 6, c = e & 63;
            float vx = 0.0f, vz = 0.0f;
            if (c < vc) {
                vx = STEP ? conv_silu(a, a.proj + r0 * a.ld + inner, ring, channels, xch + c, 0, p0)
                          : a.conv_out[(r0 + t) * channels + xch + c];
                vz = silu_f(a.proj[(r0 + t) * a.ld + xch + c]);
            }
            x_s[e] = vx;
            z_s[e] = vz;
        }
        if (threadIdx.x < n) {
            const float dt = softplus_f(a.proj[(r0 + threadIdx.x) * a.ld + inner + channels + head] + bias);
            dt_s[threadIdx.x] = dt;
            dec_s[threadIdx.x] = expf(a_neg * dt);
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float dec = dec_s[t], x = x_s[t * 64 + col], dx = dt_s[t] * x;
            float y0 = 0.0f, y1 = 0.0f;
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const float4 bb = *reinterpret_cast<const float4*>(b_s + t * NP + 16 * j + 4 * ln);
                const float4 cc = *reinterpret_cast<const float4*>(c_s + t * NP + 16 * j + 4 * ln);
                s[j].x = fmaf(dec, s[j].x, dx * bb.x);
                s[j].y = fmaf(dec, s[j].y, dx * bb.y);
                s[j].z = fmaf(dec, s[j].z, dx * bb.z);
                s[j].w = fmaf(dec, s[j].w, dx * bb.w);
                y0 = fmaf(s[j].x, cc.x, y0); y1 = fmaf(s[j].y, cc.y, y1);
                y0 = fmaf(s[j].z, cc.z, y0); y1 = fmaf(s[j].w, cc.w, y1);
            }
            float y = y0 + y1;
            y += __shfl_xor_sync(0xffffffffu, y, 1);
            y += __shfl_xor_sync(0xffffffffu, y, 2);
            if (live && ln == (t & 3)) a.y[(r0 + t) * inner + xch + col] = fmaf(dskip, x, y) * z_s[t * 64 + col];
        }
    }
    if (live)
#pragma unroll
        for (int j = 0; j < NJ; ++j) *reinterpret_cast<float4*>(state + 16 * j + 4 * ln) = s[j];
    // the last inputs of the convolution: this CTA's x channels; the group's B and C channels by its first head
    const int keep = min(a.q_rows, a.taps);
    const bool owns_bc = head % (a.heads / a.groups) == 0 && blockIdx.y == 0;
    const int nch = vc + (owns_bc ? 2 * N : 0);
    for (int e = threadIdx.x; e < keep * nch; e += 256) {
        const int k = e / nch, c = e - k * nch;
        const int ch = c < vc ? xch + c : (c < vc + N ? bch + c - vc : cch + c - vc - N);
        const int i = a.q_rows - keep + k;
        ring[(int64_t)((p0 + i) % a.taps) * channels + ch] = a.proj[((int64_t)b * a.q_rows + i) * a.ld + inner + ch];
    }
}

template <int NJ, bool STEP>
cudaError_t scan_launch(const SsmArgs& a, cudaStream_t s, bool pdl) {
    constexpr int TT = STEP ? 1 : kSsmTokens;
    const int channels = a.heads * a.vdim + 2 * a.groups * a.state;
    const size_t smem = (size_t)(2 * TT * 16 * NJ + 2 * TT * 64 + 2 * TT) * sizeof(float);
    return launch_pdl(ssm_scan_kernel<NJ, STEP>, dim3((unsigned)a.heads, (unsigned)((a.vdim + 63) / 64), (unsigned)a.batch), dim3(256),
                      smem, s, pdl, a, channels);
}
template <bool STEP>
cudaError_t scan_launch_n(const SsmArgs& a, cudaStream_t s, bool pdl) {
    switch (a.state_pad) {
        case 16: return scan_launch<1, STEP>(a, s, pdl);
        case 32: return scan_launch<2, STEP>(a, s, pdl);
        case 64: return scan_launch<4, STEP>(a, s, pdl);
        case 128: return scan_launch<8, STEP>(a, s, pdl);
        case 256: return scan_launch<16, STEP>(a, s, pdl);
    }
    return cudaErrorInvalidValue;
}

}  // namespace

int ssm_state_pad(int state) {
    if (state < 1 || state > 256) return 0;
    int p = 16;
    while (p < state) p *= 2;
    return p;
}

cudaError_t launch_ssm_step(const SsmArgs& a, cudaStream_t s, bool pdl) {
    if (a.q_rows != 1) return cudaErrorInvalidValue;
    return scan_launch_n<true>(a, s, pdl);
}

cudaError_t launch_ssm_prefill(const SsmArgs& a, cudaStream_t s) {
    const int channels = a.heads * a.vdim + 2 * a.groups * a.state;
    ssm_conv_kernel<<<dim3((unsigned)((channels + 255) / 256), (unsigned)((a.q_rows + kConvTokens - 1) / kConvTokens), (unsigned)a.batch), 256, 0, s>>>(a, channels);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    return scan_launch_n<false>(a, s, false);
}

}  // namespace bt
