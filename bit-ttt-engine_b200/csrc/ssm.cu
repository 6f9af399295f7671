// State-space recurrence with a scalar decay per head (the Mamba-2 form):
//   S <- exp(-exp(A_log) dt) S + dt B x^T,   y = S^T C + D x,
// x, B and C after a causal convolution per channel and silu, dt = softplus(dt + dt_bias).  The result leaves gated:
// y * silu(z).  State, decays, step sizes and every sum of the recurrence are f32.
#include "bt_dense.cuh"
#include "bt_ptx.cuh"

namespace bt {

namespace {

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float silu_fast(float v) { return __fdividef(v, 1.0f + __expf(-v)); }  // where the result is rounded to bf16
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
// Output columns: x | B | C.  PAD: bf16, every head's x and every group's B and C padded to a multiple of 8 (zeros), so that
// each starts on a 16-byte boundary.
constexpr int kConvTokens = 8;
__host__ __device__ inline int pad8(int n) { return (n + 7) / 8 * 8; }
__host__ __device__ inline int conv_cols(const SsmArgs& a) { return a.heads * pad8(a.vdim) + 2 * a.groups * pad8(a.state); }
template <bool PAD>
__global__ void __launch_bounds__(256) ssm_conv_kernel(const SsmArgs a, int channels) {
    const int col = blockIdx.x * blockDim.x + threadIdx.x;
    const int cols = PAD ? conv_cols(a) : channels;
    if (col >= cols) return;
    int ch = col;
    if (PAD) {
        const int vp = pad8(a.vdim), np = pad8(a.state), xw = a.heads * vp;
        if (col < xw) {
            const int h = col / vp, c = col - h * vp;
            ch = c < a.vdim ? h * a.vdim + c : -1;
        } else {
            const int q = (col - xw) / np, c = (col - xw) - q * np;  // group of B, then group of C
            ch = c < a.state ? a.heads * a.vdim + q * a.state + c : -1;
        }
    }
    const int b = blockIdx.z, i0 = blockIdx.y * kConvTokens, i1 = min(i0 + kConvTokens, a.q_rows);
    const int inner = a.heads * a.vdim, p0 = a.pos[b];
    const float* ring = a.ring + (int64_t)b * a.taps * channels;
    auto put = [&](int i, float v) {
        const int64_t r = (int64_t)b * a.q_rows + i;
        if (PAD) reinterpret_cast<__nv_bfloat16*>(a.conv_out)[r * cols + col] = __float2bfloat16_rn(v);
        else a.conv_out[r * channels + ch] = v;
    };
    const float* x = a.proj + (int64_t)b * a.q_rows * a.ld + inner + ch;
    if (ch < 0) {
        for (int i = i0; i < i1; ++i) put(i, 0.0f);
    } else if (a.taps <= 4) {
        // the inputs of the block and the three before it in registers
        float w[4], v[kConvTokens + 3];
#pragma unroll
        for (int j = 0; j < 4; ++j) w[j] = j < a.taps ? a.conv_w[(int64_t)ch * a.taps + a.taps - 1 - j] : 0.0f;  // by distance back
#pragma unroll
        for (int j = 0; j < kConvTokens + 3; ++j) {
            const int i = i0 + j - 3;
            v[j] = i >= 0 && i < i1 ? x[(int64_t)i * a.ld] : 0.0f;
        }
        if (i0 == 0)
#pragma unroll
            for (int j = 0; j < 3; ++j) {
                const int q = p0 + j - 3;
                if (q >= 0 && 3 - j < a.taps) v[j] = ring[(int64_t)(q % a.taps) * channels + ch];
            }
        const float bias = a.conv_b[ch];
#pragma unroll
        for (int j = 0; j < kConvTokens; ++j)
            if (i0 + j < i1) {
                float s = bias;
#pragma unroll
                for (int k = 3; k >= 0; --k) s = fmaf(w[k], v[j + 3 - k], s);
                put(i0 + j, PAD ? silu_fast(s) : silu_f(s));
            }
    } else {
        for (int i = i0; i < i1; ++i) put(i, conv_silu(a, a.proj + ((int64_t)b * a.q_rows + i) * a.ld + inner, ring, channels, ch, i, p0 + i));
    }
}

// The last inputs of the convolution stay behind for the next tokens: a CTA keeps its x channels, the group's B and C
// channels are kept by its first head.
__device__ __forceinline__ void keep_inputs(const SsmArgs& a, float* ring, int channels, int b, int head, int v0, int vc, int p0) {
    const int N = a.state, inner = a.heads * a.vdim, g = head / (a.heads / a.groups);
    const int xch = head * a.vdim + v0, bch = inner + g * N, cch = inner + (a.groups + g) * N;
    const int keep = min(a.q_rows, a.taps);
    const bool owns_bc = head % (a.heads / a.groups) == 0 && v0 == 0;
    const int nch = vc + (owns_bc ? 2 * N : 0);
    for (int e = threadIdx.x; e < keep * nch; e += blockDim.x) {
        const int k = e / nch, c = e - k * nch;
        const int ch = c < vc ? xch + c : (c < vc + N ? bch + c - vc : cch + c - vc - N);
        const int i = a.q_rows - keep + k;
        ring[(int64_t)((p0 + i) % a.taps) * channels + ch] = a.proj[((int64_t)b * a.q_rows + i) * a.ld + inner + ch];
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
    // everything the kernel in front does not write may be requested ahead of the wait on it
    const int p0 = a.pos[b];
    float4 s[NJ];
#pragma unroll
    for (int j = 0; j < NJ; ++j)
        s[j] = live ? *reinterpret_cast<const float4*>(state + 16 * j + 4 * ln) : make_float4(0.f, 0.f, 0.f, 0.f);
    if (p0 <= 0)
#pragma unroll
        for (int j = 0; j < NJ; ++j) s[j] = make_float4(0.f, 0.f, 0.f, 0.f);

    for (int i0 = 0; i0 < a.q_rows; i0 += TT) {
        const int n = min(TT, a.q_rows - i0);
        const int64_t r0 = (int64_t)b * a.q_rows + i0;
        if (STEP) {
            // one channel per thread and turn: B, C, then x and z
            const float* xr = a.proj + r0 * a.ld + inner;
            bool waited = false;
            for (int e = threadIdx.x; e < 2 * NP + 128; e += 256) {
                const int c = e < NP ? e : (e < 2 * NP ? e - NP : (e - 2 * NP) & 63);
                const bool is_z = e >= 2 * NP + 64;
                const int ch = e < NP ? bch + c : (e < 2 * NP ? cch + c : xch + c);
                const bool used = c < (e < 2 * NP ? N : vc);
                float hist = 0.0f, wl = 0.0f;
                if (used && !is_z) {  // the taps on earlier inputs
                    hist = a.conv_b[ch];
                    wl = a.conv_w[(int64_t)ch * a.taps + a.taps - 1];
#pragma unroll 4
                    for (int back = a.taps - 1; back > 0; --back) {
                        const int q = p0 - back;
                        if (q >= 0) hist = fmaf(a.conv_w[(int64_t)ch * a.taps + a.taps - 1 - back], ring[(int64_t)(q % a.taps) * channels + ch], hist);
                    }
                }
                if (!waited) { ptx::pdl_wait(); ptx::pdl_launch_dependents(); waited = true; }
                float v = 0.0f;
                if (used) v = is_z ? silu_f(xr[ch - inner]) : silu_f(fmaf(wl, xr[ch], hist));
                (e < NP ? b_s : (e < 2 * NP ? c_s : (is_z ? z_s : x_s)))[c] = v;
            }
            if (!waited) { ptx::pdl_wait(); ptx::pdl_launch_dependents(); }
        } else {
            __syncthreads();
            for (int e = threadIdx.x; e < n * NP; e += 256) {
                const int t = e / NP, c = e - t * NP;
                b_s[e] = c < N ? a.conv_out[(r0 + t) * channels + bch + c] : 0.0f;
                c_s[e] = c < N ? a.conv_out[(r0 + t) * channels + cch + c] : 0.0f;
            }
            for (int e = threadIdx.x; e < n * 64; e += 256) {
                const int t = e >> 6, c = e & 63;
                x_s[e] = c < vc ? a.conv_out[(r0 + t) * channels + xch + c] : 0.0f;
                z_s[e] = c < vc ? silu_f(a.proj[(r0 + t) * a.ld + xch + c]) : 0.0f;
            }
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
    keep_inputs(a, ring, channels, b, head, v0, vc, p0);
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

// ---------------------------------------------------------------------------------------
// recurrence, 64 tokens at a time on the tensor cores (prefill of bf16 models)
// ---------------------------------------------------------------------------------------
// With c_t the running sum of the decays' logarithms inside a chunk, the recurrence over the chunk is
//   y_t = exp(c_t) C_t S + sum_{s <= t} (C_t . B_s) exp(c_t - c_s) dt_s x_s,   S <- exp(c_last) S + sum_s B_s (exp(c_last - c_s) dt_s x_s)^T.
// B, C and x are bf16 (convolution outputs); every f32 factor enters its product as bf16 hi + lo (16 significand bits):
// the state, the weights of the pairs (t, s) and the scaled x.  The state itself, the sums and all decays stay f32.
// A CTA owns 64 columns of one head and walks the chunks in order; the next chunk is copied while one is computed.
// Sixteen warps as 4 x 4 over (16 tokens) x (16 earlier tokens | 16 columns): each makes its tile of pair weights, leaves it
// in shared memory and then its tile of outputs; the state is cut over the warps by rows of 16 elements and columns.
constexpr int kChunk = 64, kChunkThreads = 512;
template <int NP>
struct ChunkCfg {
    static constexpr int WN = NP / 16 < 8 ? NP / 16 : 8, WP = 16 / WN < 4 ? 16 / WN : 4;  // warps over state rows / columns
    static constexpr int TN = NP / 16 / WN, TP = 8 / WP;                                  // 16-row tiles, 8-column tiles per warp
    static constexpr int NS = NP * 2 + 16, PS = 64 * 2 + 16;                              // bytes per shared-memory row
    static constexpr int kIn = kChunk * (2 * NS + PS);                                    // B, C, x of a chunk
    static constexpr int kStages = NP <= 128 ? 2 : 1;
    static constexpr size_t kSmem = (size_t)kStages * kIn + 2 * NP * PS + 4 * kChunk * PS + 3 * kChunk * 4;
};

template <int NP>
__global__ void __launch_bounds__(kChunkThreads, 1) ssm_chunk_kernel(const SsmArgs a, int channels) {
    using Cfg = ChunkCfg<NP>;
    constexpr int NS = Cfg::NS, PS = Cfg::PS, TN = Cfg::TN, TP = Cfg::TP;
    extern __shared__ __align__(16) uint8_t csm[];
    uint8_t* s_hi = csm + Cfg::kStages * Cfg::kIn;   // state [NP][64] hi, lo
    uint8_t* s_lo = s_hi + NP * PS;
    uint8_t* w_hi = s_lo + NP * PS;                  // scaled x [64][64] hi, lo
    uint8_t* w_lo = w_hi + kChunk * PS;
    uint8_t* m_hi = w_lo + kChunk * PS;              // pair weights [64][64] hi, lo
    uint8_t* m_lo = m_hi + kChunk * PS;
    float* dt_s = reinterpret_cast<float*>(m_lo + kChunk * PS);
    float* cum_s = dt_s + kChunk;
    float* wt_s = cum_s + kChunk;                    // exp(c_last - c_t) dt_t
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.x, v0 = blockIdx.y * 64, b = blockIdx.z;
    const int vc = min(64, a.vdim - v0), inner = a.heads * a.vdim, g = head / (a.heads / a.groups);
    const int vp = pad8(a.vdim), np = pad8(a.state), cols = conv_cols(a);
    const __nv_bfloat16* in = reinterpret_cast<const __nv_bfloat16*>(a.conv_out) + (int64_t)b * a.q_rows * cols;
    const int xcol = head * vp + v0, bcol = a.heads * vp + g * np, ccol = bcol + a.groups * np;
    const int xlive = min(64, vp - v0);
    const float a_neg = -expf(a.a_log[head]), bias = a.dt_bias[head], dskip = a.d[head];
    const int p0 = a.pos[b];
    float* ring = a.ring + (int64_t)b * a.taps * channels;
    float* state = a.s + (((int64_t)b * a.heads + head) * a.vdim + v0) * a.state_pad;
    const int wn = warp % Cfg::WN, wp = warp / Cfg::WN;
    const bool s_live = wp < Cfg::WP;
    const int tt = warp >> 2, qq = warp & 3;         // tokens 16 tt ..; earlier tokens / columns 16 qq ..

    float st[TN][TP][4];  // (n = g / g + 8 of the tile, p = 2 t, 2 t + 1)
#pragma unroll
    for (int i = 0; i < TN; ++i)
#pragma unroll
        for (int k = 0; k < TP; ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int n = (wn * TN + i) * 16 + (lane >> 2) + (e >> 1) * 8, p = (wp * TP + k) * 8 + (lane & 3) * 2 + (e & 1);
                st[i][k][e] = s_live && p < vc && p0 > 0 ? state[(int64_t)p * a.state_pad + n] : 0.0f;
            }

    auto load = [&](int t0, int buf) {
        const uint32_t dst = ptx::smem_u32(csm) + buf * Cfg::kIn;
        constexpr int NQ = NP / 8;
        for (int e = threadIdx.x; e < kChunk * (2 * NQ + 8); e += kChunkThreads) {
            const int t = e / (2 * NQ + 8), q = e - t * (2 * NQ + 8);
            const __nv_bfloat16* row = in + (int64_t)(t0 + t) * cols;
            const bool tok = t0 + t < a.q_rows;
            if (q < NQ) {
                const bool live = tok && q * 8 < np;
                ptx::cp16(dst + t * NS + q * 16, live ? row + bcol + q * 8 : in, live);
            } else if (q < 2 * NQ) {
                const bool live = tok && (q - NQ) * 8 < np;
                ptx::cp16(dst + kChunk * NS + t * NS + (q - NQ) * 16, live ? row + ccol + (q - NQ) * 8 : in, live);
            } else {
                const bool live = tok && (q - 2 * NQ) * 8 < xlive;
                ptx::cp16(dst + 2 * kChunk * NS + t * PS + (q - 2 * NQ) * 16, live ? row + xcol + (q - 2 * NQ) * 8 : in, live);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto raw_dt = [&](int t0) {  // threads 0-63: this chunk's step-size projections
        const int t = t0 + (int)threadIdx.x;
        return threadIdx.x < kChunk && t < a.q_rows ? a.proj[((int64_t)b * a.q_rows + t) * a.ld + inner + channels + head] : 0.0f;
    };
    load(0, 0);
    float dt_raw = raw_dt(0);

    int buf = 0;
    for (int t0 = 0; t0 < a.q_rows; t0 += kChunk) {
        const int n = min(kChunk, a.q_rows - t0);
        const int ta = tt * 16 + (lane >> 2), tb = ta + 8;  // this lane's tokens
        // ---- step sizes and running decay; the state as hi | lo for the products; the gates are requested ----
        if (threadIdx.x < kChunk) dt_s[threadIdx.x] = (int)threadIdx.x < n ? softplus_f(dt_raw + bias) : 0.0f;
        dt_raw = raw_dt(t0 + kChunk);
        float z[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = (e >> 1) ? tb : ta, c = qq * 16 + i * 8 + (lane & 3) * 2 + (e & 1);
                z[i][e] = t < n && c < vc ? a.proj[((int64_t)b * a.q_rows + t0 + t) * a.ld + head * a.vdim + v0 + c] : 0.0f;
            }
        if (s_live)
#pragma unroll
            for (int i = 0; i < TN; ++i)
#pragma unroll
                for (int k = 0; k < TP; ++k)
#pragma unroll
                    for (int e = 0; e < 4; e += 2) {
                        const int o = ((wn * TN + i) * 16 + (lane >> 2) + (e >> 1) * 8) * PS + ((wp * TP + k) * 8 + (lane & 3) * 2) * 2;
                        const uint32_t hi = ptx::pack2(st[i][k][e], st[i][k][e + 1]);
                        *reinterpret_cast<uint32_t*>(s_hi + o) = hi;
                        *reinterpret_cast<uint32_t*>(s_lo + o) = ptx::pack2(st[i][k][e] - __uint_as_float(hi << 16), st[i][k][e + 1] - __uint_as_float(hi & 0xffff0000u));
                    }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (Cfg::kStages == 2 && t0 + kChunk < a.q_rows) load(t0 + kChunk, buf ^ 1);
        uint8_t* bt = csm + buf * Cfg::kIn;
        uint8_t* xt = bt + 2 * kChunk * NS;
        const uint32_t b_sm = ptx::smem_u32(bt), c_sm = b_sm + kChunk * NS, x_sm = b_sm + 2 * kChunk * NS;
        // ---- running sums of the decays' logarithms, while the other warps multiply ----
        if (warp == 0) {
            const float c0 = a_neg * dt_s[2 * lane], c1 = a_neg * dt_s[2 * lane + 1];
            float sum = c0 + c1;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += up;
            }
            const float last = __shfl_sync(0xffffffffu, sum, 31);
            const float before = sum - (c0 + c1);
            cum_s[2 * lane] = before + c0;
            cum_s[2 * lane + 1] = sum;
            wt_s[2 * lane] = expf(last - (before + c0)) * dt_s[2 * lane];
            wt_s[2 * lane + 1] = expf(last - sum) * dt_s[2 * lane + 1];
        }
        // ---- C S (16 tokens x 16 columns) and C B^T (16 x 16 pairs) ----
        float y[2][4] = {}, gm[2][4] = {};
        const bool live = tt * 16 < n, pairs = live && qq <= tt;
        if (live) {
            const uint32_t c_addr = c_sm + (tt * 16 + (lane & 15)) * NS + (lane >> 4) * 16;
            const uint32_t b_addr = b_sm + (qq * 16 + (lane & 7) + ((lane >> 4) << 3)) * NS + ((lane >> 3) & 1) * 16;
            const uint32_t s_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * PS + (qq * 16 + (lane >> 4) * 8) * 2;
            const uint32_t sh = ptx::smem_u32(s_hi) + s_off, sl = ptx::smem_u32(s_lo) + s_off;
#pragma unroll
            for (int kk = 0; kk < NP / 16; ++kk) {
                uint32_t ca[4], f[4];
                ptx::ldsm4(ca, c_addr + kk * 32);
                ptx::ldsm4t(f, sh + kk * 16 * PS);
                ptx::mma_bf16(y[0], ca, f[0], f[1]);
                ptx::mma_bf16(y[1], ca, f[2], f[3]);
                ptx::ldsm4t(f, sl + kk * 16 * PS);
                ptx::mma_bf16(y[0], ca, f[0], f[1]);
                ptx::mma_bf16(y[1], ca, f[2], f[3]);
                if (pairs) {
                    ptx::ldsm4(f, b_addr + kk * 32);
                    ptx::mma_bf16(gm[0], ca, f[0], f[1]);
                    ptx::mma_bf16(gm[1], ca, f[2], f[3]);
                }
            }
        }
        __syncthreads();  // running sums
        // ---- x scaled for the state update; pair weights ----
        for (int e = threadIdx.x; e < kChunk * 32; e += kChunkThreads) {
            const int t = e >> 5, o = t * PS + (e & 31) * 4;
            const uint32_t u = *reinterpret_cast<const uint32_t*>(xt + o);
            const float w = wt_s[t], lo = __uint_as_float(u << 16) * w, hi = __uint_as_float(u & 0xffff0000u) * w;
            const uint32_t h = ptx::pack2(lo, hi);
            *reinterpret_cast<uint32_t*>(w_hi + o) = h;
            *reinterpret_cast<uint32_t*>(w_lo + o) = ptx::pack2(lo - __uint_as_float(h << 16), hi - __uint_as_float(h & 0xffff0000u));
        }
        const float cum_a = cum_s[ta], cum_b = cum_s[tb];
        if (pairs)
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int e = 0; e < 4; e += 2) {
                    const int s0 = qq * 16 + i * 8 + (lane & 3) * 2, row = e ? tb : ta;
                    const float cr = e ? cum_b : cum_a;
                    const float w0 = s0 <= row ? gm[i][e] * __expf(cr - cum_s[s0]) * dt_s[s0] : 0.0f;
                    const float w1 = s0 + 1 <= row ? gm[i][e + 1] * __expf(cr - cum_s[s0 + 1]) * dt_s[s0 + 1] : 0.0f;
                    const uint32_t hi = ptx::pack2(w0, w1);
                    *reinterpret_cast<uint32_t*>(m_hi + row * PS + s0 * 2) = hi;
                    *reinterpret_cast<uint32_t*>(m_lo + row * PS + s0 * 2) = ptx::pack2(w0 - __uint_as_float(hi << 16), w1 - __uint_as_float(hi & 0xffff0000u));
                }
        __syncthreads();
        // ---- outputs ----
        if (live) {
            const float ea = __expf(cum_a), eb = __expf(cum_b);
#pragma unroll
            for (int i = 0; i < 2; ++i) { y[i][0] *= ea; y[i][1] *= ea; y[i][2] *= eb; y[i][3] *= eb; }
            const uint32_t m_off = (tt * 16 + (lane & 15)) * PS + (lane >> 4) * 16;
            const uint32_t mh = ptx::smem_u32(m_hi) + m_off, ml = ptx::smem_u32(m_lo) + m_off;
            const uint32_t x_addr = x_sm + ((lane & 7) + ((lane >> 3) & 1) * 8) * PS + (qq * 16 + (lane >> 4) * 8) * 2;
#pragma unroll
            for (int s2 = 0; s2 < 4; ++s2)
                if (s2 <= tt) {
                    uint32_t hi[4], lo[4], f[4];
                    ptx::ldsm4(hi, mh + s2 * 32);
                    ptx::ldsm4(lo, ml + s2 * 32);
                    ptx::ldsm4t(f, x_addr + s2 * 16 * PS);
                    ptx::mma_bf16(y[0], hi, f[0], f[1]);
                    ptx::mma_bf16(y[1], hi, f[2], f[3]);
                    ptx::mma_bf16(y[0], lo, f[0], f[1]);
                    ptx::mma_bf16(y[1], lo, f[2], f[3]);
                }
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int t = (e >> 1) ? tb : ta, c = qq * 16 + i * 8 + (lane & 3) * 2 + (e & 1);
                    if (t < n && c < vc) {
                        const float x = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(xt + t * PS + c * 2));
                        a.y[((int64_t)b * a.q_rows + t0 + t) * inner + head * a.vdim + v0 + c] = fmaf(dskip, x, y[i][e]) * silu_fast(z[i][e]);
                    }
                }
        }
        // ---- state ----
        if (s_live) {
            const float dec = expf(cum_s[kChunk - 1]);
#pragma unroll
            for (int i = 0; i < TN; ++i)
#pragma unroll
                for (int k = 0; k < TP; ++k)
#pragma unroll
                    for (int e = 0; e < 4; ++e) st[i][k][e] *= dec;
#pragma unroll
            for (int kk = 0; kk < kChunk / 16; ++kk)
                if (kk * 16 < n) {
                    const uint32_t wrow = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PS + (wp * TP * 8 + (lane >> 4) * 8) * 2;
#pragma unroll
                    for (int i = 0; i < TN; ++i) {
                        uint32_t af[4];
                        ptx::ldsm4t(af, b_sm + (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * NS + ((wn * TN + i) * 16 + ((lane >> 3) & 1) * 8) * 2);
#pragma unroll
                        for (int k2 = 0; k2 < TP / 2; ++k2) {
                            uint32_t f[4];
                            ptx::ldsm4t(f, ptx::smem_u32(w_hi) + wrow + k2 * 32);
                            ptx::mma_bf16(st[i][2 * k2], af, f[0], f[1]);
                            ptx::mma_bf16(st[i][2 * k2 + 1], af, f[2], f[3]);
                            ptx::ldsm4t(f, ptx::smem_u32(w_lo) + wrow + k2 * 32);
                            ptx::mma_bf16(st[i][2 * k2], af, f[0], f[1]);
                            ptx::mma_bf16(st[i][2 * k2 + 1], af, f[2], f[3]);
                        }
                    }
                }
        }
        __syncthreads();
        if (Cfg::kStages == 1) { if (t0 + kChunk < a.q_rows) load(t0 + kChunk, 0); } else buf ^= 1;
    }
#pragma unroll
    for (int i = 0; i < TN; ++i)
#pragma unroll
        for (int k = 0; k < TP; ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int n = (wn * TN + i) * 16 + (lane >> 2) + (e >> 1) * 8, p = (wp * TP + k) * 8 + (lane & 3) * 2 + (e & 1);
                if (s_live && p < vc) state[(int64_t)p * a.state_pad + n] = st[i][k][e];
            }
    keep_inputs(a, ring, channels, b, head, v0, vc, p0);
}

template <int NP>
cudaError_t chunk_launch(const SsmArgs& a, cudaStream_t s) {
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(ssm_chunk_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ChunkCfg<NP>::kSmem); });
    if (e != cudaSuccess) return e;
    ssm_chunk_kernel<NP><<<dim3((unsigned)a.heads, (unsigned)((a.vdim + 63) / 64), (unsigned)a.batch), kChunkThreads, ChunkCfg<NP>::kSmem, s>>>(
        a, a.heads * a.vdim + 2 * a.groups * a.state);
    return cudaGetLastError();
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

int64_t ssm_conv_floats(const SsmArgs& a) {  // per row, for either form
    const int64_t plain = a.heads * (int64_t)a.vdim + 2ll * a.groups * a.state, padded = (conv_cols(a) + 1) / 2;
    return plain > padded ? plain : padded;
}

cudaError_t launch_ssm_prefill(const SsmArgs& a, bool bf16, cudaStream_t s) {
    const int channels = a.heads * a.vdim + 2 * a.groups * a.state, cols = bf16 ? conv_cols(a) : channels;
    const dim3 grid((unsigned)((cols + 255) / 256), (unsigned)((a.q_rows + kConvTokens - 1) / kConvTokens), (unsigned)a.batch);
    if (bf16) ssm_conv_kernel<true><<<grid, 256, 0, s>>>(a, channels);
    else ssm_conv_kernel<false><<<grid, 256, 0, s>>>(a, channels);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    if (!bf16) return scan_launch_n<false>(a, s, false);
    switch (a.state_pad) {
        case 16: return chunk_launch<16>(a, s);
        case 32: return chunk_launch<32>(a, s);
        case 64: return chunk_launch<64>(a, s);
        case 128: return chunk_launch<128>(a, s);
        case 256: return chunk_launch<256>(a, s);
    }
    return cudaErrorInvalidValue;
}

}  // namespace bt
