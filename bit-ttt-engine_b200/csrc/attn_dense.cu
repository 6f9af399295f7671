// Softmax attention over a 16- or 32-bit cache: query and key norm over the whole projection, query temperature by
// position, capped scores, a learned sink in the denominator, mixing of the values with an earlier layer's.
// Scores, softmax and the running sums are f32 throughout.
#include <cooperative_groups.h>

#include "bt_dense.cuh"
#include "bt_ptx.cuh"

namespace cg = cooperative_groups;

namespace bt {

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

template <typename T>
__device__ __forceinline__ T to_cache(float v);
template <>
__device__ __forceinline__ float to_cache<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 to_cache<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// eight consecutive cache values as they are loaded
template <typename T>
struct Raw8;
template <>
struct Raw8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) { a = *reinterpret_cast<const float4*>(p); b = *reinterpret_cast<const float4*>(p + 4); }
    __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
    __device__ __forceinline__ void widen(float (&v)[8]) const { v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w; }
};

__device__ __forceinline__ float temperature(const DenseAttn& a, int pos) {
    if (a.temp_coef == 0.0f) return 1.0f;
    const float steps = a.temp_every_int > 0 ? (float)((unsigned)(pos + 1) / (unsigned)a.temp_every_int)
                                             : (float)floor((double)(pos + 1) / a.temp_every);
    return 1.0f + a.temp_coef * logf(steps + 1.0f);
}

// ---------------------------------------------------------------------------------------
// preparation of the new tokens' rows (prefill): one CTA per row
// ---------------------------------------------------------------------------------------
// sums of squares of the whole query and key rows; `red` holds 2 x 32 floats
__device__ __forceinline__ void qk_sums(const DenseAttn& a, const float* row, float* red, float& inv_q, float& inv_k) {
    const int nq = a.heads * a.dk, nk = a.n_kv * a.dk;
    float sq = 0.0f, sk = 0.0f;
#pragma unroll 16
    for (int c = threadIdx.x; c < nq; c += blockDim.x) sq = fmaf(row[c], row[c], sq);
#pragma unroll 8
    for (int c = threadIdx.x; c < nk; c += blockDim.x) sk = fmaf(row[nq + c], row[nq + c], sk);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
    if (l == 0) { red[w] = sq; red[32 + w] = sk; }
    __syncthreads();
    sq = 0.0f; sk = 0.0f;
    for (int i = 0; i < nw; ++i) { sq += red[i]; sk += red[32 + i]; }
    inv_q = a.q_norm ? 1.0f / sqrtf(sq / (float)nq + a.eps) : 1.0f;
    inv_k = a.k_norm ? 1.0f / sqrtf(sk / (float)nk + a.eps) : 1.0f;
}

template <typename T, bool QBF16>
__global__ void __launch_bounds__(256) attn_prep_kernel(const DenseAttn a) {
    __shared__ float red[64];
    const int64_t r = blockIdx.x;
    const int b = (int)(r / a.q_rows), p = a.pos[b] + (int)(r % a.q_rows);
    const float* row = a.qkv + r * a.ld;
    const int dk = a.dk, dv = a.dv, ks = a.kv.k_stride, vs = a.kv.v_stride;
    const int nq = a.heads * dk, nk = a.n_kv * dk, nv = a.n_kv * dv;
    float inv_q, inv_k;
    qk_sums(a, row, red, inv_q, inv_k);
    inv_q *= temperature(a, p);
    // a warp per head and turn
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int h = warp; h < a.heads; h += 8)
#pragma unroll 4
        for (int c = lane; c < ks; c += 32) {
            const int s = h * dk + c;
            const float v = c < dk ? row[s] * inv_q * (a.q_norm ? a.q_norm[s] : 1.0f) : 0.0f;
            const int64_t o = (r * a.heads + h) * ks + c;
            if (QBF16) reinterpret_cast<__nv_bfloat16*>(a.q_buf)[o] = __float2bfloat16_rn(v);
            else reinterpret_cast<float*>(a.q_buf)[o] = v;
        }
    if (p < 0 || p >= a.kv.max_seq) return;
    for (int g = warp; g < a.n_kv; g += 8) {
        const int64_t at = ((int64_t)b * a.n_kv + g) * a.kv.max_seq + p;
#pragma unroll 4
        for (int c = lane; c < ks; c += 32) {
            const int s = g * dk + c;
            const float v = c < dk ? row[nq + s] * inv_k * (a.k_norm ? a.k_norm[s] : 1.0f) : 0.0f;
            reinterpret_cast<T*>(a.kv.k)[at * ks + c] = to_cache<T>(v);
        }
        for (int c = lane; c < vs; c += 32) {
            const int s = g * dv + c;
            float v = 0.0f;
            if (c < dv) {
                v = row[nq + nk + s];
                if (a.v_first_out) a.v_first_out[r * nv + s] = v;
                if (a.v_first_in) v = (1.0f - a.v_lambda) * v + a.v_lambda * a.v_first_in[r * nv + s];
            }
            reinterpret_cast<T*>(a.kv.v)[at * vs + c] = to_cache<T>(v);
        }
    }
}

// The end of a span kernel: every CTA of the cluster holds (maximum, sum, un-normed output [h][c] at o_s[h * W + c]) of
// its span for nr heads; rank 0 reads them all, adds the sink and writes the rows of `head0 ..`.
__device__ __forceinline__ void merge_spans(const DenseAttn& a, float* m_s, float* l_s, float* o_s, int W, int nr, int head0,
                                            int64_t r, int split, int splits, int threads, const ActOut& out) {
    cg::cluster_group cluster = cg::this_cluster();
    if (splits > 1) cluster.sync(); else __syncthreads();
    if (split == 0) {
        for (int i = threadIdx.x; i < nr * a.dv; i += threads) {
            const int h = i / a.dv, c = i - h * a.dv, head = head0 + h;
            float ms[8], ls[8], os[8];
#pragma unroll
            for (int s = 0; s < 8; ++s) {  // all remote reads in flight together
                ms[s] = -INFINITY; ls[s] = os[s] = 0.0f;
                if (s < splits) {
                    ms[s] = *(splits > 1 ? cluster.map_shared_rank(m_s, s) + h : m_s + h);
                    ls[s] = *(splits > 1 ? cluster.map_shared_rank(l_s, s) + h : l_s + h);
                    os[s] = *(splits > 1 ? cluster.map_shared_rank(o_s, s) + h * W + c : o_s + h * W + c);
                }
            }
            const float sink = a.sink ? a.sink[head] : -INFINITY;
            float m = sink;
#pragma unroll
            for (int s = 0; s < 8; ++s) m = fmaxf(m, ms[s]);
            float den = a.sink ? expf(sink - m) : 0.0f, num = 0.0f;
#pragma unroll
            for (int s = 0; s < 8; ++s) {
                const float f = expf(ms[s] - m);  // an empty span: exp(-inf) = 0
                den = fmaf(ls[s], f, den);
                num = fmaf(os[s], f, num);
            }
            const float v = num / den;
            const int col = head * a.dv + c;
            if (out.tiles) *reinterpret_cast<__nv_bfloat16*>(out.tiles + dense_off(r, col, out.m_pad)) = __float2bfloat16_rn(v);
            else out.rows[r * out.ld + col] = v;
        }
    }
    if (splits > 1) cluster.sync();  // no CTA leaves while its sums are being read
}
// spans per query position: enough CTAs for the device, no span below 64 positions
int span_splits(const DenseAttn& a, int64_t groups) {
    int splits = 1;
    while (splits < 8 && groups * splits * 2 <= 2ll * a.sm_count && splits * 64 < a.kv.max_seq) splits *= 2;
    return splits;
}
template <typename... KArgs, typename... Args>
cudaError_t launch_spans(void (*kernel)(KArgs...), dim3 grid, int threads, size_t smem, cudaStream_t s, bool pdl, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3((unsigned)threads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = grid.x; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}

// ---------------------------------------------------------------------------------------
// one query position per CTA group: (row, KV head, up to 8 of its query heads), the positions cut into spans over the
// CTAs of a cluster.  This form computes in f32 on the FMA units (32-bit models).
// ---------------------------------------------------------------------------------------
// A CTA takes its span in tiles of 128 positions.  Scores: four lanes share a key (pieces of 8 dimensions in turn), two
// keys per lane, all heads of the group on the widened key.  Softmax: a warp per head over the tile.  Values: LPV lanes
// share a value row (8 dimensions each), the tile's value rows are requested before the scores are computed.
constexpr int kSpanThreads = 256, kSpanTile = 128;

template <typename T, int NR, int LPV>
__global__ void __launch_bounds__(kSpanThreads) attn_span_kernel(const DenseAttn a, bool prepared, int splits, const ActOut out) {
    extern __shared__ __align__(16) float sm[];
    constexpr int VPW = kSpanTile / 8;             // value rows per warp and tile
    constexpr int KPS = 32 / LPV;                  // value rows per step of a warp
    constexpr int VLD = VPW / KPS;
    const int dk = a.dk, dv = a.dv, ks = a.kv.k_stride, vs = a.kv.v_stride;
    float* q_s = sm;                               // [NR][ks]
    float* p_s = q_s + NR * ks;                    // [NR][128]
    float* alpha_s = p_s + NR * kSpanTile;         // [NR]
    float* m_s = alpha_s + 8;                      // [NR] running maximum; later the span's (maximum, sum)
    float* l_s = m_s + 8;
    float* red = l_s + 8;                          // 64
    float* o_s = red + 64;                         // [8 warps][NR][LPV * 8]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rep = a.heads / a.n_kv, hchunks = (rep + NR - 1) / NR;
    const int g = blockIdx.y / hchunks, h0 = (blockIdx.y % hchunks) * NR;  // first head inside the group
    const int nr = min(NR, rep - h0);
    const int64_t r = blockIdx.z;
    const int b = (int)(r / a.q_rows), split = blockIdx.x;
    const int nq = a.heads * dk, nk = a.n_kv * dk, nv = a.n_kv * dv;
    ptx::pdl_wait();
    ptx::pdl_launch_dependents();
    const int p = a.pos[b] + (int)(r % a.q_rows);
    const int total = min(p + 1, a.kv.max_seq);
    const int span = ((total + splits - 1) / splits + 7) / 8 * 8;
    const int t0 = min(split * span, total), t1 = min(t0 + span, total);
    T* kc = reinterpret_cast<T*>(a.kv.k) + ((int64_t)b * a.n_kv + g) * a.kv.max_seq * ks;
    T* vc = reinterpret_cast<T*>(a.kv.v) + ((int64_t)b * a.n_kv + g) * a.kv.max_seq * vs;

    if (!prepared) {
        const float* row = a.qkv + r * a.ld;
        float inv_q, inv_k;
        qk_sums(a, row, red, inv_q, inv_k);
        inv_q *= temperature(a, p);
        for (int i = threadIdx.x; i < NR * ks; i += kSpanThreads) {
            const int h = i / ks, c = i - h * ks, s = (g * rep + h0 + h) * dk + c;
            q_s[i] = (h < nr && c < dk) ? row[s] * inv_q * (a.q_norm ? a.q_norm[s] : 1.0f) : 0.0f;
        }
        if (t1 == p + 1 && t0 < t1) {  // the span that ends with the new token appends it (head chunks write the same values)
            for (int c = threadIdx.x; c < ks; c += kSpanThreads) {
                const int s = g * dk + c;
                kc[(int64_t)p * ks + c] = to_cache<T>(c < dk ? row[nq + s] * inv_k * (a.k_norm ? a.k_norm[s] : 1.0f) : 0.0f);
            }
            for (int c = threadIdx.x; c < vs; c += kSpanThreads) {
                const int s = g * dv + c;
                float v = 0.0f;
                if (c < dv) {
                    v = row[nq + nk + s];
                    if (a.v_first_out) a.v_first_out[r * nv + s] = v;
                    if (a.v_first_in) v = (1.0f - a.v_lambda) * v + a.v_lambda * a.v_first_in[r * nv + s];
                }
                vc[(int64_t)p * vs + c] = to_cache<T>(v);
            }
        }
    } else {
        const float* qb = reinterpret_cast<const float*>(a.q_buf) + (r * a.heads + g * rep + h0) * ks;
        for (int i = threadIdx.x; i < NR * ks; i += kSpanThreads) q_s[i] = i < nr * ks ? qb[i] : 0.0f;
    }
    if (threadIdx.x < NR) { m_s[threadIdx.x] = -INFINITY; l_s[threadIdx.x] = 0.0f; }
    __syncthreads();

    float acc[NR][8];
#pragma unroll
    for (int h = 0; h < NR; ++h)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[h][j] = 0.0f;
    const int kpieces = ks >> 3, vpiece = lane % LPV, vsub = lane / LPV;
    const bool v_live = vpiece * 8 < vs;

    for (int base = t0; base < t1; base += kSpanTile) {
        Raw8<T> vr[VLD];
#pragma unroll
        for (int i = 0; i < VLD; ++i) {
            const int t = base + warp * VPW + i * KPS + vsub;
            if (t < t1 && v_live) vr[i].load(vc + (int64_t)t * vs + vpiece * 8); else vr[i].zero();
        }
        {   // scores of this warp's 16 keys
            const int k0 = base + warp * 16 + (lane >> 2), k1 = k0 + 8, j0 = lane & 3;
            const T* r0 = kc + (int64_t)min(k0, t1 - 1) * ks;
            const T* r1 = kc + (int64_t)min(k1, t1 - 1) * ks;
            float s0[NR], s1[NR];
#pragma unroll
            for (int h = 0; h < NR; ++h) s0[h] = s1[h] = 0.0f;
#pragma unroll 4
            for (int c = j0; c < kpieces; c += 4) {
                Raw8<T> x0, x1;
                x0.load(r0 + c * 8);
                x1.load(r1 + c * 8);
                float f0[8], f1[8];
                x0.widen(f0);
                x1.widen(f1);
#pragma unroll
                for (int h = 0; h < NR; ++h) {
                    const float4 qa = *reinterpret_cast<const float4*>(q_s + h * ks + c * 8);
                    const float4 qb = *reinterpret_cast<const float4*>(q_s + h * ks + c * 8 + 4);
                    const float qv[8] = {qa.x, qa.y, qa.z, qa.w, qb.x, qb.y, qb.z, qb.w};
#pragma unroll
                    for (int j = 0; j < 8; ++j) { s0[h] = fmaf(f0[j], qv[j], s0[h]); s1[h] = fmaf(f1[j], qv[j], s1[h]); }
                }
            }
#pragma unroll
            for (int h = 0; h < NR; ++h) {
                s0[h] += __shfl_xor_sync(0xffffffffu, s0[h], 1);
                s1[h] += __shfl_xor_sync(0xffffffffu, s1[h], 1);
                s0[h] += __shfl_xor_sync(0xffffffffu, s0[h], 2);
                s1[h] += __shfl_xor_sync(0xffffffffu, s1[h], 2);
                if ((h & 3) == j0) {  // the four lanes of a key share the heads
                    float x0 = s0[h] * a.scale, x1 = s1[h] * a.scale;
                    if (a.softcap > 0.0f) { x0 = a.softcap * tanhf(x0 / a.softcap); x1 = a.softcap * tanhf(x1 / a.softcap); }
                    p_s[h * kSpanTile + warp * 16 + (lane >> 2)] = k0 < t1 ? x0 : -INFINITY;
                    p_s[h * kSpanTile + warp * 16 + 8 + (lane >> 2)] = k1 < t1 ? x1 : -INFINITY;
                }
            }
        }
        __syncthreads();
        if (warp < nr) {
            float* ph = p_s + warp * kSpanTile;
            float v[4], mx = -INFINITY;
#pragma unroll
            for (int i = 0; i < 4; ++i) { v[i] = ph[lane + 32 * i]; mx = fmaxf(mx, v[i]); }
            mx = warp_max(mx);
            const float m_old = m_s[warp], m_new = fmaxf(m_old, mx);
            float sum = 0.0f;
#pragma unroll
            for (int i = 0; i < 4; ++i) { const float e = expf(v[i] - m_new); ph[lane + 32 * i] = e; sum += e; }
            sum = warp_sum(sum);
            if (lane == 0) {
                const float al = expf(m_old - m_new);  // 0 for the first tile
                alpha_s[warp] = al;
                m_s[warp] = m_new;
                l_s[warp] = l_s[warp] * al + sum;
            }
        }
        __syncthreads();
#pragma unroll
        for (int h = 0; h < NR; ++h)
            if (h < nr) {
                const float al = alpha_s[h];
#pragma unroll
                for (int j = 0; j < 8; ++j) acc[h][j] *= al;
            }
#pragma unroll
        for (int i = 0; i < VLD; ++i) {
            float f[8];
            vr[i].widen(f);
            const int o = warp * VPW + i * KPS + vsub;
#pragma unroll
            for (int h = 0; h < NR; ++h)
                if (h < nr) {
                    const float w = p_s[h * kSpanTile + o];
#pragma unroll
                    for (int j = 0; j < 8; ++j) acc[h][j] = fmaf(w, f[j], acc[h][j]);
                }
        }
        __syncthreads();
    }
    // the warps' sums: first the row subgroups of a warp, then the warps
    constexpr int W = LPV * 8;
#pragma unroll
    for (int h = 0; h < NR; ++h)
#pragma unroll
        for (int j = 0; j < 8; ++j) {
#pragma unroll
            for (int o = LPV; o < 32; o <<= 1) acc[h][j] += __shfl_xor_sync(0xffffffffu, acc[h][j], o);
            if (lane < LPV) o_s[(warp * NR + h) * W + lane * 8 + j] = acc[h][j];
        }
    __syncthreads();
    for (int i = threadIdx.x; i < nr * W; i += kSpanThreads) {
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < 8; ++w) v += o_s[w * NR * W + i];
        o_s[i] = v;  // row 0 of the eight: read and written by this thread only
    }
    merge_spans(a, m_s, l_s, o_s, W, nr, g * rep + h0, r, split, splits, kSpanThreads, out);
}

template <typename T, int NR, int LPV>
cudaError_t span_launch(const DenseAttn& a, bool prepared, const ActOut& out, cudaStream_t s, bool pdl) {
    const int rep = a.heads / a.n_kv, hchunks = (rep + NR - 1) / NR;
    const int64_t groups = (int64_t)a.n_kv * hchunks * a.batch * a.q_rows;
    const int splits = span_splits(a, groups);
    const size_t smem = ((size_t)NR * a.kv.k_stride + NR * kSpanTile + 24 + 64 + (size_t)8 * NR * LPV * 8) * sizeof(float);
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(attn_span_kernel<T, NR, LPV>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024); });
    if (e != cudaSuccess) return e;
    if (smem > 100 * 1024) return cudaErrorInvalidConfiguration;
    return launch_spans(attn_span_kernel<T, NR, LPV>, dim3((unsigned)splits, (unsigned)(a.n_kv * hchunks), (unsigned)(a.batch * a.q_rows)),
                        kSpanThreads, smem, s, pdl, a, prepared, splits, out);
}
template <typename T, int NR>
cudaError_t span_launch_v(const DenseAttn& a, bool prepared, const ActOut& out, cudaStream_t s, bool pdl) {
    if (a.kv.v_stride <= 64) return span_launch<T, NR, 8>(a, prepared, out, s, pdl);
    if (a.kv.v_stride <= 128) return span_launch<T, NR, 16>(a, prepared, out, s, pdl);
    return span_launch<T, NR, 32>(a, prepared, out, s, pdl);
}
template <typename T>
cudaError_t span_launch_r(const DenseAttn& a, bool prepared, const ActOut& out, cudaStream_t s, bool pdl) {
    const int rep = a.heads / a.n_kv;
    if (rep == 1) return span_launch_v<T, 1>(a, prepared, out, s, pdl);
    if (rep <= 4) return span_launch_v<T, 4>(a, prepared, out, s, pdl);
    return span_launch_v<T, 8>(a, prepared, out, s, pdl);
}

// ---------------------------------------------------------------------------------------
// tiles of 64 query positions (prefill, bf16)
// ---------------------------------------------------------------------------------------
// Four warps, 16 query positions each, key tiles of 64 through a double buffer of cp.async copies.  Scores are bf16 products
// accumulated in f32; the softmax weights enter the product with the values as bf16 hi + lo (16 significand bits).
// Rows in shared memory are padded by 16 bytes, so that the eight rows of an ldmatrix fall into different banks.
constexpr int kTileQ = 64, kTileKeys = 64, kTileThreads = 128;

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// A raw score in units of ln 2, so that its exponential is one ex2: s * scale, or capped: cap * tanh(s * scale / cap) with
// tanh(u) = 1 - 2 / (e^2u + 1), whose absolute error is of the order of 1e-7 cap.
struct ScoreMap {
    float k, cap2;  // factor on the raw score; 2 cap / ln 2, 0: no cap
    __device__ __forceinline__ ScoreMap(float scale, float cap) {
        const float log2e = 1.4426950408889634f;
        k = cap > 0.0f ? scale / cap * (2.0f * log2e) : scale * log2e;
        cap2 = cap > 0.0f ? 2.0f * cap * log2e : 0.0f;
    }
    __device__ __forceinline__ float operator()(float s) const {
        const float u = s * k;
        return cap2 > 0.0f ? fmaf(-cap2, rcp(ex2(u) + 1.0f), 0.5f * cap2) : u;
    }
};
constexpr float kLn2 = 0.6931471805599453f;

// ---------------------------------------------------------------------------------------
// one query position per CTA group on the tensor cores (bf16 cache, decode)
// ---------------------------------------------------------------------------------------
// The heads of a group are the rows of the products: rows 0-7 the queries' (softmax weights') bf16 values, rows 8-15 what
// bf16 left over of them, so that the sum of the two accumulator rows carries 16 significand bits.  Every warp walks its
// own blocks of 16 positions with its own copy ring, maximum and sums - no CTA barrier inside - and the first blocks are
// requested before the wait on the projection in front (only the block of the new token has to come after it).
constexpr int kMmaThreads = 128, kMmaWarps = 4;
template <int V>
struct Const { static constexpr int value = V; };
template <int DK, int DV>
struct MmaCfg {
    static constexpr int kStages = DK + DV <= 128 ? 4 : (DK + DV <= 256 ? 3 : 2);
    static constexpr int KS = DK * 2 + 16, VS = DV * 2 + 16;   // bytes per row
    static constexpr int kStage = 16 * (KS + VS);
    static constexpr int kRing = kMmaWarps * kStages * kStage;
    static constexpr int kMerge = kMmaWarps * 8 * DV * 4;       // the warps' outputs, in the ring's place
    static constexpr size_t kBase = (size_t)(kRing > kMerge ? kRing : kMerge) + 16 * KS + (64 + 2 * kMmaWarps * 8) * 4;
    static constexpr size_t kSpan = (8 * DV + 16) * 4;          // a span's outputs, maxima and sums
    static constexpr size_t smem(int splits) { return kBase + splits * kSpan; }
};

template <int DK, int DV>
__global__ void __launch_bounds__(kMmaThreads) attn_span_mma_kernel(const DenseAttn a, bool prepared, int splits, const ActOut out) {
    using Cfg = MmaCfg<DK, DV>;
    constexpr int S = Cfg::kStages, KS = Cfg::KS, VS = Cfg::VS;
    extern __shared__ __align__(16) uint8_t tsm[];
    uint8_t* q_sm = tsm + (Cfg::kRing > Cfg::kMerge ? Cfg::kRing : Cfg::kMerge);   // [16][KS]: 8 rows hi, 8 rows lo
    float* red = reinterpret_cast<float*>(q_sm + 16 * KS);  // 64
    float* mw_s = red + 64;                                  // [4 warps][8]
    float* lw_s = mw_s + kMmaWarps * 8;
    float* span_s = lw_s + kMmaWarps * 8;                    // rank 0: [splits][8 maxima, 8 sums, 8 x DV outputs]
    cg::cluster_group cluster = cg::this_cluster();
    if (splits > 1) cluster.barrier_arrive();                // every CTA of the cluster runs before one writes to another
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int dk = a.dk, dv = a.dv, ks = a.kv.k_stride, vs = a.kv.v_stride;
    const int nk = (ks + 15) / 16, nv = (vs + 15) / 16;
    const int rep = a.heads / a.n_kv, hchunks = (rep + 7) / 8;
    const int g = blockIdx.y / hchunks, h0 = (blockIdx.y % hchunks) * 8;
    const int nr = min(8, rep - h0);
    const int64_t r = blockIdx.z;
    const int b = (int)(r / a.q_rows), split = blockIdx.x;
    const int nq = a.heads * dk, nkw = a.n_kv * dk, nvw = a.n_kv * dv;
    // positions move on long before the kernel in front of this one: they may be read ahead of the wait
    const int p = a.pos[b] + (int)(r % a.q_rows);
    const int total = min(p + 1, a.kv.max_seq);
    const int span = ((total + splits - 1) / splits + 15) / 16 * 16;
    const int t0 = min(split * span, total), t1 = min(t0 + span, total);
    __nv_bfloat16* kc = reinterpret_cast<__nv_bfloat16*>(a.kv.k) + ((int64_t)b * a.n_kv + g) * a.kv.max_seq * ks;
    __nv_bfloat16* vc = reinterpret_cast<__nv_bfloat16*>(a.kv.v) + ((int64_t)b * a.n_kv + g) * a.kv.max_seq * vs;
    const int blocks = (t1 - t0 + 15) / 16;
    const bool owner = !prepared && t1 == p + 1 && t0 < t1;    // appends the new token
    const uint32_t ring = ptx::smem_u32(tsm) + warp * S * Cfg::kStage;
    const int kp = nk * 2, vp = nv * 2;                          // 16-byte pieces per row
    // 16 rows of `stride` elements; FULL: the template's size, whose piece count is a constant
    auto copy_rows = [&](auto full, uint32_t dst, int dst_stride, const __nv_bfloat16* src, int stride, int pieces_rt, int base) {
        constexpr int kFull = decltype(full)::value;
        const int pieces = kFull ? kFull : pieces_rt;
#pragma unroll 4
        for (int e = lane; e < 16 * pieces; e += 32) {
            const int row = e / pieces, c = e - row * pieces;
            const bool live = base + row < t1 && (kFull || c * 8 < stride);
            ptx::cp16(dst + row * dst_stride + c * 16, live ? src + (int64_t)(base + row) * stride + c * 8 : src, live);
        }
    };
    auto load = [&](int i) {                                     // this warp's i-th block
        const int blk = warp + i * kMmaWarps;
        if (blk < blocks) {
            const int base = t0 + blk * 16;
            const uint32_t st = ring + (i % S) * Cfg::kStage;
            if (ks == DK) copy_rows(Const<DK / 8>(), st, KS, kc, ks, 0, base);
            else copy_rows(Const<0>(), st, KS, kc, ks, kp, base);
            if (vs == DV) copy_rows(Const<DV / 8>(), st + 16 * KS, VS, vc, vs, 0, base);
            else copy_rows(Const<0>(), st + 16 * KS, VS, vc, vs, vp, base);
        }
    };
    auto is_new = [&](int i) { return owner && warp + i * kMmaWarps == blocks - 1; };
    auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };
    if (prepared) { ptx::pdl_wait(); }                           // the cache rows come from the kernel in front
#pragma unroll 1
    for (int i = 0; i < S - 1; ++i) { if (!is_new(i)) load(i); commit(); }
    if (!prepared) ptx::pdl_wait();
    ptx::pdl_launch_dependents();

    // ---- queries as bf16 hi | lo rows, zero beyond the heads and sizes in use ----
    float inv_q = 1.0f, inv_k = 1.0f;
    const float* row = a.qkv + r * a.ld;
    if (!prepared) {
        qk_sums(a, row, red, inv_q, inv_k);
        inv_q *= temperature(a, p);
    }
    const int kw = nk * 16;
    for (int c = threadIdx.x; c < kw; c += kMmaThreads) {
        float v[8];
#pragma unroll
        for (int h = 0; h < 8; ++h) {  // all heads requested together
            v[h] = 0.0f;
            if (h < nr && c < dk) {
                const int head = g * rep + h0 + h, s = head * dk + c;
                v[h] = prepared ? reinterpret_cast<const float*>(a.q_buf)[(r * a.heads + head) * ks + c]
                                : row[s] * inv_q * (a.q_norm ? a.q_norm[s] : 1.0f);
            }
        }
#pragma unroll
        for (int h = 0; h < 8; ++h) {
            const __nv_bfloat16 hi = __float2bfloat16_rn(v[h]);
            *reinterpret_cast<__nv_bfloat16*>(q_sm + h * KS + c * 2) = hi;
            *reinterpret_cast<__nv_bfloat16*>(q_sm + (8 + h) * KS + c * 2) = __float2bfloat16_rn(v[h] - __bfloat162float(hi));
        }
    }
    if (owner) {  // (head chunks of one KV head write the same values)
        for (int c = threadIdx.x; c < ks; c += kMmaThreads) {
            const int s = g * dk + c;
            kc[(int64_t)p * ks + c] = __float2bfloat16_rn(c < dk ? row[nq + s] * inv_k * (a.k_norm ? a.k_norm[s] : 1.0f) : 0.0f);
        }
        for (int c = threadIdx.x; c < vs; c += kMmaThreads) {
            const int s = g * dv + c;
            float v = 0.0f;
            if (c < dv) {
                v = row[nq + nkw + s];
                if (a.v_first_out) a.v_first_out[r * nvw + s] = v;
                if (a.v_first_in) v = (1.0f - a.v_lambda) * v + a.v_lambda * a.v_first_in[r * nvw + s];
            }
            vc[(int64_t)p * vs + c] = __float2bfloat16_rn(v);
        }
    }
    __syncthreads();
#pragma unroll 1
    for (int i = 0; i < S - 1; ++i)
        if (is_new(i)) { load(i); commit(); }

    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j] = 0.0f;
    float m_run = -INFINITY, l_run = 0.0f;
    const ScoreMap score(a.scale, a.softcap);
    const uint32_t q_addr = ptx::smem_u32(q_sm) + (lane & 15) * KS + (lane >> 4) * 16;
    constexpr bool kQRegs = DK <= 128;
    uint32_t qf[kQRegs ? DK / 16 : 1][4];
    if (kQRegs) {
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk)
            if (kk < nk) ptx::ldsm4(qf[kQRegs ? kk : 0], q_addr + kk * 32);
    }
    for (int i = 0; warp + i * kMmaWarps < blocks; ++i) {
        if (is_new(i)) asm volatile("cp.async.wait_group 0;" ::: "memory");
        else asm volatile("cp.async.wait_group %0;" ::"n"(S - 2) : "memory");
        __syncwarp();
        load(i + S - 1);  // into the slot of the block before this one
        commit();
        const uint32_t kb = ring + (i % S) * Cfg::kStage, vb = kb + 16 * KS;
        float s[2][4] = {};
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk)
            if (kk < nk) {
                uint32_t kf[4];
                ptx::ldsm4(kf, kb + ((lane & 7) + ((lane >> 4) << 3)) * KS + kk * 32 + ((lane >> 3) & 1) * 16);
                if (!kQRegs) ptx::ldsm4(qf[0], q_addr + kk * 32);
                ptx::mma_bf16(s[0], qf[kQRegs ? kk : 0], kf[0], kf[1]);
                ptx::mma_bf16(s[1], qf[kQRegs ? kk : 0], kf[2], kf[3]);
            }
        // head = lane / 4; positions 2 (lane % 4) + {0, 1} of both halves
        const int key0 = t0 + (warp + i * kMmaWarps) * 16 + (lane & 3) * 2;
        float x[4], mx = m_run;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            x[j] = score(s[j >> 1][j & 1] + s[j >> 1][2 + (j & 1)]);
            if (key0 + (j >> 1) * 8 + (j & 1) >= t1) x[j] = -INFINITY;
            mx = fmaxf(mx, x[j]);
        }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float al = ex2(m_run - mx);
        m_run = mx;
        l_run *= al;
        uint32_t pf[4];
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
            const float e0 = ex2(x[j] - mx), e1 = ex2(x[j + 1] - mx);
            l_run += e0 + e1;
            const uint32_t hi = ptx::pack2(e0, e1);
            pf[j] = hi;                                                                          // rows 0-7: hi
            pf[j + 1] = ptx::pack2(e0 - __uint_as_float(hi << 16), e1 - __uint_as_float(hi & 0xffff0000u));  // rows 8-15: the rest
        }
#pragma unroll
        for (int n2 = 0; n2 < DV / 16; ++n2)
            if (n2 < nv) {
                uint32_t vf[4];
                ptx::ldsm4t(vf, vb + ((lane & 7) + ((lane >> 3) & 1) * 8) * VS + n2 * 32 + (lane >> 4) * 16);
#pragma unroll
                for (int j = 0; j < 4; ++j) { o[2 * n2][j] *= al; o[2 * n2 + 1][j] *= al; }
                ptx::mma_bf16(o[2 * n2], pf, vf[0], vf[1]);
                ptx::mma_bf16(o[2 * n2 + 1], pf, vf[2], vf[3]);
            }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    l_run += __shfl_xor_sync(0xffffffffu, l_run, 1);
    l_run += __shfl_xor_sync(0xffffffffu, l_run, 2);
    if ((lane & 3) == 0) { mw_s[warp * 8 + (lane >> 2)] = m_run * kLn2; lw_s[warp * 8 + (lane >> 2)] = l_run; }
    __syncthreads();  // the ring is free on every warp
    float* o_w = reinterpret_cast<float*>(tsm);  // [4 warps][8][DV]
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) o_w[(warp * 8 + (lane >> 2)) * DV + i * 8 + (lane & 3) * 2 + j] = o[i][j] + o[i][2 + j];
    __syncthreads();
    // this span's sums go straight to the CTA that finishes them
    float* dst = span_s + split * (Cfg::kSpan / 4);
    if (splits > 1) {
        cluster.barrier_wait();
        dst = cluster.map_shared_rank(dst, 0);
    }
#pragma unroll 4
    for (int i = threadIdx.x; i < nr * DV; i += kMmaThreads) {
        const int h = i / DV;
        float m = -INFINITY;
#pragma unroll
        for (int w = 0; w < kMmaWarps; ++w) m = fmaxf(m, mw_s[w * 8 + h]);
        float v = 0.0f, l = 0.0f;
#pragma unroll
        for (int w = 0; w < kMmaWarps; ++w) {
            const float f = mw_s[w * 8 + h] == -INFINITY ? 0.0f : __expf(mw_s[w * 8 + h] - m);
            v = fmaf(o_w[w * 8 * DV + i], f, v);
            l = fmaf(lw_s[w * 8 + h], f, l);
        }
        dst[16 + i] = v;
        if (i == h * DV) { dst[h] = m; dst[8 + h] = l; }
    }
    if (splits > 1) cluster.sync(); else __syncthreads();
    if (split != 0) return;
#pragma unroll 4
    for (int i = threadIdx.x; i < nr * dv; i += kMmaThreads) {
        const int h = i / dv, c = i - h * dv, head = g * rep + h0 + h;
        const float sink = a.sink ? a.sink[head] : -INFINITY;
        float m = sink;
        for (int s = 0; s < splits; ++s) m = fmaxf(m, span_s[s * (Cfg::kSpan / 4) + h]);
        float den = a.sink ? expf(sink - m) : 0.0f, num = 0.0f;
        for (int s = 0; s < splits; ++s) {
            const float* e = span_s + s * (Cfg::kSpan / 4);
            const float f = expf(e[h] - m);  // an empty span: exp(-inf) = 0
            den = fmaf(e[8 + h], f, den);
            num = fmaf(e[16 + h * DV + c], f, num);
        }
        const float v = num / den;
        const int col = head * dv + c;
        if (out.tiles) *reinterpret_cast<__nv_bfloat16*>(out.tiles + dense_off(r, col, out.m_pad)) = __float2bfloat16_rn(v);
        else out.rows[r * out.ld + col] = v;
    }
}

template <int DK, int DV>
cudaError_t span_mma_launch(const DenseAttn& a, bool prepared, const ActOut& out, cudaStream_t s, bool pdl) {
    const int hchunks = (a.heads / a.n_kv + 7) / 8;
    const int splits = span_splits(a, (int64_t)a.n_kv * hchunks * a.batch * a.q_rows);
    const size_t smem = MmaCfg<DK, DV>::smem(splits);
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(attn_span_mma_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MmaCfg<DK, DV>::smem(8)); });
    if (e != cudaSuccess) return e;
    return launch_spans(attn_span_mma_kernel<DK, DV>, dim3((unsigned)splits, (unsigned)(a.n_kv * hchunks), (unsigned)(a.batch * a.q_rows)),
                        kMmaThreads, smem, s, pdl, a, prepared, splits, out);
}
template <int DK>
cudaError_t span_mma_launch_v(const DenseAttn& a, bool prepared, const ActOut& out, cudaStream_t s, bool pdl) {
    if (a.kv.v_stride <= 64) return span_mma_launch<DK, 64>(a, prepared, out, s, pdl);
    if (a.kv.v_stride <= 128) return span_mma_launch<DK, 128>(a, prepared, out, s, pdl);
    return span_mma_launch<DK, 256>(a, prepared, out, s, pdl);
}

// LATENT: keys and values are bf16 rows expanded from the latents, the last key columns the rotated part all heads share.
struct LatentTile {
    const __nv_bfloat16* kv = nullptr;  // [sequence][kv_rows][heads k_main | heads v_stride]
    int64_t kv_ld = 0, kv_seq = 0;      // elements between positions and between sequences
    int k_main = 0;                     // columns of a head's own key part
    LatentView latent;
    int b0 = 0;
    const float* gate = nullptr;        // output gates of the rows
    int64_t gate_ld = 0;
};
template <int DK, int DV, bool LATENT>  // upper bounds of the (padded) head sizes
__global__ void __launch_bounds__(kTileThreads) attn_tile_kernel(const DenseAttn a, const LatentTile lt, const ActOut out) {
    extern __shared__ __align__(16) uint8_t tsm[];
    constexpr int KS = DK * 2 + 16, VS = DV * 2 + 16;  // bytes per row
    const uint32_t q_sm = ptx::smem_u32(tsm);
    const uint32_t k_sm = q_sm + kTileQ * KS, v_sm = k_sm + 2 * kTileKeys * KS;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int qt = gridDim.x - 1 - blockIdx.x;  // the longest first
    const int head = blockIdx.y, b = blockIdx.z + (LATENT ? lt.b0 : 0), g = LATENT ? 0 : head / (a.heads / a.n_kv);
    const int ks = a.kv.k_stride, vs = a.kv.v_stride;
    const int nk = (ks + 15) / 16, nv = (vs + 15) / 16;  // 16-wide steps in use
    const int past = a.pos[b], q0 = qt * kTileQ, rows = min(kTileQ, a.q_rows - q0);
    const int last = past + q0 + rows - 1;               // last position any row of this tile sees
    const int key_tiles = last / kTileKeys + 1;
    const __nv_bfloat16* qg = reinterpret_cast<const __nv_bfloat16*>(a.q_buf) + (((int64_t)b * a.q_rows + q0) * a.heads + head) * ks;
    const __nv_bfloat16* kg = LATENT ? lt.kv + blockIdx.z * lt.kv_seq + head * lt.k_main
                                     : reinterpret_cast<const __nv_bfloat16*>(a.kv.k) + ((int64_t)b * a.n_kv + g) * a.kv.max_seq * ks;
    const __nv_bfloat16* vg = LATENT ? lt.kv + blockIdx.z * lt.kv_seq + a.heads * lt.k_main + head * vs
                                     : reinterpret_cast<const __nv_bfloat16*>(a.kv.v) + ((int64_t)b * a.n_kv + g) * a.kv.max_seq * vs;
    const int64_t k_ld = LATENT ? lt.kv_ld : ks, v_ld = LATENT ? lt.kv_ld : vs;

    const int qpieces = nk * 2, vpieces = nv * 2;        // 16-byte pieces per row
    for (int i = threadIdx.x; i < kTileQ * qpieces; i += kTileThreads) {
        const int r = i / qpieces, c = i - r * qpieces;
        const bool live = r < rows && c * 8 < ks;
        ptx::cp16(q_sm + r * KS + c * 16, live ? qg + (int64_t)r * a.heads * ks + c * 8 : qg, live);
    }
    auto load = [&](int kt, int bufi) {
        const int base = kt * kTileKeys;
        for (int i = threadIdx.x; i < kTileKeys * qpieces; i += kTileThreads) {
            const int r = i / qpieces, c = i - r * qpieces;
            const bool live = base + r <= last && c * 8 < ks;
            const void* src = kg + (int64_t)(base + r) * k_ld + c * 8;
            if (LATENT && c * 8 >= lt.k_main) src = reinterpret_cast<const uint8_t*>(lt.latent.rows) + b * lt.latent.seq_bytes() + lt.latent.off(base + r, lt.latent.rot_col() + c * 8 - lt.k_main);
            ptx::cp16(k_sm + (bufi * kTileKeys + r) * KS + c * 16, live ? src : kg, live);
        }
        for (int i = threadIdx.x; i < kTileKeys * vpieces; i += kTileThreads) {
            const int r = i / vpieces, c = i - r * vpieces;
            const bool live = base + r <= last && c * 8 < vs;
            ptx::cp16(v_sm + (bufi * kTileKeys + r) * VS + c * 16, live ? vg + (int64_t)(base + r) * v_ld + c * 8 : vg, live);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0, 0);

    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j] = 0.0f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
    const int row_a = past + q0 + warp * 16 + (lane >> 2);  // positions of this lane's two query rows: row_a, row_a + 8
    const ScoreMap score(a.scale, a.softcap);
    const uint32_t q_addr = q_sm + (warp * 16 + (lane & 15)) * KS + (lane >> 4) * 16;

    for (int kt = 0; kt < key_tiles; ++kt) {
        const int bufi = kt & 1;
        if (kt + 1 < key_tiles) {
            load(kt + 1, bufi ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        float s[kTileKeys / 8][4];
#pragma unroll
        for (int i = 0; i < kTileKeys / 8; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) s[i][j] = 0.0f;
        const uint32_t kb = k_sm + bufi * kTileKeys * KS, vb = v_sm + bufi * kTileKeys * VS;
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk)
            if (kk < nk) {
                uint32_t qa[4];
                ptx::ldsm4(qa, q_addr + kk * 32);
#pragma unroll
                for (int n2 = 0; n2 < kTileKeys / 16; ++n2) {  // 16 keys: two n-tiles
                    uint32_t kf[4];
                    ptx::ldsm4(kf, kb + (n2 * 16 + (lane & 7) + ((lane >> 4) << 3)) * KS + kk * 32 + ((lane >> 3) & 1) * 16);
                    ptx::mma_bf16(s[2 * n2], qa, kf[0], kf[1]);
                    ptx::mma_bf16(s[2 * n2 + 1], qa, kf[2], kf[3]);
                }
            }
        const int key0 = kt * kTileKeys + (lane & 3) * 2;
        const bool mask = kt * kTileKeys + kTileKeys - 1 > past + q0 + warp * 16;
        float mx[2] = {m_run[0], m_run[1]};
#pragma unroll
        for (int i = 0; i < kTileKeys / 8; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                float x = score(s[i][j]);
                if (mask && key0 + i * 8 + (j & 1) > row_a + (j >> 1) * 8) x = -INFINITY;
                s[i][j] = x;
                mx[j >> 1] = fmaxf(mx[j >> 1], x);
            }
        float al[2];
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            mx[q] = fmaxf(mx[q], __shfl_xor_sync(0xffffffffu, mx[q], 1));
            mx[q] = fmaxf(mx[q], __shfl_xor_sync(0xffffffffu, mx[q], 2));
            al[q] = ex2(m_run[q] - mx[q]);  // position 0 is visible to every row, so mx is finite after the first tile
            m_run[q] = mx[q];
            l_run[q] *= al[q];
        }
#pragma unroll
        for (int i = 0; i < kTileKeys / 8; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float e = ex2(s[i][j] - mx[j >> 1]);
                s[i][j] = e;
                l_run[j >> 1] += e;
            }
#pragma unroll
        for (int i = 0; i < DV / 8; ++i) { o[i][0] *= al[0]; o[i][1] *= al[0]; o[i][2] *= al[1]; o[i][3] *= al[1]; }
#pragma unroll
        for (int k2 = 0; k2 < kTileKeys / 16; ++k2) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int f = 0; f < 4; ++f) {
                const float x = s[2 * k2 + (f >> 1)][(f & 1) * 2], y = s[2 * k2 + (f >> 1)][(f & 1) * 2 + 1];
                hi[f] = ptx::pack2(x, y);
                lo[f] = ptx::pack2(x - __uint_as_float(hi[f] << 16), y - __uint_as_float(hi[f] & 0xffff0000u));
            }
#pragma unroll
            for (int n2 = 0; n2 < DV / 16; ++n2)
                if (n2 < nv) {
                    uint32_t vf[4];
                    ptx::ldsm4t(vf, vb + (k2 * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VS + n2 * 32 + (lane >> 4) * 16);
                    ptx::mma_bf16(o[2 * n2], hi, vf[0], vf[1]);
                    ptx::mma_bf16(o[2 * n2], lo, vf[0], vf[1]);
                    ptx::mma_bf16(o[2 * n2 + 1], hi, vf[2], vf[3]);
                    ptx::mma_bf16(o[2 * n2 + 1], lo, vf[2], vf[3]);
                }
        }
        __syncthreads();  // before the buffer is refilled
    }
    float f[2];
#pragma unroll
    for (int q = 0; q < 2; ++q) {
        l_run[q] += __shfl_xor_sync(0xffffffffu, l_run[q], 1);
        l_run[q] += __shfl_xor_sync(0xffffffffu, l_run[q], 2);
        const float m_nat = m_run[q] * kLn2;
        float m = m_nat, den = l_run[q];
        f[q] = 1.0f;
        if (a.sink) {
            const float sk = a.sink[head];
            m = fmaxf(m, sk);
            f[q] = expf(m_nat - m);
            den = den * f[q] + expf(sk - m);
        }
        f[q] /= den;
        const int lr = warp * 16 + (lane >> 2) + q * 8;
        if (LATENT && lt.gate && lr < rows) f[q] /= 1.0f + expf(-lt.gate[((int64_t)b * a.q_rows + q0 + lr) * lt.gate_ld + head]);
    }
    const int dv = a.dv;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            const int lr = warp * 16 + (lane >> 2) + q * 8, c = i * 8 + (lane & 3) * 2;
            if (lr >= rows || c >= dv) continue;
            const int64_t r = (int64_t)b * a.q_rows + q0 + lr;
            const int col = head * dv + c;
            const float x = o[i][2 * q] * f[q], y = o[i][2 * q + 1] * f[q];
            if ((dv & 1) == 0) {
                *reinterpret_cast<uint32_t*>(out.tiles + dense_off(r, col, out.m_pad)) = ptx::pack2(x, y);
            } else {
                *reinterpret_cast<__nv_bfloat16*>(out.tiles + dense_off(r, col, out.m_pad)) = __float2bfloat16_rn(x);
                if (c + 1 < dv) *reinterpret_cast<__nv_bfloat16*>(out.tiles + dense_off(r, col + 1, out.m_pad)) = __float2bfloat16_rn(y);
            }
        }
}

template <int DK, int DV, bool LATENT>
cudaError_t tile_launch(const DenseAttn& a, const LatentTile& lt, const ActOut& out, cudaStream_t s) {
    constexpr size_t smem = (size_t)kTileQ * (DK * 2 + 16) + 2 * kTileKeys * (DK * 2 + 16 + DV * 2 + 16);
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(attn_tile_kernel<DK, DV, LATENT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); });
    if (e != cudaSuccess) return e;
    attn_tile_kernel<DK, DV, LATENT><<<dim3((unsigned)((a.q_rows + kTileQ - 1) / kTileQ), (unsigned)a.heads, (unsigned)a.batch), kTileThreads, smem, s>>>(a, lt, out);
    return cudaGetLastError();
}
template <int DK, bool LATENT>
cudaError_t tile_launch_v(const DenseAttn& a, const LatentTile& lt, const ActOut& out, cudaStream_t s) {
    if (a.kv.v_stride <= 64) return tile_launch<DK, 64, LATENT>(a, lt, out, s);
    if (a.kv.v_stride <= 128) return tile_launch<DK, 128, LATENT>(a, lt, out, s);
    return tile_launch<DK, 256, LATENT>(a, lt, out, s);
}
template <bool LATENT>
cudaError_t tile_launch_k(const DenseAttn& a, const LatentTile& lt, const ActOut& out, cudaStream_t s) {
    if (a.kv.k_stride <= 64) return tile_launch_v<64, LATENT>(a, lt, out, s);
    if (a.kv.k_stride <= 128) return tile_launch_v<128, LATENT>(a, lt, out, s);
    if (LATENT && a.kv.k_stride <= 192) return tile_launch_v<192, LATENT>(a, lt, out, s);
    return tile_launch_v<256, LATENT>(a, lt, out, s);
}
int pad8(int n) { return (n + 7) / 8 * 8; }

}  // namespace

int attn_max_dim() { return 256; }

cudaError_t launch_attn_prep(const DenseAttn& a, cudaStream_t s) {
    const unsigned grid = (unsigned)(a.batch * a.q_rows);
    if (a.kv.f32) attn_prep_kernel<float, false><<<grid, 256, 0, s>>>(a);
    else if (a.q_bf16) attn_prep_kernel<__nv_bfloat16, true><<<grid, 256, 0, s>>>(a);
    else attn_prep_kernel<__nv_bfloat16, false><<<grid, 256, 0, s>>>(a);
    return cudaGetLastError();
}

cudaError_t launch_attn_span(const DenseAttn& a, bool prepared, const ActOut& out, cudaStream_t s, bool pdl) {
    if (a.kv.k_stride > 256 || a.kv.v_stride > 256 || (!prepared && a.q_rows != 1) || (prepared && a.q_bf16)) return cudaErrorInvalidValue;
    if (a.kv.f32) return span_launch_r<float>(a, prepared, out, s, pdl);
    if (a.kv.k_stride <= 64) return span_mma_launch_v<64>(a, prepared, out, s, pdl);
    if (a.kv.k_stride <= 128) return span_mma_launch_v<128>(a, prepared, out, s, pdl);
    return span_mma_launch_v<256>(a, prepared, out, s, pdl);
}

bool attn_tile_fits(const DenseAttn& a) { return !a.kv.f32 && a.kv.k_stride <= 256 && a.kv.v_stride <= 256; }

cudaError_t launch_attn_tile(const DenseAttn& a, const ActOut& out, cudaStream_t s) {
    if (!attn_tile_fits(a) || !a.q_bf16 || !out.tiles) return cudaErrorInvalidValue;
    return tile_launch_k<false>(a, LatentTile(), out, s);
}

bool latent_tile_fits(const LatentAttn& a) { return !a.kv.f32 && pad8(a.dim) + pad8(a.rot) <= 256 && pad8(a.vdim) <= 256; }

cudaError_t launch_latent_tile(const LatentAttn& l, const __nv_bfloat16* kv16, int64_t kv_rows, int b0, int nb, const ActOut& out, cudaStream_t s) {
    if (!latent_tile_fits(l) || !l.q_buf || !out.tiles) return cudaErrorInvalidValue;
    DenseAttn a;
    a.q_buf = l.q_buf; a.q_bf16 = true;
    a.scale = l.scale; a.pos = l.pos; a.batch = nb; a.q_rows = l.q_rows; a.heads = l.heads; a.n_kv = l.heads;
    a.kv.k_stride = pad8(l.dim) + pad8(l.rot); a.kv.v_stride = pad8(l.vdim); a.kv.max_seq = l.kv.max_seq;
    a.dk = a.kv.k_stride; a.dv = l.vdim;
    LatentTile t;
    t.kv = kv16; t.k_main = pad8(l.dim); t.kv_ld = (int64_t)l.heads * (t.k_main + a.kv.v_stride); t.kv_seq = kv_rows * t.kv_ld;
    t.latent = l.kv; t.b0 = b0;
    t.gate = l.gate ? l.proj + l.heads * (l.dim + l.rot) + l.rank + l.rot : nullptr;
    t.gate_ld = l.ld;
    return tile_launch_k<true>(a, t, out, s);
}

}  // namespace bt
