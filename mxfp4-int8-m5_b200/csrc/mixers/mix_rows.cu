// Row kernels around the mixers: embedding lookup (optionally with a table row per pair of tokens), residual update with a norm on
// the sublayer's output and an optional average over all layers' results, residual update followed by the next sublayer's norm,
// row norm, causal depthwise convolution + SiLU, per-head norm + gate.
// The residual stream is float32; a bfloat16 copy for the next matrix product is written beside it.
#include <cooperative_groups.h>
#include "mix_common.cuh"

namespace cg = cooperative_groups;

namespace scmx {

// ---- embedding ----------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) embed_kernel(const int64_t* tok, const T* table, int64_t V, int W, float* x, T* h) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x;
    int64_t id = tok[t];
    id = id < 0 ? 0 : (id >= V ? V - 1 : id);
    for (int i = threadIdx.x; i < W; i += 256) {
        const T raw = table[id * W + i];
        x[t * W + i] = ldf(&raw);
        if (h != nullptr) h[t * W + i] = raw;
    }
}

// x[t] = scale table[tok[t]] + pairs[row], row = (before mul_prev + tok mul_cur) mod buckets, or `buckets` at the start of a
// sequence (prev < 0).  Only the first CTA reads and advances prev.
struct EmbedPairArgs {
    const int64_t* tok;
    int64_t* prev;           // token before this portion, negative: none
    float* x;
    int64_t V, T, buckets, mul_prev, mul_cur;
    int W;
    float scale;
};
template <typename T>
__global__ void __launch_bounds__(256) embed_pair_kernel(const T* table, const T* pairs, const EmbedPairArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x;
    int64_t id = a.tok[t];
    id = id < 0 ? 0 : (id >= a.V ? a.V - 1 : id);
    const T* pr = nullptr;
    if (pairs != nullptr) {
        const int64_t before = t > 0 ? a.tok[t - 1] : *a.prev;
        int64_t row = a.buckets;
        if (before >= 0) {
            row = (before * a.mul_prev + id * a.mul_cur) % a.buckets;
            if (row < 0) row += a.buckets;
        }
        pr = pairs + row * a.W;
    }
    for (int i = threadIdx.x; i < a.W; i += 256) {
        const float e = ldf(table + id * a.W + i) * a.scale;
        a.x[t * a.W + i] = pr != nullptr ? e + ldf(pr + i) : e;
    }
    if (t == 0 && a.prev != nullptr) {
        __syncthreads();
        if (threadIdx.x == 0) *a.prev = a.tok[a.T - 1];
    }
}

// ---- residual + next norm -----------------------------------------------------------------------------------------------
struct AddNormArgs {
    const float* y;        // [T, ldy] sublayer output, or null
    const float* x;        // [T, W]
    const float* w;        // [W] norm weight of the next sublayer
    float* x_out;          // [T, W], or null (nothing to add); may be x
    void* h_out;           // [T, W] activation type
    int64_t ldy;
    int W;
    float mult, eps;
};

// r = x + mult y;  h = r / rms(r) w.  A cluster of CTAs shares one row; each thread keeps its first groups of V values.
template <typename T, int V>
__global__ void __launch_bounds__(256) add_norm_kernel(const AddNormArgs a) {
    constexpr int KEEP = 4;
    __shared__ float red[33];
    __shared__ float part;
    pdl_launch_dependents();
    cg::cluster_group cl = cg::this_cluster();
    const int nc = (int)cl.num_blocks(), rank = (int)cl.block_rank();
    const int64_t t = blockIdx.x / nc;
    const int nv = a.W / V, per = (nv + nc - 1) / nc;
    const int v0 = rank * per, v1 = min(nv, v0 + per);
    pdl_wait();
    const float *y = a.y == nullptr ? nullptr : a.y + t * a.ldy, *x = a.x + t * a.W;
    float* xo = a.x_out == nullptr ? nullptr : a.x_out + t * a.W;
    float keep[KEEP][V], ss = 0.0f;
    auto read = [&](int i, float (&r)[V]) {
        if (V == 4) {
            const float4 p = *reinterpret_cast<const float4*>(x + 4 * i);
            r[0] = p.x; r[1 % V] = p.y; r[2 % V] = p.z; r[3 % V] = p.w;
            if (y != nullptr) {
                const float4 q = *reinterpret_cast<const float4*>(y + 4 * i);
                r[0] = fmaf(a.mult, q.x, r[0]); r[1 % V] = fmaf(a.mult, q.y, r[1 % V]); r[2 % V] = fmaf(a.mult, q.z, r[2 % V]); r[3 % V] = fmaf(a.mult, q.w, r[3 % V]);
            }
        } else {
            r[0] = x[i];
            if (y != nullptr) r[0] = fmaf(a.mult, y[i], r[0]);
        }
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int i = v0 + (int)threadIdx.x + 256 * k;
        if (i < v1) {
            read(i, keep[k]);
        } else {
#pragma unroll
            for (int e = 0; e < V; ++e) keep[k][e] = 0.0f;
        }
    }
#pragma unroll
    for (int k = 0; k < KEEP; ++k)
#pragma unroll
        for (int e = 0; e < V; ++e) ss += keep[k][e] * keep[k][e];
    for (int i = v0 + (int)threadIdx.x + 256 * KEEP; i < v1; i += 256) {
        float r[V];
        read(i, r);
#pragma unroll
        for (int e = 0; e < V; ++e) ss += r[e] * r[e];
    }
    ss = block_sumf(ss, red);
    if (nc > 1) {
        if (threadIdx.x == 0) part = ss;
        cl.sync();
        ss = 0.0f;
        for (int r = 0; r < nc; ++r) ss += *cl.map_shared_rank(&part, r);
        cl.sync();              // nobody leaves while its partial sum may still be read
    }
    const float inv = rms_inv_f32(ss, a.W, a.eps);
    T* h = static_cast<T*>(a.h_out) + t * a.W;
    auto write = [&](int i, const float (&r)[V]) {
        if (V == 4) {
            const float4 w = *reinterpret_cast<const float4*>(a.w + 4 * i);
            if (xo != nullptr) st4(xo + 4 * i, r[0], r[1 % V], r[2 % V], r[3 % V]);
            st4(h + 4 * i, r[0] * inv * w.x, r[1 % V] * inv * w.y, r[2 % V] * inv * w.z, r[3 % V] * inv * w.w);
        } else {
            if (xo != nullptr) xo[i] = r[0];
            stf(h + i, r[0] * inv * a.w[i]);
        }
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int i = v0 + (int)threadIdx.x + 256 * k;
        if (i < v1) write(i, keep[k]);
    }
    for (int i = v0 + (int)threadIdx.x + 256 * KEEP; i < v1; i += 256) {
        float r[V];
        read(i, r);
        write(i, r);
    }
}

// ---- residual + output norm + depth average -----------------------------------------------------------------------------
struct ResNormArgs {
    const float* y;        // [T, ldy] sublayer output
    const float* x;        // [T, W]   residual stream the sublayer has read
    const float* w;        // [W]      norm weight
    float* xs;             // [n, .]   results of the embedding and all layers so far, or null
    const float* dwa;      // [n]
    float* x_out;          // [T, W]
    void* h_out;           // [T, W] activation type, or null
    int64_t ldy, xs_stride;
    int n, keep, W;        // n = 0: no average; keep: store this layer's own result at xs[n - 1]
    float eps;
};

// A cluster of CTAs shares one row (column slices); the sum of squares is exchanged through distributed shared memory.
template <typename T, int V>
__global__ void __launch_bounds__(256) res_norm_kernel(const ResNormArgs a) {
    __shared__ float red[33];
    __shared__ float part;
    pdl_launch_dependents();
    pdl_wait();
    cg::cluster_group cl = cg::this_cluster();
    const int nc = (int)cl.num_blocks(), rank = (int)cl.block_rank();
    const int64_t t = blockIdx.x / nc;
    const int nv = a.W / V, per = (nv + nc - 1) / nc;
    const int v0 = rank * per, v1 = min(nv, v0 + per);
    const float* y = a.y + t * a.ldy;
    float ss = 0.0f;
    for (int i = v0 + (int)threadIdx.x; i < v1; i += 256) {
        if (V == 4) {
            const float4 q = *reinterpret_cast<const float4*>(y + 4 * i);
            ss += q.x * q.x + q.y * q.y + q.z * q.z + q.w * q.w;
        } else {
            ss += y[i] * y[i];
        }
    }
    ss = block_sumf(ss, red);
    if (nc > 1) {
        if (threadIdx.x == 0) part = ss;
        cl.sync();
        ss = 0.0f;
        for (int r = 0; r < nc; ++r) ss += *cl.map_shared_rank(&part, r);
        cl.sync();              // nobody leaves while its partial sum may still be read
    }
    const float inv = rms_inv_f32(ss, a.W, a.eps);
    const float self = a.n > 0 ? a.dwa[a.n - 1] : 1.0f;
    T* h = static_cast<T*>(a.h_out);
    for (int i = v0 + (int)threadIdx.x; i < v1; i += 256) {
        const int64_t o = t * a.W + (int64_t)V * i;
        float r[V];
        if (V == 4) {
            const float4 q = *reinterpret_cast<const float4*>(y + 4 * i), x = *reinterpret_cast<const float4*>(a.x + o);
            const float4 w = *reinterpret_cast<const float4*>(a.w + 4 * i);
            r[0] = x.x + q.x * inv * w.x;
            r[1 % V] = x.y + q.y * inv * w.y;
            r[2 % V] = x.z + q.z * inv * w.z;
            r[3 % V] = x.w + q.w * inv * w.w;
        } else {
            r[0] = a.x[o] + y[i] * inv * a.w[i];
        }
        if (a.n > 0) {
            float s[V];
#pragma unroll
            for (int e = 0; e < V; ++e) s[e] = 0.0f;
#pragma unroll 8
            for (int j = 0; j < a.n - 1; ++j) {
                const float c = a.dwa[j];
                if (V == 4) {
                    const float4 q = *reinterpret_cast<const float4*>(a.xs + j * a.xs_stride + o);
                    s[0] += c * q.x; s[1 % V] += c * q.y; s[2 % V] += c * q.z; s[3 % V] += c * q.w;
                } else {
                    s[0] += c * a.xs[j * a.xs_stride + o];
                }
            }
#pragma unroll
            for (int e = 0; e < V; ++e) {
                if (a.keep) a.xs[(a.n - 1) * a.xs_stride + o + e] = r[e];
                r[e] = s[e] + self * r[e];
            }
        }
        if (V == 4) {
            st4(a.x_out + o, r[0], r[1 % V], r[2 % V], r[3 % V]);
            if (h != nullptr) st4(h + o, r[0], r[1 % V], r[2 % V], r[3 % V]);
        } else {
            a.x_out[o] = r[0];
            if (h != nullptr) stf(h + o, r[0]);
        }
    }
}

// ---- row norm with gather -----------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) norm_rows_kernel(const float* x, const int64_t* rows, const float* w, float eps, int W, T* out) {
    __shared__ float red[33];
    pdl_launch_dependents();
    pdl_wait();
    const int64_t m = blockIdx.x, r = rows != nullptr ? rows[m] : m;
    const float* p = x + r * W;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < W; i += 256) ss += p[i] * p[i];
    const float inv = rms_inv_f32(block_sumf(ss, red), W, eps);
    for (int i = threadIdx.x; i < W; i += 256) stf(out + m * W + i, p[i] * inv * w[i]);
}

// ---- causal depthwise convolution + SiLU --------------------------------------------------------------------------------
constexpr int CONV_T = 8;       // tokens per thread

// TAPS > 0: two channels per thread, all inputs of the thread's tokens in registers; TAPS = 0: one channel, any number of taps.
template <typename T, int TAPS>
__global__ void __launch_bounds__(256) conv_silu_kernel(const T* x, int64_t ldx, int64_t n_tok, int C, int taps, const float* w,
                                                        const float* b, const float* tail, T* out, int64_t ldo) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t0 = (int64_t)blockIdx.y * CONV_T;
    const int64_t t1 = t0 + CONV_T < n_tok ? t0 + CONV_T : n_tok;
    if (TAPS > 0) {
        constexpr int W = CONV_T + (TAPS > 0 ? TAPS : 1) - 1;
        const int c = 2 * (blockIdx.x * 256 + threadIdx.x);
        if (c >= C) return;
        // C is even and rows are 2-element aligned (host side); a token before this portion lies in the carried tail
        float2 in[W];
        if (t0 >= TAPS - 1 && t1 == t0 + CONV_T) {
#pragma unroll
            for (int i = 0; i < W; ++i) {
                const T* p = x + (t0 - (TAPS - 1) + i) * ldx + c;
                if (sizeof(T) == 2) {
                    const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
                    in[i] = make_float2(bf16_lo(u), bf16_hi(u));
                } else {
                    in[i] = make_float2(ldf(p), ldf(p + 1));
                }
            }
        } else {
#pragma unroll
            for (int i = 0; i < W; ++i) {
                const int64_t t = t0 - (TAPS - 1) + i;
                in[i] = make_float2(0.0f, 0.0f);
                if (t >= 0 && t < t1) in[i] = make_float2(ldf(x + t * ldx + c), ldf(x + t * ldx + c + 1));
                if (t < 0) in[i] = make_float2(tail[(int64_t)c * (TAPS - 1) + t + TAPS - 1], tail[(int64_t)(c + 1) * (TAPS - 1) + t + TAPS - 1]);
            }
        }
        const float2 bias = b == nullptr ? make_float2(0.0f, 0.0f) : make_float2(b[c], b[c + 1]);
        float2 ww[TAPS > 0 ? TAPS : 1];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) ww[j] = make_float2(w[(int64_t)c * TAPS + j], w[(int64_t)(c + 1) * TAPS + j]);
#pragma unroll
        for (int i = 0; i < CONV_T; ++i) {
            if (t0 + i >= t1) break;
            float2 s = bias;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
                s.x = fmaf(ww[j].x, in[i + j].x, s.x);
                s.y = fmaf(ww[j].y, in[i + j].y, s.y);
            }
            T* o = out + (t0 + i) * ldo + c;
            if (sizeof(T) == 2) {
                *reinterpret_cast<uint32_t*>(o) = pack_bf16x2(silu_f32(s.x), silu_f32(s.y));
            } else {
                stf(o, silu_f32(s.x));
                stf(o + 1, silu_f32(s.y));
            }
        }
    } else {
        const int c = blockIdx.x * 256 + threadIdx.x;
        if (c >= C) return;
        for (int64_t t = t0; t < t1; ++t) {
            float s = b == nullptr ? 0.0f : b[c];
            for (int j = 0; j < taps; ++j) {
                const int64_t u = t - (taps - 1) + j;
                s = fmaf(w[(int64_t)c * taps + j], u >= 0 ? ldf(x + u * ldx + c) : tail[(int64_t)c * (taps - 1) + (u + taps - 1)], s);
            }
            stf(out + t * ldo + c, silu_f32(s));
        }
    }
}

// The last taps - 1 inputs, oldest first; a portion shorter than that keeps the younger part of the old tail.
template <typename T>
__global__ void __launch_bounds__(256) conv_tail_kernel(const T* x, int64_t ldx, int64_t n_tok, int C, int taps, float* tail) {
    pdl_launch_dependents();
    pdl_wait();
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (c >= C) return;
    float* tl = tail + (int64_t)c * (taps - 1);
    for (int j = 0; j < taps - 1; ++j) {
        const int64_t t = n_tok - (taps - 1) + j;      // ascending j: an old entry is read before it is overwritten
        tl[j] = t >= 0 ? ldf(x + t * ldx + c) : tl[t + taps - 1];
    }
}

// ---- per-head norm + gate -----------------------------------------------------------------------------------------------
// out[t, h, :] = o[t, h, :] / rms * w * gate(g[t, h, :]), gate = SiLU or the sigmoid; one warp per (token, head).
template <typename T, bool SIG>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* o, const T* g, int64_t ldg, const float* w, int64_t n, int H, int dv,
                                                             float eps, int vec, T* out) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t i = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (i >= n) return;
    const int lane = threadIdx.x & 31;
    const int64_t t = i / H;
    const int h = (int)(i - t * H);
    const float* p = o + i * dv;
    const T* gp = g + t * ldg + (int64_t)h * dv;
    auto gate = [](float z) { return SIG ? sigmoid_f32(z) : silu_f32(z); };
    float ss = 0.0f;
    if (vec) {                      // rows of four aligned values; up to 4 groups per lane stay in registers
        float4 v[4], gv[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int e = 4 * (lane + 32 * j);
            v[j] = e < dv ? *reinterpret_cast<const float4*>(p + e) : make_float4(0, 0, 0, 0);
            gv[j] = e < dv ? ld4(gp + e) : make_float4(0, 0, 0, 0);
            ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
        }
        const float inv = rms_inv_f32(warp_sumf(ss), dv, eps);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int e = 4 * (lane + 32 * j);
            if (e >= dv) continue;
            const float4 ww = w != nullptr ? *reinterpret_cast<const float4*>(w + e) : make_float4(1, 1, 1, 1);
            st4(out + i * dv + e, v[j].x * inv * ww.x * gate(gv[j].x), v[j].y * inv * ww.y * gate(gv[j].y), v[j].z * inv * ww.z * gate(gv[j].z),
                v[j].w * inv * ww.w * gate(gv[j].w));
        }
        return;
    }
    for (int e = lane; e < dv; e += 32) ss += p[e] * p[e];
    const float inv = rms_inv_f32(warp_sumf(ss), dv, eps);
    for (int e = lane; e < dv; e += 32) stf(out + i * dv + e, p[e] * inv * (w != nullptr ? w[e] : 1.0f) * gate(ldf(gp + e)));
}

// ---- xIELU of float32 values, in place ------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) xielu_kernel(float* x, int64_t n, float a_pos, float a_neg) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
    if (i < n) x[i] = xielu_f32(x[i], a_pos, a_neg);
}

// out[r, j] = gelu(gate) up of rows whose columns alternate 16 gate and 16 up values.
__global__ void __launch_bounds__(256) gated_gelu_kernel(const float* x, int64_t ldx, int64_t rows, int n, float* out) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= rows * n) return;
    const int64_t r = i / n;
    const int j = (int)(i - r * n);
    const float* p = x + r * ldx + 32 * (j >> 4) + (j & 15);
    out[i] = gelu_tanh_f32(p[0]) * p[16];
}

template <typename T>
static int run_add_norm(const AddNormArgs& a, int64_t T_, cudaStream_t st) {
    const int vec = (a.W % 4 == 0 && a.ldy % 4 == 0) ? 4 : 1;
    const int slices = (a.W / vec + 255) / 256;
    int nc = 1;
    while (nc < 8 && nc < slices && T_ * nc * 2 <= 148) nc *= 2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)(T_ * nc));
    cfg.blockDim = dim3(256);
    cfg.stream = st;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = nc;
    at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at;
    cfg.numAttrs = g_use_pdl ? 2 : 1;
    SCMX_PDL_OK("add_norm_kernel", vec == 4 ? cudaLaunchKernelEx(&cfg, add_norm_kernel<T, 4>, a)
                                            : cudaLaunchKernelEx(&cfg, add_norm_kernel<T, 1>, a));
    return SCMX_OK;
}

template <typename T>
static int run_res_norm(const ResNormArgs& a, int64_t T_, cudaStream_t st) {
    // few rows: a row is spread over a cluster so that the reads of all layers' results come from several SMs
    const int vec = (a.W % 4 == 0 && a.ldy % 4 == 0 && a.xs_stride % 4 == 0) ? 4 : 1;
    const int slices = (a.W / vec + 255) / 256;
    int nc = 1;
    while (nc < 8 && nc < slices && T_ * nc * 2 <= 148) nc *= 2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)(T_ * nc));
    cfg.blockDim = dim3(256);
    cfg.stream = st;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = nc;
    at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at;
    cfg.numAttrs = g_use_pdl ? 2 : 1;
    SCMX_PDL_OK("res_norm_kernel", vec == 4 ? cudaLaunchKernelEx(&cfg, res_norm_kernel<T, 4>, a)
                                            : cudaLaunchKernelEx(&cfg, res_norm_kernel<T, 1>, a));
    return SCMX_OK;
}

template <typename T>
static int run_conv(const T* x, int64_t ldx, int64_t n_tok, int C, int taps, const float* w, const float* b, float* tail, T* out,
                    int64_t ldo, cudaStream_t st) {
    const bool pairs = C % 2 == 0 && ldx % 2 == 0 && ldo % 2 == 0 && ((uintptr_t)x & 3) == 0 && taps <= 4;
    const int per = pairs ? 512 : 256;
    const dim3 grid((C + per - 1) / per, (unsigned)((n_tok + CONV_T - 1) / CONV_T)), block(256);
    const float* ct = tail;
    cudaError_t e;
#define CASE(n) case n: e = launch_pdl(conv_silu_kernel<T, n>, grid, block, 0, st, x, ldx, n_tok, C, taps, w, b, ct, out, ldo); break
    switch (pairs ? taps : 0) {
        CASE(1); CASE(2); CASE(3); CASE(4);
        default: e = launch_pdl(conv_silu_kernel<T, 0>, grid, block, 0, st, x, ldx, n_tok, C, taps, w, b, ct, out, ldo);
    }
#undef CASE
    SCMX_PDL_OK("conv_silu_kernel", e);
    if (taps > 1)
        SCMX_PDL_OK("conv_tail_kernel", launch_pdl(conv_tail_kernel<T>, dim3((C + 255) / 256), block, 0, st, x, ldx, n_tok, C, taps, tail));
    return SCMX_OK;
}

}  // namespace scmx

using namespace scmx;

extern "C" int scmx_embed(const int64_t* tokens, const void* table, int dt, int64_t V, int64_t T, int W, float* x, void* h, void* stream) {
    SCMX_DT_OK("embed", dt);
    SCMX_REQUIRE(tokens && table && x && V > 0 && T >= 0 && W > 0, SCMX_EINVAL, "embed: bad argument");
    if (T == 0) return SCMX_OK;
    const cudaStream_t st = (cudaStream_t)stream;
    if (dt == 0)
        SCMX_PDL_OK("embed_kernel", launch_pdl(embed_kernel<bf16_t>, dim3((unsigned)T), dim3(256), 0, st, tokens, (const bf16_t*)table, V, W, x, (bf16_t*)h));
    else
        SCMX_PDL_OK("embed_kernel", launch_pdl(embed_kernel<float>, dim3((unsigned)T), dim3(256), 0, st, tokens, (const float*)table, V, W, x, (float*)h));
    return SCMX_OK;
}

extern "C" int scmx_res_norm(const float* y, int64_t ldy, const float* x, const float* w, float eps, int64_t T, int W, float* xs,
                             int64_t xs_stride, const float* dwa, int n, int keep, float* x_out, void* h_out, int dt, void* stream) {
    SCMX_DT_OK("res_norm", dt);
    SCMX_REQUIRE(y && x && w && x_out && T >= 0 && W > 0 && ldy >= W, SCMX_EINVAL, "res_norm: bad argument");
    SCMX_REQUIRE(n >= 0 && (n == 0 || (xs && dwa && xs_stride >= T * W)), SCMX_EINVAL, "res_norm: average over %d results without a store", n);
    if (T == 0) return SCMX_OK;
    ResNormArgs a;
    a.y = y; a.x = x; a.w = w; a.xs = xs; a.dwa = dwa; a.x_out = x_out; a.h_out = h_out;
    a.ldy = ldy; a.xs_stride = xs_stride; a.n = n; a.keep = keep; a.W = W; a.eps = eps;
    return dt == 0 ? run_res_norm<bf16_t>(a, T, (cudaStream_t)stream) : run_res_norm<float>(a, T, (cudaStream_t)stream);
}

extern "C" int scmx_norm_rows(const float* x, const int64_t* rows, const float* w, float eps, int64_t M, int W, void* out, int dt, void* stream) {
    SCMX_DT_OK("norm_rows", dt);
    SCMX_REQUIRE(x && w && out && M >= 0 && W > 0, SCMX_EINVAL, "norm_rows: bad argument");
    if (M == 0) return SCMX_OK;
    const cudaStream_t st = (cudaStream_t)stream;
    if (dt == 0)
        SCMX_PDL_OK("norm_rows_kernel", launch_pdl(norm_rows_kernel<bf16_t>, dim3((unsigned)M), dim3(256), 0, st, x, rows, w, eps, W, (bf16_t*)out));
    else
        SCMX_PDL_OK("norm_rows_kernel", launch_pdl(norm_rows_kernel<float>, dim3((unsigned)M), dim3(256), 0, st, x, rows, w, eps, W, (float*)out));
    return SCMX_OK;
}

extern "C" int scmx_conv_silu(const void* x, int64_t ldx, int dt, int64_t T, int C, int taps, const float* w, const float* b, float* tail,
                              void* out, int64_t ldo, void* stream) {
    SCMX_DT_OK("conv_silu", dt);
    SCMX_REQUIRE(x && w && out && T >= 0 && C > 0 && taps >= 1 && ldx >= C && ldo >= C, SCMX_EINVAL, "conv_silu: bad argument");
    SCMX_REQUIRE(taps == 1 || tail != nullptr, SCMX_EINVAL, "conv_silu: %d taps need the carried inputs", taps);
    if (T == 0) return SCMX_OK;
    if (dt == 0) return run_conv((const bf16_t*)x, ldx, T, C, taps, w, b, tail, (bf16_t*)out, ldo, (cudaStream_t)stream);
    return run_conv((const float*)x, ldx, T, C, taps, w, b, tail, (float*)out, ldo, (cudaStream_t)stream);
}

extern "C" int scmx_embed_pair(const int64_t* tokens, const void* table, const void* pairs, int dt, int64_t V, int64_t T, int W, float scale,
                               int64_t buckets, int64_t mul_prev, int64_t mul_cur, int64_t* prev, float* x, void* stream) {
    SCMX_DT_OK("embed_pair", dt);
    SCMX_REQUIRE(tokens && table && x && V > 0 && T >= 0 && W > 0, SCMX_EINVAL, "embed_pair: bad argument");
    SCMX_REQUIRE(pairs == nullptr || (prev && buckets > 0), SCMX_EINVAL, "embed_pair: a pair table needs buckets and the token before");
    if (T == 0) return SCMX_OK;
    EmbedPairArgs a;
    a.tok = tokens; a.prev = prev; a.x = x; a.V = V; a.T = T; a.buckets = buckets; a.mul_prev = mul_prev; a.mul_cur = mul_cur; a.W = W; a.scale = scale;
    const cudaStream_t st = (cudaStream_t)stream;
    if (dt == 0)
        SCMX_PDL_OK("embed_pair_kernel", launch_pdl(embed_pair_kernel<bf16_t>, dim3((unsigned)T), dim3(256), 0, st, (const bf16_t*)table, (const bf16_t*)pairs, a));
    else
        SCMX_PDL_OK("embed_pair_kernel", launch_pdl(embed_pair_kernel<float>, dim3((unsigned)T), dim3(256), 0, st, (const float*)table, (const float*)pairs, a));
    return SCMX_OK;
}

extern "C" int scmx_add_norm(const float* y, int64_t ldy, const float* x, const float* w, float mult, float eps, int64_t T, int W, float* x_out,
                             void* h_out, int dt, void* stream) {
    SCMX_DT_OK("add_norm", dt);
    SCMX_REQUIRE(x && w && h_out && T >= 0 && W > 0, SCMX_EINVAL, "add_norm: bad argument");
    SCMX_REQUIRE(y == nullptr || (x_out && ldy >= W), SCMX_EINVAL, "add_norm: a sublayer's output needs a pitch and a place for the sum");
    if (T == 0) return SCMX_OK;
    AddNormArgs a;
    a.y = y; a.x = x; a.w = w; a.x_out = y != nullptr ? x_out : nullptr; a.h_out = h_out; a.ldy = y != nullptr ? ldy : 0; a.W = W; a.mult = mult; a.eps = eps;
    return dt == 0 ? run_add_norm<bf16_t>(a, T, (cudaStream_t)stream) : run_add_norm<float>(a, T, (cudaStream_t)stream);
}

extern "C" int scmx_head_norm_gate(const float* o, const void* g, int64_t ldg, int dt, const float* w, int gate, int64_t T, int H, int dv, float eps,
                                   void* out, void* stream) {
    SCMX_DT_OK("head_norm_gate", dt);
    SCMX_REQUIRE(o && g && out && T >= 0 && H > 0 && dv > 0 && ldg >= (int64_t)H * dv, SCMX_EINVAL, "head_norm_gate: bad argument");
    SCMX_REQUIRE(gate == 0 || gate == 1, SCMX_EINVAL, "head_norm_gate: gate=%d (0 = SiLU, 1 = sigmoid)", gate);
    if (T == 0) return SCMX_OK;
    const int64_t n = T * H;
    const int esz = dt == 0 ? 2 : 4;
    const int vec = dv % 4 == 0 && dv <= 512 && ldg % 4 == 0 && (uintptr_t)g % (4 * esz) == 0 && (uintptr_t)w % 16 == 0;
    const dim3 grid((unsigned)((n + 7) / 8)), block(256);
    const cudaStream_t st = (cudaStream_t)stream;
#define GO(T_, S_) SCMX_PDL_OK("head_norm_gate_kernel", launch_pdl(head_norm_gate_kernel<T_, S_>, grid, block, 0, st, o, (const T_*)g, ldg, w, n, H, dv, eps, vec, (T_*)out))
    if (dt == 0 && gate == 0) GO(bf16_t, false);
    else if (dt == 0) GO(bf16_t, true);
    else if (gate == 0) GO(float, false);
    else GO(float, true);
#undef GO
    return SCMX_OK;
}

extern "C" int scmx_gated_gelu(const float* x, int64_t ldx, int64_t rows, int n, float* out, void* stream) {
    SCMX_REQUIRE(x && out && rows >= 0 && n > 0 && n % 16 == 0 && ldx >= 2 * n, SCMX_EINVAL, "gated_gelu: %d outputs per row", n);
    if (rows == 0) return SCMX_OK;
    SCMX_PDL_OK("gated_gelu_kernel", launch_pdl(gated_gelu_kernel, dim3((unsigned)((rows * n + 255) / 256)), dim3(256), 0, (cudaStream_t)stream, x, ldx, rows, n, out));
    return SCMX_OK;
}

extern "C" int scmx_xielu(float* x, int64_t n, float a_pos, float a_neg, void* stream) {
    SCMX_REQUIRE(x && n >= 0, SCMX_EINVAL, "xielu: bad argument");
    if (n == 0) return SCMX_OK;
    SCMX_PDL_OK("xielu_kernel", launch_pdl(xielu_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, (cudaStream_t)stream, x, n, a_pos, a_neg));
    return SCMX_OK;
}
