// Matrix-vector product of the decode step: out [N] = W [N, K] x, weights bfloat16 or float, x and out float32, float32
// accumulation.  Each warp owns two rows (or a slice of their columns) and keeps up to 16 weight loads of 16 bytes per lane in
// flight; the first batch is issued before the previous kernel of the chain has finished (weights never change).
// Epilogues: none; xIELU; the causal convolution + SiLU of the first C rows, whose carried inputs are shifted in place; gelu(gate) up
// of rows that alternate 16 gate and 16 up rows (a warp owns one of each).
#include "mix_common.cuh"

namespace scmx {

struct GvArgs {
    const void* W;          // [N, ldw], zero padded to a multiple of 8 columns
    const float* x;         // [K]
    float* out;             // [N]
    int64_t ldw;
    int N, K, ks;           // ks: warps that share a row (1, 2, 4 or 8)
    float a_pos, a_neg;     // xIELU
    const float *cw, *cb;   // convolution weights [C, taps] and bias [C]
    float* tail;            // [C, taps - 1]
    int C, taps;
};

constexpr int GV_ROWS = 2;

template <typename T> struct Vec8;
template <> struct Vec8<bf16_t> {
    uint4 w;
    __device__ __forceinline__ void load(const bf16_t* p) { w = __ldg(reinterpret_cast<const uint4*>(p)); }
    __device__ __forceinline__ void zero() { w = make_uint4(0, 0, 0, 0); }
    __device__ __forceinline__ float dot(float4 lo, float4 hi, float s) const {
        s = fmaf(bf16_lo(w.x), lo.x, s); s = fmaf(bf16_hi(w.x), lo.y, s); s = fmaf(bf16_lo(w.y), lo.z, s); s = fmaf(bf16_hi(w.y), lo.w, s);
        s = fmaf(bf16_lo(w.z), hi.x, s); s = fmaf(bf16_hi(w.z), hi.y, s); s = fmaf(bf16_lo(w.w), hi.z, s); s = fmaf(bf16_hi(w.w), hi.w, s);
        return s;
    }
};
template <> struct Vec8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) {
        a = __ldg(reinterpret_cast<const float4*>(p));
        b = __ldg(reinterpret_cast<const float4*>(p) + 1);
    }
    __device__ __forceinline__ void zero() { a = b = make_float4(0, 0, 0, 0); }
    __device__ __forceinline__ float dot(float4 lo, float4 hi, float s) const {
        s = fmaf(a.x, lo.x, s); s = fmaf(a.y, lo.y, s); s = fmaf(a.z, lo.z, s); s = fmaf(a.w, lo.w, s);
        s = fmaf(b.x, hi.x, s); s = fmaf(b.y, hi.y, s); s = fmaf(b.z, hi.z, s); s = fmaf(b.w, hi.w, s);
        return s;
    }
};

template <typename T, int EPI>
__global__ void __launch_bounds__(256) gemv_x_kernel(const GvArgs a) {
    constexpr int U = sizeof(T) == 2 ? 8 : 4;          // vectors per lane and row in flight
    extern __shared__ __align__(16) float4 xs[];       // [2][nv]: elements 0..3 and 4..7 of every vector of 8
    __shared__ float part[8][GV_ROWS];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int nv = (a.K + 7) >> 3, ks = a.ks;
    const int r0 = (blockIdx.x * (8 / ks) + warp / ks) * GV_ROWS, first = (warp % ks) * 32 + lane, step = 32 * ks;
    const T* W = static_cast<const T*>(a.W);
    auto row_of = [&](int r) { return EPI == 3 ? 32 * (r0 >> 5) + ((r0 >> 1) & 15) + 16 * r : r0 + r; };
    Vec8<T> w[GV_ROWS][U];
    auto fetch = [&](int v0) {
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int r = 0; r < GV_ROWS; ++r) {
                const int v = v0 + u * step;
                if (v < nv && r0 + r < a.N) w[r][u].load(W + (int64_t)row_of(r) * a.ldw + 8 * (int64_t)v);
                else w[r][u].zero();
            }
    };
    fetch(first);
    pdl_wait();
    if ((a.K & 3) == 0 && ((uintptr_t)a.x & 15) == 0) {
#pragma unroll 8
        for (int i = tid; i < 2 * nv; i += 256)
            xs[(i & 1) * nv + (i >> 1)] = 4 * i < a.K ? *reinterpret_cast<const float4*>(a.x + 4 * i) : make_float4(0, 0, 0, 0);
    } else {
        for (int i = tid; i < nv * 8; i += 256) {
            const float x = i < a.K ? a.x[i] : 0.0f;
            reinterpret_cast<float*>(xs + ((i >> 2) & 1) * nv + (i >> 3))[i & 3] = x;
        }
    }
    __syncthreads();
    float s[GV_ROWS] = {};
    for (int v0 = first; v0 < nv; v0 += U * step) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int v = v0 + u * step;
            if (v < nv) {
                const float4 lo = xs[v], hi = xs[nv + v];
#pragma unroll
                for (int r = 0; r < GV_ROWS; ++r) s[r] = w[r][u].dot(lo, hi, s[r]);
            }
        }
        if (v0 + U * step < nv) fetch(v0 + U * step);
    }
#pragma unroll
    for (int r = 0; r < GV_ROWS; ++r) s[r] = warp_sumf(s[r]);
    if (ks > 1) {
        if (lane == 0)
#pragma unroll
            for (int r = 0; r < GV_ROWS; ++r) part[warp][r] = s[r];
        __syncthreads();
        if (warp % ks) return;
#pragma unroll
        for (int r = 0; r < GV_ROWS; ++r) {
            s[r] = 0.0f;
            for (int i = 0; i < ks; ++i) s[r] += part[warp + i][r];
        }
    }
    if (EPI == 3) {
        if (lane == 0 && r0 < a.N) a.out[r0 >> 1] = gelu_tanh_f32(s[0]) * s[1];
        return;
    }
    const int row = r0 + lane;
    if (lane >= GV_ROWS || row >= a.N) return;
    float y = lane == 0 ? s[0] : s[1];
    if (EPI == 1) y = xielu_f32(y, a.a_pos, a.a_neg);
    if (EPI == 2 && row < a.C) {
        const float* cw = a.cw + (int64_t)row * a.taps;
        float* tl = a.tail + (int64_t)row * (a.taps - 1);
        float c = fmaf(cw[a.taps - 1], y, a.cb == nullptr ? 0.0f : a.cb[row]);
        for (int j = 0; j < a.taps - 1; ++j) {
            c = fmaf(cw[j], tl[j], c);
            tl[j] = j + 1 < a.taps - 1 ? tl[j + 1] : y;
        }
        y = silu_f32(c);
    }
    a.out[row] = y;
}

template <typename T>
static int run_gemv(GvArgs a, int epi, cudaStream_t st) {
    const int nv = (a.K + 7) / 8;
    const size_t smem = (size_t)nv * 32;
    SCMX_REQUIRE(smem <= 200 * 1024, SCMX_ELIMIT, "gemv_x: K=%d", a.K);
    int ks = 1;                                        // enough CTAs for every SM, at least a few vectors per lane
    while (ks < 8 && (a.N + 16 / ks - 1) / (16 / ks) < 2 * sm_count() && nv > 64 * ks) ks *= 2;
    a.ks = ks;
    const int rows = 8 / ks * GV_ROWS;
    const dim3 grid((unsigned)((a.N + rows - 1) / rows)), block(256);
    auto kernel = epi == 0 ? gemv_x_kernel<T, 0> : epi == 1 ? gemv_x_kernel<T, 1> : epi == 2 ? gemv_x_kernel<T, 2> : gemv_x_kernel<T, 3>;
    if (smem > 40 * 1024) SCMX_CUDA_OK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    SCMX_PDL_OK("gemv_x_kernel", launch_pdl(kernel, grid, block, smem, st, a));
    return SCMX_OK;
}

}  // namespace scmx

using namespace scmx;

extern "C" int scmx_gemv_x(const void* W, int64_t ldw, int dt, const float* x, int64_t N, int64_t K, int epi, float a_pos, float a_neg,
                           const float* conv_w, const float* conv_b, float* tail, int C, int taps, float* out, void* stream) {
    SCMX_DT_OK("gemv_x", dt);
    SCMX_REQUIRE(W && x && out && N > 0 && K > 0 && N < (1ll << 30) && K < (1ll << 30), SCMX_EINVAL, "gemv_x: N=%lld K=%lld", (long long)N, (long long)K);
    SCMX_REQUIRE(ldw % 8 == 0 && ldw >= K && ((uintptr_t)W & 15) == 0, SCMX_EINVAL, "gemv_x: row pitch %lld", (long long)ldw);
    SCMX_REQUIRE(epi >= 0 && epi <= 3 && (epi != 3 || N % 32 == 0), SCMX_EINVAL, "gemv_x: epi=%d on %lld rows", epi, (long long)N);
    SCMX_REQUIRE(epi != 2 || (conv_w && C > 0 && C <= N && taps >= 1 && (taps == 1 || tail)), SCMX_EINVAL, "gemv_x: convolution epilogue");
    GvArgs a;
    a.W = W; a.x = x; a.out = out; a.ldw = ldw; a.N = (int)N; a.K = (int)K; a.ks = 1; a.a_pos = a_pos; a.a_neg = a_neg;
    a.cw = conv_w; a.cb = conv_b; a.tail = tail; a.C = C; a.taps = taps;
    return dt == 0 ? run_gemv<bf16_t>(a, epi, (cudaStream_t)stream) : run_gemv<float>(a, epi, (cudaStream_t)stream);
}
