// Selective scan (Mamba): per channel c and state n, S <- exp(dt_c A[c, n]) S + dt_c x_c B_n, y_c = sum_n S C_n + D_c x_c, then
// y silu(z).  The recurrence is float32 throughout; the state is carried between calls.
//
// Prefill: a group of `lpc` lanes owns one channel and walks the whole portion, NS states per lane in registers, so the
// exponentials are evaluated once and the state never leaves the SM.  Tiles of tokens are double-staged: the global loads
// of the next tile are in flight in registers while the current one is consumed from shared memory.
// Decode: one token; the step-size projection (dt_rank inputs) is part of the kernel.
#include "mix_common.cuh"

namespace scmx {

constexpr int SC_THREADS = 128;

template <typename T>
struct ScanArgs {
    const T* x;            // [n, ldx] convolved input
    const float* dtp;      // [n, ldt] step size before bias and softplus
    const T* bc;           // [n, ldbc]: B at column 0, C at column N
    const T* z;            // [n, ldz] gate
    const float* dt_bias;  // [C]
    const float* A2;       // [C, N]: -exp(A_log) log2(e)
    const float* D;        // [C]
    float* state;          // [C, N]
    T* y;                  // [n, ldy]
    int64_t n, ldx, ldt, ldbc, ldz, ldy;
    int C, N;
};

// NS states per lane, LPC lanes per channel (a power of two), N <= NS * LPC.
template <typename T, int NS, int LPC>
__global__ void __launch_bounds__(SC_THREADS) scan_kernel(const ScanArgs<T> a) {
    constexpr int CPC = SC_THREADS / LPC;         // channels per CTA
    constexpr int NP = NS * LPC;                  // padded states
    constexpr int SC_T = NP > 128 ? 16 : 32;      // tokens per tile
    constexpr int XE = (SC_T * CPC + SC_THREADS - 1) / SC_THREADS;      // staged x / dt / z values per thread and tile
    constexpr int BE = (SC_T * NP + SC_THREADS - 1) / SC_THREADS;
    __shared__ __align__(16) float2 sd[SC_T][CPC];       // step, step * x
    __shared__ __align__(16) float2 so[SC_T][CPC];       // D x, silu(z)
    __shared__ __align__(16) float sB[SC_T][NP], sC[SC_T][NP];
    __shared__ float sy[SC_T][CPC + 1];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid % LPC, ch = tid / LPC;
    const int c0 = blockIdx.x * CPC, c = c0 + ch;
    float S[NS], A2[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int n = lane * NS + i;
        A2[i] = (c < a.C && n < a.N) ? a.A2[(int64_t)c * a.N + n] : 0.0f;
    }
    pdl_wait();
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int n = lane * NS + i;
        S[i] = (c < a.C && n < a.N) ? a.state[(int64_t)c * a.N + n] : 0.0f;
    }
    // what this thread stages: column fc of rows fr, fr + FS, ...
    constexpr int FS = SC_THREADS / CPC;          // = LPC rows per sweep
    const int fc = tid % CPC, fr = tid / CPC;
    const bool fok = c0 + fc < a.C;
    const float bias = fok ? a.dt_bias[c0 + fc] : 0.0f, Dc = fok ? a.D[c0 + fc] : 0.0f;
    float pd[XE];
    T px[XE], pz[XE], pB[BE], pC[BE];       // as stored: converted when staged, so that the loads stay in flight
    auto fetch = [&](int64_t t0) {
#pragma unroll
        for (int i = 0; i < XE; ++i) {
            const int64_t t = t0 + fr + i * FS;
            const bool ok = fok && fr + i * FS < SC_T && t < a.n;
            px[i] = ok ? a.x[t * a.ldx + c0 + fc] : T(0);
            pd[i] = ok ? a.dtp[t * a.ldt + c0 + fc] : 0.0f;
            pz[i] = ok ? a.z[t * a.ldz + c0 + fc] : T(0);
        }
#pragma unroll
        for (int i = 0; i < BE; ++i) {
            const int e = tid + i * SC_THREADS, r = e / NP, n = e % NP;
            const int64_t t = t0 + r;
            const bool ok = r < SC_T && n < a.N && t < a.n;
            pB[i] = ok ? a.bc[t * a.ldbc + n] : T(0);
            pC[i] = ok ? a.bc[t * a.ldbc + a.N + n] : T(0);
        }
    };
    fetch(0);
    for (int64_t t0 = 0; t0 < a.n; t0 += SC_T) {
#pragma unroll
        for (int i = 0; i < XE; ++i) {
            const int r = fr + i * FS;
            if (r >= SC_T) break;
            // a zero step leaves the state unchanged
            const float step = t0 + r < a.n ? softplus_f32(pd[i] + bias) : 0.0f, x = ldf(&px[i]);
            sd[r][fc] = make_float2(step, step * x);
            so[r][fc] = make_float2(Dc * x, silu_f32(ldf(&pz[i])));
        }
#pragma unroll
        for (int i = 0; i < BE; ++i) {
            const int e = tid + i * SC_THREADS;
            if (e < SC_T * NP) {
                sB[e / NP][e % NP] = ldf(&pB[i]);
                sC[e / NP][e % NP] = ldf(&pC[i]);
            }
        }
        __syncthreads();
        if (t0 + SC_T < a.n) fetch(t0 + SC_T);
        // eight tokens at a time: everything but the chain through S is independent; the partial outputs of the channel's lanes
        // are summed by halving (a lane keeps half of the tokens and hands over the other half), 7 shuffles for 8 tokens
#pragma unroll 1
        for (int r0 = 0; r0 < SC_T; r0 += 8) {
            float y[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const float2 d = sd[r0 + u][ch];
                y[u] = 0.0f;
#pragma unroll
                for (int i = 0; i < NS; ++i) {
                    S[i] = fmaf(ex2_approx(d.x * A2[i]), S[i], d.y * sB[r0 + u][lane * NS + i]);
                    y[u] = fmaf(S[i], sC[r0 + u][lane * NS + i], y[u]);
                }
            }
            int first = 0;                  // the token(s) whose sum this lane ends up with
#pragma unroll
            for (int o = 1, cnt = 8; o < LPC; o *= 2) {
                if (cnt > 1) {
                    cnt /= 2;
                    const bool up = lane & o;
#pragma unroll
                    for (int u = 0; u < cnt; ++u) {
                        const float give = up ? y[u] : y[u + cnt], keep = up ? y[u + cnt] : y[u];
                        y[u] = keep + __shfl_xor_sync(0xffffffffu, give, o);
                    }
                    first += up ? cnt : 0;
                } else {
                    y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
                }
            }
            constexpr int OUT = LPC >= 8 ? 1 : 8 / LPC;
            if (lane < 8)
#pragma unroll
                for (int u = 0; u < OUT; ++u) sy[r0 + first + u][ch] = y[u];
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < XE; ++i) {
            const int r = fr + i * FS;
            const int64_t t = t0 + r;
            if (fok && r < SC_T && t < a.n) stf(a.y + t * a.ldy + c0 + fc, (sy[r][fc] + so[r][fc].x) * so[r][fc].y);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int n = lane * NS + i;
        if (c < a.C && n < a.N) a.state[(int64_t)c * a.N + n] = S[i];
    }
}

// ---- one token ------------------------------------------------------------------------------------------------------------
struct ScanStepArgs {
    const float* x;         // [C] convolved input
    const float* z;         // [C]
    const float* dbc;       // [R + 2 N]: step-size inputs, B, C
    const void* w_dt;       // [C, ldw] weight type
    const float *dt_bias, *A2, *D;
    float* state;
    float* y;               // [C]
    int64_t ldw;
    int C, N, R;
};

constexpr int SS_LANES = 8;       // lanes per channel

template <typename T>
__global__ void __launch_bounds__(256) scan_step_kernel(const ScanStepArgs a) {
    extern __shared__ float sdbc[];
    pdl_launch_dependents();
    const int lane = threadIdx.x % SS_LANES;
    const int c = blockIdx.x * (256 / SS_LANES) + threadIdx.x / SS_LANES;
    const bool ok = c < a.C;
    pdl_wait();
    for (int i = threadIdx.x; i < a.R + 2 * a.N; i += 256) sdbc[i] = a.dbc[i];
    __syncthreads();
    float dt = 0.0f;
    if (ok) {
        const T* w = static_cast<const T*>(a.w_dt) + (int64_t)c * a.ldw;
        for (int k = lane * 8; k < a.R; k += SS_LANES * 8) {      // rows are padded to a multiple of 8 inputs with zeros
            float v[8];
            ld8(w + k, v);
#pragma unroll
            for (int i = 0; i < 8; ++i)
                if (k + i < a.R) dt = fmaf(v[i], sdbc[k + i], dt);
        }
    }
#pragma unroll
    for (int o = SS_LANES / 2; o > 0; o >>= 1) dt += __shfl_xor_sync(0xffffffffu, dt, o);
    dt = ok ? softplus_f32(dt + a.dt_bias[c]) : 0.0f;
    const float x = ok ? a.x[c] : 0.0f, dx = dt * x;
    float y = 0.0f;
    if (ok) {
        float* S = a.state + (int64_t)c * a.N;
        for (int n = lane; n < a.N; n += SS_LANES) {
            const float s = fmaf(ex2_approx(dt * a.A2[(int64_t)c * a.N + n]), S[n], dx * sdbc[a.R + n]);
            S[n] = s;
            y = fmaf(s, sdbc[a.R + a.N + n], y);
        }
    }
#pragma unroll
    for (int o = SS_LANES / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (ok && lane == 0) a.y[c] = (y + a.D[c] * x) * silu_f32(a.z[c]);
}

template <typename T, int NS>
static cudaError_t launch_scan(const ScanArgs<T>& a, int lpc, cudaStream_t st) {
    const int cpc = SC_THREADS / lpc;
    const dim3 grid((unsigned)((a.C + cpc - 1) / cpc)), block(SC_THREADS);
    switch (lpc) {
        case 4: return launch_pdl(scan_kernel<T, NS, 4>, grid, block, 0, st, a);
        case 8: return launch_pdl(scan_kernel<T, NS, 8>, grid, block, 0, st, a);
        case 16: return launch_pdl(scan_kernel<T, NS, 16>, grid, block, 0, st, a);
        default: return launch_pdl(scan_kernel<T, NS, 32>, grid, block, 0, st, a);
    }
}

template <typename T>
static int run_scan(const ScanArgs<T>& a, cudaStream_t st) {
    // the fewest padded states, 4 states per lane at most while 32 lanes suffice
    int best_ns = 0, best_lpc = 32, best_pad = 1 << 30;
    for (int ns = 4; ns >= 2; --ns) {
        int lpc = 4;
        while (lpc < 32 && ns * lpc < a.N) lpc *= 2;
        if (ns * lpc >= a.N && ns * lpc < best_pad) { best_ns = ns; best_lpc = lpc; best_pad = ns * lpc; }
    }
    if (best_ns == 0) best_ns = 8;
    cudaError_t e = best_ns == 2 ? launch_scan<T, 2>(a, best_lpc, st)
                  : best_ns == 3 ? launch_scan<T, 3>(a, best_lpc, st)
                  : best_ns == 4 ? launch_scan<T, 4>(a, best_lpc, st) : launch_pdl(scan_kernel<T, 8, 32>, dim3((a.C + 3) / 4), dim3(SC_THREADS), 0, st, a);
    SCMX_PDL_OK("scan_kernel", e);
    return SCMX_OK;
}

}  // namespace scmx

using namespace scmx;

extern "C" int scmx_selective_scan(const void* x, int64_t ldx, const float* dtp, int64_t ldt, const void* bc, int64_t ldbc, const void* z,
                                   int64_t ldz, int dt, int64_t n, int C, int N, const float* dt_bias, const float* A2, const float* D,
                                   float* state, void* y, int64_t ldy, void* stream) {
    SCMX_DT_OK("selective_scan", dt);
    SCMX_REQUIRE(x && dtp && bc && z && dt_bias && A2 && D && state && y, SCMX_EINVAL, "selective_scan: null buffer");
    SCMX_REQUIRE(n >= 0 && C > 0 && N > 0 && ldx >= C && ldt >= C && ldz >= C && ldy >= C && ldbc >= 2 * N, SCMX_EINVAL,
                 "selective_scan: n=%lld C=%d N=%d", (long long)n, C, N);
    SCMX_REQUIRE(N <= 256, SCMX_ELIMIT, "selective_scan: %d states per channel (256 at most)", N);
    if (n == 0) return SCMX_OK;
#define FILL(T)                                                                                                              \
    ScanArgs<T> a;                                                                                                            \
    a.x = (const T*)x; a.dtp = dtp; a.bc = (const T*)bc; a.z = (const T*)z; a.dt_bias = dt_bias; a.A2 = A2; a.D = D;          \
    a.state = state; a.y = (T*)y; a.n = n; a.ldx = ldx; a.ldt = ldt; a.ldbc = ldbc; a.ldz = ldz; a.ldy = ldy; a.C = C; a.N = N
    if (dt == 0) {
        FILL(bf16_t);
        return run_scan<bf16_t>(a, (cudaStream_t)stream);
    }
    FILL(float);
    return run_scan<float>(a, (cudaStream_t)stream);
#undef FILL
}

extern "C" int scmx_scan_step(const float* x, const float* z, const float* dbc, const void* w_dt, int64_t ldw, int dt, int C, int N, int R,
                              const float* dt_bias, const float* A2, const float* D, float* state, float* y, void* stream) {
    SCMX_DT_OK("scan_step", dt);
    SCMX_REQUIRE(x && z && dbc && w_dt && dt_bias && A2 && D && state && y, SCMX_EINVAL, "scan_step: null buffer");
    SCMX_REQUIRE(C > 0 && N > 0 && R > 0 && ldw >= R && ldw % 8 == 0, SCMX_EINVAL, "scan_step: C=%d N=%d R=%d ldw=%lld", C, N, R, (long long)ldw);
    const size_t smem = (size_t)(R + 2 * N) * 4;
    SCMX_REQUIRE(smem <= 48 * 1024, SCMX_ELIMIT, "scan_step: %d step inputs and %d states do not fit shared memory", R, N);
    ScanStepArgs a;
    a.x = x; a.z = z; a.dbc = dbc; a.w_dt = w_dt; a.dt_bias = dt_bias; a.A2 = A2; a.D = D; a.state = state; a.y = y;
    a.ldw = ldw; a.C = C; a.N = N; a.R = R;
    const dim3 grid((unsigned)((C + 256 / SS_LANES - 1) / (256 / SS_LANES))), block(256);
    SCMX_PDL_OK("scan_step_kernel", dt == 0 ? launch_pdl(scan_step_kernel<bf16_t>, grid, block, smem, (cudaStream_t)stream, a)
                                            : launch_pdl(scan_step_kernel<float>, grid, block, smem, (cudaStream_t)stream, a));
    return SCMX_OK;
}
