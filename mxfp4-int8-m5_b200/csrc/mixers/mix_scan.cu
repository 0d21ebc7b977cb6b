// Selective scan (Mamba): per channel c and state n, S <- exp(dt_c A[c, n]) S + dt_c x_c B_n, y_c = sum_n S C_n + D_c x_c, then
// y silu(z).  The recurrence is float32 throughout; the state is carried between calls.
//
// Prefill: a group of `lpc` lanes owns one channel and walks the whole portion, NS states per lane in registers, so the
// exponentials are evaluated once and the state never leaves the SM.  8 warps of a CTA run the recurrence; 8 more load the tiles,
// apply softplus and SiLU, and write the gated outputs, one tile ahead and one behind, through double-buffered shared memory.
// Decode: one token; the step-size projection (dt_rank inputs) is part of the kernel.
#include "mix_common.cuh"

namespace scmx {

constexpr int SC_THREADS = 256;       // recurrence
constexpr int SC_STAGERS = 256;       // loads, activations, stores

// ex2_approx that the compiler keeps in program order.
__device__ __forceinline__ float ex2_ordered(float x) {
    float y;
    asm volatile("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

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
    int pairs, bc_pairs;   // two neighbouring channels (states) can be read with one load
};

// Two neighbouring values as stored; aligned: as one load.
template <typename T> struct Pair;
template <> struct Pair<bf16_t> {
    uint32_t w;
    __device__ __forceinline__ void load(const bf16_t* p, bool two, bool aligned) {
        if (aligned) w = *reinterpret_cast<const uint32_t*>(p);
        else w = (uint32_t)p[0] | (two ? (uint32_t)p[1] << 16 : 0u);
    }
    __device__ __forceinline__ void zero() { w = 0; }
    __device__ __forceinline__ float2 get() const { return make_float2(bf16_lo(w), bf16_hi(w)); }
};
template <> struct Pair<float> {
    float2 w;
    __device__ __forceinline__ void load(const float* p, bool two, bool aligned) {
        if (aligned) w = *reinterpret_cast<const float2*>(p);
        else w = make_float2(p[0], two ? p[1] : 0.0f);
    }
    __device__ __forceinline__ void zero() { w = make_float2(0, 0); }
    __device__ __forceinline__ float2 get() const { return w; }
};

// NS states per lane, LPC lanes per channel (a power of two, >= 4), N <= NS * LPC.
template <typename T, int NS, int LPC>
__global__ void __launch_bounds__(SC_THREADS + SC_STAGERS, 1) scan_kernel(const ScanArgs<T> a) {
    constexpr int CPC = SC_THREADS / LPC;         // channels per CTA: 64 .. 8
    constexpr int NP = NS * LPC;                  // padded states, even
    constexpr int SC_T = NP > 128 ? 8 : 16;       // tokens per tile
    constexpr int CW = CPC / 2;                   // channel pairs: a staging thread handles one pair of some rows
    constexpr int FS = SC_STAGERS / CW;           // rows per sweep
    constexpr int XE = (SC_T + FS - 1) / FS;
    constexpr int BU = SC_T * NP;                 // pairs of B and of C values per tile
    constexpr int BE = (BU + SC_STAGERS - 1) / SC_STAGERS;
    __shared__ __align__(16) float2 sd[2][SC_T][CPC];       // step, step * x
    __shared__ __align__(16) float2 so[2][SC_T][CPC];       // D x, silu(z)
    __shared__ __align__(16) float sBC[2][2][SC_T][NP];
    __shared__ float sy[2][SC_T][CPC + 1];
    pdl_launch_dependents();
    const int c0 = blockIdx.x * CPC;
    const int tiles = (int)((a.n + SC_T - 1) / SC_T);
    if (threadIdx.x >= SC_THREADS) {
        // ---- staging: channels fc, fc + 1 of rows fr, fr + FS, ...; a thread writes out the same elements it has staged
        const int tid = threadIdx.x - SC_THREADS;
        const int fc = 2 * (tid % CW), fr = tid / CW, c = c0 + fc;
        const bool ok0 = c < a.C, two = c + 1 < a.C, al = two && a.pairs;
        const float2 bias = make_float2(ok0 ? a.dt_bias[c] : 0.0f, two ? a.dt_bias[c + 1] : 0.0f);
        const float2 Dc = make_float2(ok0 ? a.D[c] : 0.0f, two ? a.D[c + 1] : 0.0f);
        Pair<T> px[XE], pz[XE], pb[BE];         // as stored: converted when staged, so that the loads stay in flight
        Pair<float> pd[XE];
        pdl_wait();
        // running addresses of this thread's next tile; rows past the end are zeros
        const T *xp = a.x + (int64_t)fr * a.ldx + c, *zp = a.z + (int64_t)fr * a.ldz + c, *bp[BE];
        const float* dp = a.dtp + (int64_t)fr * a.ldt + c;
        const int n_tok = (int)a.n;
        int left = ok0 ? n_tok - fr : 0;
#pragma unroll
        for (int i = 0; i < BE; ++i) {          // unit e: row, B or C, pair of states
            const int e = tid + i * SC_STAGERS;
            bp[i] = a.bc + (int64_t)(e / NP) * a.ldbc + ((e % NP) / (NP / 2)) * a.N + 2 * (e % (NP / 2));
        }
        auto fetch = [&](int tile) {
#pragma unroll
            for (int i = 0; i < XE; ++i) {
                if ((SC_T % FS == 0 || fr + i * FS < SC_T) && i * FS < left) {
                    px[i].load(xp + (int64_t)(i * FS) * a.ldx, two, al);
                    pd[i].load(dp + (int64_t)(i * FS) * a.ldt, two, al);
                    pz[i].load(zp + (int64_t)(i * FS) * a.ldz, two, al);
                } else {
                    px[i].zero();
                    pd[i].zero();
                    pz[i].zero();
                }
            }
            xp += SC_T * a.ldx;
            dp += SC_T * a.ldt;
            zp += SC_T * a.ldz;
            left -= SC_T;
#pragma unroll
            for (int i = 0; i < BE; ++i) {
                const int e = tid + i * SC_STAGERS, r = e / NP, n = 2 * (e % (NP / 2));
                if ((BU % SC_STAGERS == 0 || e < BU) && n < a.N && tile * SC_T + r < n_tok) pb[i].load(bp[i], n + 1 < a.N, n + 1 < a.N && a.bc_pairs);
                else pb[i].zero();
                bp[i] += SC_T * a.ldbc;
            }
        };
        auto put = [&](int tile) {
            const int buf = tile & 1;
#pragma unroll
            for (int i = 0; i < XE; ++i) {
                const int r = fr + i * FS;
                if (SC_T % FS != 0 && r >= SC_T) break;
                const bool live = tile * SC_T + r < n_tok;      // a zero step leaves the state unchanged
                const float2 x = px[i].get(), z = pz[i].get(), d = pd[i].get();
                const float s0 = live ? softplus_f32(d.x + bias.x) : 0.0f, s1 = live ? softplus_f32(d.y + bias.y) : 0.0f;
                *reinterpret_cast<float4*>(&sd[buf][r][fc]) = make_float4(s0, s0 * x.x, s1, s1 * x.y);
                *reinterpret_cast<float4*>(&so[buf][r][fc]) = make_float4(Dc.x * x.x, silu_f32(z.x), Dc.y * x.y, silu_f32(z.y));
            }
#pragma unroll
            for (int i = 0; i < BE; ++i) {
                const int e = tid + i * SC_STAGERS, r = e / NP, w = (e % NP) / (NP / 2), n = 2 * (e % (NP / 2));
                if (BU % SC_STAGERS == 0 || e < BU) *reinterpret_cast<float2*>(&sBC[buf][w][r][n]) = pb[i].get();
            }
        };
        T* yp = a.y + (int64_t)fr * a.ldy + c;
        auto write = [&](int tile) {
            const int buf = tile & 1;
#pragma unroll
            for (int i = 0; i < XE; ++i) {
                const int r = fr + i * FS;
                if (!ok0 || (SC_T % FS != 0 && r >= SC_T) || tile * SC_T + r >= n_tok) continue;
                const float4 o = *reinterpret_cast<const float4*>(&so[buf][r][fc]);
                const float y0 = (sy[buf][r][fc] + o.x) * o.y, y1 = (sy[buf][r][fc + 1] + o.z) * o.w;
                T* p = yp + (int64_t)(i * FS) * a.ldy;
                if (al && sizeof(T) == 2) {
                    *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(y0, y1);
                } else {
                    stf(p, y0);
                    if (two) stf(p + 1, y1);
                }
            }
            yp += SC_T * a.ldy;
        };
        fetch(0);
        put(0);
        if (tiles > 1) fetch(1);
        __syncthreads();
        for (int t = 0; t < tiles; ++t) {      // while the recurrence runs on tile t
            if (t > 0) write(t - 1);
            if (t + 1 < tiles) put(t + 1);
            if (t + 2 < tiles) fetch(t + 2);
            __syncthreads();
        }
        write(tiles - 1);
        return;
    }
    // ---- recurrence
    const int lane = threadIdx.x % LPC, ch = threadIdx.x / LPC, c = c0 + ch;
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
    uint64_t A22[(NS + 1) / 2], S2[(NS + 1) / 2];
    if constexpr (NS % 2 == 0) {
#pragma unroll
        for (int i = 0; i < NS / 2; ++i) {
            A22[i] = pack2(A2[2 * i], A2[2 * i + 1]);
            S2[i] = pack2(S[2 * i], S[2 * i + 1]);
        }
    }
    __syncthreads();
    for (int t = 0; t < tiles; ++t) {
        const int buf = t & 1;
        // eight tokens at a time: everything but the chain through S is independent; the partial outputs of the channel's lanes
        // are summed by halving (a lane keeps half of the tokens and hands over the other half), 7 shuffles for 8 tokens
#pragma unroll 1
        for (int r0 = 0; r0 < SC_T; r0 += 8) {
            float y[8];
            if constexpr (NS % 2 == 0) {
                // two states per instruction
                uint64_t f[8][NS / 2], in[8][NS / 2];
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    const float2 d = sd[buf][r0 + u][ch];
                    const uint64_t dt2 = pack2(d.x, d.x), dx2 = pack2(d.y, d.y);
                    const float* B = &sBC[buf][0][r0 + u][lane * NS];
#pragma unroll
                    for (int i = 0; i < NS / 2; ++i) {
                        const float2 e = unpack2(mul2(dt2, A22[i]));
                        f[u][i] = pack2(ex2_ordered(e.x), ex2_ordered(e.y));
                        in[u][i] = mul2(dx2, *reinterpret_cast<const uint64_t*>(B + 2 * i));
                    }
                }
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    const float* Cc = &sBC[buf][1][r0 + u][lane * NS];
                    uint64_t acc = 0;
#pragma unroll
                    for (int i = 0; i < NS / 2; ++i) {
                        S2[i] = fma2(f[u][i], S2[i], in[u][i]);
                        acc = fma2(S2[i], *reinterpret_cast<const uint64_t*>(Cc + 2 * i), acc);
                    }
                    const float2 s = unpack2(acc);
                    y[u] = s.x + s.y;
                }
            } else {
                float f[8][NS], in[8][NS];
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    const float2 d = sd[buf][r0 + u][ch];
#pragma unroll
                    for (int i = 0; i < NS; ++i) {
                        f[u][i] = ex2_ordered(d.x * A2[i]);
                        in[u][i] = d.y * sBC[buf][0][r0 + u][lane * NS + i];
                    }
                }
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    y[u] = 0.0f;
#pragma unroll
                    for (int i = 0; i < NS; ++i) {
                        S[i] = fmaf(f[u][i], S[i], in[u][i]);
                        y[u] = fmaf(S[i], sBC[buf][1][r0 + u][lane * NS + i], y[u]);
                    }
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
                for (int u = 0; u < OUT; ++u) sy[buf][r0 + first + u][ch] = y[u];
        }
        __syncthreads();
    }
    if constexpr (NS % 2 == 0) {
#pragma unroll
        for (int i = 0; i < NS / 2; ++i) {
            const float2 s = unpack2(S2[i]);
            S[2 * i] = s.x;
            S[2 * i + 1] = s.y;
        }
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
    const dim3 grid((unsigned)((a.C + cpc - 1) / cpc)), block(SC_THREADS + SC_STAGERS);
    switch (lpc) {
        case 4: return launch_pdl(scan_kernel<T, NS, 4>, grid, block, 0, st, a);
        case 8: return launch_pdl(scan_kernel<T, NS, 8>, grid, block, 0, st, a);
        case 16: return launch_pdl(scan_kernel<T, NS, 16>, grid, block, 0, st, a);
        default: return launch_pdl(scan_kernel<T, NS, 32>, grid, block, 0, st, a);
    }
}

template <typename T>
static int run_scan(ScanArgs<T> a, cudaStream_t st) {
    auto al = [&](const void* p, int64_t ld, int esz) { return ld % 2 == 0 && (uintptr_t)p % (2 * esz) == 0; };
    const int esz = (int)sizeof(T);
    a.pairs = al(a.x, a.ldx, esz) && al(a.z, a.ldz, esz) && al(a.y, a.ldy, esz) && al(a.dtp, a.ldt, 4);
    a.bc_pairs = a.N % 2 == 0 && al(a.bc, a.ldbc, esz);
    // the most states per lane that wastes little padding and still gives most SMs a CTA; otherwise the most CTAs
    int least = 1 << 30;
    for (int ns = 4; ns >= 1; --ns) {
        int lpc = 4;
        while (lpc < 32 && ns * lpc < a.N) lpc *= 2;
        if (ns * lpc >= a.N && ns * lpc < least) least = ns * lpc;
    }
    int best_ns = 0, best_lpc = 32;
    for (int ns = 4; ns >= 1; --ns) {
        int lpc = 4;
        while (lpc < 32 && ns * lpc < a.N) lpc *= 2;
        if (ns * lpc < a.N || 4 * ns * lpc > 5 * least) continue;
        if (best_ns == 0 || (int64_t)a.C * best_lpc < 120ll * SC_THREADS) { best_ns = ns; best_lpc = lpc; }
    }
    cudaError_t e = best_ns == 1 ? launch_scan<T, 1>(a, best_lpc, st)
                  : best_ns == 2 ? launch_scan<T, 2>(a, best_lpc, st)
                  : best_ns == 3 ? launch_scan<T, 3>(a, best_lpc, st)
                  : best_ns == 4 ? launch_scan<T, 4>(a, best_lpc, st)
                  : launch_pdl(scan_kernel<T, 8, 32>, dim3((a.C + 7) / 8), dim3(SC_THREADS + SC_STAGERS), 0, st, a);
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
    SCMX_REQUIRE(N <= 256 && n < (1ll << 30), SCMX_ELIMIT, "selective_scan: %d states per channel (256 at most), %lld tokens", N, (long long)n);
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
