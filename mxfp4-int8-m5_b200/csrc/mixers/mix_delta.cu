// Gated delta rule: a [d, dv] state per head, S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q, with one decay g per head
// or one per head and key channel.  q and k arrive after convolution and SiLU and are made unit vectors here (q also scaled by
// d^(-1/2)); head h reads q / k head h / (H / G).  beta = sigmoid(b), log g = nA_h softplus(a + dt_bias) with nA = -exp(A_log).
//
// delta_scan_kernel   any storage type, heads up to 256: token by token, float32 (bfloat16 prompts: delta_tc, tensor cores)
// delta_step_kernel   one token with the low-rank second products of decays and gates, head norm and gate, a cluster per head
#include <cooperative_groups.h>
#include "mix_delta.cuh"

namespace cg = cooperative_groups;

namespace scmx {

constexpr int DS_T = 8;       // tokens staged together

// Grid (heads, column slices of 32), 128 threads: four lanes share a column of the state, each holds a quarter of its rows (float4
// groups 4 r + sub).  With o = (g S)^T q + (q . k) u both sums over the old state are taken in one pass.
template <typename T, int R4, bool CH>
__global__ void __launch_bounds__(128) delta_scan_kernel(const DeltaArgs a) {
    constexpr int D = 16 * R4;
    __shared__ __align__(16) float sq[DS_T][D], sk[DS_T][D], sg[CH ? DS_T : 1][D];
    __shared__ float sv[DS_T][32], sb[DS_T], sqk[DS_T], sgs[DS_T];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, e0 = blockIdx.y * 32, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int kh = h / (a.H / a.G), sub = lane & 3, col = 8 * warp + (lane >> 2);
    const bool ok = e0 + col < a.dv;
    const T *q = static_cast<const T*>(a.q) + (int64_t)kh * a.d, *k = static_cast<const T*>(a.k) + (int64_t)kh * a.d;
    const T *v = static_cast<const T*>(a.v) + (int64_t)h * a.dv + e0, *b = static_cast<const T*>(a.b) + h;
    const float nA = a.nA[h], qs = rsqrtf((float)a.d);
    float* gS = a.state + (int64_t)h * a.d * a.dv + e0 + col;
    float4 S[R4];
#pragma unroll
    for (int r = 0; r < R4; ++r) {
        const int i = 16 * r + 4 * sub;
        S[r].x = ok && i < a.d ? gS[(int64_t)i * a.dv] : 0.0f;
        S[r].y = ok && i + 1 < a.d ? gS[(int64_t)(i + 1) * a.dv] : 0.0f;
        S[r].z = ok && i + 2 < a.d ? gS[(int64_t)(i + 2) * a.dv] : 0.0f;
        S[r].w = ok && i + 3 < a.d ? gS[(int64_t)(i + 3) * a.dv] : 0.0f;
    }
    for (int64_t t0 = 0; t0 < a.n; t0 += DS_T) {
        const int nt = (int)min((int64_t)DS_T, a.n - t0);
        __syncthreads();                       // the previous tokens are consumed
        for (int t = warp; t < nt; t += 4) {
            const T *qr = q + (t0 + t) * a.ldq, *kr = k + (t0 + t) * a.ldk;
            constexpr int E = (D + 31) / 32;
            float x[E], y[E], qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
            for (int j = 0; j < E; ++j) {
                const int e = lane + 32 * j;
                x[j] = e < a.d ? ldf(qr + e) : 0.0f;
                y[j] = e < a.d ? ldf(kr + e) : 0.0f;
                qq += x[j] * x[j];
                kk += y[j] * y[j];
                qk += x[j] * y[j];
            }
            const float iq = qs / sqrtf(warp_sumf(qq) + 1e-6f), ik = 1.0f / sqrtf(warp_sumf(kk) + 1e-6f);
            qk = warp_sumf(qk);
#pragma unroll
            for (int j = 0; j < E; ++j) {
                const int e = lane + 32 * j;
                if (e < D) {
                    sq[t][e] = x[j] * iq;
                    sk[t][e] = y[j] * ik;
                    if (CH)
                        sg[CH ? t : 0][e] = e < a.d ? expf(nA * softplus_f32(static_cast<const float*>(a.a)[(t0 + t) * a.lda + (int64_t)h * a.d + e] +
                                                                             a.dtb[(int64_t)h * a.d + e])) : 0.0f;
                }
            }
            if (lane == 0) {
                sqk[t] = qk * iq * ik;
                sb[t] = 1.0f / (1.0f + expf(-ldf(b + (t0 + t) * a.ldb)));
                if (!CH) sgs[t] = expf(nA * softplus_f32(ldf(static_cast<const T*>(a.a) + (t0 + t) * a.lda + h) + a.dtb[h]));
            }
        }
        for (int i = tid; i < nt * 32; i += 128) {
            const int t = i >> 5, e = i & 31;
            sv[t][e] = e0 + e < a.dv ? ldf(v + (t0 + t) * a.ldv + e) : 0.0f;
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float4 *k4 = reinterpret_cast<const float4*>(sk[t]), *q4 = reinterpret_cast<const float4*>(sq[t]);
            const float4* g4 = reinterpret_cast<const float4*>(sg[CH ? t : 0]);
            const float g = CH ? 0.0f : sgs[t];
            float pk = 0.0f, pq = 0.0f;
#pragma unroll
            for (int r = 0; r < R4; ++r) {
                const float4 kk = k4[4 * r + sub], qq = q4[4 * r + sub];
                const float4 gg = CH ? g4[4 * r + sub] : make_float4(g, g, g, g);
                S[r].x *= gg.x; S[r].y *= gg.y; S[r].z *= gg.z; S[r].w *= gg.w;
                pk = fmaf(S[r].x, kk.x, pk); pk = fmaf(S[r].y, kk.y, pk); pk = fmaf(S[r].z, kk.z, pk); pk = fmaf(S[r].w, kk.w, pk);
                pq = fmaf(S[r].x, qq.x, pq); pq = fmaf(S[r].y, qq.y, pq); pq = fmaf(S[r].z, qq.z, pq); pq = fmaf(S[r].w, qq.w, pq);
            }
            pk += __shfl_xor_sync(0xffffffffu, pk, 1);
            pq += __shfl_xor_sync(0xffffffffu, pq, 1);
            pk += __shfl_xor_sync(0xffffffffu, pk, 2);
            pq += __shfl_xor_sync(0xffffffffu, pq, 2);
            const float u = sb[t] * (sv[t][col] - pk);
#pragma unroll
            for (int r = 0; r < R4; ++r) {
                const float4 kk = k4[4 * r + sub];
                S[r].x = fmaf(kk.x, u, S[r].x); S[r].y = fmaf(kk.y, u, S[r].y); S[r].z = fmaf(kk.z, u, S[r].z); S[r].w = fmaf(kk.w, u, S[r].w);
            }
            if (sub == 0 && ok) a.o[((t0 + t) * a.H + h) * a.dv + e0 + col] = fmaf(sqk[t], u, pq);
        }
    }
#pragma unroll
    for (int r = 0; r < R4; ++r) {
        const int i = 16 * r + 4 * sub;
        if (ok && i < a.d) gS[(int64_t)i * a.dv] = S[r].x;
        if (ok && i + 1 < a.d) gS[(int64_t)(i + 1) * a.dv] = S[r].y;
        if (ok && i + 2 < a.d) gS[(int64_t)(i + 2) * a.dv] = S[r].z;
        if (ok && i + 3 < a.d) gS[(int64_t)(i + 3) * a.dv] = S[r].w;
    }
}

template <typename T, bool CH>
static int run_delta_scan(const DeltaArgs& a, cudaStream_t st) {
    const dim3 grid(a.H, (a.dv + 31) / 32), block(128);
    cudaError_t e;
    if (a.d <= 16) e = launch_pdl(delta_scan_kernel<T, 1, CH>, grid, block, 0, st, a);
    else if (a.d <= 32) e = launch_pdl(delta_scan_kernel<T, 2, CH>, grid, block, 0, st, a);
    else if (a.d <= 64) e = launch_pdl(delta_scan_kernel<T, 4, CH>, grid, block, 0, st, a);
    else if (a.d <= 128) e = launch_pdl(delta_scan_kernel<T, 8, CH>, grid, block, 0, st, a);
    else e = launch_pdl(delta_scan_kernel<T, 16, CH>, grid, block, 0, st, a);
    SCMX_PDL_OK("delta_scan_kernel", e);
    return SCMX_OK;
}

// ---- one token ------------------------------------------------------------------------------------------------------------
struct DeltaStepArgs {
    const float *q, *k, *v, *b;      // one row each, after convolution and SiLU (b: logits)
    const float *a, *g;              // decay logits [H] and gates [H dv], or the low-rank vectors [ra], [rg]
    const void *wa, *wg;             // second low-rank products [H d, lwa], [H dv, lwg], rows zero padded to a multiple of 8
    const float *nA, *dtb, *w;       // -exp(A_log) [H], dt_bias, head norm weight [dv]
    float* state;                    // [H, d, dv]
    float* y;                        // [H dv]
    int H, G, d, dv, ra, rg, lwa, lwg, cw;      // cw: state columns per CTA (<= 256)
    float eps;
};

// Products of stored rows (multiples of 8 columns) with a vector in shared memory, a group of lanes per row.  The first vector of the
// first PASS rows per group is requested by `request`, which may run before the vector is known.
template <typename T>
struct RowDots {
    static constexpr int PASS = 2;
    Raw8<T> pre[PASS];
    int lpr, sub, first, step;
    __device__ __forceinline__ void setup(int n, int lane, int warp) {
        lpr = 1;
        while (lpr < 32 && 8 * lpr < n) lpr *= 2;
        sub = lane & (lpr - 1);
        step = 256 / lpr;
        first = (32 * warp + lane) / lpr;
    }
    __device__ __forceinline__ void request(const T* w, int n, int rows) {
#pragma unroll
        for (int k = 0; k < PASS; ++k)
            if (first + k * step < rows && 8 * sub < n) pre[k].load(w + (int64_t)(first + k * step) * n + 8 * sub);
    }
    // done(row, product) for every row, on the lanes of its group; the warps of the CTA call it together
    template <typename F>
    __device__ __forceinline__ void run(const T* w, const float* x, int n, int rows, F done) {
        auto dot = [&](const Raw8<T>& u, int e, float s) -> float {
            float v[8];
            u.get(v);
#pragma unroll
            for (int i = 0; i < 8; ++i) s = fmaf(v[i], x[e + i], s);
            return s;
        };
        auto finish = [&](int row, float s) {
            for (int e = 8 * (sub + lpr); e < n; e += 8 * lpr)
                if (row < rows) {
                    Raw8<T> u;
                    u.load(w + (int64_t)row * n + e);
                    s = dot(u, e, s);
                }
            for (int o = lpr / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
            if (row < rows) done(row, s);
        };
#pragma unroll
        for (int k = 0; k < PASS; ++k) {
            const int row = first + k * step;
            finish(row, row < rows && 8 * sub < n ? dot(pre[k], 8 * sub, 0.0f) : 0.0f);
        }
        for (int r0 = PASS * step; r0 < rows; r0 += step) {
            const int row = first + r0;
            float s = 0.0f;
            if (row < rows && 8 * sub < n) {
                Raw8<T> u;
                u.load(w + (int64_t)row * n + 8 * sub);
                s = dot(u, 8 * sub, 0.0f);
            }
            finish(row, s);
        }
    }
};

template <typename T, bool CH>
__global__ void __launch_bounds__(256) delta_step_kernel(const DeltaStepArgs a) {
    extern __shared__ __align__(16) float sm[];
    float *sa = sm, *sg1 = sa + a.lwa, *sq = sg1 + a.lwg, *sk = sq + a.d, *sg = sk + a.d, *so = sg + a.d, *su = so + 512, *sgate = su + 256;
    __shared__ float red[33];
    __shared__ float ssq;
    pdl_launch_dependents();
    cg::cluster_group cl = cg::this_cluster();
    const int h = blockIdx.y, rank = (int)cl.block_rank(), nc = (int)cl.num_blocks(), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int kh = h / (a.H / a.G);
    const int e0 = rank * a.cw, cw = min(a.cw, a.dv - e0);      // cw may be <= 0 on a trailing rank
    const int groups = cw > 0 ? 256 / cw : 0, grp = cw > 0 ? tid / cw : 0, col = cw > 0 ? tid - grp * cw : 0;
    const bool work = grp < groups;
    // low-rank weights of this CTA's channels and values never change: requested before the previous kernel ends
    const int per = (a.d + nc - 1) / nc, ch0 = min(a.d, rank * per), nch = min(per, a.d - ch0);
    const T *wa = static_cast<const T*>(a.wa) + ((int64_t)h * a.d + ch0) * a.lwa, *wg = static_cast<const T*>(a.wg) + ((int64_t)h * a.dv + e0) * a.lwg;
    RowDots<T> da, dg;
    if (CH) {
        da.setup(a.lwa, lane, warp);
        dg.setup(a.lwg, lane, warp);
        da.request(wa, a.lwa, nch);
        dg.request(wg, a.lwg, cw);
        cl.sync();                   // every CTA of the cluster runs: its shared memory may be written
    }
    pdl_wait();
    constexpr int PRE = 16;          // the first rows of this thread's column are requested before anything else
    float* S = a.state + (int64_t)h * a.d * a.dv + e0 + col;
    float pre[PRE];
#pragma unroll
    for (int j = 0; j < PRE; ++j) {
        const int i = grp + j * groups;
        pre[j] = work && i < a.d ? S[(int64_t)i * a.dv] : 0.0f;
    }
    const float v = tid < cw ? a.v[(int64_t)h * a.dv + e0 + tid] : 0.0f;
    const float beta = 1.0f / (1.0f + expf(-a.b[h])), nA = a.nA[h];
    if (CH) {
        for (int i = tid; i < a.lwa; i += 256) sa[i] = i < a.ra ? a.a[i] : 0.0f;
        for (int i = tid; i < a.lwg; i += 256) sg1[i] = i < a.rg ? a.g[i] : 0.0f;
    }
    // unit vectors: every warp takes the three sums for itself
    float qq = 0.0f, kk = 0.0f, qk = 0.0f;
    for (int i = lane; i < a.d; i += 32) {
        const float x = a.q[(int64_t)kh * a.d + i], y = a.k[(int64_t)kh * a.d + i];
        qq += x * x;
        kk += y * y;
        qk += x * y;
    }
    const float iq = rsqrtf((float)a.d) / sqrtf(warp_sumf(qq) + 1e-6f), ik = 1.0f / sqrtf(warp_sumf(kk) + 1e-6f);
    qk = warp_sumf(qk) * iq * ik;
    for (int i = tid; i < a.d; i += 256) {
        sq[i] = a.q[(int64_t)kh * a.d + i] * iq;
        sk[i] = a.k[(int64_t)kh * a.d + i] * ik;
        if (!CH) sg[i] = expf(nA * softplus_f32(a.a[h] + a.dtb[h]));
    }
    float gate = 0.0f;
    if (CH) {
        __syncthreads();
        da.run(wa, sa, a.lwa, nch, [&](int c, float z) {
            if (da.sub >= nc) return;
            const float g = expf(nA * softplus_f32(z + a.dtb[(int64_t)h * a.d + ch0 + c]));
            for (int r = da.sub; r < nc; r += da.lpr) *cl.map_shared_rank(sg + ch0 + c, r) = g;
        });
        dg.run(wg, sg1, a.lwg, cw, [&](int c, float z) {
            if (dg.sub == 0) sgate[c] = 1.0f / (1.0f + expf(-z));
        });
        cl.sync();
        if (tid < cw) gate = sgate[tid];
    } else {
        if (tid < cw) gate = silu_f32(a.g[(int64_t)h * a.dv + e0 + tid]);
        __syncthreads();
    }
    float pk = 0.0f, pq = 0.0f;
    if (work) {
#pragma unroll
        for (int j = 0; j < PRE; ++j) {
            const int i = grp + j * groups;
            if (i < a.d) {
                pre[j] *= sg[i];
                pk = fmaf(pre[j], sk[i], pk);
                pq = fmaf(pre[j], sq[i], pq);
            }
        }
#pragma unroll 8
        for (int i = grp + PRE * groups; i < a.d; i += groups) {
            const float s = S[(int64_t)i * a.dv] * sg[i];
            pk = fmaf(s, sk[i], pk);
            pq = fmaf(s, sq[i], pq);
        }
    }
    so[tid] = pk;
    so[256 + tid] = pq;
    __syncthreads();
    float o = 0.0f;
    if (tid < cw) {
        float k0 = 0.0f, q0 = 0.0f;
        for (int r = 0; r < groups; ++r) {
            k0 += so[r * cw + tid];
            q0 += so[256 + r * cw + tid];
        }
        const float u = beta * (v - k0);
        su[tid] = u;
        o = fmaf(qk, u, q0);
    }
    const float ss = block_sumf(o * o, red);      // (its barriers also publish su)
    if (work) {
        const float u = su[col];
#pragma unroll
        for (int j = 0; j < PRE; ++j) {
            const int i = grp + j * groups;
            if (i < a.d) S[(int64_t)i * a.dv] = fmaf(sk[i], u, pre[j]);
        }
#pragma unroll 8
        for (int i = grp + PRE * groups; i < a.d; i += groups) S[(int64_t)i * a.dv] = fmaf(sk[i], u, S[(int64_t)i * a.dv] * sg[i]);
    }
    float total = ss;
    if (nc > 1) {
        if (tid == 0) ssq = ss;
        cl.sync();
        total = 0.0f;
        for (int r = 0; r < nc; ++r) total += *cl.map_shared_rank(&ssq, r);
        cl.sync();
    }
    if (tid < cw) a.y[(int64_t)h * a.dv + e0 + tid] = o * rms_inv_f32(total, a.dv, a.eps) * a.w[e0 + tid] * gate;
}

template <typename T, bool CH>
static int run_delta_step(DeltaStepArgs a, cudaStream_t st) {
    int nc = 1;                                   // CTAs per head: slices of at least 32 columns, 256 at most
    while (nc < 8 && (a.dv + nc - 1) / nc > 32) nc *= 2;
    a.cw = (a.dv + nc - 1) / nc;
    SCMX_REQUIRE(a.cw <= 256, SCMX_ELIMIT, "delta_step: %d values per head (2048 at most)", a.dv);
    const size_t smem = (size_t)(a.lwa + a.lwg + 3 * a.d + 512 + 256 + 256) * 4;
    SCMX_REQUIRE(smem <= 48 * 1024, SCMX_ELIMIT, "delta_step: head size %d, inner sizes %d and %d", a.d, a.ra, a.rg);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(nc, a.H);
    cfg.blockDim = dim3(256);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = nc;
    at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at;
    cfg.numAttrs = g_use_pdl ? 2 : 1;
    SCMX_PDL_OK("delta_step_kernel", cudaLaunchKernelEx(&cfg, delta_step_kernel<T, CH>, a));
    return SCMX_OK;
}

}  // namespace scmx

using namespace scmx;

extern "C" int64_t scmx_delta_scratch(int64_t n, int H, int d, int dv, int64_t ldv) {
    return n > 0 && H > 0 && d > 0 && dv > 0 && delta_tc_supported(n, H, d, dv, ldv) ? delta_tc_scratch(n, H, d, dv) : 0;
}

extern "C" int scmx_delta(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* v, int64_t ldv, const void* b, int64_t ldb,
                          const void* a_, int64_t lda, int dt, int channel, int64_t n, int H, int G, int d, int dv, const float* nA,
                          const float* dt_bias, float* state, float* o, void* scratch, int64_t scratch_bytes, int32_t* status, void* stream) {
    SCMX_DT_OK("delta", dt);
    SCMX_REQUIRE(q && k && v && b && a_ && nA && dt_bias && state && o, SCMX_EINVAL, "delta: null buffer");
    SCMX_REQUIRE(n >= 0 && H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0, SCMX_EINVAL, "delta: n=%lld heads=%d over %d, sizes %d / %d", (long long)n, H, G, d, dv);
    SCMX_REQUIRE(d <= 256, SCMX_ELIMIT, "delta: head size %d (256 at most)", d);
    if (n == 0) return SCMX_OK;
    DeltaArgs a;
    a.q = q; a.k = k; a.v = v; a.b = b; a.a = a_; a.nA = nA; a.dtb = dt_bias; a.state = state; a.o = o;
    a.n = n; a.ldq = ldq; a.ldk = ldk; a.ldv = ldv; a.ldb = ldb; a.lda = lda; a.H = H; a.G = G; a.d = d; a.dv = dv;
    const cudaStream_t st = (cudaStream_t)stream;
    if (scratch != nullptr) {
        SCMX_REQUIRE(dt == 0 && status && delta_tc_supported(n, H, d, dv, ldv), SCMX_ELIMIT, "delta: no tensor-core form for head sizes %d / %d", d, dv);
        SCMX_REQUIRE(((uintptr_t)v & 15) == 0 && ((uintptr_t)scratch & 255) == 0 && scratch_bytes >= delta_tc_scratch(n, H, d, dv), SCMX_EINVAL,
                     "delta: scratch of %lld bytes or an unaligned pointer", (long long)scratch_bytes);
        return delta_tc(a, channel != 0, scratch, status, st);
    }
    if (dt == 0) return channel ? run_delta_scan<bf16_t, true>(a, st) : run_delta_scan<bf16_t, false>(a, st);
    return channel ? run_delta_scan<float, true>(a, st) : run_delta_scan<float, false>(a, st);
}

extern "C" int scmx_delta_step(const float* q, const float* k, const float* v, const float* b, const float* a_, const float* g, const void* wa,
                               int64_t lwa, int ra, const void* wg, int64_t lwg, int rg, int dt, int H, int G, int d, int dv, const float* nA,
                               const float* dt_bias, const float* w, float eps, float* state, float* y, void* stream) {
    SCMX_DT_OK("delta_step", dt);
    SCMX_REQUIRE(q && k && v && b && a_ && g && nA && dt_bias && w && state && y, SCMX_EINVAL, "delta_step: null buffer");
    SCMX_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0, SCMX_EINVAL, "delta_step: heads=%d over %d, sizes %d / %d", H, G, d, dv);
    SCMX_REQUIRE((wa != nullptr) == (wg != nullptr), SCMX_EINVAL, "delta_step: low-rank products of decays and gates come together");
    SCMX_REQUIRE(wa == nullptr || (ra > 0 && rg > 0 && lwa % 8 == 0 && lwg % 8 == 0 && lwa >= ra && lwg >= rg && lwa < (1 << 16) && lwg < (1 << 16) &&
                                   (((uintptr_t)wa | (uintptr_t)wg) & 15) == 0), SCMX_EINVAL, "delta_step: pitches %lld, %lld of inner sizes %d, %d",
                 (long long)lwa, (long long)lwg, ra, rg);
    DeltaStepArgs s;
    s.q = q; s.k = k; s.v = v; s.b = b; s.a = a_; s.g = g; s.wa = wa; s.wg = wg; s.nA = nA; s.dtb = dt_bias; s.w = w; s.state = state; s.y = y;
    s.H = H; s.G = G; s.d = d; s.dv = dv; s.ra = wa ? ra : 0; s.rg = wa ? rg : 0; s.lwa = wa ? (int)lwa : 0; s.lwg = wa ? (int)lwg : 0; s.cw = 0; s.eps = eps;
    const cudaStream_t st = (cudaStream_t)stream;
    if (wa == nullptr) return run_delta_step<float, false>(s, st);
    return dt == 0 ? run_delta_step<bf16_t, true>(s, st) : run_delta_step<float, true>(s, st);
}
