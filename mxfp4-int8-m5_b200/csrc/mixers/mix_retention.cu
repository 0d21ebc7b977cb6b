// Retention: linear attention with a fixed decay per head.  S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t; q and k are rotated
// (rotate-half, table of cosines and sines per position) and k is scaled when they are read, in float32.
//
// retention_scan_kernel   any sizes, any storage type: token by token, float32 (bfloat16 prompts: retention_tc, tensor cores)
// retention_step_kernel   one token: state update, output, head norm and gate, a cluster of CTAs per head
#include <cooperative_groups.h>
#include "mix_common.cuh"

namespace cg = cooperative_groups;

namespace scmx {

bool retention_tc_supported(int64_t n, int H, int d, int dv, int dims, int64_t ldv);
int64_t retention_tc_scratch(int64_t n, int H, int d, int dv);
int retention_tc(const bf16_t* q, int64_t ldq, const bf16_t* k, int64_t ldk, const bf16_t* v, int64_t ldv, int64_t n, int H, int d, int dv,
                 const float* cs, int dims, float kscale, const float* decay, float* state, float* o, void* scratch, int32_t* status,
                 cudaStream_t st);

template <typename T>
struct RetArgs {
    const T *q, *k, *v;       // [n, ld*]: heads side by side
    const float* cs;          // [n, dims] cos / sin rows of this portion's positions
    const float* decay;       // [H]
    float* state;             // [H, d, dv]
    float* o;                 // [n, H, dv]
    int64_t n, ldq, ldk, ldv;
    int H, d, dv, dims;
    float kscale;
};

constexpr int RS_T = 8;       // tokens staged together

// Grid (heads, column slices of 32): a lane owns a column of the state, the 8 warps split its rows.
template <typename T>
__global__ void __launch_bounds__(256) retention_scan_kernel(const RetArgs<T> a) {
    extern __shared__ float sm[];
    float* S = sm;                            // [d][32]
    float* sq = S + a.d * 32;                 // [RS_T][d]
    float* sk = sq + RS_T * a.d;              // [RS_T][d]
    float* sv = sk + RS_T * a.d;              // [RS_T][32]
    float* so = sv + RS_T * 32;               // [8][RS_T][32]
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, e0 = blockIdx.y * 32, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const bool ok = e0 + lane < a.dv;
    float* gS = a.state + (int64_t)h * a.d * a.dv + e0 + lane;
    for (int i = warp; i < a.d; i += 8) S[i * 32 + lane] = ok ? gS[(int64_t)i * a.dv] : 0.0f;
    const float decay = a.decay[h];
    for (int64_t t0 = 0; t0 < a.n; t0 += RS_T) {
        const int nt = (int)min((int64_t)RS_T, a.n - t0);
        for (int i = tid; i < nt * a.d; i += 256) {
            const int t = i / a.d, e = i - t * a.d;
            const float* cs = a.cs + (t0 + t) * a.dims;
            sq[i] = rotated(a.q + (t0 + t) * a.ldq + (int64_t)h * a.d, e, a.dims, cs);
            sk[i] = rotated(a.k + (t0 + t) * a.ldk + (int64_t)h * a.d, e, a.dims, cs) * a.kscale;
        }
        for (int i = tid; i < nt * 32; i += 256) {
            const int t = i >> 5, e = e0 + (i & 31);
            sv[i] = e < a.dv ? ldf(a.v + (t0 + t) * a.ldv + (int64_t)h * a.dv + e) : 0.0f;
        }
        __syncthreads();
        float part[RS_T];
#pragma unroll
        for (int t = 0; t < RS_T; ++t) part[t] = 0.0f;
        for (int i = warp; i < a.d; i += 8) {
            float s = S[i * 32 + lane];
#pragma unroll
            for (int t = 0; t < RS_T; ++t)
                if (t < nt) {
                    s = fmaf(decay, s, sk[t * a.d + i] * sv[t * 32 + lane]);
                    part[t] = fmaf(sq[t * a.d + i], s, part[t]);
                }
            S[i * 32 + lane] = s;
        }
#pragma unroll
        for (int t = 0; t < RS_T; ++t) so[(warp * RS_T + t) * 32 + lane] = part[t];
        __syncthreads();
        for (int i = tid; i < nt * 32; i += 256) {
            float s = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; ++w) s += so[w * RS_T * 32 + i];
            const int t = i >> 5, e = e0 + (i & 31);
            if (e < a.dv) a.o[((t0 + t) * a.H + h) * a.dv + e] = s;
        }
    }
    for (int i = warp; i < a.d; i += 8)
        if (ok) gS[(int64_t)i * a.dv] = S[i * 32 + lane];
}

// ---- one token ------------------------------------------------------------------------------------------------------------
struct RetStepArgs {
    const float *q, *k, *v, *g;      // one row each
    const float* cs;                 // cos / sin table, row = position
    const int32_t* pos_dev;
    const float* decay;
    float* state;
    float* y;                        // [H * dv]: normalized and gated
    int64_t pos, cs_rows;
    int H, d, dv, dims, cw;          // cw: state columns per CTA (<= 256)
    float kscale, eps;
};

__global__ void __launch_bounds__(256) retention_step_kernel(const RetStepArgs a) {
    extern __shared__ float sm[];
    float *sq = sm, *sk = sm + a.d, *so = sm + 2 * a.d;      // so: [256] partial outputs
    __shared__ float red[33];
    __shared__ float ssq;
    pdl_launch_dependents();
    pdl_wait();
    cg::cluster_group cl = cg::this_cluster();
    const int h = blockIdx.y, rank = (int)cl.block_rank(), nc = (int)cl.num_blocks(), tid = threadIdx.x;
    const int64_t pos = min(a.pos_dev != nullptr ? (int64_t)a.pos_dev[0] : a.pos, a.cs_rows - 1);
    const float* cs = a.cs + pos * a.dims;
    const int e0 = rank * a.cw, cw = min(a.cw, a.dv - e0);      // cw may be <= 0 on a trailing rank
    const int groups = cw > 0 ? 256 / cw : 0;
    const int grp = cw > 0 ? tid / cw : 0, col = cw > 0 ? tid - grp * cw : 0;
    const bool work = grp < groups;
    const float decay = a.decay[h];
    // the first rows of this thread's column, its value and gate are requested before q and k are staged
    constexpr int PRE = 16;
    float* S = a.state + (int64_t)h * a.d * a.dv + e0 + col;
    float pre[PRE], v = 0.0f;
#pragma unroll
    for (int j = 0; j < PRE; ++j) {
        const int i = grp + j * groups;
        pre[j] = work && i < a.d ? S[(int64_t)i * a.dv] : 0.0f;
    }
    if (work) v = a.v[(int64_t)h * a.dv + e0 + col];
    const float gate = tid < cw ? a.g[(int64_t)h * a.dv + e0 + tid] : 0.0f;
    for (int i = tid; i < a.d; i += 256) {
        sq[i] = rotated(a.q + (int64_t)h * a.d, i, a.dims, cs);
        sk[i] = rotated(a.k + (int64_t)h * a.d, i, a.dims, cs) * a.kscale;
    }
    __syncthreads();
    float part = 0.0f;
    if (work) {
#pragma unroll
        for (int j = 0; j < PRE; ++j) {
            const int i = grp + j * groups;
            if (i < a.d) {
                const float s = fmaf(decay, pre[j], sk[i] * v);
                S[(int64_t)i * a.dv] = s;
                part = fmaf(sq[i], s, part);
            }
        }
#pragma unroll 8
        for (int i = grp + PRE * groups; i < a.d; i += groups) {
            const float s = fmaf(decay, S[(int64_t)i * a.dv], sk[i] * v);
            S[(int64_t)i * a.dv] = s;
            part = fmaf(sq[i], s, part);
        }
    }
    so[tid] = part;
    __syncthreads();
    float o = 0.0f;
    if (tid < cw)
        for (int r = 0; r < groups; ++r) o += so[r * cw + tid];
    const float ss = block_sumf(o * o, red);
    float total = ss;
    if (nc > 1) {
        if (tid == 0) ssq = ss;
        cl.sync();
        total = 0.0f;
        for (int r = 0; r < nc; ++r) total += *cl.map_shared_rank(&ssq, r);
        cl.sync();
    }
    if (tid < cw) {
        const int64_t i = (int64_t)h * a.dv + e0 + tid;
        a.y[i] = o * rms_inv_f32(total, a.dv, a.eps) * silu_f32(gate);
    }
}

template <typename T>
static int run_ret_scan(const RetArgs<T>& a, cudaStream_t st) {
    const size_t smem = ((size_t)a.d * 32 + 2 * RS_T * a.d + RS_T * 32 + 8 * RS_T * 32) * 4;
    SCMX_REQUIRE(smem <= 200 * 1024, SCMX_ELIMIT, "retention: head size %d", a.d);
    if (smem > 48 * 1024)
        SCMX_CUDA_OK(cudaFuncSetAttribute(retention_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    SCMX_PDL_OK("retention_scan_kernel", launch_pdl(retention_scan_kernel<T>, dim3(a.H, (a.dv + 31) / 32), dim3(256), smem, st, a));
    return SCMX_OK;
}

}  // namespace scmx

using namespace scmx;

extern "C" int64_t scmx_retention_scratch(int64_t n, int H, int d, int dv, int dims, int64_t ldv) {
    return n > 0 && H > 0 && d > 0 && dv > 0 && retention_tc_supported(n, H, d, dv, dims, ldv) ? retention_tc_scratch(n, H, d, dv) : 0;
}

extern "C" int scmx_retention(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* v, int64_t ldv, int dt, int64_t n, int H,
                              int d, int dv, const float* cs, int dims, float kscale, const float* decay, float* state, float* o,
                              void* scratch, int64_t scratch_bytes, int32_t* status, void* stream) {
    SCMX_DT_OK("retention", dt);
    SCMX_REQUIRE(q && k && v && decay && state && o, SCMX_EINVAL, "retention: null buffer");
    SCMX_REQUIRE(n >= 0 && H > 0 && d > 0 && dv > 0 && dims >= 0 && dims <= d && dims % 2 == 0 && (dims == 0 || cs), SCMX_EINVAL,
                 "retention: n=%lld heads=%d size=%d values=%d rotated=%d", (long long)n, H, d, dv, dims);
    if (n == 0) return SCMX_OK;
    if (scratch != nullptr) {
        SCMX_REQUIRE(dt == 0 && status && retention_tc_supported(n, H, d, dv, dims, ldv), SCMX_ELIMIT,
                     "retention: no tensor-core form for head sizes %d / %d", d, dv);
        SCMX_REQUIRE(((uintptr_t)v & 15) == 0 && ((uintptr_t)scratch & 255) == 0 && scratch_bytes >= retention_tc_scratch(n, H, d, dv), SCMX_EINVAL,
                     "retention: scratch of %lld bytes or an unaligned pointer", (long long)scratch_bytes);
        return retention_tc((const bf16_t*)q, ldq, (const bf16_t*)k, ldk, (const bf16_t*)v, ldv, n, H, d, dv, cs, dims, kscale, decay, state, o,
                            scratch, status, (cudaStream_t)stream);
    }
#define FILL(T)                                                                                                           \
    RetArgs<T> a;                                                                                                          \
    a.q = (const T*)q; a.k = (const T*)k; a.v = (const T*)v; a.cs = cs; a.decay = decay; a.state = state; a.o = o;         \
    a.n = n; a.ldq = ldq; a.ldk = ldk; a.ldv = ldv; a.H = H; a.d = d; a.dv = dv; a.dims = dims; a.kscale = kscale
    if (dt == 0) {
        FILL(bf16_t);
        return run_ret_scan<bf16_t>(a, (cudaStream_t)stream);
    }
    FILL(float);
    return run_ret_scan<float>(a, (cudaStream_t)stream);
#undef FILL
}

extern "C" int scmx_retention_step(const float* q, const float* k, const float* v, const float* g, int H, int d, int dv, const float* cs,
                                   int64_t cs_rows, int dims, int64_t pos, const int32_t* pos_dev, float kscale, const float* decay,
                                   float eps, float* state, float* y, void* stream) {
    SCMX_REQUIRE(q && k && v && g && decay && state && y, SCMX_EINVAL, "retention_step: null buffer");
    SCMX_REQUIRE(H > 0 && d > 0 && dv > 0 && dims >= 0 && dims <= d && dims % 2 == 0 && (dims == 0 || cs) && cs_rows >= 1, SCMX_EINVAL,
                 "retention_step: heads=%d size=%d values=%d rotated=%d", H, d, dv, dims);
    SCMX_REQUIRE(pos_dev != nullptr || (pos >= 0 && pos < cs_rows), SCMX_EINVAL, "retention_step: position %lld outside the table of %lld rows",
                 (long long)pos, (long long)cs_rows);
    RetStepArgs a;
    a.q = q; a.k = k; a.v = v; a.g = g; a.cs = cs; a.pos_dev = pos_dev; a.decay = decay; a.state = state; a.y = y;
    a.pos = pos; a.cs_rows = cs_rows; a.H = H; a.d = d; a.dv = dv; a.dims = dims; a.kscale = kscale; a.eps = eps;
    int nc = 1;                                   // CTAs per head: slices of at least 32 columns, 256 at most
    while (nc < 8 && (dv + nc - 1) / nc > 32) nc *= 2;
    a.cw = (dv + nc - 1) / nc;
    SCMX_REQUIRE(a.cw <= 256, SCMX_ELIMIT, "retention_step: %d values per head (2048 at most)", dv);
    const size_t smem = (size_t)(2 * d + 256) * 4;
    SCMX_REQUIRE(smem <= 48 * 1024, SCMX_ELIMIT, "retention_step: head size %d", d);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(nc, H);
    cfg.blockDim = dim3(256);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = (cudaStream_t)stream;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = nc;
    at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at;
    cfg.numAttrs = g_use_pdl ? 2 : 1;
    SCMX_PDL_OK("retention_step_kernel", cudaLaunchKernelEx(&cfg, retention_step_kernel, a));
    return SCMX_OK;
}
