// Differential attention: every head has two maps over the same values; o = a1 - lambda a2, normalized over the head's values
// and scaled.  Keys are cached after their norm: K [2 G, cap, d] (map m of key/value head g at row 2 g + m), V [G, cap, dv].
//
// qk_norm_append_kernel   q / k RMS norm per head and map, K / V rows appended to the cache
// diff_attn_kernel        prompt portions, any sizes and storage types, float32 arithmetic on the CUDA cores (bfloat16 with head
//                         sizes up to 128: diff_attn_tc, tensor cores)
// diff_decode_kernel      one query row: positions split over CTAs, the last CTA of a key/value head combines
#include "mix_common.cuh"

namespace scmx {

bool diff_attn_tc_supported(int64_t n, int64_t pos, int d, int dv, float scale);
int diff_attn_tc(const bf16_t* q, const bf16_t* kc, const bf16_t* vc, int64_t n, int64_t pos, int64_t cap, int H, int G, int d, int dv, float scale,
                 float lambda, float diff, float eps, bf16_t* o, int32_t* status, cudaStream_t st);

// ---- q / k norm + cache append ------------------------------------------------------------------------------------------
template <typename TI, typename TC, typename TQ>
struct PrepArgs {
    const TI *q, *k, *v;             // [n, ld*]
    const float *qw, *kw;            // [d]
    TQ* qo;                          // [2 H, n, d]
    TC *kc, *vc;                     // caches
    const int32_t* pos_dev;
    int64_t n, ldq, ldk, ldv, pos, cap;
    int nq, nk, nv, d, dv;           // nq = 2 H, nk = 2 G, nv = G
    int lpv;                         // lanes per q / k vector in the vector form, 0: element by element
    float eps;
};

template <typename TI, typename TC, typename TQ>
__global__ void __launch_bounds__(256) qk_norm_append_kernel(const PrepArgs<TI, TC, TQ> a) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x;
    const int64_t row = (a.pos_dev != nullptr ? (int64_t)a.pos_dev[0] : a.pos) + t;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (a.lpv > 0) {
        // vectors of at most 256 elements, multiples of 8, aligned: lpv lanes (a power of two) hold 8 elements each
        const int per = 32 / a.lpv, sub = lane / a.lpv, e = 8 * (lane % a.lpv);
        for (int u0 = warp * per; u0 < a.nq + a.nk; u0 += 8 * per) {      // uniform over the warp
            const int u = u0 + sub;
            const bool ok = u < a.nq + a.nk && e < a.d, isq = u < a.nq;
            const int j = isq ? u : u - a.nq;
            float x[8] = {};
            if (ok) ld8((isq ? a.q + t * a.ldq : a.k + t * a.ldk) + (int64_t)j * a.d + e, x);
            float ss = 0.0f;
#pragma unroll
            for (int i = 0; i < 8; ++i) ss += x[i] * x[i];
            for (int o = a.lpv / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            if (!ok) continue;
            const float inv = rms_inv_f32(ss, a.d, a.eps);
            float w[8];
            ld8((isq ? a.qw : a.kw) + e, w);
#pragma unroll
            for (int i = 0; i < 8; ++i) x[i] *= inv * w[i];
            if (isq) {
                TQ* o = a.qo + ((int64_t)j * a.n + t) * a.d + e;
                st4(o, x[0], x[1], x[2], x[3]);
                st4(o + 4, x[4], x[5], x[6], x[7]);
            } else if (row < a.cap) {
                TC* o = a.kc + ((int64_t)j * a.cap + row) * a.d + e;
                st4(o, x[0], x[1], x[2], x[3]);
                st4(o + 4, x[4], x[5], x[6], x[7]);
            }
        }
        if (row < a.cap)
            for (int i = 8 * threadIdx.x; i < a.nv * a.dv; i += 2048) {
                const int j = i / a.dv, f = i - j * a.dv;
                float x[8];
                ld8(a.v + t * a.ldv + i, x);
                TC* o = a.vc + ((int64_t)j * a.cap + row) * a.dv + f;
                st4(o, x[0], x[1], x[2], x[3]);
                st4(o + 4, x[4], x[5], x[6], x[7]);
            }
        return;
    }
    for (int u = warp; u < a.nq + a.nk + a.nv; u += 8) {
        if (u < a.nq + a.nk) {
            const bool isq = u < a.nq;
            const int j = isq ? u : u - a.nq;
            const TI* p = (isq ? a.q + t * a.ldq : a.k + t * a.ldk) + (int64_t)j * a.d;
            const float* w = isq ? a.qw : a.kw;
            float ss = 0.0f;
            for (int e = lane; e < a.d; e += 32) {
                const float x = ldf(p + e);
                ss += x * x;
            }
            const float inv = rms_inv_f32(warp_sumf(ss), a.d, a.eps);
            if (isq) {
                TQ* o = a.qo + ((int64_t)j * a.n + t) * a.d;
                for (int e = lane; e < a.d; e += 32) stf(o + e, ldf(p + e) * inv * w[e]);
            } else if (row < a.cap) {                   // a device-side step beyond the cache drops the row
                TC* o = a.kc + ((int64_t)j * a.cap + row) * a.d;
                for (int e = lane; e < a.d; e += 32) stf(o + e, ldf(p + e) * inv * w[e]);
            }
        } else if (row < a.cap) {
            const int j = u - a.nq - a.nk;
            const TI* p = a.v + t * a.ldv + (int64_t)j * a.dv;
            TC* o = a.vc + ((int64_t)j * a.cap + row) * a.dv;
            for (int e = lane; e < a.dv; e += 32) stf(o + e, ldf(p + e));
        }
    }
}

// ---- prompt portions, general form --------------------------------------------------------------------------------------
template <typename T>
struct DiffAttnArgs {
    const T* q;              // [2 H, n, d]
    const T *k, *v;          // caches
    T* o;                    // [n, H dv]
    int64_t n, pos, cap;
    int H, G, d, dv;
    float scale, lambda, diff, eps;
};

constexpr int DG_Q = 16;      // query rows per CTA
constexpr int DG_K = 32;      // keys per tile

template <typename T>
__global__ void __launch_bounds__(256) diff_attn_kernel(const DiffAttnArgs<T> a) {
    extern __shared__ float sm[];
    const int d = a.d, dv = a.dv, dp = d + 1;
    float* sq = sm;                           // [2][DG_Q][d + 1]
    float* sk = sq + 2 * DG_Q * dp;           // [2][DG_K][d + 1]
    float* sv = sk + 2 * DG_K * dp;           // [DG_K][dv]
    float* sp = sv + DG_K * dv;               // [2][DG_Q][DG_K] scores, then weights
    float* so = sp + 2 * DG_Q * DG_K;         // [2][DG_Q][dv]
    float* ml = so + 2 * DG_Q * dv;           // [2][DG_Q][3]: running maximum, running sum, correction
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, g = h / (a.H / a.G), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int64_t q0 = (int64_t)blockIdx.x * DG_Q;
    const int nq = (int)min((int64_t)DG_Q, a.n - q0);
    for (int i = tid; i < 2 * DG_Q * d; i += 256) {
        const int r = i / d, e = i - r * d, m = r / DG_Q, t = r - m * DG_Q;
        sq[r * dp + e] = t < nq ? ldf(a.q + ((int64_t)(2 * h + m) * a.n + q0 + t) * d + e) * a.scale : 0.0f;
    }
    for (int i = tid; i < 2 * DG_Q * dv; i += 256) so[i] = 0.0f;
    for (int i = tid; i < 2 * DG_Q; i += 256) {
        ml[3 * i] = -INFINITY;
        ml[3 * i + 1] = 0.0f;
    }
    const int64_t last = a.pos + q0 + nq;     // first key no row of the tile sees
    for (int64_t k0 = 0; k0 < last; k0 += DG_K) {
        __syncthreads();
        for (int i = tid; i < 2 * DG_K * d; i += 256) {
            const int r = i / d, e = i - r * d, m = r / DG_K, t = r - m * DG_K;
            sk[r * dp + e] = k0 + t < last ? ldf(a.k + ((int64_t)(2 * g + m) * a.cap + k0 + t) * d + e) : 0.0f;
        }
        for (int i = tid; i < DG_K * dv; i += 256) {
            const int t = i / dv, e = i - t * dv;
            sv[i] = k0 + t < last ? ldf(a.v + ((int64_t)g * a.cap + k0 + t) * dv + e) : 0.0f;
        }
        __syncthreads();
        for (int i = tid; i < 2 * DG_Q * DG_K; i += 256) {
            const int kk = i % DG_K, r = i / DG_K, m = r / DG_Q, t = r - m * DG_Q;
            float s = 0.0f;
            for (int e = 0; e < d; ++e) s = fmaf(sq[r * dp + e], sk[(m * DG_K + kk) * dp + e], s);
            sp[i] = k0 + kk <= a.pos + q0 + t ? s : -INFINITY;
        }
        __syncthreads();
        for (int r = warp; r < 2 * DG_Q; r += 8) {      // one warp per row: DG_K = 32 scores
            const float s = sp[r * DG_K + lane], m0 = ml[3 * r], mn = fmaxf(m0, warp_max(s));
            const float p = mn == -INFINITY ? 0.0f : expf(s - mn);
            const float corr = mn == -INFINITY ? 1.0f : expf(m0 - mn), l = warp_sumf(p);
            sp[r * DG_K + lane] = p;
            __syncwarp();
            if (lane == 0) {
                ml[3 * r] = mn;
                ml[3 * r + 1] = ml[3 * r + 1] * corr + l;
                ml[3 * r + 2] = corr;
            }
        }
        __syncthreads();
        for (int i = tid; i < 2 * DG_Q * dv; i += 256) {
            const int r = i / dv, e = i - r * dv;
            float o = so[i] * ml[3 * r + 2];
#pragma unroll 8
            for (int kk = 0; kk < DG_K; ++kk) o = fmaf(sp[r * DG_K + kk], sv[kk * dv + e], o);
            so[i] = o;
        }
    }
    __syncthreads();
    for (int t = warp; t < nq; t += 8) {
        const float i1 = 1.0f / ml[3 * t + 1], i2 = a.lambda / ml[3 * (DG_Q + t) + 1];
        const float *o1 = so + t * dv, *o2 = so + (DG_Q + t) * dv;
        float ss = 0.0f;
        for (int e = lane; e < dv; e += 32) {
            const float x = o1[e] * i1 - o2[e] * i2;
            ss += x * x;
        }
        const float inv = rms_inv_f32(warp_sumf(ss), dv, a.eps) * (1.0f - a.diff);
        for (int e = lane; e < dv; e += 32) stf(a.o + ((q0 + t) * a.H + h) * dv + e, (o1[e] * i1 - o2[e] * i2) * inv);
    }
}

// ---- one query row ------------------------------------------------------------------------------------------------------
template <typename T>
struct DiffDecodeArgs {
    const float* q;          // [2 H, d]
    const T *k, *v;          // caches
    const int32_t* pos_dev;
    float* part;             // [groups, nsplit, 2 R, dv + 2]: unnormalized output, running maximum (log2), running sum
    int32_t* counters;       // [groups], zero before the first call; left at zero
    float* o;                // [H dv]
    int64_t n_pos, cap;
    int H, G, d, dv, nsplit, ct, nch;      // G: groups of query heads, nch of them per key/value head
    float scale, lambda, diff, eps;
};

constexpr int DD_P = 64;          // positions per tile
constexpr int DD_MIN_CHUNK = 64;  // positions per split at least

// Query vectors of a key/value head: 2 r + m for head r of the group, map m; QP = their number padded to 4, 8, 16 or 32.  For the
// weighted values a thread owns columns c and c + CT (CT a power of two, dv <= 2 CT) of every query vector over every
// (256 / CT)-th position of a tile, so that a value read from shared memory serves all query vectors.
template <typename T, int QP>
__global__ void __launch_bounds__(256) diff_decode_kernel(const DiffDecodeArgs<T> a) {
    extern __shared__ __align__(16) float sm[];
    const int d = a.d, dv = a.dv, R = a.H / a.G, Q = 2 * R;
    const int dq = (d + 7) & ~7;
    float* sp = sm;                          // [DD_P][QP] scores, then weights
    float* sq = sp + DD_P * QP;              // [Q][dq], zero padded
    float* sv = sq + Q * dq;                 // [DD_P][dv] values; at the end [groups][QP][2 CT] and the splits' weights
    __shared__ float ml[QP][3];              // running maximum (log2), running sum, correction
    __shared__ int ticket;
    pdl_launch_dependents();
    pdl_wait();
    const int g = blockIdx.x, kvh = g / a.nch, split = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    int64_t n = a.pos_dev != nullptr ? (int64_t)a.pos_dev[0] + 1 : a.n_pos;
    n = n < 1 ? 1 : (n > a.cap ? a.cap : n);
    int64_t chunk = (n + a.nsplit - 1) / a.nsplit;
    chunk = chunk < DD_MIN_CHUNK ? DD_MIN_CHUNK : (chunk + DD_P - 1) / DD_P * DD_P;
    const int active = (int)((n + chunk - 1) / chunk);
    if (split >= active) return;
    const int64_t t0 = split * chunk, t1 = min(n, t0 + chunk);
    for (int i = tid; i < Q * dq; i += 256) {
        const int r = i / dq, e = i - r * dq;
        sq[i] = e < d ? a.q[(int64_t)(g * Q + r) * d + e] * (a.scale * 1.4426950408889634f) : 0.0f;
    }
    for (int i = tid; i < QP; i += 256) {
        ml[i][0] = -INFINITY;
        ml[i][1] = 0.0f;
    }
    const int CT = a.ct, col = tid & (CT - 1), grp = tid / CT, groups = 256 / CT;
    const bool c1 = col + CT < dv;
    float acc[QP][2];
#pragma unroll
    for (int r = 0; r < QP; ++r) acc[r][0] = acc[r][1] = 0.0f;
    const bool vec = (d & 7) == 0, vecv = (dv & 7) == 0 && dv <= 256;
    const int p = tid >> 2, j4 = tid & 3;    // scores: four lanes per position
    for (int64_t tb = t0; tb < t1; tb += DD_P) {
        const int np = (int)min((int64_t)DD_P, t1 - tb);
        const T* vr = a.v + ((int64_t)kvh * a.cap + tb) * dv;
        // the tile's values: up to 8 loads of 8 elements per thread, in flight while the scores are computed
        constexpr int VL = sizeof(T) == 2 ? 8 : 4;
        Raw8<T> vreg[VL];
        const int nvec = DD_P * dv / 8;
        if (vecv) {
#pragma unroll
            for (int i = 0; i < VL; ++i)
                if (tid + 256 * i < nvec && 8 * (tid + 256 * i) < np * dv) vreg[i].load(vr + 8 * (tid + 256 * i));
        }
        __syncthreads();                     // queries staged; the previous tile's weights and values are consumed
        const int64_t t = tb + p;
        for (int m = 0; m < 2; ++m) {
            const T* kr = a.k + ((int64_t)(2 * kvh + m) * a.cap + (t < t1 ? t : t0)) * d;
            for (int r0 = 0; r0 < R; r0 += 4) {
                float s[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll 4
                for (int e = 8 * j4; e < dq; e += 32) {
                    float kv[8];
                    if (vec) ld8(kr + e, kv);
                    else
#pragma unroll
                        for (int i = 0; i < 8; ++i) kv[i] = e + i < d ? ldf(kr + e + i) : 0.0f;
#pragma unroll
                    for (int r = 0; r < 4; ++r)
                        if (r0 + r < R) {
                            const float4* qq = reinterpret_cast<const float4*>(sq + (2 * (r0 + r) + m) * dq + e);
                            const float4 x = qq[0], y = qq[1];
                            s[r] = fmaf(x.x, kv[0], s[r]); s[r] = fmaf(x.y, kv[1], s[r]); s[r] = fmaf(x.z, kv[2], s[r]); s[r] = fmaf(x.w, kv[3], s[r]);
                            s[r] = fmaf(y.x, kv[4], s[r]); s[r] = fmaf(y.y, kv[5], s[r]); s[r] = fmaf(y.z, kv[6], s[r]); s[r] = fmaf(y.w, kv[7], s[r]);
                        }
                }
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    s[r] += __shfl_xor_sync(0xffffffffu, s[r], 1);
                    s[r] += __shfl_xor_sync(0xffffffffu, s[r], 2);
                    if (j4 == 0 && r0 + r < R) sp[p * QP + 2 * (r0 + r) + m] = t < t1 ? s[r] : -INFINITY;
                }
            }
        }
        if (vecv) {
#pragma unroll
            for (int i = 0; i < VL; ++i) {
                const int o = 8 * (tid + 256 * i);
                if (o < 8 * nvec) {
                    float x[8] = {};
                    if (o < np * dv) vreg[i].get(x);
                    reinterpret_cast<float4*>(sv + o)[0] = make_float4(x[0], x[1], x[2], x[3]);
                    reinterpret_cast<float4*>(sv + o)[1] = make_float4(x[4], x[5], x[6], x[7]);
                }
            }
            for (int o = 8 * (tid + 256 * VL); o < 8 * nvec; o += 2048) {
                float x[8] = {};
                if (o < np * dv) ld8(vr + o, x);
                reinterpret_cast<float4*>(sv + o)[0] = make_float4(x[0], x[1], x[2], x[3]);
                reinterpret_cast<float4*>(sv + o)[1] = make_float4(x[4], x[5], x[6], x[7]);
            }
        } else {
            for (int i = tid; i < DD_P * dv; i += 256) sv[i] = i < np * dv ? ldf(vr + i) : 0.0f;
        }
        __syncthreads();
        for (int r = warp; r < Q; r += 8) {
            const float s0 = sp[lane * QP + r], s1 = sp[(32 + lane) * QP + r], m0 = ml[r][0];
            const float mn = fmaxf(m0, warp_max(fmaxf(s0, s1)));      // finite: the tile has at least one position
            const float p0 = ex2_approx(s0 - mn), p1 = ex2_approx(s1 - mn), l = warp_sumf(p0 + p1);
            sp[lane * QP + r] = p0;
            sp[(32 + lane) * QP + r] = p1;
            __syncwarp();
            if (lane == 0) {
                const float corr = ex2_approx(m0 - mn);
                ml[r][0] = mn;
                ml[r][1] = ml[r][1] * corr + l;
                ml[r][2] = corr;
            }
        }
        __syncthreads();
#pragma unroll
        for (int r = 0; r < QP; ++r)
            if (r < Q) {
                acc[r][0] *= ml[r][2];
                acc[r][1] *= ml[r][2];
            }
        if (col < dv)
#pragma unroll 4
            for (int i = grp; i < DD_P; i += groups) {
                const float v0 = sv[i * dv + col], v1 = c1 ? sv[i * dv + col + CT] : 0.0f;
#pragma unroll
                for (int r = 0; r < QP; r += 4) {
                    const float4 w = *reinterpret_cast<const float4*>(sp + i * QP + r);
                    acc[r][0] = fmaf(w.x, v0, acc[r][0]); acc[r][1] = fmaf(w.x, v1, acc[r][1]);
                    acc[r + 1][0] = fmaf(w.y, v0, acc[r + 1][0]); acc[r + 1][1] = fmaf(w.y, v1, acc[r + 1][1]);
                    acc[r + 2][0] = fmaf(w.z, v0, acc[r + 2][0]); acc[r + 2][1] = fmaf(w.z, v1, acc[r + 2][1]);
                    acc[r + 3][0] = fmaf(w.w, v0, acc[r + 3][0]); acc[r + 3][1] = fmaf(w.w, v1, acc[r + 3][1]);
                }
            }
    }
    // sum over the position groups, then this split's partial state
    __syncthreads();
#pragma unroll
    for (int r = 0; r < QP; ++r)
        if (r < Q) {
            sv[(grp * Q + r) * 2 * CT + col] = acc[r][0];
            sv[(grp * Q + r) * 2 * CT + CT + col] = acc[r][1];
        }
    __syncthreads();
    const int ps = dv + 2;
    float* part = a.part + ((int64_t)g * a.nsplit + split) * Q * ps;
    for (int i = tid; i < Q * dv; i += 256) {
        const int r = i / dv, e = i - r * dv;
        float s = 0.0f;
        for (int k = 0; k < groups; ++k) s += sv[(k * Q + r) * 2 * CT + e];
        part[r * ps + e] = s;
    }
    for (int r = tid; r < Q; r += 256) {
        part[r * ps + dv] = ml[r][0];
        part[r * ps + dv + 1] = ml[r][1];
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) ticket = atomicAdd(a.counters + g, 1);
    __syncthreads();
    if (ticket != active - 1) return;
    __threadfence();
    // the last CTA of this key/value head: weights of the splits, then both maps, the difference, its norm
    const float* pg = a.part + (int64_t)g * a.nsplit * Q * ps;
    float* cf = sv;                          // [Q][32]: 2^(m_s - m) / sum
    float* sx = sv + Q * 32;                 // [R][dv]
    for (int r = warp; r < Q; r += 8) {
        const float m = lane < active ? __ldcg(pg + ((int64_t)lane * Q + r) * ps + dv) : -INFINITY;
        const float l = lane < active ? __ldcg(pg + ((int64_t)lane * Q + r) * ps + dv + 1) : 0.0f;
        const float mm = warp_max(m), c = lane < active ? ex2_approx(m - mm) : 0.0f;
        const float sum = warp_sumf(c * l);
        cf[r * 32 + lane] = c / sum;
    }
    __syncthreads();
    for (int i = tid; i < R * dv; i += 256) {
        const int r = i / dv, e = i - r * dv;
        const float* pr = pg + 2 * r * ps + e;
        float a1 = 0.0f, a2 = 0.0f;
        for (int s0 = 0; s0 < active; s0 += 8) {
            float u[8], v[8];
#pragma unroll
            for (int s = 0; s < 8; ++s) {
                const bool ok = s0 + s < active;
                u[s] = ok ? __ldcg(pr + (int64_t)(s0 + s) * Q * ps) : 0.0f;
                v[s] = ok ? __ldcg(pr + (int64_t)(s0 + s) * Q * ps + ps) : 0.0f;
            }
#pragma unroll
            for (int s = 0; s < 8; ++s) {
                a1 = fmaf(cf[(2 * r) * 32 + s0 + s], u[s], a1);
                a2 = fmaf(cf[(2 * r + 1) * 32 + s0 + s], v[s], a2);
            }
        }
        sx[i] = a1 - a.lambda * a2;
    }
    __syncthreads();
    for (int r = warp; r < R; r += 8) {
        float ss = 0.0f;
        for (int e = lane; e < dv; e += 32) ss += sx[r * dv + e] * sx[r * dv + e];
        const float inv = rms_inv_f32(warp_sumf(ss), dv, a.eps) * (1.0f - a.diff);
        for (int e = lane; e < dv; e += 32) a.o[(int64_t)(g * R + r) * dv + e] = sx[r * dv + e] * inv;
    }
    if (tid == 0) a.counters[g] = 0;
}

template <typename T>
static int run_diff_attn(const DiffAttnArgs<T>& a, cudaStream_t st) {
    const size_t smem = ((size_t)2 * (DG_Q + DG_K) * (a.d + 1) + (size_t)(DG_K + 2 * DG_Q) * a.dv + 2 * DG_Q * DG_K + 6 * DG_Q) * 4;
    SCMX_REQUIRE(smem <= 220 * 1024, SCMX_ELIMIT, "diff_attn: head sizes %d / %d", a.d, a.dv);
    SCMX_CUDA_OK(cudaFuncSetAttribute(diff_attn_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    SCMX_PDL_OK("diff_attn_kernel", launch_pdl(diff_attn_kernel<T>, dim3((unsigned)((a.n + DG_Q - 1) / DG_Q), a.H), dim3(256), smem, st, a));
    return SCMX_OK;
}

template <typename T, int QP>
static int run_diff_decode_q(const DiffDecodeArgs<T>& a, cudaStream_t st) {
    const int Q = 2 * (a.H / a.G), groups = 256 / a.ct;
    size_t stage = (size_t)DD_P * a.dv;                                   // values, group sums, combination share this area
    stage = stage > (size_t)groups * Q * 2 * a.ct ? stage : (size_t)groups * Q * 2 * a.ct;
    stage = stage > (size_t)Q * 32 + (size_t)Q / 2 * a.dv ? stage : (size_t)Q * 32 + (size_t)Q / 2 * a.dv;
    const size_t smem = ((size_t)DD_P * QP + (size_t)Q * ((a.d + 7) & ~7) + stage) * 4;
    SCMX_REQUIRE(smem <= 220 * 1024, SCMX_ELIMIT, "diff_decode: %d query heads per key/value head of sizes %d / %d", Q / 2, a.d, a.dv);
    SCMX_CUDA_OK(cudaFuncSetAttribute(diff_decode_kernel<T, QP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    SCMX_PDL_OK("diff_decode_kernel", launch_pdl(diff_decode_kernel<T, QP>, dim3(a.G, a.nsplit), dim3(256), smem, st, a));
    return SCMX_OK;
}
template <typename T>
static int run_diff_decode(DiffDecodeArgs<T> a, cudaStream_t st) {
    // at most 16 query heads per CTA: larger groups are cut into equal parts that read the same keys and values
    const int R = a.H / a.G;
    int part = R < 16 ? R : 16;
    while (R % part) --part;
    a.nch = R / part;
    a.G *= a.nch;
    const int Q = 2 * part;
    SCMX_REQUIRE(a.dv <= 512, SCMX_ELIMIT, "diff_decode: %d values per head (512 at most)", a.dv);
    a.ct = 1;
    while (2 * a.ct < a.dv) a.ct *= 2;
    if (Q <= 4) return run_diff_decode_q<T, 4>(a, st);
    if (Q <= 8) return run_diff_decode_q<T, 8>(a, st);
    if (Q <= 16) return run_diff_decode_q<T, 16>(a, st);
    return run_diff_decode_q<T, 32>(a, st);
}

template <typename TI, typename TC, typename TQ>
static int run_prep(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* v, int64_t ldv, int64_t n, int H, int G, int d, int dv,
                    const float* qw, const float* kw, float eps, int64_t pos, const int32_t* pos_dev, void* qo, void* kc, void* vc,
                    int64_t cap, cudaStream_t st) {
    PrepArgs<TI, TC, TQ> a;
    a.q = (const TI*)q; a.k = (const TI*)k; a.v = (const TI*)v; a.qw = qw; a.kw = kw; a.qo = (TQ*)qo; a.kc = (TC*)kc; a.vc = (TC*)vc;
    a.pos_dev = pos_dev; a.n = n; a.ldq = ldq; a.ldk = ldk; a.ldv = ldv; a.pos = pos; a.cap = cap;
    a.nq = 2 * H; a.nk = 2 * G; a.nv = G; a.d = d; a.dv = dv; a.eps = eps;
    auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    a.lpv = 0;
    if (d % 8 == 0 && d <= 256 && dv % 8 == 0 && ldq % 8 == 0 && ldk % 8 == 0 && ldv % 8 == 0 && al(q) && al(k) && al(v) && al(qw) && al(kw) && al(qo)) {
        a.lpv = 1;
        while (8 * a.lpv < d) a.lpv *= 2;
    }
    SCMX_PDL_OK("qk_norm_append_kernel", launch_pdl(qk_norm_append_kernel<TI, TC, TQ>, dim3((unsigned)n), dim3(256), 0, st, a));
    return SCMX_OK;
}

}  // namespace scmx

using namespace scmx;

extern "C" int scmx_qk_norm_append(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* v, int64_t ldv, int in_dt, int cache_dt,
                                   int q_dt, int64_t n, int H, int G, int d, int dv, const float* qw, const float* kw, float eps,
                                   int64_t pos, const int32_t* pos_dev, void* q_out, void* k_cache, void* v_cache, int64_t cap, void* stream) {
    SCMX_DT_OK("qk_norm_append", in_dt);
    SCMX_DT_OK("qk_norm_append", cache_dt);
    SCMX_DT_OK("qk_norm_append", q_dt);
    SCMX_REQUIRE(q && k && v && qw && kw && q_out && k_cache && v_cache, SCMX_EINVAL, "qk_norm_append: null buffer");
    SCMX_REQUIRE(n >= 0 && H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0, SCMX_EINVAL, "qk_norm_append: heads %d / %d of %d / %d", H, G, d, dv);
    SCMX_REQUIRE(pos_dev != nullptr || (pos >= 0 && pos + n <= cap), SCMX_EINVAL, "qk_norm_append: %lld rows at %lld in a cache of %lld",
                 (long long)n, (long long)pos, (long long)cap);
    if (n == 0) return SCMX_OK;
    const cudaStream_t st = (cudaStream_t)stream;
    const int key = 4 * in_dt + 2 * cache_dt + q_dt;
#define GO(TI, TC, TQ) return run_prep<TI, TC, TQ>(q, ldq, k, ldk, v, ldv, n, H, G, d, dv, qw, kw, eps, pos, pos_dev, q_out, k_cache, v_cache, cap, st)
    if (key == 0) GO(bf16_t, bf16_t, bf16_t);      // prompt, bf16
    if (key == 5) GO(float, bf16_t, float);        // one token, bf16 cache
    if (key == 7) GO(float, float, float);         // float32
#undef GO
    SCMX_REQUIRE(false, SCMX_EINVAL, "qk_norm_append: unsupported types %d %d %d", in_dt, cache_dt, q_dt);
}

extern "C" int scmx_diff_attn(const void* q, const void* k_cache, const void* v_cache, int dt, int64_t n, int64_t pos, int64_t cap, int H, int G,
                              int d, int dv, float scale, float lambda, float diff, float eps, void* o, int form, int32_t* status, void* stream) {
    SCMX_DT_OK("diff_attn", dt);
    SCMX_REQUIRE(q && k_cache && v_cache && o, SCMX_EINVAL, "diff_attn: null buffer");
    SCMX_REQUIRE(n >= 0 && pos >= 0 && pos + n <= cap && H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0, SCMX_EINVAL,
                 "diff_attn: %lld rows at %lld in a cache of %lld, heads %d / %d of %d / %d", (long long)n, (long long)pos, (long long)cap, H, G, d, dv);
    SCMX_REQUIRE(form >= 0 && form <= 2, SCMX_EINVAL, "diff_attn: form=%d", form);
    if (n == 0) return SCMX_OK;
    const bool tc = dt == 0 && status != nullptr && diff_attn_tc_supported(n, pos, d, dv, scale);
    SCMX_REQUIRE(form != 2 || tc, SCMX_ELIMIT, "diff_attn: no tensor-core form for head sizes %d / %d", d, dv);
    if (tc && form != 1)
        return diff_attn_tc((const bf16_t*)q, (const bf16_t*)k_cache, (const bf16_t*)v_cache, n, pos, cap, H, G, d, dv, scale, lambda, diff, eps,
                            (bf16_t*)o, status, (cudaStream_t)stream);
#define FILL(T)                                                                                                           \
    DiffAttnArgs<T> a;                                                                                                     \
    a.q = (const T*)q; a.k = (const T*)k_cache; a.v = (const T*)v_cache; a.o = (T*)o; a.n = n; a.pos = pos; a.cap = cap;   \
    a.H = H; a.G = G; a.d = d; a.dv = dv; a.scale = scale; a.lambda = lambda; a.diff = diff; a.eps = eps
    if (dt == 0) {
        FILL(bf16_t);
        return run_diff_attn<bf16_t>(a, (cudaStream_t)stream);
    }
    FILL(float);
    return run_diff_attn<float>(a, (cudaStream_t)stream);
#undef FILL
}

extern "C" int scmx_diff_decode(const float* q, const void* k_cache, const void* v_cache, int dt, int64_t n_pos, const int32_t* pos_dev,
                                int64_t cap, int H, int G, int d, int dv, float scale, float lambda, float diff, float eps, int nsplit,
                                float* part, int32_t* counters, float* o, void* stream) {
    SCMX_DT_OK("diff_decode", dt);
    SCMX_REQUIRE(q && k_cache && v_cache && part && counters && o, SCMX_EINVAL, "diff_decode: null buffer");
    SCMX_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0 && nsplit >= 1 && nsplit <= 32, SCMX_EINVAL,
                 "diff_decode: heads %d / %d of %d / %d, %d splits", H, G, d, dv, nsplit);
    SCMX_REQUIRE(cap >= 1 && (pos_dev != nullptr || (n_pos >= 1 && n_pos <= cap)), SCMX_EINVAL, "diff_decode: %lld positions in a cache of %lld",
                 (long long)n_pos, (long long)cap);
#define FILL(T)                                                                                                           \
    DiffDecodeArgs<T> a;                                                                                                   \
    a.q = q; a.k = (const T*)k_cache; a.v = (const T*)v_cache; a.pos_dev = pos_dev; a.part = part; a.counters = counters;  \
    a.o = o; a.n_pos = n_pos; a.cap = cap; a.H = H; a.G = G; a.d = d; a.dv = dv; a.nsplit = nsplit;                        \
    a.scale = scale; a.lambda = lambda; a.diff = diff; a.eps = eps
    if (dt == 0) {
        FILL(bf16_t);
        return run_diff_decode<bf16_t>(a, (cudaStream_t)stream);
    }
    FILL(float);
    return run_diff_decode<float>(a, (cudaStream_t)stream);
#undef FILL
}
