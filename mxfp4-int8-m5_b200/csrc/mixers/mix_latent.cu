// Latent attention: keys and values of all heads are products of one latent vector per token, k_h = W_uk,h c and v_h = W_uv,h c,
// beside one rotated key part shared by the heads.  Cached per position: [c (R), zero padded to 8; rotated part (r), padded to 8].
// Positions may be limited to a sliding window.
//
// latent_append_kernel   norms of the query latent and of c, rotation of the shared key part, cache rows
// rotate_q_kernel        rotation of the queries' rotated parts in place (prompt portions before latent_attn_tc)
// latent_absorb_kernel   queries in the latent space: [W_uk,h^T q_h, rotated part]
// latent_rows_*_kernel   attention of such queries over the cache, positions split over CTAs (decode, short portions, float32):
//                        _mma for a bfloat16 cache, the plain one for float32
// latent_value_kernel    combination of the splits and W_uv,h
#include "../scmx_ptx.cuh"
#include "mix_common.cuh"

namespace scmx {

int latent_attn_tc(const bf16_t* q, int64_t ldq, const bf16_t* kv, int64_t ldkv, const bf16_t* rot, int64_t ldrot, int64_t n, int64_t pos, int64_t k0,
                   int64_t window, int H, int d, int r, int dv, float scale, bf16_t* o, int32_t* status, cudaStream_t st);
bool latent_attn_tc_supported(int64_t n, int64_t pos, int d, int r, int dv, float scale);

__host__ __device__ __forceinline__ int up8(int n) { return (n + 7) & ~7; }

// Element i of a vector whose pairs (2 j, 2 j + 1) are rotated; cs: the position's row, cos (dims / 2) then sin (dims / 2).
template <typename T>
__device__ __forceinline__ float rotated_pair(const T* v, int i, int dims, const float* cs) {
    const int j = i >> 1, half = dims >> 1;
    const float c = cs[j], s = cs[half + j];
    return (i & 1) == 0 ? ldf(v + i) * c - ldf(v + i + 1) * s : ldf(v + i) * c + ldf(v + i - 1) * s;
}

// ---- cache append -------------------------------------------------------------------------------------------------------
template <typename TI, typename TC, typename TQ>
struct LatentAppendArgs {
    const TI* y;                 // [n, ldy]: query latent (Q), latent (R), shared key part (r)
    const float *qw, *cw, *cs;   // norm weights, rotation table [cs_rows, r]
    TQ* cq;                      // [n, ldcq]
    TC* cache;                   // [cap, ldc]
    const int32_t* pos_dev;
    int64_t ldy, ldcq, ldc, pos, cap, cs_rows;
    int Q, R, r;
    float eps;
};
// Vectors of eight elements, up to AV_KEEP per thread in registers (sizes multiples of 8, aligned rows).
constexpr int AV_THREADS = 128, AV_KEEP = 4;
template <typename TI, typename TC, typename TQ>
__global__ void __launch_bounds__(AV_THREADS) latent_append_vec_kernel(const LatentAppendArgs<TI, TC, TQ> a) {
    __shared__ float red[2][AV_THREADS / 32];
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x, row = (a.pos_dev != nullptr ? (int64_t)a.pos_dev[0] : a.pos) + t;
    const TI* y = a.y + t * a.ldy;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nq = a.Q / 8, nv = (a.Q + a.R) / 8;
    float x[AV_KEEP][8], s0 = 0.0f, s1 = 0.0f;
#pragma unroll
    for (int k = 0; k < AV_KEEP; ++k) {
        const int v = tid + AV_THREADS * k;
        if (v < nv) {
            ld8(y + 8 * v, x[k]);
        } else {
#pragma unroll
            for (int i = 0; i < 8; ++i) x[k][i] = 0.0f;
        }
    }
#pragma unroll
    for (int k = 0; k < AV_KEEP; ++k) {
        float s = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; ++i) s = fmaf(x[k][i], x[k][i], s);
        if (tid + AV_THREADS * k < nq) s0 += s;
        else s1 += s;
    }
    s0 = warp_sumf(s0);
    s1 = warp_sumf(s1);
    if (lane == 0) {
        red[0][warp] = s0;
        red[1][warp] = s1;
    }
    __syncthreads();
    const float iq = rms_inv_f32(red[0][0] + red[0][1] + red[0][2] + red[0][3], a.Q, a.eps);
    const float ic = rms_inv_f32(red[1][0] + red[1][1] + red[1][2] + red[1][3], a.R, a.eps);
    const bool fits = row < a.cap;               // a device-side step beyond the cache drops the row
#pragma unroll
    for (int k = 0; k < AV_KEEP; ++k) {
        const int v = tid + AV_THREADS * k;
        if (v >= nv) continue;
        float w[8];
        if (v < nq) {
            ld8(a.qw + 8 * v, w);
            TQ* o = a.cq + t * a.ldcq + 8 * v;
            st4(o, x[k][0] * iq * w[0], x[k][1] * iq * w[1], x[k][2] * iq * w[2], x[k][3] * iq * w[3]);
            st4(o + 4, x[k][4] * iq * w[4], x[k][5] * iq * w[5], x[k][6] * iq * w[6], x[k][7] * iq * w[7]);
        } else if (fits) {
            ld8(a.cw + 8 * (v - nq), w);
            TC* o = a.cache + row * a.ldc + 8 * (v - nq);
            st4(o, x[k][0] * ic * w[0], x[k][1] * ic * w[1], x[k][2] * ic * w[2], x[k][3] * ic * w[3]);
            st4(o + 4, x[k][4] * ic * w[4], x[k][5] * ic * w[5], x[k][6] * ic * w[6], x[k][7] * ic * w[7]);
        }
    }
    if (!fits) return;
    const float* cs = a.cs + (row < a.cs_rows ? row : a.cs_rows - 1) * a.r;
    for (int i = tid; i < a.r; i += AV_THREADS) stf(a.cache + row * a.ldc + a.R + i, rotated_pair(y + a.Q + a.R, i, a.r, cs));
}

template <typename TI, typename TC, typename TQ>
__global__ void __launch_bounds__(256) latent_append_kernel(const LatentAppendArgs<TI, TC, TQ> a) {
    __shared__ float red[2][9];
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x, row = (a.pos_dev != nullptr ? (int64_t)a.pos_dev[0] : a.pos) + t;
    const TI *q = a.y + t * a.ldy, *c = q + a.Q, *kr = c + a.R;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float s0 = 0.0f, s1 = 0.0f;
    for (int i = tid; i < a.Q; i += 256) {
        const float x = ldf(q + i);
        s0 += x * x;
    }
    for (int i = tid; i < a.R; i += 256) {
        const float x = ldf(c + i);
        s1 += x * x;
    }
    s0 = warp_sumf(s0);
    s1 = warp_sumf(s1);
    if (lane == 0) {
        red[0][warp] = s0;
        red[1][warp] = s1;
    }
    __syncthreads();
    s0 = s1 = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
        s0 += red[0][w];
        s1 += red[1][w];
    }
    const float iq = rms_inv_f32(s0, a.Q, a.eps), ic = rms_inv_f32(s1, a.R, a.eps);
    for (int i = tid; i < a.Q; i += 256) stf(a.cq + t * a.ldcq + i, ldf(q + i) * iq * a.qw[i]);
    if (row >= a.cap) return;                    // a device-side step beyond the cache drops the row
    TC* out = a.cache + row * a.ldc;
    for (int i = tid; i < a.R; i += 256) stf(out + i, ldf(c + i) * ic * a.cw[i]);
    const float* cs = a.cs + (row < a.cs_rows ? row : a.cs_rows - 1) * a.r;
    for (int i = tid; i < a.r; i += 256) stf(out + up8(a.R) + i, rotated_pair(kr, i, a.r, cs));
}

template <typename T>
__global__ void __launch_bounds__(256) rotate_q_kernel(T* q, int64_t ldq, const float* cs, int H, int d, int r) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x;
    const float* row = cs + t * r;
    const int half = r >> 1;
    for (int i = threadIdx.x; i < H * half; i += 256) {
        const int h = i / half, j = i - h * half;
        T* p = q + t * ldq + (int64_t)h * (d + r) + d + 2 * j;
        const float u = ldf(p), v = ldf(p + 1);
        stf(p, u * row[j] - v * row[half + j]);
        stf(p + 1, v * row[j] + u * row[half + j]);
    }
}

// ---- queries in the latent space ----------------------------------------------------------------------------------------
template <typename TQ, typename TW>
struct AbsorbArgs {
    const TQ* q;                 // [n, ldq]: heads of d + r
    const TW* wuk;               // [H d, ldw]
    const float* cs;
    float* out;                  // [n, H, R + r]
    const int32_t* pos_dev;
    int64_t ldq, ldw, pos, cs_rows;
    int H, d, R, r;
};
constexpr int LB_COLS = 64;      // latent columns per CTA, two per lane; the 8 warps share the rows
template <typename TQ, typename TW>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const AbsorbArgs<TQ, TW> a) {
    __shared__ float part[8][LB_COLS];
    pdl_launch_dependents();
    const int h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int64_t t = blockIdx.z;
    const int c0 = blockIdx.x * LB_COLS, c = c0 + 2 * lane;      // the pitch covers pairs (rows are padded to 8 columns)
    const TW* w = a.wuk + (int64_t)h * a.d * a.ldw + c;
    // the first rows are requested before the previous kernel ends: weights never change
    constexpr int PRE = 16;
    float2 pre[PRE];
    auto load = [&](int e) -> float2 {
        if (sizeof(TW) == 2) {
            const uint32_t u = __ldg(reinterpret_cast<const uint32_t*>(w + (int64_t)e * a.ldw));
            return make_float2(bf16_lo(u), bf16_hi(u));
        }
        return __ldg(reinterpret_cast<const float2*>(w + (int64_t)e * a.ldw));
    };
#pragma unroll
    for (int i = 0; i < PRE; ++i) pre[i] = c < a.R && warp + 8 * i < a.d ? load(warp + 8 * i) : make_float2(0.0f, 0.0f);
    pdl_wait();
    const TQ* q = a.q + t * a.ldq + (int64_t)h * (a.d + a.r);
    float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
    for (int i = 0; i < PRE; ++i)
        if (warp + 8 * i < a.d) {
            const float x = ldf(q + warp + 8 * i);
            s0 = fmaf(pre[i].x, x, s0);
            s1 = fmaf(pre[i].y, x, s1);
        }
    if (c < a.R)
#pragma unroll 8
        for (int e = warp + 8 * PRE; e < a.d; e += 8) {
            const float x = ldf(q + e);
            const float2 u = load(e);
            s0 = fmaf(u.x, x, s0);
            s1 = fmaf(u.y, x, s1);
        }
    part[warp][2 * lane] = s0;
    part[warp][2 * lane + 1] = s1;
    __syncthreads();
    float* o = a.out + (t * a.H + h) * (a.R + a.r);
    if (tid < LB_COLS && c0 + tid < a.R) {
        float s = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; ++i) s += part[i][tid];
        o[c0 + tid] = s;
    }
    if (blockIdx.x == 0 && a.r > 0) {
        int64_t pos = (a.pos_dev != nullptr ? (int64_t)a.pos_dev[0] : a.pos) + t;
        pos = pos < a.cs_rows ? pos : a.cs_rows - 1;
        for (int i = tid; i < a.r; i += 256) o[a.R + i] = rotated_pair(q + a.d, i, a.r, a.cs + pos * a.r);
    }
}

// ---- attention of absorbed queries --------------------------------------------------------------------------------------
constexpr int LR_P = 32;         // positions per tile
constexpr int LR_SPLITS = 64;    // ranges of positions at most

// Pitch of a partial result: R values, maximum and sum, 16-byte aligned; maximum and sum start at column up4.
__host__ __device__ __forceinline__ int up4(int n) { return (n + 3) & ~3; }
__host__ __device__ __forceinline__ int part_pitch(int R) { return up4(R) + 4; }

// Positions of a row's window cut into splits of whole tiles; how many splits have any.
struct LatentSpan {
    int64_t lo, end, chunk;
    int active;
};
__device__ __forceinline__ LatentSpan latent_span(int64_t pos, int64_t cap, int64_t window, int nsplit) {
    LatentSpan s;
    s.end = (pos < cap ? pos : cap - 1) + 1;
    s.lo = window > 0 && s.end > window ? s.end - window : 0;
    s.chunk = ((s.end - s.lo + nsplit - 1) / nsplit + LR_P - 1) / LR_P * LR_P;
    s.active = (int)((s.end - s.lo + s.chunk - 1) / s.chunk);
    return s;
}

template <typename T>
struct LatentRowsArgs {
    const float* q;              // [n, H, R + r]
    const T* cache;              // [cap, ldc]
    const int32_t* pos_dev;
    float* part;                 // [n, H, nsplit, part_pitch(R)]: unnormalized latent, running maximum (log2), running sum
    int64_t pos, cap, ldc, window;
    int H, R, r, nsplit, ct;     // ct: threads across the column pairs (a power of two)
    float scale;
};

// Two neighbouring values.
__device__ __forceinline__ float2 ld2(const bf16_t* p) {
    const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
    return make_float2(bf16_lo(u), bf16_hi(u));
}
__device__ __forceinline__ float2 ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }

// Grid (splits, groups of HG heads, rows).  Scores: a warp takes four positions of a tile, lanes stride over vectors of eight
// elements, partial sums are exchanged so that every lane ends with whole ones; the next tile is requested as soon as the scores of
// one are formed (its first KEEP vectors per lane and position).  Values: a thread owns NC pairs of latent columns of all HG heads
// over every (256 / ct)-th position.
template <typename T, int HG, int NC>
__global__ void __launch_bounds__(256) latent_rows_kernel(const LatentRowsArgs<T> a) {
    extern __shared__ __align__(16) uint8_t smb[];
    const int Rp = up8(a.R), nv = (Rp + up8(a.r)) / 8;
    T* sc = reinterpret_cast<T*>(smb);                                   // [LR_P][Rp] latents of the tile; at the end column sums
    float* sq = reinterpret_cast<float*>(smb + (size_t)LR_P * Rp * sizeof(T));      // [HG][2][nv][4] (halves of eight apart)
    __shared__ __align__(16) float sp[LR_P][HG];
    __shared__ float ml[HG][3];
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h0 = blockIdx.y * HG;
    const int64_t row = blockIdx.z, pos = (a.pos_dev != nullptr ? (int64_t)a.pos_dev[0] : a.pos) + row;
    const LatentSpan span = latent_span(pos, a.cap, a.window, a.nsplit);
    if ((int)blockIdx.x >= span.active) return;
    const int64_t t0 = span.lo + blockIdx.x * span.chunk, t1 = min(span.end, t0 + span.chunk);
    for (int i = tid; i < HG * nv * 8; i += 256) {
        const int h = i / (nv * 8), e = i - h * nv * 8;
        float x = 0.0f;
        if (h0 + h < a.H) {
            const float* q = a.q + (row * a.H + h0 + h) * (a.R + a.r);
            if (e < a.R) x = q[e];
            else if (e >= Rp && e - Rp < a.r) x = q[a.R + e - Rp];
        }
        sq[((h * 2 + ((e >> 2) & 1)) * nv + (e >> 3)) * 4 + (e & 3)] = x * (a.scale * 1.4426950408889634f);
    }
    if (tid < HG) {
        ml[tid][0] = -INFINITY;
        ml[tid][1] = 0.0f;
    }
    const int col = tid & (a.ct - 1), grp = tid / a.ct, groups = 256 / a.ct;
    float acc[HG][NC][2];
#pragma unroll
    for (int h = 0; h < HG; ++h)
#pragma unroll
        for (int c = 0; c < NC; ++c) acc[h][c][0] = acc[h][c][1] = 0.0f;
    constexpr int KEEP = sizeof(T) == 2 ? 3 : 1;
    Raw8<T> raw[KEEP][4];
    auto row_of = [&](int64_t tb, int p) -> const T* {
        const int64_t t = tb + 4 * warp + p;
        return a.cache + (t < t1 ? t : t0) * a.ldc;
    };
    auto request = [&](int64_t tb) {
#pragma unroll
        for (int k = 0; k < KEEP; ++k)
            if (lane + 32 * k < nv)
#pragma unroll
                for (int p = 0; p < 4; ++p) raw[k][p].load(row_of(tb, p) + 8 * (lane + 32 * k));
    };
    request(t0);
    for (int64_t tb = t0; tb < t1; tb += LR_P) {
        __syncthreads();                         // queries staged; the previous tile is consumed
        float s[4 * HG];
#pragma unroll
        for (int i = 0; i < 4 * HG; ++i) s[i] = 0.0f;
        auto use = [&](int v, const Raw8<T> (&w)[4]) {
            float x[4][8];
#pragma unroll
            for (int p = 0; p < 4; ++p) {
                w[p].get(x[p]);
                if (8 * v < Rp) w[p].store(sc + (4 * warp + p) * Rp + 8 * v);
            }
#pragma unroll
            for (int h = 0; h < HG; ++h) {
                const float4 lo = reinterpret_cast<const float4*>(sq)[(2 * h) * nv + v], hi = reinterpret_cast<const float4*>(sq)[(2 * h + 1) * nv + v];
#pragma unroll
                for (int p = 0; p < 4; ++p) {
                    float& r = s[4 * h + p];
                    r = fmaf(x[p][0], lo.x, r); r = fmaf(x[p][1], lo.y, r); r = fmaf(x[p][2], lo.z, r); r = fmaf(x[p][3], lo.w, r);
                    r = fmaf(x[p][4], hi.x, r); r = fmaf(x[p][5], hi.y, r); r = fmaf(x[p][6], hi.z, r); r = fmaf(x[p][7], hi.w, r);
                }
            }
        };
#pragma unroll
        for (int k = 0; k < KEEP; ++k)
            if (lane + 32 * k < nv) use(lane + 32 * k, raw[k]);
        for (int v = lane + 32 * KEEP; v < nv; v += 32) {
            Raw8<T> w[4];
#pragma unroll
            for (int p = 0; p < 4; ++p) w[p].load(row_of(tb, p) + 8 * v);
            use(v, w);
        }
        if (tb + LR_P < t1) request(tb + LR_P);
        // lane bits from the highest choose which half of the sums a lane keeps; what is left is added over the remaining bits
        int idx = 0;
#pragma unroll
        for (int n = 2 * HG, off = 16; off > 0; off >>= 1, n >>= 1) {
            if (n >= 1) {
                const bool up = (lane & off) != 0;
#pragma unroll
                for (int i = 0; i < n; ++i) {
                    const float keep = up ? s[i + n] : s[i], give = up ? s[i] : s[i + n];
                    s[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
                }
                idx += up ? n : 0;
            } else {
                s[0] += __shfl_xor_sync(0xffffffffu, s[0], off);
            }
        }
        // 4 HG = 32: one sum per lane; 16: two lanes hold the same one
        sp[4 * warp + (idx & 3)][idx >> 2] = tb + 4 * warp + (idx & 3) < t1 ? s[0] : -INFINITY;
        __syncthreads();
        if (warp < HG) {
            const float x = sp[lane][warp], m0 = ml[warp][0];
            const float mn = fmaxf(m0, warp_max(x)), p = ex2_approx(x - mn), l = warp_sumf(p);      // finite: a tile has a position
            sp[lane][warp] = p;
            __syncwarp();
            if (lane == 0) {
                const float corr = ex2_approx(m0 - mn);
                ml[warp][0] = mn;
                ml[warp][1] = ml[warp][1] * corr + l;
                ml[warp][2] = corr;
            }
        }
        __syncthreads();
#pragma unroll
        for (int h = 0; h < HG; ++h)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                acc[h][c][0] *= ml[h][2];
                acc[h][c][1] *= ml[h][2];
            }
#pragma unroll 4
        for (int p = grp; p < LR_P; p += groups) {
            float w[HG];
#pragma unroll
            for (int h = 0; h < HG; h += 4) *reinterpret_cast<float4*>(w + h) = *reinterpret_cast<const float4*>(&sp[p][h]);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const int e = 2 * (col + a.ct * c);
                if (e >= Rp) continue;
                const float2 v = ld2(sc + p * Rp + e);
#pragma unroll
                for (int h = 0; h < HG; ++h) {
                    acc[h][c][0] = fmaf(w[h], v.x, acc[h][c][0]);
                    acc[h][c][1] = fmaf(w[h], v.y, acc[h][c][1]);
                }
            }
        }
    }
    // sums over the position groups, one head at a time
    float* sum = reinterpret_cast<float*>(smb);
#pragma unroll
    for (int h = 0; h < HG; ++h) {
        __syncthreads();
        if (groups > 1) {
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                sum[(grp * NC + c) * 2 * a.ct + 2 * col] = acc[h][c][0];
                sum[(grp * NC + c) * 2 * a.ct + 2 * col + 1] = acc[h][c][1];
            }
            __syncthreads();
        }
        if (h0 + h >= a.H) continue;             // uniform over the CTA
        float* part = a.part + ((row * a.H + h0 + h) * a.nsplit + blockIdx.x) * part_pitch(a.R);
        if (grp == 0) {
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const int e = 2 * (col + a.ct * c);
                float x = acc[h][c][0], y = acc[h][c][1];
                for (int g = 1; g < groups; ++g) {
                    x += sum[(g * NC + c) * 2 * a.ct + 2 * col];
                    y += sum[(g * NC + c) * 2 * a.ct + 2 * col + 1];
                }
                if (e < a.R) part[e] = x;
                if (e + 1 < a.R) part[e + 1] = y;
            }
        }
        if (tid == 0) {
            part[up4(a.R)] = ml[h][0];
            part[up4(a.R) + 1] = ml[h][1];
        }
    }
}

// The same on mma (bfloat16 cache): eight heads per CTA, tiles of 32 positions brought by cp.async a tile ahead.  Scores: positions
// are rows, heads columns, the warps share the inner index (each keeps its part of the queries, two terms, in registers) and their
// sums meet in shared memory.  Values: the weights' two terms are the rows 0-7 and 8-15 of one operand, a warp owns NTV blocks of
// eight latent columns.  KPW: 16-steps of the inner index per warp.
__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}

constexpr int LM_H = 8;
__host__ __device__ __forceinline__ int lm_pitch(int R, int r) { return (up8(R) + up8(r) + 15) / 16 * 16 + 8; }      // elements; rows fall into distinct banks

template <int KPW, int NTV>
__global__ void __launch_bounds__(256) latent_rows_mma_kernel(const LatentRowsArgs<bf16_t> a) {
    extern __shared__ __align__(16) uint8_t smb[];
    __shared__ __align__(16) float red[8][LR_P][LM_H];
    __shared__ __align__(16) bf16_t ps[2][LM_H][LR_P + 8];               // weights, high and remainder terms
    __shared__ float corr[LM_H];
    const int Rp = up8(a.R), K = Rp + up8(a.r), KS = (K + 15) / 16, pitch = lm_pitch(a.R, a.r);
    bf16_t* tile = reinterpret_cast<bf16_t*>(smb);                       // [2][LR_P][pitch]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3, h0 = blockIdx.y * LM_H;
    pdl_launch_dependents();
    if (16 * KS > K)                                                     // the last 16-step's missing columns
        for (int i = tid; i < 2 * LR_P; i += 256) *reinterpret_cast<uint4*>(tile + i * pitch + K) = make_uint4(0, 0, 0, 0);
    pdl_wait();
    const int64_t row = blockIdx.z, pos = (a.pos_dev != nullptr ? (int64_t)a.pos_dev[0] : a.pos) + row;
    const LatentSpan span = latent_span(pos, a.cap, a.window, a.nsplit);
    if ((int)blockIdx.x >= span.active) return;
    const int64_t t0 = span.lo + blockIdx.x * span.chunk, t1 = min(span.end, t0 + span.chunk);
    const int chunks = K / 8;
    auto request = [&](int64_t tb, int buf) {
        for (int i = tid; i < LR_P * chunks; i += 256) {
            const int p = i / chunks, c = i - p * chunks;
            const int64_t t = tb + p < t1 ? tb + p : t0;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(tile + (buf * LR_P + p) * pitch + 8 * c)), "l"(a.cache + t * a.ldc + 8 * c) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    request(t0, 0);
    // queries of head g, this warp's 16-steps, scaled, as two terms
    uint32_t qh[KPW][2], ql[KPW][2];
    {
        const float* q = a.q + (row * a.H + h0 + g) * (a.R + a.r);
        const bool in = h0 + g < a.H;
        const float f = a.scale * 1.4426950408889634f;
        auto at = [&](int k) -> float {
            if (!in) return 0.0f;
            if (k < a.R) return q[k];
            return k >= Rp && k - Rp < a.r ? q[a.R + k - Rp] : 0.0f;
        };
        float x[KPW][4];
#pragma unroll
        for (int i = 0; i < KPW; ++i) {
            const int k = 16 * (warp + 8 * i) + 2 * t4;
            x[i][0] = at(k); x[i][1] = at(k + 1); x[i][2] = at(k + 8); x[i][3] = at(k + 9);
        }
#pragma unroll
        for (int i = 0; i < KPW; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const float u = x[i][2 * e] * f, v = x[i][2 * e + 1] * f;
                qh[i][e] = pack_bf16x2(u, v);
                ql[i][e] = pack_bf16x2(u - bf16_lo(qh[i][e]), v - bf16_hi(qh[i][e]));
            }
    }
    float acc[NTV][4] = {};
    float m = -INFINITY, l = 0.0f;               // of head h0 + warp
    int buf = 0;
    for (int64_t tb = t0; tb < t1; tb += LR_P, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                         // the tile has arrived; the other buffer is consumed
        if (tb + LR_P < t1) request(tb + LR_P, buf ^ 1);
        const uint32_t base = smem_u32(tile + buf * LR_P * pitch);
        float s[2][4] = {};
        // a lane's address: rows 0-15 by lane % 16, the second eight columns for the upper half
        const uint32_t arow = base + 2 * ((lane & 15) * pitch + 8 * (lane >> 4));
#pragma unroll
        for (int i = 0; i < KPW; ++i)
            if (warp + 8 * i < KS)
#pragma unroll
                for (int mt = 0; mt < 2; ++mt) {
                    uint32_t x[4];
                    ldsm4(x, arow + 2 * (16 * mt * pitch + 16 * (warp + 8 * i)));
                    mma_bf16(s[mt], x[0], x[1], x[2], x[3], qh[i][0], qh[i][1]);
                    mma_bf16(s[mt], x[0], x[1], x[2], x[3], ql[i][0], ql[i][1]);
                }
#pragma unroll
        for (int mt = 0; mt < 2; ++mt) {
            *reinterpret_cast<float2*>(&red[warp][16 * mt + g][2 * t4]) = make_float2(s[mt][0], s[mt][1]);
            *reinterpret_cast<float2*>(&red[warp][16 * mt + g + 8][2 * t4]) = make_float2(s[mt][2], s[mt][3]);
        }
        __syncthreads();
        {                                        // softmax: a warp per head, a lane per position
            float x = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; ++w) x += red[w][lane][warp];
            if (tb + lane >= t1) x = -INFINITY;
            const float mn = fmaxf(m, warp_max(x)), p = ex2_approx(x - mn), c = ex2_approx(m - mn);      // finite: a tile has a position
            l = l * c + warp_sumf(p);
            m = mn;
            const bf16_t hi = f32_to_bf16(p);
            ps[0][warp][lane] = hi;
            ps[1][warp][lane] = f32_to_bf16(p - bf16_to_f32(hi));
            if (lane == 0) corr[warp] = c;
        }
        __syncthreads();
        const float c = corr[g];
#pragma unroll
        for (int j = 0; j < NTV; ++j) {
            acc[j][0] *= c; acc[j][1] *= c; acc[j][2] *= c; acc[j][3] *= c;
        }
        const uint32_t brow = base + 2 * ((lane & 15) * pitch + 8 * (lane >> 4));
#pragma unroll
        for (int kb = 0; kb < 2; ++kb) {
            const uint32_t w0 = *reinterpret_cast<const uint32_t*>(&ps[0][g][16 * kb + 2 * t4]), w1 = *reinterpret_cast<const uint32_t*>(&ps[1][g][16 * kb + 2 * t4]);
            const uint32_t w2 = *reinterpret_cast<const uint32_t*>(&ps[0][g][16 * kb + 2 * t4 + 8]), w3 = *reinterpret_cast<const uint32_t*>(&ps[1][g][16 * kb + 2 * t4 + 8]);
#pragma unroll
            for (int j = 0; j < NTV; j += 2) {
                const int col = 8 * (warp * NTV + j);
                if (col >= Rp) break;
                uint32_t v[4];                   // tokens 0-7 and 8-15 of columns col .., then of col + 8 ..
                ldsm4_t(v, brow + 2 * (16 * kb * pitch + col));
                mma_bf16(acc[j], w0, w1, w2, w3, v[0], v[1]);
                mma_bf16(acc[j + 1], w0, w1, w2, w3, v[2], v[3]);
            }
        }
    }
    const int pp = part_pitch(a.R);
    if (h0 + g < a.H) {
        float* part = a.part + ((row * a.H + h0 + g) * a.nsplit + blockIdx.x) * pp;
#pragma unroll
        for (int j = 0; j < NTV; ++j) {
            const int col = 8 * (warp * NTV + j) + 2 * t4;
            if (col < a.R) *reinterpret_cast<float2*>(part + col) = make_float2(acc[j][0] + acc[j][2], acc[j][1] + acc[j][3]);
        }
    }
    if (lane == 0 && h0 + warp < a.H) *reinterpret_cast<float2*>(a.part + ((row * a.H + h0 + warp) * a.nsplit + blockIdx.x) * pp + up4(a.R)) = make_float2(m, l);
}

// ---- combination of the splits and the value product --------------------------------------------------------------------
template <typename TW, typename TO>
struct LatentValueArgs {
    const float* part;           // [n, H, nsplit, R + 2]
    const TW* wuv;               // [H dv, ldw]
    TO* out;                     // [n, ldo]
    const int32_t* pos_dev;
    int64_t ldw, ldo, pos, cap, window;
    int H, R, dv, nsplit;
};
constexpr int LV_ROWS = 32;      // values per CTA, four per warp
template <typename TW, typename TO>
__global__ void __launch_bounds__(256) latent_value_kernel(const LatentValueArgs<TW, TO> a) {
    extern __shared__ __align__(16) float ctx[];         // [2][ldw]: halves of the sum, then the latent in the first
    __shared__ float cf[LR_SPLITS];
    pdl_launch_dependents();
    const int h = blockIdx.x, e0 = blockIdx.y * LV_ROWS, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    // the first vectors of this warp's rows are requested before the previous kernel ends: weights never change
    constexpr int ROWS = LV_ROWS / 8, PRE = sizeof(TW) == 2 ? 2 : 1;
    const TW* w = a.wuv + ((int64_t)h * a.dv + e0 + warp) * a.ldw + 8 * lane;
    Raw8<TW> pre[ROWS][PRE];
#pragma unroll
    for (int j = 0; j < ROWS; ++j)
#pragma unroll
        for (int k = 0; k < PRE; ++k)
            if (e0 + warp + 8 * j < a.dv && 8 * lane + 256 * k < a.ldw) pre[j][k].load(w + 8 * j * a.ldw + 256 * k);
    pdl_wait();
    const int64_t row = blockIdx.z, pos = (a.pos_dev != nullptr ? (int64_t)a.pos_dev[0] : a.pos) + row;
    const int active = latent_span(pos, a.cap, a.window, a.nsplit).active;
    const int pp = part_pitch(a.R);
    const float* part = a.part + (row * a.H + h) * a.nsplit * pp;
    if (warp == 0) {
        float2 ml[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int sp = lane + 32 * i;
            ml[i] = sp < active ? *reinterpret_cast<const float2*>(part + sp * pp + up4(a.R)) : make_float2(-INFINITY, 0.0f);
        }
        const float mm = warp_max(fmaxf(ml[0].x, ml[1].x)), c0 = ex2_approx(ml[0].x - mm), c1 = ex2_approx(ml[1].x - mm);
        const float inv = 1.0f / warp_sumf(c0 * ml[0].y + c1 * ml[1].y);
        cf[lane] = c0 * inv;
        cf[lane + 32] = c1 * inv;
    }
    __syncthreads();
    // two halves of the CTA take every second range, four columns per thread; the halves meet in shared memory
    {
        const int half = tid >> 7;
        for (int e0_ = 4 * (tid & 127); e0_ < a.ldw; e0_ += 512) {
            float4 s = make_float4(0, 0, 0, 0);
            if (e0_ < a.R)
#pragma unroll 16
                for (int i = half; i < active; i += 2) {
                    const float c = cf[i];
                    const float4 v = *reinterpret_cast<const float4*>(part + i * pp + e0_);
                    s.x = fmaf(c, v.x, s.x); s.y = fmaf(c, v.y, s.y); s.z = fmaf(c, v.z, s.z); s.w = fmaf(c, v.w, s.w);
                }
            // columns from R on are not results
            if (e0_ + 1 >= a.R) s.y = 0.0f;
            if (e0_ + 2 >= a.R) s.z = 0.0f;
            if (e0_ + 3 >= a.R) s.w = 0.0f;
            *reinterpret_cast<float4*>(ctx + half * a.ldw + e0_) = s;
        }
        __syncthreads();
        for (int e = tid; e < a.ldw; e += 256) ctx[e] += ctx[a.ldw + e];
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int e = e0 + warp + 8 * j;
        if (e >= a.dv) continue;
        float s = 0.0f;
        auto add = [&](const Raw8<TW>& u, int i) {
            float v[8];
            u.get(v);
#pragma unroll
            for (int k = 0; k < 8; ++k) s = fmaf(v[k], ctx[i + k], s);
        };
#pragma unroll
        for (int k = 0; k < PRE; ++k)
            if (8 * lane + 256 * k < a.ldw) add(pre[j][k], 8 * lane + 256 * k);
        for (int i = 8 * lane + 256 * PRE; i < a.ldw; i += 256) {
            Raw8<TW> u;
            u.load(w + 8 * j * a.ldw + (i - 8 * lane));
            add(u, i);
        }
        s = warp_sumf(s);
        if (lane == 0) stf(a.out + row * a.ldo + (int64_t)h * a.dv + e, s);
    }
}

template <typename T, int HG, int NC>
static int run_latent_rows(LatentRowsArgs<T> a, int64_t n, cudaStream_t st) {
    const int Rp = up8(a.R), nv = (Rp + up8(a.r)) / 8;
    a.ct = 1;
    while (a.ct < 256 && 2 * a.ct * NC < Rp) a.ct *= 2;
    size_t head = (size_t)LR_P * Rp * sizeof(T);
    const size_t smem = head + (size_t)HG * nv * 32;
    const size_t sums = (size_t)(256 / a.ct) * NC * 2 * a.ct * 4;      // overlays latents and queries
    const size_t total = smem > sums ? smem : sums;
    SCMX_REQUIRE(total <= 200 * 1024, SCMX_ELIMIT, "latent_rows: latent size %d", a.R);
    SCMX_CUDA_OK(cudaFuncSetAttribute(latent_rows_kernel<T, HG, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)total));
    SCMX_PDL_OK("latent_rows_kernel", launch_pdl(latent_rows_kernel<T, HG, NC>, dim3(a.nsplit, (a.H + HG - 1) / HG, (unsigned)n), dim3(256), total, st, a));
    return SCMX_OK;
}

template <int KPW, int NTV>
static int run_latent_mma_n(const LatentRowsArgs<bf16_t>& a, int64_t n, cudaStream_t st) {
    const size_t smem = (size_t)2 * LR_P * lm_pitch(a.R, a.r) * 2;
    SCMX_CUDA_OK(cudaFuncSetAttribute(latent_rows_mma_kernel<KPW, NTV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    SCMX_PDL_OK("latent_rows_mma_kernel", launch_pdl(latent_rows_mma_kernel<KPW, NTV>, dim3(a.nsplit, (a.H + LM_H - 1) / LM_H, (unsigned)n), dim3(256), smem, st, a));
    return SCMX_OK;
}
static int run_latent_mma(const LatentRowsArgs<bf16_t>& a, int64_t n, cudaStream_t st) {
    const int KS = (up8(a.R) + up8(a.r) + 15) / 16;
    SCMX_REQUIRE(KS <= 72, SCMX_ELIMIT, "latent_rows: latent size %d and rotated part %d", a.R, a.r);
    if (KS <= 8 && a.R <= 128) return run_latent_mma_n<1, 2>(a, n, st);
    if (KS <= 40 && a.R <= 512) return run_latent_mma_n<5, 8>(a, n, st);
    return run_latent_mma_n<9, 16>(a, n, st);
}

template <typename TI, typename TC, typename TQ>
static int run_append(const void* y, int64_t ldy, int64_t n, int Q, int R, int r, const float* qw, const float* cw, const float* cs, int64_t cs_rows,
                      float eps, int64_t pos, const int32_t* pos_dev, void* cq, int64_t ldcq, void* cache, int64_t ldc, int64_t cap, cudaStream_t st) {
    LatentAppendArgs<TI, TC, TQ> a;
    a.y = (const TI*)y; a.qw = qw; a.cw = cw; a.cs = cs; a.cq = (TQ*)cq; a.cache = (TC*)cache; a.pos_dev = pos_dev; a.ldy = ldy; a.ldcq = ldcq; a.ldc = ldc;
    a.pos = pos; a.cap = cap; a.cs_rows = cs_rows; a.Q = Q; a.R = R; a.r = r; a.eps = eps;
    auto al = [](const void* x) { return ((uintptr_t)x & 15) == 0; };
    if (Q % 8 == 0 && R % 8 == 0 && (Q + R) / 8 <= AV_THREADS * AV_KEEP && ldy % 8 == 0 && ldcq % 8 == 0 && ldc % 8 == 0 && al(y) && al(qw) && al(cw) &&
        al(cq) && al(cache)) {
        SCMX_PDL_OK("latent_append_kernel", launch_pdl(latent_append_vec_kernel<TI, TC, TQ>, dim3((unsigned)n), dim3(AV_THREADS), 0, st, a));
        return SCMX_OK;
    }
    SCMX_PDL_OK("latent_append_kernel", launch_pdl(latent_append_kernel<TI, TC, TQ>, dim3((unsigned)n), dim3(256), 0, st, a));
    return SCMX_OK;
}

template <typename TQ, typename TW>
static int run_absorb(const void* q, int64_t ldq, const void* wuk, int64_t ldw, const float* cs, int64_t cs_rows, int64_t n, int H, int d, int R, int r,
                      int64_t pos, const int32_t* pos_dev, float* out, cudaStream_t st) {
    AbsorbArgs<TQ, TW> a;
    a.q = (const TQ*)q; a.wuk = (const TW*)wuk; a.cs = cs; a.out = out; a.pos_dev = pos_dev; a.ldq = ldq; a.ldw = ldw; a.pos = pos; a.cs_rows = cs_rows;
    a.H = H; a.d = d; a.R = R; a.r = r;
    SCMX_PDL_OK("latent_absorb_kernel", launch_pdl(latent_absorb_kernel<TQ, TW>, dim3((R + LB_COLS - 1) / LB_COLS, H, (unsigned)n), dim3(256), 0, st, a));
    return SCMX_OK;
}

}  // namespace scmx

using namespace scmx;

#define LATENT_ROWS_OK(who, n) SCMX_REQUIRE((n) >= 0 && (n) <= 65535, SCMX_ELIMIT, "%s: %lld rows", who, (long long)(n))

extern "C" int scmx_latent_append(const void* y, int64_t ldy, int in_dt, int cache_dt, int q_dt, int64_t n, int Q, int R, int r, const float* qw,
                                  const float* cw, const float* cs, int64_t cs_rows, float eps, int64_t pos, const int32_t* pos_dev, void* cq,
                                  int64_t ldcq, void* cache, int64_t ldc, int64_t cap, void* stream) {
    SCMX_DT_OK("latent_append", in_dt);
    SCMX_DT_OK("latent_append", cache_dt);
    SCMX_DT_OK("latent_append", q_dt);
    SCMX_REQUIRE(y && qw && cw && cq && cache && (r == 0 || cs), SCMX_EINVAL, "latent_append: null buffer");
    SCMX_REQUIRE(Q > 0 && R > 0 && r >= 0 && r % 2 == 0 && ldy >= Q + R + r && ldcq >= Q && ldc >= up8(R) + up8(r) && cs_rows >= 1, SCMX_EINVAL,
                 "latent_append: sizes %d, %d, %d", Q, R, r);
    SCMX_REQUIRE(pos_dev != nullptr || (pos >= 0 && pos + n <= cap && pos + n <= cs_rows), SCMX_EINVAL,
                 "latent_append: %lld rows at %lld in a cache of %lld, table of %lld", (long long)n, (long long)pos, (long long)cap, (long long)cs_rows);
    if (n == 0) return SCMX_OK;
    const int key = 4 * in_dt + 2 * cache_dt + q_dt;
#define GO(TI, TC, TQ) return run_append<TI, TC, TQ>(y, ldy, n, Q, R, r, qw, cw, cs, cs_rows, eps, pos, pos_dev, cq, ldcq, cache, ldc, cap, (cudaStream_t)stream)
    if (key == 0) GO(bf16_t, bf16_t, bf16_t);      // prompt, bf16
    if (key == 5) GO(float, bf16_t, float);        // one token, bf16 cache
    if (key == 7) GO(float, float, float);         // float32
#undef GO
    SCMX_REQUIRE(false, SCMX_EINVAL, "latent_append: unsupported types %d %d %d", in_dt, cache_dt, q_dt);
}

extern "C" int scmx_latent_rotate(void* q, int64_t ldq, int dt, const float* cs, int64_t n, int H, int d, int r, void* stream) {
    SCMX_DT_OK("latent_rotate", dt);
    SCMX_REQUIRE(q && (r == 0 || cs) && n >= 0 && H > 0 && d >= 0 && r >= 0 && r % 2 == 0 && ldq >= (int64_t)H * (d + r), SCMX_EINVAL, "latent_rotate: heads of %d + %d", d, r);
    if (n == 0 || r == 0) return SCMX_OK;
    if (dt == 0) SCMX_PDL_OK("rotate_q_kernel", launch_pdl(rotate_q_kernel<bf16_t>, dim3((unsigned)n), dim3(256), 0, (cudaStream_t)stream, (bf16_t*)q, ldq, cs, H, d, r));
    else SCMX_PDL_OK("rotate_q_kernel", launch_pdl(rotate_q_kernel<float>, dim3((unsigned)n), dim3(256), 0, (cudaStream_t)stream, (float*)q, ldq, cs, H, d, r));
    return SCMX_OK;
}

extern "C" int scmx_latent_absorb(const void* q, int64_t ldq, int q_dt, const void* wuk, int64_t ldw, int w_dt, const float* cs, int64_t cs_rows,
                                  int64_t n, int H, int d, int R, int r, int64_t pos, const int32_t* pos_dev, float* out, void* stream) {
    SCMX_DT_OK("latent_absorb", q_dt);
    SCMX_DT_OK("latent_absorb", w_dt);
    LATENT_ROWS_OK("latent_absorb", n);
    SCMX_REQUIRE(q && wuk && out && (r == 0 || cs) && H > 0 && d > 0 && R > 0 && r >= 0 && r % 2 == 0 && ldw % 8 == 0 && ldw >= R && cs_rows >= 1 &&
                 ((uintptr_t)wuk & 15) == 0, SCMX_EINVAL, "latent_absorb: heads of %d + %d, latent %d", d, r, R);
    SCMX_REQUIRE(pos_dev != nullptr || (pos >= 0 && pos + n <= cs_rows), SCMX_EINVAL, "latent_absorb: position %lld outside the table of %lld rows",
                 (long long)(pos + n), (long long)cs_rows);
    if (n == 0) return SCMX_OK;
    const cudaStream_t st = (cudaStream_t)stream;
#define GO(TQ, TW) return run_absorb<TQ, TW>(q, ldq, wuk, ldw, cs, cs_rows, n, H, d, R, r, pos, pos_dev, out, st)
    if (q_dt == 0 && w_dt == 0) GO(bf16_t, bf16_t);
    if (q_dt == 1 && w_dt == 0) GO(float, bf16_t);
    if (q_dt == 1 && w_dt == 1) GO(float, float);
#undef GO
    SCMX_REQUIRE(false, SCMX_EINVAL, "latent_absorb: unsupported types %d %d", q_dt, w_dt);
}

extern "C" int scmx_latent_rows(const float* q, const void* cache, int64_t ldc, int dt, int64_t n, int64_t pos, const int32_t* pos_dev, int64_t cap,
                                int64_t window, int H, int R, int r, float scale, int nsplit, float* part, void* stream) {
    SCMX_DT_OK("latent_rows", dt);
    LATENT_ROWS_OK("latent_rows", n);
    SCMX_REQUIRE(q && cache && part && H > 0 && R > 0 && r >= 0 && ldc % 8 == 0 && ldc >= up8(R) + up8(r) && ((uintptr_t)cache & 15) == 0, SCMX_EINVAL,
                 "latent_rows: heads %d, latent %d, rotated %d, pitch %lld", H, R, r, (long long)ldc);
    SCMX_REQUIRE(nsplit >= 1 && nsplit <= LR_SPLITS && window >= 0 && cap >= 1, SCMX_EINVAL, "latent_rows: %d splits, window %lld", nsplit, (long long)window);
    SCMX_REQUIRE(pos_dev != nullptr || (pos >= 0 && pos + n <= cap), SCMX_EINVAL, "latent_rows: %lld rows at %lld in a cache of %lld", (long long)n,
                 (long long)pos, (long long)cap);
    SCMX_REQUIRE(R <= 1024, SCMX_ELIMIT, "latent_rows: latent size %d (1024 at most)", R);
    if (n == 0) return SCMX_OK;
#define FILL(T)                                                                                                           \
    LatentRowsArgs<T> a;                                                                                                   \
    a.q = q; a.cache = (const T*)cache; a.pos_dev = pos_dev; a.part = part; a.pos = pos; a.cap = cap; a.ldc = ldc;         \
    a.window = window; a.H = H; a.R = R; a.r = r; a.nsplit = nsplit; a.ct = 0; a.scale = scale;
    if (dt == 0) {
        FILL(bf16_t);
        return run_latent_mma(a, n, (cudaStream_t)stream);
    }
    FILL(float);
    return R <= 512 ? run_latent_rows<float, 8, 1>(a, n, (cudaStream_t)stream) : run_latent_rows<float, 8, 2>(a, n, (cudaStream_t)stream);
#undef FILL
}

extern "C" int scmx_latent_value(const float* part, const void* wuv, int64_t ldw, int w_dt, int64_t n, int64_t pos, const int32_t* pos_dev, int64_t cap,
                                 int64_t window, int H, int R, int dv, int nsplit, void* out, int64_t ldo, int out_dt, void* stream) {
    SCMX_DT_OK("latent_value", w_dt);
    SCMX_DT_OK("latent_value", out_dt);
    LATENT_ROWS_OK("latent_value", n);
    SCMX_REQUIRE(part && wuv && out && H > 0 && R > 0 && dv > 0 && ldw % 8 == 0 && ldw >= R && ldw <= 4096 && ((uintptr_t)wuv & 15) == 0 &&
                 ldo >= (int64_t)H * dv && nsplit >= 1 && nsplit <= LR_SPLITS && window >= 0 && cap >= 1, SCMX_EINVAL, "latent_value: heads %d of %d, latent %d", H, dv, R);
    SCMX_REQUIRE(pos_dev != nullptr || (pos >= 0 && pos + n <= cap), SCMX_EINVAL, "latent_value: %lld rows at %lld in a cache of %lld", (long long)n,
                 (long long)pos, (long long)cap);
    if (n == 0) return SCMX_OK;
    const dim3 grid(H, (dv + LV_ROWS - 1) / LV_ROWS, (unsigned)n), block(256);
#define GO(TW, TO)                                                                                                        \
    do {                                                                                                                   \
        LatentValueArgs<TW, TO> a;                                                                                         \
        a.part = part; a.wuv = (const TW*)wuv; a.out = (TO*)out; a.pos_dev = pos_dev; a.ldw = ldw; a.ldo = ldo; a.pos = pos; \
        a.cap = cap; a.window = window; a.H = H; a.R = R; a.dv = dv; a.nsplit = nsplit;                                    \
        SCMX_PDL_OK("latent_value_kernel", launch_pdl(latent_value_kernel<TW, TO>, grid, block, (size_t)ldw * 8, (cudaStream_t)stream, a)); \
        return SCMX_OK;                                                                                                    \
    } while (0)
    if (w_dt == 0 && out_dt == 0) GO(bf16_t, bf16_t);
    if (w_dt == 0 && out_dt == 1) GO(bf16_t, float);
    if (w_dt == 1 && out_dt == 1) GO(float, float);
#undef GO
    SCMX_REQUIRE(false, SCMX_EINVAL, "latent_value: unsupported types %d %d", w_dt, out_dt);
}

extern "C" int scmx_latent_attn(const void* q, int64_t ldq, const void* kv, int64_t ldkv, const void* rot, int64_t ldrot, int64_t n, int64_t pos,
                                int64_t k0, int64_t window, int H, int d, int r, int dv, float scale, void* o, int32_t* status, void* stream) {
    SCMX_REQUIRE(q && kv && o && status && (r == 0 || rot), SCMX_EINVAL, "latent_attn: null buffer");
    SCMX_REQUIRE(n >= 0 && H > 0 && pos >= 0 && window >= 0 && k0 >= 0 && k0 <= (window > 0 && pos + 1 > window ? pos + 1 - window : 0), SCMX_EINVAL,
                 "latent_attn: keys from %lld on for rows at %lld with a window of %lld", (long long)k0, (long long)pos, (long long)window);
    SCMX_REQUIRE(ldq % 8 == 0 && ldkv % 8 == 0 && ldrot % 8 == 0 && ldq >= (int64_t)H * (d + r) && ldkv >= (int64_t)H * (d + dv) &&
                 (((uintptr_t)q | (uintptr_t)kv | (uintptr_t)rot | (uintptr_t)o) & 15) == 0, SCMX_EINVAL, "latent_attn: pitches %lld, %lld, %lld",
                 (long long)ldq, (long long)ldkv, (long long)ldrot);
    SCMX_REQUIRE(latent_attn_tc_supported(n, pos, d, r, dv, scale), SCMX_ELIMIT, "latent_attn: head sizes %d + %d / %d", d, r, dv);
    if (n == 0) return SCMX_OK;
    return latent_attn_tc((const bf16_t*)q, ldq, (const bf16_t*)kv, ldkv, (const bf16_t*)rot, ldrot, n, pos, k0, window, H, d, r, dv, scale, (bf16_t*)o, status,
                          (cudaStream_t)stream);
}
