// Gated delta rule of prompt portions on tcgen05 (bfloat16 activations, d up to 128, sizes multiples of 8), in chunks of 64 tokens.
// With a chunk's inclusive decay products c_i (per key channel or per head), every correction u_i = beta_i (v_i - S^T k_i) depends
// on the state S at the chunk's start and on the earlier corrections:
//   (I + N) U = beta (V - (c K) S),   N_ij = beta_i (k_i . c_i / c_j k_j) for j < i,   T = (I + N)^-1 diag(beta)
//   U = T V - W S,  W = T (c K);   O = (c Q) S + B U,  B_ij = q_i . c_i / c_j k_j for j <= i;   S' = c_end S + E^T U,  E = c_end / c K
//
// delta_prep_kernel    per chunk and head, all in parallel: unit vectors, decays, N, B, T, W.  Ratios c_i / c_j are formed by running
//                      products of decays, so nothing overflows however strong the decay is
// delta_state_kernel   per head and 128 values, chunk after chunk: S^T lives in tensor memory (a lane per value), three products per
//                      chunk with S or U as the tensor-memory operand
// Operands that enter the recurrence are stored as two bfloat16 terms (16 significant bits; three MMAs per product, two with V,
// which is bfloat16 as projected); S itself is carried in float32.  Waits are bounded (status word codes 61..64).
#include "mix_delta.cuh"
#include "mix_tc.cuh"

namespace scmx {

constexpr int DC = 64;                   // tokens per chunk
constexpr int DC_BLK = 64 * 128;         // bytes of a [64 rows x 64 values] operand block
constexpr int DP_THREADS = 512;
constexpr int DP_PITCH = 68;             // row pitch of the 64 x 64 matrices in shared memory

struct DeltaTcArgs {
    DeltaArgs p;
    bf16_t *wh, *wl, *qh, *ql, *eh, *el;     // [items][64][D]: -W, c Q, E
    bf16_t *th, *tl, *bh, *bl;               // [items][64][64]
    float* gend;                             // [items][D]: c at the chunk's end
    int32_t* status;
    uint64_t wait_ns;
    int nc;                                  // chunks; item = chunk * H + head
};

// Two or four values as two bfloat16 terms.
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16x2(x, y);
    lo = pack_bf16x2(x - bf16_lo(hi), y - bf16_hi(hi));
}

// D = A B + D, 16 x 8 x 16, bfloat16 operands.
__device__ __forceinline__ void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// The same with both operands in two terms (three products).
__device__ __forceinline__ void mma_split(float (&d)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[2], const uint32_t (&bl)[2]) {
    mma_16816(d, ah, bh[0], bh[1]);
    mma_16816(d, ah, bl[0], bl[1]);
    mma_16816(d, al, bh[0], bh[1]);
}

// Shared memory of the preparation, in floats.  Per channel decays: K, Q, G hold k, q, g, later k f, q f, k e with the decay products
// f from the start of a block of 16 tokens and e to its end; PB the products of whole blocks.  One decay per head: K, Q stay, the
// products are per token (F, E), RAT holds the ratios within a block.
template <int D, bool CH>
struct DpSmem {
    static constexpr int P = D + 16;         // row pitch: eight lanes of a 128-bit load fall into distinct banks
    static constexpr int K = 0, Q = K + 64 * P, G = Q + 64 * P, N = G + (CH ? 64 * P : 64), B = N + 64 * DP_PITCH, X = B + 64 * DP_PITCH,
                         T = X + 64 * DP_PITCH, BETA = T + 32 * 36, PB = BETA + 64, F = PB + (CH ? 4 * D : 64), E = F + 64, RAT = E + 64,
                         FLOATS = RAT + (CH ? 0 : 64 * 17);
};

__device__ __forceinline__ void split4(const float4 v, uint32_t& h0, uint32_t& h1, uint32_t& l0, uint32_t& l1) {
    split2(v.x, v.y, h0, l0);
    split2(v.z, v.w, h1, l1);
}
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float4 mul4(float4 a, float b) { return make_float4(a.x * b, a.y * b, a.z * b, a.w * b); }
__device__ __forceinline__ void half_bar() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

template <int D, bool CH>
__global__ void __launch_bounds__(DP_THREADS, 1) delta_prep_kernel(const DeltaTcArgs a) {
    using L = DpSmem<D, CH>;
    constexpr int P = L::P;
    extern __shared__ __align__(16) float sm[];
    float *sk = sm + L::K, *sq = sm + L::Q, *sg = sm + L::G, *sN = sm + L::N, *sB = sm + L::B, *sX = sm + L::X, *sT = sm + L::T;
    float *beta = sm + L::BETA, *pb = sm + L::PB, *sf = sm + L::F, *se = sm + L::E, *rat = sm + L::RAT;
    pdl_launch_dependents();
    pdl_wait();
    const DeltaArgs& p = a.p;
    const int item = blockIdx.x, h = item % p.H, kh = h / (p.H / p.G);
    const int64_t t0 = (int64_t)(item / p.H) * DC;
    const int nt = (int)min((int64_t)DC, p.n - t0);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    // ---- unit vectors, decays, beta; tokens past the end become neutral (k = q = 0, beta = 0, decay 1)
    {
        constexpr int V = D / 32;
        const int e = V * lane;
        const bool in = e < p.d;
        const bf16_t *q = static_cast<const bf16_t*>(p.q) + (int64_t)kh * p.d + e, *k = static_cast<const bf16_t*>(p.k) + (int64_t)kh * p.d + e;
        float x[4][V], y[4][V], z[4][V], bl = 0.0f, al = 0.0f, dtb[V];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int t = warp + 16 * r;
#pragma unroll
            for (int i = 0; i < V; ++i) x[r][i] = y[r][i] = z[r][i] = 0.0f;
            if (t < nt && in) {
                // rows are 4-byte aligned, decay rows 8-byte (host side)
#pragma unroll
                for (int i = 0; i < V; i += 2) {
                    const uint32_t u = *reinterpret_cast<const uint32_t*>(q + (t0 + t) * p.ldq + i), w = *reinterpret_cast<const uint32_t*>(k + (t0 + t) * p.ldk + i);
                    x[r][i] = bf16_lo(u); x[r][i + 1] = bf16_hi(u);
                    y[r][i] = bf16_lo(w); y[r][i + 1] = bf16_hi(w);
                    if (CH) {
                        const float2 v = *reinterpret_cast<const float2*>(static_cast<const float*>(p.a) + (t0 + t) * p.lda + (int64_t)h * p.d + e + i);
                        z[r][i] = v.x; z[r][i + 1] = v.y;
                    }
                }
            }
            if (lane == r && t < nt) {           // lane r keeps token r's scalars
                bl = ldf(static_cast<const bf16_t*>(p.b) + (t0 + t) * p.ldb + h);
                if (!CH) al = ldf(static_cast<const bf16_t*>(p.a) + (t0 + t) * p.lda + h);
            }
        }
        const float qs = rsqrtf((float)p.d), nA2 = p.nA[h] * 1.4426950408889634f;
#pragma unroll
        for (int i = 0; i < V; ++i) dtb[i] = CH ? (in ? p.dtb[(int64_t)h * p.d + e + i] : 0.0f) : p.dtb[h];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int t = warp + 16 * r;
            float qq = 0.0f, kk = 0.0f;
#pragma unroll
            for (int i = 0; i < V; ++i) {
                qq = fmaf(x[r][i], x[r][i], qq);
                kk = fmaf(y[r][i], y[r][i], kk);
            }
            // two sums in six shuffles: the halves of the warp take one each
            const bool up = (lane & 16) != 0;
            float s = (up ? kk : qq) + __shfl_xor_sync(0xffffffffu, up ? qq : kk, 16);
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
            const float other = __shfl_xor_sync(0xffffffffu, s, 16);
            const float iq = qs * rsqrtf((up ? other : s) + 1e-6f), ik = rsqrtf((up ? s : other) + 1e-6f);
#pragma unroll
            for (int i = 0; i < V; ++i) {
                sq[t * P + e + i] = x[r][i] * iq;
                sk[t * P + e + i] = y[r][i] * ik;
                if (CH) sg[t * P + e + i] = t < nt ? ex2_approx(nA2 * softplus_f32(z[r][i] + dtb[i])) : 1.0f;
            }
        }
        if (lane < 4) {
            const int t = warp + 16 * lane;
            beta[t] = t < nt ? sigmoid_f32(bl) : 0.0f;
            if (!CH) sg[t] = t < nt ? ex2_approx(nA2 * softplus_f32(al + dtb[0])) : 1.0f;
        }
    }
    __syncthreads();
    if (CH) {
        // ---- diagonal blocks of N and B: a warp carries four keys j of a block, c_i / c_j k_j, from i = j on; lanes split the channels
        constexpr int V = D / 32;
        const int b0 = 16 * (warp >> 2), jg = 4 * (warp & 3);
        float kc[4][V];
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int i = 0; i < V; ++i) kc[j][i] = sk[(b0 + jg + j) * P + V * lane + i];
        for (int i0 = jg; i0 < 16; i0 += 4) {
            float s[32];
#pragma unroll
            for (int ii = 0; ii < 4; ++ii) {
                const int o = (b0 + i0 + ii) * P + V * lane;
                float k[V], q[V], g[V];
                if (V == 4) {
                    *reinterpret_cast<float4*>(k) = *reinterpret_cast<const float4*>(sk + o);
                    *reinterpret_cast<float4*>(q) = *reinterpret_cast<const float4*>(sq + o);
                    *reinterpret_cast<float4*>(g) = *reinterpret_cast<const float4*>(sg + o);
                } else {
                    *reinterpret_cast<float2*>(k) = *reinterpret_cast<const float2*>(sk + o);
                    *reinterpret_cast<float2*>(q) = *reinterpret_cast<const float2*>(sq + o);
                    *reinterpret_cast<float2*>(g) = *reinterpret_cast<const float2*>(sg + o);
                }
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    float n = 0.0f, m = 0.0f;
#pragma unroll
                    for (int i = 0; i < V; ++i) {
                        if (i0 > jg || ii > j) kc[j][i] *= g[i];
                        n = fmaf(kc[j][i], k[i], n);
                        m = fmaf(kc[j][i], q[i], m);
                    }
                    s[8 * ii + 2 * j] = n;
                    s[8 * ii + 2 * j + 1] = m;
                }
            }
            // 32 sums over the warp, one per lane: lane bits from the highest choose the half that a lane keeps
#pragma unroll
            for (int n = 16; n > 0; n >>= 1) {
                const bool up = (lane & n) != 0;
#pragma unroll
                for (int i = 0; i < n; ++i) {
                    const float keep = up ? s[i + n] : s[i], give = up ? s[i] : s[i + n];
                    s[i] = keep + __shfl_xor_sync(0xffffffffu, give, n);
                }
            }
            const int i = b0 + i0 + (lane >> 3), j = b0 + jg + ((lane >> 1) & 3);
            if (lane & 1) {
                if (i >= j) sB[i * DP_PITCH + j] = s[0];
            } else if (i > j) {
                sN[i * DP_PITCH + j] = beta[i] * s[0];
            }
        }
        __syncthreads();
        // ---- decay products within the blocks, a thread per channel and block
        for (int u = tid; u < 4 * D; u += DP_THREADS) {
            const int c = u % D, b = u / D;
            float *k = sk + 16 * b * P + c, *q = sq + 16 * b * P + c, *g = sg + 16 * b * P + c;
            float kk[16], gg[16], f = 1.0f, e = 1.0f;
#pragma unroll
            for (int t = 0; t < 16; ++t) {
                kk[t] = k[t * P];
                gg[t] = g[t * P];
            }
#pragma unroll
            for (int t = 0; t < 16; ++t) {
                f *= gg[t];
                k[t * P] = kk[t] * f;
                q[t * P] *= f;
            }
            pb[b * D + c] = f;
#pragma unroll
            for (int t = 15; t >= 0; --t) {
                g[t * P] = kk[t] * e;
                e *= gg[t];
            }
        }
    } else {
        // ---- the same per token: products from the block's start, to its end, and between its tokens
        if (tid < 64) {
            const int b0 = tid & ~15, j = tid & 15;
            float f = 1.0f, e = 1.0f, r = 1.0f;
            for (int t = 0; t < 16; ++t) {
                const float g = sg[b0 + t];
                if (t <= j) f *= g;
                if (t > j) {
                    e *= g;
                    r *= g;
                }
                rat[tid * 17 + t] = r;           // key j, token t >= j
            }
            sf[tid] = f;
            se[tid] = e;
            if (j == 15) pb[tid >> 4] = f;
        }
    }
    __syncthreads();
    // ---- N and B by blocks of 16 rows x 8 keys: row block I against key block b (the diagonal only with one decay per head).  The inner
    // index is permuted so that a lane's four values of a 16-step are neighbours.
    {
        const int g = lane >> 2, t4 = lane & 3;
        constexpr int TASKS = CH ? 12 : 20;
        for (int task = warp; task < TASKS; task += 16) {
            const int pair = task >> 1, j0 = 8 * (task & 1);
            int I, b;
            if (CH) {
                I = pair == 0 ? 1 : pair < 3 ? 2 : 3;
                b = pair == 0 ? 0 : pair < 3 ? pair - 1 : pair - 3;
            } else {
                I = pair == 0 ? 0 : pair < 3 ? 1 : pair < 6 ? 2 : 3;
                b = pair - I * (I + 1) / 2;
            }
            const float *kr = sk + (16 * I + g) * P + 4 * t4, *qr = sq + (16 * I + g) * P + 4 * t4, *kc = (CH ? sg : sk) + (16 * b + j0 + g) * P + 4 * t4;
            float n[4] = {}, m[4] = {};
#pragma unroll 2
            for (int s = 0; s < D; s += 16) {
                uint32_t ah[4], al[4], bh[2], bl[2];
                float4 v = *reinterpret_cast<const float4*>(kc + s);
                if (CH) {                        // decay of the blocks between
                    if (I - b >= 2) v = mul4(v, *reinterpret_cast<const float4*>(pb + (b + 1) * D + s + 4 * t4));
                    if (I - b == 3) v = mul4(v, *reinterpret_cast<const float4*>(pb + (b + 2) * D + s + 4 * t4));
                }
                split4(v, bh[0], bh[1], bl[0], bl[1]);
                split4(*reinterpret_cast<const float4*>(kr + s), ah[0], ah[2], al[0], al[2]);
                split4(*reinterpret_cast<const float4*>(kr + 8 * P + s), ah[1], ah[3], al[1], al[3]);
                mma_split(n, ah, al, bh, bl);
                split4(*reinterpret_cast<const float4*>(qr + s), ah[0], ah[2], al[0], al[2]);
                split4(*reinterpret_cast<const float4*>(qr + 8 * P + s), ah[1], ah[3], al[1], al[3]);
                mma_split(m, ah, al, bh, bl);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = 16 * I + g + 8 * (e >> 1), j = 16 * b + j0 + 2 * t4 + (e & 1);
                float r = 1.0f;
                if (!CH) {
                    if (I == b) r = i >= j ? rat[j * 17 + (i & 15)] : 0.0f;
                    else {
                        r = sf[i] * se[j];
                        for (int u = b + 1; u < I; ++u) r *= pb[u];
                    }
                }
                if (i > j) sN[i * DP_PITCH + j] = beta[i] * n[e] * r;
                if (i >= j) sB[i * DP_PITCH + j] = m[e] * r;
            }
        }
    }
    __syncthreads();
    if (warp < 8) {
        // ---- X = (I + N)^-1: diagonal blocks of 16 (a lane per column), then 32 from 16 and 64 from 32: X21 = -X22 (N21 X11)
        if (warp < 4) {
            const int b0 = 16 * warp;
            float x[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                float s = i == lane ? 1.0f : 0.0f;
#pragma unroll
                for (int j = 0; j < i; ++j) s = fmaf(-sN[(b0 + i) * DP_PITCH + b0 + j], x[j], s);
                x[i] = s;
            }
            if (lane < 16)
#pragma unroll
                for (int i = 0; i < 16; ++i) sX[(b0 + i) * DP_PITCH + b0 + lane] = x[i];
        }
        half_bar();
        {
            const int pr = tid >> 7, r = (tid >> 3) & 15, c = 2 * (tid & 7), b0 = 32 * pr;
            float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
            for (int k = 0; k < 16; ++k) {
                const float n = sN[(b0 + 16 + r) * DP_PITCH + b0 + k];
                const float2 xx = *reinterpret_cast<const float2*>(sX + (b0 + k) * DP_PITCH + b0 + c);
                s0 = fmaf(n, xx.x, s0);
                s1 = fmaf(n, xx.y, s1);
            }
            *reinterpret_cast<float2*>(sT + (pr * 16 + r) * 36 + c) = make_float2(s0, s1);
            half_bar();
            s0 = s1 = 0.0f;
#pragma unroll
            for (int k = 0; k < 16; ++k) {
                const float n = sX[(b0 + 16 + r) * DP_PITCH + b0 + 16 + k];
                const float2 tt = *reinterpret_cast<const float2*>(sT + (pr * 16 + k) * 36 + c);
                s0 = fmaf(n, tt.x, s0);
                s1 = fmaf(n, tt.y, s1);
            }
            *reinterpret_cast<float2*>(sX + (b0 + 16 + r) * DP_PITCH + b0 + c) = make_float2(-s0, -s1);
            *reinterpret_cast<float2*>(sX + (b0 + r) * DP_PITCH + b0 + 16 + c) = make_float2(0.0f, 0.0f);   // read by the products of 32
            half_bar();
        }
        {
            const int r = tid >> 3, c = 4 * (tid & 7);
            float4 s = make_float4(0, 0, 0, 0);
#pragma unroll 16
            for (int k = 0; k < 32; ++k) {
                const float n = sN[(32 + r) * DP_PITCH + k];
                const float4 x = *reinterpret_cast<const float4*>(sX + k * DP_PITCH + c);
                s.x = fmaf(n, x.x, s.x); s.y = fmaf(n, x.y, s.y); s.z = fmaf(n, x.z, s.z); s.w = fmaf(n, x.w, s.w);
            }
            *reinterpret_cast<float4*>(sT + r * 36 + c) = s;
            half_bar();
            s = make_float4(0, 0, 0, 0);
#pragma unroll 16
            for (int k = 0; k < 32; ++k) {
                const float n = sX[(32 + r) * DP_PITCH + 32 + k];
                const float4 x = *reinterpret_cast<const float4*>(sT + k * 36 + c);
                s.x = fmaf(n, x.x, s.x); s.y = fmaf(n, x.y, s.y); s.z = fmaf(n, x.z, s.z); s.w = fmaf(n, x.w, s.w);
            }
            *reinterpret_cast<float4*>(sX + (32 + r) * DP_PITCH + c) = make_float4(-s.x, -s.y, -s.z, -s.w);
        }
    } else {
        // ---- meanwhile: c Q, E, B and c at the chunk's end
        for (int u = tid - 256; u < 64 * (D / 8); u += 256) {
            const int t = u / (D / 8), c = 8 * (u % (D / 8)), b = t >> 4;
            const int64_t o = ((int64_t)item * DC + t) * D + c;
            uint32_t hw[4], lw[4];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                float4 v = *reinterpret_cast<const float4*>(sq + t * P + c + 4 * e);
                if (!CH) v = mul4(v, sf[t]);
                for (int w = 0; w < b; ++w) v = CH ? mul4(v, *reinterpret_cast<const float4*>(pb + w * D + c + 4 * e)) : mul4(v, pb[w]);
                split4(v, hw[2 * e], hw[2 * e + 1], lw[2 * e], lw[2 * e + 1]);
            }
            *reinterpret_cast<uint4*>(a.qh + o) = make_uint4(hw[0], hw[1], hw[2], hw[3]);
            *reinterpret_cast<uint4*>(a.ql + o) = make_uint4(lw[0], lw[1], lw[2], lw[3]);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                float4 v = *reinterpret_cast<const float4*>((CH ? sg : sk) + t * P + c + 4 * e);
                if (!CH) v = mul4(v, se[t]);
                for (int w = b + 1; w < 4; ++w) v = CH ? mul4(v, *reinterpret_cast<const float4*>(pb + w * D + c + 4 * e)) : mul4(v, pb[w]);
                split4(v, hw[2 * e], hw[2 * e + 1], lw[2 * e], lw[2 * e + 1]);
            }
            *reinterpret_cast<uint4*>(a.eh + o) = make_uint4(hw[0], hw[1], hw[2], hw[3]);
            *reinterpret_cast<uint4*>(a.el + o) = make_uint4(lw[0], lw[1], lw[2], lw[3]);
        }
        for (int u = tid - 256; u < 512; u += 256) {
            const int i = u >> 3, j = 8 * (u & 7);
            uint32_t hw[4], lw[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int c = j + 2 * e;
                split2(c <= i ? sB[i * DP_PITCH + c] : 0.0f, c + 1 <= i ? sB[i * DP_PITCH + c + 1] : 0.0f, hw[e], lw[e]);
            }
            const int64_t o = ((int64_t)item * DC + i) * 64 + j;
            *reinterpret_cast<uint4*>(a.bh + o) = make_uint4(hw[0], hw[1], hw[2], hw[3]);
            *reinterpret_cast<uint4*>(a.bl + o) = make_uint4(lw[0], lw[1], lw[2], lw[3]);
        }
        for (int c = tid - 256; c < D; c += 256)
            a.gend[(int64_t)item * D + c] = CH ? pb[c] * pb[D + c] * pb[2 * D + c] * pb[3 * D + c] : pb[0] * pb[1] * pb[2] * pb[3];
    }
    __syncthreads();
    // ---- T = X diag(beta)
    {
        const int i = tid >> 3, j = 8 * (tid & 7);
        uint32_t hw[4], lw[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = j + 2 * e;
            split2(c <= i ? sX[i * DP_PITCH + c] * beta[c] : 0.0f, c + 1 <= i ? sX[i * DP_PITCH + c + 1] * beta[c + 1] : 0.0f, hw[e], lw[e]);
        }
        const int64_t o = ((int64_t)item * DC + i) * 64 + j;
        *reinterpret_cast<uint4*>(a.th + o) = make_uint4(hw[0], hw[1], hw[2], hw[3]);
        *reinterpret_cast<uint4*>(a.tl + o) = make_uint4(lw[0], lw[1], lw[2], lw[3]);
    }
    // ---- -W = -X (beta c K): a warp owns 16 channels and two row blocks (D = 128: {0, 3} or {1, 2}; D = 64: one).  Inner index (tokens):
    // lane t4 holds tokens t4 + 4 e of a block; columns: a lane's four channels are neighbours.
    {
        const int g = lane >> 2, t4 = lane & 3;
        constexpr int CG = D / 16, ROWS = CG == 8 ? 2 : 1;
        const int c0 = 16 * (warp % CG), rs = warp / CG;
        float acc[ROWS][2][4] = {};
        const int last = ROWS == 2 ? (rs == 0 ? 3 : 2) : rs;
        float pre[2] = {1.0f, 1.0f};             // decay of the blocks before, for this lane's two columns
        const int ca = c0 + 4 * (g >> 1) + (g & 1);
        for (int jb = 0; jb <= last; ++jb) {
            uint32_t bh[2][2], bl[2][2];
            float v[2][4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int j = 16 * jb + t4 + 4 * e;
                const float w = beta[j] * (CH ? 1.0f : sf[j]);
                v[0][e] = sk[j * P + ca] * (w * pre[0]);
                v[1][e] = sk[j * P + ca + 2] * (w * pre[1]);
            }
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                split2(v[n][0], v[n][1], bh[n][0], bl[n][0]);
                split2(v[n][2], v[n][3], bh[n][1], bl[n][1]);
                pre[n] *= CH ? pb[jb * D + ca + 2 * n] : pb[jb];
            }
#pragma unroll
            for (int r = 0; r < ROWS; ++r) {
                const int I = ROWS == 2 ? (r == 0 ? last : rs) : rs;
                if (jb > I) continue;
                const float* x = sX + (16 * I + g) * DP_PITCH + 16 * jb + t4;
                uint32_t ah[4], al[4];
                split2(x[0], x[4], ah[0], al[0]);
                split2(x[8 * DP_PITCH], x[8 * DP_PITCH + 4], ah[1], al[1]);
                split2(x[8], x[12], ah[2], al[2]);
                split2(x[8 * DP_PITCH + 8], x[8 * DP_PITCH + 12], ah[3], al[3]);
#pragma unroll
                for (int n = 0; n < 2; ++n) mma_split(acc[r][n], ah, al, bh[n], bl[n]);
            }
        }
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            const int I = ROWS == 2 ? (r == 0 ? last : rs) : rs;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                uint32_t h0, l0, h1, l1;
                split2(-acc[r][0][2 * e], -acc[r][0][2 * e + 1], h0, l0);
                split2(-acc[r][1][2 * e], -acc[r][1][2 * e + 1], h1, l1);
                const int64_t o = ((int64_t)item * DC + 16 * I + g + 8 * e) * D + c0 + 4 * t4;
                *reinterpret_cast<uint2*>(a.wh + o) = make_uint2(h0, h1);
                *reinterpret_cast<uint2*>(a.wl + o) = make_uint2(l0, l1);
            }
        }
    }
}

// ---- the recurrence over chunks -----------------------------------------------------------------------------------------
// 576 threads: TMA warp, MMA warp (converged, one lane issues), four warpgroups that turn S into tensor-memory operands (a thread per
// value row, 32 channels each); the first two do the same with U (32 tokens each), the others store O.  Operands stream through a ring of 16 KB slots, per chunk:
//   V (two blocks of 64 values), {T high, T remainder}, per 64 channels {-W}, {c Q}, {E}, then {B}.
// Tensor memory: S^T float32 0..127, its two terms 128..255 (per 32 channels: 16 columns high, 16 remainder), U^T 256..319, its
// terms 320..383, O^T 384..511 (two buffers).
constexpr int DT_THREADS = 576;
constexpr int DT_SLOTS = 13, DT_SLOT = 2 * DC_BLK;
constexpr int DT_G_OFF = DT_SLOTS * DT_SLOT;                  // float [4][128]
constexpr int DT_BAR_OFF = DT_G_OFF + 4 * 512;                // full[], empty[], g[4], u, uw, s, sw, of[2], oe[2]
constexpr int DT_NBAR = 2 * DT_SLOTS + 12;
constexpr int DT_MISC_OFF = DT_BAR_OFF + 8 * DT_NBAR;
constexpr int DT_SMEM = DT_MISC_OFF + 16 + 1024;
constexpr uint32_t DT_SP = 128, DT_U = 256, DT_UP = 320, DT_O = 384;

// 32 float32 values as two bfloat16 terms: 16 columns high, 16 columns remainder.
__device__ __forceinline__ void split32(const uint32_t (&v)[32], uint32_t (&pk)[32]) {
#pragma unroll
    for (int i = 0; i < 16; ++i) split2(__uint_as_float(v[2 * i]), __uint_as_float(v[2 * i + 1]), pk[i], pk[16 + i]);
}

template <int DB>
__global__ void __launch_bounds__(DT_THREADS, 1)
    delta_state_kernel(const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmTh, const __grid_constant__ CUtensorMap tmTl,
                       const __grid_constant__ CUtensorMap tmWh, const __grid_constant__ CUtensorMap tmWl, const __grid_constant__ CUtensorMap tmQh,
                       const __grid_constant__ CUtensorMap tmQl, const __grid_constant__ CUtensorMap tmEh, const __grid_constant__ CUtensorMap tmEl,
                       const __grid_constant__ CUtensorMap tmBh, const __grid_constant__ CUtensorMap tmBl, const DeltaTcArgs a) {
    constexpr int D = 64 * DB;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    const uint32_t sbase = smem_u32(smem);
    const uint32_t b_f = sbase + DT_BAR_OFF, b_e = b_f + 8 * DT_SLOTS, b_g = b_e + 8 * DT_SLOTS, b_u = b_g + 32, b_uw = b_u + 8, b_s = b_uw + 8,
                   b_sw = b_s + 8, b_of = b_sw + 8, b_oe = b_of + 16;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + DT_MISC_OFF);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + DT_MISC_OFF + 4);
    const int warp = __shfl_sync(0xffffffffu, (int)(threadIdx.x >> 5), 0), lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (const CUtensorMap* m : {&tmV, &tmTh, &tmTl, &tmWh, &tmWl, &tmQh, &tmQl, &tmEh, &tmEl, &tmBh, &tmBl}) prefetch_map(m);
        for (int i = 0; i < DT_NBAR; ++i) {
            const uint32_t b = b_f + 8 * i;
            mbar_init(b, b == b_uw || b == b_oe || b == b_oe + 8 ? 8 : b == b_sw ? 8 * DB : 1);
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        tmem_alloc(smem_u32(tmem_slot), 512);
        tmem_relinquish();
    }
    pdl_launch_dependents();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = __shfl_sync(0xffffffffu, *tmem_slot, 0);
    pdl_wait();
    const DeltaArgs& p = a.p;
    const int h = blockIdx.x, v0 = blockIdx.y * 128, nc = a.nc;
    int fail = 0;

    if (warp == 0) {
        if (lane == 0) {
            int i = 0;
            uint32_t s, bar;
            auto slot = [&]() -> bool {       // next free slot, armed for its 16 KB
                const int st = i % DT_SLOTS;
                if (int w = mbar_wait(b_e + 8 * st, ((i / DT_SLOTS) & 1) ^ 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 61 : -1; return false; }
                s = sbase + st * DT_SLOT;
                bar = b_f + 8 * st;
                mbar_expect_tx(bar, DT_SLOT);
                ++i;
                return true;
            };
            for (int c = 0; c < nc && fail == 0; ++c) {
                const int item = c * p.H + h, row = item * DC;
                if (!slot()) break;
                tma_load_3d(s, &tmV, 2 * v0, c * DC, h, bar);
                tma_load_3d(s + DC_BLK, &tmV, 2 * v0 + 128, c * DC, h, bar);
                // slot c & 3 of the decays is free: it was read before the products of chunk c - 4, whose operands left the ring
                mbar_expect_tx(b_g + 8 * (c & 3), 4 * D);
                bulk_load(sbase + DT_G_OFF + 512 * (c & 3), a.gend + (int64_t)item * D, 4 * D, b_g + 8 * (c & 3));
                if (!slot()) break;
                tma_load_2d(s, &tmTh, 0, row, bar);
                tma_load_2d(s + DC_BLK, &tmTl, 0, row, bar);
                for (int b = 0; b < DB && fail == 0; ++b)
                    if (slot()) {
                        tma_load_2d(s, &tmWh, 128 * b, row, bar);
                        tma_load_2d(s + DC_BLK, &tmWl, 128 * b, row, bar);
                    }
                for (int b = 0; b < DB && fail == 0; ++b)
                    if (slot()) {
                        tma_load_2d(s, &tmQh, 128 * b, row, bar);
                        tma_load_2d(s + DC_BLK, &tmQl, 128 * b, row, bar);
                    }
                for (int b = 0; b < DB && fail == 0; ++b)
                    if (slot()) {
                        tma_load_2d(s, &tmEh, 128 * b, row, bar);
                        tma_load_2d(s + DC_BLK, &tmEl, 128 * b, row, bar);
                    }
                if (fail || !slot()) break;
                tma_load_2d(s, &tmBh, 0, row, bar);
                tma_load_2d(s + DC_BLK, &tmBl, 0, row, bar);
            }
        }
    } else if (warp == 1) {
        // the whole warp walks through the chunks; `on` is the lane that issues
        constexpr uint32_t idesc = umma_idesc_bf16(128, 64), idesc_v = idesc | IDESC_A_MN, idesc_e = idesc | IDESC_B_MN;
        const uint32_t on = elect_lane();
        int st = 0;
        uint32_t ph = 0, s = 0;
        auto wait = [&](uint32_t bar, uint32_t parity, int code) -> bool {
            const int w = mbar_wait(bar, parity, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) { fail = w == 1 ? code : -1; return false; }
            tc_fence_after();
            return true;
        };
        auto next = [&]() -> bool {
            if (!wait(b_f + 8 * st, ph, 62)) return false;
            s = sbase + st * DT_SLOT;
            return true;
        };
        auto done = [&]() {
            umma_commit_on(on, b_e + 8 * st);
            if (++st == DT_SLOTS) { st = 0; ph ^= 1; }
        };
        // D (+)= terms at `op` (per 32 values of K: 16 columns high, 16 remainder) times the K-major block pair at s, 64 of K
        auto split_product = [&](uint32_t d, uint32_t op, uint32_t fresh) {
            const uint64_t bh = umma_desc(s), bl = umma_desc(s + DC_BLK);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const uint32_t x = op + (k >> 1) * 32 + (k & 1) * 8;
                umma_bf16_ts_on(on, d, x, bh + 2 * k, idesc, k > 0 ? 1u : 1u - fresh);
                umma_bf16_ts_on(on, d, x, bl + 2 * k, idesc, 1);
                umma_bf16_ts_on(on, d, x + 16, bh + 2 * k, idesc, 1);
            }
        };
        auto values = [&]() -> bool {      // U = T V
            if (!next()) return false;
            const uint64_t v = umma_desc_mn(s, DC_BLK);
            const uint32_t vfree = b_e + 8 * st;
            if (++st == DT_SLOTS) { st = 0; ph ^= 1; }
            if (!next()) return false;
            const uint64_t th = umma_desc(s), tl = umma_desc(s + DC_BLK);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                umma_bf16_on(on, tmem + DT_U, v + 128 * k, th + 2 * k, idesc_v, k > 0);
                umma_bf16_on(on, tmem + DT_U, v + 128 * k, tl + 2 * k, idesc_v, 1);
            }
            umma_commit_on(on, vfree);
            done();
            return true;
        };
        bool ok = values();
        for (int c = 0; c < nc && ok; ++c) {
            if (!wait(b_sw, c & 1, 63)) break;
#pragma unroll
            for (int b = 0; b < DB; ++b) {
                if (!(ok = next())) break;
                split_product(tmem + DT_U, tmem + DT_SP + 64 * b, 0);
                done();
            }
            if (!ok) break;
            umma_commit_on(on, b_u);
            const uint32_t o = tmem + DT_O + 64 * (c & 1);
            if (!wait(b_oe + 8 * (c & 1), ((c >> 1) & 1) ^ 1, 63)) break;
#pragma unroll
            for (int b = 0; b < DB; ++b) {
                if (!(ok = next())) break;
                split_product(o, tmem + DT_SP + 64 * b, b == 0);
                done();
            }
            if (!ok || !wait(b_uw, c & 1, 63)) break;
#pragma unroll
            for (int b = 0; b < DB; ++b) {
                if (!(ok = next())) break;
                const uint64_t eh = umma_desc_mn(s, DC_BLK), el = umma_desc_mn(s + DC_BLK, DC_BLK);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const uint32_t u = tmem + DT_UP + (k >> 1) * 32 + (k & 1) * 8;
                    umma_bf16_ts_on(on, tmem + 64 * b, u, eh + 128 * k, idesc_e, 1);
                    umma_bf16_ts_on(on, tmem + 64 * b, u, el + 128 * k, idesc_e, 1);
                    umma_bf16_ts_on(on, tmem + 64 * b, u + 16, eh + 128 * k, idesc_e, 1);
                }
                done();
            }
            if (!ok) break;
            umma_commit_on(on, b_s);
            if (!(ok = next())) break;
            split_product(o, tmem + DT_UP, 0);
            done();
            umma_commit_on(on, b_of + 8 * (c & 1));
            if (c + 1 < nc) ok = values();
        }
        if (!on) fail = fail > 0 ? -1 : fail;      // one lane reports
    } else {
        const int wg = (warp - 2) >> 2, q = warp & 3, v = v0 + 32 * q + lane;
        const uint32_t lane_base = (uint32_t)(32 * q) << 16;
        const bool in = v < p.dv, owner = wg < 2 * DB;       // owner: holds 32 channels of S
        const int ch = 32 * wg;
        float* gS = p.state + ((int64_t)h * p.d + ch) * p.dv + v;
        auto wait = [&](uint32_t bar, uint32_t parity) -> bool {
            const int w = mbar_wait(bar, parity, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) { fail = w == 1 ? 64 : -1; return false; }
            tc_fence_after();
            return true;
        };
        for (int c = 0; c <= nc; ++c) {
            // S at the start of chunk c: its terms, and c_end S for the sum; after the last chunk the state is stored
            if (owner) {
                if (c < nc && !wait(b_g + 8 * (c & 3), (c >> 2) & 1)) break;
                if (c > 0 && !wait(b_s, (c - 1) & 1)) break;
                uint32_t s[32];
                if (c > 0) {
                    tmem_ld32(tmem + ch + lane_base, s);
                    tmem_ld_fence(s);
                } else {
#pragma unroll
                    for (int i = 0; i < 32; ++i) s[i] = in && ch + i < p.d ? __float_as_uint(gS[(int64_t)i * p.dv]) : 0u;
                }
                if (c == nc) {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (in && ch + i < p.d) gS[(int64_t)i * p.dv] = __uint_as_float(s[i]);
                } else {
                    uint32_t pk[32];
                    split32(s, pk);
                    tmem_st32(tmem + DT_SP + ch + lane_base, pk);
                    const float4* g = reinterpret_cast<const float4*>(smem + DT_G_OFF + 512 * (c & 3)) + ch / 4;
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        const float4 f = g[i];
                        s[4 * i] = __float_as_uint(__uint_as_float(s[4 * i]) * f.x);
                        s[4 * i + 1] = __float_as_uint(__uint_as_float(s[4 * i + 1]) * f.y);
                        s[4 * i + 2] = __float_as_uint(__uint_as_float(s[4 * i + 2]) * f.z);
                        s[4 * i + 3] = __float_as_uint(__uint_as_float(s[4 * i + 3]) * f.w);
                    }
                    tmem_st32(tmem + ch + lane_base, s);
                    tmem_st_wait();
                    tc_fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive(b_sw);
                }
            }
            if (wg < 2) {
                if (c == nc) break;
                // the corrections of this warpgroup's 32 tokens
                if (!wait(b_u, c & 1)) break;
                uint32_t u[32], pk[32];
                tmem_ld32(tmem + DT_U + 32 * wg + lane_base, u);
                tmem_ld_fence(u);
                split32(u, pk);
                tmem_st32(tmem + DT_UP + 32 * wg + lane_base, pk);
                tmem_st_wait();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(b_uw);
            } else if (c > 0) {
                // outputs of the previous chunk, 32 tokens per warpgroup
                const int b = (c - 1) & 1;
                if (!wait(b_of + 8 * b, ((c - 1) >> 1) & 1)) break;
                uint32_t x[32];
                tmem_ld32(tmem + DT_O + 64 * b + 32 * (wg - 2) + lane_base, x);
                tmem_ld_fence(x);
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(b_oe + 8 * b);
                const int64_t t0 = (int64_t)(c - 1) * DC + 32 * (wg - 2);
                const int nt = (int)min((int64_t)32, p.n - t0);
                float* out = p.o + (t0 * p.H + h) * p.dv + v;
                const int64_t step = (int64_t)p.H * p.dv;
                if (in)
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (i < nt) out[i * step] = __uint_as_float(x[i]);
            }
        }
    }

    if (fail > 0) {
        if (atomicCAS(a.status, 0, fail) == 0) {
            a.status[1] = blockIdx.x;
            a.status[2] = threadIdx.x;
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (*abort_flag) {
        const uint64_t w0 = globaltimer_ns();
        while (globaltimer_ns() - w0 < 200000ull) __nanosleep(1000);   // 0.2 ms for outstanding TMA writes
        __syncthreads();
    }
    if (warp == 1) tmem_dealloc(tmem, 512);
}

bool delta_tc_supported(int64_t n, int H, int d, int dv, int64_t ldv) {
    return d % 8 == 0 && dv % 8 == 0 && d <= 128 && ldv % 8 == 0 && n < (1ll << 24) && (n + DC - 1) / DC * H < (1ll << 24);
}

static int64_t align256(int64_t b) { return (b + 255) / 256 * 256; }
static int width(int d) { return d <= 64 ? 64 : 128; }
int64_t delta_tc_scratch(int64_t n, int H, int d) {
    const int64_t items = (n + DC - 1) / DC * H;
    return 6 * align256(items * DC * width(d) * 2) + 4 * align256(items * DC_BLK) + align256(items * width(d) * 4);
}

template <int D, bool CH>
static int run_prep_tc(const DeltaTcArgs& a, cudaStream_t st) {
    constexpr int smem = DpSmem<D, CH>::FLOATS * 4;
    static bool configured[64] = {};
    const int dev = current_device();
    SCMX_REQUIRE(dev >= 0, SCMX_ECUDA, "no current CUDA device (ordinal 0..63)");
    if (!configured[dev]) {
        SCMX_CUDA_OK(cudaFuncSetAttribute(delta_prep_kernel<D, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        configured[dev] = true;
    }
    SCMX_PDL_OK("delta_prep_kernel", launch_pdl(delta_prep_kernel<D, CH>, dim3((unsigned)a.nc * a.p.H), dim3(DP_THREADS), (size_t)smem, st, a));
    return SCMX_OK;
}

template <int DB>
static int run_state(const CUtensorMap (&m)[11], const DeltaTcArgs& a, cudaStream_t st) {
    static bool configured[64] = {};
    const int dev = current_device();
    SCMX_REQUIRE(dev >= 0, SCMX_ECUDA, "no current CUDA device (ordinal 0..63)");
    if (!configured[dev]) {
        SCMX_CUDA_OK(cudaFuncSetAttribute(delta_state_kernel<DB>, cudaFuncAttributeMaxDynamicSharedMemorySize, DT_SMEM));
        configured[dev] = true;
    }
    SCMX_PDL_OK("delta_state_kernel", launch_pdl(delta_state_kernel<DB>, dim3(a.p.H, (a.p.dv + 127) / 128), dim3(DT_THREADS), (size_t)DT_SMEM, st, m[0], m[1],
                                                 m[2], m[3], m[4], m[5], m[6], m[7], m[8], m[9], m[10], a));
    return SCMX_OK;
}

int delta_tc(const DeltaArgs& p, bool channel, void* scratch, int32_t* status, cudaStream_t st) {
    SCMX_REQUIRE(p.ldq % 2 == 0 && p.ldk % 2 == 0 && (((uintptr_t)p.q | (uintptr_t)p.k) & 3) == 0 &&
                 (!channel || (p.lda % 2 == 0 && ((uintptr_t)p.a & 7) == 0)), SCMX_EINVAL, "delta: unaligned rows");
    DeltaTcArgs a;
    a.p = p; a.status = status; a.wait_ns = g_wait_limit_ns; a.nc = (int)((p.n + DC - 1) / DC);
    const int64_t items = (int64_t)a.nc * p.H;
    const int D = width(p.d);
    uint8_t* s = static_cast<uint8_t*>(scratch);
    bf16_t** wide[6] = {&a.wh, &a.wl, &a.qh, &a.ql, &a.eh, &a.el};
    for (auto x : wide) { *x = reinterpret_cast<bf16_t*>(s); s += align256(items * DC * D * 2); }
    bf16_t** square[4] = {&a.th, &a.tl, &a.bh, &a.bl};
    for (auto x : square) { *x = reinterpret_cast<bf16_t*>(s); s += align256(items * DC_BLK); }
    a.gend = reinterpret_cast<float*>(s);
    CUtensorMap m[11];
    int rc = make_map_planes(&m[0], p.v, p.H, p.n, 2 * p.dv, 2 * p.ldv, 2 * p.dv, DC);
    const bf16_t* src[10] = {a.th, a.tl, a.wh, a.wl, a.qh, a.ql, a.eh, a.el, a.bh, a.bl};
    for (int i = 0; i < 10 && !rc; ++i) rc = make_map_u8(&m[i + 1], src[i], items * DC, i >= 2 && i < 8 ? 2 * D : 128, 128, DC, 128, 0);
    if (rc) return rc;
    if (D == 64) rc = channel ? run_prep_tc<64, true>(a, st) : run_prep_tc<64, false>(a, st);
    else rc = channel ? run_prep_tc<128, true>(a, st) : run_prep_tc<128, false>(a, st);
    if (rc) return rc;
    return D == 64 ? run_state<1>(m, a, st) : run_state<2>(m, a, st);
}

}  // namespace scmx
