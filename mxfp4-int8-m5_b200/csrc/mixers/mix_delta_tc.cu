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

template <int D, bool CH>
struct DpSmem {
    static constexpr int Q = 0, K = Q + 64 * D, G = K + 64 * D, N = G + (CH ? 64 * D : 64), B = N + 64 * DP_PITCH, T = B + 64 * DP_PITCH,
                         BETA = T + 32 * 34, FLOATS = BETA + 64;
};

template <int D, bool CH>
__global__ void __launch_bounds__(DP_THREADS, 1) delta_prep_kernel(const DeltaTcArgs a) {
    using L = DpSmem<D, CH>;
    extern __shared__ __align__(16) float sm[];
    float *sq = sm + L::Q, *sk = sm + L::K, *sg = sm + L::G, *sN = sm + L::N, *sB = sm + L::B, *sT = sm + L::T, *beta = sm + L::BETA;
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
        const bf16_t *q = static_cast<const bf16_t*>(p.q) + (int64_t)kh * p.d, *k = static_cast<const bf16_t*>(p.k) + (int64_t)kh * p.d;
        const float qs = rsqrtf((float)p.d), nA2 = p.nA[h] * 1.4426950408889634f;
        const int e = V * lane;
        const bool in = e < p.d;
        float dtb[V];
#pragma unroll
        for (int i = 0; i < V; ++i) dtb[i] = CH ? (in ? p.dtb[(int64_t)h * p.d + e + i] : 0.0f) : p.dtb[h];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int t = warp + 16 * r;
            float x[V], y[V], z[V];
#pragma unroll
            for (int i = 0; i < V; ++i) x[i] = y[i] = z[i] = 0.0f;
            if (t < nt && in) {
                const bf16_t *qr = q + (t0 + t) * p.ldq + e, *kr = k + (t0 + t) * p.ldk + e;
                // rows are 4-byte aligned (host side)
#pragma unroll
                for (int i = 0; i < V; i += 2) {
                    const uint32_t u = *reinterpret_cast<const uint32_t*>(qr + i), w = *reinterpret_cast<const uint32_t*>(kr + i);
                    x[i] = bf16_lo(u); x[i + 1] = bf16_hi(u);
                    y[i] = bf16_lo(w); y[i + 1] = bf16_hi(w);
                }
                if (CH) {
                    const float* ar = static_cast<const float*>(p.a) + (t0 + t) * p.lda + (int64_t)h * p.d + e;
#pragma unroll
                    for (int i = 0; i < V; i += 2) {
                        const float2 u = *reinterpret_cast<const float2*>(ar + i);
                        z[i] = u.x; z[i + 1] = u.y;
                    }
                }
            }
            float qq = 0.0f, kk = 0.0f;
#pragma unroll
            for (int i = 0; i < V; ++i) {
                qq = fmaf(x[i], x[i], qq);
                kk = fmaf(y[i], y[i], kk);
            }
            const float iq = qs / sqrtf(warp_sumf(qq) + 1e-6f), ik = 1.0f / sqrtf(warp_sumf(kk) + 1e-6f);
#pragma unroll
            for (int i = 0; i < V; ++i) {
                sq[t * D + e + i] = x[i] * iq;
                sk[t * D + e + i] = y[i] * ik;
                if (CH) sg[t * D + e + i] = t < nt ? ex2_approx(nA2 * softplus_f32(z[i] + dtb[i])) : 1.0f;
            }
            if (lane == 0) {
                beta[t] = t < nt ? sigmoid_f32(ldf(static_cast<const bf16_t*>(p.b) + (t0 + t) * p.ldb + h)) : 0.0f;
                if (!CH) sg[t] = t < nt ? ex2_approx(nA2 * softplus_f32(ldf(static_cast<const bf16_t*>(p.a) + (t0 + t) * p.lda + h) + dtb[0])) : 1.0f;
            }
        }
    }
    __syncthreads();
    // ---- N and B.  Eight lanes share a key j (float4 groups sub + 8 v); they carry c_i / c_j k_j from i = j on.  Work falls with j:
    // the four warps of a scheduler take columns from both ends.
    const int wk = warp >> 2, ws = warp & 3, pw = wk == 0 ? ws : wk == 1 ? 7 - ws : wk == 2 ? 8 + ws : 15 - ws;
    {
        constexpr int NV = D / 32;
        const int sub = lane & 7, j = 4 * pw + (lane >> 3);
        uint64_t kc[2 * NV];
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(sk + j * D + 4 * (sub + 8 * v));
            kc[2 * v] = u.x;
            kc[2 * v + 1] = u.y;
        }
        float ratio = 1.0f;
        for (int i0 = (4 * pw) & ~7; i0 < DC; i0 += 8) {
            float s[16];
#pragma unroll
            for (int ii = 0; ii < 8; ++ii) {
                const int i = i0 + ii;
                if (CH) {
                    if (i > j)
#pragma unroll
                        for (int v = 0; v < NV; ++v) {
                            const ulonglong2 g = *reinterpret_cast<const ulonglong2*>(sg + i * D + 4 * (sub + 8 * v));
                            kc[2 * v] = mul2(kc[2 * v], g.x);
                            kc[2 * v + 1] = mul2(kc[2 * v + 1], g.y);
                        }
                } else if (i > j) {
                    ratio *= sg[i];
                }
                uint64_t s0 = 0, s1 = 0, s2 = 0, s3 = 0;
#pragma unroll
                for (int v = 0; v < NV; ++v) {
                    const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(sk + i * D + 4 * (sub + 8 * v));
                    const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(sq + i * D + 4 * (sub + 8 * v));
                    s0 = fma2(kc[2 * v], k.x, s0);
                    s1 = fma2(kc[2 * v + 1], k.y, s1);
                    s2 = fma2(kc[2 * v], q.x, s2);
                    s3 = fma2(kc[2 * v + 1], q.y, s3);
                }
                const float2 x0 = unpack2(s0), x1 = unpack2(s1), y0 = unpack2(s2), y1 = unpack2(s3);
                s[2 * ii] = (x0.x + x0.y) + (x1.x + x1.y);
                s[2 * ii + 1] = (y0.x + y0.y) + (y1.x + y1.y);
                if (!CH) {
                    s[2 * ii] *= ratio;
                    s[2 * ii + 1] *= ratio;
                }
            }
            // sums over the eight lanes; lane `sub` ends with those of i0 + sub
#pragma unroll
            for (int n = 8, off = 4; off > 0; off >>= 1, n >>= 1) {
                const bool up = (lane & off) != 0;
#pragma unroll
                for (int i = 0; i < n; ++i) {
                    const float keep = up ? s[i + n] : s[i], give = up ? s[i] : s[i + n];
                    s[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
                }
            }
            const int i = i0 + sub;
            if (i > j) sN[i * DP_PITCH + j] = beta[i] * s[0];
            if (i >= j) sB[i * DP_PITCH + j] = s[1];
        }
    }
    __syncthreads();
    // ---- four warps invert the diagonal blocks of 16 (a lane per column), the others store B
    float x[16];
    if (warp < 4) {
        const int b0 = 16 * warp;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float s = i == lane ? 1.0f : 0.0f;
#pragma unroll
            for (int j = 0; j < i; ++j) s = fmaf(-sN[(b0 + i) * DP_PITCH + b0 + j], x[j], s);
            x[i] = s;
        }
    } else {
        for (int u = tid - 128; u < 512; u += DP_THREADS - 128) {
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
    }
    __syncthreads();
    float* sX = sB;
    if (warp < 4 && lane < 16) {
#pragma unroll
        for (int i = 0; i < 16; ++i) sX[(16 * warp + i) * DP_PITCH + 16 * warp + lane] = x[i];
    }
    // ---- decay products: forward over the tokens for c Q and c K (beta folded in, in place of q), backward for E
    {
        constexpr int PAIRS = D / 2, SEG = DP_THREADS / PAIRS / 2, LEN = DC / SEG;
        const int c = 2 * (tid % PAIRS), g0 = tid / PAIRS, s = g0 < SEG ? g0 : g0 - SEG;
        auto decay = [&](int t) -> float2 { return CH ? *reinterpret_cast<const float2*>(sg + t * D + c) : make_float2(sg[t], sg[t]); };
        float2 m = make_float2(1.0f, 1.0f);
        if (g0 < SEG) {
#pragma unroll 8
            for (int t = 0; t < s * LEN; ++t) {
                const float2 g = decay(t);
                m.x *= g.x; m.y *= g.y;
            }
#pragma unroll
            for (int i = 0; i < LEN; ++i) {
                const int t = s * LEN + i;
                const float2 g = decay(t), q = *reinterpret_cast<const float2*>(sq + t * D + c), k = *reinterpret_cast<const float2*>(sk + t * D + c);
                m.x *= g.x; m.y *= g.y;
                uint32_t hw, lw;
                split2(m.x * q.x, m.y * q.y, hw, lw);
                const int64_t o = ((int64_t)item * DC + t) * D + c;
                *reinterpret_cast<uint32_t*>(a.qh + o) = hw;
                *reinterpret_cast<uint32_t*>(a.ql + o) = lw;
                const float bt = beta[t];
                *reinterpret_cast<float2*>(sq + t * D + c) = make_float2(m.x * k.x * bt, m.y * k.y * bt);
            }
            if (s == SEG - 1) *reinterpret_cast<float2*>(a.gend + (int64_t)item * D + c) = m;
        } else {
#pragma unroll 8
            for (int t = DC - 1; t >= (s + 1) * LEN; --t) {
                const float2 g = decay(t);
                m.x *= g.x; m.y *= g.y;
            }
#pragma unroll
            for (int i = LEN - 1; i >= 0; --i) {
                const int t = s * LEN + i;
                const float2 g = decay(t), k = *reinterpret_cast<const float2*>(sk + t * D + c);
                uint32_t hw, lw;
                split2(m.x * k.x, m.y * k.y, hw, lw);
                const int64_t o = ((int64_t)item * DC + t) * D + c;
                *reinterpret_cast<uint32_t*>(a.eh + o) = hw;
                *reinterpret_cast<uint32_t*>(a.el + o) = lw;
                m.x *= g.x; m.y *= g.y;
            }
        }
    }
    __syncthreads();
    // ---- the rest of the inverse: blocks of 32 from blocks of 16, then 64 from 32: X21 = -X22 (N21 X11)
    {
        const int pr = tid >> 8, r = (tid >> 4) & 15, c = tid & 15, b0 = 32 * pr;
        float s = 0.0f;
#pragma unroll
        for (int k = 0; k < 16; ++k) s = fmaf(sN[(b0 + 16 + r) * DP_PITCH + b0 + k], sX[(b0 + k) * DP_PITCH + b0 + c], s);
        sT[(pr * 16 + r) * 17 + c] = s;
        __syncthreads();
        s = 0.0f;
#pragma unroll
        for (int k = 0; k < 16; ++k) s = fmaf(sX[(b0 + 16 + r) * DP_PITCH + b0 + 16 + k], sT[(pr * 16 + k) * 17 + c], s);
        sX[(b0 + 16 + r) * DP_PITCH + b0 + c] = -s;
        sX[(b0 + r) * DP_PITCH + b0 + 16 + c] = 0.0f;        // the upper block is read by the products of 32
        __syncthreads();
    }
    {
        const int r = tid >> 4, c = 2 * (tid & 15);
        float s0 = 0.0f, s1 = 0.0f;
#pragma unroll 8
        for (int k = 0; k < 32; ++k) {
            const float n = sN[(32 + r) * DP_PITCH + k];
            const float2 xx = *reinterpret_cast<const float2*>(sX + k * DP_PITCH + c);
            s0 = fmaf(n, xx.x, s0);
            s1 = fmaf(n, xx.y, s1);
        }
        *reinterpret_cast<float2*>(sT + r * 34 + c) = make_float2(s0, s1);
        __syncthreads();
        s0 = s1 = 0.0f;
#pragma unroll 8
        for (int k = 0; k < 32; ++k) {
            const float n = sX[(32 + r) * DP_PITCH + 32 + k];
            const float2 tt = *reinterpret_cast<const float2*>(sT + k * 34 + c);
            s0 = fmaf(n, tt.x, s0);
            s1 = fmaf(n, tt.y, s1);
        }
        *reinterpret_cast<float2*>(sX + (32 + r) * DP_PITCH + c) = make_float2(-s0, -s1);
        __syncthreads();
    }
    // ---- T = X diag(beta) and -W = -X (beta c K)
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
    {
        constexpr int RPT = D / 32;              // rows per thread
        const int row = D == 128 ? 4 * pw : 4 * pw + 2 * (lane >> 4), c = 4 * (D == 128 ? lane : lane & 15);
        uint64_t acc[RPT][2];
#pragma unroll
        for (int r = 0; r < RPT; ++r) acc[r][0] = acc[r][1] = 0;
        for (int j = 0; j < 4 * pw + 4; j += 4) {
            float xr[RPT][4];
#pragma unroll
            for (int r = 0; r < RPT; ++r) *reinterpret_cast<float4*>(xr[r]) = *reinterpret_cast<const float4*>(sX + (row + r) * DP_PITCH + j);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(sq + (j + e) * D + c);
#pragma unroll
                for (int r = 0; r < RPT; ++r) {
                    const uint64_t w = pack2(xr[r][e], xr[r][e]);
                    acc[r][0] = fma2(w, k.x, acc[r][0]);
                    acc[r][1] = fma2(w, k.y, acc[r][1]);
                }
            }
        }
#pragma unroll
        for (int r = 0; r < RPT; ++r) {
            const float2 u = unpack2(acc[r][0]), v = unpack2(acc[r][1]);
            uint32_t h0, l0, h1, l1;
            split2(-u.x, -u.y, h0, l0);
            split2(-v.x, -v.y, h1, l1);
            const int64_t o = ((int64_t)item * DC + row + r) * D + c;
            *reinterpret_cast<uint2*>(a.wh + o) = make_uint2(h0, h1);
            *reinterpret_cast<uint2*>(a.wl + o) = make_uint2(l0, l1);
        }
    }
}

// ---- the recurrence over chunks -----------------------------------------------------------------------------------------
// 448 threads: TMA warp, MMA warp, two warpgroups that turn S and U into tensor-memory operands (a thread per value row; each
// takes half of the channels or tokens), one warpgroup that stores O.  Operands stream through a ring of 16 KB slots, per chunk:
//   V (two blocks of 64 values), {T high, T remainder}, per 64 channels {-W}, {c Q}, {E}, then {B}.
// Tensor memory: S^T float32 0..127, its two terms 128..255 (per 32 channels: 16 columns high, 16 remainder), U^T 256..319, its
// terms 320..383, O^T 384..511 (two buffers).
constexpr int DT_THREADS = 448;
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
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (const CUtensorMap* m : {&tmV, &tmTh, &tmTl, &tmWh, &tmWl, &tmQh, &tmQl, &tmEh, &tmEl, &tmBh, &tmBl}) prefetch_map(m);
        for (int i = 0; i < DT_NBAR; ++i) {
            const uint32_t b = b_f + 8 * i;
            mbar_init(b, b == b_uw || b == b_sw ? 8 : b == b_oe || b == b_oe + 8 ? 4 : 1);
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
    const uint32_t tmem = *tmem_slot;
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
        if (lane == 0) {
            constexpr uint32_t idesc = umma_idesc_bf16(128, 64), idesc_v = idesc | IDESC_A_MN, idesc_e = idesc | IDESC_B_MN;
            int i = 0;
            uint32_t s = 0;
            auto next = [&]() -> bool {
                const int st = i % DT_SLOTS;
                if (int w = mbar_wait(b_f + 8 * st, (i / DT_SLOTS) & 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 62 : -1; return false; }
                tc_fence_after();
                s = sbase + st * DT_SLOT;
                return true;
            };
            auto done = [&]() { umma_commit(b_e + 8 * (i % DT_SLOTS)); ++i; };
            auto wait = [&](uint32_t bar, uint32_t parity) -> bool {
                if (int w = mbar_wait(bar, parity, abort_flag, a.wait_ns)) { fail = w == 1 ? 63 : -1; return false; }
                tc_fence_after();
                return true;
            };
            // D (+)= terms at `op` (per 32 values of K: 16 columns high, 16 remainder) times a K-major block pair at s, `steps` x 16 of K
            auto split_product = [&](uint32_t d, uint32_t op, int steps, bool fresh) {
                const uint64_t bh = umma_desc(s), bl = umma_desc(s + DC_BLK);
                for (int k = 0; k < steps; ++k) {
                    const uint32_t x = op + (k >> 1) * 32 + (k & 1) * 8;
                    umma_bf16_ts(d, x, bh + 2 * k, idesc, !fresh || k > 0);
                    umma_bf16_ts(d, x, bl + 2 * k, idesc, 1);
                    umma_bf16_ts(d, x + 16, bh + 2 * k, idesc, 1);
                }
            };
            auto values = [&]() -> bool {      // U = T V
                if (!next()) return false;
                const uint64_t v = umma_desc_mn(s, DC_BLK);
                ++i;                           // V's slot is freed together with T's below
                if (!next()) return false;
                const uint64_t th = umma_desc(s), tl = umma_desc(s + DC_BLK);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    umma_bf16(tmem + DT_U, v + 128 * k, th + 2 * k, idesc_v, k > 0);
                    umma_bf16(tmem + DT_U, v + 128 * k, tl + 2 * k, idesc_v, 1);
                }
                umma_commit(b_e + 8 * ((i - 1) % DT_SLOTS));
                done();
                return true;
            };
            bool ok = values();
            for (int c = 0; c < nc && ok; ++c) {
                if (!wait(b_sw, c & 1)) break;
                for (int b = 0; b < DB && ok; ++b) {
                    if (!(ok = next())) break;
                    split_product(tmem + DT_U, tmem + DT_SP + 64 * b, 4, false);
                    done();
                }
                if (!ok) break;
                umma_commit(b_u);
                const uint32_t o = tmem + DT_O + 64 * (c & 1);
                if (!wait(b_oe + 8 * (c & 1), ((c >> 1) & 1) ^ 1)) break;
                for (int b = 0; b < DB && ok; ++b) {
                    if (!(ok = next())) break;
                    split_product(o, tmem + DT_SP + 64 * b, 4, b == 0);
                    done();
                }
                if (!ok || !wait(b_uw, c & 1)) break;
                for (int b = 0; b < DB && ok; ++b) {
                    if (!(ok = next())) break;
                    const uint64_t eh = umma_desc_mn(s, DC_BLK), el = umma_desc_mn(s + DC_BLK, DC_BLK);
#pragma unroll
                    for (int k = 0; k < 4; ++k) {
                        const uint32_t u = tmem + DT_UP + (k >> 1) * 32 + (k & 1) * 8;
                        umma_bf16_ts(tmem + 64 * b, u, eh + 128 * k, idesc_e, 1);
                        umma_bf16_ts(tmem + 64 * b, u, el + 128 * k, idesc_e, 1);
                        umma_bf16_ts(tmem + 64 * b, u + 16, eh + 128 * k, idesc_e, 1);
                    }
                    done();
                }
                if (!ok) break;
                umma_commit(b_s);
                if (!(ok = next())) break;
                split_product(o, tmem + DT_UP, 4, false);
                done();
                umma_commit(b_of + 8 * (c & 1));
                if (c + 1 < nc) ok = values();
            }
        }
    } else if (warp < 10) {
        const int wg = (warp - 2) >> 2, q = warp & 3, v = v0 + 32 * q + lane;
        const uint32_t lane_base = (uint32_t)(32 * q) << 16;
        const bool in = v < p.dv;
        float* gS = p.state + ((int64_t)h * p.d + wg * (D / 2)) * p.dv + v;
        auto wait = [&](uint32_t bar, uint32_t parity) -> bool {
            const int w = mbar_wait(bar, parity, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) { fail = w == 1 ? 64 : -1; return false; }
            return true;
        };
        for (int c = 0; c <= nc; ++c) {
            // S at the start of chunk c: its terms, and c_end S for the sum; after the last chunk the state is stored
            if (c < nc && !wait(b_g + 8 * (c & 3), (c >> 2) & 1)) break;
            if (c > 0) {
                if (!wait(b_s, (c - 1) & 1)) break;
                tc_fence_after();
            }
            const float* g = reinterpret_cast<const float*>(smem + DT_G_OFF + 512 * (c & 3)) + wg * (D / 2);
#pragma unroll
            for (int b = 0; b < DB; ++b) {
                const int ch = 32 * b;                       // within this warpgroup's half
                const uint32_t col = wg * (D / 2) + ch;
                uint32_t s[32], pk[32];
                if (c > 0) {
                    tmem_ld32(tmem + col + lane_base, s);
                    tmem_ld_fence(s);
                } else {
#pragma unroll
                    for (int i = 0; i < 32; ++i) s[i] = in && wg * (D / 2) + ch + i < p.d ? __float_as_uint(gS[(int64_t)(ch + i) * p.dv]) : 0u;
                }
                if (c == nc) {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (in && wg * (D / 2) + ch + i < p.d) gS[(int64_t)(ch + i) * p.dv] = __uint_as_float(s[i]);
                } else {
                    split32(s, pk);
                    tmem_st32(tmem + DT_SP + col + lane_base, pk);
#pragma unroll
                    for (int i = 0; i < 32; i += 4) {
                        const float4 f = *reinterpret_cast<const float4*>(g + ch + i);
                        s[i] = __float_as_uint(__uint_as_float(s[i]) * f.x);
                        s[i + 1] = __float_as_uint(__uint_as_float(s[i + 1]) * f.y);
                        s[i + 2] = __float_as_uint(__uint_as_float(s[i + 2]) * f.z);
                        s[i + 3] = __float_as_uint(__uint_as_float(s[i + 3]) * f.w);
                    }
                    tmem_st32(tmem + col + lane_base, s);
                }
            }
            if (c == nc) break;
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(b_sw);
            // the corrections of this warpgroup's 32 tokens
            if (!wait(b_u, c & 1)) break;
            tc_fence_after();
            uint32_t u[32], pk[32];
            tmem_ld32(tmem + DT_U + 32 * wg + lane_base, u);
            tmem_ld_fence(u);
            split32(u, pk);
            tmem_st32(tmem + DT_UP + 32 * wg + lane_base, pk);
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(b_uw);
        }
    } else {
        const int q = warp & 3, v = v0 + 32 * q + lane;
        const uint32_t lane_base = (uint32_t)(32 * q) << 16;
        for (int c = 0; c < nc; ++c) {
            const int w = mbar_wait(b_of + 8 * (c & 1), (c >> 1) & 1, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) { fail = w == 1 ? 64 : -1; break; }
            tc_fence_after();
            uint32_t x[2][32];
            tmem_ld32(tmem + DT_O + 64 * (c & 1) + lane_base, x[0]);
            tmem_ld32(tmem + DT_O + 64 * (c & 1) + 32 + lane_base, x[1]);
            tmem_ld_fence(x[0]);
            tmem_ld_fence(x[1]);
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(b_oe + 8 * (c & 1));
            const int64_t t0 = (int64_t)c * DC;
            const int nt = (int)min((int64_t)DC, p.n - t0);
            float* out = p.o + (t0 * p.H + h) * p.dv + v;
            const int64_t step = (int64_t)p.H * p.dv;
            if (v < p.dv)
#pragma unroll
                for (int b = 0; b < 2; ++b)
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (32 * b + i < nt) out[(32 * b + i) * step] = __uint_as_float(x[b][i]);
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
