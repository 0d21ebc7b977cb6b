// Gated delta rule of prompt portions on tcgen05 (bfloat16 activations, d up to 128, sizes multiples of 8), in chunks of 64 tokens.
// With a chunk's inclusive decay products c_i (per key channel or per head), every correction u_i = beta_i (v_i - S^T k_i) depends
// on the state S at the chunk's start and on the earlier corrections:
//   (I + N) U = beta (V - (c K) S),   N_ij = beta_i (k_i . c_i / c_j k_j) for j < i,   T = (I + N)^-1 diag(beta)
//   U = T V - W S,  W = T (c K);   O = (c Q) S + B U,  B_ij = q_i . c_i / c_j k_j for j <= i;   S' = c_end S + E^T U,  E = c_end / c K
//
// delta_prep_*_kernel  per chunk and head, all in parallel: unit vectors, decays, N, B, the inverse, W, T V (one kernel per kind of
//                      decay).  Ratios c_i / c_j are products of decays, so that nothing overflows however strong the decay is
// delta_state_kernel   per head and 128 values, chunk after chunk: S^T lives in tensor memory (a lane per value), the products of a
//                      chunk take S or U as the tensor-memory operand
// delta_join_kernel    long portions with few heads run as several segments side by side: a first pass without outputs gives every
//                      segment's end from a zero start and, from unit vectors in place of values, the matrix that a start is
//                      multiplied with; the true starts follow from these; a second pass with them gives the outputs
// Operands that enter the recurrence are stored as two bfloat16 terms (16 significant bits, three MMAs per product; raw keys,
// queries and values are bfloat16 as projected and take one term); S itself is carried in float32.  Waits are bounded (status word
// codes 61..64).
#include "mix_delta.cuh"
#include "mix_tc.cuh"

namespace scmx {

constexpr int DC = 64;                   // tokens per chunk
constexpr int DC_BLK = 64 * 128;         // bytes of a [64 rows x 64 values] operand block
constexpr int DP_PITCH = 68;             // row pitch of the 64 x 64 matrices in shared memory

struct DeltaTcArgs {
    DeltaArgs p;
    bf16_t *wh, *wl, *qh, *ql, *eh, *el;     // [items][64][D]: -W, c Q, E
    bf16_t *bh, *bl;                         // [items][64][64]: B
    float* uv;                               // [items][value tiles][64][128]: T V
    float* gend;                             // [items][D]: c at the chunk's end
    int32_t* status;
    uint64_t wait_ns;
    int nc, nvt;                             // chunks, item = chunk * H + head; tiles of 128 values
    int nseg, len;                           // segments of `len` chunks (the last may be shorter)
    float *ends, *mats, *starts;             // [nseg][H, d, dv], [nseg][H, d, d], [nseg][H, d, dv]; one segment: unused
};

// Segments: as many CTAs as SMs in either pass, four chunks each at least.
constexpr int DT_SMS = 148;
static int segments(int nc, int H, int nvt) {
    int best = 1;
    for (int s = 3; s <= 16; ++s)
        if (nc / s >= 4 && H * nvt + (s - 2) * H * (nvt + 1) <= DT_SMS && s * H * nvt <= DT_SMS) best = s;
    return best;
}

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

__device__ __forceinline__ void split4(const float4 v, uint32_t& h0, uint32_t& h1, uint32_t& l0, uint32_t& l1) {
    split2(v.x, v.y, h0, l0);
    split2(v.z, v.w, h1, l1);
}
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float4 mul4(float4 a, float b) { return make_float4(a.x * b, a.y * b, a.z * b, a.w * b); }
template <int N> __device__ __forceinline__ void part_bar() { asm volatile("bar.sync 1, %0;" ::"n"(N) : "memory"); }

// 2^(nA softplus(z) log2 e) with z2 = z log2 e: the logarithm of the sum directly in base two.
__device__ __forceinline__ float decay_f32(float nA, float z2) {
    float l;
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(l) : "f"(1.0f + ex2_approx(-fabsf(z2))));
    return ex2_approx(nA * (fmaxf(z2, 0.0f) + l));
}

// Operands of one 16 x 16 (A) or 16 x 8 (B) block in shared memory as two terms.  Inner index: lane t4 holds t4 + 4 e of the 16.
__device__ __forceinline__ void block_a(const float* m, int lane, uint32_t (&ah)[4], uint32_t (&al)[4]) {
    const float *x = m + (lane >> 2) * DP_PITCH + (lane & 3), *y = x + 8 * DP_PITCH;
    split2(x[0], x[4], ah[0], al[0]);
    split2(y[0], y[4], ah[1], al[1]);
    split2(x[8], x[12], ah[2], al[2]);
    split2(y[8], y[12], ah[3], al[3]);
}
template <int PITCH>
__device__ __forceinline__ void block_b(const float* m, int lane, uint32_t (&bh)[2], uint32_t (&bl)[2]) {
    const float* x = m + (lane & 3) * PITCH + (lane >> 2);
    split2(x[0], x[4 * PITCH], bh[0], bl[0]);
    split2(x[8 * PITCH], x[12 * PITCH], bh[1], bl[1]);
}

// X = (I + N)^-1 by the first four warps: diagonal blocks of 16 (a lane per column), then 32 from 16 and 64 from 32 with
// X21 = -X22 (N21 X11), a warp per 8 columns.  Only entries below the diagonal of N are read; X above it is zero within blocks of 32.
// sT: four areas of [32][8] floats.
__device__ __forceinline__ void invert_unit_lower(const float* sN, float* sX, float* sT, int tid) {
    const int lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    {
        const int b0 = 16 * warp;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float s = i == lane ? 1.0f : 0.0f, s2 = 0.0f;
#pragma unroll
            for (int j = 0; j < i; ++j) {
                if (j & 1) s2 = fmaf(-sN[(b0 + i) * DP_PITCH + b0 + j], x[j], s2);
                else s = fmaf(-sN[(b0 + i) * DP_PITCH + b0 + j], x[j], s);
            }
            x[i] = s + s2;
        }
        if (lane < 16)
#pragma unroll
            for (int i = 0; i < 16; ++i) sX[(b0 + i) * DP_PITCH + b0 + lane] = x[i];
    }
    part_bar<128>();
    float* tile = sT + warp * 256;
    auto keep = [&](const float (&d)[4], float* out, int pitch, float sign) {      // a 16 x 8 result
        *reinterpret_cast<float2*>(out + g * pitch + 2 * t4) = make_float2(sign * d[0], sign * d[1]);
        *reinterpret_cast<float2*>(out + (g + 8) * pitch + 2 * t4) = make_float2(sign * d[2], sign * d[3]);
    };
    uint32_t ah[4], al[4], bh[2], bl[2];
    {
        const int b0 = 32 * (warp >> 1), c = b0 + 8 * (warp & 1);
        float d[4] = {};
        block_a(sN + (b0 + 16) * DP_PITCH + b0, lane, ah, al);
        block_b<DP_PITCH>(sX + b0 * DP_PITCH + c, lane, bh, bl);
        mma_split(d, ah, al, bh, bl);
        keep(d, tile, 8, 1.0f);
        __syncwarp();
        float x[4] = {};
        block_a(sX + (b0 + 16) * DP_PITCH + b0 + 16, lane, ah, al);
        block_b<8>(tile, lane, bh, bl);
        mma_split(x, ah, al, bh, bl);
        keep(x, sX + (b0 + 16) * DP_PITCH + c, DP_PITCH, -1.0f);
        const float zero[4] = {};
        keep(zero, sX + b0 * DP_PITCH + c + 16, DP_PITCH, 1.0f);      // above the diagonal, read by the products of 32
    }
    part_bar<128>();
    float d[2][4] = {}, x[2][4] = {};
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        block_b<DP_PITCH>(sX + 16 * k * DP_PITCH + 8 * warp, lane, bh, bl);
#pragma unroll
        for (int m = 0; m < 2; ++m) {
            block_a(sN + (32 + 16 * m) * DP_PITCH + 16 * k, lane, ah, al);
            mma_split(d[m], ah, al, bh, bl);
        }
    }
    __syncwarp();
    keep(d[0], tile, 8, 1.0f);
    keep(d[1], tile + 128, 8, 1.0f);
    __syncwarp();
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        block_b<8>(tile + 128 * k, lane, bh, bl);
#pragma unroll
        for (int m = 0; m < 2; ++m) {
            block_a(sX + (32 + 16 * m) * DP_PITCH + 32 + 16 * k, lane, ah, al);
            mma_split(x[m], ah, al, bh, bl);
        }
    }
    keep(x[0], sX + 32 * DP_PITCH + 8 * warp, DP_PITCH, -1.0f);
    keep(x[1], sX + 48 * DP_PITCH + 8 * warp, DP_PITCH, -1.0f);
}

// T = X diag(beta) as two terms in the order of the A operand: per block of 16 columns, word t4 + 4 u holds columns t4 + 8 u and
// t4 + 4 + 8 u.
constexpr int DT_PITCH = 36;             // words per row
__device__ __forceinline__ void pack_t(const float* sX, const float* beta, uint32_t* th, uint32_t* tl, int tid, int n) {
    for (int u = tid; u < 64 * 32; u += n) {
        const int i = u >> 5, w = u & 31, c = 16 * (w >> 3) + (w & 3) + 8 * ((w >> 2) & 1);
        if (16 * (w >> 3) > i) continue;             // blocks above the diagonal are not read
        split2(c <= i ? sX[i * DP_PITCH + c] * beta[c] : 0.0f, c + 4 <= i ? sX[i * DP_PITCH + c + 4] * beta[c + 4] : 0.0f, th[i * DT_PITCH + w],
               tl[i * DT_PITCH + w]);
    }
}

// The lower triangle of a 64 x 64 matrix as two terms, by `n` threads.
__device__ __forceinline__ void store_lower(const float* m, bf16_t* hi, bf16_t* lo, int item, int tid, int n) {
    for (int u = tid; u < 512; u += n) {
        const int i = u >> 3, j = 8 * (u & 7);
        uint32_t hw[4], lw[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = j + 2 * e;
            split2(c <= i ? m[i * DP_PITCH + c] : 0.0f, c + 1 <= i ? m[i * DP_PITCH + c + 1] : 0.0f, hw[e], lw[e]);
        }
        const int64_t o = ((int64_t)item * DC + i) * 64 + j;
        *reinterpret_cast<uint4*>(hi + o) = make_uint4(hw[0], hw[1], hw[2], hw[3]);
        *reinterpret_cast<uint4*>(lo + o) = make_uint4(lw[0], lw[1], lw[2], lw[3]);
    }
}

// Values of 64 tokens, columns v0 .. v0 + 127, -> shared memory, zeros outside.
constexpr int DV_PITCH = 136;
template <int NT>
__device__ __forceinline__ void load_values(const DeltaArgs& p, bf16_t* sV, int h, int64_t t0, int nt, int v0, int tid) {
#pragma unroll
    for (int i = 0; i < 1024 / NT; ++i) {
        const int u = tid + NT * i, t = u >> 4, c = 8 * (u & 15);
        uint4 w = make_uint4(0, 0, 0, 0);
        if (t < nt && v0 + c < p.dv) w = *reinterpret_cast<const uint4*>(static_cast<const bf16_t*>(p.v) + (t0 + t) * p.ldv + (int64_t)h * p.dv + v0 + c);
        *reinterpret_cast<uint4*>(sV + t * DV_PITCH + c) = w;
    }
}

// One warp: T Y for 16 columns of Y, all 64 rows.  Inner index as in T; columns: a lane's four results of a row are neighbours, 4 t4 ..
// column(j0, n, bh, bl): the operand of tokens j0 + t4 + 4 e, column 4 (g / 2) + (g & 1) + 2 n, in one (TERMS = 1) or two terms.
// put(row, four results).
template <int TERMS, typename Col, typename Put>
__device__ __forceinline__ void lower_product(const uint32_t* th, const uint32_t* tl, int lane, Col column, Put put) {
    const int g = lane >> 2, t4 = lane & 3;
    float acc[4][2][4] = {};
#pragma unroll
    for (int jb = 0; jb < 4; ++jb) {
        uint32_t bh[2][2], bl[2][2];
#pragma unroll
        for (int n = 0; n < 2; ++n) column(16 * jb, n, bh[n], bl[n]);
#pragma unroll
        for (int I = jb; I < 4; ++I) {
            const int o = (16 * I + g) * DT_PITCH + 8 * jb + t4;
            const uint32_t ah[4] = {th[o], th[o + 8 * DT_PITCH], th[o + 4], th[o + 8 * DT_PITCH + 4]};
            const uint32_t al[4] = {tl[o], tl[o + 8 * DT_PITCH], tl[o + 4], tl[o + 8 * DT_PITCH + 4]};
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                mma_16816(acc[I][n], ah, bh[n][0], bh[n][1]);
                mma_16816(acc[I][n], al, bh[n][0], bh[n][1]);
                if (TERMS == 2) mma_16816(acc[I][n], ah, bl[n][0], bl[n][1]);
            }
        }
    }
#pragma unroll
    for (int I = 0; I < 4; ++I)
#pragma unroll
        for (int e = 0; e < 2; ++e)
            put(16 * I + g + 8 * e, make_float4(acc[I][0][2 * e], acc[I][0][2 * e + 1], acc[I][1][2 * e], acc[I][1][2 * e + 1]));
}

// T V of the staged values, 16 columns per warp task.
__device__ __forceinline__ void values_product(const DeltaTcArgs& a, const uint32_t* th, const uint32_t* tl, const bf16_t* sV, int item, int v0, int group, int lane) {
    const int g = lane >> 2, t4 = lane & 3, ca = 16 * group + 4 * (g >> 1) + (g & 1), co = 16 * group + 4 * t4;
    float* out = a.uv + ((int64_t)item * a.nvt + (v0 >> 7)) * DC * 128;
    lower_product<1>(th, tl, lane,
        [&](int j0, int n, uint32_t (&bh)[2], uint32_t (&)[2]) {
            const bf16_t* v = sV + (j0 + t4) * DV_PITCH + ca + 2 * n;
            bh[0] = (uint32_t)v[0] | (uint32_t)v[4 * DV_PITCH] << 16;
            bh[1] = (uint32_t)v[8 * DV_PITCH] | (uint32_t)v[12 * DV_PITCH] << 16;
        },
        [&](int row, float4 r) { *reinterpret_cast<float4*>(out + row * 128 + co) = r; });
}

// -W: results of a row as two terms.
template <int D>
__device__ __forceinline__ void store_w(const DeltaTcArgs& a, int item, int row, int c, float4 r) {
    uint32_t h0, l0, h1, l1;
    split2(-r.x, -r.y, h0, l0);
    split2(-r.z, -r.w, h1, l1);
    const int64_t o = ((int64_t)item * DC + row) * D + c;
    *reinterpret_cast<uint2*>(a.wh + o) = make_uint2(h0, h1);
    *reinterpret_cast<uint2*>(a.wl + o) = make_uint2(l0, l1);
}

// Eight values as two terms, 16 bytes each.
__device__ __forceinline__ void store_terms8(bf16_t* hi, bf16_t* lo, float4 u, float4 v) {
    uint32_t hw[4], lw[4];
    split4(u, hw[0], hw[1], lw[0], lw[1]);
    split4(v, hw[2], hw[3], lw[2], lw[3]);
    *reinterpret_cast<uint4*>(hi) = make_uint4(hw[0], hw[1], hw[2], hw[3]);
    *reinterpret_cast<uint4*>(lo) = make_uint4(lw[0], lw[1], lw[2], lw[3]);
}

// The sums of x and y over the warp, in six shuffles.
__device__ __forceinline__ float2 warp_sum2(float x, float y, int lane) {
    const bool up = (lane & 16) != 0;
    float s = (up ? y : x) + __shfl_xor_sync(0xffffffffu, up ? x : y, 16);
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    const float other = __shfl_xor_sync(0xffffffffu, s, 16);
    return up ? make_float2(other, s) : make_float2(s, other);
}

// Row block I and key block b <= I of the pair-th pair of blocks of 16.
__device__ __forceinline__ void block_pair(int pair, int& I, int& b) {
    I = pair == 0 ? 0 : pair < 3 ? 1 : pair < 6 ? 2 : 3;
    b = pair - I * (I + 1) / 2;
}

// ---- a decay per key channel ----------------------------------------------------------------------------------------------
// Shared memory, in floats.  K, Q, G hold k, q, g, later k f, q f, k e with the decay products f from the start of a block of 16
// tokens and e to its end; PB the products of whole blocks, PI their reciprocals.  Within a block c_i / c_j = f_i e_j / product; a
// block with a channel below 2^-64 forms its ratios by running products instead.
constexpr int DPC_THREADS = 512;
template <int D>
struct DpcSmem {
    static constexpr int P = D + 16;         // row pitch: eight lanes of a 128-bit load fall into distinct banks
    static constexpr int K = 0, Q = K + 64 * P, G = Q + 64 * P, N = G + 64 * P, B = N + 64 * DP_PITCH, X = B + 64 * DP_PITCH, T = X + 64 * DP_PITCH,
                         V = T + 32 * 36, BETA = V + 64 * DV_PITCH / 2, PB = BETA + 64, PI = PB + 4 * D, STRONG = PI + 4 * D, FLOATS = STRONG + 4;
};

template <int D>
__global__ void __launch_bounds__(DPC_THREADS, 1) delta_prep_channel_kernel(const DeltaTcArgs a) {
    using L = DpcSmem<D>;
    constexpr int P = L::P, VC = D / 32;
    extern __shared__ __align__(16) float sm[];
    float *sk = sm + L::K, *sq = sm + L::Q, *sg = sm + L::G, *sN = sm + L::N, *sB = sm + L::B, *sX = sm + L::X;
    float *beta = sm + L::BETA, *pb = sm + L::PB, *pi = sm + L::PI;
    bf16_t* sV = reinterpret_cast<bf16_t*>(sm + L::V);
    int* strong = reinterpret_cast<int*>(sm + L::STRONG);
    pdl_launch_dependents();
    pdl_wait();
    const DeltaArgs& p = a.p;
    const int item = blockIdx.x, h = item % p.H, kh = h / (p.H / p.G);
    const int64_t t0 = (int64_t)(item / p.H) * DC;
    const int nt = (int)min((int64_t)DC, p.n - t0);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    // ---- unit vectors, decays, beta; tokens past the end become neutral (k = q = 0, beta = 0, decay 1)
    {
        const int e = VC * lane;
        const bool in = e < p.d;
        const bf16_t *q = static_cast<const bf16_t*>(p.q) + (int64_t)kh * p.d + e, *k = static_cast<const bf16_t*>(p.k) + (int64_t)kh * p.d + e;
        const float* ar = static_cast<const float*>(p.a) + (int64_t)h * p.d + e;
        uint32_t qw[4][VC / 2], kw[4][VC / 2];
        float z[4][VC], bl = 0.0f, dtb[VC];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int t = warp + 16 * r;
#pragma unroll
            for (int i = 0; i < VC / 2; ++i) qw[r][i] = kw[r][i] = 0;
#pragma unroll
            for (int i = 0; i < VC; ++i) z[r][i] = 0.0f;
            if (t < nt && in) {                  // rows are aligned for these loads (host side)
                if (VC == 4) {
                    *reinterpret_cast<uint2*>(qw[r]) = *reinterpret_cast<const uint2*>(q + (t0 + t) * p.ldq);
                    *reinterpret_cast<uint2*>(kw[r]) = *reinterpret_cast<const uint2*>(k + (t0 + t) * p.ldk);
                    *reinterpret_cast<float4*>(z[r]) = *reinterpret_cast<const float4*>(ar + (t0 + t) * p.lda);
                } else {
                    qw[r][0] = *reinterpret_cast<const uint32_t*>(q + (t0 + t) * p.ldq);
                    kw[r][0] = *reinterpret_cast<const uint32_t*>(k + (t0 + t) * p.ldk);
                    *reinterpret_cast<float2*>(z[r]) = *reinterpret_cast<const float2*>(ar + (t0 + t) * p.lda);
                }
            }
        }
        if (lane < 4 && warp + 16 * lane < nt) bl = ldf(static_cast<const bf16_t*>(p.b) + (t0 + warp + 16 * lane) * p.ldb + h);
#pragma unroll
        for (int i = 0; i < VC; ++i) dtb[i] = in ? p.dtb[(int64_t)h * p.d + e + i] : 0.0f;
        const float qs = rsqrtf((float)p.d), nA = p.nA[h];
        load_values<DPC_THREADS>(p, sV, h, t0, nt, 0, tid);
        if (tid < 4) strong[tid] = 0;
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int t = warp + 16 * r;
            float x[VC], y[VC], g[VC], qq = 0.0f, kk = 0.0f;
#pragma unroll
            for (int i = 0; i < VC / 2; ++i) {
                x[2 * i] = bf16_lo(qw[r][i]); x[2 * i + 1] = bf16_hi(qw[r][i]);
                y[2 * i] = bf16_lo(kw[r][i]); y[2 * i + 1] = bf16_hi(kw[r][i]);
            }
#pragma unroll
            for (int i = 0; i < VC; ++i) {
                qq = fmaf(x[i], x[i], qq);
                kk = fmaf(y[i], y[i], kk);
                g[i] = t < nt ? decay_f32(nA, (z[r][i] + dtb[i]) * 1.4426950408889634f) : 1.0f;
            }
            const float2 s = warp_sum2(qq, kk, lane);
            const float iq = qs * rsqrtf(s.x + 1e-6f), ik = rsqrtf(s.y + 1e-6f);
            const int o = t * P + e;
            if (VC == 4) {
                *reinterpret_cast<float4*>(sq + o) = make_float4(x[0] * iq, x[1] * iq, x[VC - 2] * iq, x[VC - 1] * iq);
                *reinterpret_cast<float4*>(sk + o) = make_float4(y[0] * ik, y[1] * ik, y[VC - 2] * ik, y[VC - 1] * ik);
                *reinterpret_cast<float4*>(sg + o) = make_float4(g[0], g[1], g[VC - 2], g[VC - 1]);
            } else {
                *reinterpret_cast<float2*>(sq + o) = make_float2(x[0] * iq, x[1] * iq);
                *reinterpret_cast<float2*>(sk + o) = make_float2(y[0] * ik, y[1] * ik);
                *reinterpret_cast<float2*>(sg + o) = make_float2(g[0], g[1]);
            }
        }
        if (lane < 4) beta[warp + 16 * lane] = warp + 16 * lane < nt ? sigmoid_f32(bl) : 0.0f;
    }
    __syncthreads();
    // ---- decay products within the blocks, a thread per channel and block
    {
        const int c = tid % D, b = tid / D;
        const bool work = b < 4;
        float *k = sk + 16 * b * P + c, *q = sq + 16 * b * P + c, *g = sg + 16 * b * P + c;
        float kk[16], gg[16], whole = 1.0f;
        if (work) {
#pragma unroll
            for (int t = 0; t < 16; ++t) {
                kk[t] = k[t * P];
                gg[t] = g[t * P];
                whole *= gg[t];
            }
            if (whole < 5.4e-20f) strong[b] = 1;
        }
        __syncthreads();
        if (strong[0] | strong[1] | strong[2] | strong[3]) {
            // diagonal blocks by running products: a warp carries four keys j, c_i / c_j k_j, from i = j on; lanes split the channels
            const int b0 = 16 * (warp >> 2), jg = 4 * (warp & 3);
            if (strong[warp >> 2]) {
                float kc[4][VC];
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int i = 0; i < VC; ++i) kc[j][i] = sk[(b0 + jg + j) * P + VC * lane + i];
                for (int i0 = jg; i0 < 16; ++i0) {
                    const int o = (b0 + i0) * P + VC * lane;
                    float s[8];
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        float n = 0.0f, m = 0.0f;
#pragma unroll
                        for (int i = 0; i < VC; ++i) {
                            if (i0 > jg + j) kc[j][i] *= sg[o + i];
                            n = fmaf(kc[j][i], sk[o + i], n);
                            m = fmaf(kc[j][i], sq[o + i], m);
                        }
                        s[2 * j] = n;
                        s[2 * j + 1] = m;
                    }
                    // eight sums over the warp: lane bits 4, 2, 1 choose, the others add
#pragma unroll
                    for (int n = 4; n > 0; n >>= 1) {
                        const bool up = (lane & n) != 0;
#pragma unroll
                        for (int i = 0; i < n; ++i) {
                            const float keep = up ? s[i + n] : s[i], give = up ? s[i] : s[i + n];
                            s[i] = keep + __shfl_xor_sync(0xffffffffu, give, n);
                        }
                    }
                    s[0] += __shfl_xor_sync(0xffffffffu, s[0], 8);
                    s[0] += __shfl_xor_sync(0xffffffffu, s[0], 16);
                    const int i = b0 + i0, j = b0 + jg + ((lane >> 1) & 3);
                    if (lane < 8) {
                        if (lane & 1) {
                            if (i >= j) sB[i * DP_PITCH + j] = s[0];
                        } else if (i > j) {
                            sN[i * DP_PITCH + j] = beta[i] * s[0];
                        }
                    }
                }
            }
            __syncthreads();
        }
        if (work) {
            float f = 1.0f, e = 1.0f;
#pragma unroll
            for (int t = 0; t < 16; ++t) {
                f *= gg[t];
                k[t * P] = kk[t] * f;
                q[t * P] *= f;
            }
            pb[b * D + c] = f;
            pi[b * D + c] = __fdividef(1.0f, f);
#pragma unroll
            for (int t = 15; t >= 0; --t) {
                g[t * P] = kk[t] * e;
                e *= gg[t];
            }
        }
    }
    __syncthreads();
    // ---- N and B by blocks of 16 x 16.  The inner index is permuted so that a lane's four values of a 16-step are neighbours.
    if (warp < 10) {
        int I, b;
        block_pair(warp, I, b);
        if (I != b || !strong[b]) {
            const int g = lane >> 2, t4 = lane & 3;
            const float *kr = sk + (16 * I + g) * P + 4 * t4, *qr = sq + (16 * I + g) * P + 4 * t4, *kc = sg + (16 * b + g) * P + 4 * t4;
            float n[2][4] = {}, m[2][4] = {};
#pragma unroll 2
            for (int s = 0; s < D; s += 16) {
                uint32_t ah[4], al[4], bh[2][2], bl[2][2];
                float4 v[2] = {*reinterpret_cast<const float4*>(kc + s), *reinterpret_cast<const float4*>(kc + 8 * P + s)};
                if (I != b + 1) {                // decay of the blocks between, or the block's own product taken back
                    float4 r = *reinterpret_cast<const float4*>((I == b ? pi + b * D : pb + (b + 1) * D) + s + 4 * t4);
                    if (I == b + 3) r = mul4(r, *reinterpret_cast<const float4*>(pb + (b + 2) * D + s + 4 * t4));
                    v[0] = mul4(v[0], r);
                    v[1] = mul4(v[1], r);
                }
#pragma unroll
                for (int j = 0; j < 2; ++j) split4(v[j], bh[j][0], bh[j][1], bl[j][0], bl[j][1]);
                split4(*reinterpret_cast<const float4*>(kr + s), ah[0], ah[2], al[0], al[2]);
                split4(*reinterpret_cast<const float4*>(kr + 8 * P + s), ah[1], ah[3], al[1], al[3]);
#pragma unroll
                for (int j = 0; j < 2; ++j) mma_split(n[j], ah, al, bh[j], bl[j]);
                split4(*reinterpret_cast<const float4*>(qr + s), ah[0], ah[2], al[0], al[2]);
                split4(*reinterpret_cast<const float4*>(qr + 8 * P + s), ah[1], ah[3], al[1], al[3]);
#pragma unroll
                for (int j = 0; j < 2; ++j) mma_split(m[j], ah, al, bh[j], bl[j]);
            }
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int e = u & 3, i = 16 * I + g + 8 * (e >> 1), j = 16 * b + 8 * (u >> 2) + 2 * t4 + (e & 1);
                if (i > j) sN[i * DP_PITCH + j] = beta[i] * n[u >> 2][e];
                if (i >= j) sB[i * DP_PITCH + j] = m[u >> 2][e];
            }
        }
    }
    __syncthreads();
    if (tid < 128) {
        invert_unit_lower(sN, sX, sm + L::T, tid);
    } else {
        // ---- meanwhile: c Q, E, B and c at the chunk's end
        for (int u = tid - 128; u < 64 * (D / 8); u += DPC_THREADS - 128) {
            const int t = u / (D / 8), c = 8 * (u % (D / 8)), b = t >> 4;
            const int64_t o = ((int64_t)item * DC + t) * D + c;
            const float4 *pf = reinterpret_cast<const float4*>(pb + c), *q = reinterpret_cast<const float4*>(sq + t * P + c), *e = reinterpret_cast<const float4*>(sg + t * P + c);
            float4 q0 = q[0], q1 = q[1], e0 = e[0], e1 = e[1];
#pragma unroll
            for (int w = 0; w < 4; ++w) {
                const float4 f0 = pf[w * (D / 4)], f1 = pf[w * (D / 4) + 1];
                if (w < b) {
                    q0 = mul4(q0, f0);
                    q1 = mul4(q1, f1);
                }
                if (w > b) {
                    e0 = mul4(e0, f0);
                    e1 = mul4(e1, f1);
                }
            }
            store_terms8(a.qh + o, a.ql + o, q0, q1);
            store_terms8(a.eh + o, a.el + o, e0, e1);
        }
        store_lower(sB, a.bh, a.bl, item, tid - 128, DPC_THREADS - 128);
        for (int c = tid - 128; c < D; c += DPC_THREADS - 128) a.gend[(int64_t)item * D + c] = pb[c] * pb[D + c] * pb[2 * D + c] * pb[3 * D + c];
    }
    __syncthreads();
    uint32_t *th = reinterpret_cast<uint32_t*>(sN), *tl = th + 64 * DT_PITCH;      // over N and B
    pack_t(sX, beta, th, tl, tid, DPC_THREADS);
    __syncthreads();
    // ---- -W = -X (beta c K) and T V
    for (int v0 = 0; v0 < p.dv; v0 += 128) {
        if (v0 > 0) {
            __syncthreads();
            load_values<DPC_THREADS>(p, sV, h, t0, nt, v0, tid);
            __syncthreads();
        }
        const int vg = min(8, (p.dv - v0 + 15) / 16), wgroups = v0 == 0 ? D / 16 : 0;
        for (int task = warp; task < wgroups + vg; task += DPC_THREADS / 32) {
            if (task < wgroups) {
                const int g = lane >> 2, t4 = lane & 3, ca = 16 * task + 4 * (g >> 1) + (g & 1);
                float pre[2] = {1.0f, 1.0f};     // decay of the blocks before, for this lane's two columns
                lower_product<2>(th, tl, lane,
                    [&](int j0, int n, uint32_t (&bh)[2], uint32_t (&bl)[2]) {
                        const float* k = sk + (j0 + t4) * P + ca + 2 * n;
                        split2(k[0] * pre[n], k[4 * P] * pre[n], bh[0], bl[0]);
                        split2(k[8 * P] * pre[n], k[12 * P] * pre[n], bh[1], bl[1]);
                        pre[n] *= pb[(j0 >> 4) * D + ca + 2 * n];
                    },
                    [&](int row, float4 r) { store_w<D>(a, item, row, 16 * task + 4 * t4, r); });
            } else {
                values_product(a, th, tl, sV, item, v0, task - wgroups, lane);
            }
        }
    }
}

// ---- a decay per head ------------------------------------------------------------------------------------------------------
// k and q stay as projected (bfloat16, exact); norms and decays are factors of rows and columns.  Two CTAs share an SM.
constexpr int DPH_THREADS = 256;
template <int D>
struct DphSmem {
    static constexpr int P = D + 8;          // bfloat16 row pitch
    static constexpr int K = 0, Q = K + 64 * P / 2, V = Q + 64 * P / 2, N = V + 64 * DV_PITCH / 2, B = N + 64 * DP_PITCH, X = B + 64 * DP_PITCH,
                         T = X + 64 * DP_PITCH, BETA = T + 32 * 36, IQ = BETA + 64, IK = IQ + 64, G = IK + 64, C = G + 64, W = C + 64, E = W + 64, FLOATS = E + 64;
};

template <int D>
__global__ void __launch_bounds__(DPH_THREADS, 2) delta_prep_head_kernel(const DeltaTcArgs a) {
    using L = DphSmem<D>;
    constexpr int P = L::P, VC = D / 32, NW = DPH_THREADS / 32;
    extern __shared__ __align__(16) float sm[];
    bf16_t *sk = reinterpret_cast<bf16_t*>(sm + L::K), *sq = reinterpret_cast<bf16_t*>(sm + L::Q), *sV = reinterpret_cast<bf16_t*>(sm + L::V);
    float *sN = sm + L::N, *sB = sm + L::B, *sX = sm + L::X;
    float *beta = sm + L::BETA, *iq = sm + L::IQ, *ik = sm + L::IK, *sg = sm + L::G, *sc = sm + L::C, *wk = sm + L::W, *we = sm + L::E;
    pdl_launch_dependents();
    pdl_wait();
    const DeltaArgs& p = a.p;
    const int item = blockIdx.x, h = item % p.H, kh = h / (p.H / p.G);
    const int64_t t0 = (int64_t)(item / p.H) * DC;
    const int nt = (int)min((int64_t)DC, p.n - t0);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    // ---- raw rows, norms, decays, beta; tokens past the end become neutral
    {
        const int e = VC * lane;
        const bool in = e < p.d;
        const bf16_t *q = static_cast<const bf16_t*>(p.q) + (int64_t)kh * p.d + e, *k = static_cast<const bf16_t*>(p.k) + (int64_t)kh * p.d + e;
        const float qs = rsqrtf((float)p.d);
        uint32_t qw[64 / NW][VC / 2], kw[64 / NW][VC / 2];
#pragma unroll
        for (int r = 0; r < 64 / NW; ++r) {
            const int t = warp + NW * r;
#pragma unroll
            for (int i = 0; i < VC / 2; ++i) qw[r][i] = kw[r][i] = 0;
            if (t < nt && in) {
                if (VC == 4) {
                    *reinterpret_cast<uint2*>(qw[r]) = *reinterpret_cast<const uint2*>(q + (t0 + t) * p.ldq);
                    *reinterpret_cast<uint2*>(kw[r]) = *reinterpret_cast<const uint2*>(k + (t0 + t) * p.ldk);
                } else {
                    qw[r][0] = *reinterpret_cast<const uint32_t*>(q + (t0 + t) * p.ldq);
                    kw[r][0] = *reinterpret_cast<const uint32_t*>(k + (t0 + t) * p.ldk);
                }
            }
        }
        if (tid < 64) {
            float bt = 0.0f, g = 1.0f;
            if (tid < nt) {
                bt = sigmoid_f32(ldf(static_cast<const bf16_t*>(p.b) + (t0 + tid) * p.ldb + h));
                g = decay_f32(p.nA[h], (ldf(static_cast<const bf16_t*>(p.a) + (t0 + tid) * p.lda + h) + p.dtb[h]) * 1.4426950408889634f);
            }
            beta[tid] = bt;
            sg[tid] = g;
        }
        load_values<DPH_THREADS>(p, sV, h, t0, nt, 0, tid);
#pragma unroll
        for (int r = 0; r < 64 / NW; ++r) {
            const int t = warp + NW * r;
            float qq = 0.0f, kk = 0.0f;
#pragma unroll
            for (int i = 0; i < VC / 2; ++i) {
                qq = fmaf(bf16_lo(qw[r][i]), bf16_lo(qw[r][i]), qq);
                qq = fmaf(bf16_hi(qw[r][i]), bf16_hi(qw[r][i]), qq);
                kk = fmaf(bf16_lo(kw[r][i]), bf16_lo(kw[r][i]), kk);
                kk = fmaf(bf16_hi(kw[r][i]), bf16_hi(kw[r][i]), kk);
                *reinterpret_cast<uint32_t*>(sq + t * P + e + 2 * i) = qw[r][i];
                *reinterpret_cast<uint32_t*>(sk + t * P + e + 2 * i) = kw[r][i];
            }
            const float2 s = warp_sum2(qq, kk, lane);
            if (lane == 0) {
                iq[t] = qs * rsqrtf(s.x + 1e-6f);
                ik[t] = rsqrtf(s.y + 1e-6f);
            }
        }
    }
    __syncthreads();
    // ---- c_i / c_j for i >= j into N's place: a thread takes key j and 16 tokens
    {
        const int j = tid & 63, s0 = 16 * (tid >> 6);
        float r = 1.0f;
#pragma unroll 8
        for (int t = 0; t < s0; ++t)
            if (t > j) r *= sg[t];
#pragma unroll
        for (int t = s0; t < s0 + 16; ++t) {
            if (t > j) r *= sg[t];
            sN[t * DP_PITCH + j] = r;            // meant for t >= j
            if (j == 0) sc[t] = r * sg[0];       // c itself
        }
    }
    __syncthreads();
    if (tid < 64) {
        wk[tid] = sc[tid] * ik[tid];
        we[tid] = sN[63 * DP_PITCH + tid] * ik[tid];      // before N is formed: the products to the chunk's end
    }
    __syncthreads();
    for (int pair = warp; pair < 10; pair += NW) {
        int I, b;
        block_pair(pair, I, b);
        const int g = lane >> 2, t4 = lane & 3;
        const bf16_t *kr = sk + (16 * I + g) * P + 2 * t4, *qr = sq + (16 * I + g) * P + 2 * t4, *kc = sk + (16 * b + g) * P + 2 * t4;
        auto at = [](const bf16_t* x) { return *reinterpret_cast<const uint32_t*>(x); };
        float n[2][4] = {}, m[2][4] = {};
#pragma unroll 4
        for (int s = 0; s < D; s += 16) {
            const uint32_t ka[4] = {at(kr + s), at(kr + 8 * P + s), at(kr + s + 8), at(kr + 8 * P + s + 8)};
            const uint32_t qa[4] = {at(qr + s), at(qr + 8 * P + s), at(qr + s + 8), at(qr + 8 * P + s + 8)};
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const uint32_t b0 = at(kc + 8 * j * P + s), b1 = at(kc + 8 * j * P + s + 8);
                mma_16816(n[j], ka, b0, b1);
                mma_16816(m[j], qa, b0, b1);
            }
        }
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int e = u & 3, i = 16 * I + g + 8 * (e >> 1), j = 16 * b + 8 * (u >> 2) + 2 * t4 + (e & 1);
            const float r = sN[i * DP_PITCH + j] * ik[j];
            if (i >= j) sB[i * DP_PITCH + j] = m[u >> 2][e] * r * iq[i];
            if (i > j) sN[i * DP_PITCH + j] = n[u >> 2][e] * r * ik[i] * beta[i];
        }
    }
    __syncthreads();
    if (tid < 128) {
        invert_unit_lower(sN, sX, sm + L::T, tid);
    } else {
        // ---- meanwhile: c Q, E, B and c at the chunk's end
        for (int u = tid - 128; u < 64 * (D / 8); u += 128) {
            const int t = u / (D / 8), c = 8 * (u % (D / 8));
            const int64_t o = ((int64_t)item * DC + t) * D + c;
            const float fq = iq[t] * sc[t], fe = we[t];
            float x[8], y[8];
            ld8(sq + t * P + c, x);
            ld8(sk + t * P + c, y);
            store_terms8(a.qh + o, a.ql + o, mul4(make_float4(x[0], x[1], x[2], x[3]), fq), mul4(make_float4(x[4], x[5], x[6], x[7]), fq));
            store_terms8(a.eh + o, a.el + o, mul4(make_float4(y[0], y[1], y[2], y[3]), fe), mul4(make_float4(y[4], y[5], y[6], y[7]), fe));
        }
        store_lower(sB, a.bh, a.bl, item, tid - 128, 128);
        for (int c = tid - 128; c < D; c += 128) a.gend[(int64_t)item * D + c] = sc[63];
    }
    __syncthreads();
    uint32_t *th = reinterpret_cast<uint32_t*>(sN), *tl = th + 64 * DT_PITCH;      // over N and B
    pack_t(sX, beta, th, tl, tid, DPH_THREADS);
    __syncthreads();
    for (int v0 = 0; v0 < p.dv; v0 += 128) {
        if (v0 > 0) {
            __syncthreads();
            load_values<DPH_THREADS>(p, sV, h, t0, nt, v0, tid);
            __syncthreads();
        }
        const int vg = min(8, (p.dv - v0 + 15) / 16), wgroups = v0 == 0 ? D / 16 : 0;
        for (int task = warp; task < wgroups + vg; task += NW) {
            if (task < wgroups) {
                const int g = lane >> 2, t4 = lane & 3, ca = 16 * task + 4 * (g >> 1) + (g & 1);
                lower_product<2>(th, tl, lane,
                    [&](int j0, int n, uint32_t (&bh)[2], uint32_t (&bl)[2]) {
                        const bf16_t* k = sk + (j0 + t4) * P + ca + 2 * n;
                        const float* w = wk + j0 + t4;
                        split2(ldf(k) * w[0], ldf(k + 4 * P) * w[4], bh[0], bl[0]);
                        split2(ldf(k + 8 * P) * w[8], ldf(k + 12 * P) * w[12], bh[1], bl[1]);
                    },
                    [&](int row, float4 r) { store_w<D>(a, item, row, 16 * task + 4 * t4, r); });
            } else {
                values_product(a, th, tl, sV, item, v0, task - wgroups, lane);
            }
        }
    }
}

// ---- the recurrence over chunks -----------------------------------------------------------------------------------------
// 576 threads: TMA warp, MMA warp (converged, one lane issues), four warpgroups that turn S into tensor-memory operands (a thread per
// value row, 32 channels each); the first two do the same with U (32 tokens each), the others store O.  Operands stream through a ring of 16 KB slots, per chunk:
//   per 64 channels {-W}, {c Q}, then E (D = 128: the high terms of all channels, the remainders; else both in one slot), {B}.
// Tensor memory: S^T float32 0..127, its two terms 128..255 (per 32 channels: 16 columns high, 16 remainder), U^T 256..319 (starts
// as T V, which the first two warpgroups put there a chunk ahead), its terms 320..383, O^T 384..511 (two buffers).
constexpr int DT_THREADS = 576;
constexpr int DT_SLOTS = 11, DT_SLOT = 2 * DC_BLK;
constexpr int DT_V_OFF = DT_SLOTS * DT_SLOT;                  // float [64][128]: T V of the next chunk
constexpr int DT_G_OFF = DT_V_OFF + 64 * 128 * 4;             // float [4][128]
constexpr int DT_BAR_OFF = DT_G_OFF + 4 * 512;                // full[], empty[], g[4], u, uw, s, sw, sc, of[2], oe[2], vf, ve
constexpr int DT_NBAR = 2 * DT_SLOTS + 15;
constexpr int DT_MISC_OFF = DT_BAR_OFF + 8 * DT_NBAR;
constexpr int DT_SMEM = DT_MISC_OFF + 16 + 1024;
constexpr uint32_t DT_SP = 128, DT_U = 256, DT_UP = 320, DT_O = 384;

// 32 float32 values as two bfloat16 terms: 16 columns high, 16 columns remainder.
__device__ __forceinline__ void split32(const uint32_t (&v)[32], uint32_t (&pk)[32]) {
#pragma unroll
    for (int i = 0; i < 16; ++i) split2(__uint_as_float(v[2 * i]), __uint_as_float(v[2 * i + 1]), pk[i], pk[16 + i]);
}

// OUT: the pass with outputs (or the only one), from `starts`.  Otherwise the first pass over segments 0 .. nseg - 2: blockIdx.y =
// value tile, or the unit vectors (nvt; not for segment 0, which starts from the carried state).
template <int DB, bool OUT>
__global__ void __launch_bounds__(DT_THREADS, 1)
    delta_state_kernel(const __grid_constant__ CUtensorMap tmWh, const __grid_constant__ CUtensorMap tmWl, const __grid_constant__ CUtensorMap tmQh,
                       const __grid_constant__ CUtensorMap tmQl, const __grid_constant__ CUtensorMap tmEh, const __grid_constant__ CUtensorMap tmEl,
                       const __grid_constant__ CUtensorMap tmBh, const __grid_constant__ CUtensorMap tmBl, const DeltaTcArgs a) {
    constexpr int D = 64 * DB;
    if (!OUT && (int)blockIdx.y == a.nvt && (int)blockIdx.z + 1 >= a.nseg - 1) return;      // the unit vectors have no further segment
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    const uint32_t sbase = smem_u32(smem);
    const uint32_t b_f = sbase + DT_BAR_OFF, b_e = b_f + 8 * DT_SLOTS, b_g = b_e + 8 * DT_SLOTS, b_u = b_g + 32, b_uw = b_u + 8, b_s = b_uw + 8,
                   b_sw = b_s + 8, b_sc = b_sw + 8, b_of = b_sc + 8, b_oe = b_of + 16, b_vf = b_oe + 16, b_ve = b_vf + 8;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + DT_MISC_OFF);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + DT_MISC_OFF + 4);
    const int warp = __shfl_sync(0xffffffffu, (int)(threadIdx.x >> 5), 0), lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (const CUtensorMap* m : {&tmWh, &tmWl, &tmQh, &tmQl, &tmEh, &tmEl, &tmBh, &tmBl}) prefetch_map(m);
        for (int i = 0; i < DT_NBAR; ++i) {
            const uint32_t b = b_f + 8 * i;
            mbar_init(b, b == b_uw || b == b_ve || b == b_oe || b == b_oe + 8 ? 8 : b == b_sw || b == b_sc ? 8 * DB : 1);
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
    const bool unit = !OUT && (int)blockIdx.y == a.nvt;
    const int h = blockIdx.x, v0 = unit ? 0 : blockIdx.y * 128, seg = blockIdx.z + (unit ? 1 : 0);
    const int cb = seg * a.len, nc = min(a.len, a.nc - cb), dv = unit ? p.d : p.dv;      // chunks cb .. cb + nc - 1
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
                const int item = (cb + c) * p.H + h, row = item * DC;
                // slot c & 3 of the decays is free: it was read before the products of chunk c - 4, whose operands left the ring
                bool first = true;
                if (int w = mbar_wait(b_ve, (c & 1) ^ 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 61 : -1; break; }
                if (!unit) mbar_expect_tx(b_vf, 64 * 128 * 4);
                if (!unit) bulk_load(sbase + DT_V_OFF, a.uv + ((int64_t)item * a.nvt + blockIdx.y) * DC * 128, 64 * 128 * 4, b_vf);
                for (int b = 0; b < DB && fail == 0; ++b)
                    if (slot()) {
                        tma_load_2d(s, &tmWh, 128 * b, row, bar);
                        tma_load_2d(s + DC_BLK, &tmWl, 128 * b, row, bar);
                        if (first) {
                            mbar_expect_tx(b_g + 8 * (c & 3), 4 * D);
                            bulk_load(sbase + DT_G_OFF + 512 * (c & 3), a.gend + (int64_t)item * D, 4 * D, b_g + 8 * (c & 3));
                        }
                        first = false;
                    }
                for (int b = 0; OUT && b < DB && fail == 0; ++b)
                    if (slot()) {
                        tma_load_2d(s, &tmQh, 128 * b, row, bar);
                        tma_load_2d(s + DC_BLK, &tmQl, 128 * b, row, bar);
                    }
                for (int b = 0; b < DB && fail == 0; ++b)
                    if (slot()) {
                        tma_load_2d(s, DB == 1 || b == 0 ? &tmEh : &tmEl, 0, row, bar);
                        tma_load_2d(s + DC_BLK, DB == 2 && b == 0 ? &tmEh : &tmEl, DB == 2 ? 128 : 0, row, bar);
                    }
                if (fail) break;
                if (!OUT) continue;
                if (!slot()) break;
                tma_load_2d(s, &tmBh, 0, row, bar);
                tma_load_2d(s + DC_BLK, &tmBl, 0, row, bar);
            }
        }
    } else if (warp == 1) {
        // the whole warp walks through the chunks; `on` is the lane that issues
        constexpr uint32_t idesc = umma_idesc_bf16(128, 64), idesc_e = umma_idesc_bf16(128, D) | IDESC_B_MN;
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
        bool ok = true;
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
            if (OUT && !wait(b_oe + 8 * (c & 1), ((c >> 1) & 1) ^ 1, 63)) break;
#pragma unroll
            for (int b = 0; OUT && b < DB; ++b) {
                if (!(ok = next())) break;
                split_product(o, tmem + DT_SP + 64 * b, b == 0);
                done();
            }
            if (!ok || !wait(b_uw, c & 1, 63) || !wait(b_sc, c & 1, 63)) break;
            {
                if (!(ok = next())) break;
                const uint64_t eh = umma_desc_mn(s, DC_BLK);
                uint64_t el = umma_desc_mn(s + DC_BLK, DC_BLK);
                const uint32_t efree = b_e + 8 * st;
                if (DB == 2) {
                    if (++st == DT_SLOTS) { st = 0; ph ^= 1; }
                    if (!(ok = next())) break;
                    el = umma_desc_mn(s, DC_BLK);
                }
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const uint32_t u = tmem + DT_UP + (k >> 1) * 32 + (k & 1) * 8;
                    umma_bf16_ts_on(on, tmem, u, eh + 128 * k, idesc_e, 1);
                    umma_bf16_ts_on(on, tmem, u, el + 128 * k, idesc_e, 1);
                    umma_bf16_ts_on(on, tmem, u + 16, eh + 128 * k, idesc_e, 1);
                }
                if (DB == 2) umma_commit_on(on, efree);
                done();
            }
            if (!ok) break;
            umma_commit_on(on, b_s);
            if (!OUT) continue;
            if (!(ok = next())) break;
            split_product(o, tmem + DT_UP, 0);
            done();
            umma_commit_on(on, b_of + 8 * (c & 1));
        }
        if (!on) fail = fail > 0 ? -1 : fail;      // one lane reports
    } else {
        const int wg = (warp - 2) >> 2, q = warp & 3, v = v0 + 32 * q + lane;
        const uint32_t lane_base = (uint32_t)(32 * q) << 16;
        const bool in = v < dv, owner = wg < 2 * DB;       // owner: holds 32 channels of S
        const int ch = 32 * wg;
        // this thread's row of a [heads, d, dv] state: channel ch, value v
        auto state_row = [&](float* base, int segment) { return base + ((int64_t)segment * p.H + h) * p.d * dv + (int64_t)ch * dv + v; };
        auto wait = [&](uint32_t bar, uint32_t parity) -> bool {
            const int w = mbar_wait(bar, parity, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) { fail = w == 1 ? 64 : -1; return false; }
            tc_fence_after();
            return true;
        };
        // T V of a chunk into U's place, this warpgroup's 32 tokens
        auto bring_values = [&](int c) -> bool {
            if (!unit && !wait(b_vf, c & 1)) return false;
            const float* src = reinterpret_cast<const float*>(smem + DT_V_OFF) + 32 * wg * 128 + 32 * q + lane;
            uint32_t u[32];
#pragma unroll
            for (int i = 0; i < 32; ++i) u[i] = in && !unit ? __float_as_uint(src[128 * i]) : 0u;
            __syncwarp();
            if (lane == 0) mbar_arrive(b_ve);
            tmem_st32(tmem + DT_U + 32 * wg + lane_base, u);
            return true;
        };
        const bool go = wg >= 2 || bring_values(0);
        for (int c = 0; c <= nc && go; ++c) {
            // S at the start of chunk c: its terms first, then c_end S for the sum; after the last chunk the state is stored
            if (owner) {
                if (c > 0 && !wait(b_s, (c - 1) & 1)) break;
                uint32_t s[32];
                if (c > 0) {
                    tmem_ld32(tmem + ch + lane_base, s);
                    tmem_ld_fence(s);
                } else {
                    const float* gS = a.nseg == 1 || (!OUT && seg == 0) ? state_row(p.state, 0) : OUT ? state_row(a.starts, seg) : nullptr;
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        float x = unit && v == ch + i ? 1.0f : 0.0f;
                        if (gS != nullptr && in && ch + i < p.d) x = gS[(int64_t)i * dv];
                        s[i] = __float_as_uint(x);
                    }
                }
                if (c == nc) {
                    float* gE = !OUT ? state_row(unit ? a.mats : a.ends, seg) : seg == a.nseg - 1 ? state_row(p.state, 0) : nullptr;
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (gE != nullptr && in && ch + i < p.d) gE[(int64_t)i * dv] = __uint_as_float(s[i]);
                } else {
                    uint32_t pk[32];
                    split32(s, pk);
                    tmem_st32(tmem + DT_SP + ch + lane_base, pk);
                    tmem_st_wait();
                    tc_fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive(b_sw);
                    if (!wait(b_g + 8 * (c & 3), (c >> 2) & 1)) break;
                    const ulonglong2* g = reinterpret_cast<const ulonglong2*>(smem + DT_G_OFF + 512 * (c & 3)) + ch / 4;
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        const ulonglong2 f = g[i];
                        const float2 x = unpack2(mul2(pack2(__uint_as_float(s[4 * i]), __uint_as_float(s[4 * i + 1])), f.x));
                        const float2 y = unpack2(mul2(pack2(__uint_as_float(s[4 * i + 2]), __uint_as_float(s[4 * i + 3])), f.y));
                        s[4 * i] = __float_as_uint(x.x); s[4 * i + 1] = __float_as_uint(x.y);
                        s[4 * i + 2] = __float_as_uint(y.x); s[4 * i + 3] = __float_as_uint(y.y);
                    }
                    tmem_st32(tmem + ch + lane_base, s);
                    tmem_st_wait();
                    tc_fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive(b_sc);
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
                if (c + 1 < nc && !bring_values(c + 1)) break;
            } else if (OUT && c > 0) {
                // outputs of the previous chunk, 32 tokens per warpgroup
                const int b = (c - 1) & 1;
                if (!wait(b_of + 8 * b, ((c - 1) >> 1) & 1)) break;
                uint32_t x[32];
                tmem_ld32(tmem + DT_O + 64 * b + 32 * (wg - 2) + lane_base, x);
                tmem_ld_fence(x);
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(b_oe + 8 * b);
                const int64_t t0 = (int64_t)(cb + c - 1) * DC + 32 * (wg - 2);
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


// Starts of the segments: start 0 is the carried state, start 1 what segment 0 ends with, start s + 1 = M_s start_s + end_s.  Grid
// (tiles of 8 NT values, heads); a warp owns 16 channels, operands in two terms.
template <int D, int NT>
__global__ void __launch_bounds__(2 * D) delta_join_kernel(const DeltaTcArgs a) {
    constexpr int PITCH = 8 * NT + 2;            // rows 4 t4 + e of four lanes fall into distinct banks
    __shared__ float sS[D * PITCH];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    const DeltaArgs& p = a.p;
    const int h = blockIdx.y, v = blockIdx.x * 8 * NT + 2 * t4, r0 = 16 * warp + g;      // results: rows r0, r0 + 8, values v + 8 n, v + 8 n + 1
    pdl_launch_dependents();
    pdl_wait();
    const int64_t head = (int64_t)h * p.d * p.dv, plane = (int64_t)p.H * p.d * p.dv;
    auto in = [&](int r, int n) { return r0 + 8 * r < p.d && v + 8 * n < p.dv; };
    const int64_t at[2] = {head + (int64_t)r0 * p.dv + v, head + (int64_t)(r0 + 8) * p.dv + v};
    // this warp's rows of M and of the end from zero; inner index: a lane's four values of a 16-step are neighbours
    struct Operand {
        float4 m[2][D / 16];
        float2 end[2][NT];
    } x, y;
    float2 cur[2][NT];
    auto request = [&](int seg, Operand& o) {
        const float* src = a.mats + ((int64_t)seg * p.H + h) * p.d * p.d;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int c = r0 + 8 * r;
#pragma unroll
            for (int k = 0; k < D / 16; ++k) {
                const int j = 16 * k + 4 * t4;
                o.m[r][k] = seg > 0 && c < p.d && j < p.d ? *reinterpret_cast<const float4*>(src + (int64_t)c * p.d + j) : make_float4(0, 0, 0, 0);
            }
#pragma unroll
            for (int n = 0; n < NT; ++n)
                o.end[r][n] = in(r, n) ? *reinterpret_cast<const float2*>(a.ends + seg * plane + at[r] + 8 * n) : make_float2(0, 0);
        }
    };
    // writes the start of a segment and forms the next one, whose operand was requested a segment ago
    auto step = [&](int seg, const Operand& o, Operand& next) -> bool {
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                if (in(r, n)) *reinterpret_cast<float2*>(a.starts + seg * plane + at[r] + 8 * n) = cur[r][n];
                *reinterpret_cast<float2*>(sS + (r0 + 8 * r) * PITCH + 8 * n + 2 * t4) = cur[r][n];
            }
        if (seg == a.nseg - 1) return false;
        if (seg + 1 < a.nseg - 1) request(seg + 1, next);
        __syncthreads();
        float acc[NT][3][4] = {};                // high high, high remainder, remainder high: shorter chains
        if (seg > 0) {
#pragma unroll
            for (int k = 0; k < D / 16; ++k) {
                uint32_t ah[4], al[4], bh[2], bl[2];
                split4(o.m[0][k], ah[0], ah[2], al[0], al[2]);
                split4(o.m[1][k], ah[1], ah[3], al[1], al[3]);
#pragma unroll
                for (int n = 0; n < NT; ++n) {
                    const float* s = sS + (16 * k + 4 * t4) * PITCH + 8 * n + g;
                    split2(s[0], s[PITCH], bh[0], bl[0]);
                    split2(s[2 * PITCH], s[3 * PITCH], bh[1], bl[1]);
                    mma_16816(acc[n][0], ah, bh[0], bh[1]);
                    mma_16816(acc[n][1], ah, bl[0], bl[1]);
                    mma_16816(acc[n][2], al, bh[0], bh[1]);
                }
            }
        }
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r)
                cur[r][n] = make_float2(o.end[r][n].x + (acc[n][0][2 * r] + (acc[n][1][2 * r] + acc[n][2][2 * r])),
                                        o.end[r][n].y + (acc[n][0][2 * r + 1] + (acc[n][1][2 * r + 1] + acc[n][2][2 * r + 1])));
        __syncthreads();
        return true;
    };
#pragma unroll
    for (int r = 0; r < 2; ++r)
#pragma unroll
        for (int n = 0; n < NT; ++n) cur[r][n] = in(r, n) ? *reinterpret_cast<const float2*>(p.state + at[r] + 8 * n) : make_float2(0, 0);
    request(0, x);
    for (int seg = 0; step(seg, x, y) && step(seg + 1, y, x); seg += 2) {
    }
}

bool delta_tc_supported(int64_t n, int H, int d, int dv, int64_t ldv) {
    return d % 8 == 0 && dv % 8 == 0 && d <= 128 && ldv % 8 == 0 && n < (1ll << 24) && (n + DC - 1) / DC * H < (1ll << 24);
}

static int64_t align256(int64_t b) { return (b + 255) / 256 * 256; }
static int width(int d) { return d <= 64 ? 64 : 128; }
static int64_t segment_bytes(int64_t n, int H, int d, int dv) {
    const int nseg = segments((int)((n + DC - 1) / DC), H, (dv + 127) / 128);
    return nseg == 1 ? 0 : 2 * align256((int64_t)nseg * H * d * dv * 4) + align256((int64_t)nseg * H * d * d * 4);
}
int64_t delta_tc_scratch(int64_t n, int H, int d, int dv) {
    const int64_t items = (n + DC - 1) / DC * H;
    return 6 * align256(items * DC * width(d) * 2) + 2 * align256(items * DC_BLK) + align256(items * ((dv + 127) / 128) * DC * 128 * 4) +
           align256(items * width(d) * 4) + segment_bytes(n, H, d, dv);
}

static int run_prep_tc(void (*kernel)(DeltaTcArgs), int smem, int threads, bool (&configured)[64], const DeltaTcArgs& a, cudaStream_t st) {
    const int dev = current_device();
    SCMX_REQUIRE(dev >= 0, SCMX_ECUDA, "no current CUDA device (ordinal 0..63)");
    if (!configured[dev]) {
        SCMX_CUDA_OK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        configured[dev] = true;
    }
    SCMX_PDL_OK("delta_prep_kernel", launch_pdl(kernel, dim3((unsigned)a.nc * a.p.H), dim3(threads), (size_t)smem, st, a));
    return SCMX_OK;
}

template <int D>
static int run_prep(bool channel, const DeltaTcArgs& a, cudaStream_t st) {
    static bool done[2][64] = {};
    return channel ? run_prep_tc(delta_prep_channel_kernel<D>, DpcSmem<D>::FLOATS * 4, DPC_THREADS, done[1], a, st)
                   : run_prep_tc(delta_prep_head_kernel<D>, DphSmem<D>::FLOATS * 4, DPH_THREADS, done[0], a, st);
}

template <int DB, bool OUT>
static int run_state(const CUtensorMap (&m)[8], const DeltaTcArgs& a, dim3 grid, cudaStream_t st) {
    static bool configured[64] = {};
    const int dev = current_device();
    SCMX_REQUIRE(dev >= 0, SCMX_ECUDA, "no current CUDA device (ordinal 0..63)");
    if (!configured[dev]) {
        SCMX_CUDA_OK(cudaFuncSetAttribute(delta_state_kernel<DB, OUT>, cudaFuncAttributeMaxDynamicSharedMemorySize, DT_SMEM));
        configured[dev] = true;
    }
    SCMX_PDL_OK("delta_state_kernel", launch_pdl(delta_state_kernel<DB, OUT>, grid, dim3(DT_THREADS), (size_t)DT_SMEM, st, m[0], m[1], m[2], m[3], m[4], m[5],
                                                 m[6], m[7], a));
    return SCMX_OK;
}
template <int DB>
static int run_states(const CUtensorMap (&m)[8], const DeltaTcArgs& a, cudaStream_t st) {
    if (a.nseg > 1) {
        // segments 0 .. nseg - 2 of the values, 1 .. nseg - 2 of the unit vectors: the latter's blockIdx.z counts from segment 1
        const int rc = run_state<DB, false>(m, a, dim3(a.p.H, a.nvt + 1, a.nseg - 1), st);
        if (rc) return rc;
        const int nt = (a.p.dv + 7) / 8 * a.p.H <= DT_SMS ? 1 : (a.p.dv + 15) / 16 * a.p.H <= DT_SMS ? 2 : 4;      // one round of CTAs
        const dim3 grid((a.p.dv + 8 * nt - 1) / (8 * nt), a.p.H), block(128 * DB);
        SCMX_PDL_OK("delta_join_kernel", nt == 1   ? launch_pdl(delta_join_kernel<64 * DB, 1>, grid, block, 0, st, a)
                                         : nt == 2 ? launch_pdl(delta_join_kernel<64 * DB, 2>, grid, block, 0, st, a)
                                                   : launch_pdl(delta_join_kernel<64 * DB, 4>, grid, block, 0, st, a));
    }
    return run_state<DB, true>(m, a, dim3(a.p.H, a.nvt, a.nseg), st);
}

int delta_tc(const DeltaArgs& p, bool channel, void* scratch, int32_t* status, cudaStream_t st) {
    SCMX_REQUIRE(p.ldq % 4 == 0 && p.ldk % 4 == 0 && (((uintptr_t)p.q | (uintptr_t)p.k) & 7) == 0 &&
                 (!channel || (p.lda % 4 == 0 && ((uintptr_t)p.a & 15) == 0)), SCMX_EINVAL, "delta: unaligned rows");
    DeltaTcArgs a;
    a.p = p; a.status = status; a.wait_ns = g_wait_limit_ns; a.nc = (int)((p.n + DC - 1) / DC); a.nvt = (p.dv + 127) / 128;
    const int64_t items = (int64_t)a.nc * p.H;
    const int D = width(p.d);
    uint8_t* s = static_cast<uint8_t*>(scratch);
    bf16_t** wide[6] = {&a.wh, &a.wl, &a.qh, &a.ql, &a.eh, &a.el};
    for (auto x : wide) { *x = reinterpret_cast<bf16_t*>(s); s += align256(items * DC * D * 2); }
    bf16_t** square[2] = {&a.bh, &a.bl};
    for (auto x : square) { *x = reinterpret_cast<bf16_t*>(s); s += align256(items * DC_BLK); }
    a.uv = reinterpret_cast<float*>(s); s += align256(items * a.nvt * DC * 128 * 4);
    a.gend = reinterpret_cast<float*>(s); s += align256(items * D * 4);
    a.nseg = segments(a.nc, p.H, a.nvt);
    a.len = (a.nc + a.nseg - 1) / a.nseg;
    a.nseg = (a.nc + a.len - 1) / a.len;         // no empty segment
    a.ends = reinterpret_cast<float*>(s); s += align256((int64_t)a.nseg * p.H * p.d * p.dv * 4);
    a.starts = reinterpret_cast<float*>(s); s += align256((int64_t)a.nseg * p.H * p.d * p.dv * 4);
    a.mats = reinterpret_cast<float*>(s);
    CUtensorMap m[8];
    int rc = 0;
    const bf16_t* src[8] = {a.wh, a.wl, a.qh, a.ql, a.eh, a.el, a.bh, a.bl};
    for (int i = 0; i < 8 && !rc; ++i) rc = make_map_u8(&m[i], src[i], items * DC, i < 6 ? 2 * D : 128, 128, DC, 128, 0);
    if (!rc) rc = D == 64 ? run_prep<64>(channel, a, st) : run_prep<128>(channel, a, st);
    if (rc) return rc;
    return D == 64 ? run_states<1>(m, a, st) : run_states<2>(m, a, st);
}

}  // namespace scmx
