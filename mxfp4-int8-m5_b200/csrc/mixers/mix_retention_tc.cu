// Retention of prompt portions on tcgen05 (bfloat16 activations, head size up to 256, sizes multiples of 8), chunk-parallel:
//   ret_prep_kernel    rotates q and k in float32 and stores each as two bfloat16 terms (high + remainder, 16 significant bits);
//                      a second copy of k carries decay^(distance to the end of its chunk)
//   ret_chunk_kernel   per chunk of RC tokens: U = sum_j decay^(end - j) k_j v_j^T, one [d, dv] matrix in float32
//   ret_carry_kernel   S_(c+1) = decay^len S_c + U_c over the chunks, float32; every S_c is stored as two bfloat16 terms
//   ret_out_kernel     o_i = sum_{j <= i, same chunk} decay^(i - j) (q_i . k_j) v_j + decay^(i - start + 1) S_c^T q_i
// Products of two split operands use three MMAs (high high, high remainder, remainder high), products with v (bfloat16 as
// projected) two, so that scores and everything that enters the state keep float32-like precision.  Waits are bounded (status
// word codes 41..45).
#include "mix_tc.cuh"

namespace scmx {

constexpr int RC = 256;                  // tokens per chunk: two tiles of 128
constexpr int RT_BLK = 128 * 128;        // bytes of a [128 rows x 64 values] operand block

struct RetTcArgs {
    const bf16_t *q, *k;     // [n, ld]: heads side by side
    const float* cs;         // [n, dims]
    const float* decay;      // [H]
    bf16_t *qh, *ql, *kh, *kl, *eh, *el;      // [H, n, d]
    float* U;                // [nc, H, d, dv]
    bf16_t *sh, *sl;         // [nc, H, d, dv]
    float* state;            // [H, d, dv]
    float* o;                // [n, H, dv]
    int32_t* status;
    uint64_t wait_ns;
    int64_t n, ldq, ldk;
    int H, d, dv, dims, nc;
    float kscale;
};

// Eight values as two bfloat16 terms.
__device__ __forceinline__ void put_split8(bf16_t* hi, bf16_t* lo, const float (&x)[8]) {
    uint32_t h[4], l[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        h[i] = pack_bf16x2(x[2 * i], x[2 * i + 1]);
        l[i] = pack_bf16x2(x[2 * i] - bf16_lo(h[i]), x[2 * i + 1] - bf16_hi(h[i]));
    }
    *reinterpret_cast<uint4*>(hi) = make_uint4(h[0], h[1], h[2], h[3]);
    *reinterpret_cast<uint4*>(lo) = make_uint4(l[0], l[1], l[2], l[3]);
}

// VEC: half of the rotated elements is a multiple of 8 and rows are 16-byte aligned, so that the eight partners of eight elements
// are one vector too.
template <bool VEC>
__global__ void __launch_bounds__(256) ret_prep_kernel(const RetTcArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x;
    const int64_t end = min(a.n, (t / RC + 1) * RC) - 1;
    const float* cs = a.cs + t * a.dims;
    const int half = a.dims >> 1;
    for (int i = 8 * threadIdx.x; i < a.H * a.d; i += 2048) {
        const int h = i / a.d, e = i - h * a.d;
        const bf16_t *q = a.q + t * a.ldq + (int64_t)h * a.d, *k = a.k + t * a.ldk + (int64_t)h * a.d;
        const float f = ex2_approx((float)(end - t) * log2f(a.decay[h]));
        const int64_t o = ((int64_t)h * a.n + t) * a.d + e;
        float x[8], y[8];
        if (VEC) {
            ld8(q + e, x);
            ld8(k + e, y);
            if (e < a.dims) {
                const bool lo = e < half;
                const int p = lo ? e + half : e - half, c = lo ? e : e - half;
                float qp[8], kp[8], cc[8], sn[8];
                ld8(q + p, qp);
                ld8(k + p, kp);
                ld8(cs + c, cc);
                ld8(cs + half + c, sn);
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const float s = lo ? -sn[j] : sn[j];
                    x[j] = fmaf(x[j], cc[j], qp[j] * s);
                    y[j] = fmaf(y[j], cc[j], kp[j] * s);
                }
            }
        } else {
            for (int j = 0; j < 8; ++j) {
                x[j] = rotated(q, e + j, a.dims, cs);
                y[j] = rotated(k, e + j, a.dims, cs);
            }
        }
        put_split8(a.qh + o, a.ql + o, x);
#pragma unroll
        for (int j = 0; j < 8; ++j) y[j] *= a.kscale;
        put_split8(a.kh + o, a.kl + o, y);
#pragma unroll
        for (int j = 0; j < 8; ++j) y[j] *= f;
        put_split8(a.eh + o, a.el + o, y);
    }
}

__global__ void __launch_bounds__(256) ret_carry_kernel(const RetTcArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t plane = (int64_t)a.d * a.dv, total = a.H * plane, i = 4 * ((int64_t)blockIdx.x * 256 + threadIdx.x);
    if (i >= total) return;                       // dv is a multiple of 4: four values of one head and row
    const float l2 = log2f(a.decay[i / plane]);
    float4 s = *reinterpret_cast<const float4*>(a.state + i);
#pragma unroll 4
    for (int c = 0; c < a.nc; ++c) {
        const float4 u = __ldcg(reinterpret_cast<const float4*>(a.U + c * total + i));
        const uint32_t h0 = pack_bf16x2(s.x, s.y), h1 = pack_bf16x2(s.z, s.w);
        *reinterpret_cast<uint2*>(a.sh + c * total + i) = make_uint2(h0, h1);
        *reinterpret_cast<uint2*>(a.sl + c * total + i) =
            make_uint2(pack_bf16x2(s.x - bf16_lo(h0), s.y - bf16_hi(h0)), pack_bf16x2(s.z - bf16_lo(h1), s.w - bf16_hi(h1)));
        const float f = exp2f((float)min((int64_t)RC, a.n - (int64_t)c * RC) * l2);
        s.x = fmaf(f, s.x, u.x); s.y = fmaf(f, s.y, u.y); s.z = fmaf(f, s.z, u.z); s.w = fmaf(f, s.w, u.w);
    }
    *reinterpret_cast<float4*>(a.state + i) = s;
}

// ---- chunk matrices -----------------------------------------------------------------------------------------------------
// Grid (chunks, heads, 128-row tiles of d x 128-column tiles of dv).  Both tiles of tokens are loaded at once; A (the weighted k)
// and B (v) are stored with the token index as rows, so both are read transposed.
constexpr int RK_THREADS = 192;
constexpr int RK_TILE = 6 * RT_BLK;      // per 128 tokens: e high 2 blocks, e remainder 2, v 2
constexpr int RK_SMEM = 2 * RK_TILE + 64 + 1024;

__global__ void __launch_bounds__(RK_THREADS, 1) ret_chunk_kernel(const __grid_constant__ CUtensorMap tmEh, const __grid_constant__ CUtensorMap tmEl,
                                                           const __grid_constant__ CUtensorMap tmV, const RetTcArgs a) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    const uint32_t sbase = smem_u32(smem), b_full = sbase + 2 * RK_TILE, b_done = b_full + 16;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + 2 * RK_TILE + 32);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + 2 * RK_TILE + 36);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        prefetch_map(&tmEh);
        prefetch_map(&tmEl);
        prefetch_map(&tmV);
        mbar_init(b_full, 1);
        mbar_init(b_full + 8, 1);
        mbar_init(b_done, 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        tmem_alloc(smem_u32(tmem_slot), 128);
        tmem_relinquish();
    }
    pdl_launch_dependents();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    pdl_wait();
    const int c = blockIdx.x, h = blockIdx.y, nvt = (a.dv + 127) / 128;
    const int d0 = (blockIdx.z / nvt) * 128, v0 = (blockIdx.z % nvt) * 128;
    const int t0 = c * RC, ntile = a.n - t0 > 128 ? 2 : 1;
    int fail = 0;
    if (warp == 0) {
        if (lane == 0)
            for (int t = 0; t < ntile; ++t) {
                const uint32_t s = sbase + t * RK_TILE, bar = b_full + 8 * t;
                mbar_expect_tx(bar, RK_TILE);
                for (int b = 0; b < 2; ++b) {
                    tma_load_3d(s + b * RT_BLK, &tmEh, 2 * d0 + 128 * b, t0 + 128 * t, h, bar);
                    tma_load_3d(s + (2 + b) * RT_BLK, &tmEl, 2 * d0 + 128 * b, t0 + 128 * t, h, bar);
                    tma_load_3d(s + (4 + b) * RT_BLK, &tmV, 2 * v0 + 128 * b, t0 + 128 * t, h, bar);
                }
            }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = umma_idesc_bf16(128, 128) | IDESC_A_MN | IDESC_B_MN;
            for (int t = 0; t < ntile; ++t) {
                if (int w = mbar_wait(b_full + 8 * t, 0, abort_flag, a.wait_ns)) { fail = w == 1 ? 41 : -1; break; }
                tc_fence_after();
                const uint32_t s = sbase + t * RK_TILE;
                const uint64_t eh = umma_desc_mn(s, RT_BLK), el = umma_desc_mn(s + 2 * RT_BLK, RT_BLK), v = umma_desc_mn(s + 4 * RT_BLK, RT_BLK);
#pragma unroll
                for (int k = 0; k < 8; ++k) {
                    umma_bf16(tmem, eh + 128 * k, v + 128 * k, idesc, (t | k) != 0);
                    umma_bf16(tmem, el + 128 * k, v + 128 * k, idesc, 1);
                }
            }
            if (fail == 0) umma_commit(b_done);
        }
    } else {
        int w = mbar_wait(b_done, 0, abort_flag, a.wait_ns);
        if (__any_sync(0xffffffffu, w)) {
            fail = w == 1 ? 42 : -1;
        } else {
            tc_fence_after();
            const int q = warp & 3, r = d0 + 32 * q + lane;
            float* out = a.U + (((int64_t)c * a.H + h) * a.d + r) * a.dv + v0;
#pragma unroll
            for (int b = 0; b < 4; ++b) {
                uint32_t v[32];
                tmem_ld32(tmem + 32 * b + ((uint32_t)(32 * q) << 16), v);
                tmem_ld_fence(v);
                if (r < a.d)
#pragma unroll
                    for (int i = 0; i < 32; i += 4)
                        if (v0 + 32 * b + i < a.dv) *reinterpret_cast<uint4*>(out + 32 * b + i) = make_uint4(v[i], v[i + 1], v[i + 2], v[i + 3]);
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
    if (warp == 1) tmem_dealloc(tmem, 128);
}

// ---- outputs ------------------------------------------------------------------------------------------------------------
// Grid (query tiles of 128, heads, 128-column tiles of dv), 320 threads: TMA warp, MMA warp, two warpgroups.  Key tile t of the
// chunk (t = 0, 1) is weighted by warpgroup t, a thread per query row, while the MMA thread runs the state product.  Operands
// other than Q stream through a ring of 32 KB stages in the order of their use:
//   per key tile and 64 elements of d: {k high, k remainder}; per 128 rows of d and 64 columns: {S high, S remainder}; per key
//   tile: v (two blocks of 64 columns).
template <int KB>
struct RoCfg {
    static constexpr int STAGES = KB == 1 ? 5 : KB == 2 ? 4 : 3;
    static constexpr int STAGE = 2 * RT_BLK;
    static constexpr int Q_BYTES = 2 * KB * RT_BLK;                    // high blocks, then remainder blocks
    static constexpr int RING_OFF = Q_BYTES;
    static constexpr int BAR_OFF = RING_OFF + STAGES * STAGE;          // q, full[], empty[], s[2], p[2], o
    static constexpr int MISC_OFF = BAR_OFF + 8 * (2 * STAGES + 6);
    static constexpr int TOTAL = MISC_OFF + 16 + 1024;
};
constexpr int RO_THREADS = 320;

template <int KB>
__global__ void __launch_bounds__(RO_THREADS, 1)
    ret_out_kernel(const __grid_constant__ CUtensorMap tmQh, const __grid_constant__ CUtensorMap tmQl, const __grid_constant__ CUtensorMap tmKh,
                   const __grid_constant__ CUtensorMap tmKl, const __grid_constant__ CUtensorMap tmSh, const __grid_constant__ CUtensorMap tmSl,
                   const __grid_constant__ CUtensorMap tmV, const RetTcArgs a) {
    using L = RoCfg<KB>;
    constexpr int STAGES = L::STAGES;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    const uint32_t sbase = smem_u32(smem), ring = sbase + L::RING_OFF;
    const uint32_t b_q = sbase + L::BAR_OFF, b_f = b_q + 8, b_e = b_f + 8 * STAGES, b_s = b_e + 8 * STAGES, b_p = b_s + 16, b_o = b_p + 16;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + L::MISC_OFF);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + L::MISC_OFF + 4);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (const CUtensorMap* m : {&tmQh, &tmQl, &tmKh, &tmKl, &tmSh, &tmSl, &tmV}) prefetch_map(m);
        for (int i = 0; i < 2 * STAGES + 6; ++i) {
            const uint32_t b = b_q + 8 * i;
            mbar_init(b, b == b_p || b == b_p + 8 ? 4 : 1);
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
    const int qt = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 128;
    const int q0 = qt * 128, c = q0 / RC, k0 = c * RC, ntile = (q0 - k0) / 128 + 1;      // key tiles up to the diagonal one
    const int rows = (int)min((int64_t)128, a.n - q0);
    const int nkb = (a.d + 63) / 64, ndt = (a.d + 127) / 128, nvb = a.dv - v0 > 64 ? 2 : 1;
    int fail = 0;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(b_q, 2 * nkb * RT_BLK);
            for (int b = 0; b < nkb; ++b) {
                tma_load_3d(sbase + b * RT_BLK, &tmQh, 128 * b, q0, h, b_q);
                tma_load_3d(sbase + (KB + b) * RT_BLK, &tmQl, 128 * b, q0, h, b_q);
            }
            int i = 0;
            auto stage = [&](uint32_t& s, uint32_t& bar) -> bool {       // next free stage, armed for its 32 KB
                const int st = i % STAGES;
                if (int w = mbar_wait(b_e + 8 * st, ((i / STAGES) & 1) ^ 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 43 : -1; return false; }
                s = ring + st * L::STAGE;
                bar = b_f + 8 * st;
                mbar_expect_tx(bar, L::STAGE);
                ++i;
                return true;
            };
            uint32_t s, bar;
            for (int t = 0; t < ntile && fail == 0; ++t)
                for (int b = 0; b < nkb; ++b) {
                    if (!stage(s, bar)) break;
                    tma_load_3d(s, &tmKh, 128 * b, k0 + 128 * t, h, bar);
                    tma_load_3d(s + RT_BLK, &tmKl, 128 * b, k0 + 128 * t, h, bar);
                }
            for (int r = 0; r < ndt && fail == 0; ++r)
                for (int b = 0; b < nvb; ++b) {
                    if (!stage(s, bar)) break;
                    tma_load_3d(s, &tmSh, 2 * v0 + 128 * b, 128 * r, c * a.H + h, bar);
                    tma_load_3d(s + RT_BLK, &tmSl, 2 * v0 + 128 * b, 128 * r, c * a.H + h, bar);
                }
            for (int t = 0; t < ntile && fail == 0; ++t) {
                if (!stage(s, bar)) break;
                tma_load_3d(s, &tmV, 2 * v0, k0 + 128 * t, h, bar);
                tma_load_3d(s + RT_BLK, &tmV, 2 * v0 + 128, k0 + 128 * t, h, bar);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc_s = umma_idesc_bf16(128, 128), idesc_v = idesc_s | IDESC_B_MN;
            constexpr uint32_t idesc_64 = umma_idesc_bf16(128, 64) | IDESC_B_MN;
            int i = 0;
            auto next = [&](uint32_t& s) -> bool {
                const int st = i % STAGES;
                if (int w = mbar_wait(b_f + 8 * st, (i / STAGES) & 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 44 : -1; return false; }
                tc_fence_after();
                s = ring + st * L::STAGE;
                return true;
            };
            auto done = [&]() { umma_commit(b_e + 8 * (i % STAGES)); ++i; };
            uint32_t s;
            if (int w = mbar_wait(b_q, 0, abort_flag, a.wait_ns)) fail = w == 1 ? 44 : -1;
            for (int t = 0; t < ntile && fail == 0; ++t) {
                for (int b = 0; b < nkb; ++b) {
                    if (!next(s)) break;
                    const uint64_t qh = umma_desc(sbase + b * RT_BLK), ql = umma_desc(sbase + (KB + b) * RT_BLK), kh = umma_desc(s), kl = umma_desc(s + RT_BLK);
                    const int steps = min(4, (a.d - 64 * b + 15) / 16);
                    for (int k = 0; k < steps; ++k) {
                        umma_bf16(tmem + 128 * t, qh + 2 * k, kh + 2 * k, idesc_s, (b | k) != 0);
                        umma_bf16(tmem + 128 * t, qh + 2 * k, kl + 2 * k, idesc_s, 1);
                        umma_bf16(tmem + 128 * t, ql + 2 * k, kh + 2 * k, idesc_s, 1);
                    }
                    done();
                }
                if (fail == 0) umma_commit(b_s + 8 * t);
            }
            for (int r = 0; r < ndt && fail == 0; ++r)
                for (int b = 0; b < nvb; ++b) {
                    if (!next(s)) break;
                    const uint64_t sh = umma_desc_mn(s, RT_BLK), sl = umma_desc_mn(s + RT_BLK, RT_BLK);
                    const int steps = min(8, (a.d - 128 * r + 15) / 16);
                    for (int k = 0; k < steps; ++k) {
                        const uint32_t qo = (2 * r + (k >> 2)) * RT_BLK;
                        const uint64_t qh = umma_desc(sbase + qo) + 2 * (k & 3), ql = umma_desc(sbase + KB * RT_BLK + qo) + 2 * (k & 3);
                        umma_bf16(tmem + 384 + 64 * b, qh, sh + 128 * k, idesc_64, (r | k) != 0);
                        umma_bf16(tmem + 384 + 64 * b, qh, sl + 128 * k, idesc_64, 1);
                        umma_bf16(tmem + 384 + 64 * b, ql, sh + 128 * k, idesc_64, 1);
                    }
                    done();
                }
            for (int t = 0; t < ntile && fail == 0; ++t) {
                if (int w = mbar_wait(b_p + 8 * t, 0, abort_flag, a.wait_ns)) { fail = w == 1 ? 44 : -1; break; }
                if (!next(s)) break;
                const uint64_t v = umma_desc_mn(s, RT_BLK);
#pragma unroll
                for (int k = 0; k < 8; ++k) {
                    const uint32_t pa = tmem + 128 * t + (k >> 1) * 32 + (k & 1) * 8;
                    umma_bf16_ts(tmem + 256, pa, v + 128 * k, idesc_v, (t | k) != 0);
                    umma_bf16_ts(tmem + 256, pa + 16, v + 128 * k, idesc_v, 1);
                }
                done();
            }
            if (fail == 0) umma_commit(b_o);
        }
    } else {
        const int t = (warp - 2) >> 2, q = warp & 3, row = 32 * q + lane;
        const uint32_t lane_base = (uint32_t)(32 * q) << 16;
        const float l2 = log2f(a.decay[h]);
        const int pos = q0 - k0 + row;            // place in the chunk
        if (t < ntile) {
            int w = mbar_wait(b_s + 8 * t, 0, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) {
                fail = w == 1 ? 45 : -1;
            } else {
                tc_fence_after();
                const uint32_t ts = tmem + 128 * t + lane_base;
                const int dist0 = pos - 128 * t;          // distance to the tile's first key
                const float far = (float)dist0 * l2;
                uint32_t r[2][32];
                tmem_ld32(ts, r[0]);
                tmem_ld_fence(r[0]);
#pragma unroll
                for (int b = 0; b < 4; ++b) {
                    uint32_t(&v)[32] = r[b & 1];
                    if (b < 3) tmem_ld32(ts + 32 * (b + 1), r[(b + 1) & 1]);
                    uint32_t pk[32];
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        float x[2];
#pragma unroll
                        for (int e = 0; e < 2; ++e) {
                            const int j = 32 * b + 2 * i + e;
                            x[e] = j <= dist0 ? __uint_as_float(v[2 * i + e]) * ex2_approx(fmaf((float)-j, l2, far)) : 0.0f;
                        }
                        const uint32_t hi = pack_bf16x2(x[0], x[1]);
                        pk[i] = hi;
                        pk[16 + i] = pack_bf16x2(x[0] - bf16_lo(hi), x[1] - bf16_hi(hi));
                    }
                    if (b < 3) tmem_ld_fence(r[(b + 1) & 1]);
                    tmem_st32(ts + 32 * b, pk);
                }
                tmem_st_wait();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(b_p + 8 * t);
            }
        }
        if (fail == 0) {
            int w = mbar_wait(b_o, 0, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) {
                fail = w == 1 ? 45 : -1;
            } else {
                // warpgroup t stores value columns 64 t .. 64 t + 63
                tc_fence_after();
                const float f = ex2_approx((float)(pos + 1) * l2);
                float* out = a.o + ((int64_t)(q0 + row) * a.H + h) * a.dv + v0;
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    const int col = 64 * t + 32 * b;
                    uint32_t u[32], v[32];
                    tmem_ld32(tmem + 256 + col + lane_base, u);
                    tmem_ld32(tmem + 384 + col + lane_base, v);
                    tmem_ld_fence(u);
                    tmem_ld_fence(v);
                    if (row < rows)
#pragma unroll
                        for (int i = 0; i < 32; i += 4)
                            if (v0 + col + i < a.dv)
                                *reinterpret_cast<float4*>(out + col + i) = make_float4(
                                    fmaf(f, __uint_as_float(v[i]), __uint_as_float(u[i])), fmaf(f, __uint_as_float(v[i + 1]), __uint_as_float(u[i + 1])),
                                    fmaf(f, __uint_as_float(v[i + 2]), __uint_as_float(u[i + 2])), fmaf(f, __uint_as_float(v[i + 3]), __uint_as_float(u[i + 3])));
                }
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

template <int KB>
static int launch_ro(const CUtensorMap (&m)[7], const RetTcArgs& a, cudaStream_t st) {
    using L = RoCfg<KB>;
    static bool configured[64] = {};
    const int dev = current_device();
    SCMX_REQUIRE(dev >= 0, SCMX_ECUDA, "no current CUDA device (ordinal 0..63)");
    if (!configured[dev]) {
        SCMX_CUDA_OK(cudaFuncSetAttribute(ret_out_kernel<KB>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL));
        configured[dev] = true;
    }
    const dim3 grid((unsigned)((a.n + 127) / 128), a.H, (a.dv + 127) / 128);
    SCMX_PDL_OK("ret_out_kernel", launch_pdl(ret_out_kernel<KB>, grid, dim3(RO_THREADS), (size_t)L::TOTAL, st, m[0], m[1], m[2], m[3], m[4], m[5], m[6], a));
    return SCMX_OK;
}

bool retention_tc_supported(int64_t n, int H, int d, int dv, int dims, int64_t ldv) {
    return d % 8 == 0 && dv % 8 == 0 && d <= 256 && ldv % 8 == 0 && dims % 2 == 0 && n < (1ll << 24) && H <= 65535;
}

// Scratch: six [H, n, d] and two [nc, H, d, dv] bfloat16 arrays, one [nc, H, d, dv] float array, 256-byte aligned each.
static int64_t align256(int64_t b) { return (b + 255) / 256 * 256; }
int64_t retention_tc_scratch(int64_t n, int H, int d, int dv) {
    const int64_t nc = (n + RC - 1) / RC;
    return 6 * align256(2 * n * H * d) + 2 * align256(2 * nc * H * d * dv) + align256(4 * nc * H * d * dv);
}

int retention_tc(const bf16_t* q, int64_t ldq, const bf16_t* k, int64_t ldk, const bf16_t* v, int64_t ldv, int64_t n, int H, int d, int dv,
                 const float* cs, int dims, float kscale, const float* decay, float* state, float* o, void* scratch, int32_t* status,
                 cudaStream_t st) {
    RetTcArgs a;
    a.q = q; a.k = k; a.cs = cs; a.decay = decay; a.state = state; a.o = o; a.status = status; a.wait_ns = g_wait_limit_ns;
    a.n = n; a.ldq = ldq; a.ldk = ldk; a.H = H; a.d = d; a.dv = dv; a.dims = dims; a.nc = (int)((n + RC - 1) / RC); a.kscale = kscale;
    uint8_t* p = static_cast<uint8_t*>(scratch);
    bf16_t** act[6] = {&a.qh, &a.ql, &a.kh, &a.kl, &a.eh, &a.el};
    for (auto x : act) { *x = reinterpret_cast<bf16_t*>(p); p += align256(2 * n * H * d); }
    const int64_t sz = (int64_t)a.nc * H * d * dv;
    a.sh = reinterpret_cast<bf16_t*>(p); p += align256(2 * sz);
    a.sl = reinterpret_cast<bf16_t*>(p); p += align256(2 * sz);
    a.U = reinterpret_cast<float*>(p);
    CUtensorMap m[7], eh, el;
    int rc = 0;
    const bf16_t* src[4] = {a.qh, a.ql, a.kh, a.kl};
    for (int i = 0; i < 4 && !rc; ++i) rc = make_map_planes(&m[i], src[i], H, n, 2 * d, 2 * d, 2 * n * d, 128);
    if (!rc) rc = make_map_planes(&m[4], a.sh, (int64_t)a.nc * H, d, 2 * dv, 2 * dv, 2ll * d * dv, 128);
    if (!rc) rc = make_map_planes(&m[5], a.sl, (int64_t)a.nc * H, d, 2 * dv, 2 * dv, 2ll * d * dv, 128);
    if (!rc) rc = make_map_planes(&m[6], v, H, n, 2 * dv, 2 * ldv, 2 * dv, 128);
    if (!rc) rc = make_map_planes(&eh, a.eh, H, n, 2 * d, 2 * d, 2 * n * d, 128);
    if (!rc) rc = make_map_planes(&el, a.el, H, n, 2 * d, 2 * d, 2 * n * d, 128);
    if (rc) return rc;
    const bool vec = dims % 16 == 0 && ldq % 8 == 0 && ldk % 8 == 0 && (((uintptr_t)q | (uintptr_t)k | (uintptr_t)cs) & 15) == 0;
    SCMX_PDL_OK("ret_prep_kernel", vec ? launch_pdl(ret_prep_kernel<true>, dim3((unsigned)n), dim3(256), 0, st, a)
                                       : launch_pdl(ret_prep_kernel<false>, dim3((unsigned)n), dim3(256), 0, st, a));
    static bool configured[64] = {};
    const int dev = current_device();
    SCMX_REQUIRE(dev >= 0, SCMX_ECUDA, "no current CUDA device (ordinal 0..63)");
    if (!configured[dev]) {
        SCMX_CUDA_OK(cudaFuncSetAttribute(ret_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, RK_SMEM));
        configured[dev] = true;
    }
    SCMX_PDL_OK("ret_chunk_kernel", launch_pdl(ret_chunk_kernel, dim3(a.nc, H, ((d + 127) / 128) * ((dv + 127) / 128)), dim3(RK_THREADS), (size_t)RK_SMEM, st,
                                               eh, el, m[6], a));
    const int64_t quads = (int64_t)H * d * dv / 4;
    SCMX_PDL_OK("ret_carry_kernel", launch_pdl(ret_carry_kernel, dim3((unsigned)((quads + 255) / 256)), dim3(256), 0, st, a));
    if (d <= 64) return launch_ro<1>(m, a, st);
    if (d <= 128) return launch_ro<2>(m, a, st);
    return launch_ro<4>(m, a, st);
}

}  // namespace scmx
