// Differential attention of prompt portions on tcgen05 (bfloat16 cache, head sizes up to 128, multiples of 8).
//
// A CTA owns 128 query rows of one head and BOTH maps: the maps share the value tiles, and while the tensor core works on one
// map the other map's softmax runs, so the two maps are each other's latency hiding.  320 threads:
//   warp 0      TMA producer: Q of both maps once, then per tile of 128 keys K of both maps and V (128-byte swizzle)
//   warp 1      one thread issues all MMAs: S_m = Q_m K_m^T (128 x 128, float32 in tensor memory), O_m += P_m V with P_m read
//               from tensor memory (it overwrites S_m) and V as stored, value index contiguous
//   warps 2-9   two softmax warpgroups, one per map, a thread per query row.  Weights stay 32-bit in effect: each is split into
//               two bfloat16 terms (high + remainder, 16 significant bits) and both are multiplied with V.  The running maximum
//               is only raised when it has grown by more than 2^8, so O is rarely rescaled.
// Tensor memory: S_0, S_1 (128 columns each), O_0, O_1 (up to 128 each).  At the end each warpgroup forms half of the value
// columns of a1 - lambda a2, the row's root mean square is completed through shared memory, and the result leaves as bfloat16.
// Every mbarrier wait is bounded (status word codes 31..36).
#include "mix_tc.cuh"

namespace scmx {

struct TcAttnArgs {
    int n, H, G, d, dv;
    int64_t pos;             // position of query row 0
    float scale_log2, lambda, out_scale, eps;
    bf16_t* o;               // [n, H dv]
    int32_t* status;
    uint64_t wait_ns;
};

constexpr int TA_THREADS = 320;
constexpr int TA_TILE = 128 * 128;       // bytes of a [128 rows x 64 values] operand block

template <int KB, int VB, int KS>
struct TaSmem {
    static constexpr int VS = 2;
    static constexpr int Q_OFF = 0;
    static constexpr int K_OFF = Q_OFF + 2 * KB * TA_TILE;
    static constexpr int V_OFF = K_OFF + KS * 2 * KB * TA_TILE;
    static constexpr int BAR_OFF = V_OFF + VS * VB * TA_TILE;
    // qfull, kfull[KS], kempty[KS], vfull[VS], vempty[VS], sfull[2], pfull[2], ofull
    static constexpr int NBAR = 1 + 2 * KS + 2 * VS + 5;
    static constexpr int MISC_OFF = BAR_OFF + 8 * NBAR;
    static constexpr int ROW_OFF = (MISC_OFF + 16 + 15) & ~15;       // float [2][128] sums, [2][128] squares
    static constexpr int TOTAL = ROW_OFF + 4 * 128 * 4 + 1024;
};

__device__ __forceinline__ void softmax_bar() { asm volatile("bar.sync 2, 256;" ::: "memory"); }

template <int KB, int VB, int KS>
__global__ void __launch_bounds__(TA_THREADS, 1) diff_attn_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                                                              const __grid_constant__ CUtensorMap tmV, const TcAttnArgs a) {
    using L = TaSmem<KB, VB, KS>;
    constexpr int VS = L::VS;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    const uint32_t sbase = smem_u32(smem), bars = sbase + L::BAR_OFF;
    const uint32_t b_q = bars, b_kf = b_q + 8, b_ke = b_kf + 8 * KS, b_vf = b_ke + 8 * KS, b_ve = b_vf + 8 * VS, b_s = b_ve + 8 * VS,
                   b_p = b_s + 16, b_o = b_p + 16;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + L::MISC_OFF);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + L::MISC_OFF + 4);
    float* s_row = reinterpret_cast<float*>(smem + L::ROW_OFF);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    if (threadIdx.x == 0) {
        for (const CUtensorMap* m : {&tmQ, &tmK, &tmV}) prefetch_map(m);
        for (int i = 0; i < L::NBAR; ++i) {
            const uint32_t b = bars + 8 * i;
            mbar_init(b, b == b_p || b == b_p + 8 ? 4 : 1);      // b_p: one arrival per softmax warp of the map
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

    const int nqt = (a.n + 127) / 128;
    const int h = blockIdx.x % a.H, qt = nqt - 1 - blockIdx.x / a.H;       // long rows first
    const int g = h / (a.H / a.G), q0 = qt * 128, rows = min(128, a.n - q0);
    const int64_t p0 = a.pos + q0;
    const int nkt = (int)((p0 + rows + 127) / 128);
    int fail = 0;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(b_q, 2 * KB * TA_TILE);
            for (int m = 0; m < 2; ++m)
                for (int c = 0; c < KB; ++c) tma_load_3d(sbase + L::Q_OFF + (m * KB + c) * TA_TILE, &tmQ, c * 128, q0, 2 * h + m, b_q);
            for (int j = 0; j < nkt; ++j) {
                const int ks = j % KS, vs = j % VS;
                if (int w = mbar_wait(b_ke + 8 * ks, ((j / KS) & 1) ^ 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 31 : -1; break; }
                mbar_expect_tx(b_kf + 8 * ks, 2 * KB * TA_TILE);
                for (int m = 0; m < 2; ++m)
                    for (int c = 0; c < KB; ++c)
                        tma_load_3d(sbase + L::K_OFF + ((ks * 2 + m) * KB + c) * TA_TILE, &tmK, c * 128, j * 128, 2 * g + m, b_kf + 8 * ks);
                if (int w = mbar_wait(b_ve + 8 * vs, ((j / VS) & 1) ^ 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 32 : -1; break; }
                mbar_expect_tx(b_vf + 8 * vs, VB * TA_TILE);
                for (int c = 0; c < VB; ++c) tma_load_3d(sbase + L::V_OFF + (vs * VB + c) * TA_TILE, &tmV, c * 128, j * 128, g, b_vf + 8 * vs);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_s = umma_idesc_bf16(128, 128);
            const uint32_t idesc_o = umma_idesc_bf16(128, (a.dv + 15) & ~15) | IDESC_B_MN;
            const int dsteps = (a.d + 15) / 16;
            auto scores = [&](int m, int ks) {
                for (int k = 0; k < dsteps; ++k) {
                    const uint32_t o = (k >> 2) * TA_TILE;
                    const uint64_t da = umma_desc(sbase + L::Q_OFF + m * KB * TA_TILE + o), db = umma_desc(sbase + L::K_OFF + (ks * 2 + m) * KB * TA_TILE + o);
                    umma_bf16(tmem + 128 * m, da + 2 * (k & 3), db + 2 * (k & 3), idesc_s, k > 0);
                }
                umma_commit(b_s + 8 * m);
            };
            do {
                if (int w = mbar_wait(b_q, 0, abort_flag, a.wait_ns)) { fail = w == 1 ? 33 : -1; break; }
                if (int w = mbar_wait(b_kf, 0, abort_flag, a.wait_ns)) { fail = w == 1 ? 33 : -1; break; }
                tc_fence_after();
                scores(0, 0);
                scores(1, 0);
                umma_commit(b_ke);
                for (int j = 0; j < nkt && fail == 0; ++j) {
                    const int vs = j % VS, kn = (j + 1) % KS;
                    for (int m = 0; m < 2; ++m) {
                        if (int w = mbar_wait(b_p + 8 * m, j & 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 34 : -1; break; }
                        if (m == 0)
                            if (int w = mbar_wait(b_vf + 8 * vs, (j / VS) & 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 33 : -1; break; }
                        tc_fence_after();
                        const uint64_t dv = umma_desc_mn(sbase + L::V_OFF + vs * VB * TA_TILE, TA_TILE);
#pragma unroll
                        for (int k = 0; k < 8; ++k) {       // 16 keys: high and remainder terms, 8 columns each
                            const uint32_t pa = tmem + 128 * m + (k >> 1) * 32 + (k & 1) * 8;
                            umma_bf16_ts(tmem + 256 + 128 * m, pa, dv + 128 * k, idesc_o, (j | k) != 0);
                            umma_bf16_ts(tmem + 256 + 128 * m, pa + 16, dv + 128 * k, idesc_o, 1);
                        }
                        if (j + 1 < nkt) {
                            if (m == 0)
                                if (int w = mbar_wait(b_kf + 8 * kn, ((j + 1) / KS) & 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 33 : -1; break; }
                            tc_fence_after();
                            scores(m, kn);
                            if (m == 1) umma_commit(b_ke + 8 * kn);
                        }
                        if (m == 1) umma_commit(b_ve + 8 * vs);
                    }
                }
                if (fail == 0) umma_commit(b_o);
            } while (false);
        }
    } else {
        const int m = (warp - 2) >> 2, q = warp & 3, row = 32 * q + lane;
        const uint32_t lane_base = (uint32_t)(32 * q) << 16, ts = tmem + 128 * m + lane_base, to = tmem + 256 + 128 * m + lane_base;
        const int dv_chunks = (a.dv + 31) / 32;
        float mx = 0.0f, sum = 0.0f;
        for (int j = 0; j < nkt; ++j) {
            int w = mbar_wait(b_s + 8 * m, j & 1, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) { fail = w == 1 ? 35 : -1; break; }
            tc_fence_after();
            const int64_t lim64 = p0 + row - (int64_t)j * 128 + 1;       // keys of this tile that the row sees
            const int lim = lim64 > 128 ? 128 : (int)lim64;
            const bool edge = __any_sync(0xffffffffu, lim < 128);
            // first pass over the scores: the maximum
            uint32_t r[2][32];
            float tm = -INFINITY;
            tmem_ld32(ts, r[0]);
            tmem_ld_fence(r[0]);
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                uint32_t(&v)[32] = r[c & 1];
                if (c < 3) tmem_ld32(ts + 32 * (c + 1), r[(c + 1) & 1]);
                if (edge) {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (32 * c + i >= lim) v[i] = 0xFF800000u;
                }
                float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
                for (int i = 0; i < 32; i += 4) {
                    t0 = fmaxf(t0, fmaxf(__uint_as_float(v[i]), __uint_as_float(v[i + 1])));
                    t1 = fmaxf(t1, fmaxf(__uint_as_float(v[i + 2]), __uint_as_float(v[i + 3])));
                }
                tm = fmaxf(tm, fmaxf(t0, t1));
                if (c < 3) tmem_ld_fence(r[(c + 1) & 1]);
            }
            if (j == 0) {
                mx = tm;                 // finite: every row sees key 0
            } else {
                const bool grow = (tm - mx) * a.scale_log2 > 8.0f;
                if (__any_sync(0xffffffffu, grow)) {
                    // S_m(j) complete implies O_m of the previous tile complete: MMAs of one thread finish in order
                    const float mn = grow ? tm : mx, f = ex2_approx((mx - mn) * a.scale_log2);
                    mx = mn;
                    sum *= f;
                    for (int c = 0; c < dv_chunks; ++c) {
                        uint32_t v[32];
                        tmem_ld32(to + 32 * c, v);
                        tmem_ld_fence(v);
#pragma unroll
                        for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * f);
                        tmem_st32(to + 32 * c, v);
                    }
                }
            }
            // second pass: weights, their two bfloat16 terms in place of the chunk's scores
            const float off = -mx * a.scale_log2;
            float s0 = 0.0f, s1 = 0.0f;
            tmem_ld32(ts, r[0]);
            tmem_ld_fence(r[0]);
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                uint32_t(&v)[32] = r[c & 1];
                if (c < 3) tmem_ld32(ts + 32 * (c + 1), r[(c + 1) & 1]);
                if (edge) {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (32 * c + i >= lim) v[i] = 0xFF800000u;
                }
                uint32_t pk[32];
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float x0 = ex2_approx(fmaf(__uint_as_float(v[2 * i]), a.scale_log2, off));
                    const float x1 = ex2_approx(fmaf(__uint_as_float(v[2 * i + 1]), a.scale_log2, off));
                    s0 += x0;
                    s1 += x1;
                    const uint32_t hi = pack_bf16x2(x0, x1);
                    pk[i] = hi;
                    pk[16 + i] = pack_bf16x2(x0 - bf16_lo(hi), x1 - bf16_hi(hi));
                }
                if (c < 3) tmem_ld_fence(r[(c + 1) & 1]);
                tmem_st32(ts + 32 * c, pk);
            }
            sum += s0 + s1;
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(b_p + 8 * m);
        }
        if (fail == 0) {
            int w = mbar_wait(b_o, 0, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) fail = w == 1 ? 36 : -1;
        }
        // the 256 threads meet twice whatever happened
        s_row[m * 128 + row] = sum;
        softmax_bar();
        const bool ok = *abort_flag == 0 && fail == 0;      // uniform over the warp
        float x[VB * 32], ss = 0.0f;
        if (ok) {
            tc_fence_after();
            const float i1 = 1.0f / s_row[row], i2 = a.lambda / s_row[128 + row];
            const uint32_t t1 = tmem + 256 + lane_base, t2 = t1 + 128;
#pragma unroll
            for (int c = 0; c < VB; ++c) {
                const int col = (m * VB + c) * 32;
                uint32_t u[32], v[32];
                tmem_ld32(t1 + col, u);
                tmem_ld32(t2 + col, v);
                tmem_ld_fence(u);
                tmem_ld_fence(v);
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    x[c * 32 + i] = col + i < a.dv ? __uint_as_float(u[i]) * i1 - __uint_as_float(v[i]) * i2 : 0.0f;
                    ss += x[c * 32 + i] * x[c * 32 + i];
                }
            }
            s_row[256 + m * 128 + row] = ss;
        }
        softmax_bar();
        if (ok && row < rows) {
            const float inv = rms_inv_f32(s_row[256 + row] + s_row[384 + row], a.dv, a.eps) * a.out_scale;
            bf16_t* o = a.o + ((int64_t)(q0 + row) * a.H + h) * a.dv;
#pragma unroll
            for (int c = 0; c < VB; ++c)
#pragma unroll
                for (int i = 0; i < 32; i += 8) {
                    const int col = (m * VB + c) * 32 + i;
                    if (col < a.dv) {
                        const float* y = x + c * 32 + i;
                        *reinterpret_cast<uint4*>(o + col) = make_uint4(pack_bf16x2(y[0] * inv, y[1] * inv), pack_bf16x2(y[2] * inv, y[3] * inv),
                                                                        pack_bf16x2(y[4] * inv, y[5] * inv), pack_bf16x2(y[6] * inv, y[7] * inv));
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
        const uint64_t t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);   // 0.2 ms for outstanding TMA writes
        __syncthreads();
    }
    if (warp == 1) tmem_dealloc(tmem, 512);
}

template <int KB, int VB, int KS>
static int launch_tc(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, const TcAttnArgs& a, cudaStream_t st) {
    using L = TaSmem<KB, VB, KS>;
    static bool configured[64] = {};
    const int dev = current_device();
    SCMX_REQUIRE(dev >= 0, SCMX_ECUDA, "no current CUDA device (ordinal 0..63)");
    if (!configured[dev]) {
        SCMX_CUDA_OK(cudaFuncSetAttribute(diff_attn_tc_kernel<KB, VB, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL));
        configured[dev] = true;
    }
    const unsigned grid = (unsigned)((a.n + 127) / 128) * a.H;
    SCMX_PDL_OK("diff_attn_tc_kernel", launch_pdl(diff_attn_tc_kernel<KB, VB, KS>, dim3(grid), dim3(TA_THREADS), (size_t)L::TOTAL, st, q, k, v, a));
    return SCMX_OK;
}

bool diff_attn_tc_supported(int64_t n, int64_t pos, int d, int dv, float scale) {
    return d % 8 == 0 && dv % 8 == 0 && d <= 128 && dv <= 128 && scale > 0.0f && pos + n < (1ll << 30);
}

int diff_attn_tc(const bf16_t* q, const bf16_t* kc, const bf16_t* vc, int64_t n, int64_t pos, int64_t cap, int H, int G, int d, int dv, float scale,
                 float lambda, float diff, float eps, bf16_t* o, int32_t* status, cudaStream_t st) {
    TcAttnArgs a;
    a.n = (int)n; a.H = H; a.G = G; a.d = d; a.dv = dv; a.pos = pos; a.scale_log2 = scale * 1.4426950408889634f; a.lambda = lambda;
    a.out_scale = 1.0f - diff; a.eps = eps; a.o = o; a.status = status; a.wait_ns = g_wait_limit_ns;
    CUtensorMap tq, tk, tv;
    // keys and values end at the last filled row: later rows of the cache are read as zeros
    int rc = make_map_planes(&tq, q, 2 * H, n, 2 * d, 2 * d, 2 * n * d, 128);
    if (!rc) rc = make_map_planes(&tk, kc, 2 * G, pos + n, 2 * d, 2 * d, 2 * cap * d, 128);
    if (!rc) rc = make_map_planes(&tv, vc, G, pos + n, 2 * dv, 2 * dv, 2 * cap * dv, 128);
    if (rc) return rc;
    if (d <= 64) return dv <= 64 ? launch_tc<1, 1, 2>(tq, tk, tv, a, st) : launch_tc<1, 2, 2>(tq, tk, tv, a, st);
    return dv <= 64 ? launch_tc<2, 1, 1>(tq, tk, tv, a, st) : launch_tc<2, 2, 1>(tq, tk, tv, a, st);
}

}  // namespace scmx
