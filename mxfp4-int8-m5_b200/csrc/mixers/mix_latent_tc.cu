// Attention of prompt portions on tcgen05 with a shared rotated key part and a sliding window (bfloat16; head sizes d, dv up to 128,
// rotated part up to 64, multiples of 8): score = (q . k_h + q_rot . k_rot) scale, position i sees j with 0 <= i - j < window.
//
// A CTA owns two tiles of 128 query rows of one head; they share the key and value tiles, and while the tensor core works on one
// tile the other tile's softmax runs.  320 threads:
//   warp 0      TMA producer: both query tiles once, then per tile of 128 keys the head's keys, the shared part and the values
//   warp 1      all MMAs (the warp stays converged, one lane issues): S_m = Q_m K^T (128 x 128, float32 in tensor memory), O_m += P_m V with P_m read from
//               tensor memory (it overwrites S_m)
//   warps 2-9   two softmax warpgroups, one per query tile, a thread per row.  Weights are split into two bfloat16 terms (16
//               significant bits); the running maximum is only raised when it has grown by more than 2^8
// Each query tile has its own range of key tiles (window and diagonal); tiles outside it are skipped for that tile only.
// Every mbarrier wait is bounded (status word codes 51..56).
#include "mix_tc.cuh"

namespace scmx {

struct LaArgs {
    int n, H, d, r, dv;
    int64_t pos, k0, window;     // position of query row 0, of key row 0; window 0: none
    float scale_log2;
    bf16_t* o;                   // [n, H dv]
    int32_t* status;
    uint64_t wait_ns;
};

constexpr int LA_THREADS = 320;
constexpr int LA_TILE = 128 * 128;       // bytes of a [128 rows x 64 values] operand block

template <int KB, int VB>
struct LaSmem {
    static constexpr int KS = KB == 3 ? 1 : 2, VS = 2;
    static constexpr int Q_OFF = 0;
    static constexpr int K_OFF = Q_OFF + 2 * KB * LA_TILE;
    static constexpr int V_OFF = K_OFF + KS * KB * LA_TILE;
    static constexpr int BAR_OFF = V_OFF + VS * VB * LA_TILE;
    // qfull, kfull[KS], kempty[KS], vfull[VS], vempty[VS], sfull[2], pfull[2], ofull[2]
    static constexpr int NBAR = 1 + 2 * KS + 2 * VS + 6;
    static constexpr int MISC_OFF = BAR_OFF + 8 * NBAR;
    static constexpr int TOTAL = MISC_OFF + 16 + 1024;
};

// DU blocks of 64 for the heads' own part, RB (0 or 1) for the shared rotated part, VB for the values.
template <int DU, int RB, int VB>
__global__ void __launch_bounds__(LA_THREADS, 1)
    latent_attn_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmQr, const __grid_constant__ CUtensorMap tmK,
                          const __grid_constant__ CUtensorMap tmKr, const __grid_constant__ CUtensorMap tmV, const LaArgs a) {
    constexpr int KB = DU + RB;
    using L = LaSmem<KB, VB>;
    constexpr int KS = L::KS, VS = L::VS;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    const uint32_t sbase = smem_u32(smem), bars = sbase + L::BAR_OFF;
    const uint32_t b_q = bars, b_kf = b_q + 8, b_ke = b_kf + 8 * KS, b_vf = b_ke + 8 * KS, b_ve = b_vf + 8 * VS, b_s = b_ve + 8 * VS, b_p = b_s + 16,
                   b_o = b_p + 16;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + L::MISC_OFF);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + L::MISC_OFF + 4);
    const int warp = __shfl_sync(0xffffffffu, (int)(threadIdx.x >> 5), 0), lane = threadIdx.x & 31;

    if (threadIdx.x == 0) {
        for (const CUtensorMap* m : {&tmQ, &tmQr, &tmK, &tmKr, &tmV}) prefetch_map(m);
        for (int i = 0; i < L::NBAR; ++i) {
            const uint32_t b = bars + 8 * i;
            mbar_init(b, b == b_p || b == b_p + 8 ? 4 : 1);      // b_p: one arrival per softmax warp of the query tile
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

    const int npair = (a.n + 255) / 256;
    const int h = blockIdx.x % a.H, q0 = 256 * (npair - 1 - blockIdx.x / a.H);       // long rows first
    // key tiles [lo[m], hi[m]) of the two query tiles; an absent second tile has none
    int lo[2], hi[2];
#pragma unroll
    for (int m = 0; m < 2; ++m) {
        const int r0 = q0 + 128 * m, r1 = min(a.n, r0 + 128);
        const int64_t first = a.window > 0 && a.pos + r0 + 1 > a.window ? a.pos + r0 + 1 - a.window : 0;
        lo[m] = first > a.k0 ? (int)((first - a.k0) / 128) : 0;
        hi[m] = r1 > r0 ? (int)((a.pos + r1 - 1 - a.k0) / 128) + 1 : lo[m];
    }
    const int jlo = lo[0], jhi = hi[1] > hi[0] ? hi[1] : hi[0];
    int fail = 0;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(b_q, 2 * KB * LA_TILE);
            for (int m = 0; m < 2; ++m) {
                for (int c = 0; c < DU; ++c) tma_load_3d(sbase + L::Q_OFF + (m * KB + c) * LA_TILE, &tmQ, c * 128, q0 + 128 * m, h, b_q);
                if (RB) tma_load_3d(sbase + L::Q_OFF + (m * KB + DU) * LA_TILE, &tmQr, 0, q0 + 128 * m, h, b_q);
            }
            for (int j = jlo; j < jhi; ++j) {
                const int i = j - jlo, ks = i % KS, vs = i % VS;
                if (int w = mbar_wait(b_ke + 8 * ks, ((i / KS) & 1) ^ 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 51 : -1; break; }
                mbar_expect_tx(b_kf + 8 * ks, KB * LA_TILE);
                for (int c = 0; c < DU; ++c) tma_load_3d(sbase + L::K_OFF + (ks * KB + c) * LA_TILE, &tmK, c * 128, j * 128, h, b_kf + 8 * ks);
                if (RB) tma_load_3d(sbase + L::K_OFF + (ks * KB + DU) * LA_TILE, &tmKr, 0, j * 128, 0, b_kf + 8 * ks);
                if (int w = mbar_wait(b_ve + 8 * vs, ((i / VS) & 1) ^ 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 52 : -1; break; }
                mbar_expect_tx(b_vf + 8 * vs, VB * LA_TILE);
                for (int c = 0; c < VB; ++c) tma_load_3d(sbase + L::V_OFF + (vs * VB + c) * LA_TILE, &tmV, c * 128, j * 128, h, b_vf + 8 * vs);
            }
        }
    } else if (warp == 1) {
        // the whole warp walks through the tiles; `on` is the lane that issues
        const uint32_t on = elect_lane();
        const uint32_t idesc_s = umma_idesc_bf16(128, 128);
        const uint32_t idesc_o = umma_idesc_bf16(128, (a.dv + 15) & ~15) | IDESC_B_MN;
        const int dsteps = (a.d + 15) / 16, rsteps = RB ? (a.r + 15) / 16 : 0;
        auto wait = [&](uint32_t bar, uint32_t parity, int code) -> bool {
            const int w = mbar_wait(bar, parity, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) { fail = w == 1 ? code : -1; return false; }
            tc_fence_after();
            return true;
        };
        auto scores = [&](int m, int ks) {
            const uint32_t d = tmem + 128 * m;
            uint32_t acc = 0;
#pragma unroll
            for (int c = 0; c < KB; ++c) {
                const uint64_t da = umma_desc(sbase + L::Q_OFF + (m * KB + c) * LA_TILE), db = umma_desc(sbase + L::K_OFF + (ks * KB + c) * LA_TILE);
                const int steps = c < DU ? dsteps - 4 * c : rsteps;
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    if (k < steps) {
                        umma_bf16_on(on, d, da + 2 * k, db + 2 * k, idesc_s, acc);
                        acc = 1;
                    }
            }
            umma_commit_on(on, b_s + 8 * m);
        };
        bool ok = wait(b_q, 0, 53) && wait(b_kf, 0, 53);
        if (ok) {
#pragma unroll
            for (int m = 0; m < 2; ++m)
                if (jlo >= lo[m] && jlo < hi[m]) scores(m, 0);
            umma_commit_on(on, b_ke);
        }
        for (int j = jlo; j < jhi && ok; ++j) {
            const int i = j - jlo, vs = i % VS, kn = (i + 1) % KS;
#pragma unroll
            for (int m = 0; m < 2; ++m) {
                const bool now = j >= lo[m] && j < hi[m];
                if (now && !(ok = wait(b_p + 8 * m, (j - lo[m]) & 1, 54))) break;
                if (m == 0 && !(ok = wait(b_vf + 8 * vs, (i / VS) & 1, 53))) break;
                if (now) {
                    const uint64_t dv = umma_desc_mn(sbase + L::V_OFF + vs * VB * LA_TILE, LA_TILE);
#pragma unroll
                    for (int k = 0; k < 8; ++k) {       // 16 keys: high and remainder terms, 8 columns each
                        const uint32_t pa = tmem + 128 * m + (k >> 1) * 32 + (k & 1) * 8;
                        umma_bf16_ts_on(on, tmem + 256 + 128 * m, pa, dv + 128 * k, idesc_o, k > 0 ? 1u : (uint32_t)(j > lo[m]));
                        umma_bf16_ts_on(on, tmem + 256 + 128 * m, pa + 16, dv + 128 * k, idesc_o, 1);
                    }
                    if (j + 1 == hi[m]) umma_commit_on(on, b_o + 8 * m);
                }
                if (j + 1 < jhi) {
                    if (m == 0 && !(ok = wait(b_kf + 8 * kn, ((i + 1) / KS) & 1, 53))) break;
                    if (j + 1 >= lo[m] && j + 1 < hi[m]) scores(m, kn);
                    if (m == 1) umma_commit_on(on, b_ke + 8 * kn);
                }
                if (m == 1) umma_commit_on(on, b_ve + 8 * vs);
            }
        }
        if (!on) fail = fail > 0 ? -1 : fail;      // one lane reports
    } else {
        const int m = (warp - 2) >> 2, q = warp & 3, row = 32 * q + lane;
        const uint32_t lane_base = (uint32_t)(32 * q) << 16, ts = tmem + 128 * m + lane_base, to = tmem + 256 + 128 * m + lane_base;
        const int dv_chunks = (a.dv + 31) / 32, mlo = m == 0 ? lo[0] : lo[1], mhi = m == 0 ? hi[0] : hi[1];
        const int64_t p = a.pos + q0 + 128 * m + row - a.k0;         // the row's own key
        const int64_t back = a.window > 0 ? p - a.window + 1 : -1;   // its first key (may be negative)
        float mx = -1e30f, sum = 0.0f;
        for (int j = mlo; j < mhi; ++j) {
            int w = mbar_wait(b_s + 8 * m, (j - mlo) & 1, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) { fail = w == 1 ? 55 : -1; break; }
            tc_fence_after();
            const int64_t up = p - (int64_t)j * 128 + 1, down = back - (int64_t)j * 128;      // this tile's keys down <= . < up
            const int lim = up > 128 ? 128 : (int)up, from = down < 0 ? 0 : down > 128 ? 128 : (int)down;
            const bool edge = __any_sync(0xffffffffu, lim < 128 || from > 0);
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
                        if (32 * c + i >= lim || 32 * c + i < from) v[i] = 0xFF800000u;
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
            // a row may see none of a tile's keys: its maximum stays at -1e30 and its weights are zero
            if (j == mlo) {
                mx = fmaxf(mx, tm);
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
                        if (32 * c + i >= lim || 32 * c + i < from) v[i] = 0xFF800000u;
                }
                uint32_t pk[32];
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float x0 = ex2_approx(fmaf(__uint_as_float(v[2 * i]), a.scale_log2, off));
                    const float x1 = ex2_approx(fmaf(__uint_as_float(v[2 * i + 1]), a.scale_log2, off));
                    s0 += x0;
                    s1 += x1;
                    const uint32_t hw = pack_bf16x2(x0, x1);
                    pk[i] = hw;
                    pk[16 + i] = pack_bf16x2(x0 - bf16_lo(hw), x1 - bf16_hi(hw));
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
        if (fail == 0 && mhi > mlo) {
            int w = mbar_wait(b_o + 8 * m, 0, abort_flag, a.wait_ns);
            if (__any_sync(0xffffffffu, w)) {
                fail = w == 1 ? 56 : -1;
            } else {
                tc_fence_after();
                const float inv = 1.0f / sum;
                const int qr = q0 + 128 * m + row;
                bf16_t* o = a.o + ((int64_t)qr * a.H + h) * a.dv;
#pragma unroll
                for (int c = 0; c < 2 * VB; ++c) {
                    uint32_t v[32];
                    if (32 * c >= a.dv) break;
                    tmem_ld32(to + 32 * c, v);
                    tmem_ld_fence(v);
                    if (qr < a.n)
#pragma unroll
                        for (int i = 0; i < 32; i += 8)
                            if (32 * c + i < a.dv) {
                                uint32_t pk[4];
#pragma unroll
                                for (int e = 0; e < 4; ++e) pk[e] = pack_bf16x2(__uint_as_float(v[i + 2 * e]) * inv, __uint_as_float(v[i + 2 * e + 1]) * inv);
                                *reinterpret_cast<uint4*>(o + 32 * c + i) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
                            }
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

template <int DU, int RB, int VB>
static int launch_la(const CUtensorMap (&m)[5], const LaArgs& a, cudaStream_t st) {
    using L = LaSmem<DU + RB, VB>;
    static bool configured[64] = {};
    const int dev = current_device();
    SCMX_REQUIRE(dev >= 0, SCMX_ECUDA, "no current CUDA device (ordinal 0..63)");
    if (!configured[dev]) {
        SCMX_CUDA_OK(cudaFuncSetAttribute(latent_attn_tc_kernel<DU, RB, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL));
        configured[dev] = true;
    }
    const unsigned grid = (unsigned)((a.n + 255) / 256) * a.H;
    SCMX_PDL_OK("latent_attn_tc_kernel", launch_pdl(latent_attn_tc_kernel<DU, RB, VB>, dim3(grid), dim3(LA_THREADS), (size_t)L::TOTAL, st, m[0], m[1], m[2],
                                                    m[3], m[4], a));
    return SCMX_OK;
}

bool latent_attn_tc_supported(int64_t n, int64_t pos, int d, int r, int dv, float scale) {
    return d > 0 && dv > 0 && r >= 0 && d % 8 == 0 && r % 8 == 0 && dv % 8 == 0 && d <= 128 && r <= 64 && dv <= 128 && scale > 0.0f && pos + n < (1ll << 30);
}

int latent_attn_tc(const bf16_t* q, int64_t ldq, const bf16_t* kv, int64_t ldkv, const bf16_t* rot, int64_t ldrot, int64_t n, int64_t pos, int64_t k0,
                   int64_t window, int H, int d, int r, int dv, float scale, bf16_t* o, int32_t* status, cudaStream_t st) {
    LaArgs a;
    a.n = (int)n; a.H = H; a.d = d; a.r = r; a.dv = dv; a.pos = pos; a.k0 = k0; a.window = window; a.scale_log2 = scale * 1.4426950408889634f; a.o = o;
    a.status = status; a.wait_ns = g_wait_limit_ns;
    const int64_t nk = pos + n - k0;          // rows past the last key are read as zeros
    CUtensorMap m[5];
    int rc = make_map_planes(&m[0], q, H, n, 2 * d, 2 * ldq, 2ll * (d + r), 128);
    if (!rc) rc = make_map_planes(&m[1], r ? q + d : q, H, n, 2 * (r ? r : d), 2 * ldq, 2ll * (d + r), 128);
    if (!rc) rc = make_map_planes(&m[2], kv, H, nk, 2 * d, 2 * ldkv, 2 * d, 128);
    if (!rc) rc = make_map_planes(&m[3], r ? rot : kv, 1, nk, 2 * (r ? r : d), 2 * (r ? ldrot : ldkv), 2 * (r ? ldrot : ldkv) * nk, 128);
    if (!rc) rc = make_map_planes(&m[4], kv + (int64_t)H * d, H, nk, 2 * dv, 2 * ldkv, 2 * dv, 128);
    if (rc) return rc;
#define GO(DU)                                                                                                            \
    do {                                                                                                                   \
        if (r == 0) return dv <= 64 ? launch_la<DU, 0, 1>(m, a, st) : launch_la<DU, 0, 2>(m, a, st);                       \
        return dv <= 64 ? launch_la<DU, 1, 1>(m, a, st) : launch_la<DU, 1, 2>(m, a, st);                                   \
    } while (0)
    if (d <= 64) GO(1);
    GO(2);
#undef GO
}

}  // namespace scmx
