// bfloat16 GEMM with float32 accumulation, out = A [M, K] . W [N, K]^T, on tcgen05.mma kind::f16.  Same structure as the INT8
// GEMM (TMA producer warp, one MMA-issuing thread, 8 epilogue warps, two accumulators in tensor memory, persistent tiles): a K
// block is 128 bytes = 64 values, so the stages, swizzle and descriptors are the INT8 kernel's.  Large shapes run on CTA pairs
// (256 x 256 tiles), others on single CTAs (128 x BN tiles).
// Epilogue: float32 or bfloat16 output, optionally through xIELU or the gated GELU.  Rows of the output are padded to a multiple of 16 bytes.
#include "mix_tc.cuh"

namespace scmx {

struct BgArgs {
    int M, N, K;
    int out_f32;                 // 1: float output, 0: bfloat16
    int act;                     // 0: none, 1: xIELU, 2: gelu(gate) up, columns alternate 16 gate and 16 up
    float a_pos, a_neg;          // xIELU: softplus(p), 1/2 + softplus(q)
    void* out;
    int64_t ldo;                 // elements
    int splits;                  // > 1: K is cut into this many ranges; range s goes to out + s * split_stride (float32, no activation)
    int64_t split_stride;        // elements
    int32_t* status;
    uint64_t wait_ns;
};

// Staged 32 rows x 128 bytes -> global memory, full lines, 4 rows per instruction; `valid` bytes of the unit (a multiple of 16).
__device__ __forceinline__ void bg_drain(const BgArgs& a, uint8_t* out, const uint8_t* stg, int lane, int row0, size_t row_bytes, size_t col_byte0, int valid) {
    const int piece = lane & 7, rsub = lane >> 3;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int rl = 4 * i + rsub, row = row0 + rl;
        const uint4 v = *reinterpret_cast<const uint4*>(stg + rl * EPI_PITCH + piece * 16);
        if (row < a.M && piece * 16 < valid)
            *reinterpret_cast<uint4*>(out + (size_t)row * row_bytes + col_byte0 + piece * 16) = v;
    }
}

// One warp's 32 rows x BN/2 accumulator columns (see epilogue_warp of the INT8 kernel for the staging layout).
// A 32-column chunk leaves as 32 values, or as 16 with the gated activation (16 gate columns, 16 up columns).  Chunks are staged
// until 128 bytes of a row are full.
template <int BN>
__device__ __forceinline__ void bg_epilogue(const BgArgs& a, uint8_t* out, uint32_t taddr, int row0, int n0, uint8_t* stg, int lane) {
    constexpr int CHUNKS = BN / 64;           // 32-column chunks
    uint8_t* my = stg + lane * EPI_PITCH;
    const int esz = a.out_f32 ? 4 : 2, cols = a.act == 2 ? 16 : 32, bytes = cols * esz, unit = 128 / bytes;
    const size_t row_bytes = (size_t)a.ldo * esz;
    const int nout = a.act == 2 ? a.N / 2 : a.N, npad = a.out_f32 ? (nout + 3) & ~3 : (nout + 7) & ~7;
    const int c0 = a.act == 2 ? n0 / 2 : n0;
    uint32_t r[2][32];
    tmem_ld32(taddr, r[0]);
    tmem_ld_fence(r[0]);
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        uint32_t(&v)[32] = r[c & 1];
        if (c + 1 < CHUNKS) tmem_ld32(taddr + (c + 1) * 32, r[(c + 1) & 1]);
        if (a.act == 1) {
#pragma unroll
            for (int j = 0; j < 32; ++j) v[j] = __float_as_uint(xielu_f32(__uint_as_float(v[j]), a.a_pos, a.a_neg));
        } else if (a.act == 2) {
#pragma unroll
            for (int j = 0; j < 16; ++j) v[j] = __float_as_uint(gelu_tanh_f32(__uint_as_float(v[j])) * __uint_as_float(v[16 + j]));
        }
        const int k = c & (unit - 1);
        uint4* o = reinterpret_cast<uint4*>(my + bytes * k);
        if (a.out_f32) {
#pragma unroll
            for (int j = 0; j < 8; ++j)
                if (4 * j < cols) o[j] = make_uint4(v[4 * j], v[4 * j + 1], v[4 * j + 2], v[4 * j + 3]);
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (8 * j < cols) {
                    uint32_t pk[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i) pk[i] = pack_bf16x2(__uint_as_float(v[8 * j + 2 * i]), __uint_as_float(v[8 * j + 2 * i + 1]));
                    o[j] = make_uint4(pk[0], pk[1], pk[2], pk[3]);
                }
        }
        if (k == unit - 1 || c + 1 == CHUNKS) {
            __syncwarp();
            const int col = c0 + (c - k) * cols;
            bg_drain(a, out, stg, lane, row0, row_bytes, (size_t)col * esz, min((k + 1) * bytes, (npad - col) * esz));
            __syncwarp();
        }
        if (c + 1 < CHUNKS) tmem_ld_fence(r[(c + 1) & 1]);
    }
}

template <int BN_, int STAGES_, bool PAIR>
struct BgSmem {
    static constexpr int BN = BN_, STAGES = STAGES_;
    static constexpr int A_BYTES = BM * BK;
    static constexpr int B_BYTES = (PAIR ? BN / 2 : BN) * BK;
    static constexpr int STAGE_BYTES = A_BYTES + B_BYTES;
    static constexpr int BAR_OFF = STAGES * STAGE_BYTES;
    static constexpr int MISC_OFF = BAR_OFF + 8 * (2 * STAGES + 4);
    static constexpr int EPI_OFF = (MISC_OFF + 16 + 127) & ~127;
    static constexpr int TOTAL = EPI_OFF + EPI_STAGE_BYTES + 1024;
};

// PAIR = false: one CTA per 128 x BN tile.  PAIR = true: launched as clusters of 2, 256 x BN tile, each CTA loads its 128 rows of
// A and its BN/2 weight rows (plain TMA loads), the leader issues the MMAs; barriers as in gemm_i8_pair_kernel.
template <int BN, int STAGES, bool PAIR>
__device__ __forceinline__ void gemm_bf16_body(const CUtensorMap& tmA, const CUtensorMap& tmB, const BgArgs& a) {
    using L = BgSmem<BN, STAGES, PAIR>;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    const uint32_t sbase = smem_u32(smem);
    const uint32_t bar_full = sbase + L::BAR_OFF, bar_empty = bar_full + 8 * STAGES;
    const uint32_t bar_tfull = bar_empty + 8 * STAGES, bar_tempty = bar_tfull + 16;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + L::MISC_OFF);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + L::MISC_OFF + 4);
    constexpr uint32_t TMEM_COLS = 2 * BN;      // 128, 256 or 512

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t rank = PAIR ? cluster_ctarank() : 0;
    const bool leader = rank == 0;

    if (threadIdx.x == 0) {
        prefetch_map(&tmA);
        prefetch_map(&tmB);
        for (int s = 0; s < STAGES; ++s) {
            mbar_init(bar_full + 8 * s, 1);
            mbar_init(bar_empty + 8 * s, 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(bar_tfull + 8 * i, 1);
            mbar_init(bar_tempty + 8 * i, PAIR ? 2 * EPI_WARPS : EPI_WARPS);
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        if (PAIR) {
            tmem_alloc2(smem_u32(tmem_slot), TMEM_COLS);
            tmem_relinquish2();
        } else {
            tmem_alloc(smem_u32(tmem_slot), TMEM_COLS);
            tmem_relinquish();
        }
    }
    pdl_launch_dependents();
    tc_fence_before();
    __syncthreads();
    if (PAIR) cluster_sync_all();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    pdl_wait();

    const uint32_t full_leader = PAIR ? mapa_u32(bar_full, 0) : bar_full;
    const uint32_t tempty_leader = PAIR ? mapa_u32(bar_tempty, 0) : bar_tempty;
    constexpr int TM_ROWS = PAIR ? 2 * BM : BM;
    const int worker = PAIR ? blockIdx.x >> 1 : blockIdx.x, nworkers = PAIR ? gridDim.x >> 1 : gridDim.x;
    const int tiles_m = (a.M + TM_ROWS - 1) / TM_ROWS, tiles_n = (a.N + BN - 1) / BN;
    const int per_split = tiles_m * tiles_n, total = per_split * a.splits;
    const int all_kb = (2 * a.K + BK - 1) / BK;
    int fail = 0;

    if (warp == 0) {
        if (lane == 0) {
            int stage = 0;
            uint32_t phase = 0;
            for (int t = worker; t < total && fail == 0; t += nworkers) {
                const int sp = t / per_split, tt = t - sp * per_split, nt = tt / tiles_m, mt = tt - nt * tiles_m;
                const int kb0 = (int)((int64_t)all_kb * sp / a.splits), num_kb = (int)((int64_t)all_kb * (sp + 1) / a.splits) - kb0;
                const int row0 = mt * TM_ROWS + (int)rank * BM, brow = nt * BN + (PAIR ? (int)rank * (BN / 2) : 0);
                for (int kb = 0; kb < num_kb; ++kb) {
                    if (int w = mbar_wait(bar_empty + 8 * stage, phase ^ 1, abort_flag, a.wait_ns)) { fail = w == 1 ? 1 : -1; break; }
                    const uint32_t sa = sbase + stage * L::STAGE_BYTES, sb = sa + L::A_BYTES;
                    if (PAIR) {
                        if (leader) mbar_expect_tx(bar_full + 8 * stage, 2 * L::STAGE_BYTES);
                        tma_load_2d_pair(sa, &tmA, (kb0 + kb) * BK, row0, full_leader + 8 * stage);
                        tma_load_2d_pair(sb, &tmB, (kb0 + kb) * BK, brow, full_leader + 8 * stage);
                    } else {
                        mbar_expect_tx(bar_full + 8 * stage, L::STAGE_BYTES);
                        tma_load_2d(sa, &tmA, (kb0 + kb) * BK, row0, bar_full + 8 * stage);
                        tma_load_2d(sb, &tmB, (kb0 + kb) * BK, brow, bar_full + 8 * stage);
                    }
                    if (++stage == STAGES) { stage = 0; phase ^= 1; }
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0 && leader) {
            constexpr uint32_t idesc = umma_idesc_bf16(TM_ROWS, BN);
            int stage = 0;
            uint32_t phase = 0, acc = 0, acc_phase = 0;
            for (int t = worker; t < total && fail == 0; t += nworkers) {
                const int w0 = PAIR ? mbar_wait_cluster(bar_tempty + 8 * acc, acc_phase ^ 1, abort_flag, a.wait_ns)
                                    : mbar_wait(bar_tempty + 8 * acc, acc_phase ^ 1, abort_flag, a.wait_ns);
                if (w0) { fail = w0 == 1 ? 2 : -1; break; }
                tc_fence_after();
                const uint32_t d_tmem = tmem_base + acc * BN;
                const int sp = t / per_split;
                const int num_kb = (int)((int64_t)all_kb * (sp + 1) / a.splits) - (int)((int64_t)all_kb * sp / a.splits);
                for (int kb = 0; kb < num_kb; ++kb) {
                    if (int w = mbar_wait(bar_full + 8 * stage, phase, abort_flag, a.wait_ns)) { fail = w == 1 ? 3 : -1; break; }
                    tc_fence_after();
                    const uint32_t sa = sbase + stage * L::STAGE_BYTES, sb = sa + L::A_BYTES;
                    const uint64_t da = umma_desc(sa), db = umma_desc(sb);
#pragma unroll
                    for (int k = 0; k < BK / UMMA_K; ++k) {       // 16 values = 32 bytes of K per instruction
                        const uint64_t o = (uint64_t)(k * (UMMA_K >> 4));
                        if (PAIR) umma_bf16_pair(d_tmem, da + o, db + o, idesc, (kb | k) != 0 ? 1u : 0u);
                        else umma_bf16(d_tmem, da + o, db + o, idesc, (kb | k) != 0 ? 1u : 0u);
                    }
                    if (PAIR) umma_commit_pair(bar_empty + 8 * stage);
                    else umma_commit(bar_empty + 8 * stage);
                    if (++stage == STAGES) { stage = 0; phase ^= 1; }
                }
                if (fail) break;
                if (PAIR) umma_commit_pair(bar_tfull + 8 * acc);
                else umma_commit(bar_tfull + 8 * acc);
                acc ^= 1;
                if (acc == 0) acc_phase ^= 1;
            }
        }
    } else {
        const int q = warp & 3, chalf = (warp - 2) >> 2;
        uint32_t acc = 0, acc_phase = 0;
        for (int t = worker; t < total && fail == 0; t += nworkers) {
            const int sp = t / per_split, tt = t - sp * per_split, nt = tt / tiles_m, mt = tt - nt * tiles_m;
            uint8_t* out = static_cast<uint8_t*>(a.out) + (size_t)sp * a.split_stride * 4;
            const int n0 = nt * BN + chalf * (BN / 2), wrow0 = mt * TM_ROWS + (int)rank * BM + 32 * q;
            if (int w = mbar_wait(bar_tfull + 8 * acc, acc_phase, abort_flag, a.wait_ns)) fail = w == 1 ? 4 : -1;
            epilogue_bar();         // the epilogue threads agree on giving up before anyone touches TMEM
            if (*abort_flag) { if (!fail) fail = -1; break; }
            tc_fence_after();
            bg_epilogue<BN>(a, out, tmem_base + acc * BN + chalf * (BN / 2) + ((uint32_t)(32 * q) << 16), wrow0, n0,
                            smem + L::EPI_OFF + (warp - 2) * EPI_STAGE_WARP, lane);
            tc_fence_before();
            __syncwarp();
            if (lane == 0) {
                if (!PAIR || leader) mbar_arrive(bar_tempty + 8 * acc);
                else mbar_arrive_cluster(tempty_leader + 8 * acc);
            }
            acc ^= 1;
            if (acc == 0) acc_phase ^= 1;
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
    if (*abort_flag) {
        const uint64_t t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);   // 0.2 ms for outstanding TMA writes
        __syncthreads();
    }
    if (PAIR) cluster_sync_all();
    tc_fence_after();
    if (warp == 1) {
        if (PAIR) tmem_dealloc2(tmem_base, TMEM_COLS);
        else tmem_dealloc(tmem_base, TMEM_COLS);
    }
}

template <int BN, int STAGES>
__global__ void __launch_bounds__(CTA_THREADS, 1) gemm_bf16_kernel(const __grid_constant__ CUtensorMap tmA,
                                                            const __grid_constant__ CUtensorMap tmB, const BgArgs a) {
    gemm_bf16_body<BN, STAGES, false>(tmA, tmB, a);
}
template <int BN, int STAGES>
__global__ void __cluster_dims__(2, 1, 1) __launch_bounds__(CTA_THREADS, 1)
    gemm_bf16_pair_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB, const BgArgs a) {
    gemm_bf16_body<BN, STAGES, true>(tmA, tmB, a);
}

template <int BN, int STAGES, bool PAIR>
static int launch_bg(const void* A, int64_t lda, const void* W, int64_t ldw, const BgArgs& a, cudaStream_t st) {
    using L = BgSmem<BN, STAGES, PAIR>;
    static bool configured[64] = {};
    const int dev = current_device();
    SCMX_REQUIRE(dev >= 0, SCMX_ECUDA, "no current CUDA device (ordinal 0..63)");
    void (*kernel)(CUtensorMap, CUtensorMap, BgArgs);
    if constexpr (PAIR) kernel = gemm_bf16_pair_kernel<BN, STAGES>;
    else kernel = gemm_bf16_kernel<BN, STAGES>;
    if (!configured[dev]) {
        SCMX_CUDA_OK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL));
        configured[dev] = true;
    }
    CUtensorMap tmA, tmB;
    int rc = make_map_u8(&tmA, A, a.M, 2 * (int64_t)a.K, BK, BM, 128, 2 * lda);
    if (rc) return rc;
    rc = make_map_u8(&tmB, W, a.N, 2 * (int64_t)a.K, BK, PAIR ? BN / 2 : BN, 128, 2 * ldw);
    if (rc) return rc;
    constexpr int rows = PAIR ? 2 * BM : BM;
    const int64_t tiles = ((a.M + rows - 1) / rows) * (int64_t)((a.N + BN - 1) / BN) * a.splits;
    int workers = PAIR ? sm_count() / 2 : sm_count();
    if (tiles < workers) workers = (int)tiles;
    SCMX_PDL_OK("gemm_bf16", launch_pdl(kernel, dim3(PAIR ? 2 * workers : workers), dim3(CTA_THREADS), (size_t)L::TOTAL, st, tmA, tmB, a));
    return SCMX_OK;
}

// Sum of the K ranges' partial products, in order of the ranges -> the output type.
__global__ void __launch_bounds__(256) gemm_reduce_kernel(const float* part, int splits, int64_t stride, int64_t rows, int quads, int64_t ldp,
                                                          int out_f32, void* out, int64_t ldo) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= rows * quads) return;
    const int64_t r = i / quads;
    const int c = 4 * (int)(i - r * quads);
    float4 s = make_float4(0, 0, 0, 0);
#pragma unroll 8
    for (int k = 0; k < splits; ++k) {
        const float4 v = __ldcg(reinterpret_cast<const float4*>(part + k * stride + r * ldp + c));
        s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
    }
    if (out_f32) st4(static_cast<float*>(out) + r * ldo + c, s.x, s.y, s.z, s.w);
    else st4(static_cast<bf16_t*>(out) + r * ldo + c, s.x, s.y, s.z, s.w);
}

}  // namespace scmx

using namespace scmx;

extern "C" int scmx_gemm_bf16(const void* A, int64_t lda, const void* W, int64_t ldw, int64_t M, int64_t N, int64_t K, int act, float a_pos,
                              float a_neg, void* out, int out_f32, int64_t ldo, int tile, int splits, float* part, int32_t* status,
                              void* stream) {
    SCMX_REQUIRE(A && W && out && status, SCMX_EINVAL, "gemm_bf16: null buffer");
    SCMX_REQUIRE(M >= 0 && N > 0 && K > 0 && M < (1ll << 30) && N < (1ll << 30) && K < (1ll << 29), SCMX_EINVAL, "gemm_bf16: M=%lld N=%lld K=%lld",
                 (long long)M, (long long)N, (long long)K);
    SCMX_REQUIRE(lda % 8 == 0 && ldw % 8 == 0 && lda >= K && ldw >= K, SCMX_EINVAL,
                 "gemm_bf16: the row pitches %lld, %lld must be multiples of 8 that hold K=%lld", (long long)lda, (long long)ldw, (long long)K);
    const int q = out_f32 ? 4 : 8;
    SCMX_REQUIRE(act >= 0 && act <= 2 && (act != 2 || N % 32 == 0), SCMX_EINVAL, "gemm_bf16: act=%d on %lld columns", act, (long long)N);
    const int64_t nout = act == 2 ? N / 2 : N;
    SCMX_REQUIRE(ldo % q == 0 && ldo >= (nout + q - 1) / q * q, SCMX_EINVAL, "gemm_bf16: output pitch %lld for %lld columns", (long long)ldo, (long long)N);
    SCMX_REQUIRE(((uintptr_t)A & 15) == 0 && ((uintptr_t)W & 15) == 0 && ((uintptr_t)out & 15) == 0, SCMX_EINVAL, "gemm_bf16: pointer not 16-byte aligned");
    SCMX_REQUIRE(tile == 0 || tile == 64 || tile == 128 || tile == 256, SCMX_EINVAL, "gemm_bf16: tile=%d", tile);
    if (M == 0) return SCMX_OK;
    BgArgs a;
    a.M = (int)M; a.N = (int)N; a.K = (int)K; a.out_f32 = out_f32 ? 1 : 0; a.act = act; a.a_pos = a_pos; a.a_neg = a_neg;
    a.out = out; a.ldo = ldo; a.status = status; a.wait_ns = g_wait_limit_ns; a.splits = 1; a.split_stride = 0;
    const cudaStream_t st = (cudaStream_t)stream;
    if (tile == 0) {
        const int64_t m = (M + 127) / 128;
        if (M > 128 && N >= 256 && ((M + 255) / 256) * ((N + 255) / 256) * 2 >= sm_count() / 2) tile = 256;
        else tile = m * ((N + 127) / 128) >= sm_count() / 2 ? 128 : 64;
    }
    if (splits > 1) {
        SCMX_REQUIRE(part && ((uintptr_t)part & 15) == 0 && act == 0 && splits <= (2 * K + BK - 1) / BK, SCMX_EINVAL,
                     "gemm_bf16: %d ranges of K=%lld need a buffer and no activation", splits, (long long)K);
        const int64_t ldp = (N + 3) / 4 * 4;
        a.out = part; a.out_f32 = 1; a.ldo = ldp; a.splits = splits; a.split_stride = M * ldp;
        const int rc = tile == 256 ? launch_bg<256, 5, true>(A, lda, W, ldw, a, st)
                     : tile == 128 ? launch_bg<128, 5, false>(A, lda, W, ldw, a, st) : launch_bg<64, 7, false>(A, lda, W, ldw, a, st);
        if (rc) return rc;
        const int quads = (int)(ldp / 4);
        SCMX_PDL_OK("gemm_reduce_kernel", launch_pdl(gemm_reduce_kernel, dim3((unsigned)((M * quads + 255) / 256)), dim3(256), 0, st, (const float*)part,
                                                     splits, a.split_stride, M, quads, ldp, out_f32 ? 1 : 0, out, ldo));
        return SCMX_OK;
    }
    if (tile == 256) return launch_bg<256, 5, true>(A, lda, W, ldw, a, st);
    if (tile == 128) return launch_bg<128, 5, false>(A, lda, W, ldw, a, st);
    return launch_bg<64, 7, false>(A, lda, W, ldw, a, st);
}
