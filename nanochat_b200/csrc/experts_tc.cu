// The experts' products for many rows, on the tensor cores (tcgen05, accumulators in tensor memory).
//
// Persistent CTAs, one per SM, walk over the tiles of all experts: 128 of an expert's sorted positions by BN
// weight rows (UP: BN / 2 gate and the BN / 2 up rows of the same channels, so that a thread holds both
// factors of an output).  A tile's K runs in steps of 64 through a ring in shared memory (128-byte
// swizzle).  Roles, connected by mbarriers:
//   warp 0      moves the weights, and without UP the positions (rows of act), by TMA
//   warps 6-13  UP: the tokens of a tile lie anywhere in h; these warps fetch them with 16-byte asynchronous copies
//               into the place the swizzle gives them, so h is never copied into sorted order (a gather by
//               TMA, four rows per instruction, was three times slower than the products).  Four of the
//               warps take the even steps, four the odd ones.
//   warp 1      one thread issues the products into one of two accumulators
//   warps 2-5   one thread per position reads the other accumulator, applies the router's weight and the
//               activation (UP) or finds the pair's place (down), and stores
// Tiles of one expert are consecutive, positions fastest: the CTAs that run side by side share weights and rows
// in L2.  What stands in a tile behind an expert's last position is not stored.  Every wait is bounded; one that
// runs out sets NCKV_ST_TIMEOUT, the roles stop, copies in flight are waited for and tensor memory is freed.
#include "experts.cuh"
#include "tc05.cuh"

namespace nckv {

constexpr int ET_M = 128, ET_K = 64;
constexpr int ET_THREADS = 192, ET_GATHER = 256;  // UP has ET_GATHER more, in two halves
constexpr int ET_MAX_EXPERTS = 1024;
constexpr int ET_A_BYTES = ET_M * ET_K * 2;

template <int BN> struct EtShape {
    static constexpr int B_BYTES = BN * ET_K * 2, STAGE = ET_A_BYTES + B_BYTES;
    static constexpr int STAGES = BN == 256 ? 4 : 6;
    static constexpr int SMEM = STAGES * STAGE + 256;
};

// One tile, found by walking on from the tile before.
struct EtCursor {
    int e, m_lo, m_hi, m0, n;
    __device__ __forceinline__ bool seek(const int *s_first, const ExpertParams &p, int n_tiles, int idx) {
        while (e < p.E && idx >= s_first[e + 1] * n_tiles) ++e;
        if (e >= p.E) return false;
        const int tiles = s_first[e + 1] - s_first[e], local = idx - s_first[e] * n_tiles;
        m_lo = p.offsets[e];
        m_hi = p.offsets[e + 1];
        n = local / tiles;
        m0 = m_lo + (local - n * tiles) * ET_M;
        return true;
    }
};

template <bool UP, int BN>
__global__ void __launch_bounds__(ET_THREADS + (UP ? ET_GATHER : 0), 1)
experts_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_w, const ExpertParams p) {
    using Shape = EtShape<BN>;
    constexpr int STAGES = Shape::STAGES;
    extern __shared__ __align__(1024) uint8_t smem[];
    __shared__ int s_first[ET_MAX_EXPERTS + 1];  // token tiles before expert e
    if ((smem_u32(smem) & 1023u) != 0) {         // uniform; checked rather than assumed
        if (threadIdx.x == 0) atomicOr(p.status, (int)NCKV_ST_TIMEOUT);
        return;
    }
    uint64_t *bars = reinterpret_cast<uint64_t *>(smem + STAGES * Shape::STAGE);
    uint64_t *bar_full = bars, *bar_free = bars + STAGES;                         // a stage's operands landed / were read
    uint64_t *bar_acc = bars + 2 * STAGES, *bar_read = bars + 2 * STAGES + 2;     // an accumulator is complete / was read
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(bars + 2 * STAGES + 4);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int n_tiles = UP ? (p.N + BN / 2 - 1) / (BN / 2) : (p.N + BN - 1) / BN, k_steps = (p.K + ET_K - 1) / ET_K;
    if (warp == 0) {
        tmem_alloc(tmem_slot, 2 * BN);
        tmem_relinquish();
    } else if (warp == 1) {
        int carry = 0;
        for (int e0 = 0; e0 < p.E; e0 += 32) {
            const int e = e0 + lane;
            const int t = e < p.E ? (p.offsets[e + 1] - p.offsets[e] + ET_M - 1) / ET_M : 0;
            int inc = t;
#pragma unroll
            for (int off = 1; off < 32; off <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, inc, off);
                if (lane >= off) inc += v;
            }
            if (e < p.E) s_first[e + 1] = carry + inc;
            carry += __shfl_sync(0xffffffffu, inc, 31);
        }
        if (lane == 0) s_first[0] = 0;
    } else if (tid == 64) {
        prefetch_tensormap(&map_a);
        prefetch_tensormap(&map_w);
        for (int i = 0; i < STAGES; ++i) {
            mbar_init(&bar_full[i], UP ? 1 + ET_GATHER / 64 : 1);
            mbar_init(&bar_free[i], 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(&bar_acc[i], 1);
            mbar_init(&bar_read[i], 4);
        }
        *abort_flag = 0;
        fence_mbar_init();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    const int total = s_first[p.E] * n_tiles;
    auto timed_out = [&]() {
        *abort_flag = 1;
        atomicOr(p.status, (int)NCKV_ST_TIMEOUT);
    };
    auto warp_wait = [&](uint64_t *bar, uint32_t parity) -> bool {  // one lane polls
        int ok = 1;
        if (lane == 0) ok = *abort_flag == 0 && mbar_wait_bounded(bar, parity) ? 1 : 0;
        ok = __shfl_sync(0xffffffffu, ok, 0);
        __syncwarp();
        return ok != 0;
    };

    EtCursor cur;
    cur.e = 0;
    if (warp == 0) {
        // =============== operands ===================================================================
        uint32_t fill = 0;  // number of the fill: stage fill % STAGES
        bool ok = true;
        for (int idx = blockIdx.x; idx < total && ok; idx += gridDim.x) {
            if (!cur.seek(s_first, p, n_tiles, idx)) break;
            for (int ks = 0; ks < k_steps; ++ks, ++fill) {
                const uint32_t st = fill % STAGES, round = fill / STAGES;
                if (round > 0 && !warp_wait(&bar_free[st], (round - 1) & 1u)) {
                    ok = false;
                    break;
                }
                uint8_t *a = smem + st * Shape::STAGE, *b = a + ET_A_BYTES;
                if (lane == 0) {
                    mbar_arrive_expect_tx(&bar_full[st], UP ? Shape::B_BYTES : Shape::STAGE);
                    if (UP) {
                        tma_load_4d(b, &map_w, &bar_full[st], ks * ET_K, cur.n * (BN / 2), 0, cur.e);
                        tma_load_4d(b + Shape::B_BYTES / 2, &map_w, &bar_full[st], ks * ET_K, cur.n * (BN / 2), 1, cur.e);
                    } else {
                        tma_load_2d(a, &map_a, &bar_full[st], ks * ET_K, cur.m0);
                        tma_load_4d(b, &map_w, &bar_full[st], ks * ET_K, cur.n * BN, 0, cur.e);
                    }
                }
            }
        }
        if (!ok) {
            if (lane == 0) {
                timed_out();
                // copies already issued land before the CTA's memory is released
                for (uint32_t f = fill > STAGES ? fill - STAGES : 0; f < fill; ++f)
                    mbar_wait_bounded(&bar_full[f % STAGES], (f / STAGES) & 1u, 100000000ull);
            }
            __syncwarp();
        }
    } else if (warp == 1) {
        // =============== products ===================================================================
        if (lane == 0) {
            constexpr uint32_t IDESC = umma_idesc(ET_M, BN, 0, 0);
            const uint64_t desc0 = smem_desc_sw128(smem_u32(smem), 16, 1024);
            uint32_t fill = 0, tile = 0;
            bool ok = true;
            for (int idx = blockIdx.x; idx < total && ok; idx += gridDim.x, ++tile) {
                const uint32_t buf = tile & 1u, use = tile >> 1;
                if (use > 0 && !mbar_wait_bounded(&bar_read[buf], (use - 1) & 1u)) {
                    ok = false;
                    break;
                }
                tc_fence_after();
                const uint32_t d = tmem + buf * BN;
                for (int ks = 0; ks < k_steps; ++ks, ++fill) {
                    const uint32_t st = fill % STAGES;
                    if (*abort_flag != 0 || !mbar_wait_bounded(&bar_full[st], (fill / STAGES) & 1u)) {
                        ok = false;
                        break;
                    }
                    tc_fence_after();
                    const uint64_t da = desc0 + (uint64_t)((st * Shape::STAGE) >> 4), db = da + (uint64_t)(ET_A_BYTES >> 4);
#pragma unroll
                    for (int kk = 0; kk < ET_K / 16; ++kk)
                        umma_bf16(d, da + (uint64_t)(kk * 2), db + (uint64_t)(kk * 2), IDESC, ks > 0 || kk > 0 ? 1u : 0u);
                    umma_commit(&bar_free[st]);
                }
                if (ok) umma_commit(&bar_acc[buf]);
            }
            if (!ok) timed_out();
        }
        __syncwarp();
    } else if (UP && warp >= 6) {
        // =============== tokens =====================================================================
        // 8 threads fetch the 128 bytes a token has in a step; a thread serves 8 tokens.  A step is handed over
        // once the LAG of its own steps behind it have been asked for.
        constexpr int LAG = STAGES / 2 - 1;
        const uint32_t odd = tid >= ET_THREADS + ET_GATHER / 2;
        const int pt = (tid - ET_THREADS) & (ET_GATHER / 2 - 1), chunk = pt & 7, r0 = pt >> 3;
        uint32_t fill = 0, mine = 0;  // steps, and those of this half: its step k is number 2 k + odd
        bool ok = true;
        auto hand_over = [&](uint32_t k) {
            fence_proxy_async_smem();  // this thread's copies, before the products read them
            __syncwarp();
            if (lane == 0) mbar_arrive(&bar_full[(2 * k + odd) % STAGES]);
        };
        for (int idx = blockIdx.x; idx < total && ok; idx += gridDim.x) {
            if (!cur.seek(s_first, p, n_tiles, idx)) break;
            const __nv_bfloat16 *src[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int m = cur.m0 + r0 + 16 * i;  // nobody reads the results of rows behind the expert's last
                src[i] = m < cur.m_hi ? static_cast<const __nv_bfloat16 *>(p.a) + (long long)(p.slot[m] / p.top) * p.K + chunk * 8 : nullptr;
            }
            for (int ks = 0; ks < k_steps; ++ks, ++fill) {
                if ((fill & 1u) != odd) continue;
                const uint32_t st = fill % STAGES, round = fill / STAGES;
                if (round > 0 && !warp_wait(&bar_free[st], (round - 1) & 1u)) {
                    ok = false;
                    break;
                }
                const uint32_t base = smem_u32(smem + st * Shape::STAGE);
                const int bytes = ks * ET_K + chunk * 8 < p.K ? 16 : 0;  // zeros behind the last channel
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    const int r = r0 + 16 * i;
                    if (src[i])
                        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(base + r * 128 + ((chunk ^ (r & 7)) << 4)),
                                     "l"(bytes ? src[i] + ks * ET_K : src[i]), "r"(bytes)
                                     : "memory");
                }
                asm volatile("cp.async.commit_group;" ::: "memory");
                if (mine >= (uint32_t)LAG) {
                    asm volatile("cp.async.wait_group %0;" ::"n"(LAG) : "memory");
                    hand_over(mine - LAG);
                }
                ++mine;
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        if (ok)
            for (uint32_t k = mine > (uint32_t)LAG ? mine - LAG : 0; k < mine; ++k) hand_over(k);
        if (!ok && lane == 0 && *abort_flag == 0) timed_out();
        __syncwarp();
    } else {
        // =============== results ====================================================================
        const int q = warp & 3, row = q * 32 + lane;  // a warp reaches tensor-memory lanes 32 (warp % 4) ..
        const uint32_t lane_sel = (uint32_t)(q * 32) << 16;
        const bool vec = p.N % 8 == 0 && (((uintptr_t)p.out) & 15) == 0;
        uint32_t tile = 0;
        for (int idx = blockIdx.x; idx < total; idx += gridDim.x, ++tile) {
            if (!cur.seek(s_first, p, n_tiles, idx)) break;
            const int m = cur.m0 + row;
            const bool have = m < cur.m_hi;
            const float s = UP && have ? p.scale[m] : 0.f;
            const int n0 = cur.n * (UP ? BN / 2 : BN);
            __nv_bfloat16 *out = static_cast<__nv_bfloat16 *>(p.out) + (long long)(UP ? m : (have ? p.slot[m] : 0)) * p.N;
            const uint32_t buf = tile & 1u;
            if (!warp_wait(&bar_acc[buf], (tile >> 1) & 1u)) {
                if (lane == 0 && *abort_flag == 0) timed_out();
                break;
            }
            tc_fence_after();
            const uint32_t acc = tmem + buf * BN + lane_sel;
#pragma unroll 1
            for (int c = 0; c < (UP ? BN / 2 : BN); c += 32) {
                if (n0 + c >= p.N) break;  // uniform over the CTA
                __syncwarp();              // the loads below are warp-wide
                float v[32];
                if (UP) {
                    float u[32];
                    tmem_ld32x2(acc + c, v, acc + BN / 2 + c, u);
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[i] = Fn<__nv_bfloat16>::silu(s * v[i]) * (s * u[i]);
                } else {
                    tmem_ld32(acc + c, v);
                }
                if (!have) continue;
#pragma unroll
                for (int i = 0; i < 32; i += 8) {
                    const int n = n0 + c + i;
                    if (vec) {
                        if (n < p.N)
                            *reinterpret_cast<uint4 *>(out + n) = make_uint4(pack_bf16x2(v[i], v[i + 1]), pack_bf16x2(v[i + 2], v[i + 3]),
                                                                             pack_bf16x2(v[i + 4], v[i + 5]), pack_bf16x2(v[i + 6], v[i + 7]));
                    } else {
#pragma unroll
                        for (int k = 0; k < 8; ++k)
                            if (n + k < p.N) out[n + k] = __float2bfloat16_rn(v[i + k]);
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&bar_read[buf]);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 0) tmem_dealloc(tmem, 2 * BN);
}

template <bool UP, int BN>
static cudaError_t et_launch(const ExpertParams &p, cudaStream_t s, int *rc) {
    CUtensorMap ma, mw;
    {
        const int64_t dims[2] = {p.K, UP ? p.R / p.top : p.R}, strides[1] = {p.K};
        const int box[2] = {ET_K, ET_M};
        *rc = make_tensor_map(&ma, p.a, 2, dims, strides, box);  // not used by UP
    }
    if (*rc != NCKV_OK) return cudaSuccess;
    const int64_t N = p.N, K = p.K, halves = UP ? 2 : 1;
    const int64_t dims[4] = {K, N, halves, p.E}, strides[3] = {K, N * K, halves * N * K};
    const int box[4] = {ET_K, UP ? BN / 2 : BN, 1, 1};
    *rc = make_tensor_map(&mw, p.w, 4, dims, strides, box);
    if (*rc != NCKV_OK) return cudaSuccess;
    const cudaError_t e = cudaFuncSetAttribute(experts_tc_kernel<UP, BN>, cudaFuncAttributeMaxDynamicSharedMemorySize, EtShape<BN>::SMEM);
    if (e != cudaSuccess) return e;
    const long long tiles = ((long long)p.R / ET_M + p.E) * ((p.N + BN / halves - 1) / (BN / halves));
    const int grid = tiles < sm_count() ? (int)tiles : sm_count();
    experts_tc_kernel<UP, BN><<<grid, ET_THREADS + (UP ? ET_GATHER : 0), EtShape<BN>::SMEM, s>>>(ma, mw, p);
    return cudaGetLastError();
}

cudaError_t experts_tc(const ExpertParams &p, bool up, cudaStream_t s, int *rc) {
    if (p.E > ET_MAX_EXPERTS) {
        set_error("experts: at most %d experts", ET_MAX_EXPERTS);
        *rc = NCKV_E_UNSUPPORTED;
        return cudaSuccess;
    }
    // Narrow tiles read the operands more often, but leave smaller last waves: take them where that wins
    // at an even spread of the positions.
    const long long m_tiles = p.R / ET_M + (p.E + 1) / 2;
    auto waves = [&](int bn) {
        const int per = up ? bn / 2 : bn;
        return (m_tiles * ((p.N + per - 1) / per) + sm_count() - 1) / sm_count();
    };
    const bool wide = 2 * waves(256) * 10 <= waves(128) * 11;
    if (up) return wide ? et_launch<true, 256>(p, s, rc) : et_launch<true, 128>(p, s, rc);
    return wide ? et_launch<false, 256>(p, s, rc) : et_launch<false, 128>(p, s, rc);
}

}  // namespace nckv
