// Shared device/host helpers for libnckv (sm_100a only).
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>

#include "../../include/nckv.h"

#define NCKV_D 128  // head_dim every kernel is specialised for

namespace nckv {

// ---- host-side error text (thread local) --------------------------------------------------
void set_error(const char *fmt, ...);
int cuda_fail(cudaError_t e, const char *what);

#define NCKV_CUDA_CHECK(expr)                                   \
    do {                                                        \
        cudaError_t _e = (expr);                                \
        if (_e != cudaSuccess) return nckv::cuda_fail(_e, #expr); \
    } while (0)

// Number of SMs of the current device (cached per device).
int sm_count();

// Tiled tensor maps over a (B, T, Hkv, D) bf16 cache view (defined in host.cu): the 4-D form
// (d, h, t, b) and the 5-D form (d within half [64], t, half [2], h, b).
int make_kv_tensor_map(CUtensorMap *map, const void *base, int B, int T, int Hkv,
                       int64_t batch_stride, int64_t token_stride, int box_tokens);

int make_kv_tensor_map_5d(CUtensorMap *map, const void *base, int B, int T, int Hkv,
                          int64_t batch_stride, int64_t token_stride, int box_tokens);

// A bf16 tensor of `rank` dimensions (innermost first, strides in elements for dimensions 1 ..) as a tiled tensor
// map with the 128-byte swizzle; elements outside read as zero.
int make_tensor_map(CUtensorMap *map, const void *base, int rank, const int64_t *dims, const int64_t *strides, const int *box);

// ---- sequence-split bookkeeping (shared by host checks and kernels) ---------------------------
// Block-cyclic ownership of key positions: position p belongs to shard (p / block) % world and
// sits at local index (p / (block*world)) * block + p % block there.  owned_below(n) = how many
// positions p < n shard `rank` owns = the local index of position n when the shard owns it.
__host__ __device__ inline int owned_below(int n, int world, int rank, int block) {
    const int cycle = block * world;
    const int full = n / cycle, rem = n - full * cycle;
    int part = rem - rank * block;
    part = part < 0 ? 0 : (part > block ? block : part);
    return full * block + part;
}
struct KvSplit {  // block == 0: the cache is not split
    int world, rank, block;
};

// Peer-memory exchange of the sequence-split path: one symmetric buffer per rank,
//     data  [2][world][per] fp32, flags [2][world] u32   (per = p2p_per_floats(rows))
#define NCKV_MAX_PEERS 16
struct PeerPtrs {
    float *buf[NCKV_MAX_PEERS];
};
__host__ __device__ inline long long p2p_per_floats(int rows) { return (long long)rows * NCKV_D + ((rows + 3) & ~3); }

// What a head's softmax ends with besides the division by its sum: a sink (one more term of score 0 in the
// sum, without a value) and a sigmoid gate per token and head.
struct HeadEnd {
    int sink;
    const __nv_bfloat16 *gate;  // rows of one logit per head, or null
    long long gate_stride;
    __host__ __device__ bool active() const { return sink || gate; }
#ifdef __CUDACC__
    // factor on the unnormalised output; max and sum of the exponentials in powers of two
    __device__ __forceinline__ float factor(float m, float l, long long row, int head) const {
        float f = 1.f / (sink ? l + exp2f(-m) : l);
        if (gate) f *= 1.f / (1.f + __expf(-__bfloat162float(gate[row * gate_stride + head])));
        return f;
    }
#endif
};

// ---- device helpers ----------------------------------------------------------------------
#ifdef __CUDACC__

__device__ __forceinline__ uint32_t smem_u32(const void *p) {
    return static_cast<uint32_t>(__cvta_generic_to_shared(p));
}

__device__ __forceinline__ float bf16_bits_to_float(uint32_t bits16) {
    return __uint_as_float(bits16 << 16);
}
__device__ __forceinline__ float bf16lo(uint32_t packed) { return __uint_as_float(packed << 16); }
__device__ __forceinline__ float bf16hi(uint32_t packed) {
    return __uint_as_float(packed & 0xffff0000u);
}
// round-to-nearest-even fp32 -> bf16 -> fp32 (the rounding an eager bf16 op applies)
__device__ __forceinline__ float round_bf16(float x) {
    return __bfloat162float(__float2bfloat16_rn(x));
}
__device__ __forceinline__ uint32_t pack_bf16x2(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t *>(&v);
}

// ---- mbarrier ----------------------------------------------------------------------------
__device__ __forceinline__ void mbar_init(uint64_t *bar, uint32_t count) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count)
                 : "memory");
}
__device__ __forceinline__ void mbar_inval(uint64_t *bar) {
    asm volatile("mbarrier.inval.shared::cta.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void mbar_arrive_expect_tx(uint64_t *bar, uint32_t bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)),
                 "r"(bytes)
                 : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint64_t *bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ bool mbar_try_wait(uint64_t *bar, uint32_t parity) {
    uint32_t ok;
    asm volatile(
        "{\n"
        ".reg .pred p;\n"
        "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n"
        "selp.u32 %0, 1, 0, p;\n"
        "}\n"
        : "=r"(ok)
        : "r"(smem_u32(bar)), "r"(parity)
        : "memory");
    return ok != 0;
}
// Non-blocking test of a phase (mbarrier.test_wait never suspends the thread).
__device__ __forceinline__ bool mbar_test(uint64_t *bar, uint32_t parity) {
    uint32_t ok;
    asm volatile(
        "{\n"
        ".reg .pred p;\n"
        "mbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n"
        "selp.u32 %0, 1, 0, p;\n"
        "}\n"
        : "=r"(ok)
        : "r"(smem_u32(bar)), "r"(parity)
        : "memory");
    return ok != 0;
}
// Bounded wait: polls until the phase completes or about `limit_ns` of wall time have passed
// (each poll may suspend for a short, hardware-defined slice) and reports failure instead of
// spinning for ever.
__device__ __forceinline__ unsigned long long global_timer_ns() {
    unsigned long long t;
    asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
    return t;
}
constexpr unsigned long long NCKV_WAIT_LIMIT_NS = 2000000000ull;  // 2 s: far beyond any legitimate wait
__device__ __forceinline__ bool mbar_wait_bounded(uint64_t *bar, uint32_t parity,
                                                  unsigned long long limit_ns = NCKV_WAIT_LIMIT_NS) {
    if (mbar_try_wait(bar, parity)) return true;
    const unsigned long long t0 = global_timer_ns();
    for (;;) {
#pragma unroll 1
        for (int i = 0; i < 64; ++i) {
            if (mbar_try_wait(bar, parity)) return true;
        }
        if (global_timer_ns() - t0 > limit_ns) return false;
    }
}

__device__ __forceinline__ void fence_proxy_async_smem() {
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}
__device__ __forceinline__ void fence_mbar_init() {
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
}

// ---- TMA (tiled bulk tensor copies, global -> shared, no multicast) -------------------------
__device__ __forceinline__ void tma_load_4d(void *smem_dst, const CUtensorMap *map, uint64_t *bar,
                                            int c0, int c1, int c2, int c3) {
    asm volatile(
        "cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes"
        " [%0], [%1, {%2, %3, %4, %5}], [%6];" ::"r"(smem_u32(smem_dst)),
        "l"(map), "r"(c0), "r"(c1), "r"(c2), "r"(c3), "r"(smem_u32(bar))
        : "memory");
}
__device__ __forceinline__ void tma_load_2d(void *smem_dst, const CUtensorMap *map, uint64_t *bar, int c0, int c1) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes"
        " [%0], [%1, {%2, %3}], [%4];" ::"r"(smem_u32(smem_dst)),
        "l"(map), "r"(c0), "r"(c1), "r"(smem_u32(bar))
        : "memory");
}
// Same, with an L2 cache policy (e.g. evict-first for data that is streamed once).
__device__ __forceinline__ void tma_load_4d_hint(void *smem_dst, const CUtensorMap *map, uint64_t *bar,
                                                 int c0, int c1, int c2, int c3, uint64_t policy) {
    asm volatile(
        "cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes.L2::cache_hint"
        " [%0], [%1, {%2, %3, %4, %5}], [%6], %7;" ::"r"(smem_u32(smem_dst)),
        "l"(map), "r"(c0), "r"(c1), "r"(c2), "r"(c3), "r"(smem_u32(bar)), "l"(policy)
        : "memory");
}
__device__ __forceinline__ uint64_t l2_policy_evict_first() {
    uint64_t pol;
    asm volatile("createpolicy.fractional.L2::evict_first.b64 %0, 1.0;" : "=l"(pol));
    return pol;
}
// Programmatic dependent launch: let the next kernel of the stream start its prologue early /
// wait until everything the previous kernel wrote is visible.  Both are no-ops for a kernel that
// was launched without the programmatic-serialization attribute.
__device__ __forceinline__ void pdl_launch_dependents() {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}
__device__ __forceinline__ void pdl_wait_prior_grids() {
    asm volatile("griddepcontrol.wait;" ::: "memory");
}
__device__ __forceinline__ void tma_load_5d(void *smem_dst, const CUtensorMap *map, uint64_t *bar,
                                            int c0, int c1, int c2, int c3, int c4) {
    asm volatile(
        "cp.async.bulk.tensor.5d.shared::cluster.global.mbarrier::complete_tx::bytes"
        " [%0], [%1, {%2, %3, %4, %5, %6}], [%7];" ::"r"(smem_u32(smem_dst)),
        "l"(map), "r"(c0), "r"(c1), "r"(c2), "r"(c3), "r"(c4), "r"(smem_u32(bar))
        : "memory");
}
__device__ __forceinline__ void tma_load_5d_hint(void *smem_dst, const CUtensorMap *map, uint64_t *bar,
                                                 int c0, int c1, int c2, int c3, int c4, uint64_t policy) {
    asm volatile(
        "cp.async.bulk.tensor.5d.shared::cluster.global.mbarrier::complete_tx::bytes.L2::cache_hint"
        " [%0], [%1, {%2, %3, %4, %5, %6}], [%7], %8;" ::"r"(smem_u32(smem_dst)),
        "l"(map), "r"(c0), "r"(c1), "r"(c2), "r"(c3), "r"(c4), "r"(smem_u32(bar)), "l"(policy)
        : "memory");
}
// L2 prefetch of a tile (no shared-memory destination, no completion to wait for)
__device__ __forceinline__ void tma_prefetch_l2_5d(const CUtensorMap *map, int c0, int c1, int c2, int c3, int c4) {
    asm volatile("cp.async.bulk.prefetch.tensor.5d.L2.global.tile [%0, {%1, %2, %3, %4, %5}];" ::"l"(map), "r"(c0),
                 "r"(c1), "r"(c2), "r"(c3), "r"(c4)
                 : "memory");
}
__device__ __forceinline__ void tma_prefetch_l2_4d(const CUtensorMap *map, int c0, int c1, int c2, int c3) {
    asm volatile("cp.async.bulk.prefetch.tensor.4d.L2.global.tile [%0, {%1, %2, %3, %4}];" ::"l"(map), "r"(c0),
                 "r"(c1), "r"(c2), "r"(c3)
                 : "memory");
}
__device__ __forceinline__ void prefetch_tensormap(const CUtensorMap *map) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(map) : "memory");
}

// ---- warp-level matrix ops (legacy tensor path, used only by the memory-bound decode kernel)
__device__ __forceinline__ void ldmatrix_x4(uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3,
                                            uint32_t saddr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
                 : "r"(saddr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t &r0, uint32_t &r1, uint32_t &r2,
                                                  uint32_t &r3, uint32_t saddr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
                 : "r"(saddr));
}
// D(16x8,f32) += A(16x16,bf16,row) * B(16x8,bf16,col)
__device__ __forceinline__ void mma_bf16_16816(float &d0, float &d1, float &d2, float &d3,
                                               uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3,
                                               uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
        "{%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d0), "+f"(d1), "+f"(d2), "+f"(d3)
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

#endif  // __CUDACC__

}  // namespace nckv
