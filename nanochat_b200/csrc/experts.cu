// Mixture of experts: routing, and the experts' products for few rows or any size.
//
//   route_kernel          a thread (few experts) or a warp per token picks the `top` largest logits (ties: the lower
//                         index) and their sigmoids; one CTA counts, sorts by expert and writes the order.
//   route_pick_kernel,    the same for many tokens: choices and counts first, then positions from a prefix sum
//   route_place_kernel    and one reservation per CTA and expert.
//   expert_rows_kernel    bf16, few rows: bound by reading each used expert's weights once.  A CTA takes
//                         16 weight rows of one expert (8 gate and 8 up rows, or 16 down rows) as the rows
//                         of mma.m16n8k16 tiles, its warps split K, and up to 32 of the expert's tokens are
//                         the columns.  A lane loads 16 consecutive bytes of a row; the order of K inside a
//                         tile is the same for both operands and otherwise free.
//   expert_plain_kernel   fp32, and sizes without 16-byte rows: 32 x 32 tiles on the fp32 pipe.
// Many bf16 rows take the tensor-memory form in experts_tc.cu.
#include "experts.cuh"

namespace nckv {

constexpr int RT_MAX_EXPERTS = 1024;
constexpr int RT_ONE_CTA = 2048;  // (token, choice) pairs that one CTA sorts

struct RouteParams {
    const float *logits;   // (rows, E)
    int32_t *offsets;      // (E + 1)
    int32_t *slot;         // (R)
    float *scale;          // (R)
    int32_t *choice;       // many tokens: (R) expert of a pair, then (E) counts, (E) cursors
    float *weight;         // many tokens: (R)
    int rows, E, top;
};

// A row's logits in the lanes of a warp, 32 NJ at most, as numbers whose unsigned order is theirs; 0: none, or taken.
template <int NJ> struct RouteRow {
    uint32_t key[NJ];
    __device__ __forceinline__ void load(const float *z, int E, int lane) {
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const int e = lane + 32 * j;
            const uint32_t bits = e < E ? __float_as_uint(z[e]) : 0u;
            key[j] = e < E ? (bits & 0x80000000u ? ~bits : bits | 0x80000000u) : 0u;
        }
    }
    // the largest that is left (ties: the lowest index) and its logit
    __device__ __forceinline__ int next(int E, int lane, float &z) {
        uint32_t best = key[0];
        int idx = lane;
#pragma unroll
        for (int j = 1; j < NJ; ++j)
            if (key[j] > best) {
                best = key[j];
                idx = lane + 32 * j;
            }
        const uint32_t top = __reduce_max_sync(0xffffffffu, best);
        const int e = (int)__reduce_min_sync(0xffffffffu, best == top ? (unsigned)idx : 0x7fffffffu);
#pragma unroll
        for (int j = 0; j < NJ; ++j)
            if (e == lane + 32 * j) key[j] = 0u;
        z = __uint_as_float(top & 0x80000000u ? top & 0x7fffffffu : ~top);
        return min(e, E - 1);
    }
};

// The same with a row's logits in one thread, EM at most.
template <int EM> struct RouteThread {
    uint32_t key[EM];
    __device__ __forceinline__ void load(const float *z, int E) {
#pragma unroll
        for (int e = 0; e < EM; ++e) {
            const uint32_t bits = e < E ? __float_as_uint(z[e]) : 0u;
            key[e] = e < E ? (bits & 0x80000000u ? ~bits : bits | 0x80000000u) : 0u;
        }
    }
    __device__ __forceinline__ int next(float &z) {
        uint32_t best = key[0];
        int idx = 0;
#pragma unroll
        for (int e = 1; e < EM; ++e)
            if (key[e] > best) {
                best = key[e];
                idx = e;
            }
#pragma unroll
        for (int e = 0; e < EM; ++e)
            if (e == idx) key[e] = 0u;
        z = __uint_as_float(best & 0x80000000u ? best & 0x7fffffffu : ~best);
        return idx;
    }
};

// Calls put(pair, expert, logit) for every choice of the rows first, first + step, .. of a CTA or grid: by threads
// (PER_THREAD experts at most) or by warps (32 NJ at most).
template <int PER_THREAD, int NJ, typename Put>
__device__ __forceinline__ void route_rows(const RouteParams &p, int cta, int ctas, Put put) {
    const int tid = threadIdx.x, lane = tid & 31, NT = blockDim.x;
    if constexpr (PER_THREAD > 0) {
        for (int row = cta * NT + tid; row < p.rows; row += ctas * NT) {
            RouteThread<PER_THREAD> z;
            z.load(p.logits + (long long)row * p.E, p.E);
            for (int j = 0; j < p.top; ++j) {
                float zl;
                const int el = z.next(zl);
                put(row * p.top + j, el, zl);
            }
        }
    } else {
        const int step = ctas * (NT >> 5);
        RouteRow<NJ> z, ahead;
        int row = cta * (NT >> 5) + (tid >> 5);
        if (row < p.rows) z.load(p.logits + (long long)row * p.E, p.E, lane);
        for (; row < p.rows; row += step) {
            if (row + step < p.rows) ahead.load(p.logits + (long long)(row + step) * p.E, p.E, lane);
            for (int j = 0; j < p.top; ++j) {
                float zl;
                const int el = z.next(p.E, lane, zl);
                if (lane == 0) put(row * p.top + j, el, zl);
            }
            z = ahead;
        }
    }
}

// exclusive prefix sums of count[0 .. E) by the first warp; the total behind the last
__device__ __forceinline__ void route_prefix(const int *count, int *first, int E) {
    if (threadIdx.x >= 32) return;
    int carry = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
        const int e = e0 + threadIdx.x, n = e < E ? count[e] : 0;
        int inc = n;
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
            const int v = __shfl_up_sync(0xffffffffu, inc, off);
            if ((int)threadIdx.x >= off) inc += v;
        }
        if (e < E) first[e] = carry + inc - n;
        carry += __shfl_sync(0xffffffffu, inc, 31);
    }
    if (threadIdx.x == 0) first[E] = carry;
}

// the next free place of every lane's expert (-1: none wanted), one addition per warp and expert
__device__ __forceinline__ int route_claim(int *next, int expert, int lane) {
    const unsigned same = __match_any_sync(0xffffffffu, expert);
    const int first = __ffs(same) - 1;
    int at = 0;
    if (lane == first && expert >= 0) at = atomicAdd(&next[expert], __popc(same));
    return __shfl_sync(0xffffffffu, at, first) + __popc(same & ((1u << lane) - 1));
}

template <int PER_THREAD, int NJ>
__global__ void __launch_bounds__(1024) route_kernel(const RouteParams p) {
    __shared__ int s_count[RT_MAX_EXPERTS], s_first[RT_MAX_EXPERTS + 1];
    __shared__ uint16_t s_choice[RT_ONE_CTA];
    __shared__ float s_logit[RT_ONE_CTA];
    const int tid = threadIdx.x, lane = tid & 31, NT = blockDim.x, R = p.rows * p.top;
    for (int e = tid; e < p.E; e += NT) s_count[e] = 0;
    route_rows<PER_THREAD, NJ>(p, 0, 1, [&](int pair, int expert, float z) {
        s_choice[pair] = (uint16_t)expert;
        s_logit[pair] = z;
    });
    __syncthreads();
    for (int i0 = 0; i0 < R; i0 += NT) route_claim(s_count, i0 + tid < R ? s_choice[i0 + tid] : -1, lane);
    __syncthreads();
    route_prefix(s_count, s_first, p.E);
    __syncthreads();
    for (int e = tid; e <= p.E; e += NT) p.offsets[e] = s_first[e];
    __syncthreads();
    for (int i0 = 0; i0 < R; i0 += NT) {
        const int i = i0 + tid, at = route_claim(s_first, i < R ? s_choice[i] : -1, lane);
        if (i < R) {
            p.slot[at] = i;
            p.scale[at] = 1.f / (1.f + expf(-s_logit[i]));
        }
    }
}

template <int PER_THREAD, int NJ>
__global__ void __launch_bounds__(256) route_pick_kernel(const RouteParams p) {
    __shared__ int s_count[RT_MAX_EXPERTS];
    const int tid = threadIdx.x;
    int32_t *counts = p.choice + p.rows * p.top;
    for (int e = tid; e < p.E; e += 256) s_count[e] = 0;
    __syncthreads();
    route_rows<PER_THREAD, NJ>(p, blockIdx.x, gridDim.x, [&](int pair, int expert, float z) {
        p.choice[pair] = expert;
        p.weight[pair] = 1.f / (1.f + expf(-z));
        atomicAdd(&s_count[expert], 1);
    });
    __syncthreads();
    for (int e = tid; e < p.E; e += 256)
        if (s_count[e]) atomicAdd(&counts[e], s_count[e]);
}

__global__ void __launch_bounds__(256) route_place_kernel(const RouteParams p, int per_cta) {
    __shared__ int s_count[RT_MAX_EXPERTS], s_first[RT_MAX_EXPERTS + 1];
    const int tid = threadIdx.x, R = p.rows * p.top, lo = blockIdx.x * per_cta, hi = min(R, lo + per_cta);
    const int32_t *counts = p.choice + R;
    int32_t *cursors = p.choice + R + p.E;
    for (int e = tid; e < p.E; e += 256) s_count[e] = counts[e];
    __syncthreads();
    route_prefix(s_count, s_first, p.E);
    __syncthreads();
    if (blockIdx.x == 0)
        for (int e = tid; e <= p.E; e += 256) p.offsets[e] = s_first[e];
    for (int e = tid; e < p.E; e += 256) s_count[e] = 0;
    __syncthreads();
    for (int i0 = lo; i0 < hi; i0 += 256) route_claim(s_count, i0 + tid < hi ? p.choice[i0 + tid] : -1, tid & 31);
    __syncthreads();
    for (int e = tid; e < p.E; e += 256)
        if (s_count[e]) s_first[e] += atomicAdd(&cursors[e], s_count[e]);
    __syncthreads();
    for (int i0 = lo; i0 < hi; i0 += 256) {
        const int i = i0 + tid, at = route_claim(s_first, i < hi ? p.choice[i] : -1, tid & 31);
        if (i < hi) {
            p.slot[at] = i;
            p.scale[at] = p.weight[i];
        }
    }
}

// ------------------------------------------------------------------------------------------------
// few rows
// ------------------------------------------------------------------------------------------------
constexpr int ER_WARPS = 8;
constexpr int ER_TILES = 4;  // column tiles of 8 tokens at a time

template <bool UP>
__global__ void __launch_bounds__(ER_WARPS * 32) expert_rows_kernel(const ExpertParams p) {
    constexpr int ROWS = UP ? 8 : 16, COLS = ER_TILES * 8;
    __shared__ float s_red[ER_WARPS][16][COLS + 1];
    const int e = blockIdx.y, m_lo = p.offsets[e], m_hi = p.offsets[e + 1];
    if (m_lo >= m_hi) return;
    const int n0 = blockIdx.x * ROWS, K = p.K, N = p.N;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tig = lane & 3;
    const __nv_bfloat16 *w = static_cast<const __nv_bfloat16 *>(p.w) + (long long)e * (UP ? 2 : 1) * N * K;
    // weight rows g and g + 8 of the tile: gate and up row of one channel, or two output rows
    const bool ok0 = n0 + g < N, ok1 = UP ? ok0 : n0 + 8 + g < N;
    const __nv_bfloat16 *w0 = w + (long long)(n0 + g) * K, *w1 = w + (long long)(UP ? N + n0 + g : n0 + 8 + g) * K;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    for (int m0 = m_lo; m0 < m_hi; m0 += COLS) {
        const int tiles = min(ER_TILES, (m_hi - m0 + 7) / 8);
        const __nv_bfloat16 *b[ER_TILES];
#pragma unroll
        for (int i = 0; i < ER_TILES; ++i) {
            const int m = min(m0 + i * 8 + g, m_hi - 1);
            b[i] = static_cast<const __nv_bfloat16 *>(p.a) + (long long)(UP ? p.slot[m] / p.top : m) * K;
        }
        float acc[ER_TILES][4];
#pragma unroll
        for (int i = 0; i < ER_TILES; ++i)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[i][c] = 0.f;
#pragma unroll 4
        for (int k = warp * 32 + tig * 8; k < K + tig * 8; k += ER_WARPS * 32) {  // the trip count is the warp's
            const bool in = k < K;
            const uint4 a0 = in && ok0 ? *reinterpret_cast<const uint4 *>(w0 + k) : zero;
            const uint4 a1 = in && ok1 ? *reinterpret_cast<const uint4 *>(w1 + k) : zero;
#pragma unroll
            for (int i = 0; i < ER_TILES; ++i) {
                if (i >= tiles) break;
                const uint4 x = in ? *reinterpret_cast<const uint4 *>(b[i] + k) : zero;
                mma_bf16_16816(acc[i][0], acc[i][1], acc[i][2], acc[i][3], a0.x, a1.x, a0.y, a1.y, x.x, x.y);
                mma_bf16_16816(acc[i][0], acc[i][1], acc[i][2], acc[i][3], a0.z, a1.z, a0.w, a1.w, x.z, x.w);
            }
        }
        __syncthreads();  // the tokens before are written out
#pragma unroll
        for (int i = 0; i < ER_TILES; ++i) {
            if (i >= tiles) break;
            s_red[warp][g][i * 8 + 2 * tig] = acc[i][0];
            s_red[warp][g][i * 8 + 2 * tig + 1] = acc[i][1];
            s_red[warp][g + 8][i * 8 + 2 * tig] = acc[i][2];
            s_red[warp][g + 8][i * 8 + 2 * tig + 1] = acc[i][3];
        }
        __syncthreads();
        for (int i = tid; i < ROWS * tiles * 8; i += ER_WARPS * 32) {
            const int r = i % ROWS, c = i / ROWS, m = m0 + c, n = n0 + r;
            if (m >= m_hi || n >= N) continue;
            float s0 = 0.f, s1 = 0.f;
#pragma unroll
            for (int q = 0; q < ER_WARPS; ++q) {
                s0 += s_red[q][r][c];
                if (UP) s1 += s_red[q][r + 8][c];
            }
            if (UP) {
                const float s = p.scale[m];
                put(static_cast<__nv_bfloat16 *>(p.out) + (long long)m * N + n, Fn<__nv_bfloat16>::silu(s * s0) * (s * s1));
            } else {
                put(static_cast<__nv_bfloat16 *>(p.out) + (long long)p.slot[m] * N + n, s0);
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------
// any size, fp32 sums on the fp32 pipe
// ------------------------------------------------------------------------------------------------
constexpr int EP_TILE = 32;

template <typename T, bool UP>
__global__ void __launch_bounds__(256) expert_plain_kernel(const ExpertParams p) {
    __shared__ float s_a[EP_TILE][EP_TILE + 1], s_w[UP ? 2 : 1][EP_TILE][EP_TILE + 1];
    // the token tile blockIdx.y of all experts' tiles in order
    int e = 0, left = blockIdx.y, m_lo = 0, m_hi = 0;
    for (; e < p.E; ++e) {
        m_lo = p.offsets[e];
        m_hi = p.offsets[e + 1];
        const int tiles = (m_hi - m_lo + EP_TILE - 1) / EP_TILE;
        if (left < tiles) break;
        left -= tiles;
    }
    if (e == p.E) return;
    const int m0 = m_lo + left * EP_TILE, n0 = blockIdx.x * EP_TILE, tid = threadIdx.x, K = p.K, N = p.N;
    const T *w = static_cast<const T *>(p.w) + (long long)e * (UP ? 2 : 1) * N * K;
    const int tx = tid % 16, ty = tid / 16;  // outputs: tokens ty, ty + 16; channels tx, tx + 16
    float acc[UP ? 2 : 1][2][2];
#pragma unroll
    for (int q = 0; q < (UP ? 2 : 1); ++q) acc[q][0][0] = acc[q][0][1] = acc[q][1][0] = acc[q][1][1] = 0.f;
    for (int k0 = 0; k0 < K; k0 += EP_TILE) {
        __syncthreads();
        for (int i = tid; i < EP_TILE * EP_TILE; i += 256) {
            const int r = i / EP_TILE, c = i % EP_TILE, k = k0 + c, m = m0 + r;
            float a = 0.f;
            if (m < m_hi && k < K) a = to_f(static_cast<const T *>(p.a)[(long long)(UP ? p.slot[m] / p.top : m) * K + k]);
            s_a[r][c] = a;
#pragma unroll
            for (int q = 0; q < (UP ? 2 : 1); ++q)
                s_w[q][r][c] = n0 + r < N && k < K ? to_f(w[(long long)(q * N + n0 + r) * K + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < EP_TILE; ++k) {
            const float a0 = s_a[ty][k], a1 = s_a[ty + 16][k];
#pragma unroll
            for (int q = 0; q < (UP ? 2 : 1); ++q) {
                const float w0 = s_w[q][tx][k], w1 = s_w[q][tx + 16][k];
                acc[q][0][0] = fmaf(a0, w0, acc[q][0][0]); acc[q][0][1] = fmaf(a0, w1, acc[q][0][1]);
                acc[q][1][0] = fmaf(a1, w0, acc[q][1][0]); acc[q][1][1] = fmaf(a1, w1, acc[q][1][1]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int m = m0 + ty + 16 * i;
        if (m >= m_hi) continue;
        const float s = UP ? p.scale[m] : 1.f;
        T *out = static_cast<T *>(p.out) + (long long)(UP ? m : p.slot[m]) * N;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int n = n0 + tx + 16 * j;
            if (n >= N) continue;
            if constexpr (UP) put(out + n, Fn<T>::silu(s * acc[0][i][j]) * (s * acc[1][i][j]));
            else put(out + n, acc[0][i][j]);
        }
    }
}

template <typename T>
static cudaError_t expert_plain(const ExpertParams &p, bool up, cudaStream_t s) {
    const dim3 grid((p.N + EP_TILE - 1) / EP_TILE, (p.R + EP_TILE - 1) / EP_TILE + p.E);
    if (up) expert_plain_kernel<T, true><<<grid, 256, 0, s>>>(p);
    else expert_plain_kernel<T, false><<<grid, 256, 0, s>>>(p);
    return cudaGetLastError();
}

// pairs above which the tensor-memory form is used
constexpr int EXPERT_MANY = 32;

}  // namespace nckv

extern "C" {

size_t nckv_route_workspace_bytes(int rows, int E, int top) {
    if (rows <= 0 || E <= 0 || top <= 0 || (long long)rows * top <= nckv::RT_ONE_CTA) return 0;
    return sizeof(int32_t) * (2 * (size_t)rows * top + 2 * (size_t)E);
}

int nckv_route(const float *logits, int32_t *offsets, int32_t *slot, float *scale, int rows, int E, int top, void *workspace,
               size_t workspace_bytes, void *stream) {
    using namespace nckv;
    if (!logits || !offsets || !slot || !scale) {
        set_error("route: null pointer argument");
        return NCKV_E_ARG;
    }
    if (rows <= 0 || E <= 0 || top <= 0 || top > E || E > RT_MAX_EXPERTS || (long long)rows * top > 0x7fffffffLL) {
        set_error("route: size out of range (rows=%d experts=%d top=%d)", rows, E, top);
        return NCKV_E_ARG;
    }
    RouteParams p = {};
    p.logits = logits; p.offsets = offsets; p.slot = slot; p.scale = scale;
    p.rows = rows; p.E = E; p.top = top;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const int R = rows * top;
    if (R <= RT_ONE_CTA) {
        const int warps = R > 992 ? 32 : (R + 31) / 32, row_warps = rows < 32 ? rows : 32;
        if (E <= 8) route_kernel<8, 0><<<1, warps * 32, 0, s>>>(p);
        else if (E <= 16) route_kernel<16, 0><<<1, warps * 32, 0, s>>>(p);
        else if (E <= 32) route_kernel<32, 0><<<1, warps * 32, 0, s>>>(p);
        else if (E <= 64) route_kernel<0, 2><<<1, row_warps * 32, 0, s>>>(p);
        else if (E <= 256) route_kernel<0, 8><<<1, row_warps * 32, 0, s>>>(p);
        else route_kernel<0, 32><<<1, row_warps * 32, 0, s>>>(p);
        NCKV_CUDA_CHECK(cudaGetLastError());
        return NCKV_OK;
    }
    if (!workspace || workspace_bytes < nckv_route_workspace_bytes(rows, E, top)) {
        set_error("route: workspace of %zu bytes given, %zu needed", workspace_bytes, nckv_route_workspace_bytes(rows, E, top));
        return NCKV_E_CAPACITY;
    }
    p.choice = static_cast<int32_t *>(workspace);
    p.weight = reinterpret_cast<float *>(p.choice + R + 2 * E);
    NCKV_CUDA_CHECK(cudaMemsetAsync(p.choice + R, 0, sizeof(int32_t) * 2 * E, s));
    const int want = E <= 32 ? (rows + 255) / 256 : (rows + 7) / 8, grid = want < 4 * sm_count() ? want : 4 * sm_count();
    if (E <= 8) route_pick_kernel<8, 0><<<grid, 256, 0, s>>>(p);
    else if (E <= 16) route_pick_kernel<16, 0><<<grid, 256, 0, s>>>(p);
    else if (E <= 32) route_pick_kernel<32, 0><<<grid, 256, 0, s>>>(p);
    else if (E <= 64) route_pick_kernel<0, 2><<<grid, 256, 0, s>>>(p);
    else if (E <= 256) route_pick_kernel<0, 8><<<grid, 256, 0, s>>>(p);
    else route_pick_kernel<0, 32><<<grid, 256, 0, s>>>(p);
    NCKV_CUDA_CHECK(cudaGetLastError());
    const int per = (R + sm_count() - 1) / sm_count() < 1024 ? 1024 : (R + sm_count() - 1) / sm_count();
    route_place_kernel<<<(R + per - 1) / per, 256, 0, s>>>(p, per);
    NCKV_CUDA_CHECK(cudaGetLastError());
    return NCKV_OK;
}

int nckv_experts(const void *a, const void *w, void *out, const int32_t *offsets, const int32_t *slot, const float *scale, int up,
                 int R, int E, int top, int N, int K, int f32, int32_t *status, void *stream) {
    using namespace nckv;
    if (!a || !w || !out || !offsets || !slot || !status || (up && !scale)) {
        set_error("experts: null pointer argument");
        return NCKV_E_ARG;
    }
    if (R <= 0 || E <= 0 || top <= 0 || N <= 0 || K <= 0 || E > 65535 || R / EP_TILE + E > 65000) {
        set_error("experts: size out of range (R=%d E=%d top=%d N=%d K=%d)", R, E, top, N, K);
        return NCKV_E_ARG;
    }
    ExpertParams p;
    p.a = a; p.w = w; p.out = out; p.offsets = offsets; p.slot = slot; p.scale = scale; p.status = status;
    p.R = R; p.E = E; p.top = top; p.N = N; p.K = K;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (f32) {
        NCKV_CUDA_CHECK(expert_plain<float>(p, up, s));
        return NCKV_OK;
    }
    if (K % 8 || (((uintptr_t)a | (uintptr_t)w) & 15)) {
        NCKV_CUDA_CHECK(expert_plain<__nv_bfloat16>(p, up, s));
        return NCKV_OK;
    }
    if (R > EXPERT_MANY) {
        int rc = NCKV_OK;
        NCKV_CUDA_CHECK(experts_tc(p, up, s, &rc));
        return rc;
    }
    if (up) expert_rows_kernel<true><<<dim3((N + 7) / 8, E), ER_WARPS * 32, 0, s>>>(p);
    else expert_rows_kernel<false><<<dim3((N + 15) / 16, E), ER_WARPS * 32, 0, s>>>(p);
    NCKV_CUDA_CHECK(cudaGetLastError());
    return NCKV_OK;
}

}  // extern "C"
