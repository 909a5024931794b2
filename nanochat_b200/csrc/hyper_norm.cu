// The step between two sublayers of a trunk with hyper-connections: instead of one residual stream there are
// S of them, mixed with each other around every sublayer.  T is the element type of activations (bf16, or
// fp32 for the exact mode); the streams, the mixing and the norm are fp32.
//
//   hyper_norm_kernel   y  = sum of the `parts` rows the last sublayer left for this token
//                       x_t' = sum_s M[s, t] x_s + o[t] y    (start of the trunk: x_t' = table[token])
//                       u  = sum_t g[t] x_t'                 (g null: the plain sum)
//                       h  = T((u - mean) / sqrt(var + eps) * w)
//
// One CTA per token.  A thread takes V consecutive channels at a time of all streams, so the mixing needs no
// exchange between threads; u stays in registers for the two reductions of the norm.
#include "vec_io.cuh"

namespace nckv {

constexpr int HN_MAX_THREADS = 512;
constexpr int HN_MAX_STREAMS = 8;

struct HyperNormParams {
    const float *x;            // (rows, S, W), or null when tokens are given
    const int64_t *tokens;     // (rows) ids into table
    const void *table;         // (vocab, W) T
    const void *y;             // (rows, parts, W) T, or null (streams pass as they are)
    const float *mix, *out;    // (S, S) from, to; (S)
    const float *in;           // (S) or null
    const float *w;            // (W)
    float *x_out;              // (rows, S, W), may be x; or null
    void *h;                   // (rows, W) T
    int rows, S, W, parts, vocab;
    float eps;
};

// sum over the CTA; s_part: one float per warp
__device__ __forceinline__ float cta_sum(float v, float *s_part) {
#pragma unroll
    for (int off = 16; off; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) s_part[threadIdx.x >> 5] = v;
    __syncthreads();
    const int lane = threadIdx.x & 31, n = blockDim.x >> 5;
    float t = lane < n ? s_part[lane] : 0.f;
#pragma unroll
    for (int off = 16; off; off >>= 1) t += __shfl_xor_sync(0xffffffffu, t, off);
    return t;
}

// NV pieces of V channels per thread: W <= NV * V * threads.  SM: streams held (S <= SM)
template <typename T, int V, int NV, int SM>
__global__ void __launch_bounds__(HN_MAX_THREADS) hyper_norm_kernel(const HyperNormParams p) {
    __shared__ float s_part[HN_MAX_THREADS / 32];
    __shared__ float s_mix[HN_MAX_STREAMS * HN_MAX_STREAMS], s_out[HN_MAX_STREAMS], s_in[HN_MAX_STREAMS];
    const int tid = threadIdx.x, NT = blockDim.x, S = p.S;
    const long long row = blockIdx.x;
    if (tid < S) {
        s_out[tid] = p.y ? p.out[tid] : 0.f;
        s_in[tid] = p.in ? p.in[tid] : 1.f;
    }
    for (int i = tid; i < S * S; i += NT) s_mix[i] = p.y ? p.mix[i] : 0.f;
    __syncthreads();
    long long id = 0;
    if (p.tokens) {
        id = p.tokens[row];
        id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    }
    float u[NV][V], sum = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (k * NT + tid) * V;
#pragma unroll
        for (int e = 0; e < V; ++e) u[k][e] = 0.f;
        if (c >= p.W) continue;
        float x[SM][V], y[V];
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = 0.f;
        if (p.tokens) {
            float e0[V];
            get_v(static_cast<const T *>(p.table) + id * p.W + c, e0);
#pragma unroll
            for (int s = 0; s < SM; ++s)
#pragma unroll
                for (int e = 0; e < V; ++e) x[s][e] = e0[e];
        } else {
#pragma unroll
            for (int s = 0; s < SM; ++s)
                if (s < S) get_v(p.x + (row * S + s) * p.W + c, x[s]);
        }
        if (p.y) {
            for (int j = 0; j < p.parts; ++j) {
                float one[V];
                get_v(static_cast<const T *>(p.y) + (row * p.parts + j) * p.W + c, one);
#pragma unroll
                for (int e = 0; e < V; ++e) y[e] += one[e];
            }
        }
#pragma unroll
        for (int t = 0; t < SM; ++t) {
            if (t >= S) break;
            float n[V];
            if (p.y) {
#pragma unroll
                for (int e = 0; e < V; ++e) n[e] = s_out[t] * y[e];
#pragma unroll
                for (int s = 0; s < SM; ++s) {
                    if (s >= S) break;
                    const float m = s_mix[s * S + t];
#pragma unroll
                    for (int e = 0; e < V; ++e) n[e] = fmaf(m, x[s][e], n[e]);
                }
            } else {
#pragma unroll
                for (int e = 0; e < V; ++e) n[e] = x[t][e];
            }
            if (p.x_out) put_v(p.x_out + (row * S + t) * p.W + c, n);
            const float g = s_in[t];
#pragma unroll
            for (int e = 0; e < V; ++e) u[k][e] = fmaf(g, n[e], u[k][e]);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) sum += u[k][e];
    }
    const float mean = cta_sum(sum, s_part) / (float)p.W;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        if ((k * NT + tid) * V >= p.W) continue;
#pragma unroll
        for (int e = 0; e < V; ++e) {
            u[k][e] -= mean;
            ss = fmaf(u[k][e], u[k][e], ss);
        }
    }
    const float inv = 1.f / sqrtf(cta_sum(ss, s_part) / (float)p.W + p.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (k * NT + tid) * V;
        if (c >= p.W) continue;
        float w[V], o[V];
        get_v(p.w + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = u[k][e] * inv * w[e];
        put_v(static_cast<T *>(p.h) + row * p.W + c, o);
    }
}

template <typename T, int V, int NV>
static cudaError_t hn_launch_streams(const HyperNormParams &p, int threads, cudaStream_t s) {
    if (p.S <= 2) hyper_norm_kernel<T, V, NV, 2><<<p.rows, threads, 0, s>>>(p);
    else if (p.S <= 4) hyper_norm_kernel<T, V, NV, 4><<<p.rows, threads, 0, s>>>(p);
    else hyper_norm_kernel<T, V, NV, HN_MAX_STREAMS><<<p.rows, threads, 0, s>>>(p);
    return cudaGetLastError();
}

template <typename T, int V>
static cudaError_t hn_launch(const HyperNormParams &p, cudaStream_t s) {
    const int pieces = (p.W + V - 1) / V;
    auto threads_for = [&](int nv) { return ((pieces + nv - 1) / nv + 31) / 32 * 32; };
    if (pieces <= HN_MAX_THREADS) return hn_launch_streams<T, V, 1>(p, threads_for(1), s);
    if (pieces <= 2 * HN_MAX_THREADS) return hn_launch_streams<T, V, 2>(p, threads_for(2), s);
    if (pieces <= 4 * HN_MAX_THREADS) return hn_launch_streams<T, V, 4>(p, threads_for(4), s);
    return hn_launch_streams<T, V, 16>(p, threads_for(16), s);
}

}  // namespace nckv

extern "C" int nckv_hyper_norm(const float *x, const int64_t *tokens, const void *table, int vocab, const void *y, int parts,
                               const float *mix, const float *out, const float *in, const float *w, float *x_out, void *h,
                               int rows, int S, int W, float eps, int f32, void *stream) {
    using namespace nckv;
    if ((!x && !tokens) || (tokens && (!table || vocab <= 0)) || (y && (!mix || !out || parts <= 0)) || !w || !h) {
        set_error("hyper_norm: missing operand");
        return NCKV_E_ARG;
    }
    if (rows <= 0 || W <= 0 || S <= 0) {
        set_error("hyper_norm: size out of range (rows=%d S=%d W=%d)", rows, S, W);
        return NCKV_E_ARG;
    }
    const uintptr_t elem = f32 ? 4 : 2;
    const uintptr_t a32 = (uintptr_t)x | (uintptr_t)w | (uintptr_t)x_out, at = (uintptr_t)table | (uintptr_t)h | (uintptr_t)y;
    const bool vec = W % 4 == 0 && (a32 & 15) == 0 && (at & (4 * elem - 1)) == 0;
    if (S > HN_MAX_STREAMS || W > (vec ? 4 : 1) * 16 * HN_MAX_THREADS) {
        set_error("hyper_norm: S=%d W=%d unsupported (at most %d streams of %d)", S, W, HN_MAX_STREAMS, (vec ? 4 : 1) * 16 * HN_MAX_THREADS);
        return NCKV_E_UNSUPPORTED;
    }
    HyperNormParams p;
    p.x = x; p.tokens = tokens; p.table = table; p.y = y; p.mix = mix; p.out = out; p.in = in; p.w = w;
    p.x_out = x_out; p.h = h;
    p.rows = rows; p.S = S; p.W = W; p.parts = parts; p.vocab = vocab; p.eps = eps;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    cudaError_t e;
    if (f32) e = vec ? hn_launch<float, 4>(p, s) : hn_launch<float, 1>(p, s);
    else e = vec ? hn_launch<__nv_bfloat16, 4>(p, s) : hn_launch<__nv_bfloat16, 1>(p, s);
    NCKV_CUDA_CHECK(e);
    return NCKV_OK;
}
