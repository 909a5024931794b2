// Elementwise steps around the matrix products of a trunk with a 32-bit residual stream and norms on
// the sublayers' outputs.  T is the element type of activations (bf16, or fp32 for the exact mode);
// the stream x and all norms are fp32.
//
//   resid_norm_kernel   x' = x + y / rms(y) * w          or  x' = table[token]         (start of the trunk)
//                       then any of
//                         h    = T(x')                                                  next sublayer's input
//                         h    = T(x' / rms(x') * wf)                                   last norm
//                         mixM = T(x' + (before - x') * mu_M), M < n_mix                token shift
//                       where `before` is the previous token's x' (the row's carried vector for the
//                       first token of a call).  A CTA walks `run` consecutive tokens of a row and keeps
//                       the last one in registers; for its first token it recomputes the one before it,
//                       so the shift needs no second pass over the stream.
//   silu_mul_kernel     out = T(silu(gate) * up) over rows [gate | up]
//   tanh_split_kernel   tanh of a fp32 row as bf16 hi | lo halves (their sum carries 16 bits), or as fp32
//   softcap_kernel      cap * tanh(z / cap), fp32 in place
#include "vec_io.cuh"

namespace nckv {

constexpr int RN_THREADS = 256;
constexpr int MAX_MIX = 8;

struct ResidNormParams {
    const float *x;            // (rows, W) or null when tokens are given
    const void *y;             // (rows, W) T or fp32, or null
    const float *w;            // (W) weight of y's norm
    const int64_t *tokens;     // start of the trunk: (rows) ids into table
    const void *table;         // (vocab, W) T
    float *x_out;              // (rows, W) or null
    void *h;                   // (rows, W) T or null
    const float *final_w;      // (W): h is the normed stream
    void *mix;                 // (n_mix, rows, W) T or null
    const float *mu;           // (n_mix, W)
    float *carry;              // (B, W) the stream of the row's previous token
    int B, T, W, run, n_mix, vocab;
    float eps;
};

__device__ __forceinline__ float block_sum(float v, float *s_part) {
#pragma unroll
    for (int off = 16; off; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) s_part[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = s_part[threadIdx.x & (RN_THREADS / 32 - 1)];
#pragma unroll
    for (int off = RN_THREADS / 64; off; off >>= 1) t += __shfl_xor_sync(0xffffffffu, t, off);
    return t;
}

// NV pieces of V channels per thread: W <= NV * V * RN_THREADS
template <typename T, typename TY, int V, int NV>
__global__ void __launch_bounds__(RN_THREADS) resid_norm_kernel(const ResidNormParams p) {
    __shared__ float s_part[RN_THREADS / 32];
    const int b = blockIdx.y, t0 = blockIdx.x * p.run, t1 = min(p.T, t0 + p.run);
    const int tid = threadIdx.x;
    float cur[NV][V], prev[NV][V];

    auto load_row = [&](long long row, float (&o)[NV][V]) {
        if (p.tokens) {
            long long id = p.tokens[row];
            id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
            const T *src = static_cast<const T *>(p.table) + id * p.W;
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const int c = (k * RN_THREADS + tid) * V;
                if (c < p.W) get_v(src + c, o[k]);
            }
            return;
        }
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = (k * RN_THREADS + tid) * V;
            if (c < p.W) get_v(p.x + row * p.W + c, o[k]);
        }
        if (!p.y) return;
        float y[NV][V], ss = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = (k * RN_THREADS + tid) * V;
            if (c < p.W) {
                get_v(static_cast<const TY *>(p.y) + row * p.W + c, y[k]);
#pragma unroll
                for (int e = 0; e < V; ++e) ss = fmaf(y[k][e], y[k][e], ss);
            }
        }
        const float inv = rsqrtf(block_sum(ss, s_part) / (float)p.W + p.eps);
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = (k * RN_THREADS + tid) * V;
            if (c < p.W) {
                float w[V];
                get_v(p.w + c, w);
#pragma unroll
                for (int e = 0; e < V; ++e) o[k][e] = fmaf(y[k][e] * inv, w[e], o[k][e]);
            }
        }
    };

    if (p.mix) {
        if (t0 > 0) {
            load_row((long long)b * p.T + t0 - 1, prev);
        } else {
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const int c = (k * RN_THREADS + tid) * V;
                if (c < p.W) get_v(p.carry + (long long)b * p.W + c, prev[k]);
            }
        }
    }
    for (int t = t0; t < t1; ++t) {
        const long long row = (long long)b * p.T + t;
        load_row(row, cur);
        float inv_f = 0.f;
        if (p.final_w) {
            float ss = 0.f;
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                if ((k * RN_THREADS + tid) * V < p.W) {
#pragma unroll
                    for (int e = 0; e < V; ++e) ss = fmaf(cur[k][e], cur[k][e], ss);
                }
            }
            inv_f = rsqrtf(block_sum(ss, s_part) / (float)p.W + p.eps);
        }
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = (k * RN_THREADS + tid) * V;
            if (c >= p.W) continue;
            if (p.x_out) put_v(p.x_out + row * p.W + c, cur[k]);
            if (p.h) {
                float o[V];
                if (p.final_w) {
                    float w[V];
                    get_v(p.final_w + c, w);
#pragma unroll
                    for (int e = 0; e < V; ++e) o[e] = cur[k][e] * inv_f * w[e];
                } else {
#pragma unroll
                    for (int e = 0; e < V; ++e) o[e] = cur[k][e];
                }
                put_v(static_cast<T *>(p.h) + row * p.W + c, o);
            }
            if (p.mix) {
                const long long plane = (long long)p.B * p.T * p.W;
#pragma unroll 5
                for (int m = 0; m < p.n_mix; ++m) {
                    float mu[V], o[V];
                    get_v(p.mu + (long long)m * p.W + c, mu);
#pragma unroll
                    for (int e = 0; e < V; ++e) o[e] = fmaf(prev[k][e] - cur[k][e], mu[e], cur[k][e]);
                    put_v(static_cast<T *>(p.mix) + m * plane + row * p.W + c, o);
                }
                // a single-token call carries the vector on here (the thread that read it writes it);
                // longer calls copy their last row afterwards
                if (p.T == 1) put_v(p.carry + (long long)b * p.W + c, cur[k]);
#pragma unroll
                for (int e = 0; e < V; ++e) prev[k][e] = cur[k][e];
            }
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(256) silu_mul_kernel(const T *__restrict__ in, T *__restrict__ out, long long rows, int F, int vec) {
    const long long step = (long long)gridDim.x * blockDim.x;
    if (vec) {
        // 8 channels at a time, a row per CTA turn
        const int per_row = F / 8, blocks_per_row = (per_row + 255) / 256;
        const long long n = rows * blocks_per_row;
        for (long long i = blockIdx.x; i < n; i += gridDim.x) {
            const long long row = i / blocks_per_row;
            const int c = ((int)(i - row * blocks_per_row) * 256 + threadIdx.x) * 8;
            if (c >= F) continue;
            float g[8], u[8], o[8];
            get_v(in + row * 2 * F + c, g);
            get_v(in + row * 2 * F + F + c, u);
#pragma unroll
            for (int e = 0; e < 8; ++e)
                o[e] = (sizeof(T) == 2 ? __fdividef(g[e], 1.f + __expf(-g[e])) : g[e] / (1.f + expf(-g[e]))) * u[e];
            put_v(out + row * F + c, o);
        }
    } else {
        const long long n = rows * F;
        for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += step) {
            const long long row = i / F;
            const int c = (int)(i - row * F);
            const float g = to_f(in[row * 2 * F + c]), u = to_f(in[row * 2 * F + F + c]);
            put(out + i, g / (1.f + expf(-g)) * u);
        }
    }
}

// z (rows, R) fp32 -> out: fp32 (rows, R), or bf16 (rows, 2 R) holding hi then lo
__global__ void __launch_bounds__(256) tanh_split_kernel(const float *__restrict__ z, void *__restrict__ out, long long rows, int R, int f32) {
    const long long n = rows * R;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        const float v = tanhf(z[i]);
        if (f32) {
            static_cast<float *>(out)[i] = v;
        } else {
            const long long row = i / R;
            const int c = (int)(i - row * R);
            const float hi = round_bf16(v);
            __nv_bfloat16 *dst = static_cast<__nv_bfloat16 *>(out) + row * 2 * R + c;
            dst[0] = __float2bfloat16_rn(hi);
            dst[R] = __float2bfloat16_rn(v - hi);
        }
    }
}

__global__ void __launch_bounds__(256) softcap_kernel(float *z, long long n, float cap) {
    const long long step = (long long)gridDim.x * blockDim.x, first = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const long long quads = (((uintptr_t)z) & 15) == 0 ? n / 4 : 0;
    for (long long i = first; i < quads; i += step) {
        float4 f = reinterpret_cast<float4 *>(z)[i];
        f.x = cap * tanhf(f.x / cap); f.y = cap * tanhf(f.y / cap);
        f.z = cap * tanhf(f.z / cap); f.w = cap * tanhf(f.w / cap);
        reinterpret_cast<float4 *>(z)[i] = f;
    }
    for (long long i = quads * 4 + first; i < n; i += step) z[i] = cap * tanhf(z[i] / cap);
}

static unsigned grid_for(long long n) {
    long long blocks = (n + 255) / 256;
    const long long cap = (long long)sm_count() * 16;
    return (unsigned)(blocks < 1 ? 1 : (blocks > cap ? cap : blocks));
}

template <typename T, typename TY, int V>
static cudaError_t rn_launch(const ResidNormParams &p, cudaStream_t s) {
    const dim3 grid((p.T + p.run - 1) / p.run, p.B);
    const int per = (p.W + V * RN_THREADS - 1) / (V * RN_THREADS);
    if (per <= 1) resid_norm_kernel<T, TY, V, 1><<<grid, RN_THREADS, 0, s>>>(p);
    else if (per <= 2) resid_norm_kernel<T, TY, V, 2><<<grid, RN_THREADS, 0, s>>>(p);
    else if (per <= 4) resid_norm_kernel<T, TY, V, 4><<<grid, RN_THREADS, 0, s>>>(p);
    else resid_norm_kernel<T, TY, V, 8><<<grid, RN_THREADS, 0, s>>>(p);
    return cudaGetLastError();
}

}  // namespace nckv

extern "C" {

int nckv_resid_norm(const float *x, const void *y, int y_f32, const float *w, const int64_t *tokens, const void *table,
                    int vocab, float *x_out, void *h, const float *final_w, void *mix, const float *mu, int n_mix,
                    float *carry, int B, int T, int W, float eps, int f32, void *stream) {
    using namespace nckv;
    if ((!x && !tokens) || (tokens && (!table || vocab <= 0)) || (y && !w) || (!x_out && !h && !mix) ||
        (mix && (!mu || !carry || !x_out || n_mix <= 0 || n_mix > MAX_MIX)) || (final_w && !h)) {
        set_error("resid_norm: missing operand");
        return NCKV_E_ARG;
    }
    if (B <= 0 || T <= 0 || W <= 0 || B > 65535) {
        set_error("resid_norm: size out of range (B=%d T=%d W=%d)", B, T, W);
        return NCKV_E_ARG;
    }
    if (mix && x_out == x) {
        set_error("resid_norm: the token shift reads neighbouring rows, so x_out must not alias x");
        return NCKV_E_ARG;
    }
    const uintptr_t elem = f32 ? 4 : 2;
    const uintptr_t a32 = (uintptr_t)x | (uintptr_t)w | (uintptr_t)x_out | (uintptr_t)final_w | (uintptr_t)mu | (uintptr_t)carry |
                          (y_f32 ? (uintptr_t)y : 0);
    const uintptr_t at = (uintptr_t)table | (uintptr_t)h | (uintptr_t)mix | (y_f32 ? 0 : (uintptr_t)y);
    const bool vec = W % 4 == 0 && (a32 & 15) == 0 && (at & (4 * elem - 1)) == 0;
    if (W > (vec ? 4 : 1) * 8 * RN_THREADS) {
        set_error("resid_norm: W=%d unsupported (at most %d)", W, (vec ? 4 : 1) * 8 * RN_THREADS);
        return NCKV_E_UNSUPPORTED;
    }
    ResidNormParams p;
    p.x = x; p.y = y; p.w = w; p.tokens = tokens; p.table = table; p.x_out = x_out; p.h = h; p.final_w = final_w;
    p.mix = mix; p.mu = mu; p.carry = carry;
    p.B = B; p.T = T; p.W = W; p.n_mix = n_mix; p.vocab = vocab; p.eps = eps;
    // longer runs save the recomputed row; short prompts keep the grid full instead
    p.run = 1;
    if (mix) while (p.run < 8 && (long long)B * T >= 2LL * p.run * 8 * sm_count()) p.run *= 2;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    cudaError_t e;
    if (f32) e = vec ? rn_launch<float, float, 4>(p, s) : rn_launch<float, float, 1>(p, s);
    else if (y_f32) e = vec ? rn_launch<__nv_bfloat16, float, 4>(p, s) : rn_launch<__nv_bfloat16, float, 1>(p, s);
    else e = vec ? rn_launch<__nv_bfloat16, __nv_bfloat16, 4>(p, s) : rn_launch<__nv_bfloat16, __nv_bfloat16, 1>(p, s);
    NCKV_CUDA_CHECK(e);
    if (mix && T > 1)
        NCKV_CUDA_CHECK(cudaMemcpy2DAsync(carry, sizeof(float) * W, x_out + (long long)(T - 1) * W, sizeof(float) * W * (size_t)T,
                                          sizeof(float) * W, B, cudaMemcpyDeviceToDevice, s));
    return NCKV_OK;
}

int nckv_silu_mul(const void *gate_up, void *out, int64_t rows, int F, int f32, void *stream) {
    using namespace nckv;
    if (!gate_up || !out || rows <= 0 || F <= 0) {
        set_error("silu_mul: null pointer or non-positive size");
        return NCKV_E_ARG;
    }
    const int vec = F % 8 == 0 && (((uintptr_t)gate_up | (uintptr_t)out) & 15) == 0;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const unsigned grid = vec ? grid_for(rows * ((F / 8 + 255) / 256) * 256) : grid_for(rows * F);
    if (f32) silu_mul_kernel<float><<<grid, 256, 0, s>>>(static_cast<const float *>(gate_up), static_cast<float *>(out), rows, F, vec);
    else silu_mul_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(static_cast<const __nv_bfloat16 *>(gate_up), static_cast<__nv_bfloat16 *>(out), rows, F, vec);
    NCKV_CUDA_CHECK(cudaGetLastError());
    return NCKV_OK;
}

int nckv_tanh_split(const float *z, void *out, int64_t rows, int R, int f32, void *stream) {
    using namespace nckv;
    if (!z || !out || rows <= 0 || R <= 0) {
        set_error("tanh_split: null pointer or non-positive size");
        return NCKV_E_ARG;
    }
    tanh_split_kernel<<<grid_for(rows * R), 256, 0, static_cast<cudaStream_t>(stream)>>>(z, out, rows, R, f32);
    NCKV_CUDA_CHECK(cudaGetLastError());
    return NCKV_OK;
}

int nckv_softcap(float *z, int64_t n, float cap, void *stream) {
    using namespace nckv;
    if (!z || n <= 0 || !(cap > 0.f)) {
        set_error("softcap: null pointer, non-positive size or cap");
        return NCKV_E_ARG;
    }
    softcap_kernel<<<grid_for((n + 3) / 4), 256, 0, static_cast<cudaStream_t>(stream)>>>(z, n, cap);
    NCKV_CUDA_CHECK(cudaGetLastError());
    return NCKV_OK;
}

}  // extern "C"
