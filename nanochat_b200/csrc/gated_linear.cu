// Short causal convolutions and the real-gated linear recurrence over channels.
//
//   short_conv_kernel   out_t = act(b + sum_j taps[j] (x_(t - K + 1 + j) + b_in)), per channel, zeros before the
//                       start of a sequence; the last K - 1 inputs of every row are carried in fp32.  A
//                       thread takes a run of tokens of 4 (or 1) channels, all inputs loaded together.
//   gated_scan_kernel   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a_t = -rate r_t and the gates
//                       r, i = sigmoid(logits + bias); out_t = S_t * gelu_tanh(y_t + b_y).  A thread per channel
//                       and segment.  Prompts are cut into segments that run side by side: a first pass
//                       finds each segment's decay product and own contribution, gated_join_kernel chains
//                       them, a second pass runs all segments from their initial states.  How the tokens
//                       are cut changes results at fp32 rounding level only.
#include "vec_io.cuh"

namespace nckv {

// ------------------------------------------------------------------------------------------------
// short causal convolution
// ------------------------------------------------------------------------------------------------
constexpr int CONV_MAX_TAPS = 16;

struct ShortConvParams {
    const void *x;          // (B * T) rows of T, row stride x_stride
    long long x_stride;
    const float *taps;      // (K, C): tap-major
    const float *in_bias, *bias;  // (C) or null
    float *carry;           // (B, K - 1, C)
    void *out;              // (B * T, C) T
    int B, T, C, K, act;
};

// KK: taps of the padded filter (the first KK - K are zero).  RUN tokens per thread, their inputs loaded together.
template <typename T, int V, int KK, int RUN>
__global__ void __launch_bounds__(128) short_conv_kernel(const ShortConvParams p) {
    const int c = (blockIdx.x * 128 + threadIdx.x) * V, b = blockIdx.z;
    if (c >= p.C) return;
    const int t0 = blockIdx.y * RUN, K = p.K, lack = KK - K;
    const T *x = static_cast<const T *>(p.x) + (long long)b * p.T * p.x_stride + c;
    float *carry = p.carry + (long long)b * (K - 1) * p.C + c;
    float in[RUN + KK - 1][V], bi[V], bo[V];  // in[j]: input of token t0 - (KK - 1) + j
#pragma unroll
    for (int e = 0; e < V; ++e) bi[e] = bo[e] = 0.f;
    if (p.in_bias) get_v(p.in_bias + c, bi);
    if (p.bias) get_v(p.bias + c, bo);
    if (t0 >= KK - 1 && t0 + RUN <= p.T) {  // inside the call: nothing stands between the loads
#pragma unroll
        for (int j = 0; j < RUN + KK - 1; ++j) get_v(x + (long long)(t0 - (KK - 1) + j) * p.x_stride, in[j]);
#pragma unroll
        for (int j = 0; j < RUN + KK - 1; ++j)
#pragma unroll
            for (int e = 0; e < V; ++e) in[j][e] = j < lack ? 0.f : in[j][e] + bi[e];
    } else {
#pragma unroll
        for (int j = 0; j < RUN + KK - 1; ++j) {
            const int t = t0 - (KK - 1) + j;
#pragma unroll
            for (int e = 0; e < V; ++e) in[j][e] = 0.f;
            if (j < lack || t >= p.T) continue;
            if (t >= 0) {
                get_v(x + t * p.x_stride, in[j]);
#pragma unroll
                for (int e = 0; e < V; ++e) in[j][e] += bi[e];
            } else {
                get_v(carry + (long long)(K - 1 + t) * p.C, in[j]);  // what is carried has its bias already
            }
        }
    }
    float w[KK][V];
#pragma unroll
    for (int j = 0; j < KK; ++j) {
#pragma unroll
        for (int e = 0; e < V; ++e) w[j][e] = 0.f;
        if (j >= lack) get_v(p.taps + (long long)(j - lack) * p.C + c, w[j]);
    }
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
        if (t0 + i >= p.T) break;
        float o[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
            o[e] = bo[e];
#pragma unroll
            for (int j = 0; j < KK; ++j) o[e] = fmaf(w[j][e], in[i + j][e], o[e]);
            if (p.act) o[e] = Fn<T>::silu(o[e]);
        }
        put_v(static_cast<T *>(p.out) + ((long long)b * p.T + t0 + i) * p.C + c, o);
    }
    if (blockIdx.y > 0) return;
    // Only the first run reads carried inputs (RUN >= KK - 1 where there are several), so it may replace them.
    if (gridDim.y > 1) {
#pragma unroll
        for (int j = 0; j < KK - 1; ++j) {
            if (j >= K - 1) break;
            float last[V];
            get_v(x + (p.T - (K - 1) + j) * p.x_stride, last);
#pragma unroll
            for (int e = 0; e < V; ++e) last[e] += bi[e];
            put_v(carry + (long long)j * p.C, last);
        }
    } else {
#pragma unroll
        for (int j = 1; j < RUN + KK - 1; ++j) {
            const int keep = j - lack - p.T;  // token t0 - (KK - 1) + j is number `keep` of the K - 1 to carry
            if (keep >= 0 && keep < K - 1) put_v(carry + (long long)keep * p.C, in[j]);
        }
    }
}

template <typename T, int V, int KK, int RUN>
static cudaError_t conv_run(const ShortConvParams &p, cudaStream_t s) {
    static_assert(RUN == 1 || RUN >= KK - 1, "one run reads the carried inputs");
    short_conv_kernel<T, V, KK, RUN><<<dim3((p.C + 128 * V - 1) / (128 * V), (p.T + RUN - 1) / RUN, p.B), 128, 0, s>>>(p);
    return cudaGetLastError();
}

template <typename T, int V>
static cudaError_t conv_launch(const ShortConvParams &p, cudaStream_t s) {
    if (p.K <= 2) return p.T == 1 ? conv_run<T, V, 2, 1>(p, s) : conv_run<T, V, 2, 8>(p, s);
    if (p.K <= 4) return p.T == 1 ? conv_run<T, V, 4, 1>(p, s) : conv_run<T, V, 4, 8>(p, s);
    if (p.K <= 8) return p.T == 1 ? conv_run<T, V, 8, 1>(p, s) : conv_run<T, V, 8, 8>(p, s);
    return p.T == 1 ? conv_run<T, V, CONV_MAX_TAPS, 1>(p, s) : conv_run<T, V, CONV_MAX_TAPS, 16>(p, s);
}

// ------------------------------------------------------------------------------------------------
// real-gated linear recurrence
// ------------------------------------------------------------------------------------------------
struct GatedScanParams {
    const void *u, *y;       // (B * T, C) T; y with its own row stride
    long long u_stride, y_stride;
    const float *gates;      // (blocks, B * T, 2 n): logits of r, then of i, of the n channels of a block
    const float *gate_bias;  // (2, C): of r, of i
    const float *y_bias;     // (C)
    const float *rate;       // (C), >= 0
    float *state;            // (B, C)
    void *out;               // (B * T, C) T
    float *parts;            // (B, n_seg, 2, C): own contribution, then initial state; decay product
    int B, T, C, n, n_seg;
};

// decay and drive of one token; sqrt(1 - a^2) from log a, which keeps its digits where a is close to 1
template <typename T> __device__ __forceinline__ void gated_terms(float zr, float zi, float rate, float u, float &a, float &d);
template <> __device__ __forceinline__ void gated_terms<float>(float zr, float zi, float rate, float u, float &a, float &d) {
    const float la = -rate * Fn<float>::sigmoid(zr);
    a = expf(la);
    d = sqrtf(-expm1f(2.f * la)) * Fn<float>::sigmoid(zi) * u;
}
template <> __device__ __forceinline__ void gated_terms<__nv_bfloat16>(float zr, float zi, float rate, float u, float &a, float &d) {
    // both sigmoids with one reciprocal; the cut changes them below 1e-17 only
    const float er = 1.f + __expf(fminf(-zr, 40.f)), ei = 1.f + __expf(fminf(-zi, 40.f)), inv = __fdividef(1.f, er * ei);
    const float la = -rate * (ei * inv), x = -2.f * la;
    a = __expf(la);
    // 1 - e^-x: its series where the difference would cancel (the first term left out is x^6 / 720)
    const float small = x * fmaf(x, fmaf(x, fmaf(x, fmaf(x, 1.f / 120.f, -1.f / 24.f), 1.f / 6.f), -0.5f), 1.f);
    const float y = x < 0.125f ? small : fmaf(-a, a, 1.f);
    d = (y > 0.f ? y * rsqrtf(y) : 0.f) * (er * inv) * u;
}

constexpr int SC_SEG = 32;  // tokens per segment

// SCAN: 0 all tokens of a row from its state (few tokens), 1 a segment's decay product and own contribution,
// 2 a segment's outputs from its initial state.  V consecutive channels per thread, AHEAD tokens loaded together.
template <typename T, int SCAN, int V, int AHEAD>
__global__ void __launch_bounds__(128) gated_scan_kernel(const GatedScanParams p) {
    const int c = (blockIdx.x * 128 + threadIdx.x) * V, b = blockIdx.z, seg = blockIdx.y;
    if (c >= p.C) return;
    const int blk = c / p.n, j = c - blk * p.n;
    float br[V], bi[V], by[V], rate[V];
    get_v(p.gate_bias + c, br);
    get_v(p.gate_bias + p.C + c, bi);
    get_v(p.y_bias + c, by);
    get_v(p.rate + c, rate);
    const int t_begin = SCAN ? seg * SC_SEG : 0, t_end = SCAN ? min(p.T, t_begin + SC_SEG) : p.T;
    const long long row = (long long)b * p.T + t_begin;
    const T *u = static_cast<const T *>(p.u) + row * p.u_stride + c, *y = static_cast<const T *>(p.y) + row * p.y_stride + c;
    const float *g = p.gates + ((long long)blk * p.B * p.T + row) * 2 * p.n + j;
    T *out = static_cast<T *>(p.out) + row * p.C + c;
    float *part = p.parts + ((long long)b * p.n_seg + seg) * 2 * p.C + c;
    float S[V], prod[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
        S[e] = 0.f;
        prod[e] = 1.f;
    }
    if (SCAN == 0) get_v(p.state + (long long)b * p.C + c, S);
    if (SCAN == 2) get_v(part, S);
    for (int left = t_end - t_begin; left > 0; left -= AHEAD) {
        float zr[AHEAD][V], zi[AHEAD][V], uu[AHEAD][V], yy[AHEAD][V];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const long long k = min(i, left - 1);  // past the end: the last token again, not used
            get_v(g + k * 2 * p.n, zr[i]);
            get_v(g + k * 2 * p.n + p.n, zi[i]);
            get_v(u + k * p.u_stride, uu[i]);
            if (SCAN != 1) get_v(y + k * p.y_stride, yy[i]);
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (i >= left) break;
#pragma unroll
            for (int e = 0; e < V; ++e) {
                float a, d;
                gated_terms<T>(zr[i][e] + br[e], zi[i][e] + bi[e], rate[e], uu[i][e], a, d);
                S[e] = fmaf(a, S[e], d);
                if (SCAN == 1) prod[e] *= a;
                else yy[i][e] = S[e] * gelu_tanh<T>(yy[i][e] + by[e]);
            }
            if (SCAN != 1) put_v(out + (long long)i * p.C, yy[i]);
        }
        g += (long long)AHEAD * 2 * p.n;
        u += AHEAD * p.u_stride;
        y += AHEAD * p.y_stride;
        out += (long long)AHEAD * p.C;
    }
    if (SCAN == 0) put_v(p.state + (long long)b * p.C + c, S);
    if (SCAN == 1) {
        put_v(part, S);
        put_v(part + p.C, prod);
    }
}

// every segment's initial state in place of its own contribution, and the row's state after the last
__global__ void __launch_bounds__(64) gated_join_kernel(const GatedScanParams p) {
    const int c = blockIdx.x * 64 + threadIdx.x, b = blockIdx.y;
    if (c >= p.C) return;
    float *part = p.parts + (long long)b * p.n_seg * 2 * p.C + c;
    float S = p.state[(long long)b * p.C + c];
    constexpr int AHEAD = 32;
    for (int s0 = 0; s0 < p.n_seg; s0 += AHEAD) {
        float own[AHEAD], prod[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const long long at = (long long)min(s0 + i, p.n_seg - 1) * 2 * p.C;
            own[i] = part[at];
            prod[i] = part[at + p.C];
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (s0 + i >= p.n_seg) break;
            part[(long long)(s0 + i) * 2 * p.C] = S;
            S = fmaf(prod[i], S, own[i]);
        }
    }
    p.state[(long long)b * p.C + c] = S;
}

static int scan_segments(int T) { return T <= SC_SEG ? 0 : (T + SC_SEG - 1) / SC_SEG; }

template <typename T, int V, int AHEAD>
static cudaError_t scan_launch(const GatedScanParams &p, cudaStream_t s) {
    const unsigned cols = (p.C + 128 * V - 1) / (128 * V);
    if (p.n_seg == 0) {
        gated_scan_kernel<T, 0, V, AHEAD><<<dim3(cols, 1, p.B), 128, 0, s>>>(p);
        return cudaGetLastError();
    }
    gated_scan_kernel<T, 1, V, AHEAD><<<dim3(cols, p.n_seg, p.B), 128, 0, s>>>(p);
    gated_join_kernel<<<dim3((p.C + 63) / 64, p.B), 64, 0, s>>>(p);
    gated_scan_kernel<T, 2, V, AHEAD><<<dim3(cols, p.n_seg, p.B), 128, 0, s>>>(p);
    return cudaGetLastError();
}

template <typename T>
static cudaError_t scan_any(const GatedScanParams &p, cudaStream_t s) {
    const uintptr_t elem = sizeof(T);
    const uintptr_t a32 = (uintptr_t)p.gates | (uintptr_t)p.gate_bias | (uintptr_t)p.y_bias | (uintptr_t)p.rate | (uintptr_t)p.state |
                          (uintptr_t)p.parts;
    const uintptr_t at = (uintptr_t)p.u | (uintptr_t)p.y | (uintptr_t)p.out | (uintptr_t)(p.u_stride | p.y_stride) * elem;
    // wide accesses where enough threads are left
    const bool vec = p.n % 4 == 0 && (a32 & 15) == 0 && (at & (4 * elem - 1)) == 0;
    const bool many = p.n_seg == 0 || (long long)p.B * p.C * p.n_seg >= 4096LL * sm_count();
    if (vec && many) return scan_launch<T, 4, 4>(p, s);
    return scan_launch<T, 1, 8>(p, s);
}

}  // namespace nckv

extern "C" {

int nckv_short_conv(const void *x, int64_t x_stride, const float *taps, const float *in_bias, const float *bias, float *carry,
                    void *out, int B, int T, int C, int K, int act, int f32, void *stream) {
    using namespace nckv;
    if (!x || !taps || !out || (K > 1 && !carry)) {
        set_error("short_conv: null pointer argument");
        return NCKV_E_ARG;
    }
    if (B <= 0 || T <= 0 || C <= 0 || K <= 0 || B > 65535 || T > 65535 * 8) {
        set_error("short_conv: size out of range (B=%d T=%d C=%d K=%d)", B, T, C, K);
        return NCKV_E_ARG;
    }
    if (K > CONV_MAX_TAPS) {
        set_error("short_conv: %d taps unsupported (at most %d)", K, CONV_MAX_TAPS);
        return NCKV_E_UNSUPPORTED;
    }
    ShortConvParams p;
    p.x = x; p.x_stride = x_stride; p.taps = taps; p.in_bias = in_bias; p.bias = bias; p.carry = carry; p.out = out;
    p.B = B; p.T = T; p.C = C; p.K = K; p.act = act;
    const uintptr_t elem = f32 ? 4 : 2;
    const uintptr_t a32 = (uintptr_t)taps | (uintptr_t)in_bias | (uintptr_t)bias | (uintptr_t)carry;
    const uintptr_t at = (uintptr_t)x | (uintptr_t)out | (uintptr_t)x_stride * elem;
    const bool vec = C % 4 == 0 && (a32 & 15) == 0 && (at & (4 * elem - 1)) == 0;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    cudaError_t e;
    if (f32) e = vec ? conv_launch<float, 4>(p, s) : conv_launch<float, 1>(p, s);
    else e = vec ? conv_launch<__nv_bfloat16, 4>(p, s) : conv_launch<__nv_bfloat16, 1>(p, s);
    NCKV_CUDA_CHECK(e);
    return NCKV_OK;
}

size_t nckv_gated_scan_workspace_bytes(int B, int T, int C) {
    if (B <= 0 || T <= 0 || C <= 0) return 0;
    return sizeof(float) * 2 * (size_t)B * nckv::scan_segments(T) * C;
}

int nckv_gated_scan(const void *u, int64_t u_stride, const void *y, int64_t y_stride, const float *gates, const float *gate_bias,
                    const float *y_bias, const float *rate, float *state, void *out, int B, int T, int C, int blocks, int f32,
                    void *workspace, size_t workspace_bytes, void *stream) {
    using namespace nckv;
    if (!u || !y || !gates || !gate_bias || !y_bias || !rate || !state || !out) {
        set_error("gated_scan: null pointer argument");
        return NCKV_E_ARG;
    }
    if (B <= 0 || T <= 0 || C <= 0 || B > 65535 || blocks <= 0 || C % blocks) {
        set_error("gated_scan: size out of range (B=%d T=%d C=%d blocks=%d)", B, T, C, blocks);
        return NCKV_E_ARG;
    }
    if (scan_segments(T) > 65535 || (scan_segments(T) && (!workspace || workspace_bytes < nckv_gated_scan_workspace_bytes(B, T, C)))) {
        set_error("gated_scan: workspace of %zu bytes given, %zu needed", workspace_bytes, nckv_gated_scan_workspace_bytes(B, T, C));
        return NCKV_E_CAPACITY;
    }
    GatedScanParams p;
    p.u = u; p.y = y; p.u_stride = u_stride; p.y_stride = y_stride;
    p.gates = gates; p.gate_bias = gate_bias; p.y_bias = y_bias; p.rate = rate; p.state = state; p.out = out;
    p.parts = static_cast<float *>(workspace);
    p.B = B; p.T = T; p.C = C; p.n = C / blocks; p.n_seg = scan_segments(T);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    NCKV_CUDA_CHECK(f32 ? scan_any<float>(p, s) : scan_any<__nv_bfloat16>(p, s));
    return NCKV_OK;
}

}  // extern "C"
