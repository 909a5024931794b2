// Short causal convolutions and the real-gated linear recurrence over channels.
//
//   short_conv_kernel   out_t = act(b + sum_j taps[j] (x_(t - K + 1 + j) + b_in)), per channel, zeros before the
//                       start of a sequence; the last K - 1 inputs of every row are carried in fp32.  A
//                       thread slides over a run of tokens of 4 (or 1) channels with the inputs in registers.
//   conv_carry_kernel   the carried inputs after a call of more than one run
//   gated_scan_kernel   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a_t = -rate r_t and the gates
//                       r, i = sigmoid(logits + bias); out_t = S_t * gelu_tanh(y_t + b_y).  A CTA owns L
//                       channels of one row; its warps (or half-warps) take SC_TOKENS consecutive tokens each,
//                       find their own decay product and contribution, chain them through shared memory and
//                       run through their tokens again from the right initial state (operands stay in
//                       registers, so global memory is read once).
//   gated_scan_step_kernel   the same for few tokens: a thread per channel, one token after the other.
#include "vec_io.cuh"

namespace nckv {

// ------------------------------------------------------------------------------------------------
// short causal convolution
// ------------------------------------------------------------------------------------------------
constexpr int CONV_RUN = 16;
constexpr int CONV_MAX_TAPS = 16;

struct ShortConvParams {
    const void *x;          // (B * T) rows of T, row stride x_stride
    long long x_stride;
    const float *taps;      // (K, C): tap-major
    const float *in_bias, *bias;  // (C) or null
    float *carry;           // (B, K - 1, C)
    void *out;              // (B * T, C) T
    int B, T, C, K, run, act;
};

template <typename T, int V, int KK>
__global__ void __launch_bounds__(128) short_conv_kernel(const ShortConvParams p) {
    const int c = (blockIdx.x * 128 + threadIdx.x) * V, b = blockIdx.z;
    if (c >= p.C) return;
    const int t0 = blockIdx.y * p.run, t1 = min(p.T, t0 + p.run);
    const int K = p.K, lack = KK - K;  // the first `lack` taps of the padded filter are zero
    float w[KK][V], win[KK][V], bi[V], bo[V];
#pragma unroll
    for (int e = 0; e < V; ++e) bi[e] = bo[e] = 0.f;
    if (p.in_bias) get_v(p.in_bias + c, bi);
    if (p.bias) get_v(p.bias + c, bo);
    const T *x = static_cast<const T *>(p.x) + (long long)b * p.T * p.x_stride + c;
    float *carry = p.carry + (long long)b * (K - 1) * p.C + c;
    auto input = [&](int t, float (&o)[V]) {  // input of token t of this call; before it: what is carried
        if (t >= 0) {
            get_v(x + t * p.x_stride, o);
#pragma unroll
            for (int e = 0; e < V; ++e) o[e] += bi[e];
        } else {
            get_v(carry + (long long)(K - 1 + t) * p.C, o);
        }
    };
#pragma unroll
    for (int j = 0; j < KK; ++j) {
#pragma unroll
        for (int e = 0; e < V; ++e) w[j][e] = win[j][e] = 0.f;
        if (j >= lack) get_v(p.taps + (long long)(j - lack) * p.C + c, w[j]);
        if (j >= lack && j < KK - 1) input(t0 - (KK - 1) + j, win[j]);
    }
    for (int t = t0; t < t1; ++t) {
        input(t, win[KK - 1]);
        float o[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
            o[e] = bo[e];
#pragma unroll
            for (int j = 0; j < KK; ++j) o[e] = fmaf(w[j][e], win[j][e], o[e]);
            if (p.act) o[e] = Fn<T>::silu(o[e]);
        }
        put_v(static_cast<T *>(p.out) + ((long long)b * p.T + t) * p.C + c, o);
#pragma unroll
        for (int j = 0; j < KK - 1; ++j)
#pragma unroll
            for (int e = 0; e < V; ++e) win[j][e] = win[j + 1][e];
    }
    if (p.run >= p.T) {  // the only run of its row: nobody else reads the carried inputs
#pragma unroll
        for (int j = 0; j < KK - 1; ++j)
            if (j >= lack) put_v(carry + (long long)(j - lack) * p.C, win[j]);
    }
}

// after a call of T >= K - 1 tokens
template <typename T>
__global__ void __launch_bounds__(256) conv_carry_kernel(const ShortConvParams p) {
    const int c = blockIdx.x * 256 + threadIdx.x, j = blockIdx.y, b = blockIdx.z;
    if (c >= p.C) return;
    const long long t = (long long)b * p.T + p.T - (p.K - 1) + j;
    p.carry[((long long)b * (p.K - 1) + j) * p.C + c] =
        to_f(static_cast<const T *>(p.x)[t * p.x_stride + c]) + (p.in_bias ? p.in_bias[c] : 0.f);
}

template <typename T, int V>
static cudaError_t conv_launch(ShortConvParams p, cudaStream_t s) {
    // runs long enough to make the K - 1 inputs read again cheap; short calls in one run
    p.run = p.T <= CONV_RUN ? p.T : CONV_RUN;
    const dim3 grid((p.C + 128 * V - 1) / (128 * V), (p.T + p.run - 1) / p.run, p.B);
    if (p.K <= 2) short_conv_kernel<T, V, 2><<<grid, 128, 0, s>>>(p);
    else if (p.K <= 4) short_conv_kernel<T, V, 4><<<grid, 128, 0, s>>>(p);
    else if (p.K <= 8) short_conv_kernel<T, V, 8><<<grid, 128, 0, s>>>(p);
    else short_conv_kernel<T, V, CONV_MAX_TAPS><<<grid, 128, 0, s>>>(p);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess || p.run >= p.T || p.K == 1) return e;
    conv_carry_kernel<T><<<dim3((p.C + 255) / 256, p.K - 1, p.B), 256, 0, s>>>(p);  // T > CONV_RUN >= K here
    return cudaGetLastError();
}
static_assert(CONV_RUN >= CONV_MAX_TAPS, "the carried inputs of a longer call are all its own");

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
    int B, T, C, n;
};

// decay and drive of one token
template <typename T>
__device__ __forceinline__ void gated_terms(float zr, float zi, float rate, float u, float &a, float &d) {
    const float la = -rate * Fn<T>::sigmoid(zr);
    a = Fn<T>::exp(la);
    d = sqrtf(-expm1f(2.f * la)) * Fn<T>::sigmoid(zi) * u;
}

template <typename T>
__global__ void __launch_bounds__(128) gated_scan_step_kernel(const GatedScanParams p) {
    const int c = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y;
    if (c >= p.C) return;
    const int blk = c / p.n, j = c - blk * p.n;
    const float br = p.gate_bias[c], bi = p.gate_bias[p.C + c], by = p.y_bias[c], rate = p.rate[c];
    float S = p.state[(long long)b * p.C + c];
    for (int t = 0; t < p.T; ++t) {
        const long long row = (long long)b * p.T + t;
        const float *g = p.gates + ((long long)blk * p.B * p.T + row) * 2 * p.n + j;
        float a, d;
        gated_terms<T>(g[0] + br, g[p.n] + bi, rate, to_f(static_cast<const T *>(p.u)[row * p.u_stride + c]), a, d);
        S = fmaf(a, S, d);
        put(static_cast<T *>(p.out) + row * p.C + c, S * gelu_tanh<T>(to_f(static_cast<const T *>(p.y)[row * p.y_stride + c]) + by));
    }
    p.state[(long long)b * p.C + c] = S;
}

constexpr int SC_TOKENS = 16;   // consecutive tokens a thread holds
constexpr int SC_THREADS = 256;

// L: channels per CTA; SC_THREADS / L groups of tokens
template <typename T, int L>
__global__ void __launch_bounds__(SC_THREADS) gated_scan_kernel(const GatedScanParams p) {
    constexpr int NG = SC_THREADS / L, CHUNK = NG * SC_TOKENS;
    __shared__ float s_prod[2][NG][L], s_end[2][NG][L];
    const int lane = threadIdx.x % L, grp = threadIdx.x / L, b = blockIdx.y;
    const int c_raw = blockIdx.x * L + lane, c = min(c_raw, p.C - 1);  // spare lanes repeat the last channel
    const bool have = c_raw < p.C;
    const int blk = c / p.n, j = c - blk * p.n;
    const float br = p.gate_bias[c], bi = p.gate_bias[p.C + c], by = p.y_bias[c], rate = p.rate[c];
    const long long row0 = (long long)b * p.T;
    const T *u = static_cast<const T *>(p.u) + row0 * p.u_stride + c, *y = static_cast<const T *>(p.y) + row0 * p.y_stride + c;
    const float *g = p.gates + ((long long)blk * p.B * p.T + row0) * 2 * p.n + j;
    T *out = static_cast<T *>(p.out) + row0 * p.C + c;
    float S = p.state[(long long)b * p.C + c];
    int parity = 0;
    for (int t0 = 0; t0 < p.T; t0 += CHUNK, parity ^= 1) {
        const int t = t0 + grp * SC_TOKENS;
        float a[SC_TOKENS], d[SC_TOKENS], yv[SC_TOKENS];
#pragma unroll
        for (int i = 0; i < SC_TOKENS; ++i) {  // all loads first
            const long long r = min(t + i, p.T - 1);
            a[i] = g[r * 2 * p.n];
            d[i] = g[r * 2 * p.n + p.n];
            yv[i] = to_f(y[r * p.y_stride]);
        }
        float prod = 1.f, end = 0.f;
#pragma unroll
        for (int i = 0; i < SC_TOKENS; ++i) {
            const long long r = min(t + i, p.T - 1);
            float an, dn;
            gated_terms<T>(a[i] + br, d[i] + bi, rate, to_f(u[r * p.u_stride]), an, dn);
            const bool in = t + i < p.T;
            a[i] = in ? an : 1.f;
            d[i] = in ? dn : 0.f;
            prod *= a[i];
            end = fmaf(a[i], end, d[i]);
        }
        s_prod[parity][grp][lane] = prod;
        s_end[parity][grp][lane] = end;
        __syncthreads();  // the other buffer is free again once all have passed here
        float mine = S;
#pragma unroll
        for (int q = 0; q < NG; ++q) {
            if (q == grp) mine = S;
            S = fmaf(s_prod[parity][q][lane], S, s_end[parity][q][lane]);
        }
#pragma unroll
        for (int i = 0; i < SC_TOKENS; ++i) {
            mine = fmaf(a[i], mine, d[i]);
            if (have && t + i < p.T) put(out + (long long)(t + i) * p.C, mine * gelu_tanh<T>(yv[i] + by));
        }
    }
    if (have && grp == 0) p.state[(long long)b * p.C + c] = S;
}

template <typename T>
static cudaError_t scan_launch(const GatedScanParams &p, cudaStream_t s) {
    if (p.T <= SC_TOKENS) {
        gated_scan_step_kernel<T><<<dim3((p.C + 127) / 128, p.B), 128, 0, s>>>(p);
    } else if ((long long)p.B * ((p.C + 31) / 32) >= 2 * sm_count()) {
        gated_scan_kernel<T, 32><<<dim3((p.C + 31) / 32, p.B), SC_THREADS, 0, s>>>(p);
    } else {
        gated_scan_kernel<T, 16><<<dim3((p.C + 15) / 16, p.B), SC_THREADS, 0, s>>>(p);
    }
    return cudaGetLastError();
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
    if (B <= 0 || T <= 0 || C <= 0 || K <= 0 || B > 65535 || (T + CONV_RUN - 1) / CONV_RUN > 65535) {
        set_error("short_conv: size out of range (B=%d T=%d C=%d K=%d)", B, T, C, K);
        return NCKV_E_ARG;
    }
    if (K > CONV_MAX_TAPS) {
        set_error("short_conv: %d taps unsupported (at most %d)", K, CONV_MAX_TAPS);
        return NCKV_E_UNSUPPORTED;
    }
    ShortConvParams p;
    p.x = x; p.x_stride = x_stride; p.taps = taps; p.in_bias = in_bias; p.bias = bias; p.carry = carry; p.out = out;
    p.B = B; p.T = T; p.C = C; p.K = K; p.run = T; p.act = act;
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

int nckv_gated_scan(const void *u, int64_t u_stride, const void *y, int64_t y_stride, const float *gates, const float *gate_bias,
                    const float *y_bias, const float *rate, float *state, void *out, int B, int T, int C, int blocks, int f32,
                    void *stream) {
    using namespace nckv;
    if (!u || !y || !gates || !gate_bias || !y_bias || !rate || !state || !out) {
        set_error("gated_scan: null pointer argument");
        return NCKV_E_ARG;
    }
    if (B <= 0 || T <= 0 || C <= 0 || B > 65535 || blocks <= 0 || C % blocks) {
        set_error("gated_scan: size out of range (B=%d T=%d C=%d blocks=%d)", B, T, C, blocks);
        return NCKV_E_ARG;
    }
    GatedScanParams p;
    p.u = u; p.y = y; p.u_stride = u_stride; p.y_stride = y_stride;
    p.gates = gates; p.gate_bias = gate_bias; p.y_bias = y_bias; p.rate = rate; p.state = state; p.out = out;
    p.B = B; p.T = T; p.C = C; p.n = C / blocks;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    NCKV_CUDA_CHECK(f32 ? scan_launch<float>(p, s) : scan_launch<__nv_bfloat16>(p, s));
    return NCKV_OK;
}

}  // extern "C"
