// Launchers of the recurrence (recurrent.cuh), the join of its segments, and the gated rms-norm behind a
// recurrence whose norm spans more than one head.
#include "recurrent.cuh"

namespace nckv {

// states (n_seg, B, H, Dk, Dv) hold every segment's own contribution on entry and every segment's
// initial state on exit; `state` (B, H, Dk, Dv) is the first segment's initial state.
__global__ void __launch_bounds__(256) recurrent_join_kernel(float *states, const float *prods, const float *state,
                                                             long long per_seg, int Dv, int n_seg) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= per_seg) return;
    float s = state[i];
    const long long key = i / Dv, per_prod = per_seg / Dv;
    constexpr int AHEAD = 8;  // segments whose operands are fetched together
    for (int g0 = 0; g0 < n_seg; g0 += AHEAD) {
        float own[AHEAD], w[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int g = min(g0 + j, n_seg - 1);
            own[j] = states[g * per_seg + i];
            w[j] = prods[g * per_prod + key];
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (g0 + j >= n_seg) break;
            states[(g0 + j) * per_seg + i] = s;
            s = fmaf(w[j], s, own[j]);
        }
    }
}

// One rms-norm group per CTA: out = x / rms(x) * w * sigmoid(gate) (or silu(gate)), x fp32.  NV quads per
// thread, loaded together; VEC false: scalar loop for sizes that do not allow 4-element accesses.
template <typename T, int NV>
__global__ void __launch_bounds__(256) gated_norm_kernel(const float *__restrict__ x, const T *__restrict__ gate,
                                                         long long gate_stride, const float *__restrict__ w, T *__restrict__ out,
                                                         int C, int group, float eps, int gate_silu) {
    __shared__ float s_part[8];
    const long long row = blockIdx.x;
    const int c0 = blockIdx.y * group, tid = threadIdx.x;
    const float *xr = x + row * C + c0;
    const T *gr = gate + row * gate_stride + c0;
    T *dst = out + row * C + c0;
    float4 a[NV > 0 ? NV : 1];
    Quad<T> g[NV > 0 ? NV : 1];
    float ss = 0.f;
    if (NV > 0) {
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = (k * 256 + tid) * 4;
            a[k] = load_quad<true>(xr + c, c < group, 4).w;
            g[k] = load_quad<true>(gr + c, c < group, 4);
            ss = fmaf(a[k].x, a[k].x, fmaf(a[k].y, a[k].y, fmaf(a[k].z, a[k].z, fmaf(a[k].w, a[k].w, ss))));
        }
    } else {
        for (int c = tid; c < group; c += 256) ss = fmaf(xr[c], xr[c], ss);
    }
#pragma unroll
    for (int off = 16; off; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    if ((tid & 31) == 0) s_part[tid >> 5] = ss;
    __syncthreads();
    ss = s_part[tid & 7];
#pragma unroll
    for (int off = 4; off; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    const float inv = rsqrtf(ss / (float)group + eps);
    auto gate_of = [&](float z) {
        const float s = silu_of<T>(z);  // z * sigmoid(z)
        return gate_silu ? s : (sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-z)) : 1.f / (1.f + expf(-z)));
    };
    if (NV > 0) {
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = (k * 256 + tid) * 4;
            if (c >= group) continue;
            const float4 gf = widen(g[k]), wf = *reinterpret_cast<const float4 *>(w + c0 + c);
            store_quad<true>(dst + c, make_float4(a[k].x * inv * wf.x * gate_of(gf.x), a[k].y * inv * wf.y * gate_of(gf.y),
                                                  a[k].z * inv * wf.z * gate_of(gf.z), a[k].w * inv * wf.w * gate_of(gf.w)), 4);
        }
    } else {
        for (int c = tid; c < group; c += 256) {
            const float z = sizeof(T) == 2 ? bf16_bits_to_float(*reinterpret_cast<const uint16_t *>(gr + c)) : *reinterpret_cast<const float *>(gr + c);
            const float v = xr[c] * inv * w[c0 + c] * gate_of(z);
            store_quad<false>(dst + c, make_float4(v, 0.f, 0.f, 0.f), 1);
        }
    }
}

// Groups of up to 512 channels: a warp per group.
template <typename T, int NV>
__global__ void __launch_bounds__(256) gated_norm_warp_kernel(const float *__restrict__ x, const T *__restrict__ gate,
                                                              long long gate_stride, const float *__restrict__ w, T *__restrict__ out,
                                                              long long n, int C, int group, float eps, int gate_silu) {
    const int lane = threadIdx.x & 31, per_row = C / group;
    const long long id = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (id >= n) return;
    const long long row = id / per_row;
    const int c0 = (int)(id - row * per_row) * group;
    float4 a[NV];
    Quad<T> g[NV];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (k * 32 + lane) * 4;
        a[k] = load_quad<true>(x + row * C + c0 + c, c < group, 4).w;
        g[k] = load_quad<true>(gate + row * gate_stride + c0 + c, c < group, 4);
        ss = fmaf(a[k].x, a[k].x, fmaf(a[k].y, a[k].y, fmaf(a[k].z, a[k].z, fmaf(a[k].w, a[k].w, ss))));
    }
#pragma unroll
    for (int off = 16; off; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    const float inv = rsqrtf(ss / (float)group + eps);
    auto gate_of = [&](float z) {
        return gate_silu ? silu_of<T>(z) : (sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-z)) : 1.f / (1.f + expf(-z)));
    };
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (k * 32 + lane) * 4;
        if (c >= group) continue;
        const float4 gf = widen(g[k]), wf = *reinterpret_cast<const float4 *>(w + c0 + c);
        store_quad<true>(out + row * C + c0 + c, make_float4(a[k].x * inv * wf.x * gate_of(gf.x), a[k].y * inv * wf.y * gate_of(gf.y),
                                                             a[k].z * inv * wf.z * gate_of(gf.z), a[k].w * inv * wf.w * gate_of(gf.w)), 4);
    }
}

template <typename T>
static cudaError_t gated_norm_launch(const float *x, const T *gate, int64_t gate_stride, const float *w, T *out, int rows, int C,
                                     int group, float eps, int gate_silu, cudaStream_t s) {
    const uintptr_t elem = sizeof(T);
    const bool vec = group % 4 == 0 && C % 4 == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0 &&
                     (((uintptr_t)gate | (uintptr_t)out | (uintptr_t)gate_stride * elem) & (4 * elem - 1)) == 0;
    const int per = (group + 1023) / 1024;
    const dim3 grid(rows, C / group);
    if (vec && group <= 512) {
        const long long n = (long long)rows * (C / group);
        const unsigned blocks = (unsigned)((n + 7) / 8);
        if (group <= 128) gated_norm_warp_kernel<T, 1><<<blocks, 256, 0, s>>>(x, gate, gate_stride, w, out, n, C, group, eps, gate_silu);
        else if (group <= 256) gated_norm_warp_kernel<T, 2><<<blocks, 256, 0, s>>>(x, gate, gate_stride, w, out, n, C, group, eps, gate_silu);
        else gated_norm_warp_kernel<T, 4><<<blocks, 256, 0, s>>>(x, gate, gate_stride, w, out, n, C, group, eps, gate_silu);
        return cudaGetLastError();
    }
    if (!vec || per > 8) gated_norm_kernel<T, 0><<<grid, 256, 0, s>>>(x, gate, gate_stride, w, out, C, group, eps, gate_silu);
    else if (per <= 1) gated_norm_kernel<T, 1><<<grid, 256, 0, s>>>(x, gate, gate_stride, w, out, C, group, eps, gate_silu);
    else if (per <= 2) gated_norm_kernel<T, 2><<<grid, 256, 0, s>>>(x, gate, gate_stride, w, out, C, group, eps, gate_silu);
    else if (per <= 4) gated_norm_kernel<T, 4><<<grid, 256, 0, s>>>(x, gate, gate_stride, w, out, C, group, eps, gate_silu);
    else gated_norm_kernel<T, 8><<<grid, 256, 0, s>>>(x, gate, gate_stride, w, out, C, group, eps, gate_silu);
    return cudaGetLastError();
}

cudaError_t recurrent_bf16(const RecurrentParams &p, bool with_out, cudaStream_t s) { return rec_launch<__nv_bfloat16>(p, with_out, s); }

// Segments for a launch of `pairs` (row, head) CTAs over T tokens.
static int rec_segments(int T, int pairs) {
    int n = 2 * sm_count() / pairs;  // about two CTAs per SM, and no straggling second wave
    if (n > T / 64) n = T / 64;      // a shorter segment does not pay for the first pass and the join
    if (n > 64) n = 64;
    return n < 3 ? 1 : n;            // two segments side by side cost more than one after the other
}

}  // namespace nckv

extern "C" {

size_t nckv_recurrent_workspace_bytes(int B, int T, int H, int Dk, int Dv) {
    using namespace nckv;
    if (B <= 0 || T <= 0 || H <= 0 || Dk <= 0 || Dv <= 0) return 0;
    const int n = rec_segments(T, B * H);
    return n == 1 ? 0 : sizeof(float) * (size_t)n * B * H * Dk * (Dv + 1);
}

int nckv_recurrent(const void *q, const void *k, const void *v, int64_t q_stride, int64_t k_stride, int64_t v_stride,
                   const float *x, int64_t x_stride, const float *x0, const float *u, const float *decay,
                   const void *gate, int64_t gate_stride, const float *norm_w, float eps, void *out, int64_t out_stride,
                   float *state, int B, int T, int H, int Dk, int Dv, int act_in, int f32, void *workspace,
                   size_t workspace_bytes, void *stream) {
    using namespace nckv;
    if (!q || !k || !v || !out || !state || (!x && !decay) || (x && (!x0 || !u)) || (norm_w && (!gate || !x))) {
        set_error("recurrent: null pointer argument");
        return NCKV_E_ARG;
    }
    if (B <= 0 || T <= 0 || H <= 0 || Dk <= 0 || Dv <= 0 || B > 65535) {
        set_error("recurrent: size out of range (B=%d T=%d H=%d Dk=%d Dv=%d)", B, T, H, Dk, Dv);
        return NCKV_E_ARG;
    }
    if (Dk > 256 || (norm_w && Dv > REC_COLS)) {
        set_error("recurrent: head sizes %d x %d unsupported (keys at most 256, gated values at most %d)", Dk, Dv, REC_COLS);
        return NCKV_E_UNSUPPORTED;
    }
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    RecurrentParams p;
    p.q = q; p.k = k; p.v = v; p.gate = gate;
    p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride; p.gate_stride = gate_stride;
    p.x = x; p.x_stride = x_stride; p.x0 = x0; p.u = u; p.decay = decay; p.norm_w = norm_w;
    p.out = out; p.out_stride = out_stride;
    p.B = B; p.T = T; p.H = H; p.Dk = Dk; p.Dv = Dv;
    p.eps = eps; p.act_in = act_in;
    p.prod_out = nullptr; p.state_last = nullptr;
    p.C = 0; p.n_cols = 1;
    const uintptr_t elem = f32 ? 4 : 2;
    uintptr_t a = (uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)gate |
                  ((uintptr_t)(q_stride | k_stride | v_stride | gate_stride | Dk | Dv) * elem);
    p.vec = (a & (4 * elem - 1)) == 0 && Dk % 4 == 0 && Dv % 4 == 0 && (!x || ((((uintptr_t)x) | (uintptr_t)(x_stride * 4)) & 15) == 0);

    const int n_seg = rec_segments(T, B * H);
    auto run = [&](const RecurrentParams &r, bool with_out) { return f32 ? recurrent_f32(r, with_out, s) : recurrent_bf16(r, with_out, s); };
    if (n_seg == 1) {
        p.seg_len = T; p.n_seg = 1;
        p.state_in = state; p.state_out = state;
        NCKV_CUDA_CHECK(run(p, true));
        return NCKV_OK;
    }
    if (!workspace || workspace_bytes < nckv_recurrent_workspace_bytes(B, T, H, Dk, Dv)) {
        set_error("recurrent: workspace of %zu bytes given, %zu needed", workspace_bytes,
                  nckv_recurrent_workspace_bytes(B, T, H, Dk, Dv));
        return NCKV_E_CAPACITY;
    }
    const long long per_seg = (long long)B * H * Dk * Dv;
    float *states = static_cast<float *>(workspace), *prods = states + n_seg * per_seg;
    p.seg_len = (T + n_seg - 1) / n_seg;
    p.n_seg = (T + p.seg_len - 1) / p.seg_len;
    RecurrentParams first = p;
    first.state_in = nullptr; first.state_out = states; first.prod_out = prods;
    first.norm_w = nullptr;
    NCKV_CUDA_CHECK(run(first, false));
    recurrent_join_kernel<<<(unsigned)((per_seg + 255) / 256), 256, 0, s>>>(states, prods, state, per_seg, Dv, p.n_seg);
    NCKV_CUDA_CHECK(cudaGetLastError());
    p.state_in = states; p.state_out = states; p.state_last = state;
    NCKV_CUDA_CHECK(run(p, true));
    return NCKV_OK;
}

int nckv_gated_norm(const float *x, const void *gate, int64_t gate_stride, const float *w, void *out, int rows, int C,
                    int group, float eps, int gate_silu, int f32, void *stream) {
    using namespace nckv;
    if (!x || !gate || !w || !out || rows <= 0 || C <= 0 || group <= 0 || C % group || C / group > 65535) {
        set_error("gated_norm: null pointer or bad size (rows=%d C=%d group=%d)", rows, C, group);
        return NCKV_E_ARG;
    }
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    NCKV_CUDA_CHECK(f32 ? gated_norm_launch(x, static_cast<const float *>(gate), gate_stride, w, static_cast<float *>(out), rows, C, group, eps, gate_silu, s)
                        : gated_norm_launch(x, static_cast<const __nv_bfloat16 *>(gate), gate_stride, w, static_cast<__nv_bfloat16 *>(out), rows, C,
                                            group, eps, gate_silu, s));
    return NCKV_OK;
}

}  // extern "C"
