// Attention pieces for heads of any size in bf16 or fp32, with 32-bit positions, scores and weights.
//
//   rope_unit_append_kernel  rotates the first `rot_dims` channels of every q and k head (pairs
//                            i, i + rot_dims / 2; fp32 cos/sin tables indexed by the absolute position),
//                            divides q and k by their root mean square over the head, multiplies q by
//                            q_scale, and stores q to q_out and k, v to the cache at
//                            cache_seqlens[b] + t.  q_out and the cache may be wider than the head
//                            (zero-filled), so heads of up to 128 channels can run on the kernels that
//                            are built for 128.  One warp per head row.
//   rms_rope_append_kernel   the same with a weighted norm over the whole projection ahead of the rotation
//   window_attn_kernel       softmax attention over the `window` latest keys, fp32 throughout, with an
//                            optional sink and head gate.  A CTA takes
//                            8 query rows of one kv head ((token, group member) pairs, token-major), a warp
//                            one of them; 32 keys at a time are staged in shared memory, a lane scores one
//                            key, and the products with V run over the lanes' value channels.  It serves
//                            the fp32 mode and head sizes the tensor-core kernels do not cover.
#include "vec_io.cuh"

namespace nckv {

struct RopeUnitParams {
    const void *q, *k, *v;  // rows of (heads * dim), own row strides
    long long q_stride, k_stride, v_stride;
    const float *cs;        // (rope_len, rot_dims) fp32: rot_dims / 2 cosines, then as many sines
    const int32_t *seqlens;
    void *q_out, *k_cache, *v_cache;
    long long cache_bs, cache_ts, vcache_bs, vcache_ts;
    int32_t *status;
    int B, T, Hq, Hkv, Dk, Dv, Dk_pad, Dv_pad, rot_dims, rope_len, T_max;
    float q_scale, eps;
};

constexpr int ROPE_MAX = 16;  // channels per lane

// V: consecutive channels a lane takes at a time (4 where sizes and strides allow 4-element accesses)
template <typename T, int V>
__global__ void __launch_bounds__(256) rope_unit_append_kernel(const RopeUnitParams p) {
    const int heads = p.Hq + 2 * p.Hkv;
    const int lane = threadIdx.x & 31;
    const long long n = (long long)p.B * p.T * heads;
    for (long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5); i < n; i += (long long)gridDim.x * 8) {
        const long long row = i / heads;
        const int hh = (int)(i - row * heads);
        const int b = (int)(row / p.T), t = (int)(row - (long long)b * p.T);
        const int L = p.seqlens[b], pos = L + t;
        if (L < 0 || pos >= p.T_max || pos >= p.rope_len) {
            if (lane == 0) atomicOr(p.status, (int)(L < 0 ? NCKV_ST_BAD_SEQLEN : NCKV_ST_OVERFLOW));
            continue;
        }
        const bool is_q = hh < p.Hq, is_v = hh >= p.Hq + p.Hkv;
        const int h = is_q ? hh : (is_v ? hh - p.Hq - p.Hkv : hh - p.Hq);
        const int D = is_v ? p.Dv : p.Dk, D_pad = is_v ? p.Dv_pad : p.Dk_pad;
        const T *src = is_q ? static_cast<const T *>(p.q) + row * p.q_stride + (long long)h * D
                            : (is_v ? static_cast<const T *>(p.v) + row * p.v_stride + (long long)h * D
                                    : static_cast<const T *>(p.k) + row * p.k_stride + (long long)h * D);
        T *dst = is_q ? static_cast<T *>(p.q_out) + (row * p.Hq + h) * D_pad
                      : (is_v ? static_cast<T *>(p.v_cache) + (long long)b * p.vcache_bs + (long long)pos * p.vcache_ts + (long long)h * D_pad
                              : static_cast<T *>(p.k_cache) + (long long)b * p.cache_bs + (long long)pos * p.cache_ts + (long long)h * D_pad);
        const int half = p.rot_dims / 2;
        const float *cs = p.cs + (long long)pos * p.rot_dims;
        auto load = [&](int c, float (&o)[V]) {
            if constexpr (V == 4 && sizeof(T) == 2) {
                const uint2 f = *reinterpret_cast<const uint2 *>(src + c);
                o[0] = bf16lo(f.x); o[1] = bf16hi(f.x); o[2] = bf16lo(f.y); o[3] = bf16hi(f.y);
            } else if constexpr (V == 4) {
                const float4 f = *reinterpret_cast<const float4 *>(src + c);
                o[0] = f.x; o[1] = f.y; o[2] = f.z; o[3] = f.w;
            } else {
                o[0] = to_f(src[c]);
            }
        };
        float x[ROPE_MAX / V][V];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < ROPE_MAX / V; ++k) {
            const int c = (k * 32 + lane) * V;
#pragma unroll
            for (int e = 0; e < V; ++e) x[k][e] = 0.f;
            if (c >= D) continue;
            load(c, x[k]);
            if (!is_v && c < 2 * half) {  // V divides half here, so a piece does not straddle the two halves
                float other[V];
                const bool first = c < half;
                load(first ? c + half : c - half, other);
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    const int i2 = (first ? c : c - half) + e;
                    const float co = cs[i2], si = cs[half + i2];
                    x[k][e] = first ? x[k][e] * co - other[e] * si : x[k][e] * co + other[e] * si;
                }
            }
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(x[k][e], x[k][e], ss);
        }
        float f = 1.f;
        if (!is_v) {
#pragma unroll
            for (int off = 16; off; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
            f = rsqrtf(ss / (float)D + p.eps);
            if (is_q) f *= p.q_scale;
        }
#pragma unroll
        for (int k = 0; k < ROPE_MAX / V; ++k) {
            const int c = (k * 32 + lane) * V;
            if (c >= D_pad) continue;
            if constexpr (V == 4 && sizeof(T) == 2) {
                *reinterpret_cast<uint2 *>(dst + c) = make_uint2(pack_bf16x2(x[k][0] * f, x[k][1] * f), pack_bf16x2(x[k][2] * f, x[k][3] * f));
            } else if constexpr (V == 4) {
                *reinterpret_cast<float4 *>(dst + c) = make_float4(x[k][0] * f, x[k][1] * f, x[k][2] * f, x[k][3] * f);
            } else {
                put(dst + c, x[k][0] * f);
            }
        }
    }
}

// The same append with the norm over the whole projection instead of each head, ahead of the rotation, and with
// a weight: q / rms(q) * wq over all Hq * Dk channels, k alike.  One CTA per token.  k null: queries only (the
// keys and values are another layer's).
struct RmsRopeParams {
    RopeUnitParams a;       // eps as there
    const float *q_w, *k_w; // (Hq * Dk), (Hkv * Dk)
};

template <typename T, int V>
__global__ void __launch_bounds__(256) rms_rope_append_kernel(const RmsRopeParams r) {
    const RopeUnitParams &p = r.a;
    __shared__ float s_part[2][8];
    const int tid = threadIdx.x;
    const long long row = blockIdx.x;
    const int b = (int)(row / p.T), t = (int)(row - (long long)b * p.T);
    const int L = p.seqlens[b], pos = L + t;
    if (L < 0 || pos >= p.T_max || pos >= p.rope_len) {  // uniform over the CTA
        if (tid == 0) atomicOr(p.status, (int)(L < 0 ? NCKV_ST_BAD_SEQLEN : NCKV_ST_OVERFLOW));
        return;
    }
    const T *q = static_cast<const T *>(p.q) + row * p.q_stride, *k = static_cast<const T *>(p.k) + row * p.k_stride;
    const int nq = p.Hq * p.Dk, nk = p.k ? p.Hkv * p.Dk : 0;
    float sq = 0.f, sk = 0.f;
    for (int c = tid * V; c < nq; c += 256 * V) {
        float x[V];
        get_v(q + c, x);
#pragma unroll
        for (int e = 0; e < V; ++e) sq = fmaf(x[e], x[e], sq);
    }
    for (int c = tid * V; c < nk; c += 256 * V) {
        float x[V];
        get_v(k + c, x);
#pragma unroll
        for (int e = 0; e < V; ++e) sk = fmaf(x[e], x[e], sk);
    }
#pragma unroll
    for (int off = 16; off; off >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, off);
        sk += __shfl_xor_sync(0xffffffffu, sk, off);
    }
    if ((tid & 31) == 0) {
        s_part[0][tid >> 5] = sq;
        s_part[1][tid >> 5] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        sq += s_part[0][i];
        sk += s_part[1][i];
    }
    const float fq = 1.f / sqrtf(sq / (float)nq + p.eps), fk = nk ? 1.f / sqrtf(sk / (float)nk + p.eps) : 0.f;
    const int half = p.rot_dims / 2;
    const float *cs = p.cs + (long long)pos * p.rot_dims;
    // heads of D channels from src to padded heads at dst; w null: copied as they are
    auto heads = [&](const T *src, T *dst, int H, int D, int D_pad, const float *w, float f, float scale) {
        const int per = D_pad / V;
        for (int i = tid; i < H * per; i += 256) {
            const int h = i / per, c = (i - h * per) * V;
            float x[V];
#pragma unroll
            for (int e = 0; e < V; ++e) x[e] = 0.f;
            if (c < D) {
                const T *s = src + (long long)h * D;
                get_v(s + c, x);
                if (w) {
                    float ww[V];
                    get_v(w + h * D + c, ww);
#pragma unroll
                    for (int e = 0; e < V; ++e) x[e] *= f * ww[e];
                    if (c < 2 * half) {  // V divides half here, so a piece does not straddle the two halves
                        const bool first = c < half;
                        const int c2 = first ? c + half : c - half;
                        float other[V];
                        get_v(s + c2, other);
                        get_v(w + h * D + c2, ww);
#pragma unroll
                        for (int e = 0; e < V; ++e) {
                            const int i2 = (first ? c : c2) + e;
                            const float o = other[e] * (f * ww[e]), co = cs[i2], si = cs[half + i2];
                            x[e] = first ? x[e] * co - o * si : x[e] * co + o * si;
                        }
                    }
#pragma unroll
                    for (int e = 0; e < V; ++e) x[e] *= scale;
                }
            }
            put_v(dst + (long long)h * D_pad + c, x);
        }
    };
    heads(q, static_cast<T *>(p.q_out) + row * p.Hq * p.Dk_pad, p.Hq, p.Dk, p.Dk_pad, r.q_w, fq, p.q_scale);
    if (!p.k) return;
    heads(k, static_cast<T *>(p.k_cache) + (long long)b * p.cache_bs + (long long)pos * p.cache_ts, p.Hkv, p.Dk, p.Dk_pad, r.k_w, fk, 1.f);
    heads(static_cast<const T *>(p.v) + row * p.v_stride, static_cast<T *>(p.v_cache) + (long long)b * p.vcache_bs + (long long)pos * p.vcache_ts,
          p.Hkv, p.Dv, p.Dv_pad, nullptr, 1.f, 1.f);
}

struct WindowAttnParams {
    const void *q, *k, *v;  // q (B, T, Hq, Dk) packed; caches with the strides below
    void *out;              // (B, T, Hq, Dv) packed
    const int32_t *seqlens;
    long long k_bs, k_ts, v_bs, v_ts;
    int B, T, Hq, Hkv, Dk, Dv, T_max, window;
    float scale;
    int sink;               // one more term of score 0, without a value, in every softmax
    const void *gate;       // (B * T) rows of one logit per head, or null
    long long gate_stride;
};

constexpr int WA_ROWS = 8, WA_KEYS = 32, WA_MAX_DV = 512;

template <typename T>
__global__ void __launch_bounds__(WA_ROWS * 32) window_attn_kernel(const WindowAttnParams p) {
    extern __shared__ __align__(16) float wa_smem[];
    const int Dk4 = (p.Dk + 3) & ~3, kst = Dk4 + 4;
    float *sq = wa_smem, *sk = sq + WA_ROWS * Dk4, *sv = sk + WA_KEYS * kst;
    const int G = p.Hq / p.Hkv, b = blockIdx.z, g0 = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rows = p.T * G, r0 = blockIdx.x * WA_ROWS, r_last = min(rows, r0 + WA_ROWS) - 1;
    const int L = max(p.seqlens[b], 0);
    const int r = min(r0 + warp, rows - 1);
    const int t = r / G, h = g0 * G + r % G, pos = L + t;
    const T *q = static_cast<const T *>(p.q) + (((long long)b * p.T + t) * p.Hq + h) * p.Dk;
    for (int c = lane; c < Dk4; c += 32) sq[warp * Dk4 + c] = c < p.Dk ? to_f(q[c]) : 0.f;
    const int lo = max(0, L + r0 / G - p.window + 1), hi = min(p.T_max, L + r_last / G + 1);
    const T *kb = static_cast<const T *>(p.k) + (long long)b * p.k_bs + (long long)g0 * p.Dk;
    const T *vb = static_cast<const T *>(p.v) + (long long)b * p.v_bs + (long long)g0 * p.Dv;

    float o[WA_MAX_DV / 32];
#pragma unroll
    for (int i = 0; i < WA_MAX_DV / 32; ++i) o[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int j0 = lo; j0 < hi; j0 += WA_KEYS) {
        __syncthreads();
        for (int i = threadIdx.x; i < WA_KEYS * Dk4; i += WA_ROWS * 32) {
            const int j = i / Dk4, c = i - j * Dk4;
            sk[j * kst + c] = j0 + j < hi && c < p.Dk ? to_f(kb[(long long)(j0 + j) * p.k_ts + c]) : 0.f;
        }
        for (int i = threadIdx.x; i < WA_KEYS * p.Dv; i += WA_ROWS * 32) {
            const int j = i / p.Dv, c = i - j * p.Dv;
            sv[i] = j0 + j < hi ? to_f(vb[(long long)(j0 + j) * p.v_ts + c]) : 0.f;
        }
        __syncthreads();
        const int j = j0 + lane;
        float s = -INFINITY;
        if (j < hi && j <= pos && pos - j < p.window) {
            const float4 *a = reinterpret_cast<const float4 *>(sq + warp * Dk4), *k4 = reinterpret_cast<const float4 *>(sk + lane * kst);
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int c = 0; c < Dk4 / 4; ++c) {
                const float4 x = a[c], y = k4[c];
                acc.x = fmaf(x.x, y.x, acc.x); acc.y = fmaf(x.y, y.y, acc.y);
                acc.z = fmaf(x.z, y.z, acc.z); acc.w = fmaf(x.w, y.w, acc.w);
            }
            s = ((acc.x + acc.y) + (acc.z + acc.w)) * p.scale;
        }
        float mx = s;
#pragma unroll
        for (int off = 16; off; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        if (mx == -INFINITY) continue;  // uniform over the warp; the barriers are at the top of the loop
        const float mn = fmaxf(m, mx), alpha = expf(m - mn), pr = expf(s - mn);
        m = mn;
        l = l * alpha + pr;  // per-lane partial sum
#pragma unroll
        for (int i = 0; i < WA_MAX_DV / 32; ++i) o[i] *= alpha;
        for (int jj = 0; jj < WA_KEYS; ++jj) {
            const float w = __shfl_sync(0xffffffffu, pr, jj);
            const float *vr = sv + jj * p.Dv;
#pragma unroll
            for (int i = 0; i < WA_MAX_DV / 32; ++i)
                if (i * 32 + lane < p.Dv) o[i] = fmaf(w, vr[i * 32 + lane], o[i]);
        }
    }
    if (r0 + warp >= rows) return;
#pragma unroll
    for (int off = 16; off; off >>= 1) l += __shfl_xor_sync(0xffffffffu, l, off);
    float inv = l > 0.f ? 1.f / (p.sink ? l + expf(-m) : l) : 0.f;
    if (p.gate) inv *= 1.f / (1.f + expf(-to_f(static_cast<const T *>(p.gate)[((long long)b * p.T + t) * p.gate_stride + h])));
    T *dst = static_cast<T *>(p.out) + (((long long)b * p.T + t) * p.Hq + h) * p.Dv;
#pragma unroll
    for (int i = 0; i < WA_MAX_DV / 32; ++i)
        if (i * 32 + lane < p.Dv) put(dst + i * 32 + lane, o[i] * inv);
}

}  // namespace nckv

extern "C" {

int nckv_rope_unit_append(const void *q, const void *k, const void *v, int64_t q_stride, int64_t k_stride, int64_t v_stride,
                          const float *cos_sin, const int32_t *cache_seqlens, void *q_out, void *k_cache, void *v_cache,
                          int64_t k_batch_stride, int64_t k_token_stride, int64_t v_batch_stride, int64_t v_token_stride,
                          int B, int T, int Hq, int Hkv, int Dk, int Dv, int Dk_pad, int Dv_pad, int rot_dims, int rope_len,
                          int T_max, float q_scale, float eps, int f32, int32_t *status, void *stream) {
    using namespace nckv;
    if (!q || !k || !v || !cache_seqlens || !q_out || !k_cache || !v_cache || !status || (rot_dims > 0 && !cos_sin)) {
        set_error("rope_unit_append: null pointer argument");
        return NCKV_E_ARG;
    }
    if (B <= 0 || T <= 0 || Hq <= 0 || Hkv <= 0 || Hq % Hkv || Dk <= 0 || Dv <= 0 || Dk_pad < Dk || Dv_pad < Dv || T_max <= 0 ||
        rot_dims < 0 || rot_dims > Dk || rot_dims % 2) {
        set_error("rope_unit_append: bad sizes (B=%d T=%d Hq=%d Hkv=%d Dk=%d Dv=%d rot=%d)", B, T, Hq, Hkv, Dk, Dv, rot_dims);
        return NCKV_E_ARG;
    }
    if (T > T_max) {
        set_error("rope_unit_append: T=%d exceeds cache capacity T_max=%d", T, T_max);
        return NCKV_E_CAPACITY;
    }
    if (Dk_pad > 32 * ROPE_MAX || Dv_pad > 32 * ROPE_MAX) {
        set_error("rope_unit_append: head sizes above %d unsupported", 32 * ROPE_MAX);
        return NCKV_E_UNSUPPORTED;
    }
    RopeUnitParams p;
    p.q = q; p.k = k; p.v = v; p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
    p.cs = cos_sin; p.seqlens = cache_seqlens; p.q_out = q_out; p.k_cache = k_cache; p.v_cache = v_cache;
    p.cache_bs = k_batch_stride; p.cache_ts = k_token_stride; p.vcache_bs = v_batch_stride; p.vcache_ts = v_token_stride;
    p.status = status;
    p.B = B; p.T = T; p.Hq = Hq; p.Hkv = Hkv; p.Dk = Dk; p.Dv = Dv; p.Dk_pad = Dk_pad; p.Dv_pad = Dv_pad;
    p.rot_dims = rot_dims; p.rope_len = rot_dims > 0 ? rope_len : 0x7fffffff; p.T_max = T_max; p.q_scale = q_scale; p.eps = eps;
    const uintptr_t elem = f32 ? 4 : 2;
    const uintptr_t a = (uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache |
                        elem * (uintptr_t)(q_stride | k_stride | v_stride | k_batch_stride | k_token_stride | v_batch_stride |
                                           v_token_stride | Dk | Dv | Dk_pad | Dv_pad);
    const bool vec = (a & (4 * elem - 1)) == 0 && rot_dims % 8 == 0;
    const long long n = (long long)B * T * (Hq + 2 * Hkv);
    long long blocks = (n + 7) / 8;
    if (blocks > 32LL * sm_count()) blocks = 32LL * sm_count();
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const unsigned grid = (unsigned)blocks;
    if (f32) {
        if (vec) rope_unit_append_kernel<float, 4><<<grid, 256, 0, s>>>(p);
        else rope_unit_append_kernel<float, 1><<<grid, 256, 0, s>>>(p);
    } else {
        if (vec) rope_unit_append_kernel<__nv_bfloat16, 4><<<grid, 256, 0, s>>>(p);
        else rope_unit_append_kernel<__nv_bfloat16, 1><<<grid, 256, 0, s>>>(p);
    }
    NCKV_CUDA_CHECK(cudaGetLastError());
    return NCKV_OK;
}

int nckv_rms_rope_append(const void *q, const void *k, const void *v, int64_t q_stride, int64_t k_stride, int64_t v_stride,
                         const float *q_weight, const float *k_weight, const float *cos_sin, const int32_t *cache_seqlens,
                         void *q_out, void *k_cache, void *v_cache, int64_t k_batch_stride, int64_t k_token_stride,
                         int64_t v_batch_stride, int64_t v_token_stride, int B, int T, int Hq, int Hkv, int Dk, int Dv,
                         int Dk_pad, int Dv_pad, int rot_dims, int rope_len, int T_max, float q_scale, float eps, int f32,
                         int32_t *status, void *stream) {
    using namespace nckv;
    if (!q || !q_weight || !cache_seqlens || !q_out || !status || (rot_dims > 0 && !cos_sin) ||
        (k && (!v || !k_weight || !k_cache || !v_cache))) {
        set_error("rms_rope_append: null pointer argument");
        return NCKV_E_ARG;
    }
    if (B <= 0 || T <= 0 || Hq <= 0 || Hkv <= 0 || Hq % Hkv || Dk <= 0 || Dv <= 0 || Dk_pad < Dk || Dv_pad < Dv || T_max <= 0 ||
        rot_dims < 0 || rot_dims > Dk || rot_dims % 2 || (long long)B * T > 0x7fffffffLL) {
        set_error("rms_rope_append: bad sizes (B=%d T=%d Hq=%d Hkv=%d Dk=%d Dv=%d rot=%d)", B, T, Hq, Hkv, Dk, Dv, rot_dims);
        return NCKV_E_ARG;
    }
    if (T > T_max) {
        set_error("rms_rope_append: T=%d exceeds cache capacity T_max=%d", T, T_max);
        return NCKV_E_CAPACITY;
    }
    RmsRopeParams r;
    RopeUnitParams &p = r.a;
    p.q = q; p.k = k; p.v = v; p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
    p.cs = cos_sin; p.seqlens = cache_seqlens; p.q_out = q_out; p.k_cache = k_cache; p.v_cache = v_cache;
    p.cache_bs = k_batch_stride; p.cache_ts = k_token_stride; p.vcache_bs = v_batch_stride; p.vcache_ts = v_token_stride;
    p.status = status;
    p.B = B; p.T = T; p.Hq = Hq; p.Hkv = Hkv; p.Dk = Dk; p.Dv = Dv; p.Dk_pad = Dk_pad; p.Dv_pad = Dv_pad;
    p.rot_dims = rot_dims; p.rope_len = rot_dims > 0 ? rope_len : 0x7fffffff; p.T_max = T_max; p.q_scale = q_scale; p.eps = eps;
    r.q_w = q_weight; r.k_w = k_weight;
    const uintptr_t elem = f32 ? 4 : 2;
    uintptr_t a = (uintptr_t)q | (uintptr_t)q_out | elem * (uintptr_t)(q_stride | Dk | Dv | Dk_pad | Dv_pad);
    if (k) a |= (uintptr_t)k | (uintptr_t)v | (uintptr_t)k_cache | (uintptr_t)v_cache |
                elem * (uintptr_t)(k_stride | v_stride | k_batch_stride | k_token_stride | v_batch_stride | v_token_stride);
    const bool vec = (a & (4 * elem - 1)) == 0 && (((uintptr_t)q_weight | (uintptr_t)k_weight) & 15) == 0 && rot_dims % 8 == 0;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const unsigned grid = (unsigned)(B * T);
    if (f32) {
        if (vec) rms_rope_append_kernel<float, 4><<<grid, 256, 0, s>>>(r);
        else rms_rope_append_kernel<float, 1><<<grid, 256, 0, s>>>(r);
    } else {
        if (vec) rms_rope_append_kernel<__nv_bfloat16, 4><<<grid, 256, 0, s>>>(r);
        else rms_rope_append_kernel<__nv_bfloat16, 1><<<grid, 256, 0, s>>>(r);
    }
    NCKV_CUDA_CHECK(cudaGetLastError());
    return NCKV_OK;
}

int nckv_window_attn(const void *q, const void *k_cache, const void *v_cache, const int32_t *cache_seqlens, void *out,
                     int64_t k_batch_stride, int64_t k_token_stride, int64_t v_batch_stride, int64_t v_token_stride, int B,
                     int T, int Hq, int Hkv, int Dk, int Dv, int T_max, int window, float scale, int sink, const void *gate,
                     int64_t gate_stride, int f32, void *stream) {
    using namespace nckv;
    if (!q || !k_cache || !v_cache || !cache_seqlens || !out) {
        set_error("window_attn: null pointer argument");
        return NCKV_E_ARG;
    }
    if (B <= 0 || T <= 0 || Hq <= 0 || Hkv <= 0 || Hq % Hkv || Dk <= 0 || Dv <= 0 || T_max <= 0 || window <= 0 || B > 65535 || Hkv > 65535) {
        set_error("window_attn: bad sizes (B=%d T=%d Hq=%d Hkv=%d Dk=%d Dv=%d window=%d)", B, T, Hq, Hkv, Dk, Dv, window);
        return NCKV_E_ARG;
    }
    const int Dk4 = (Dk + 3) & ~3;
    const size_t smem = sizeof(float) * ((size_t)WA_ROWS * Dk4 + WA_KEYS * (Dk4 + 4) + (size_t)WA_KEYS * Dv);
    if (Dv > WA_MAX_DV || smem > 200 * 1024) {
        set_error("window_attn: head sizes %d / %d unsupported", Dk, Dv);
        return NCKV_E_UNSUPPORTED;
    }
    WindowAttnParams p;
    p.q = q; p.k = k_cache; p.v = v_cache; p.out = out; p.seqlens = cache_seqlens;
    p.k_bs = k_batch_stride; p.k_ts = k_token_stride; p.v_bs = v_batch_stride; p.v_ts = v_token_stride;
    p.B = B; p.T = T; p.Hq = Hq; p.Hkv = Hkv; p.Dk = Dk; p.Dv = Dv; p.T_max = T_max; p.window = window; p.scale = scale;
    p.sink = sink; p.gate = gate; p.gate_stride = gate_stride;
    const long long rows = (long long)T * (Hq / Hkv);
    const dim3 grid((unsigned)((rows + WA_ROWS - 1) / WA_ROWS), Hkv, B);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (smem > 48 * 1024) {
        if (f32) NCKV_CUDA_CHECK(cudaFuncSetAttribute(window_attn_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        else NCKV_CUDA_CHECK(cudaFuncSetAttribute(window_attn_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    }
    if (f32) window_attn_kernel<float><<<grid, WA_ROWS * 32, smem, s>>>(p);
    else window_attn_kernel<__nv_bfloat16><<<grid, WA_ROWS * 32, smem, s>>>(p);
    NCKV_CUDA_CHECK(cudaGetLastError());
    return NCKV_OK;
}

}  // extern "C"
