// Linear recurrences with a matrix state per head: one kernel for prompts and for decoding (included by
// recurrent.cu for bf16 and recurrent_f32.cu for fp32 activations).
//
//   S_t = diag(w_t) S_(t-1) + k_t v_t^T          S: (Dk, Dv) per (row, head), fp32, kept in registers
//   o_t = S_t^T q_t                               (inclusive form)
//   o_t = (S_(t-1) + diag(u) k_t v_t^T)^T q_t     (bonus form: the current token enters through u)
//
// The decay w is a constant per head (scaled linear attention) or, per token and key channel,
// exp(-exp(x + x0)) of a projection x (RWKV-style time mixing); both are parameters of the call.
// q, k, v may pass through silu on the way in; o may leave through a per-head rms-norm, a weight and
// a silu gate.  All arithmetic is fp32.  The recurrence is applied token by token, so the state after
// a token has the same bits however the sequence was cut into calls (see the segments below for the
// one exception, which is at fp32 rounding level).
//
// Mapping.  A CTA owns up to 128 value columns of one (row, head, segment).  A warp owns VG*8 of them:
// lane = vg * KG + kg holds key channels {4 KG i + 4 kg + j : i < U, j < 4} of columns {8 vg + c : c < 8}.
// Pairs of key channels are the two halves of packed fp32 instructions; a step is three of them per
// pair and column.  Tokens run in batches of 4: their partial outputs are summed over the KG lanes
// together (a reduce-scatter that leaves a lane 2 or 4 columns of one token), so the latency of the
// shuffles is paid once per batch.  Batches are padded with tokens that leave the state as it is
// (k = 0, w = 1).  Per warp and token 3 U + 2 16-byte shared-memory loads stand against 48 U packed
// multiply-adds: the fp32 pipe is the bound, shared memory and the issue slots are just below it.  Tokens are staged C at a time through two buffers
// (converted, activated and exponentiated once per head on the way, by all warps evenly); the next
// chunk's bytes wait in registers meanwhile.  8 threads normalise, gate and store a token of the
// chunk before.
//
// Single tokens.  recurrent_step_kernel: a decode step is bound by reading and writing the state, so it
// runs more and smaller threads: a thread owns 4 value columns of every (256 / column quads)-th or so key
// row, a row of the state is one coalesced run, and 8 rows per thread are in flight before the first
// is needed.
//
// Segments.  Few (row, head) pairs and a long prompt leave most SMs idle.  Then the prompt is cut
// into segments that run side by side: a first pass finds each segment's own contribution to the
// state and its product of decays, recurrent_join_kernel chains them into every segment's initial
// state, and the ordinary pass runs all segments at once.
#pragma once

#include "nckv_common.cuh"
#include "tc05.cuh"

namespace nckv {

struct RecurrentParams {
    const void *q, *k, *v, *gate;     // (B * T) rows; heads packed inside a row
    long long q_stride, k_stride, v_stride, gate_stride;  // elements between rows
    const float *x;                   // per-channel decay logits, (B * T) rows of x_stride floats; null: per-head decay
    long long x_stride;
    const float *x0, *u;              // (H, Dk) fp32, per-channel form / bonus form
    const float *decay;               // (H) fp32, per-head form
    const float *norm_w;              // (H * Dv) fp32 or null (no epilogue)
    void *out;                        // gated: element type of q; else fp32.  (B * T) rows of out_stride elements
    long long out_stride;
    const float *state_in;            // (B, H, Dk, Dv) or, segmented, (n_seg, B, H, Dk, Dv); null: zero
    float *state_out;                 // same shape, or null: not kept
    float *state_last;                // segmented: where the last segment's state goes instead
    float *prod_out;                  // segmented first pass: (n_seg, B, H, Dk) products of decays
    int B, T, H, Dk, Dv;
    int C;                            // tokens per chunk
    int seg_len, n_seg;
    int n_cols;                       // column blocks per head (1 when gated)
    float eps;
    int act_in;                       // silu on q, k, v
    int vec;                          // all rows allow 4-element loads
};

constexpr int REC_COLS = 128;  // value columns per CTA
constexpr int REC_BATCH = 4;   // tokens whose outputs are reduced together
constexpr int REC_MAXQ = 2;    // 4-element pieces a thread stages per vector and chunk

// fp32 activations get the full-precision functions, bf16 ones the fast intrinsics (a few fp32 ulps)
template <typename T> __device__ __forceinline__ float exp_of(float x);
template <> __device__ __forceinline__ float exp_of<float>(float x) { return expf(x); }
template <> __device__ __forceinline__ float exp_of<__nv_bfloat16>(float x) { return __expf(x); }
template <typename T> __device__ __forceinline__ float silu_of(float z);
template <> __device__ __forceinline__ float silu_of<float>(float z) { return z / (1.f + expf(-z)); }
template <> __device__ __forceinline__ float silu_of<__nv_bfloat16>(float z) { return __fdividef(z, 1.f + __expf(-z)); }
template <typename T> __device__ __forceinline__ float4 silu4(float4 a) {
    return make_float4(silu_of<T>(a.x), silu_of<T>(a.y), silu_of<T>(a.z), silu_of<T>(a.w));
}

template <typename T> struct Quad;
template <> struct Quad<__nv_bfloat16> { uint2 w; };
template <> struct Quad<float> { float4 w; };

__device__ __forceinline__ float4 widen(const Quad<__nv_bfloat16> &q) {
    return make_float4(bf16lo(q.w.x), bf16hi(q.w.x), bf16lo(q.w.y), bf16hi(q.w.y));
}
__device__ __forceinline__ float4 widen(const Quad<float> &q) { return q.w; }

// elements [0, 4) at p when `in`, zeros otherwise; `left` elements are there (VEC: all four or none)
template <bool VEC>
__device__ __forceinline__ Quad<__nv_bfloat16> load_quad(const __nv_bfloat16 *p, bool in, int left) {
    Quad<__nv_bfloat16> r;
    r.w = make_uint2(0u, 0u);
    if (VEC) {
        if (in) r.w = *reinterpret_cast<const uint2 *>(p);
    } else if (in) {
        uint32_t e[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) e[j] = j < left ? (uint32_t)*reinterpret_cast<const uint16_t *>(p + j) : 0u;
        r.w = make_uint2(e[0] | (e[1] << 16), e[2] | (e[3] << 16));
    }
    return r;
}
template <bool VEC>
__device__ __forceinline__ Quad<float> load_quad(const float *p, bool in, int left) {
    Quad<float> r;
    r.w = make_float4(0.f, 0.f, 0.f, 0.f);
    if (VEC) {
        if (in) r.w = *reinterpret_cast<const float4 *>(p);
    } else if (in) {
        r.w.x = p[0];
        if (left > 1) r.w.y = p[1];
        if (left > 2) r.w.z = p[2];
        if (left > 3) r.w.w = p[3];
    }
    return r;
}
template <bool VEC> __device__ __forceinline__ void store_quad(float *p, float4 a, int left) {
    if (VEC) {
        *reinterpret_cast<float4 *>(p) = a;
    } else {
        p[0] = a.x;
        if (left > 1) p[1] = a.y;
        if (left > 2) p[2] = a.z;
        if (left > 3) p[3] = a.w;
    }
}
template <bool VEC> __device__ __forceinline__ void store_quad(__nv_bfloat16 *p, float4 a, int left) {
    if (VEC) {
        *reinterpret_cast<uint2 *>(p) = make_uint2(pack_bf16x2(a.x, a.y), pack_bf16x2(a.z, a.w));
    } else {
        p[0] = __float2bfloat16_rn(a.x);
        if (left > 1) p[1] = __float2bfloat16_rn(a.y);
        if (left > 2) p[2] = __float2bfloat16_rn(a.z);
        if (left > 3) p[3] = __float2bfloat16_rn(a.w);
    }
}

__device__ __forceinline__ float2 fmul2(float2 a, float2 b) {
    float2 d;
    asm("{\n.reg .b64 ra, rb, rd;\nmov.b64 ra, {%2, %3};\nmov.b64 rb, {%4, %5};\nmul.rn.f32x2 rd, ra, rb;\n"
        "mov.b64 {%0, %1}, rd;\n}"
        : "=f"(d.x), "=f"(d.y)
        : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
    return d;
}

// Sums of o[0 .. LEN) over the lanes that differ in the bits BIT, BIT / 2, .. 1 of `kg`: each level halves
// what a lane still holds (a single element is summed by both).  Returns the index of the first element left.
template <int BIT, int LEN> __device__ __forceinline__ int reduce_scatter(float *o, int kg) {
    if constexpr (BIT == 0) {
        return 0;
    } else if constexpr (LEN == 1) {
        o[0] += __shfl_xor_sync(0xffffffffu, o[0], BIT);
        return reduce_scatter<BIT / 2, 1>(o, kg);
    } else {
        constexpr int HALF = LEN / 2;
        const bool up = (kg & BIT) != 0;
#pragma unroll
        for (int c = 0; c < HALF; ++c) {
            const float keep = up ? o[c + HALF] : o[c], give = up ? o[c] : o[c + HALF];
            o[c] = keep + __shfl_xor_sync(0xffffffffu, give, BIT);
        }
        return (up ? HALF : 0) + reduce_scatter<BIT / 2, HALF>(o, kg);
    }
}

// CHANNEL: decay per token and key channel, bonus form.  OUT: false in the first pass over segments.
template <typename T, int KG, int U, bool CHANNEL, bool OUT, bool VEC>
__global__ void __launch_bounds__(REC_COLS / (256 / KG) * 32) recurrent_kernel(const RecurrentParams p) {
    constexpr int TB = REC_BATCH, VG = 32 / KG, KP = 4 * KG * U, KQ = KP / 4, WC = 8 * VG;  // WC: columns per warp
    constexpr int NB = KQ > 32 ? KQ / 32 : 1;                               // partial bonus sums per token
    const int NT = blockDim.x, NW = NT >> 5;
    const int VP = NW * WC, VQ = VP / 4;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, kg = lane % KG, vg = lane / KG;
    const int h = blockIdx.x / p.n_cols, b = blockIdx.y, seg = blockIdx.z;
    const int col0 = (blockIdx.x % p.n_cols) * VP, Dk = p.Dk, Dv = min(p.Dv - col0, VP);  // this CTA's columns of the head
    const int C = p.C;
    const int t_begin = seg * p.seg_len, t_end = min(p.T, t_begin + p.seg_len);
    const bool gated = CHANNEL && OUT && p.norm_w != nullptr;

    extern __shared__ __align__(16) float rec_smem[];
    // [x0 | u | norm weights], two buffers of [k | v | q | w | bonus], two output tiles
    const int per_buf = C * (KP + VP + (OUT ? KP : 0) + (CHANNEL ? KP : 0)) + (CHANNEL && OUT ? C * 4 : 0);
    float *s_x0 = rec_smem, *s_u = s_x0 + KP, *s_nw = s_u + KP, *s_buf = s_nw + VP, *s_out = s_buf + 2 * per_buf;
    const int off_v = C * KP, off_q = off_v + C * VP, off_w = off_q + (OUT ? C * KP : 0), off_b = off_w + (CHANNEL ? C * KP : 0);

    // ---- this lane's part of the state: all loads in flight together ----------------------------------
    float2 S[U * 2][8];  // [pair of key channels][column]
    const int v0 = warp * WC + vg * 8;
    const long long state_base = (((long long)seg * p.B + b) * p.H + h) * (long long)Dk * p.Dv + col0;
    {
        const float *src = p.state_in + state_base;
        const bool have = p.state_in != nullptr;
#pragma unroll
        for (int i = 0; i < U * 4; ++i) {
            const int kc = (i >> 2) * 4 * KG + kg * 4 + (i & 3);
#pragma unroll
            for (int c = 0; c < 8; c += 4) {
                const float4 f = load_quad<VEC>(src + (long long)kc * p.Dv + v0 + c, have && kc < Dk && v0 + c < Dv, Dv - v0 - c).w;
                const float e[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    if (i & 1) S[i >> 1][c + j].y = e[j];
                    else S[i >> 1][c + j].x = e[j];
                }
            }
        }
    }
    float2 prod2[!OUT ? U * 2 : 1];
    if (!OUT) {
#pragma unroll
        for (int i = 0; i < U * 2; ++i) prod2[i] = make_float2(1.f, 1.f);
    }
    const float w_head = CHANNEL ? 1.f : p.decay[h];

    // ---- staging ---------------------------------------------------------------------------------------
    const long long row0 = (long long)b * p.T;
    const int tv = tid / VQ, cv = (tid % VQ) * 4, tv_step = NT / VQ;  // this thread's piece of v: token, column
    const int et = tid >> 3, ec = (tid & 7) * 4, et_step = NT >> 3;    // and of the output: token, first column
    const T *gk = static_cast<const T *>(p.k) + row0 * p.k_stride + (long long)h * Dk;
    const T *gq = static_cast<const T *>(p.q) + row0 * p.q_stride + (long long)h * Dk;
    const float *gx = p.x + row0 * p.x_stride + (long long)h * Dk;
    const T *gv = static_cast<const T *>(p.v) + row0 * p.v_stride + (long long)h * p.Dv + col0 + cv;
    const T *gg = static_cast<const T *>(p.gate) + row0 * p.gate_stride + (long long)h * p.Dv + ec;
    Quad<T> rq[REC_MAXQ], rk[REC_MAXQ], rv[REC_MAXQ];
    Quad<float> rx[REC_MAXQ];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int i = 0; i < REC_MAXQ; ++i) {
            const int idx = tid + i * NT, tk = idx / KQ, ck = (idx % KQ) * 4;
            const bool in = tk < C && t0 + tk < t_end && ck < Dk;
            rk[i] = load_quad<VEC>(gk + (t0 + tk) * p.k_stride + ck, in, Dk - ck);
            if (OUT) rq[i] = load_quad<VEC>(gq + (t0 + tk) * p.q_stride + ck, in, Dk - ck);
            if (CHANNEL) rx[i] = load_quad<VEC>(gx + (t0 + tk) * p.x_stride + ck, in, Dk - ck);
            const int t = tv + i * tv_step;
            rv[i] = load_quad<VEC>(gv + (t0 + t) * p.v_stride, t < C && t0 + t < t_end && cv < Dv, Dv - cv);
        }
    };
    auto stage = [&](float *buf, int n_staged) {  // tokens [n_staged, C) are padding
#pragma unroll
        for (int i = 0; i < REC_MAXQ; ++i) {
            const int idx = tid + i * NT, tk = idx / KQ, ck = (idx % KQ) * 4;
            float4 k4 = widen(rk[i]), q4;
            if (p.act_in) k4 = silu4<T>(k4);
            if (tk < C) *reinterpret_cast<float4 *>(buf + tk * KP + ck) = k4;
            if (OUT) {
                q4 = widen(rq[i]);
                if (p.act_in) q4 = silu4<T>(q4);
                if (tk < C) *reinterpret_cast<float4 *>(buf + off_q + tk * KP + ck) = q4;
            }
            if (CHANNEL) {
                const float4 z = *reinterpret_cast<const float4 *>(s_x0 + ck);
                float4 a = rx[i].w;
                const bool pad = tk >= n_staged;
                a.x = pad ? 1.f : exp_of<T>(-exp_of<T>(a.x + z.x));
                a.y = pad ? 1.f : exp_of<T>(-exp_of<T>(a.y + z.y));
                a.z = pad ? 1.f : exp_of<T>(-exp_of<T>(a.z + z.z));
                a.w = pad ? 1.f : exp_of<T>(-exp_of<T>(a.w + z.w));
                if (tk < C) *reinterpret_cast<float4 *>(buf + off_w + tk * KP + ck) = a;
            }
            if (CHANNEL && OUT) {  // sum over the key channels of q u k, the bonus' factor on v
                const float4 z = *reinterpret_cast<const float4 *>(s_u + ck);
                float s = fmaf(q4.x * z.x, k4.x, fmaf(q4.y * z.y, k4.y, fmaf(q4.z * z.z, k4.z, q4.w * z.w * k4.w)));
#pragma unroll
                for (int off = (KQ < 32 ? KQ : 32) / 2; off; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
                if (tk < C && (idx % (KQ < 32 ? KQ : 32)) == 0) buf[off_b + tk * 4 + (idx % KQ) / 32] = s;
            }
            const int t = tv + i * tv_step;
            if (t < C) {
                float4 v4 = widen(rv[i]);
                if (p.act_in) v4 = silu4<T>(v4);
                *reinterpret_cast<float4 *>(buf + off_v + t * VP + cv) = v4;
            }
        }
    };

    fetch(t_begin);
    for (int c = tid; c < KP; c += NT) {
        s_x0[c] = CHANNEL && c < Dk ? p.x0[h * Dk + c] : 0.f;
        s_u[c] = CHANNEL && OUT && c < Dk ? p.u[h * Dk + c] : 0.f;
    }
    if (gated)
        for (int c = tid; c < VP; c += NT) s_nw[c] = c < Dv ? p.norm_w[h * p.Dv + c] : 0.f;
    __syncthreads();
    stage(s_buf, min(C, t_end - t_begin));
    __syncthreads();

    int parity = 0;
    for (int t0 = t_begin; t0 < t_end; t0 += C, parity ^= 1) {
        const int n = min(C, t_end - t0);
        const float *buf = s_buf + parity * per_buf;
        float *so = s_out + parity * C * VP;
        const bool more = t0 + C < t_end;
        if (more) fetch(t0 + C);
        Quad<T> rg[REC_COLS / 32];
        if (gated) {  // the gate of this chunk, needed at its end (later tokens of a short CTA's share: loaded there)
#pragma unroll
            for (int j = 0; j < REC_COLS / 32; ++j)
                rg[j] = load_quad<VEC>(gg + (t0 + et) * p.gate_stride + j * 32, et < n && ec + j * 32 < Dv, Dv - ec - j * 32);
        }

        const float *bk = buf + kg * 4, *bv = buf + off_v + v0;
#pragma unroll 1
        for (int tb = 0; tb < n; tb += TB) {
            float o[TB * 8];  // [token][column], partial sums over this lane's key channels
#pragma unroll
            for (int tt = 0; tt < TB; ++tt) {
                const int t = tb + tt;
                float2 k2[U * 2], w2[U * 2], q2[OUT ? U * 2 : 1];
                float vv[8];
#pragma unroll
                for (int i = 0; i < U; ++i) {
                    float4 f = *reinterpret_cast<const float4 *>(bk + t * KP + i * 4 * KG);
                    k2[2 * i] = make_float2(f.x, f.y);
                    k2[2 * i + 1] = make_float2(f.z, f.w);
                    if (OUT) {
                        f = *reinterpret_cast<const float4 *>(bk + off_q + t * KP + i * 4 * KG);
                        q2[2 * i] = make_float2(f.x, f.y);
                        q2[2 * i + 1] = make_float2(f.z, f.w);
                    }
                    if (CHANNEL) {
                        f = *reinterpret_cast<const float4 *>(bk + off_w + t * KP + i * 4 * KG);
                        w2[2 * i] = make_float2(f.x, f.y);
                        w2[2 * i + 1] = make_float2(f.z, f.w);
                    } else {
                        const float wt = t < n ? w_head : 1.f;
                        w2[2 * i] = w2[2 * i + 1] = make_float2(wt, wt);
                    }
                }
#pragma unroll
                for (int c = 0; c < 8; c += 4) {
                    const float4 f = *reinterpret_cast<const float4 *>(bv + t * VP + c);
                    vv[c] = f.x; vv[c + 1] = f.y; vv[c + 2] = f.z; vv[c + 3] = f.w;
                }
                if (!OUT && CHANNEL) {
#pragma unroll
                    for (int i = 0; i < U * 2; ++i) prod2[i] = fmul2(prod2[i], w2[i]);
                }
#pragma unroll
                for (int c = 0; c < 8; ++c) {
                    const float2 vd = make_float2(vv[c], vv[c]);
                    float2 acc = make_float2(0.f, 0.f);
#pragma unroll
                    for (int i = 0; i < U * 2; ++i) {
                        if (OUT && CHANNEL) acc = i ? ffma2(q2[i], S[i][c], acc) : fmul2(q2[i], S[i][c]);
                        S[i][c] = ffma2(w2[i], S[i][c], fmul2(k2[i], vd));
                        if (OUT && !CHANNEL) acc = i ? ffma2(q2[i], S[i][c], acc) : fmul2(q2[i], S[i][c]);
                    }
                    if (OUT) o[tt * 8 + c] = acc.x + acc.y;
                }
            }
            if (OUT) {
                const int first = reduce_scatter<KG / 2, TB * 8>(o, kg);
                constexpr int HELD = TB * 8 / KG;  // 4 or 2 columns of one token
                const int t = tb + first / 8, col = v0 + first % 8;
                float bonus = 0.f;
                if (CHANNEL) {
                    bonus = buf[off_b + t * 4];
                    if (NB > 1) bonus += buf[off_b + t * 4 + 1];
                }
#pragma unroll
                for (int c = 0; c < HELD; ++c) {
                    if (CHANNEL) o[c] = fmaf(bonus, buf[off_v + t * VP + col + c], o[c]);
                    so[t * VP + col + c] = o[c];
                }
            }
        }
        if (more) stage(s_buf + (parity ^ 1) * per_buf, min(C, t_end - t0 - C));
        __syncthreads();
        if (OUT) {
            // 8 threads write a token; the buffers in use by the next chunk are the other ones
            for (int tb = 0; tb < n; tb += et_step) {  // the same trip count for all threads: the shuffles need whole warps
                const int t = tb + et;
                const long long row = row0 + t0 + t;
                if (gated) {
                    float4 o4[REC_COLS / 32];
                    float ss = 0.f;
#pragma unroll
                    for (int j = 0; j < REC_COLS / 32; ++j) {
                        o4[j] = make_float4(0.f, 0.f, 0.f, 0.f);
                        if (t < n && ec + j * 32 < VP) o4[j] = *reinterpret_cast<const float4 *>(so + t * VP + ec + j * 32);
                        ss = fmaf(o4[j].x, o4[j].x, fmaf(o4[j].y, o4[j].y, fmaf(o4[j].z, o4[j].z, fmaf(o4[j].w, o4[j].w, ss))));
                        if (tb > 0) rg[j] = load_quad<VEC>(gg + (t0 + t) * p.gate_stride + j * 32, t < n && ec + j * 32 < Dv, Dv - ec - j * 32);
                    }
#pragma unroll
                    for (int off = 4; off; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
                    const float inv = rsqrtf(ss / (float)Dv + p.eps);
                    T *dst = static_cast<T *>(p.out) + row * p.out_stride + (long long)h * p.Dv + ec;
#pragma unroll
                    for (int j = 0; j < REC_COLS / 32; ++j) {
                        if (t < n && ec + j * 32 < Dv) {
                            const float4 g = silu4<T>(widen(rg[j])), w = *reinterpret_cast<const float4 *>(s_nw + ec + j * 32);
                            store_quad<VEC>(dst + j * 32, make_float4(o4[j].x * inv * w.x * g.x, o4[j].y * inv * w.y * g.y,
                                                                      o4[j].z * inv * w.z * g.z, o4[j].w * inv * w.w * g.w), Dv - ec - j * 32);
                        }
                    }
                } else if (t < n) {
                    float *dst = static_cast<float *>(p.out) + row * p.out_stride + (long long)h * p.Dv + col0 + ec;
#pragma unroll
                    for (int j = 0; j < REC_COLS / 32; ++j)
                        if (ec + j * 32 < Dv)
                            store_quad<VEC>(dst + j * 32, *reinterpret_cast<const float4 *>(so + t * VP + ec + j * 32), Dv - ec - j * 32);
                }
            }
        }
    }

    if (p.state_out) {
        float *dst = p.state_last && seg == p.n_seg - 1
                         ? p.state_last + ((long long)b * p.H + h) * Dk * p.Dv + col0
                         : p.state_out + state_base;
#pragma unroll
        for (int i = 0; i < U * 4; ++i) {
            const int kc = (i >> 2) * 4 * KG + kg * 4 + (i & 3);
#pragma unroll
            for (int c = 0; c < 8; c += 4) {
                float e[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) e[j] = (i & 1) ? S[i >> 1][c + j].y : S[i >> 1][c + j].x;
                if (kc < Dk && v0 + c < Dv)
                    store_quad<VEC>(dst + (long long)kc * p.Dv + v0 + c, make_float4(e[0], e[1], e[2], e[3]), Dv - v0 - c);
            }
        }
    }
    if (!OUT && p.prod_out && col0 == 0 && warp == 0 && vg == 0) {
        float *dst = p.prod_out + (((long long)seg * p.B + b) * p.H + h) * Dk;
#pragma unroll
        for (int i = 0; i < U * 4; ++i) {
            const int kc = (i >> 2) * 4 * KG + kg * 4 + (i & 3);
            const float w = CHANNEL ? ((i & 1) ? prod2[i >> 1].y : prod2[i >> 1].x) : powf(w_head, (float)(t_end - t_begin));
            if (kc < Dk) dst[kc] = w;
        }
    }
}

// One token per row.  Thread = row group * CQ + column quad; CQ (a power of two) quads cover the CTA's columns.
template <typename T, bool CHANNEL>
__global__ void __launch_bounds__(256) recurrent_step_kernel(const RecurrentParams p, int CQ) {
    constexpr int ROWS = 8;  // state rows a thread has in flight
    extern __shared__ __align__(16) float step_smem[];
    float4 *s_kqw = reinterpret_cast<float4 *>(step_smem);       // (Dk): k, q, w
    float4 *s_red = s_kqw + p.Dk;                                 // (warps, CQ) partial outputs
    __shared__ float s_bonus[8];
    const int NT = blockDim.x, RG = NT / CQ, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.x / p.n_cols, b = blockIdx.y, col0 = (blockIdx.x % p.n_cols) * CQ * 4;
    const int Dk = p.Dk, cq = tid % CQ, rg = tid / CQ, col = col0 + cq * 4;
    const bool have_col = col < p.Dv;
    const long long base = ((long long)b * p.H + h) * Dk * p.Dv + col;
    const float *src = p.state_in + base;
    float *dst = p.state_out + base;

    float4 S[ROWS];
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const int r = rg + i * RG;
        S[i] = load_quad<true>(src + (long long)r * p.Dv, have_col && r < Dk, 4).w;
    }
    const float4 v_raw = widen(load_quad<true>(static_cast<const T *>(p.v) + b * p.v_stride + (long long)h * p.Dv + col, have_col, 4));
    const bool gated = CHANNEL && p.norm_w != nullptr, last = tid < CQ && have_col;
    const Quad<T> gate = load_quad<true>(static_cast<const T *>(p.gate) + b * p.gate_stride + (long long)h * p.Dv + col, gated && last, 4);
    const float4 nw = load_quad<true>(p.norm_w + (long long)h * p.Dv + col, gated && last, 4).w;
    float bonus = 0.f;
    const float w_head = CHANNEL ? 0.f : p.decay[h];
    for (int c = tid; c < Dk; c += NT) {
        auto one = [](const T *ptr) {
            if constexpr (sizeof(T) == 2) return bf16_bits_to_float(*reinterpret_cast<const uint16_t *>(ptr));
            else return *ptr;
        };
        float q = one(static_cast<const T *>(p.q) + b * p.q_stride + (long long)h * Dk + c);
        float k = one(static_cast<const T *>(p.k) + b * p.k_stride + (long long)h * Dk + c);
        if (p.act_in) {
            q = silu_of<T>(q);
            k = silu_of<T>(k);
        }
        float w = w_head;
        if (CHANNEL) {
            w = exp_of<T>(-exp_of<T>(p.x[b * p.x_stride + (long long)h * Dk + c] + p.x0[h * Dk + c]));
            bonus = fmaf(q * p.u[h * Dk + c], k, bonus);
        }
        s_kqw[c] = make_float4(k, q, w, 0.f);
    }
    const float4 v4 = p.act_in ? silu4<T>(v_raw) : v_raw;
    if (CHANNEL) {
#pragma unroll
        for (int off = 16; off; off >>= 1) bonus += __shfl_xor_sync(0xffffffffu, bonus, off);
        if (lane == 0) s_bonus[warp] = bonus;
    }
    __syncthreads();

    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int r0 = 0; r0 < Dk; r0 += ROWS * RG) {
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            const int r = r0 + rg + i * RG;
            if (r0 > 0) S[i] = load_quad<true>(src + (long long)r * p.Dv, have_col && r < Dk, 4).w;
        }
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            const int r = r0 + rg + i * RG;
            if (r >= Dk) continue;
            const float4 f = s_kqw[r];
            float4 n;
            n.x = fmaf(f.z, S[i].x, f.x * v4.x); n.y = fmaf(f.z, S[i].y, f.x * v4.y);
            n.z = fmaf(f.z, S[i].z, f.x * v4.z); n.w = fmaf(f.z, S[i].w, f.x * v4.w);
            const float4 o = CHANNEL ? S[i] : n;
            acc.x = fmaf(f.y, o.x, acc.x); acc.y = fmaf(f.y, o.y, acc.y);
            acc.z = fmaf(f.y, o.z, acc.z); acc.w = fmaf(f.y, o.w, acc.w);
            if (have_col) *reinterpret_cast<float4 *>(dst + (long long)r * p.Dv) = n;
        }
    }
    for (int off = 16; off >= CQ; off >>= 1) {
        acc.x += __shfl_xor_sync(0xffffffffu, acc.x, off); acc.y += __shfl_xor_sync(0xffffffffu, acc.y, off);
        acc.z += __shfl_xor_sync(0xffffffffu, acc.z, off); acc.w += __shfl_xor_sync(0xffffffffu, acc.w, off);
    }
    if (lane < CQ) s_red[warp * CQ + lane] = acc;
    __syncthreads();
    if (warp > 0) return;  // CQ <= 32: the first warp finishes
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (last) {
        float bn = 0.f;
        for (int i = 0; i < (NT >> 5); ++i) {
            const float4 f = s_red[i * CQ + cq];
            o.x += f.x; o.y += f.y; o.z += f.z; o.w += f.w;
            if (CHANNEL) bn += s_bonus[i];
        }
        o.x = fmaf(bn, v4.x, o.x); o.y = fmaf(bn, v4.y, o.y); o.z = fmaf(bn, v4.z, o.z); o.w = fmaf(bn, v4.w, o.w);
    }
    if (gated) {
        float ss = fmaf(o.x, o.x, fmaf(o.y, o.y, fmaf(o.z, o.z, o.w * o.w)));
#pragma unroll
        for (int off = 16; off; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
        const float inv = rsqrtf(ss / (float)p.Dv + p.eps);
        const float4 g = silu4<T>(widen(gate));
        if (last)
            store_quad<true>(static_cast<T *>(p.out) + b * p.out_stride + (long long)h * p.Dv + col,
                             make_float4(o.x * inv * nw.x * g.x, o.y * inv * nw.y * g.y, o.z * inv * nw.z * g.z, o.w * inv * nw.w * g.w), 4);
    } else if (last) {
        store_quad<true>(static_cast<float *>(p.out) + b * p.out_stride + (long long)h * p.Dv + col, o, 4);
    }
}

template <typename T, bool CHANNEL>
static cudaError_t rec_step_launch(RecurrentParams p, cudaStream_t s) {
    const int cols = p.Dv < REC_COLS ? p.Dv : REC_COLS;
    int CQ = 1;
    while (CQ * 4 < cols) CQ *= 2;
    p.n_cols = (p.Dv + CQ * 4 - 1) / (CQ * 4);
    const int NT = p.Dk * CQ > 1024 ? 256 : (p.Dk * CQ > 512 ? 128 : 64);  // about 8 rows of the state per thread
    const size_t smem = sizeof(float4) * (p.Dk + (size_t)(NT / 32) * CQ);
    recurrent_step_kernel<T, CHANNEL><<<dim3(p.H * p.n_cols, p.B), NT, smem, s>>>(p, CQ);
    return cudaGetLastError();
}

template <typename T, int KG, int U, bool CHANNEL, bool OUT, bool VEC>
static cudaError_t rec_launch_one(RecurrentParams p, cudaStream_t s) {
    constexpr int TB = REC_BATCH, WC = 256 / KG, KP = 4 * KG * U;
    const int cols = p.Dv < REC_COLS ? p.Dv : REC_COLS;
    int NW = (cols + WC - 1) / WC;
    while (REC_MAXQ * NW * 32 < TB * (KP / 4)) ++NW;  // room to stage a batch (wide keys, few value columns)
    const int NT = NW * 32, VP = NW * WC;
    int C = REC_MAXQ * NT / (KP / 4);
    const int Cv = REC_MAXQ * (NT / (VP / 4));
    if (Cv < C) C = Cv;
    if (C > 16) C = 16;
    p.C = C -= C % TB;
    p.n_cols = (p.Dv + VP - 1) / VP;
    const size_t smem = sizeof(float) * (2ull * KP + VP + 2ull * C * (KP + VP + (OUT ? KP : 0) + (CHANNEL ? KP : 0) + (OUT && CHANNEL ? 4 : 0)) +
                                         (OUT ? 2ull * C * VP : 0));
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(recurrent_kernel<T, KG, U, CHANNEL, OUT, VEC>,
                                                   cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    recurrent_kernel<T, KG, U, CHANNEL, OUT, VEC><<<dim3(p.H * p.n_cols, p.B, p.n_seg), NT, smem, s>>>(p);
    return cudaGetLastError();
}

template <typename T, bool CHANNEL, bool OUT, bool VEC>
static cudaError_t rec_launch_dims(const RecurrentParams &p, cudaStream_t s) {
    if (p.Dk <= 32) return rec_launch_one<T, 8, 1, CHANNEL, OUT, VEC>(p, s);
    if (p.Dk <= 64) return rec_launch_one<T, 16, 1, CHANNEL, OUT, VEC>(p, s);
    if (p.Dk <= 128) return rec_launch_one<T, 16, 2, CHANNEL, OUT, VEC>(p, s);
    return rec_launch_one<T, 16, 4, CHANNEL, OUT, VEC>(p, s);
}

template <typename T>
static cudaError_t rec_launch(const RecurrentParams &p, bool with_out, cudaStream_t s) {
    if (p.T == 1 && p.vec && with_out) return p.x ? rec_step_launch<T, true>(p, s) : rec_step_launch<T, false>(p, s);
    if (p.vec) {
        if (p.x) return with_out ? rec_launch_dims<T, true, true, true>(p, s) : rec_launch_dims<T, true, false, true>(p, s);
        return with_out ? rec_launch_dims<T, false, true, true>(p, s) : rec_launch_dims<T, false, false, true>(p, s);
    }
    if (p.x) return with_out ? rec_launch_dims<T, true, true, false>(p, s) : rec_launch_dims<T, true, false, false>(p, s);
    return with_out ? rec_launch_dims<T, false, true, false>(p, s) : rec_launch_dims<T, false, false, false>(p, s);
}

cudaError_t recurrent_bf16(const RecurrentParams &p, bool with_out, cudaStream_t s);
cudaError_t recurrent_f32(const RecurrentParams &p, bool with_out, cudaStream_t s);

}  // namespace nckv
