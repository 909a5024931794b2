// Linear recurrences with a matrix state per head: one kernel for prompts and for decoding.
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
// Mapping.  A CTA owns up to 128 value columns of one (row, head, segment); a warp owns 4*VT of them,
// a lane KV4*4 key channels x VT columns of S: lane = vg * 8 + kg, key channels {32 i + 4 kg + j}, columns
// {vg VT + c}.  Pairs of key channels are the two halves of packed fp32 instructions.  A step costs
// three packed multiply-adds per pair and column; the sum over key channels is a reduce-scatter over
// the 8 lanes kg.  Tokens are staged C at a time through two shared-memory buffers (converted,
// activated and exponentiated on the way), the next chunk's bytes wait in registers meanwhile.
// A single-token call is the same code with one chunk: 16-byte state loads and stores that all sit
// in flight together, which is what a decode step is bound by.
//
// Segments.  Few (row, head) pairs and a long prompt leave most SMs idle.  Then the prompt is cut
// into segments that run side by side: a first pass finds each segment's own contribution to the
// state and its product of decays, recurrent_join_kernel chains them into every segment's initial
// state, and the ordinary pass runs all segments at once.
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
constexpr int REC_MAXQ = 2;  // 4-element pieces a thread stages per vector and chunk

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }

template <typename T> struct Quad;
template <> struct Quad<__nv_bfloat16> { uint2 w; };
template <> struct Quad<float> { float4 w; };

__device__ __forceinline__ float4 widen(const Quad<__nv_bfloat16> &q) {
    return make_float4(bf16lo(q.w.x), bf16hi(q.w.x), bf16lo(q.w.y), bf16hi(q.w.y));
}
__device__ __forceinline__ float4 widen(const Quad<float> &q) { return q.w; }

// elements [c, c + 4) of a row of `n`, zeros beyond it
__device__ __forceinline__ Quad<__nv_bfloat16> load_quad(const __nv_bfloat16 *row, int c, int n, bool vec) {
    Quad<__nv_bfloat16> r;
    if (vec && c + 4 <= n) {
        r.w = *reinterpret_cast<const uint2 *>(row + c);
    } else {
        uint32_t e[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) e[j] = c + j < n ? (uint32_t)*reinterpret_cast<const uint16_t *>(row + c + j) : 0u;
        r.w = make_uint2(e[0] | (e[1] << 16), e[2] | (e[3] << 16));
    }
    return r;
}
__device__ __forceinline__ Quad<float> load_quad(const float *row, int c, int n, bool vec) {
    Quad<float> r;
    if (vec && c + 4 <= n) {
        r.w = *reinterpret_cast<const float4 *>(row + c);
    } else {
        r.w.x = c < n ? row[c] : 0.f;
        r.w.y = c + 1 < n ? row[c + 1] : 0.f;
        r.w.z = c + 2 < n ? row[c + 2] : 0.f;
        r.w.w = c + 3 < n ? row[c + 3] : 0.f;
    }
    return r;
}
__device__ __forceinline__ float4 silu4(float4 a) { return make_float4(silu_f(a.x), silu_f(a.y), silu_f(a.z), silu_f(a.w)); }

__device__ __forceinline__ void store_elem(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void store_elem(float *p, float v) { *p = v; }

__device__ __forceinline__ float2 fmul2(float2 a, float2 b) {
    float2 d;
    asm("{\n.reg .b64 ra, rb, rd;\nmov.b64 ra, {%2, %3};\nmov.b64 rb, {%4, %5};\nmul.rn.f32x2 rd, ra, rb;\n"
        "mov.b64 {%0, %1}, rd;\n}"
        : "=f"(d.x), "=f"(d.y)
        : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
    return d;
}

// CHANNEL: decay per token and key channel, bonus form.  OUT: false in the first pass over segments.
template <typename T, int KV4, int VT, bool CHANNEL, bool OUT>
__global__ void __launch_bounds__(REC_COLS / (4 * VT) * 32)
recurrent_kernel(const RecurrentParams p) {
    constexpr int KP = KV4 * 32;
    const int NT = blockDim.x, NW = NT >> 5;
    const int VP = NW * 4 * VT;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, kg = lane & 7, vg = lane >> 3;
    const int h = blockIdx.x / p.n_cols, b = blockIdx.y, seg = blockIdx.z;
    const int col0 = (blockIdx.x % p.n_cols) * VP, Dv = min(p.Dv - col0, VP);  // this CTA's columns of the head
    const int C = p.C;
    const int t_begin = seg * p.seg_len, t_end = min(p.T, t_begin + p.seg_len);
    const bool gated = OUT && p.norm_w != nullptr;

    extern __shared__ __align__(16) float rec_smem[];
    // two buffers of [k | v | q | w | gate], then two output tiles
    const int per_buf = C * (KP + VP + (OUT ? KP : 0) + (CHANNEL ? KP : 0) + (OUT && CHANNEL ? VP : 0));
    float *s_out = rec_smem + 2 * per_buf;
    const int off_v = C * KP, off_q = off_v + C * VP, off_w = off_q + (OUT ? C * KP : 0),
              off_g = off_w + (CHANNEL ? C * KP : 0);

    const T *gq = static_cast<const T *>(p.q) + (long long)h * p.Dk;
    const T *gk = static_cast<const T *>(p.k) + (long long)h * p.Dk;
    const T *gv = static_cast<const T *>(p.v) + (long long)h * p.Dv + col0;
    const T *gg = static_cast<const T *>(p.gate) + (long long)h * p.Dv + col0;
    const float *gx = p.x + (long long)h * p.Dk;
    const long long row0 = (long long)b * p.T;

    // ---- this lane's part of the state --------------------------------------------------------------
    float2 S[KV4 * 2][VT];  // [pair of key channels][column]
    const int v0 = warp * 4 * VT + vg * VT;
    const long long state_base = (((long long)seg * p.B + b) * p.H + h) * (long long)p.Dk * p.Dv + col0;
    const bool state_vec = (p.Dv & 3) == 0;
#pragma unroll
    for (int i = 0; i < KV4 * 4; ++i) {
        const int kc = (i >> 2) * 32 + kg * 4 + (i & 3);
#pragma unroll
        for (int c = 0; c < VT; c += 4) {
            float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
            if (p.state_in && kc < p.Dk) {
                const float *src = p.state_in + state_base + (long long)kc * p.Dv;
                f = load_quad(src, v0 + c, Dv, state_vec).w;
            }
            const float e[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (i & 1) S[i >> 1][c + j].y = e[j];
                else S[i >> 1][c + j].x = e[j];
            }
        }
    }
    float2 u2[CHANNEL && OUT ? KV4 * 2 : 1], prod2[!OUT ? KV4 * 2 : 1];
    if (CHANNEL && OUT) {
#pragma unroll
        for (int i = 0; i < KV4 * 2; ++i) {
            const int kc = (i >> 1) * 32 + kg * 4 + (i & 1) * 2;
            u2[i].x = kc < p.Dk ? p.u[h * p.Dk + kc] : 0.f;
            u2[i].y = kc + 1 < p.Dk ? p.u[h * p.Dk + kc + 1] : 0.f;
        }
    }
    if (!OUT) {
#pragma unroll
        for (int i = 0; i < KV4 * 2; ++i) prod2[i] = make_float2(1.f, 1.f);
    }
    const float w_head = CHANNEL ? 1.f : p.decay[h];

    // ---- staging ---------------------------------------------------------------------------------------
    Quad<T> rq[REC_MAXQ], rk[REC_MAXQ], rv[REC_MAXQ], rg[REC_MAXQ];
    Quad<float> rx[REC_MAXQ];
    const bool vec = p.vec != 0;
    auto fetch = [&](int t0) {
#pragma unroll
        for (int i = 0; i < REC_MAXQ; ++i) {
            const int idx = tid + i * NT;
            const int tk = idx / (KP / 4), ck = (idx % (KP / 4)) * 4;
            if (tk < C && t0 + tk < t_end && ck < p.Dk) {
                const long long row = row0 + t0 + tk;
                rk[i] = load_quad(gk + row * p.k_stride, ck, p.Dk, vec);
                if (OUT) rq[i] = load_quad(gq + row * p.q_stride, ck, p.Dk, vec);
                if (CHANNEL) rx[i] = load_quad(gx + row * p.x_stride, ck, p.Dk, vec);
            }
            const int tv = idx / (VP / 4), cv = (idx % (VP / 4)) * 4;
            if (tv < C && t0 + tv < t_end && cv < Dv) {
                const long long row = row0 + t0 + tv;
                rv[i] = load_quad(gv + row * p.v_stride, cv, Dv, vec);
                if (CHANNEL && gated) rg[i] = load_quad(gg + row * p.gate_stride, cv, Dv, vec);
            }
        }
    };
    auto stage = [&](int t0, float *buf) {
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < REC_MAXQ; ++i) {
            const int idx = tid + i * NT;
            const int tk = idx / (KP / 4), ck = (idx % (KP / 4)) * 4;
            if (tk < C && t0 + tk < t_end) {
                const bool in = ck < p.Dk;
                float4 a = in ? widen(rk[i]) : zero;
                *reinterpret_cast<float4 *>(buf + tk * KP + ck) = p.act_in ? silu4(a) : a;
                if (OUT) {
                    a = in ? widen(rq[i]) : zero;
                    *reinterpret_cast<float4 *>(buf + off_q + tk * KP + ck) = p.act_in ? silu4(a) : a;
                }
                if (CHANNEL) {
                    a = in ? rx[i].w : zero;
                    const float *z = p.x0 + h * p.Dk + ck;
                    a.x = ck < p.Dk ? expf(-expf(a.x + z[0])) : 0.f;
                    a.y = ck + 1 < p.Dk ? expf(-expf(a.y + z[1])) : 0.f;
                    a.z = ck + 2 < p.Dk ? expf(-expf(a.z + z[2])) : 0.f;
                    a.w = ck + 3 < p.Dk ? expf(-expf(a.w + z[3])) : 0.f;
                    *reinterpret_cast<float4 *>(buf + off_w + tk * KP + ck) = a;
                }
            }
            const int tv = idx / (VP / 4), cv = (idx % (VP / 4)) * 4;
            if (tv < C && t0 + tv < t_end) {
                const bool in = cv < Dv;
                float4 a = in ? widen(rv[i]) : zero;
                *reinterpret_cast<float4 *>(buf + off_v + tv * VP + cv) = p.act_in ? silu4(a) : a;
                if (CHANNEL && gated) {
                    a = in ? silu4(widen(rg[i])) : zero;
                    const float *z = p.norm_w + h * p.Dv + col0 + cv;
                    a.x *= cv < Dv ? z[0] : 0.f;
                    a.y *= cv + 1 < Dv ? z[1] : 0.f;
                    a.z *= cv + 2 < Dv ? z[2] : 0.f;
                    a.w *= cv + 3 < Dv ? z[3] : 0.f;
                    *reinterpret_cast<float4 *>(buf + off_g + tv * VP + cv) = a;
                }
            }
        }
    };

    fetch(t_begin);
    stage(t_begin, rec_smem);
    __syncthreads();

    int parity = 0;
    for (int t0 = t_begin; t0 < t_end; t0 += C, parity ^= 1) {
        const int n = min(C, t_end - t0);
        const float *buf = rec_smem + parity * per_buf;
        float *so = s_out + parity * C * VP;
        const bool more = t0 + C < t_end;
        if (more) fetch(t0 + C);

#pragma unroll 2
        for (int t = 0; t < n; ++t) {
            float2 k2[KV4 * 2], w2[CHANNEL ? KV4 * 2 : 1], q2[OUT ? KV4 * 2 : 1];
            float vv[VT];
#pragma unroll
            for (int i = 0; i < KV4; ++i) {
                float4 f = *reinterpret_cast<const float4 *>(buf + t * KP + i * 32 + kg * 4);
                k2[2 * i] = make_float2(f.x, f.y);
                k2[2 * i + 1] = make_float2(f.z, f.w);
                if (OUT) {
                    f = *reinterpret_cast<const float4 *>(buf + off_q + t * KP + i * 32 + kg * 4);
                    q2[2 * i] = make_float2(f.x, f.y);
                    q2[2 * i + 1] = make_float2(f.z, f.w);
                }
                if (CHANNEL) {
                    f = *reinterpret_cast<const float4 *>(buf + off_w + t * KP + i * 32 + kg * 4);
                    w2[2 * i] = make_float2(f.x, f.y);
                    w2[2 * i + 1] = make_float2(f.z, f.w);
                }
            }
#pragma unroll
            for (int c = 0; c < VT; c += 4) {
                const float4 f = *reinterpret_cast<const float4 *>(buf + off_v + t * VP + v0 + c);
                vv[c] = f.x; vv[c + 1] = f.y; vv[c + 2] = f.z; vv[c + 3] = f.w;
            }
            const float2 wh2 = make_float2(w_head, w_head);
            float o[VT];
            float bonus = 0.f;
            if (CHANNEL && OUT) {
                float2 b2 = make_float2(0.f, 0.f);
#pragma unroll
                for (int i = 0; i < KV4 * 2; ++i) b2 = ffma2(fmul2(q2[i], u2[i]), k2[i], b2);
                bonus = b2.x + b2.y;
            }
            if (!OUT && CHANNEL) {
#pragma unroll
                for (int i = 0; i < KV4 * 2; ++i) prod2[i] = fmul2(prod2[i], w2[i]);
            }
#pragma unroll
            for (int c = 0; c < VT; ++c) {
                const float2 vd = make_float2(vv[c], vv[c]);
                float2 acc = make_float2(0.f, 0.f);
#pragma unroll
                for (int i = 0; i < KV4 * 2; ++i) {
                    if (OUT && CHANNEL) acc = ffma2(q2[i], S[i][c], acc);
                    S[i][c] = ffma2(CHANNEL ? w2[i] : wh2, S[i][c], fmul2(k2[i], vd));
                    if (OUT && !CHANNEL) acc = ffma2(q2[i], S[i][c], acc);
                }
                if (OUT) o[c] = CHANNEL ? fmaf(bonus, vv[c], acc.x + acc.y) : acc.x + acc.y;
            }
            if (OUT) {
                // sum over the 8 lanes kg, every lane keeping a share of the columns
                int col = 0;
                float r4[VT / 2];
#pragma unroll
                for (int c = 0; c < VT / 2; ++c) {
                    const float keep = (kg & 4) ? o[c + VT / 2] : o[c];
                    const float give = (kg & 4) ? o[c] : o[c + VT / 2];
                    r4[c] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
                }
                col += (kg & 4) ? VT / 2 : 0;
                float r2[VT / 4];
#pragma unroll
                for (int c = 0; c < VT / 4; ++c) {
                    const float keep = (kg & 2) ? r4[c + VT / 4] : r4[c];
                    const float give = (kg & 2) ? r4[c] : r4[c + VT / 4];
                    r2[c] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
                }
                col += (kg & 2) ? VT / 4 : 0;
                if (VT == 8) {
                    const float keep = (kg & 1) ? r2[VT / 4 - 1] : r2[0];
                    const float give = (kg & 1) ? r2[0] : r2[VT / 4 - 1];
                    const float r1 = keep + __shfl_xor_sync(0xffffffffu, give, 1);
                    so[t * VP + v0 + col + (kg & 1)] = r1;
                } else {
                    const float r1 = r2[0] + __shfl_xor_sync(0xffffffffu, r2[0], 1);
                    if (!(kg & 1)) so[t * VP + v0 + col] = r1;
                }
            }
        }
        if (more) stage(t0 + C, rec_smem + (parity ^ 1) * per_buf);
        __syncthreads();
        if (OUT) {
            // a warp writes whole tokens; the other buffers are in use by the next chunk meanwhile
            for (int t = warp; t < n; t += NW) {
                const long long row = row0 + t0 + t;
                if (CHANNEL && gated) {
                    float ss = 0.f;
                    for (int c = lane; c < Dv; c += 32) ss = fmaf(so[t * VP + c], so[t * VP + c], ss);
#pragma unroll
                    for (int off = 16; off; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
                    const float inv = 1.f / sqrtf(ss / (float)Dv + p.eps);
                    T *dst = static_cast<T *>(p.out) + row * p.out_stride + (long long)h * p.Dv + col0;
                    for (int c = lane; c < Dv; c += 32) store_elem(dst + c, so[t * VP + c] * inv * buf[off_g + t * VP + c]);
                } else {
                    float *dst = static_cast<float *>(p.out) + row * p.out_stride + (long long)h * p.Dv + col0;
                    for (int c = lane; c < Dv; c += 32) dst[c] = so[t * VP + c];
                }
            }
            if (CHANNEL && gated) __syncthreads();  // the gate sits in the buffer that is refilled next
        }
    }

    if (p.state_out) {
#pragma unroll
        for (int i = 0; i < KV4 * 4; ++i) {
            const int kc = (i >> 2) * 32 + kg * 4 + (i & 3);
            if (kc >= p.Dk) continue;
            float *dst = p.state_out + state_base + (long long)kc * p.Dv;
#pragma unroll
            for (int c = 0; c < VT; c += 4) {
                float e[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) e[j] = (i & 1) ? S[i >> 1][c + j].y : S[i >> 1][c + j].x;
                if (state_vec && v0 + c + 4 <= Dv) {
                    *reinterpret_cast<float4 *>(dst + v0 + c) = make_float4(e[0], e[1], e[2], e[3]);
                } else {
#pragma unroll
                    for (int j = 0; j < 4; ++j)
                        if (v0 + c + j < Dv) dst[v0 + c + j] = e[j];
                }
            }
        }
    }
    if (!OUT && p.prod_out && col0 == 0 && warp == 0 && vg == 0) {
        float *dst = p.prod_out + (((long long)seg * p.B + b) * p.H + h) * p.Dk;
#pragma unroll
        for (int i = 0; i < KV4 * 4; ++i) {
            const int kc = (i >> 2) * 32 + kg * 4 + (i & 3);
            const float w = CHANNEL ? ((i & 1) ? prod2[i >> 1].y : prod2[i >> 1].x) : powf(w_head, (float)(t_end - t_begin));
            if (kc < p.Dk) dst[kc] = w;
        }
    }
}

// states (n_seg, B, H, Dk, Dv) hold every segment's own contribution on entry and every segment's
// initial state on exit; `state` (B, H, Dk, Dv) is the first segment's initial state.
__global__ void __launch_bounds__(256) recurrent_join_kernel(float *states, const float *prods, const float *state,
                                                             long long per_seg, int Dv, int n_seg) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= per_seg) return;
    float s = state[i];
    const long long key = i / Dv, per_prod = per_seg / Dv;
    for (int g = 0; g < n_seg; ++g) {
        const float own = states[g * per_seg + i];
        states[g * per_seg + i] = s;
        s = fmaf(prods[g * per_prod + key], s, own);
    }
}

// One rms-norm group per CTA: out = x / rms(x) * w * sigmoid(gate) (or silu(gate)), x fp32.
template <typename T>
__global__ void __launch_bounds__(128) gated_norm_kernel(const float *__restrict__ x, const T *__restrict__ gate,
                                                         long long gate_stride, const float *__restrict__ w, T *__restrict__ out,
                                                         int C, int group, float eps, int gate_silu) {
    __shared__ float s_part[4];
    const long long row = blockIdx.x;
    const int c0 = blockIdx.y * group, tid = threadIdx.x;
    const float *xr = x + row * C + c0;
    float ss = 0.f;
    for (int c = tid; c < group; c += 128) ss = fmaf(xr[c], xr[c], ss);
#pragma unroll
    for (int off = 16; off; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    if ((tid & 31) == 0) s_part[tid >> 5] = ss;
    __syncthreads();
    ss = (s_part[0] + s_part[1]) + (s_part[2] + s_part[3]);
    const float inv = 1.f / sqrtf(ss / (float)group + eps);
    for (int c = tid; c < group; c += 128) {
        const float g = (float)gate[row * gate_stride + c0 + c];
        const float sig = 1.f / (1.f + expf(-g));
        store_elem(out + row * C + c0 + c, xr[c] * inv * w[c0 + c] * (gate_silu ? g * sig : sig));
    }
}

template <typename T, int KV4, int VT, bool CHANNEL, bool OUT>
static cudaError_t rec_launch_one(RecurrentParams p, cudaStream_t s) {
    const int cols = p.Dv < REC_COLS ? p.Dv : REC_COLS;
    const int NW = (cols + 4 * VT - 1) / (4 * VT), NT = NW * 32;
    const int KP = KV4 * 32, VP = NW * 4 * VT;
    int C = REC_MAXQ * NT * 4 / KP;
    const int Cv = REC_MAXQ * NT * 4 / VP;
    if (Cv < C) C = Cv;
    if (C > (KV4 > 2 ? 8 : 16)) C = KV4 > 2 ? 8 : 16;
    if (C > p.seg_len) C = p.seg_len;
    p.C = C;
    p.n_cols = (p.Dv + VP - 1) / VP;
    const size_t smem = sizeof(float) * (2ull * C * (KP + VP + (OUT ? KP : 0) + (CHANNEL ? KP : 0) + (OUT && CHANNEL ? VP : 0)) +
                                         (OUT ? 2ull * C * VP : 0));
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(recurrent_kernel<T, KV4, VT, CHANNEL, OUT>,
                                                   cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    recurrent_kernel<T, KV4, VT, CHANNEL, OUT><<<dim3(p.H * p.n_cols, p.B, p.n_seg), NT, smem, s>>>(p);
    return cudaGetLastError();
}

template <typename T, bool CHANNEL, bool OUT>
static cudaError_t rec_launch(const RecurrentParams &p, cudaStream_t s) {
    const int kv4 = (p.Dk + 31) / 32;
    if (kv4 == 1) return rec_launch_one<T, 1, 8, CHANNEL, OUT>(p, s);
    if (kv4 == 2) return rec_launch_one<T, 2, 8, CHANNEL, OUT>(p, s);
    if (kv4 <= 4) return rec_launch_one<T, 4, 4, CHANNEL, OUT>(p, s);
    return rec_launch_one<T, 8, 4, CHANNEL, OUT>(p, s);
}

// Segments for a launch of `pairs` (row, head) CTAs over T tokens.
static int rec_segments(int T, int pairs) {
    const int want = (4 * sm_count() + pairs - 1) / pairs;  // CTAs of two to four warps: several fit on an SM
    int n = T / 128;                                        // a segment of less than 128 tokens does not pay for the joins
    if (n > want) n = want;
    if (n > 64) n = 64;
    return n < 3 ? 1 : n;
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
    p.prod_out = nullptr;
    p.C = 0; p.n_cols = 1;
    const uintptr_t elem = f32 ? 4 : 2;
    uintptr_t a = (uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)gate |
                  ((uintptr_t)(q_stride | k_stride | v_stride | gate_stride | Dk | Dv) * elem);
    p.vec = (a & (4 * elem - 1)) == 0 && (!x || ((((uintptr_t)x) | (uintptr_t)(x_stride * 4)) & 15) == 0);

    const int n_seg = rec_segments(T, B * H);
    const bool channel = x != nullptr;
    auto run = [&](const RecurrentParams &r, bool with_out) -> cudaError_t {
        if (f32) {
            if (channel) return with_out ? rec_launch<float, true, true>(r, s) : rec_launch<float, true, false>(r, s);
            return with_out ? rec_launch<float, false, true>(r, s) : rec_launch<float, false, false>(r, s);
        }
        if (channel) return with_out ? rec_launch<__nv_bfloat16, true, true>(r, s) : rec_launch<__nv_bfloat16, true, false>(r, s);
        return with_out ? rec_launch<__nv_bfloat16, false, true>(r, s) : rec_launch<__nv_bfloat16, false, false>(r, s);
    };
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
    p.state_in = states; p.state_out = states;
    NCKV_CUDA_CHECK(run(p, true));
    NCKV_CUDA_CHECK(cudaMemcpyAsync(state, states + (p.n_seg - 1) * per_seg, per_seg * sizeof(float), cudaMemcpyDeviceToDevice, s));
    return NCKV_OK;
}

int nckv_gated_norm(const float *x, const void *gate, int64_t gate_stride, const float *w, void *out, int rows, int C,
                    int group, float eps, int gate_silu, int f32, void *stream) {
    using namespace nckv;
    if (!x || !gate || !w || !out || rows <= 0 || C <= 0 || group <= 0 || C % group || C / group > 65535) {
        set_error("gated_norm: null pointer or bad size (rows=%d C=%d group=%d)", rows, C, group);
        return NCKV_E_ARG;
    }
    const dim3 grid(rows, C / group);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (f32)
        gated_norm_kernel<float><<<grid, 128, 0, s>>>(x, static_cast<const float *>(gate), gate_stride, w,
                                                      static_cast<float *>(out), C, group, eps, gate_silu);
    else
        gated_norm_kernel<__nv_bfloat16><<<grid, 128, 0, s>>>(x, static_cast<const __nv_bfloat16 *>(gate), gate_stride, w,
                                                              static_cast<__nv_bfloat16 *>(out), C, group, eps, gate_silu);
    NCKV_CUDA_CHECK(cudaGetLastError());
    return NCKV_OK;
}

}  // extern "C"
