// Gated delta rule with a decay per key channel: a matrix state per head that is corrected, not only added to.
//
//   S <- diag(w_t) S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t
//
// S: (Dk, Dv) per (row, head), fp32, kept in registers.  q and k are made unit vectors (q also scaled by
// Dk^-1/2), w = exp(-rate softplus(x + x0)), beta = sigmoid(b), all in fp32.
//
// Prompts run in batches of 4 tokens.  With c_t = w_1 .. w_t (products from the batch's first token on) the
// four corrections follow from the state before the batch:
//   u_t = beta_t (v_t - S^T (c_t k_t) - sum_{i<t} A_ti u_i)      A_ti = sum_c k_t k_i w_(i+1) .. w_t
//   o_t = S^T (c_t q_t) + sum_{i<=t} Q_ti u_i                     Q_ti = sum_c q_t k_i w_(i+1) .. w_t
//   S   <- diag(c_4) S + sum_i (w_(i+1) .. w_4 k_i) u_i^T
// so a batch costs one exchange between the lanes that share a column instead of four, and 13 instead of 16
// multiply-adds per state element.  Only products of decays appear (each <= 1): nothing overflows however
// strong the decay.  Everything that does not depend on the state is found once per head by
//
//   delta_prepare_kernel   one warp per (row, head, batch): norms, decays, the three scaled key / query rows
//                          per token, A, Q and beta, as one record of fp32 numbers
//   delta_kernel           a CTA owns some value columns of one (row, head) and walks over the records,
//                          which arrive through a ring in shared memory (cp.async); lane = vg * KG + kg
//                          holds key channels {4 KG i + 4 kg + j} of 4 columns.  Partial products are
//                          summed over the KG lanes with the columns scattered first, every lane solves
//                          the batch's four corrections of its column, and the lanes of a warp exchange them.
//   delta_step_kernel      single tokens: bound by reading and writing the state, so a whole head per CTA,
//                          a row of the state as one coalesced run, the head's norm and gate included.
//
// How a prompt is cut into calls moves the batch borders, which changes results at fp32 rounding level only.
#include "tc05.cuh"
#include "vec_io.cuh"

namespace nckv {

constexpr int DL_TB = 4;     // tokens per batch
constexpr int DL_TAIL = 32;  // floats after the rows of a record: A (6), Q (10), beta (4), padding
constexpr int DL_COLS = 4;   // value columns per lane
constexpr int DL_WARPS = 4;
constexpr int DL_RING = 4;   // records in flight

// record: [c_t k_t : 4 rows][c_t q_t : 4][k_i to the end : 4][c_4 : 1] of KP floats, then the tail
__host__ __device__ constexpr int delta_record(int KP) { return 13 * KP + DL_TAIL; }

struct DeltaParams {
    const void *q, *k, *v;      // (B * T) rows of T; heads packed inside a row
    long long q_stride, k_stride, v_stride;
    const float *x;             // (B * T) rows of H * Dk decay logits
    long long x_stride;
    const float *x0, *rate;     // (H * Dk), (H)
    const void *b;              // (B * T) rows of H step-size logits
    long long b_stride;
    float *records;             // (B, H, batches, delta_record(KP))
    float *state;               // (B, H, Dk, Dv)
    void *out;                  // prompts: (B * T, H * Dv) fp32; single tokens: T
    const void *gate;           // single tokens: rows of H * Dv
    long long gate_stride;
    const float *norm_w;        // single tokens: (Dv)
    int B, T, H, G, Dk, Dv, KP, n_batches, n_cols;
    float eps;
};

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int off = 16; off; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
    return v;
}

// NJ channels per lane: c = lane + 32 j
template <typename T, int NJ>
__global__ void __launch_bounds__(128) delta_prepare_kernel(const DeltaParams p) {
    const int lane = threadIdx.x & 31;
    const long long id = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);  // (batch, head, row), heads fastest: rows are read once
    if (id >= (long long)p.B * p.n_batches * p.H) return;
    const int h = (int)(id % p.H), bt = (int)(id / p.H % p.n_batches), b = (int)(id / p.H / p.n_batches);
    const int g = h / (p.H / p.G), t0 = bt * DL_TB;
    const float rate = p.rate[h], q_scale = rsqrtf((float)p.Dk);
    float q[DL_TB][NJ], k[DL_TB][NJ], w[DL_TB][NJ], beta = 0.f;
#pragma unroll
    for (int t = 0; t < DL_TB; ++t) {
        const long long row = (long long)b * p.T + t0 + t;
        const bool in = t0 + t < p.T;  // the tokens behind the last leave the state as it is
        float qq = 0.f, kk = 0.f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const int c = lane + 32 * j;
            const bool on = in && c < p.Dk;
            q[t][j] = on ? to_f(static_cast<const T *>(p.q)[row * p.q_stride + (long long)g * p.Dk + c]) : 0.f;
            k[t][j] = on ? to_f(static_cast<const T *>(p.k)[row * p.k_stride + (long long)g * p.Dk + c]) : 0.f;
            const float x = on ? p.x[row * p.x_stride + (long long)h * p.Dk + c] + p.x0[h * p.Dk + c] : 0.f;
            w[t][j] = on ? Fn<T>::exp(-rate * softplus(x)) : 1.f;
            qq = fmaf(q[t][j], q[t][j], qq);
            kk = fmaf(k[t][j], k[t][j], kk);
        }
        const float iq = q_scale / sqrtf(warp_sum(qq) + 1e-6f), ik = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            q[t][j] *= iq;
            k[t][j] *= ik;
        }
        if (lane == t && in) beta = Fn<T>::sigmoid(to_f(static_cast<const T *>(p.b)[row * p.b_stride + h]));
    }
    float A[6], Q[10];  // (1,0) (2,0) (2,1) (3,0) ..; (0,0) (1,0) (1,1) (2,0) ..
#pragma unroll
    for (int i = 0; i < 6; ++i) A[i] = 0.f;
#pragma unroll
    for (int i = 0; i < 10; ++i) Q[i] = 0.f;
    float *rec = p.records + (((long long)b * p.H + h) * p.n_batches + bt) * delta_record(p.KP);
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        const int c = lane + 32 * j;
        float ki[DL_TB];  // k_i carried to the current token
#pragma unroll
        for (int t = 0; t < DL_TB; ++t) {
#pragma unroll
            for (int i = 0; i < t; ++i) {
                ki[i] *= w[t][j];
                A[t * (t - 1) / 2 + i] = fmaf(k[t][j], ki[i], A[t * (t - 1) / 2 + i]);
                Q[t * (t + 1) / 2 + i] = fmaf(q[t][j], ki[i], Q[t * (t + 1) / 2 + i]);
            }
            ki[t] = k[t][j];
            Q[t * (t + 1) / 2 + t] = fmaf(q[t][j], ki[t], Q[t * (t + 1) / 2 + t]);
        }
        if (c < p.KP) {
            float cum = 1.f;
#pragma unroll
            for (int t = 0; t < DL_TB; ++t) {
                cum *= w[t][j];
                rec[t * p.KP + c] = cum * k[t][j];
                rec[(DL_TB + t) * p.KP + c] = cum * q[t][j];
                rec[(2 * DL_TB + t) * p.KP + c] = ki[t];
            }
            rec[3 * DL_TB * p.KP + c] = cum;
        }
    }
    float *tail = rec + 13 * p.KP;
#pragma unroll
    for (int i = 0; i < 6; ++i) {
        const float s = warp_sum(A[i]);
        if (lane == 0) tail[i] = s;
    }
#pragma unroll
    for (int i = 0; i < 10; ++i) {
        const float s = warp_sum(Q[i]);
        if (lane == 0) tail[6 + i] = s;
    }
    if (lane < DL_TB) tail[16 + lane] = beta;
}

__device__ __forceinline__ void cp_async16(void *smem, const void *gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ float2 fmul2_(float2 a, float2 b) {
    float2 d;
    asm("{\n.reg .b64 ra, rb, rd;\nmov.b64 ra, {%2, %3};\nmov.b64 rb, {%4, %5};\nmul.rn.f32x2 rd, ra, rb;\n"
        "mov.b64 {%0, %1}, rd;\n}"
        : "=f"(d.x), "=f"(d.y)
        : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
    return d;
}

template <typename T, int KG, int U>
__global__ void __launch_bounds__(DL_WARPS * 32) delta_kernel(const DeltaParams p) {
    constexpr int KP = 4 * KG * U, VG = 32 / KG, WC = VG * DL_COLS, REC = delta_record(KP), NT = DL_WARPS * 32;
    static_assert(DL_COLS == 4, "two bits of kg choose the column");
    extern __shared__ __align__(16) float dl_smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, kg = lane % KG, vg = lane / KG;
    const int h = blockIdx.x / p.n_cols, b = blockIdx.y;
    const int col_lane = (blockIdx.x % p.n_cols) * DL_WARPS * WC + warp * WC + vg * DL_COLS;  // first of this lane's columns
    // after the scatter a lane answers for one column: the upper two bits of kg choose it
    const int my_col = col_lane + kg / (KG / 4), n = p.n_batches;
    const bool have = my_col < p.Dv;
    const float *src = p.records + ((long long)b * p.H + h) * n * REC;
    auto fetch = [&](int i) {
        if (i < n) {
            float *dst = dl_smem + (i % DL_RING) * REC;
            const float *from = src + (long long)i * REC;
            for (int c = tid; c < REC / 4; c += NT) cp_async16(dst + c * 4, from + c * 4);
        }
        cp_async_commit();
    };
#pragma unroll
    for (int i = 0; i < DL_RING - 1; ++i) fetch(i);

    float2 S[U * 2][DL_COLS];  // pairs of key channels
    float *state = p.state + ((long long)b * p.H + h) * p.Dk * p.Dv;
#pragma unroll
    for (int i = 0; i < U * 2; ++i) {
        const int kc = (i >> 1) * 4 * KG + kg * 4 + (i & 1) * 2;
#pragma unroll
        for (int c = 0; c < DL_COLS; ++c) {
            const bool in = col_lane + c < p.Dv;
            S[i][c].x = in && kc < p.Dk ? state[(long long)kc * p.Dv + col_lane + c] : 0.f;
            S[i][c].y = in && kc + 1 < p.Dk ? state[(long long)(kc + 1) * p.Dv + col_lane + c] : 0.f;
        }
    }
    const T *v = static_cast<const T *>(p.v) + (long long)b * p.T * p.v_stride + (long long)h * p.Dv + my_col;
    float *out = static_cast<float *>(p.out) + (long long)b * p.T * p.H * p.Dv + (long long)h * p.Dv + my_col;
    float v_next[DL_TB];
    auto load_v = [&](int i) {
#pragma unroll
        for (int t = 0; t < DL_TB; ++t) {
            const int tt = i * DL_TB + t;
            v_next[t] = have && tt < p.T ? to_f(v[(long long)tt * p.v_stride]) : 0.f;
        }
    };
    load_v(0);

    for (int i = 0; i < n; ++i) {
        cp_async_wait<DL_RING - 2>();
        __syncthreads();  // record i has landed for all threads, and record i - 1 has been read by all
        fetch(i + DL_RING - 1);
        const float *rec = dl_smem + (i % DL_RING) * REC, *tail = rec + 13 * KP;
        float vt[DL_TB];
#pragma unroll
        for (int t = 0; t < DL_TB; ++t) vt[t] = v_next[t];
        load_v(i + 1);

        // S^T (c_t k_t) and S^T (c_t q_t): [column][4 k, 4 q]
        float r[DL_COLS * 8];
#pragma unroll
        for (int t = 0; t < 8; ++t) {
            float2 a2[U * 2];
#pragma unroll
            for (int j = 0; j < U; ++j) {
                const float4 f = *reinterpret_cast<const float4 *>(rec + t * KP + j * 4 * KG + kg * 4);
                a2[2 * j] = make_float2(f.x, f.y);
                a2[2 * j + 1] = make_float2(f.z, f.w);
            }
#pragma unroll
            for (int c = 0; c < DL_COLS; ++c) {
                float2 acc = fmul2_(a2[0], S[0][c]);
#pragma unroll
                for (int j = 1; j < U * 2; ++j) acc = ffma2(a2[j], S[j][c], acc);
                r[c * 8 + t] = acc.x + acc.y;
            }
        }
        // columns 0..3 are split over the upper two bits of kg, the rest is summed
        {
            const bool up = (kg & (KG / 2)) != 0;
#pragma unroll
            for (int e = 0; e < 16; ++e) {
                const float keep = up ? r[16 + e] : r[e], give = up ? r[e] : r[16 + e];
                r[e] = keep + __shfl_xor_sync(0xffffffffu, give, KG / 2);
            }
            const bool up2 = (kg & (KG / 4)) != 0;
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const float keep = up2 ? r[8 + e] : r[e], give = up2 ? r[e] : r[8 + e];
                r[e] = keep + __shfl_xor_sync(0xffffffffu, give, KG / 4);
            }
#pragma unroll
            for (int off = KG / 8; off; off >>= 1)
#pragma unroll
                for (int e = 0; e < 8; ++e) r[e] += __shfl_xor_sync(0xffffffffu, r[e], off);
        }
        float u[DL_TB], tl[20];
#pragma unroll
        for (int e = 0; e < 20; e += 4) {
            const float4 f = *reinterpret_cast<const float4 *>(tail + e);
            tl[e] = f.x; tl[e + 1] = f.y; tl[e + 2] = f.z; tl[e + 3] = f.w;
        }
#pragma unroll
        for (int t = 0; t < DL_TB; ++t) {
            float z = vt[t] - r[t];
#pragma unroll
            for (int j = 0; j < t; ++j) z = fmaf(-tl[t * (t - 1) / 2 + j], u[j], z);
            u[t] = tl[16 + t] * z;
        }
        // all four columns' corrections to every lane of the column group
        float ua[DL_COLS][DL_TB];
        {
            float lo[2][DL_TB];
            const bool up2 = (kg & (KG / 4)) != 0, up = (kg & (KG / 2)) != 0;
#pragma unroll
            for (int t = 0; t < DL_TB; ++t) {
                const float other = __shfl_xor_sync(0xffffffffu, u[t], KG / 4);
                lo[0][t] = up2 ? other : u[t];
                lo[1][t] = up2 ? u[t] : other;
            }
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
                for (int t = 0; t < DL_TB; ++t) {
                    const float other = __shfl_xor_sync(0xffffffffu, lo[c][t], KG / 2);
                    ua[c][t] = up ? other : lo[c][t];
                    ua[2 + c][t] = up ? lo[c][t] : other;
                }
        }
        // S <- diag(c_4) S + sum_i k_i u_i^T
#pragma unroll
        for (int j = 0; j < U; ++j) {
            float4 f = *reinterpret_cast<const float4 *>(rec + 12 * KP + j * 4 * KG + kg * 4);
            const float2 d0 = make_float2(f.x, f.y), d1 = make_float2(f.z, f.w);
            float2 k0[DL_TB], k1[DL_TB];
#pragma unroll
            for (int t = 0; t < DL_TB; ++t) {
                f = *reinterpret_cast<const float4 *>(rec + (8 + t) * KP + j * 4 * KG + kg * 4);
                k0[t] = make_float2(f.x, f.y);
                k1[t] = make_float2(f.z, f.w);
            }
#pragma unroll
            for (int c = 0; c < DL_COLS; ++c) {
                float2 s0 = fmul2_(d0, S[2 * j][c]), s1 = fmul2_(d1, S[2 * j + 1][c]);
#pragma unroll
                for (int t = 0; t < DL_TB; ++t) {
                    const float2 uu = make_float2(ua[c][t], ua[c][t]);
                    s0 = ffma2(k0[t], uu, s0);
                    s1 = ffma2(k1[t], uu, s1);
                }
                S[2 * j][c] = s0;
                S[2 * j + 1][c] = s1;
            }
        }
        // outputs: the lanes that answer for one column write a token each
        if (have) {
#pragma unroll
            for (int t = 0; t < DL_TB; ++t) {
                float o = r[4 + t];
#pragma unroll
                for (int j = 0; j <= t; ++j) o = fmaf(tl[6 + t * (t + 1) / 2 + j], u[j], o);
                const int tt = i * DL_TB + t;
                if (t % (KG / 4) == kg % (KG / 4) && tt < p.T) out[(long long)tt * p.H * p.Dv] = o;
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int i = 0; i < U * 2; ++i) {
        const int kc = (i >> 1) * 4 * KG + kg * 4 + (i & 1) * 2;
#pragma unroll
        for (int c = 0; c < DL_COLS; ++c) {
            const bool in = col_lane + c < p.Dv;
            if (in && kc < p.Dk) state[(long long)kc * p.Dv + col_lane + c] = S[i][c].x;
            if (in && kc + 1 < p.Dk) state[(long long)(kc + 1) * p.Dv + col_lane + c] = S[i][c].y;
        }
    }
}

// One token per row, the head's norm and sigmoid gate included.  Thread = row group * CQ + column quad; CQ (a
// power of two, at most 32) quads cover the head's columns.  ROWS state rows per thread are kept in
// registers; larger states (rows beyond ROWS * groups) are read a second time.
constexpr int DL_STEP_THREADS = 256;
template <typename T, int ROWS>
__global__ void __launch_bounds__(DL_STEP_THREADS) delta_step_kernel(const DeltaParams p, int CQ) {
    extern __shared__ __align__(16) float dl_smem[];
    float4 *s_kqw = reinterpret_cast<float4 *>(dl_smem);  // (Dk): k, q, w
    float4 *s_red = s_kqw + p.Dk;                          // (2, warps, CQ)
    __shared__ float s_part[3][DL_STEP_THREADS / 32];
    constexpr int NT = DL_STEP_THREADS, NW = NT / 32;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, RG = NT / CQ;
    const int h = blockIdx.x, b = blockIdx.y, g = h / (p.H / p.G), Dk = p.Dk, Dv = p.Dv;
    const int cq = tid % CQ, rg = tid / CQ, col = cq * 4;
    const bool have = col < Dv;
    float *state = p.state + ((long long)b * p.H + h) * Dk * Dv + col;
    float4 S[ROWS];
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const int r = rg + i * RG;
        S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (have && r < Dk) S[i] = *reinterpret_cast<const float4 *>(state + (long long)r * Dv);
    }
    float v4[4] = {0.f, 0.f, 0.f, 0.f}, gate[4] = {0.f, 0.f, 0.f, 0.f}, nw[4] = {0.f, 0.f, 0.f, 0.f};
    if (have) {
        get_v(static_cast<const T *>(p.v) + b * p.v_stride + (long long)h * Dv + col, v4);
        if (rg == 0) {
            get_v(static_cast<const T *>(p.gate) + b * p.gate_stride + (long long)h * Dv + col, gate);
            get_v(p.norm_w + col, nw);
        }
    }
    const float beta = Fn<T>::sigmoid(to_f(static_cast<const T *>(p.b)[b * p.b_stride + h])), rate = p.rate[h];
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int c = tid; c < Dk; c += NT) {
        const float q = to_f(static_cast<const T *>(p.q)[b * p.q_stride + (long long)g * Dk + c]);
        const float k = to_f(static_cast<const T *>(p.k)[b * p.k_stride + (long long)g * Dk + c]);
        const float w = Fn<T>::exp(-rate * softplus(p.x[b * p.x_stride + (long long)h * Dk + c] + p.x0[h * Dk + c]));
        s_kqw[c] = make_float4(k, q, w, 0.f);
        qq = fmaf(q, q, qq);
        kk = fmaf(k, k, kk);
        qk = fmaf(q, k, qk);
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    qk = warp_sum(qk);
    if (lane == 0) {
        s_part[0][warp] = qq;
        s_part[1][warp] = kk;
        s_part[2][warp] = qk;
    }
    __syncthreads();
    qq = kk = qk = 0.f;
#pragma unroll
    for (int i = 0; i < NW; ++i) {
        qq += s_part[0][i];
        kk += s_part[1][i];
        qk += s_part[2][i];
    }
    const float iq = rsqrtf((float)Dk) / sqrtf(qq + 1e-6f), ik = 1.f / sqrtf(kk + 1e-6f);
    // with the decayed state S: S^T k and S^T q in one pass; o = S^T q + (q . k) u
    float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
    auto pass = [&](float4 &s, int r) {
        const float4 f = s_kqw[r];
        s.x *= f.z; s.y *= f.z; s.z *= f.z; s.w *= f.z;
        ak.x = fmaf(f.x, s.x, ak.x); ak.y = fmaf(f.x, s.y, ak.y); ak.z = fmaf(f.x, s.z, ak.z); ak.w = fmaf(f.x, s.w, ak.w);
        aq.x = fmaf(f.y, s.x, aq.x); aq.y = fmaf(f.y, s.y, aq.y); aq.z = fmaf(f.y, s.z, aq.z); aq.w = fmaf(f.y, s.w, aq.w);
    };
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const int r = rg + i * RG;
        if (r < Dk) pass(S[i], r);
    }
    for (int r = rg + ROWS * RG; r < Dk; r += RG) {
        if (!have) break;
        float4 s = *reinterpret_cast<const float4 *>(state + (long long)r * Dv);
        pass(s, r);
    }
    for (int off = 16; off >= CQ; off >>= 1) {
        ak.x += __shfl_xor_sync(0xffffffffu, ak.x, off); ak.y += __shfl_xor_sync(0xffffffffu, ak.y, off);
        ak.z += __shfl_xor_sync(0xffffffffu, ak.z, off); ak.w += __shfl_xor_sync(0xffffffffu, ak.w, off);
        aq.x += __shfl_xor_sync(0xffffffffu, aq.x, off); aq.y += __shfl_xor_sync(0xffffffffu, aq.y, off);
        aq.z += __shfl_xor_sync(0xffffffffu, aq.z, off); aq.w += __shfl_xor_sync(0xffffffffu, aq.w, off);
    }
    if (lane < CQ) {
        s_red[warp * CQ + lane] = ak;
        s_red[(NW + warp) * CQ + lane] = aq;
    }
    __syncthreads();
    ak = aq = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NW; ++i) {
        const float4 x = s_red[i * CQ + cq], y = s_red[(NW + i) * CQ + cq];
        ak.x += x.x; ak.y += x.y; ak.z += x.z; ak.w += x.w;
        aq.x += y.x; aq.y += y.y; aq.z += y.z; aq.w += y.w;
    }
    float4 u;
    u.x = beta * (v4[0] - ik * ak.x); u.y = beta * (v4[1] - ik * ak.y);
    u.z = beta * (v4[2] - ik * ak.z); u.w = beta * (v4[3] - ik * ak.w);
    if (have) {
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            const int r = rg + i * RG;
            if (r >= Dk) continue;
            const float k = s_kqw[r].x * ik;
            *reinterpret_cast<float4 *>(state + (long long)r * Dv) =
                make_float4(fmaf(k, u.x, S[i].x), fmaf(k, u.y, S[i].y), fmaf(k, u.z, S[i].z), fmaf(k, u.w, S[i].w));
        }
        for (int r = rg + ROWS * RG; r < Dk; r += RG) {
            float4 s = *reinterpret_cast<const float4 *>(state + (long long)r * Dv);
            const float4 f = s_kqw[r];
            const float k = f.x * ik;
            *reinterpret_cast<float4 *>(state + (long long)r * Dv) =
                make_float4(fmaf(k, u.x, s.x * f.z), fmaf(k, u.y, s.y * f.z), fmaf(k, u.z, s.z * f.z), fmaf(k, u.w, s.w * f.z));
        }
    }
    if (warp > 0) return;  // CQ <= 32: the first warp holds every column
    const float dot = qk * iq * ik;
    float o[4] = {0.f, 0.f, 0.f, 0.f};
    if (rg == 0 && have) {
        o[0] = fmaf(dot, u.x, iq * aq.x); o[1] = fmaf(dot, u.y, iq * aq.y);
        o[2] = fmaf(dot, u.z, iq * aq.z); o[3] = fmaf(dot, u.w, iq * aq.w);
    }
    const float ss = warp_sum(fmaf(o[0], o[0], fmaf(o[1], o[1], fmaf(o[2], o[2], o[3] * o[3]))));
    const float inv = 1.f / sqrtf(ss / (float)Dv + p.eps);
    if (rg == 0 && have) {
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] *= inv * nw[e] * Fn<T>::sigmoid(gate[e]);
        put_v(static_cast<T *>(p.out) + ((long long)b * p.H + h) * Dv + col, o);
    }
}

static int delta_key_pad(int Dk) { return Dk <= 32 ? 32 : (Dk <= 64 ? 64 : (Dk <= 128 ? 128 : 256)); }

template <typename T, int KG, int U>
static cudaError_t delta_run(DeltaParams p, cudaStream_t s) {
    constexpr int cols = DL_WARPS * (32 / KG) * DL_COLS;
    const int smem = DL_RING * delta_record(4 * KG * U) * (int)sizeof(float);
    p.n_cols = (p.Dv + cols - 1) / cols;
    const cudaError_t e = cudaFuncSetAttribute(delta_kernel<T, KG, U>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    delta_kernel<T, KG, U><<<dim3(p.H * p.n_cols, p.B), DL_WARPS * 32, smem, s>>>(p);
    return cudaGetLastError();
}

template <typename T>
static cudaError_t delta_prompt(const DeltaParams &p, cudaStream_t s) {
    const long long warps = (long long)p.B * p.n_batches * p.H;
    const unsigned grid = (unsigned)((warps + 3) / 4);
    if (p.KP == 32) delta_prepare_kernel<T, 1><<<grid, 128, 0, s>>>(p);
    else if (p.KP == 64) delta_prepare_kernel<T, 2><<<grid, 128, 0, s>>>(p);
    else if (p.KP == 128) delta_prepare_kernel<T, 4><<<grid, 128, 0, s>>>(p);
    else delta_prepare_kernel<T, 8><<<grid, 128, 0, s>>>(p);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    // fewer lanes per column do the same work with fewer shuffles, but leave fewer warps
    const long long cols = (long long)p.B * p.H * p.Dv;
    const long long warps_at_8 = cols / 16;
    const bool many = warps_at_8 >= 8LL * sm_count(), some = 2 * warps_at_8 >= 8LL * sm_count();
    if (p.KP == 32) return delta_run<T, 8, 1>(p, s);
    if (p.KP == 64) return many ? delta_run<T, 8, 2>(p, s) : delta_run<T, 16, 1>(p, s);
    if (p.KP == 128) return many ? delta_run<T, 8, 4>(p, s) : (some ? delta_run<T, 16, 2>(p, s) : delta_run<T, 32, 1>(p, s));
    return many ? delta_run<T, 16, 4>(p, s) : delta_run<T, 32, 2>(p, s);
}

template <typename T>
static cudaError_t delta_step(const DeltaParams &p, cudaStream_t s) {
    int CQ = 1;
    while (CQ * 4 < p.Dv) CQ *= 2;
    const size_t smem = sizeof(float4) * (p.Dk + 2ull * (DL_STEP_THREADS / 32) * CQ);
    const dim3 grid(p.H, p.B);
    const int rows = (p.Dk * CQ + DL_STEP_THREADS - 1) / DL_STEP_THREADS;
    if (rows <= 4) delta_step_kernel<T, 4><<<grid, DL_STEP_THREADS, smem, s>>>(p, CQ);
    else if (rows <= 8) delta_step_kernel<T, 8><<<grid, DL_STEP_THREADS, smem, s>>>(p, CQ);
    else delta_step_kernel<T, 16><<<grid, DL_STEP_THREADS, smem, s>>>(p, CQ);
    return cudaGetLastError();
}

}  // namespace nckv

extern "C" {

size_t nckv_delta_workspace_bytes(int B, int T, int H, int Dk) {
    using namespace nckv;
    if (B <= 0 || T <= 0 || H <= 0 || Dk <= 0 || Dk > 256) return 0;
    return sizeof(float) * (size_t)B * H * ((T + DL_TB - 1) / DL_TB) * delta_record(delta_key_pad(Dk));
}

int nckv_delta_rule(const void *q, const void *k, const void *v, int64_t q_stride, int64_t k_stride, int64_t v_stride,
                    const float *x, int64_t x_stride, const float *x0, const float *rate, const void *b, int64_t b_stride,
                    float *out, float *state, int B, int T, int H, int G, int Dk, int Dv, int f32, void *workspace,
                    size_t workspace_bytes, void *stream) {
    using namespace nckv;
    if (!q || !k || !v || !x || !x0 || !rate || !b || !out || !state) {
        set_error("delta_rule: null pointer argument");
        return NCKV_E_ARG;
    }
    if (B <= 0 || T <= 0 || H <= 0 || G <= 0 || H % G || Dk <= 0 || Dv <= 0 || B > 65535) {
        set_error("delta_rule: size out of range (B=%d T=%d H=%d G=%d Dk=%d Dv=%d)", B, T, H, G, Dk, Dv);
        return NCKV_E_ARG;
    }
    if (Dk > 256) {
        set_error("delta_rule: %d key channels per head unsupported (at most 256)", Dk);
        return NCKV_E_UNSUPPORTED;
    }
    if (!workspace || ((uintptr_t)workspace & 15) || workspace_bytes < nckv_delta_workspace_bytes(B, T, H, Dk)) {
        set_error("delta_rule: workspace of %zu bytes given, %zu needed", workspace_bytes, nckv_delta_workspace_bytes(B, T, H, Dk));
        return NCKV_E_CAPACITY;
    }
    DeltaParams p = {};
    p.q = q; p.k = k; p.v = v; p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
    p.x = x; p.x_stride = x_stride; p.x0 = x0; p.rate = rate; p.b = b; p.b_stride = b_stride;
    p.records = static_cast<float *>(workspace); p.state = state; p.out = out;
    p.B = B; p.T = T; p.H = H; p.G = G; p.Dk = Dk; p.Dv = Dv;
    p.KP = delta_key_pad(Dk); p.n_batches = (T + DL_TB - 1) / DL_TB;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    NCKV_CUDA_CHECK(f32 ? delta_prompt<float>(p, s) : delta_prompt<__nv_bfloat16>(p, s));
    return NCKV_OK;
}

int nckv_delta_step(const void *q, const void *k, const void *v, int64_t q_stride, int64_t k_stride, int64_t v_stride,
                    const float *x, int64_t x_stride, const float *x0, const float *rate, const void *b, int64_t b_stride,
                    const void *gate, int64_t gate_stride, const float *norm_w, float eps, void *out, float *state, int B,
                    int H, int G, int Dk, int Dv, int f32, void *stream) {
    using namespace nckv;
    if (!q || !k || !v || !x || !x0 || !rate || !b || !gate || !norm_w || !out || !state) {
        set_error("delta_step: null pointer argument");
        return NCKV_E_ARG;
    }
    if (B <= 0 || H <= 0 || G <= 0 || H % G || Dk <= 0 || Dv <= 0 || B > 65535) {
        set_error("delta_step: size out of range (B=%d H=%d G=%d Dk=%d Dv=%d)", B, H, G, Dk, Dv);
        return NCKV_E_ARG;
    }
    const uintptr_t elem = f32 ? 4 : 2;
    const uintptr_t at = (uintptr_t)v | (uintptr_t)gate | (uintptr_t)out | (uintptr_t)(v_stride | gate_stride) * elem;
    if (Dv % 4 || Dv > 128 || Dk > 1024 || (at & (4 * elem - 1)) || (((uintptr_t)state | (uintptr_t)norm_w) & 15)) {
        set_error("delta_step: %d key and %d value channels or their alignment unsupported", Dk, Dv);
        return NCKV_E_UNSUPPORTED;
    }
    DeltaParams p = {};
    p.q = q; p.k = k; p.v = v; p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
    p.x = x; p.x_stride = x_stride; p.x0 = x0; p.rate = rate; p.b = b; p.b_stride = b_stride;
    p.gate = gate; p.gate_stride = gate_stride; p.norm_w = norm_w; p.eps = eps; p.out = out; p.state = state;
    p.B = B; p.T = 1; p.H = H; p.G = G; p.Dk = Dk; p.Dv = Dv;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    NCKV_CUDA_CHECK(f32 ? delta_step<float>(p, s) : delta_step<__nv_bfloat16>(p, s));
    return NCKV_OK;
}

}  // extern "C"
