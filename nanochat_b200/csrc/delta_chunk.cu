// The gated delta rule of delta.cu for bf16 prompts, in chunks of 16 tokens whose products run as m16n8k8 tf32
// matrix instructions.  Every fp32 operand enters as two tf32 terms (hi * hi + hi * lo + lo * hi, fp32 sums), which
// keeps about 22 bits of it; the state itself stays in fp32 accumulators.
//
// With c_t = w_1 .. w_t (products from the chunk's first token on) and the state S before the chunk
//   R_t = S^T (c_t k_t)      P_t = S^T (c_t q_t)
//   u = T (v - R)            T = (1 + diag(beta) A)^-1 diag(beta),   A_ti = sum_c k_t k_i w_(i+1) .. w_t  (i < t)
//   o = P + Q u              Q_ti = sum_c q_t k_i w_(i+1) .. w_t  (i <= t)
//   S <- diag(c_16) S + sum_i (w_(i+1) .. w_16 k_i) u_i^T
// Only products of decays appear (each <= 1), so nothing overflows however strong the decay.
//
//   delta_chunk_prepare_kernel   one CTA per (row, head, chunk), a thread per key channel: norms, decays, the scaled
//                                rows, A, Q and T, left as one record in the order the matrix fragments want
//   delta_chunk_kernel           a warp owns 16 value columns of one (row, head).  S^T (16 x Dk) lives in
//                                accumulator fragments: they are the left operand of the next chunk's products
//                                as they stand (the order of the summed index is free), so no value crosses
//                                lanes.  Records arrive by bulk copies through a ring in shared memory.
#include "vec_io.cuh"

namespace nckv {

constexpr int DC_T = 16;     // tokens per chunk
constexpr int DC_RING = 3;   // records in flight

__host__ __device__ constexpr int dc_row(int KP) { return KP + 16; }  // keeps 16-byte reads of 8 rows free of conflicts
// record: [c_t k_t : 16 rows][c_t q_t : 16 rows][k_i to the end : KP x 16 tokens][c_16 : KP][T : 16 x 16][Q : 16 x 16]
__host__ __device__ constexpr int dc_record(int KP) { return 2 * DC_T * dc_row(KP) + KP * DC_T + KP + 2 * DC_T * DC_T; }
// place of token i among the 16 summed positions: the four a lane of a fragment needs lie together
__device__ __forceinline__ int dc_place(int i) { return ((i & 7) >> 1) * 4 + ((i >> 3) << 1) + (i & 1); }

struct DeltaChunkParams {
    const __nv_bfloat16 *q, *k, *v;  // (B * T) rows; heads packed inside a row
    long long q_stride, k_stride, v_stride;
    const float *x;                  // (B * T) rows of H * Dk decay logits
    long long x_stride;
    const float *x0, *rate;          // (H * Dk), (H)
    const __nv_bfloat16 *b;          // (B * T) rows of H step-size logits
    long long b_stride;
    float *records;                  // (B, H, chunks, dc_record(KP))
    float *state;                    // (B, H, Dk, Dv)
    float *out;                      // (B * T, H * Dv)
    int32_t *status;
    int B, T, H, G, Dk, Dv, n_chunks, n_cols;
};

// sums of o[0 .. LEN) over the warp: each level halves what a lane still holds.  Returns the index a lane ends with.
template <int BIT, int LEN> __device__ __forceinline__ int scatter_sum(float *o, int lane) {
    if constexpr (LEN == 1) {
        return 0;
    } else {
        constexpr int HALF = LEN / 2;
        const bool up = (lane & BIT) != 0;
#pragma unroll
        for (int c = 0; c < HALF; ++c) {
            const float keep = up ? o[c + HALF] : o[c], give = up ? o[c] : o[c + HALF];
            o[c] = keep + __shfl_xor_sync(0xffffffffu, give, BIT);
        }
        return (up ? HALF : 0) + scatter_sum<BIT / 2, HALF>(o, lane);
    }
}

template <int KP>
__global__ void __launch_bounds__(KP, 640 / KP) delta_chunk_prepare_kernel(const DeltaChunkParams p) {
    constexpr int NW = KP / 32;
    __shared__ float s_sum[DC_T / 2][NW][32], s_pair[DC_T * DC_T], s_beta[DC_T], s_scale[2][DC_T];
    const int c = threadIdx.x, lane = c & 31, warp = c >> 5;
    const int h = blockIdx.x % p.H, chunk = blockIdx.x / p.H, b = blockIdx.y;  // heads fastest: rows are shared in L2
    const int g = h / (p.H / p.G), t0 = chunk * DC_T, n = min(DC_T, p.T - t0);
    const bool on = c < p.Dk;
    const float rate = p.rate[h], x0 = on ? p.x0[h * p.Dk + c] : 0.f;
    const long long row = (long long)b * p.T + t0;
    const __nv_bfloat16 *gq = p.q + row * p.q_stride + (long long)g * p.Dk + c, *gk = p.k + row * p.k_stride + (long long)g * p.Dk + c;
    const float *gx = p.x + row * p.x_stride + (long long)h * p.Dk + c;
    float q[DC_T], k[DC_T], w[DC_T];  // tokens behind the last leave the state as it is
#pragma unroll
    for (int t = 0; t < DC_T; ++t) {
        const bool in = on && t < n;
        q[t] = in ? to_f(gq[t * p.q_stride]) : 0.f;
        k[t] = in ? to_f(gk[t * p.k_stride]) : 0.f;
        w[t] = in ? gx[t * p.x_stride] : 0.f;
    }
    if (c < DC_T) s_beta[c] = c < n ? Fn<__nv_bfloat16>::sigmoid(to_f(p.b[(row + c) * p.b_stride + h])) : 0.f;
    float part[32];
#pragma unroll
    for (int t = 0; t < DC_T; ++t) {
        part[t] = q[t] * q[t];
        part[DC_T + t] = k[t] * k[t];
        // softplus in the fast functions: what it loses for very negative logits is far below one rounding of w
        const float z = w[t] + x0;
        w[t] = on && t < n ? __expf(-rate * (fmaxf(z, 0.f) + __logf(1.f + __expf(-fabsf(z))))) : 1.f;
    }
    {
        const int at = scatter_sum<16, 32>(part, lane);
        s_sum[0][warp][at] = part[0];
    }
    __syncthreads();
    if (c < 32) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < NW; ++i) s += s_sum[0][i][c];
        s_scale[c >> 4][c & 15] = (c < DC_T ? rsqrtf((float)p.Dk) : 1.f) / sqrtf(s + 1e-6f);
    }
    __syncthreads();  // also: the sums above have been read
#pragma unroll
    for (int t = 0; t < DC_T; ++t) {
        q[t] *= s_scale[0][t];
        k[t] *= s_scale[1][t];
    }
    float *rec = p.records + (((long long)b * p.H + h) * p.n_chunks + chunk) * dc_record(KP);
    {
        float cum = 1.f;
#pragma unroll
        for (int t = 0; t < DC_T; ++t) {
            cum *= w[t];
            rec[t * dc_row(KP) + c] = cum * k[t];
            rec[(DC_T + t) * dc_row(KP) + c] = cum * q[t];
        }
        rec[2 * DC_T * dc_row(KP) + KP * DC_T + c] = cum;
    }
    // Row t of A and Q: k_i carried to token t, times k_t and q_t, summed over the channels.  The t + (t + 1) entries
    // of row t are numbers t^2 .. of 256 (A_ti is t^2 + i, Q_ti is t^2 + t + i); 32 at a time are summed.
    float ki[DC_T];
#pragma unroll
    for (int t = 0; t < DC_T; ++t) {
#pragma unroll
        for (int i = 0; i < t; ++i) ki[i] *= w[t];
        ki[t] = k[t];
#pragma unroll
        for (int e = 0; e < 2 * t + 1; ++e) {
            const int at = t * t + e;
            part[at % 32] = e < t ? k[t] * ki[e] : q[t] * ki[e >= t ? e - t : 0];
            if (at % 32 == 31) {
                const int mine = scatter_sum<16, 32>(part, lane);
                s_sum[at / 32][warp][mine] = part[0];
            }
        }
    }
    {
        // this channel's 16 tokens in the order of dc_place
        float4 *dst = reinterpret_cast<float4 *>(rec + 2 * DC_T * dc_row(KP) + c * DC_T);
#pragma unroll
        for (int i = 0; i < 4; ++i) dst[i] = make_float4(ki[2 * i], ki[2 * i + 1], ki[8 + 2 * i], ki[9 + 2 * i]);
    }
    __syncthreads();
    for (int i = c; i < DC_T * DC_T; i += KP) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < NW; ++j) s += s_sum[i >> 5][j][i & 31];
        s_pair[i] = s;
    }
    __syncthreads();
    float *tail = rec + 2 * DC_T * dc_row(KP) + KP * DC_T + KP;
    if (c < DC_T) {  // column c of T by forward substitution
        float u[DC_T];
#pragma unroll
        for (int t = 0; t < DC_T; ++t) {
            float s = t == c ? 1.f : 0.f;
#pragma unroll
            for (int i = 0; i < DC_T; ++i)
                if (i < t) s = fmaf(-s_pair[t * t + i], u[i], s);  // u[i] is zero for i < c
            u[t] = s_beta[t] * s;
            tail[t * DC_T + dc_place(c)] = u[t];
        }
    }
    for (int i = c; i < DC_T * DC_T; i += KP) {
        const int t = i / DC_T, j = i % DC_T;
        tail[DC_T * DC_T + t * DC_T + dc_place(j)] = j <= t ? s_pair[t * t + t + j] : 0.f;
    }
}

__device__ __forceinline__ void mma_tf32(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x = hi + lo: hi keeps the bits a tf32 operand has, lo the rest
__device__ __forceinline__ void split_tf32(float x, uint32_t &hi, uint32_t &lo) {
    hi = __float_as_uint(x) & 0xffffe000u;
    lo = __float_as_uint(x - __uint_as_float(hi));
}
struct Pair4 {  // the B values of two summed steps (x, y and z, w) in two terms
    uint32_t hi[4], lo[4];
    __device__ __forceinline__ explicit Pair4(const float4 &f) {
        split_tf32(f.x, hi[0], lo[0]);
        split_tf32(f.y, hi[1], lo[1]);
        split_tf32(f.z, hi[2], lo[2]);
        split_tf32(f.w, hi[3], lo[3]);
    }
};
struct LeftFrag {  // an accumulator fragment as left operand
    uint32_t hi[4], lo[4];
    __device__ __forceinline__ explicit LeftFrag(const float (&s)[4]) {
        // accumulator (g, 2t) (g, 2t+1) (g+8, 2t) (g+8, 2t+1); operand (g, t) (g+8, t) (g, t+4) (g+8, t+4)
        split_tf32(s[0], hi[0], lo[0]);
        split_tf32(s[2], hi[1], lo[1]);
        split_tf32(s[1], hi[2], lo[2]);
        split_tf32(s[3], hi[3], lo[3]);
    }
};

// d (16 x 16 tokens) = x times the transpose of a lower triangular 16 x 16 matrix; at: row g, this lane's four places
__device__ __forceinline__ void small_product(float (&d)[2][4], const LeftFrag &x0, const LeftFrag &x1, const float *at) {
    const Pair4 b0(*reinterpret_cast<const float4 *>(at)), b1(*reinterpret_cast<const float4 *>(at + 8 * DC_T));
    float t[9][4];
#pragma unroll
    for (int i = 0; i < 9; ++i) t[i][0] = t[i][1] = t[i][2] = t[i][3] = 0.f;
    mma_tf32(t[0], x0.hi, b0.hi[0], b0.hi[1]);  // tokens 0-7 take nothing from 8-15
    mma_tf32(t[1], x0.hi, b0.lo[0], b0.lo[1]);
    mma_tf32(t[2], x0.lo, b0.hi[0], b0.hi[1]);
    mma_tf32(t[3], x0.hi, b1.hi[0], b1.hi[1]);
    mma_tf32(t[4], x0.hi, b1.lo[0], b1.lo[1]);
    mma_tf32(t[5], x0.lo, b1.hi[0], b1.hi[1]);
    mma_tf32(t[6], x1.hi, b1.hi[2], b1.hi[3]);
    mma_tf32(t[7], x1.hi, b1.lo[2], b1.lo[3]);
    mma_tf32(t[8], x1.lo, b1.hi[2], b1.hi[3]);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        d[0][e] = t[0][e] + (t[1][e] + t[2][e]);
        d[1][e] = (t[3][e] + t[6][e]) + ((t[4][e] + t[5][e]) + (t[7][e] + t[8][e]));
    }
}

__device__ __forceinline__ void bulk_load(void *smem_dst, const void *src, uint32_t bytes, uint64_t *bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(smem_dst)),
                 "l"(src), "r"(bytes), "r"(smem_u32(bar))
                 : "memory");
}

// fragment tiles 2 j and 2 j + 1 hold channels 16 j + 4 t + {0, 1} and + {2, 3} in columns 2 t and 2 t + 1.
// SPLIT > 1 (few heads): the CTA's SPLIT warps share 16 columns, each holding KP / SPLIT key channels; their
// partial R and P meet in shared memory, everything else stays apart.
template <int KP, int SPLIT>
__global__ void __launch_bounds__(128) delta_chunk_kernel(const DeltaChunkParams p) {
    constexpr int J = KP / 16 / SPLIT, RS = dc_row(KP), REC = dc_record(KP);
    static_assert(J >= 2 && J % 2 == 0, "the update takes two channel groups at a time");
    extern __shared__ __align__(128) float dc_smem[];
    __shared__ uint64_t bar[DC_RING];
    __shared__ float4 s_part[SPLIT > 1 ? 2 : 1][SPLIT][4][32];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tg = lane & 3;
    const int part = SPLIT > 1 ? warp : 0, c0 = part * (KP / SPLIT);  // this warp's first key channel
    const int h = blockIdx.x / p.n_cols, b = blockIdx.y;
    const int groups = SPLIT > 1 ? 1 : blockDim.x >> 5;
    const int col = ((blockIdx.x % p.n_cols) * groups + (SPLIT > 1 ? 0 : warp)) * 16 + g;  // this lane's columns: col, col + 8
    const bool on0 = col < p.Dv, on1 = col + 8 < p.Dv;
    const float *src = p.records + ((long long)b * p.H + h) * p.n_chunks * REC;
    auto fetch = [&](int i) {  // by one thread
        mbar_arrive_expect_tx(&bar[i % DC_RING], REC * 4);
        bulk_load(dc_smem + (i % DC_RING) * REC, src + (long long)i * REC, REC * 4, &bar[i % DC_RING]);
    };
    int fetched = 0;
    if (tid == 0) {
        for (int i = 0; i < DC_RING; ++i) mbar_init(&bar[i], 1);
        fence_mbar_init();
        for (; fetched < DC_RING && fetched < p.n_chunks; ++fetched) fetch(fetched);
    }

    float S[2 * J][4];
    float *state = p.state + (((long long)b * p.H + h) * p.Dk + c0) * p.Dv + col;
#pragma unroll
    for (int i = 0; i < 2 * J; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int ch = (i >> 1) * 16 + 4 * tg + (i & 1) * 2 + e;
            S[i][e] = on0 && c0 + ch < p.Dk ? state[(long long)ch * p.Dv] : 0.f;
            S[i][2 + e] = on1 && c0 + ch < p.Dk ? state[(long long)ch * p.Dv + 8] : 0.f;
        }
    const __nv_bfloat16 *v = p.v + (long long)b * p.T * p.v_stride + (long long)h * p.Dv + col;
    float *out = p.out + (long long)b * p.T * p.H * p.Dv + (long long)h * p.Dv + col;
    const long long out_row = (long long)p.H * p.Dv;
    __nv_bfloat16 v_raw[2][4];  // [half of the tokens][(g, 2t) (g, 2t+1) (g+8, 2t) (g+8, 2t+1)]
    auto load_v = [&](int i) {
#pragma unroll
        for (int s = 0; s < 2; ++s)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = i * DC_T + 8 * s + 2 * tg + e;
                const __nv_bfloat16 *at = v + t * p.v_stride;
                v_raw[s][e] = on0 && t < p.T ? at[0] : __float2bfloat16_rn(0.f);
                v_raw[s][2 + e] = on1 && t < p.T ? at[8] : __float2bfloat16_rn(0.f);
            }
    };
    load_v(0);
    __syncthreads();

    bool failed = false;
    for (int i = 0; i < p.n_chunks; ++i) {
        int ok = 1;
        if (lane == 0) ok = mbar_wait_bounded(&bar[i % DC_RING], (i / DC_RING) & 1u) ? 1 : 0;
        ok = __shfl_sync(0xffffffffu, ok, 0);
        __syncwarp();
        const float *rec = dc_smem + (i % DC_RING) * REC;
        // A matrix instruction takes longer to finish than to issue: neighbours in the order below add to
        // different accumulators.
        // R^T (tokens 0-7, 8-15) and P^T: 16 columns of v by 32 token rows; cross terms summed apart
        float r[4][4], rc[4][4];
#pragma unroll
        for (int m = 0; m < 4; ++m)
#pragma unroll
            for (int e = 0; e < 4; ++e) r[m][e] = rc[m][e] = 0.f;
        if (ok) {
#pragma unroll
            for (int j = 0; j < J; ++j) {
                const LeftFrag a0(S[2 * j]), a1(S[2 * j + 1]);
                const float *at = rec + g * RS + c0 + 16 * j + 4 * tg;
                const Pair4 bb[4] = {Pair4(*reinterpret_cast<const float4 *>(at)), Pair4(*reinterpret_cast<const float4 *>(at + 8 * RS)),
                                     Pair4(*reinterpret_cast<const float4 *>(at + 16 * RS)), Pair4(*reinterpret_cast<const float4 *>(at + 24 * RS))};
#pragma unroll
                for (int m = 0; m < 4; ++m) mma_tf32(r[m], a0.hi, bb[m].hi[0], bb[m].hi[1]);
#pragma unroll
                for (int m = 0; m < 4; ++m) mma_tf32(rc[m], a0.hi, bb[m].lo[0], bb[m].lo[1]);
#pragma unroll
                for (int m = 0; m < 4; ++m) mma_tf32(r[m], a1.hi, bb[m].hi[2], bb[m].hi[3]);
#pragma unroll
                for (int m = 0; m < 4; ++m) mma_tf32(rc[m], a0.lo, bb[m].hi[0], bb[m].hi[1]);
#pragma unroll
                for (int m = 0; m < 4; ++m) mma_tf32(rc[m], a1.hi, bb[m].lo[2], bb[m].lo[3]);
#pragma unroll
                for (int m = 0; m < 4; ++m) mma_tf32(rc[m], a1.lo, bb[m].hi[2], bb[m].hi[3]);
            }
        }
#pragma unroll
        for (int m = 0; m < 4; ++m)
#pragma unroll
            for (int e = 0; e < 4; ++e) r[m][e] += rc[m][e];
        if (SPLIT > 1) {
#pragma unroll
            for (int m = 0; m < 4; ++m) s_part[i & 1][part][m][lane] = make_float4(r[m][0], r[m][1], r[m][2], r[m][3]);
        }
        failed = __syncthreads_or(!ok);  // behind it nobody reads the record before this one any more
        if (failed) break;
        if (tid == 0 && i > 0 && fetched < p.n_chunks) fetch(fetched++);
        if (SPLIT > 1) {
#pragma unroll
            for (int m = 0; m < 4; ++m) {
                if (m >= 2 && part != m - 2) continue;  // warp 0 and 1 answer for the outputs of 8 tokens each
                r[m][0] = r[m][1] = r[m][2] = r[m][3] = 0.f;
#pragma unroll
                for (int w = 0; w < SPLIT; ++w) {  // in the same order in every warp
                    const float4 f = s_part[i & 1][w][m][lane];
                    r[m][0] += f.x; r[m][1] += f.y; r[m][2] += f.z; r[m][3] += f.w;
                }
            }
        }
        const float *tail = rec + 2 * DC_T * RS + KP * DC_T + KP;
        float u[2][4];
#pragma unroll
        for (int s = 0; s < 2; ++s)
#pragma unroll
            for (int e = 0; e < 4; ++e) r[s][e] = to_f(v_raw[s][e]) - r[s][e];
        if (i + 1 < p.n_chunks) load_v(i + 1);
        // u^T = (v - R)^T T^T
        small_product(u, LeftFrag(r[0]), LeftFrag(r[1]), tail + g * DC_T + 4 * tg);
        const LeftFrag u0(u[0]), u1(u[1]);
        // S^T <- S^T diag(c_16) + u^T K, four tiles at a time
        const float *kt = rec + 2 * DC_T * RS, *cw = kt + KP * DC_T;
#pragma unroll
        for (int j = 0; j < J; j += 2) {
            float (&s0)[4] = S[2 * j], (&s1)[4] = S[2 * j + 1], (&s2)[4] = S[2 * j + 2], (&s3)[4] = S[2 * j + 3];
            const float4 f = *reinterpret_cast<const float4 *>(cw + c0 + 16 * j + 4 * tg);
            const float4 f2 = *reinterpret_cast<const float4 *>(cw + c0 + 16 * j + 16 + 4 * tg);
            s0[0] *= f.x; s0[1] *= f.y; s0[2] *= f.x; s0[3] *= f.y;
            s1[0] *= f.z; s1[1] *= f.w; s1[2] *= f.z; s1[3] *= f.w;
            s2[0] *= f2.x; s2[1] *= f2.y; s2[2] *= f2.x; s2[3] *= f2.y;
            s3[0] *= f2.z; s3[1] *= f2.w; s3[2] *= f2.z; s3[3] *= f2.w;
            const float *at = kt + (c0 + 16 * j + 4 * (g >> 1) + (g & 1)) * DC_T + 4 * tg;
            const Pair4 b0(*reinterpret_cast<const float4 *>(at)), b1(*reinterpret_cast<const float4 *>(at + 2 * DC_T)),
                b2(*reinterpret_cast<const float4 *>(at + 16 * DC_T)), b3(*reinterpret_cast<const float4 *>(at + 18 * DC_T));
            auto term = [&](const uint32_t (&a)[4], int lo, int at0) {
                mma_tf32(s0, a, lo ? b0.lo[at0] : b0.hi[at0], lo ? b0.lo[at0 + 1] : b0.hi[at0 + 1]);
                mma_tf32(s1, a, lo ? b1.lo[at0] : b1.hi[at0], lo ? b1.lo[at0 + 1] : b1.hi[at0 + 1]);
                mma_tf32(s2, a, lo ? b2.lo[at0] : b2.hi[at0], lo ? b2.lo[at0 + 1] : b2.hi[at0 + 1]);
                mma_tf32(s3, a, lo ? b3.lo[at0] : b3.hi[at0], lo ? b3.lo[at0 + 1] : b3.hi[at0 + 1]);
            };
            term(u0.hi, 0, 0);
            term(u1.hi, 0, 2);
            term(u0.hi, 1, 0);
            term(u1.hi, 1, 2);
            term(u0.lo, 0, 0);
            term(u1.lo, 0, 2);
        }
        // o^T = P^T + u^T Q^T
        if (SPLIT == 1 || part < 2) {
            float o[2][4];
            small_product(o, u0, u1, tail + DC_T * DC_T + g * DC_T + 4 * tg);
#pragma unroll
            for (int s = 0; s < 2; ++s) {
                if (SPLIT > 1 && part != s) continue;
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int t = i * DC_T + 8 * s + 2 * tg + e;
                    if (t < p.T && on0) out[t * out_row] = r[2 + s][e] + o[s][e];
                    if (t < p.T && on1) out[t * out_row + 8] = r[2 + s][2 + e] + o[s][2 + e];
                }
            }
        }
    }
    if (failed) {
        if (tid == 0) {
            atomicOr(p.status, (int)NCKV_ST_TIMEOUT);
            // copies already issued land before the CTA's memory is released
            for (int f = fetched > DC_RING ? fetched - DC_RING : 0; f < fetched; ++f)
                mbar_wait_bounded(&bar[f % DC_RING], (f / DC_RING) & 1u, 100000000ull);
        }
        __syncthreads();
        return;
    }
#pragma unroll
    for (int j = 0; j < 2 * J; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int ch = (j >> 1) * 16 + 4 * tg + (j & 1) * 2 + e;
            if (on0 && c0 + ch < p.Dk) state[(long long)ch * p.Dv] = S[j][e];
            if (on1 && c0 + ch < p.Dk) state[(long long)ch * p.Dv + 8] = S[j][2 + e];
        }
}

static int dc_pad(int Dk) { return Dk <= 32 ? 32 : (Dk <= 64 ? 64 : 128); }

template <int KP, int SPLIT> static cudaError_t dc_rule(const DeltaChunkParams &p, int warps, cudaStream_t s) {
    const int smem = DC_RING * dc_record(KP) * (int)sizeof(float);
    const cudaError_t e = cudaFuncSetAttribute(delta_chunk_kernel<KP, SPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    delta_chunk_kernel<KP, SPLIT><<<dim3(p.H * p.n_cols, p.B), warps * 32, smem, s>>>(p);
    return cudaGetLastError();
}

template <int KP> static cudaError_t dc_run(DeltaChunkParams p, cudaStream_t s) {
    delta_chunk_prepare_kernel<KP><<<dim3(p.n_chunks * p.H, p.B), KP, 0, s>>>(p);
    const cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    // few heads: several warps to 16 columns; many: CTAs whose warps share a record between their columns
    constexpr int MOST = KP / 32;
    const int per_head = (p.Dv + 15) / 16;
    const long long groups = (long long)p.B * p.H * per_head;
    p.n_cols = per_head;
    if (MOST >= 4 && groups * 2 <= 4LL * sm_count()) return dc_rule<KP, MOST >= 4 ? 4 : 1>(p, 4, s);
    if (MOST >= 2 && groups <= 4LL * sm_count()) return dc_rule<KP, MOST >= 2 ? 2 : 1>(p, 2, s);
    int warps = 1;
    while (warps < 4 && warps < per_head && (long long)p.B * p.H * ((per_head + 2 * warps - 1) / (2 * warps)) >= sm_count()) warps *= 2;
    p.n_cols = (per_head + warps - 1) / warps;
    return dc_rule<KP, 1>(p, warps, s);
}

}  // namespace nckv

extern "C" {

size_t nckv_delta_chunk_workspace_bytes(int B, int T, int H, int Dk) {
    using namespace nckv;
    if (B <= 0 || T <= 0 || H <= 0 || Dk <= 0 || Dk > 128) return 0;
    return sizeof(float) * (size_t)B * H * ((T + DC_T - 1) / DC_T) * dc_record(dc_pad(Dk));
}

int nckv_delta_chunk(const void *q, const void *k, const void *v, int64_t q_stride, int64_t k_stride, int64_t v_stride,
                     const float *x, int64_t x_stride, const float *x0, const float *rate, const void *b, int64_t b_stride,
                     float *out, float *state, int B, int T, int H, int G, int Dk, int Dv, void *workspace,
                     size_t workspace_bytes, int32_t *status, void *stream) {
    using namespace nckv;
    if (!q || !k || !v || !x || !x0 || !rate || !b || !out || !state || !status) {
        set_error("delta_chunk: null pointer argument");
        return NCKV_E_ARG;
    }
    if (B <= 0 || T <= 0 || H <= 0 || G <= 0 || H % G || Dk <= 0 || Dv <= 0 || B > 65535) {
        set_error("delta_chunk: size out of range (B=%d T=%d H=%d G=%d Dk=%d Dv=%d)", B, T, H, G, Dk, Dv);
        return NCKV_E_ARG;
    }
    if (Dk > 128) {
        set_error("delta_chunk: %d key channels per head unsupported (at most 128)", Dk);
        return NCKV_E_UNSUPPORTED;
    }
    if (!workspace || ((uintptr_t)workspace & 15) || workspace_bytes < nckv_delta_chunk_workspace_bytes(B, T, H, Dk)) {
        set_error("delta_chunk: workspace of %zu bytes given, %zu needed", workspace_bytes, nckv_delta_chunk_workspace_bytes(B, T, H, Dk));
        return NCKV_E_CAPACITY;
    }
    DeltaChunkParams p;
    p.q = static_cast<const __nv_bfloat16 *>(q); p.k = static_cast<const __nv_bfloat16 *>(k); p.v = static_cast<const __nv_bfloat16 *>(v);
    p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
    p.x = x; p.x_stride = x_stride; p.x0 = x0; p.rate = rate;
    p.b = static_cast<const __nv_bfloat16 *>(b); p.b_stride = b_stride;
    p.records = static_cast<float *>(workspace); p.state = state; p.out = out; p.status = status;
    p.B = B; p.T = T; p.H = H; p.G = G; p.Dk = Dk; p.Dv = Dv;
    p.n_chunks = (T + DC_T - 1) / DC_T; p.n_cols = 1;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const int KP = dc_pad(Dk);
    NCKV_CUDA_CHECK(KP == 32 ? dc_run<32>(p, s) : (KP == 64 ? dc_run<64>(p, s) : dc_run<128>(p, s)));
    return NCKV_OK;
}

}  // extern "C"
