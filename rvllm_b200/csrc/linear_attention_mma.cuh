// The tensor-core forms of linear_attention.cu's `state` and `out` kernels (bfloat16 rows, d and dv
// in multiples of 16, d up to 128); included by that file, whose first comment explains them.
#pragma once

#define LM_LD 72            // padded row of 64 bfloat16 columns

__device__ __forceinline__ unsigned lm_silu2(unsigned u) {
    const float2 f = lm_pair(u);
    const __nv_bfloat162 r = __floats2bfloat162_rn(la_silu(f.x), la_silu(f.y));
    return *(const unsigned*)&r;
}
// Eight projections of one token, as the recurrence reads them.
__device__ __forceinline__ uint4 lm_in8(const bf16* p, bool there, int act) {
    uint4 v = there ? *(const uint4*)p : make_uint4(0, 0, 0, 0);
    if (act) {
        v.x = lm_silu2(v.x);
        v.y = lm_silu2(v.y);
        v.z = lm_silu2(v.z);
        v.w = lm_silu2(v.w);
    }
    return v;
}
__device__ __forceinline__ float lm_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// z -> B: what the tokens of a chunk up to and with this one keep of a channel, as a power of two
// (sums of log2 a), in place, so that neither of the kernels below repeats it for its tiles.  A
// warp has eight tokens of 32 channels.
#define LM_STRONG -57.7f    // -40 log2 e
__global__ void __launch_bounds__(256) la_decay_kernel(float* __restrict__ z, const float* __restrict__ bias,
                                                       float scale, const int* __restrict__ q_start,
                                                       const int* __restrict__ state_slot, int first_req,
                                                       int n_reqs, int width) {
    rv_pdl_launch_dependents();
    __shared__ float tot[8][32];
    __shared__ int at[2];
    const int lane = threadIdx.x & 31, g = threadIdx.x >> 5, c = blockIdx.y * 32 + lane;
    if (threadIdx.x < 32) {
        int r = -1, before = 0;
        const bool ok = la_find(q_start, state_slot, first_req, n_reqs, blockIdx.x, lane, r, before);
        if (lane == 0) {
            at[0] = ok ? q_start[r] + ((int)blockIdx.x - before) * LA_C : -1;
            at[1] = ok ? min(LA_C, q_start[r + 1] - at[0]) : 0;
        }
    }
    __syncthreads();
    const int t0 = at[0], L = at[1];
    const float b = c < width ? bias[c] : 0.f;
    rv_pdl_wait();
    if (t0 < 0) return;
    float v[8], s = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j)
        v[j] = 8 * g + j < L && c < width ? z[(size_t)(t0 + 8 * g + j) * width + c] : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        s += la_logsigmoid(v[j] + b) * scale;
        v[j] = s;
    }
    tot[g][lane] = s;
    __syncthreads();
    float before = 0.f;
    for (int i = 0; i < g; ++i) before += tot[i][lane];
#pragma unroll
    for (int j = 0; j < 8; ++j)
        if (8 * g + j < L && c < width) z[(size_t)(t0 + 8 * g + j) * width + c] = before + v[j];
}

// KV = sum_j (k_j e^(B_L - B_j)) v_j^T for 64 channels by 64 columns: a warp has 16 channels.
template <int MODE>
__global__ void __launch_bounds__(128) la_state_mma_kernel(
    const bf16* __restrict__ rows, int stride, const LaRows lr, const LaToken tk, const float* __restrict__ zb,
    const float* __restrict__ log_decay,
    const int* __restrict__ q_start, const int* __restrict__ state_slot, int first_req, int n_reqs,
    float* __restrict__ kv, float* __restrict__ dec, int H, int d, int dv, int act) {
    constexpr bool CHANNEL = MODE == LA_CHANNEL, TOKEN = MODE == LA_TOKEN;
    rv_pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char smraw[];
    bf16* ks = (bf16*)smraw;                            // [3][64 tokens][LM_LD]
    bf16* vs = ks + 3 * LA_C * LM_LD;                   // [64 tokens][LM_LD]
    __shared__ int at[2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int item = blockIdx.x, h = blockIdx.y;
    const int tiles_v = (dv + LA_T - 1) / LA_T;
    const int d0 = (blockIdx.z / tiles_v) * LA_T, v0 = (blockIdx.z % tiles_v) * LA_T;
    lm_locate(q_start, state_slot, first_req, n_reqs, item, at);
    const int t0 = at[0], L = at[1];
    rv_pdl_wait();
    if (t0 < 0) return;
    const int dn = min(LA_T, d - d0), vn = min(LA_T, dv - v0);
    const bf16* base = rows + (size_t)t0 * stride;
    const float ld = MODE != LA_CONST ? 0.f : log_decay[h];
    const int kh = h / lr.share;
    const double last = TOKEN ? tk.B[(size_t)(t0 + L - 1) * H + h] : 0.;
    // eight columns a thread: 8 chunks a row, 16 rows a round, 4 rounds
    const int ch = tid & 7, jr = tid >> 3;
    uint4 kreg[4], vreg[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
        const int j = jr + 16 * u;
        const bf16* row = base + (size_t)j * stride;
        kreg[u] = lm_in8(row + lr.k + kh * d + d0 + 8 * ch, j < L && 8 * ch < dn, act);
        vreg[u] = lm_in8(row + lr.v + h * dv + v0 + 8 * ch, j < L && 8 * ch < vn, act);
    }
    float bl[8];                                        // CHANNEL: B of the chunk's last token
    if (CHANNEL) {
        const float* p = zb + (size_t)(t0 + L - 1) * H * d + h * d + d0;
#pragma unroll
        for (int e = 0; e < 8; ++e) bl[e] = 8 * ch < dn ? p[8 * ch + e] : 0.f;
        if (v0 == 0 && jr == 0 && 8 * ch < dn)
#pragma unroll
            for (int e = 0; e < 8; ++e)
                dec[((size_t)item * H + h) * d + d0 + 8 * ch + e] = lm_exp2(bl[e]);
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
        const int j = jr + 16 * u;
        *(uint4*)(vs + j * LM_LD + 8 * ch) = vreg[u];
        const unsigned in[4] = {kreg[u].x, kreg[u].y, kreg[u].z, kreg[u].w};
        unsigned o[3][4];
        float f = 0.f, bj[8];
        if (MODE == LA_CONST) f = expf(ld * (float)(L - 1 - min(j, L - 1)));
        if (TOKEN) {
            const size_t at_j = (size_t)(t0 + min(j, L - 1)) * H + h;
            f = expf((float)(last - tk.B[at_j])) * tk.w[at_j];
        }
        if (CHANNEL) {
            const float* p = zb + (size_t)(t0 + min(j, L - 1)) * H * d + h * d + d0 + 8 * ch;
#pragma unroll
            for (int e = 0; e < 8; e += 4) {
                const float4 x = 8 * ch < dn ? *(const float4*)(p + e) : make_float4(0.f, 0.f, 0.f, 0.f);
                bj[e] = x.x; bj[e + 1] = x.y; bj[e + 2] = x.z; bj[e + 3] = x.w;
            }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float2 k2 = lm_pair(in[e]);
            float fx = f, fy = f;
            if (CHANNEL) {
                fx = lm_exp2(bl[2 * e] - bj[2 * e]);
                fy = lm_exp2(bl[2 * e + 1] - bj[2 * e + 1]);
            }
            lm_split(k2.x * fx, k2.y * fy, o[0][e], o[1][e], o[2][e]);
        }
#pragma unroll
        for (int s = 0; s < 3; ++s)
            *(uint4*)(ks + (s * LA_C + j) * LM_LD + 8 * ch) = make_uint4(o[s][0], o[s][1], o[s][2], o[s][3]);
    }
    __syncthreads();
    if (16 * warp >= dn) return;
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const int nk = (L + 15) >> 4;
    for (int kk = 0; kk < nk; ++kk) {
        unsigned a[3][4];
#pragma unroll
        for (int s = 0; s < 3; ++s)
            ldmatrix_x4_trans(a[s], ks + (s * LA_C + kk * 16 + (lane & 7) + (lane >> 4) * 8) * LM_LD +
                                        16 * warp + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int nd = 0; nd < 4; ++nd) {
            if (16 * nd >= vn) continue;
            unsigned b[4];
            ldmatrix_x4_trans(b, vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LM_LD + nd * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int s = 2; s >= 0; --s) {
                mma_bf16(acc[2 * nd], a[s], b[0], b[1]);
                mma_bf16(acc[2 * nd + 1], a[s], b[2], b[3]);
            }
        }
    }
    float* o = kv + ((size_t)item * H + h) * d * dv + (size_t)(d0 + 16 * warp + (lane >> 2)) * dv + v0 + (lane & 3) * 2;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        if (8 * i >= vn) continue;
        *(float2*)(o + 8 * i) = make_float2(acc[i][0], acc[i][1]);
        *(float2*)(o + (size_t)8 * dv + 8 * i) = make_float2(acc[i][2], acc[i][3]);
    }
}

// (B in powers of two here: zb is what la_decay left.)
// o = (scores, masked) V + (q e^(B_i)) S for the chunk's 64 tokens by 64 columns: a warp has 16
// tokens.  CHANNEL: B is kept whole (bs), q e^(B_i) is formed in fragments, k e^(-B_j) in shared memory.
template <int MODE>
__global__ void __launch_bounds__(128) la_out_mma_kernel(
    const bf16* __restrict__ rows, int stride, const LaRows lr, const LaToken tk, const float* __restrict__ zb,
    const float* __restrict__ log_decay,
    const int* __restrict__ q_start, const int* __restrict__ state_slot, int first_req, int n_reqs,
    const float* __restrict__ kv, float* __restrict__ num, int H, int d, int dv, int act, float q_scale) {
    constexpr bool CHANNEL = MODE == LA_CHANNEL, TOKEN = MODE == LA_TOKEN;
    rv_pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char smraw[];
    const int LQ = d + 8, LB = d + 2;
    bf16* ss = (bf16*)smraw;                            // [3][d][LM_LD]: the state's columns
    bf16* vs = ss + 3 * d * LM_LD;                      // [64][LM_LD]
    bf16* qs = vs + LA_C * LM_LD;                       // [64][LQ]
    bf16* ks = qs + LA_C * LQ;                          // [1 or 3][64][LQ]
    float* bs = (float*)(ks + (CHANNEL ? 3 : 1) * LA_C * LQ);   // CHANNEL: [64][LB]
    __shared__ float pw[LA_C + 1];                      // constant decay: its powers; TOKEN: weights
    __shared__ double bt[TOKEN ? LA_C : 1];             // TOKEN: B
    __shared__ int at[2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int item = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * LA_T;
    lm_locate(q_start, state_slot, first_req, n_reqs, item, at);
    const int t0 = at[0], L = at[1];
    if (MODE == LA_CONST && tid <= LA_C) pw[tid] = expf(log_decay[h] * (float)tid);
    rv_pdl_wait();
    if (t0 < 0) return;
    if (TOKEN && tid < LA_C) {
        const size_t at_j = (size_t)(t0 + min(tid, L - 1)) * H + h;
        bt[tid] = tk.B[at_j];
        pw[tid] = tid < L ? tk.w[at_j] : 0.f;
    }
    const int kh = h / lr.share;
    const int vn = min(LA_T, dv - v0);
    const bf16* base = rows + (size_t)t0 * stride;
    // values, queries, keys: eight columns a thread and access
    {
        const int ch = tid & 7, jr = tid >> 3;
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int j = jr + 16 * u;
            *(uint4*)(vs + j * LM_LD + 8 * ch) =
                lm_in8(base + (size_t)j * stride + lr.v + h * dv + v0 + 8 * ch, j < L && 8 * ch < vn, act);
        }
        const int cpr = d >> 3;                         // chunks a row
#pragma unroll 4
        for (int n = tid; n < LA_C * cpr; n += 128) {
            const int j = n / cpr, c = (n - j * cpr) * 8;
            const bf16* row = base + (size_t)j * stride + kh * d + c;
            *(uint4*)(qs + j * LQ + c) = lm_in8(row + lr.q, j < L, act);
            *(uint4*)(ks + j * LQ + c) = lm_in8(row + lr.k, j < L, act);
        }
    }
    // the state before the chunk, in three parts
    {
        const float* S = kv + ((size_t)item * H + h) * d * dv + v0;
        const int c = (tid & 15) * 4;
#pragma unroll 4
        for (int r = tid >> 4; r < d; r += 8) {
            const float4 x = c < vn ? *(const float4*)(S + (size_t)r * dv + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            uint2 p[3];
            lm_split(x.x, x.y, p[0].x, p[1].x, p[2].x);
            lm_split(x.z, x.w, p[0].y, p[1].y, p[2].y);
#pragma unroll
            for (int s = 0; s < 3; ++s) *(uint2*)(ss + (s * d + r) * LM_LD + c) = p[s];
        }
    }
    bool strong = false;
    if (CHANNEL) {
        const int cpr = d >> 2;
        bool low = false;
#pragma unroll 4
        for (int n = tid; n < LA_C * cpr; n += 128) {
            const int j = n / cpr, c = (n - j * cpr) * 4;
            const float4 x = *(const float4*)(zb + (size_t)(t0 + min(j, L - 1)) * H * d + h * d + c);
            *(float2*)(bs + j * LB + c) = make_float2(x.x, x.y);
            *(float2*)(bs + j * LB + c + 2) = make_float2(x.z, x.w);
            low |= fminf(fminf(x.x, x.y), fminf(x.z, x.w)) < LM_STRONG;
        }
        strong = __syncthreads_or(low);
        if (!strong) {
#pragma unroll 2
            for (int n = tid; n < LA_C * (d >> 1); n += 128) {
                const int j = n / (d >> 1), c = (n - j * (d >> 1)) * 2;
                unsigned* k0 = (unsigned*)(ks + j * LQ + c);
                const float2 k2 = lm_pair(*k0), b2 = *(const float2*)(bs + j * LB + c);
                unsigned p[3];
                lm_split(k2.x * lm_exp2(-b2.x), k2.y * lm_exp2(-b2.y), p[0], p[1], p[2]);
                k0[0] = p[0];
                *(unsigned*)(ks + LA_C * LQ + j * LQ + c) = p[1];
                *(unsigned*)(ks + 2 * LA_C * LQ + j * LQ + c) = p[2];
            }
        }
    }
    __syncthreads();
    const int row_a = 16 * warp + (lane >> 2), row_b = row_a + 8;   // this thread's tokens
    if (16 * warp >= L) return;
    float p[8][4], o[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) p[i][e] = o[i][e] = 0.f;
    for (int kk = 0; kk < (d >> 4); ++kk) {
        unsigned a[CHANNEL ? 3 : 1][4];
        ldmatrix_x4(a[0], qs + (16 * warp + (lane & 15)) * LQ + kk * 16 + (lane >> 4) * 8);
        if (CHANNEL) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 q2 = lm_pair(a[0][e]);
                const float2 b2 = *(const float2*)(bs + ((e & 1) ? row_b : row_a) * LB + kk * 16 + (e >> 1) * 8 + (lane & 3) * 2);
                lm_split(q2.x * lm_exp2(b2.x), q2.y * lm_exp2(b2.y), a[0][e], a[CHANNEL ? 1 : 0][e], a[CHANNEL ? 2 : 0][e]);
            }
        }
        // scores: keys up to the warp's own tokens
        if (!CHANNEL || !strong) {
#pragma unroll
            for (int nb = 0; nb < 4; ++nb) {
                if (nb > warp) continue;
                unsigned b[CHANNEL ? 3 : 1][4];
#pragma unroll
                for (int s = 0; s < (CHANNEL ? 3 : 1); ++s)
                    ldmatrix_x4(b[s], ks + (s * LA_C + nb * 16 + (lane & 7) + (lane >> 4) * 8) * LQ + kk * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
                for (int x = (CHANNEL ? 2 : 0); x >= 0; --x)         // smallest products first
#pragma unroll
                    for (int y = 0; y <= x; ++y) {
                        mma_bf16(p[2 * nb], a[y], b[x - y][0], b[x - y][1]);
                        mma_bf16(p[2 * nb + 1], a[y], b[x - y][2], b[x - y][3]);
                    }
            }
        }
        // the state's share
#pragma unroll
        for (int nd = 0; nd < 4; ++nd) {
            if (16 * nd >= vn) continue;
            unsigned b[3][4];
#pragma unroll
            for (int s = 0; s < 3; ++s)
                ldmatrix_x4_trans(b[s], ss + (s * d + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LM_LD + nd * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int x = 2; x >= 0; --x)
#pragma unroll
                for (int y = 0; y <= (CHANNEL ? x : 0); ++y) {
                    mma_bf16(o[2 * nd], a[y], b[x - y][0], b[x - y][1]);
                    mma_bf16(o[2 * nd + 1], a[y], b[x - y][2], b[x - y][3]);
                }
        }
    }
    // a chunk with strong decays: every pair's own difference
    if (CHANNEL && strong) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (i > 2 * warp + 1) continue;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = e < 2 ? row_a : row_b, j = 8 * i + (lane & 3) * 2 + (e & 1);
                float s = 0.f;
                if (j <= r)
                    for (int c = 0; c < d; ++c)
                        s = fmaf(__bfloat162float(qs[r * LQ + c]) * __bfloat162float(ks[j * LQ + c]),
                                 lm_exp2(bs[r * LB + c] - bs[j * LB + c]), s);
                p[i][e] = s;
            }
        }
    }
    if (!CHANNEL) {
        const float fa = TOKEN ? expf((float)bt[row_a]) : pw[row_a + 1];
        const float fb = TOKEN ? expf((float)bt[row_b]) : pw[row_b + 1];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            o[i][0] *= fa; o[i][1] *= fa;
            o[i][2] *= fb; o[i][3] *= fb;
        }
    }
    // decays between the pairs (those of whole heads) and the mask, then the values
    auto pair = [&](int r, int j) {
        return TOKEN ? expf((float)(bt[r] - bt[j])) * pw[j] : pw[r - j];
    };
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
        if (kk > warp) continue;
        unsigned a[3][4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = 2 * kk + (e >> 1), r = (e & 1) ? row_b : row_a, j = 8 * i + (lane & 3) * 2;
            float x = p[i][(e & 1) * 2], y = p[i][(e & 1) * 2 + 1];
            x = j <= r ? (CHANNEL ? x : x * pair(r, j)) : 0.f;
            y = j + 1 <= r ? (CHANNEL ? y : y * pair(r, j + 1)) : 0.f;
            lm_split(x, y, a[0][e], a[1][e], a[2][e]);
        }
#pragma unroll
        for (int nd = 0; nd < 4; ++nd) {
            if (16 * nd >= vn) continue;
            unsigned b[4];
            ldmatrix_x4_trans(b, vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LM_LD + nd * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int s = 2; s >= 0; --s) {
                mma_bf16(o[2 * nd], a[s], b[0], b[1]);
                mma_bf16(o[2 * nd + 1], a[s], b[2], b[3]);
            }
        }
    }
    float* dst = num + ((size_t)t0 * H + h) * dv + v0 + (lane & 3) * 2;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        if (8 * i >= vn) continue;
        if (row_a < L)
            *(float2*)(dst + (size_t)row_a * H * dv + 8 * i) = make_float2(o[i][0] * q_scale, o[i][1] * q_scale);
        if (row_b < L)
            *(float2*)(dst + (size_t)row_b * H * dv + 8 * i) = make_float2(o[i][2] * q_scale, o[i][3] * q_scale);
    }
}

static inline size_t lm_state_smem() {
    return (size_t)4 * LA_C * LM_LD * 2;
}
static inline size_t lm_out_smem(bool channel, int d) {
    return (size_t)(3 * d + LA_C) * LM_LD * 2 + (size_t)(channel ? 4 : 2) * LA_C * (d + 8) * 2 +
           (channel ? (size_t)LA_C * (d + 2) * 4 : 0);
}
