// The gated delta rule with one decay per head over portions in chunks of 64 tokens, on the tensor
// cores (bfloat16 rows; included by gated_delta.cu, whose first comment has the recurrence).
//
// For a head and the tokens 0..63 of a chunk let k_i, q_i be the activated keys and queries (bfloat16),
// a_i, b_i what makes them unit vectors (and q scaled), B_i the sum of the log decays up to token i
// and S_0 the state before the chunk.  The correction of token i,
//
//     u_i = beta_i (v_i - e^(B_i) a_i S_0^T k_i - sum_(j < i) e^(B_i - B_j) a_i a_j <k_i, k_j> u_j),
//
// is linear in the others, so with A_ij = beta_i e^(B_i - B_j) a_i a_j <k_i, k_j> (j < i) and
// T = (I + A)^(-1) diag(beta):
//
//     U = T (V - diag(e^(B_i) a_i) K S_0);      S = e^(B_L) S_0 + K^T diag(e^(B_L - B_j) a_j) U
//     o_i = e^(B_i) b_i S_0^T q_i + sum_(j <= i) e^(B_i - B_j) b_i a_j <q_i, k_j> u_j
//
//   conv_silu   q | k | v pass the convolutions and silu -> rows [n, C] bfloat16 (conv_silu.cuh)
//   gdc_chunk   block per (chunk, head): norms, decays, A, its inverse, T
//   gdc_scan    block per (head, 16 value columns, request): over the chunks one after another, the
//               three products with S in float32 accumulators; the state before every chunk and U go
//               out, the last state is the record
//   gdc_out     block per (chunk, head, 32 value columns): o
//
// No factor is ever above 1.  Float32 operands (S, V - .., T, U, the scores) enter the bfloat16
// products as three parts (chunks.cuh): three products with a bfloat16 operand, the six of nine that
// reach a float32's last bits with another float32 one.  Sums of log decays are float64, so that their
// differences stay exact enough behind a token that forgets all.
#pragma once
#include "conv_silu.cuh"

#define GC_THREADS 256      // threads of a block of gdc_chunk
#define GC_T 32             // value columns of a block of gdc_out
#define GC_COLS 16          // value columns of a block of gdc_scan
#define GC_LT 72            // padded row of 64 bfloat16
#define GC_SC 384           // floats of a (chunk, head)'s scalars: rho | sigma | eq | sq | sk | e^(B_L), ...

struct GcArgs {
    const float *proj, *lowrank, *a_log, *dt_bias;
    const bf16* rows;                        // [n, C]
    const int *q_start, *state_slot;
    int P, LW, C, first_req, n_reqs, H, G, d, dv;
    float unit_eps;
    bf16* T;                                 // [items, H, 3, 64, 64]
    float* sc;                               // [items, H, GC_SC]
    double* B;                               // [items, H, 64]
    float *S0, *U;                           // [items, H, dv, d], [items, H, dv, 64]
};

__device__ __forceinline__ float gc_norm2(const bf16* p, int d, int sub) {       // eight lanes a row
    float s = 0.f;
    for (int c = sub * 8; c < d; c += 64) {
        const uint4 v = *(const uint4*)(p + c);
        const unsigned u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float2 f = lm_pair(u[e]);
            s += f.x * f.x + f.y * f.y;
        }
    }
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    s += __shfl_xor_sync(0xffffffffu, s, 2);
    s += __shfl_xor_sync(0xffffffffu, s, 4);
    return s;
}

__global__ void __launch_bounds__(GC_THREADS) gdc_chunk_kernel(const GcArgs g) {
    rv_pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char smraw[];
    const int d = g.d, LK = d + 8;
    float* As = (float*)smraw;                            // [64][65]: A, then rows of its inverse below it
    float* Xs = As + 64 * 65;                             // [64][65]: the inverse
    bf16* ks = (bf16*)(Xs + 64 * 65);                     // [64][LK]
    __shared__ float sk[64], sq[64], beta[64];
    __shared__ double bt[64];
    __shared__ int at[2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int item = blockIdx.x, h = blockIdx.y, kh = h / (g.H / g.G);
    lm_locate(g.q_start, g.state_slot, g.first_req, g.n_reqs, item, at);
    const int t0 = at[0], L = at[1];
    rv_pdl_wait();
    if (t0 < 0) return;
    const bf16* base = g.rows + (size_t)t0 * g.C;
    for (int n = tid; n < 64 * (d >> 3); n += GC_THREADS) {
        const int j = n / (d >> 3), c = (n - j * (d >> 3)) * 8;
        *(uint4*)(ks + j * LK + c) = j < L ? *(const uint4*)(base + (size_t)j * g.C + (g.G + kh) * d + c)
                                           : make_uint4(0, 0, 0, 0);
    }
    // norms: eight lanes a token
    #pragma unroll
    for (int u = 0; u < 64 * 8 / GC_THREADS; ++u) {
        const int j = (tid >> 3) + u * (GC_THREADS / 8);
        const bf16* row = base + (size_t)min(j, L - 1) * g.C + kh * d;
        const float nq = gc_norm2(row, d, tid & 7), nk = gc_norm2(row + g.G * d, d, tid & 7);
        if ((tid & 7) == 0) {
            sq[j] = j < L ? 1.f / sqrtf((float)d) / sqrtf(nq + g.unit_eps) : 0.f;
            sk[j] = j < L ? 1.f / sqrtf(nk + g.unit_eps) : 0.f;
        }
    }
    if (warp == 7) {                                      // two tokens a lane
        const float rate = expf(g.a_log[h]), bias = g.dt_bias[h];
        double l[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int j = 2 * lane + e;
            const size_t t = t0 + min(j, L - 1);
            l[e] = j < L ? -(double)(rate * la_softplus(g.lowrank[t * g.LW + h] + bias)) : 0.;
            beta[j] = j < L ? 1.f / (1.f + expf(-g.proj[t * g.P + g.C + h])) : 0.f;
        }
        double incl = l[0] + l[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, incl, o);
            if (lane >= o) incl += up;
        }
        bt[2 * lane + 1] = incl;
        bt[2 * lane] = incl - l[1];
    }
    __syncthreads();
    // A: two warps have 16 rows, half of the columns each
    {
        const int rg = warp >> 1, half = warp & 1;
        float p[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) p[i][0] = p[i][1] = p[i][2] = p[i][3] = 0.f;
        for (int kk = 0; kk < (d >> 4); ++kk) {
            unsigned a[4];
            ldmatrix_x4(a, ks + (16 * rg + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int nb = 2 * half + u;
                if (nb > rg) continue;
                unsigned b[4];
                ldmatrix_x4(b, ks + (nb * 16 + (lane & 7) + (lane >> 4) * 8) * LK + kk * 16 + ((lane >> 3) & 1) * 8);
                mma_bf16(p[2 * u], a, b[0], b[1]);
                mma_bf16(p[2 * u + 1], a, b[2], b[3]);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = 16 * rg + (lane >> 2) + (e >> 1) * 8, j = 32 * half + 8 * i + (lane & 3) * 2 + (e & 1);
                As[r * 65 + j] = j < r ? beta[r] * sk[r] * sk[j] * expf((float)(bt[r] - bt[j])) * p[i][e] : 0.f;
            }
    }
    __syncthreads();
    // The inverse X of I + A.  First its four diagonal blocks of 16, a warp each, two lanes a column:
    // x_i = (i = j) - sum_(j <= m < i) A_im x_m.
    if (warp < 4) {
        const int o = 16 * warp, j = lane >> 1, half = lane & 1;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float s = 0.f;
#pragma unroll
            for (int m = 0; m < i; ++m)
                if ((m & 1) == half) s = fmaf(As[(o + i) * 65 + o + m], x[m], s);
            s += __shfl_xor_sync(0xffffffffu, s, 1);
            x[i] = (i == j ? 1.f : 0.f) - s;
        }
#pragma unroll
        for (int i = 0; i < 16; ++i)
            if ((i & 1) == half) Xs[(o + i) * 65 + o + j] = x[i];
    } else {                                              // beside the blocks: zeros
        for (int n = tid - 128; n < 64 * 64; n += GC_THREADS - 128)
            if (((n >> 4) & 3) != (n >> 10)) Xs[(n >> 6) * 65 + (n & 63)] = 0.f;
    }
    __syncthreads();
    // Then pairs of blocks of 16, and the pair of 32: X_21 = -X_22 (A_21 X_11); the inner product goes
    // where A_21 was, once it has been read.
#pragma unroll
    for (int w = 16; w <= 32; w <<= 1) {
        const int per = w * w, pairs = 32 / w;            // outputs of a pair; pairs
        constexpr int MAXO = 32 * 32 / GC_THREADS;
        float tmp[MAXO];
        for (int pass = 0; pass < 2; ++pass) {
#pragma unroll
            for (int u = 0; u < MAXO; ++u) {
                const int n = tid + GC_THREADS * u;
                if (n >= pairs * per) continue;
                const int q = n / per, e = n - q * per, i = e / w, j = e - i * w, o = 2 * q * w;
                float s = 0.f;
                if (pass == 0)
#pragma unroll 8
                    for (int m = j; m < w; ++m)
                        s = fmaf(As[(o + w + i) * 65 + o + m], Xs[(o + m) * 65 + o + j], s);
                else
#pragma unroll 8
                    for (int m = 0; m <= i; ++m)
                        s = fmaf(Xs[(o + w + i) * 65 + o + w + m], As[(o + w + m) * 65 + o + j], s);
                tmp[u] = s;
            }
            __syncthreads();
#pragma unroll
            for (int u = 0; u < MAXO; ++u) {
                const int n = tid + GC_THREADS * u;
                if (n >= pairs * per) continue;
                const int q = n / per, e = n - q * per, i = e / w, j = e - i * w, o = 2 * q * w;
                if (pass == 0) As[(o + w + i) * 65 + o + j] = tmp[u];
                else Xs[(o + w + i) * 65 + o + j] = -tmp[u];
            }
            __syncthreads();
        }
    }
    const size_t ih = (size_t)item * g.H + h;
    bf16* T = g.T + ih * 3 * 64 * 64;
    for (int n = tid; n < 64 * 32; n += GC_THREADS) {
        const int i = n >> 5, j = (n & 31) * 2;
        unsigned p[3];
        lm_split(Xs[i * 65 + j] * beta[j], Xs[i * 65 + j + 1] * beta[j + 1], p[0], p[1], p[2]);
#pragma unroll
        for (int s = 0; s < 3; ++s) *(unsigned*)(T + (s * 64 + i) * 64 + j) = p[s];
    }
    if (tid < 64) {
        float* sc = g.sc + ih * GC_SC;
        const float e = expf((float)bt[tid]);
        sc[tid] = e * sk[tid];
        sc[64 + tid] = expf((float)(bt[L - 1] - bt[tid])) * sk[tid];
        sc[128 + tid] = e * sq[tid];
        sc[192 + tid] = sq[tid];
        sc[256 + tid] = sk[tid];
        if (tid == 0) sc[320] = expf((float)bt[L - 1]);
        g.B[ih * 64 + tid] = bt[tid];
    }
}

// S^T lies in accumulators, 16 columns by d = 16 UNITS rows: a warp has 16 rows, or 32.  The products of
// the operands' three parts have accumulators of their own, so that none is a long chain.
template <int UNITS>
__global__ void __launch_bounds__(128) gdc_scan_kernel(const GcArgs g, float* __restrict__ state, long long rec,
                                                       int taps) {
    rv_pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char smraw[];
    constexpr int d = 16 * UNITS, LK = d + 8, NU = (UNITS + 3) / 4;
    const int dv = g.dv;
    bf16* ss = (bf16*)smraw;                              // [3][16][LK]: the state
    bf16* rs = ss + 3 * GC_COLS * LK;                     // [3][16][GC_LT]: V - rho Y
    bf16* us = rs + 3 * GC_COLS * GC_LT;                  // [3][16][GC_LT]: sigma U
    bf16* kbuf = us + 3 * GC_COLS * GC_LT;                // [2][64][LK]
    bf16* tbuf = kbuf + 2 * 64 * LK;                      // [2][3][64][GC_LT]
    bf16* vbuf = tbuf + 2 * 3 * 64 * GC_LT;               // [2][64][24]
    float* cbuf = (float*)(vbuf + 2 * 64 * 24);           // [2][132]: rho | sigma | e^(B_L), ...
    __shared__ int first_item;
    const int col_blocks = dv / GC_COLS;
    const int h = blockIdx.x / col_blocks, c0 = (blockIdx.x - h * col_blocks) * GC_COLS, kh = h / (g.H / g.G);
    const int r = g.first_req + blockIdx.y;
    const int slot = g.state_slot[r];
    const int t0 = g.q_start[r], qlen = g.q_start[r + 1] - t0;
    const int n = slot < 0 ? 0 : (qlen + LA_C - 1) / LA_C;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    if (tid < 32) {
        int before = 0;
        for (int b = g.first_req + tid; b < r; b += 32) before += la_chunks(g.q_start, g.state_slot, b);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
        if (tid == 0) first_item = before;
    }
    __syncthreads();
    rv_pdl_wait();
    if (n == 0) return;
    constexpr int cpr = d >> 3;
    auto load = [&](int c) {                              // chunk c's operands into buffer c & 1
        const int L = min(LA_C, qlen - c * LA_C);
        const bf16* base = g.rows + (size_t)(t0 + c * LA_C) * g.C;
        bf16* kd = kbuf + (c & 1) * 64 * LK;
#pragma unroll
        for (int m = tid; m < 64 * cpr; m += 128) {
            const int j = m / cpr, ch = (m - j * cpr) * 8;
            cp_async_16(kd + j * LK + ch, base + (size_t)min(j, L - 1) * g.C + (g.G + kh) * d + ch, j < L);
        }
        const size_t ih = (size_t)(first_item + c) * g.H + h;
        const bf16* T = g.T + ih * 3 * 64 * 64;
        bf16* td = tbuf + (c & 1) * 3 * 64 * GC_LT;
#pragma unroll 4
        for (int m = tid; m < 3 * 64 * 8; m += 128) cp_async_16(td + (m >> 3) * GC_LT + (m & 7) * 8, T + m * 8, true);
        bf16* vd = vbuf + (c & 1) * 64 * 24;
        const int j = tid >> 1, ch = (tid & 1) * 8;
        cp_async_16(vd + j * 24 + ch, base + (size_t)min(j, L - 1) * g.C + 2 * g.G * d + h * dv + c0 + ch, j < L);
        float* cd = cbuf + (c & 1) * 132;
        const float* sc = g.sc + ih * GC_SC;
        if (tid < 32) cp_async_16(cd + tid * 4, sc + tid * 4, true);
        if (tid == 32) cp_async_16(cd + 128, sc + 320, true);
        cp_async_commit();
    };
    load(0);
    // the record's rows, [column][d]: this thread has columns ca and ca + 8 of its row pairs
    const int ca = lane >> 2;
    float* Sg = state + (size_t)slot * rec + (size_t)(taps - 1) * g.C + ((size_t)h * dv + c0) * d;
    const bool wide = (((uintptr_t)Sg) & 7) == 0;
    float S[2 * NU][4];
#pragma unroll
    for (int i = 0; i < 2 * NU; ++i) {
        const int un = warp + 4 * (i >> 1), row = un * 16 + (i & 1) * 8 + (lane & 3) * 2;
        S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
        if (un < UNITS) {
            const float *p = Sg + (size_t)ca * d + row, *q = p + (size_t)8 * d;
            if (wide) {
                const float2 a = *(const float2*)p, b = *(const float2*)q;
                S[i][0] = a.x; S[i][1] = a.y; S[i][2] = b.x; S[i][3] = b.y;
            } else {
                S[i][0] = p[0]; S[i][1] = p[1]; S[i][2] = q[0]; S[i][3] = q[1];
            }
        }
    }
    auto split_pair = [&](bf16* dst, int ld, int row, int col, float x, float y) {
        unsigned p[3];
        lm_split(x, y, p[0], p[1], p[2]);
#pragma unroll
        for (int s = 0; s < 3; ++s) *(unsigned*)(dst + (s * GC_COLS + row) * ld + col) = p[s];
    };
    auto put_state = [&]() {
#pragma unroll
        for (int i = 0; i < 2 * NU; ++i) {
            const int un = warp + 4 * (i >> 1), row = un * 16 + (i & 1) * 8 + (lane & 3) * 2;
            if (un >= UNITS) continue;
            split_pair(ss, LK, ca, row, S[i][0], S[i][1]);
            split_pair(ss, LK, ca + 8, row, S[i][2], S[i][3]);
        }
    };
    put_state();
    for (int c = 0; c < n; ++c) {
        if (c + 1 < n) {
            load(c + 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();                                  // chunk c is here, and so is the state
        const int L = min(LA_C, qlen - c * LA_C);
        const bf16 *ks = kbuf + (c & 1) * 64 * LK, *ts = tbuf + (c & 1) * 3 * 64 * GC_LT, *vs = vbuf + (c & 1) * 64 * 24;
        const float* cs = cbuf + (c & 1) * 132;
        const size_t ih = (size_t)(first_item + c) * g.H + h;
        // the state before the chunk
        float* S0 = g.S0 + (ih * dv + c0) * d;
#pragma unroll
        for (int i = 0; i < 2 * NU; ++i) {
            const int un = warp + 4 * (i >> 1), row = un * 16 + (i & 1) * 8 + (lane & 3) * 2;
            if (un >= UNITS) continue;
            *(float2*)(S0 + (size_t)ca * d + row) = make_float2(S[i][0], S[i][1]);
            *(float2*)(S0 + (size_t)(ca + 8) * d + row) = make_float2(S[i][2], S[i][3]);
        }
        // Y^T = S^T K^T for this warp's 16 tokens
        float y3[3][2][4], y[2][4];
        auto clear = [&]() {
#pragma unroll
            for (int s = 0; s < 3; ++s)
#pragma unroll
                for (int i = 0; i < 2; ++i) y3[s][i][0] = y3[s][i][1] = y3[s][i][2] = y3[s][i][3] = 0.f;
        };
        auto sum = [&]() {                                // smallest first
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) y[i][e] = (y3[2][i][e] + y3[1][i][e]) + y3[0][i][e];
        };
        clear();
#pragma unroll
        for (int kk = 0; kk < UNITS; ++kk) {
            unsigned a[3][4], b[4];
#pragma unroll
            for (int s = 0; s < 3; ++s)
                ldmatrix_x4(a[s], ss + (s * GC_COLS + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8);
            ldmatrix_x4(b, ks + (16 * warp + (lane & 7) + (lane >> 4) * 8) * LK + kk * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int s = 2; s >= 0; --s) {
                mma_bf16(y3[s][0], a[s], b[0], b[1]);
                mma_bf16(y3[s][1], a[s], b[2], b[3]);
            }
        }
        sum();
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int j = 16 * warp + 8 * i + (lane & 3) * 2;
            const float r0 = cs[j], r1 = cs[j + 1];
#pragma unroll
            for (int e = 0; e < 2; ++e)
                split_pair(rs, GC_LT, ca + 8 * e, j,
                           fmaf(-r0, y[i][2 * e], __bfloat162float(vs[j * 24 + ca + 8 * e])),
                           fmaf(-r1, y[i][2 * e + 1], __bfloat162float(vs[(j + 1) * 24 + ca + 8 * e])));
        }
        __syncthreads();
        // U^T = R^T T^T
        clear();
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            if (kk > warp) continue;
            unsigned a[3][4], b[3][4];
#pragma unroll
            for (int s = 0; s < 3; ++s) {
                ldmatrix_x4(a[s], rs + (s * GC_COLS + (lane & 15)) * GC_LT + kk * 16 + (lane >> 4) * 8);
                ldmatrix_x4(b[s], ts + (s * 64 + 16 * warp + (lane & 7) + (lane >> 4) * 8) * GC_LT + kk * 16 +
                                      ((lane >> 3) & 1) * 8);
            }
#pragma unroll
            for (int z = 0; z < 3; ++z)
#pragma unroll
                for (int x = 2; x >= z; --x) {
                    mma_bf16(y3[x][0], a[z], b[x - z][0], b[x - z][1]);
                    mma_bf16(y3[x][1], a[z], b[x - z][2], b[x - z][3]);
                }
        }
        sum();
        float* U = g.U + (ih * dv + c0) * 64;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int j = 16 * warp + 8 * i + (lane & 3) * 2;
            const float s0 = cs[64 + j], s1 = cs[64 + j + 1];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                *(float2*)(U + (size_t)(ca + 8 * e) * 64 + j) = make_float2(y[i][2 * e], y[i][2 * e + 1]);
                split_pair(us, GC_LT, ca + 8 * e, j, y[i][2 * e] * s0, y[i][2 * e + 1] * s1);
            }
        }
        __syncthreads();
        // S^T <- e^(B_L) S^T + (sigma U)^T K
        const float keep = cs[128];
#pragma unroll
        for (int i = 0; i < 2 * NU; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) S[i][e] *= keep;
        float low[2 * NU][4];
#pragma unroll
        for (int i = 0; i < 2 * NU; ++i) low[i][0] = low[i][1] = low[i][2] = low[i][3] = 0.f;
        const int nk = (L + 15) >> 4;
        for (int kk = 0; kk < nk; ++kk) {
            unsigned a[3][4];
#pragma unroll
            for (int s = 0; s < 3; ++s)
                ldmatrix_x4(a[s], us + (s * GC_COLS + (lane & 15)) * GC_LT + kk * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < NU; ++i) {
                const int un = warp + 4 * i;
                if (un >= UNITS) continue;
                unsigned b[4];
                ldmatrix_x4_trans(b, ks + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LK + un * 16 + (lane >> 4) * 8);
#pragma unroll
                for (int s = 2; s > 0; --s) {
                    mma_bf16(low[2 * i], a[s], b[0], b[1]);
                    mma_bf16(low[2 * i + 1], a[s], b[2], b[3]);
                }
                mma_bf16(S[2 * i], a[0], b[0], b[1]);
                mma_bf16(S[2 * i + 1], a[0], b[2], b[3]);
            }
        }
#pragma unroll
        for (int i = 0; i < 2 * NU; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) S[i][e] += low[i][e];
        put_state();                                      // (every warp has read the old one)
        // the buffer that chunk c + 2 goes to is this chunk's: everyone has to be done with it
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2 * NU; ++i) {
        const int un = warp + 4 * (i >> 1), row = un * 16 + (i & 1) * 8 + (lane & 3) * 2;
        if (un >= UNITS) continue;
        float *p = Sg + (size_t)ca * d + row, *q = p + (size_t)8 * d;
        if (wide) {
            *(float2*)p = make_float2(S[i][0], S[i][1]);
            *(float2*)q = make_float2(S[i][2], S[i][3]);
        } else {
            p[0] = S[i][0]; p[1] = S[i][1]; q[0] = S[i][2]; q[1] = S[i][3];
        }
    }
}

__global__ void __launch_bounds__(128) gdc_out_kernel(const GcArgs g, float* __restrict__ o_out) {
    rv_pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char smraw[];
    const int d = g.d, dv = g.dv, LK = d + 8;
    bf16* ss = (bf16*)smraw;                              // [3][GC_T columns][LK]: the state before the chunk
    bf16* us = ss + 3 * GC_T * LK;                        // [3][GC_T columns][GC_LT]: U
    bf16* qs = us + 3 * GC_T * GC_LT;                     // [64][LK]
    bf16* ks = qs + 64 * LK;                              // [64][LK]
    __shared__ float eq[64], sq[64], sk[64];
    __shared__ double bt[64];
    __shared__ int at[2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int item = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * GC_T, kh = h / (g.H / g.G);
    lm_locate(g.q_start, g.state_slot, g.first_req, g.n_reqs, item, at);
    const int t0 = at[0], L = at[1];
    rv_pdl_wait();
    if (t0 < 0) return;
    const int vn = min(GC_T, dv - v0);                    // a multiple of 16
    const size_t ih = (size_t)item * g.H + h;
    if (tid < 64) {
        const float* sc = g.sc + ih * GC_SC;
        eq[tid] = sc[128 + tid];
        sq[tid] = sc[192 + tid];
        sk[tid] = sc[256 + tid];
        bt[tid] = g.B[ih * 64 + tid];
    }
    const bf16* base = g.rows + (size_t)t0 * g.C + kh * d;
    const int cpr = d >> 3;
#pragma unroll 4
    for (int n = tid; n < 64 * cpr; n += 128) {
        const int j = n / cpr, c = (n - j * cpr) * 8;
        const bf16* row = base + (size_t)min(j, L - 1) * g.C + c;
        *(uint4*)(qs + j * LK + c) = j < L ? *(const uint4*)row : make_uint4(0, 0, 0, 0);
        *(uint4*)(ks + j * LK + c) = j < L ? *(const uint4*)(row + g.G * d) : make_uint4(0, 0, 0, 0);
    }
    const float *S0 = g.S0 + (ih * dv + v0) * d, *U = g.U + (ih * dv + v0) * 64;
    auto split4 = [&](bf16* dst, int rows, int ld, int row, int col, const float4& x) {
        uint2 p[3];
        lm_split(x.x, x.y, p[0].x, p[1].x, p[2].x);
        lm_split(x.z, x.w, p[0].y, p[1].y, p[2].y);
#pragma unroll
        for (int s = 0; s < 3; ++s) *(uint2*)(dst + (s * rows + row) * ld + col) = p[s];
    };
#pragma unroll 4
    for (int n = tid; n < vn * (d >> 2); n += 128) {
        const int row = n / (d >> 2), c = (n - row * (d >> 2)) * 4;
        split4(ss, GC_T, LK, row, c, *(const float4*)(S0 + (size_t)row * d + c));
    }
#pragma unroll 4
    for (int n = tid; n < vn * 16; n += 128)
        split4(us, GC_T, GC_LT, n >> 4, (n & 15) * 4, *(const float4*)(U + (size_t)(n >> 4) * 64 + (n & 15) * 4));
    __syncthreads();
    if (16 * warp >= L) return;
    const int row_a = 16 * warp + (lane >> 2), row_b = row_a + 8;
    float p[8][4], o[GC_T / 8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            p[i][e] = 0.f;
            if (i < GC_T / 8) o[i][e] = 0.f;
        }
    for (int kk = 0; kk < (d >> 4); ++kk) {
        unsigned a[4];
        ldmatrix_x4(a, qs + (16 * warp + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) {
            if (nb > warp) continue;
            unsigned b[4];
            ldmatrix_x4(b, ks + (nb * 16 + (lane & 7) + (lane >> 4) * 8) * LK + kk * 16 + ((lane >> 3) & 1) * 8);
            mma_bf16(p[2 * nb], a, b[0], b[1]);
            mma_bf16(p[2 * nb + 1], a, b[2], b[3]);
        }
#pragma unroll
        for (int nd = 0; nd < GC_T / 16; ++nd) {
            if (16 * nd >= vn) continue;
#pragma unroll
            for (int s = 2; s >= 0; --s) {
                unsigned b[4];
                ldmatrix_x4(b, ss + (s * GC_T + nd * 16 + (lane & 7) + (lane >> 4) * 8) * LK + kk * 16 + ((lane >> 3) & 1) * 8);
                mma_bf16(o[2 * nd], a, b[0], b[1]);
                mma_bf16(o[2 * nd + 1], a, b[2], b[3]);
            }
        }
    }
    const float fa = eq[row_a], fb = eq[row_b];
#pragma unroll
    for (int i = 0; i < GC_T / 8; ++i) {
        o[i][0] *= fa; o[i][1] *= fa;
        o[i][2] *= fb; o[i][3] *= fb;
    }
    auto pair = [&](int r, int j) { return j <= r ? expf((float)(bt[r] - bt[j])) * sq[r] * sk[j] : 0.f; };
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
        if (kk > warp) continue;
        unsigned a[3][4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = 2 * kk + (e >> 1), r = (e & 1) ? row_b : row_a, j = 8 * i + (lane & 3) * 2;
            lm_split(p[i][(e & 1) * 2] * pair(r, j), p[i][(e & 1) * 2 + 1] * pair(r, j + 1), a[0][e], a[1][e], a[2][e]);
        }
#pragma unroll
        for (int nd = 0; nd < GC_T / 16; ++nd) {
            if (16 * nd >= vn) continue;
            unsigned b[3][4];
#pragma unroll
            for (int s = 0; s < 3; ++s)
                ldmatrix_x4(b[s], us + (s * GC_T + nd * 16 + (lane & 7) + (lane >> 4) * 8) * GC_LT + kk * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int x = 2; x >= 0; --x)
#pragma unroll
                for (int z = 0; z <= x; ++z) {
                    mma_bf16(o[2 * nd], a[z], b[x - z][0], b[x - z][1]);
                    mma_bf16(o[2 * nd + 1], a[z], b[x - z][2], b[x - z][3]);
                }
        }
    }
    float* dst = o_out + ((size_t)t0 * g.H + h) * dv + v0 + (lane & 3) * 2;
#pragma unroll
    for (int i = 0; i < GC_T / 8; ++i) {
        if (8 * i >= vn) continue;
        if (row_a < L) *(float2*)(dst + (size_t)row_a * g.H * dv + 8 * i) = make_float2(o[i][0], o[i][1]);
        if (row_b < L) *(float2*)(dst + (size_t)row_b * g.H * dv + 8 * i) = make_float2(o[i][2], o[i][3]);
    }
}

// ---------------------------------------------------------------------------------
struct GcScratch {
    long long rows, T, sc, B, S0, U, total;               // in floats
};
static GcScratch gc_layout(int n_tokens, long long items, int H, int d, int dv, int C) {
    auto align = [](long long f) { return (f + 3) & ~3LL; };
    GcScratch s;
    s.rows = 0;
    s.T = align(((long long)n_tokens * C + 1) / 2);
    s.sc = s.T + items * H * (3 * 64 * 64 / 2);
    s.B = s.sc + items * H * GC_SC;
    s.S0 = s.B + items * H * 128;
    s.U = s.S0 + align(items * H * dv * d);
    s.total = s.U + items * H * dv * 64;
    return s;
}

// Which sizes the chunk form takes.
static bool gc_sizes_ok(int H, int G, int d, int dv) {
    return d % 16 == 0 && d <= 128 && dv % 16 == 0 && (2 * G * d + H * dv) % 8 == 0;
}

#define GC_SMEM(kernel, bytes)                                                                        \
    {                                                                                                 \
        static size_t have = 40 * 1024;       /* the default 48 KB hold the static arrays too */        \
        if ((bytes) > have) {                                                                         \
            if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,             \
                                     (int)(bytes)) != cudaSuccess)                                    \
                RV_FAIL("gated_delta: %zu bytes of shared memory are not to be had", (size_t)(bytes)); \
            have = (bytes);                                                                           \
        }                                                                                             \
    }

// Portions of requests [first_req, n_reqs), tokens [first_token, n_tokens): o [n, H dv].
static int gc_run(GcArgs g, const float* filt, float* state, long long rec, int taps, const int* token_req,
                  int first_token, int n_tokens, float* scratch, float* o, cudaStream_t s) {
    const long long items = la_items(n_tokens - first_token, g.n_reqs - g.first_req);
    if (items > 65535LL * 32) RV_FAIL("gated_delta: too many tokens");
    const GcScratch lay = gc_layout(n_tokens, items, g.H, g.d, g.dv, g.C);
    bf16* rows = (bf16*)(scratch + lay.rows);
    g.rows = rows;
    g.T = (bf16*)(scratch + lay.T);
    g.sc = scratch + lay.sc;
    g.B = (double*)(scratch + lay.B);
    g.S0 = scratch + lay.S0;
    g.U = scratch + lay.U;
    const ConvSilu conv = {g.proj, filt, nullptr, state, rec, token_req, g.q_start, g.state_slot, g.P, 0,
                           first_token, n_tokens, g.C, taps};
    conv_silu<bf16>(conv, rows, s);
    RV_CHECK_LAUNCH("gated_delta conv");
    const int LK = g.d + 8;
    const size_t sm1 = (size_t)2 * 64 * 65 * 4 + (size_t)64 * LK * 2;
    GC_SMEM(gdc_chunk_kernel, sm1)
    rv_launch(gdc_chunk_kernel, dim3((unsigned)items, g.H), dim3(GC_THREADS), sm1, s, g);
    RV_CHECK_LAUNCH("gated_delta chunk");
    const size_t sm2 = ((size_t)(3 * GC_COLS + 2 * 64) * LK + (size_t)(6 * GC_COLS + 6 * 64) * GC_LT + 2 * 64 * 24) * 2 +
                       2 * 132 * 4;
    const dim3 grid2(g.H * (g.dv / GC_COLS), g.n_reqs - g.first_req);
#define GC_SCAN(U)                                                                            \
    case U:                                                                                   \
        GC_SMEM(gdc_scan_kernel<U>, sm2)                                                      \
        rv_launch(gdc_scan_kernel<U>, grid2, dim3(128), sm2, s, g, state, rec, taps);         \
        break;
    switch (g.d >> 4) {
        GC_SCAN(1) GC_SCAN(2) GC_SCAN(3) GC_SCAN(4) GC_SCAN(5) GC_SCAN(6) GC_SCAN(7) GC_SCAN(8)
    }
#undef GC_SCAN
    RV_CHECK_LAUNCH("gated_delta scan");
    const size_t sm3 = ((size_t)(3 * GC_T + 2 * 64) * LK + (size_t)3 * GC_T * GC_LT) * 2;
    GC_SMEM(gdc_out_kernel, sm3)
    rv_launch(gdc_out_kernel, dim3((unsigned)items, g.H, (g.dv + GC_T - 1) / GC_T), dim3(128), sm3, s, g, o);
    RV_CHECK_LAUNCH("gated_delta out");
    return 0;
}
