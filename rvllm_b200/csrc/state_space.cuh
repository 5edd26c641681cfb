// A selective state space with one decay per token and head (the Mamba-2 form), on the kernels of
// linear_attention.cu, which includes this file: per head a float32 matrix S [N, dv],
//
//     S <- a_t S + dt_t B_t x_t^T;   y_t = S^T C_t + D x_t
//     dt = softplus(t + dt_bias),  a = exp(-exp(A_log) dt)
//
// that is a linear attention with keys B, queries C, values x, the decay a and the keys' weights dt.
// B and C are shared by the heads of a group.
//
//   proj [n, P] float32: z [H dv] | x [H dv] | B [G N] | C [G N] | t [H] | anything else
//   conv_silu  x, B and C pass the convolution and silu -> rows [n, C] of the compute type
//              (conv_silu.cuh; records [taps-1][C])
//   ss_decay   dt of every token of a portion, and the sums of the log decays of its chunk's tokens
//              up to it (float64), once per chunk and head
//   state, scan, out / token: linear_attention.cu with LA_TOKEN
//   ss_finish  y + D x, times silu(z), RMS-normed in equal parts of the row, times the weight; and
//              the convolution's inputs move on (the last taps-1 of old record | this step's rows)
// Plain reference: tests/plain_ops.py state_space.
#pragma once
#include "conv_silu.cuh"

// A warp has eight tokens of 32 heads.
__global__ void __launch_bounds__(256) ss_decay_kernel(
    const float* __restrict__ t_raw, int P, const float* __restrict__ dt_bias,
    const float* __restrict__ a_log, const int* __restrict__ q_start, const int* __restrict__ state_slot,
    int first_req, int n_reqs, double* __restrict__ B, float* __restrict__ w, float* __restrict__ dec, int H) {
    rv_pdl_launch_dependents();
    __shared__ double tot[8][32];
    __shared__ int at[2];
    const int lane = threadIdx.x & 31, g = threadIdx.x >> 5, h = blockIdx.y * 32 + lane;
    lm_locate(q_start, state_slot, first_req, n_reqs, blockIdx.x, at);
    const int t0 = at[0], L = at[1];
    const float bias = h < H ? dt_bias[h] : 0.f, rate = h < H ? expf(a_log[h]) : 0.f;
    rv_pdl_wait();
    if (t0 < 0) return;
    float v[8];
    double sum[8], s = 0.;
#pragma unroll
    for (int j = 0; j < 8; ++j)
        v[j] = 8 * g + j < L && h < H ? t_raw[(size_t)(t0 + 8 * g + j) * P + h] : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        v[j] = la_softplus(v[j] + bias);
        if (8 * g + j < L) s -= (double)(rate * v[j]);
        sum[j] = s;
    }
    tot[g][lane] = s;
    __syncthreads();
    double before = 0.;
    for (int i = 0; i < g; ++i) before += tot[i][lane];
    if (h >= H) return;
#pragma unroll
    for (int j = 0; j < 8; ++j)
        if (8 * g + j < L) {
            const size_t to = (size_t)(t0 + 8 * g + j) * H + h;
            B[to] = before + sum[j];
            w[to] = v[j];
        }
    if (g == 7) dec[(size_t)blockIdx.x * H + h] = expf((float)(before + s));
}

// Blocks (token, part of the row); then a block per request.
template <typename T, int V>
__global__ void ss_finish_kernel(const float* __restrict__ num, const T* __restrict__ rows,
                                 const float* __restrict__ proj, int P, const float* __restrict__ D,
                                 const float* __restrict__ norm_w, float eps, float* __restrict__ conv_state,
                                 const int* __restrict__ token_req, const int* __restrict__ q_start,
                                 const int* __restrict__ state_slot, T* __restrict__ out, int n_tokens,
                                 int inner, int C, int dv, int part, int taps) {
    rv_pdl_launch_dependents();
    extern __shared__ __align__(16) float vals[];                // [part]
    __shared__ float scratch[33];
    if ((int)blockIdx.x >= n_tokens) {
        // oldest first, so that what a place receives is read before that place is overwritten
        const int r = blockIdx.x - n_tokens;
        const int slot = state_slot[r];
        const int t0 = q_start[r], qlen = q_start[r + 1] - t0;
        if (slot < 0 || qlen <= 0) return;
        rv_pdl_wait();
        float* record = conv_state + (size_t)slot * (taps - 1) * C;
        for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x)
            for (int i = 0; i < taps - 1; ++i) {
                const int idx = qlen - (taps - 1) + i;           // among this step's rows; negative: older
                record[(size_t)i * C + c] = idx >= 0 ? proj[(size_t)(t0 + idx) * P + inner + c]
                                                     : record[(size_t)(taps - 1 + idx) * C + c];
            }
        return;
    }
    const int t = blockIdx.x, c0 = blockIdx.y * part;
    const bool pad = state_slot[token_req[t]] < 0;
    rv_pdl_wait();
    T* o = out + (size_t)t * inner + c0;
    if (pad) {
        for (int c = threadIdx.x; c < part; c += blockDim.x) rv_store(o + c, 0.f);
        return;
    }
    const float* nm = num + (size_t)t * inner + c0;
    const float* z = proj + (size_t)t * P + c0;
    const T* xr = rows + (size_t)t * C + c0;
    float ss = 0.f;
    for (int c = threadIdx.x * V; c < part; c += blockDim.x * V) {
        float y[V], zz[V], x[V];
        la_load<float, V>(nm + c, y);
        la_load<float, V>(z + c, zz);
        la_load<T, V>(xr + c, x);
        const float skip = D[(c0 + c) / dv];
#pragma unroll
        for (int e = 0; e < V; ++e) {
            y[e] = fmaf(skip, x[e], y[e]) * (zz[e] / (1.f + expf(-zz[e])));
            ss += y[e] * y[e];
            vals[c + e] = y[e];
        }
    }
    const float inv = 1.f / sqrtf(rv_block_sum(ss, scratch) / (float)part + eps);
    for (int c = threadIdx.x * V; c < part; c += blockDim.x * V) {
        float y[V], w[V];
        la_load<float, V>(norm_w + c0 + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = vals[c + e] * inv * w[e];
        la_store<T, V>(o + c, y);
    }
}

// ---------------------------------------------------------------------------------
// Where the parts of the scratch begin, in floats.
struct SsScratch {
    long long num, kv, dec, B, w, rows, total;
};
static SsScratch ss_layout(int n_tokens, int n_decode, int n_reqs, int H, int dv, int N, int G, int el) {
    auto align = [](long long f) { return (f + 3) & ~3LL; };
    const int portions = n_reqs > n_decode && n_tokens > n_decode;
    const long long items = portions ? la_items(n_tokens - n_decode, n_reqs - n_decode) : 0;
    const long long nh = portions ? (long long)n_tokens * H : 0;
    SsScratch s;
    s.num = 0;
    s.kv = align((long long)n_tokens * H * dv);
    s.dec = s.kv + align(items * H * N * dv);
    s.B = s.dec + align(items * H);
    s.w = s.B + align(2 * nh);
    s.rows = s.w + align(nh);
    s.total = s.rows + align(((long long)n_tokens * (H * dv + 2LL * G * N) * el + 3) / 4);
    return s;
}
extern "C" long long rv_state_space_scratch(int n_tokens, int n_decode, int n_reqs, int H, int dv, int N, int G,
                                            int dtype) {
    return ss_layout(n_tokens, n_decode, n_reqs, H, dv, N, G, dtype == RV_DTYPE_BF16 ? 2 : 4).total;
}

template <typename T>
static int ss_run(const float* proj, int P, const float* filt, const float* conv_bias, const float* D,
                  float* conv_state, LaArgs a, const SsScratch& lay, T* out, int G, int taps, int norm_groups,
                  cudaStream_t s) {
    const int inner = a.H * a.dv, C = inner + 2 * G * a.d;
    float* num = a.scratch + lay.num;
    T* rows = (T*)(a.scratch + lay.rows);
    const ConvSilu conv = {proj, filt, conv_bias, conv_state, (long long)(taps - 1) * C, a.token_req, a.q_start,
                           a.state_slot, P, inner, 0, a.n_tokens, C, taps};
    conv_silu<T>(conv, rows, s);
    RV_CHECK_LAUNCH("state_space_conv");
    if (a.n_decode > 0 && la_tokens<T, true>((const T*)rows, a, num, s)) return 1;
    if (a.n_tokens > a.n_decode && a.n_reqs > a.n_decode) {
        const unsigned items = (unsigned)la_items(a.n_tokens - a.n_decode, a.n_reqs - a.n_decode);
        double* B = (double*)(a.scratch + lay.B);
        float *w = a.scratch + lay.w, *dec = a.scratch + lay.dec;
        rv_launch(ss_decay_kernel, dim3(items, (a.H + 31) / 32), dim3(256), 0, s, (const float*)a.z, a.z_stride,
                  a.bias, a.log_decay, a.q_start, a.state_slot, a.n_decode, a.n_reqs, B, w, dec, a.H);
        RV_CHECK_LAUNCH("state_space_decay");
        a.tk = {B, w};
        if (la_portions<T, LA_TOKEN>((const T*)rows, a, num, a.scratch + lay.kv, dec, items, s)) return 1;
    }
    const int part = inner / norm_groups;
    const bool vec = part % 4 == 0 && a.dv % 4 == 0 && C % 4 == 0 && P % 4 == 0 &&
                     (((uintptr_t)proj | (uintptr_t)rows | (uintptr_t)out | (uintptr_t)a.norm_w) & 15) == 0;
    const int lanes = vec ? part / 4 : part;
    const int threads = lanes >= 256 ? 256 : ((lanes + 31) / 32) * 32;
    const size_t smem = (size_t)part * sizeof(float);
    if (smem > 200 * 1024) RV_FAIL("state_space: a norm over %d values does not fit shared memory", part);
    const dim3 grid(a.n_tokens + (taps > 1 ? a.n_reqs : 0), norm_groups);
    if (vec) {
        LA_SMEM((ss_finish_kernel<T, 4>), smem)
        rv_launch(ss_finish_kernel<T, 4>, grid, dim3(threads), smem, s, (const float*)num, (const T*)rows, proj, P,
                  D, a.norm_w, a.eps, conv_state, a.token_req, a.q_start, a.state_slot, out, a.n_tokens, inner, C,
                  a.dv, part, taps);
    } else {
        LA_SMEM((ss_finish_kernel<T, 1>), smem)
        rv_launch(ss_finish_kernel<T, 1>, grid, dim3(threads), smem, s, (const float*)num, (const T*)rows, proj, P,
                  D, a.norm_w, a.eps, conv_state, a.token_req, a.q_start, a.state_slot, out, a.n_tokens, inner, C,
                  a.dv, part, taps);
    }
    RV_CHECK_LAUNCH("state_space_finish");
    return 0;
}

// filt [C, taps], conv_bias [C] with C = H dv + 2 G N; dt_bias, a_log, D [H]; norm_w [H dv];
// conv_state [slots, taps-1, C] (taps > 1); state [slots, H, N, dv]; scratch:
// rv_state_space_scratch floats, 16-byte aligned; out [n, H dv] of type `dtype`.  Requests
// [0, n_decode) bring one token each.  `tensor`: whether portions may take the tensor-core forms.
extern "C" int rv_state_space(const float* proj, int P, const float* filt, const float* conv_bias,
                              const float* dt_bias, const float* a_log, const float* D, const float* norm_w,
                              float* conv_state, float* state, const int* token_req, const int* q_start,
                              const int* state_slot, float* scratch, void* out, int dtype, int n_tokens,
                              int n_decode, int n_reqs, int H, int dv, int N, int G, int taps, int norm_groups,
                              float eps, int tensor, void* stream) {
    if (n_tokens == 0 || n_reqs == 0) return 0;
    if (n_tokens < 0 || n_decode < 0 || n_decode > n_reqs || n_decode > n_tokens || H < 1 || dv < 1 || N < 1 ||
        G < 1 || H % G || taps < 1 || norm_groups < 1 || (H * dv) % norm_groups)
        RV_FAIL("state_space: bad sizes");
    const int inner = H * dv, C = inner + 2 * G * N;
    if (P < inner + C + H) RV_FAIL("state_space: rows are too short");
    const int tiles_d = (N + LA_T - 1) / LA_T, tiles_v = (dv + LA_T - 1) / LA_T;
    if (n_reqs > 65535 || H > 65535 || N > 2048 || dv > 65535 || tiles_d * tiles_v > 65535 ||
        norm_groups > 65535 || n_tokens > 65535 * CS_TOKENS)
        RV_FAIL("state_space: too many tokens, requests or heads, or heads that are too large");
    if (((uintptr_t)scratch & 15) || (taps > 1 && !conv_state))
        RV_FAIL("state_space: the scratch must be 16-byte aligned, and the convolution needs its records");
    // (the tensor-core form's tiles of B, C and the state fit shared memory up to 256 rows here)
    tensor = tensor && dtype == RV_DTYPE_BF16 && N % 16 == 0 && dv % 16 == 0 && N <= 256 && C % 8 == 0;
    const SsScratch lay = ss_layout(n_tokens, n_decode, n_reqs, H, dv, N, G, dtype == RV_DTYPE_BF16 ? 2 : 4);
    const LaArgs a = {{inner + G * N, inner, 0, H / G}, {nullptr, nullptr}, (float*)proj + inner + C, a_log, dt_bias,
                      norm_w, state, scratch, token_req, q_start, state_slot, 1.f, 1.f, eps, C, P, n_tokens,
                      n_decode, n_reqs, H, N, dv, 0, 0, 0, tensor};
    RV_DISPATCH_DTYPE(dtype, "state_space",
                      return ss_run<T>(proj, P, filt, conv_bias, D, conv_state, a, lay, (T*)out, G, taps,
                                       norm_groups, (cudaStream_t)stream));
    return 0;
}
