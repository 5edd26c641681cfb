// A causal convolution over time per channel and silu, ahead of a recurrence (state_space.cuh,
// gated_delta_chunk.cuh): float32 columns [off, off + C) of rows [n, P], filter [C, taps] (last column
// the current token's), bias [C] or null; inputs before a request's first token of the step come from its
// record, [taps-1][C] oldest first, records `rec` floats apart.  Output [n, C] of the compute type.  A
// thread has some channels of eight tokens, whose inputs it requests together (of one token, where
// they are few).
#pragma once
#include "chunks.cuh"

#define CS_TOKENS 8         // tokens a thread takes where there are many

template <int V>
__device__ __forceinline__ void cs_load(const float* p, float (&x)[V]) {
    if (V == 4) {
        const float4 f = *(const float4*)p;
        x[0] = f.x; x[1 % V] = f.y; x[2 % V] = f.z; x[3 % V] = f.w;
    } else {
        x[0] = *p;
    }
}

// TAPS 0: any number, `taps`.
template <typename T, int TAPS, int TT, int V>
__global__ void __launch_bounds__(128) conv_silu_kernel(
    const float* __restrict__ proj, int P, int off, const float* __restrict__ filt,
    const float* __restrict__ bias, const float* __restrict__ conv_state, long long rec,
    const int* __restrict__ token_req, const int* __restrict__ q_start,
    const int* __restrict__ state_slot, T* __restrict__ out, int first_token, int n_tokens, int C,
    int taps_any) {
    rv_pdl_launch_dependents();
    const int taps = TAPS ? TAPS : taps_any;
    const int c = (blockIdx.x * 128 + threadIdx.x) * V;
    const int first = first_token + blockIdx.y * TT;
    constexpr int KT = TAPS ? TAPS : 1;
    float w[KT][V], b[V];
    if (c < C) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
            b[e] = bias ? bias[c + e] : 0.f;
            if (TAPS)
#pragma unroll
                for (int j = 0; j < KT; ++j) w[j][e] = filt[(size_t)(c + e) * TAPS + j];
        }
    }
    rv_pdl_wait();
    if (c >= C) return;
    // input `m` of the request whose first token is t0 (m < t0: from its record)
    auto input = [&](int m, int t0, int slot, float (&x)[V]) {
        if (m >= t0) cs_load<V>(proj + (size_t)m * P + off + c, x);
        else cs_load<V>(conv_state + slot * rec + (size_t)(taps - 1 + m - t0) * C + c, x);
    };
    float x[TT][V];
#pragma unroll
    for (int i = 0; i < TT; ++i)
        if (first + i < n_tokens) cs_load<V>(proj + (size_t)(first + i) * P + off + c, x[i]);
    float before[KT > 1 ? KT - 1 : 1][V];                // the taps-1 inputs before the token
    int held = -1;                                       // the request they belong to
#pragma unroll
    for (int i = 0; i < TT; ++i) {
        const int t = first + i;
        if (t >= n_tokens) break;
        const int r = token_req[t];
        const int slot = state_slot[r];
        if (slot < 0) continue;
        const int t0 = q_start[r];
        float acc[V];
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = 0.f;
        if (TAPS) {
            if (r != held) {
#pragma unroll
                for (int j = 0; j < KT - 1; ++j) input(t - (KT - 1) + j, t0, slot, before[j]);
                held = r;
            }
#pragma unroll
            for (int e = 0; e < V; ++e) {
#pragma unroll
                for (int j = 0; j < KT - 1; ++j) acc[e] = fmaf(w[j][e], before[j][e], acc[e]);
                acc[e] = fmaf(w[KT - 1][e], x[i][e], acc[e]);
#pragma unroll
                for (int j = 0; j + 1 < KT - 1; ++j) before[j][e] = before[j + 1][e];
                if (KT > 1) before[KT > 1 ? KT - 2 : 0][e] = x[i][e];
            }
        } else {
            for (int j = 0; j < taps; ++j) {
                float xj[V];
                input(t - (taps - 1 - j), t0, slot, xj);
#pragma unroll
                for (int e = 0; e < V; ++e) acc[e] = fmaf(filt[(size_t)(c + e) * taps + j], xj[e], acc[e]);
            }
        }
#pragma unroll
        for (int e = 0; e < V; ++e) {
            acc[e] += b[e];
            acc[e] = acc[e] / (1.f + expf(-acc[e]));
        }
        la_store<T, V>(out + (size_t)t * C + c, acc);
    }
}

struct ConvSilu {
    const float *proj, *filt, *bias, *state;     // the state's first float of record 0
    long long rec;
    const int *token_req, *q_start, *state_slot;
    int P, off, first_token, n_tokens, C, taps;
};

template <typename T, int TT, int V>
static void conv_silu_launch(const ConvSilu& a, T* out, cudaStream_t s) {
    const dim3 grid((a.C / V + 127) / 128, (a.n_tokens - a.first_token + TT - 1) / TT);
#define CS_CONV(K)                                                                                         \
    rv_launch(conv_silu_kernel<T, K, TT, V>, grid, dim3(128), 0, s, a.proj, a.P, a.off, a.filt, a.bias,    \
              a.state, a.rec, a.token_req, a.q_start, a.state_slot, out, a.first_token, a.n_tokens, a.C, a.taps)
    if (a.taps == 2) CS_CONV(2);
    else if (a.taps == 3) CS_CONV(3);
    else if (a.taps == 4) CS_CONV(4);
    else CS_CONV(0);
#undef CS_CONV
}
// Tokens [first_token, n_tokens), at most 65,535 x 8 of them.
template <typename T>
static void conv_silu(const ConvSilu& a, T* out, cudaStream_t s) {
    if (a.n_tokens <= a.first_token) return;
    const bool v4 = a.C % 4 == 0 && a.P % 4 == 0 && a.off % 4 == 0 && a.rec % 4 == 0 &&
                    (((uintptr_t)a.proj | (uintptr_t)a.state | (uintptr_t)out) & 15) == 0;
    const bool few = (long long)(a.n_tokens - a.first_token) * ((a.C + 511) / 512) < 4 * rv_sm_count();
    if (v4 && few) conv_silu_launch<T, 1, 4>(a, out, s);
    else if (v4) conv_silu_launch<T, CS_TOKENS, 4>(a, out, s);
    else if (few) conv_silu_launch<T, 1, 1>(a, out, s);
    else conv_silu_launch<T, CS_TOKENS, 1>(a, out, s);
}
