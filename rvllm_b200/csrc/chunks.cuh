// What kernels that work on portions in chunks of 64 tokens share (linear_attention.cu,
// state_space.cuh, gated_delta_chunk.cuh): which tokens a chunk has, float32 operands as three bfloat16
// parts, and vector accesses.
#pragma once
#include "common.cuh"
#include "mma_bf16.cuh"

#define LA_C 64             // tokens a chunk
__device__ __forceinline__ float la_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// Chunk `item` of the portions of requests [first_req, n_reqs): its request and its number there;
// and how many chunks lie before the request.  Requests without a slot have none.  Whole warp.
__device__ __forceinline__ int la_chunks(const int* q_start, const int* state_slot, int r) {
    return state_slot[r] < 0 ? 0 : (q_start[r + 1] - q_start[r] + LA_C - 1) / LA_C;
}
__device__ __forceinline__ bool la_find(const int* q_start, const int* state_slot, int first_req,
                                        int n_reqs, int item, int lane, int& r, int& before) {
    before = 0;
    for (int base = first_req; base < n_reqs; base += 32) {
        const int n = base + lane < n_reqs ? la_chunks(q_start, state_slot, base + lane) : 0;
        int incl = n;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int up = __shfl_up_sync(0xffffffffu, incl, o);
            if (lane >= o) incl += up;
        }
        const unsigned hit = __ballot_sync(0xffffffffu, before + incl > item);
        if (hit) {
            const int l = __ffs(hit) - 1;
            r = base + l;
            before += __shfl_sync(0xffffffffu, incl - n, l);
            return true;
        }
        before += __shfl_sync(0xffffffffu, incl, 31);
    }
    return false;
}

// The most chunks the portions of `n_tokens` tokens in `n_reqs` requests can have.
static long long la_items(int n_tokens, int n_reqs) { return (long long)n_tokens / LA_C + n_reqs; }

// The pair (x, y) as three pairs of bfloat16 whose sum it is.
__device__ __forceinline__ void lm_split(float x, float y, unsigned& a, unsigned& b, unsigned& c) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 hf = __bfloat1622float2(h);
    x -= hf.x;
    y -= hf.y;
    const __nv_bfloat162 m = __floats2bfloat162_rn(x, y);
    const float2 mf = __bfloat1622float2(m);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - mf.x, y - mf.y);
    a = *(const unsigned*)&h;
    b = *(const unsigned*)&m;
    c = *(const unsigned*)&l;
}
__device__ __forceinline__ float2 lm_pair(unsigned u) { return __bfloat1622float2(*(const __nv_bfloat162*)&u); }
// Where a chunk lies: first token and token count (0: no such chunk).  Whole block.
__device__ __forceinline__ void lm_locate(const int* q_start, const int* state_slot, int first_req,
                                          int n_reqs, int item, int* at) {
    if (threadIdx.x < 32) {
        int r = -1, before = 0;
        const bool ok = la_find(q_start, state_slot, first_req, n_reqs, item, threadIdx.x, r, before);
        if (threadIdx.x == 0) {
            at[0] = ok ? q_start[r] + (item - before) * LA_C : -1;
            at[1] = ok ? min(LA_C, q_start[r + 1] - at[0]) : 0;
        }
    }
    __syncthreads();
}
// Four neighbouring values (16- and 8-byte accesses) or one.
template <typename T, int V>
__device__ __forceinline__ void la_load(const T* p, float (&x)[V]) {
    if (V == 4 && sizeof(T) == 4) {
        const float4 f = *(const float4*)p;
        x[0] = f.x; x[1 % V] = f.y; x[2 % V] = f.z; x[3 % V] = f.w;
    } else if (V == 4) {
        const uint2 u = *(const uint2*)p;
        const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&u.x), b = __bfloat1622float2(*(const __nv_bfloat162*)&u.y);
        x[0] = a.x; x[1 % V] = a.y; x[2 % V] = b.x; x[3 % V] = b.y;
    } else {
        x[0] = rv_load(p);
    }
}
template <typename T, int V>
__device__ __forceinline__ void la_store(T* p, const float (&x)[V]) {
    if (V == 4 && sizeof(T) == 4) {
        *(float4*)p = make_float4(x[0], x[1 % V], x[2 % V], x[3 % V]);
    } else if (V == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(x[0], x[1 % V]), b = __floats2bfloat162_rn(x[2 % V], x[3 % V]);
        uint2 u;
        u.x = *(const unsigned*)&a;
        u.y = *(const unsigned*)&b;
        *(uint2*)p = u;
    } else {
        rv_store(p, x[0]);
    }
}
