// Rotation, cache write and the rows of pooled blocks, for attention over a window of tokens and the
// blocks before it.  Rows [n, stride] of the storage type:
//   [ q: H heads of d | k: G heads of d | v: G heads of d, unless values are keys ]
// Queries are rotated in place; keys go rotated to the key pages, values as they are (or the keys
// before the rotation) to the value pages: as in rope_partial.cu, which see for the rotation.
//
// A block of `pool` tokens has one row of its own: the means of its cached keys and values.  It is
// formed in the step that brings the block's last token: the tokens of earlier steps are read from
// their pages, those of this step are added as they are written (rounded to the storage type), all
// in the order of their positions in float32, so a block's row does not depend on how its tokens
// were cut into steps.
//
// Thread blocks [0, n) take the keys: block t works if token t is the first of its pooled block in
// this step and then walks the pooled block's tokens, a warp per key/value head (so no two warps
// meet).  The others take the queries: a warp per token and RP_QH heads, which share a pair's sine
// and cosine.  Plain reference: tests/plain_ops.py rope_pool_write.
#include "common.cuh"

#define RP_QH 4

__device__ __forceinline__ float rp_round(float x, const float*) { return x; }
__device__ __forceinline__ float rp_round(float x, const __nv_bfloat16*) {
    return __bfloat162float(__float2bfloat16_rn(x));
}

template <typename T>
__global__ void __launch_bounds__(128) rope_pool_write_kernel(
    T* __restrict__ rows, int stride, int n_tokens, int H, int G, int d, const float* __restrict__ freq,
    int rot_dims, float amplitude, int v_is_k, const int* __restrict__ positions,
    const int* __restrict__ token_req, const int* __restrict__ q_start,
    const int* __restrict__ slot_mapping, const int* __restrict__ block_table, int max_blocks,
    int page_size, int pool, const int* __restrict__ pool_slots, T* __restrict__ k_cache,
    T* __restrict__ v_cache, T* __restrict__ pk, T* __restrict__ pv) {
    rv_pdl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int half = rot_dims >> 1;
    if (blockIdx.x >= n_tokens) {                        // queries
        const int groups = (H + RP_QH - 1) / RP_QH;
        const long long w = (long long)(blockIdx.x - n_tokens) * 4 + warp;
        const int t = (int)(w / groups), h0 = (int)(w - (long long)t * groups) * RP_QH;
        const float pos = t < n_tokens && freq ? (float)positions[t] : 0.f;
        rv_pdl_wait();
        if (t >= n_tokens || !freq) return;
        T* row = rows + (size_t)t * stride;
        for (int i = lane; i < half; i += 32) {
            float sn, cs, u[RP_QH], v[RP_QH];
#pragma unroll
            for (int x = 0; x < RP_QH; ++x)
                if (h0 + x < H) {
                    u[x] = rv_load(row + (size_t)(h0 + x) * d + i);
                    v[x] = rv_load(row + (size_t)(h0 + x) * d + i + half);
                }
            sincosf(pos * freq[i], &sn, &cs);
            sn *= amplitude;
            cs *= amplitude;
#pragma unroll
            for (int x = 0; x < RP_QH; ++x)
                if (h0 + x < H) {
                    rv_store(row + (size_t)(h0 + x) * d + i, u[x] * cs - v[x] * sn);
                    rv_store(row + (size_t)(h0 + x) * d + i + half, v[x] * cs + u[x] * sn);
                }
        }
        return;
    }
    // keys: index arrays of the step come before the wait
    const int t = blockIdx.x;
    const int r = token_req[t], p = positions[t];
    const bool leads = slot_mapping[t] >= 0 && (p % pool == 0 || t == q_start[r]);
    const int p0 = p - p % pool;                         // the pooled block's first position
    const int n = min(q_start[r + 1] - t, p0 + pool - p);          // its tokens in this step
    const bool complete = leads && p + n == p0 + pool;
    const int out_slot = complete ? pool_slots[t + n - 1] : -1;
    const int* table = block_table + (size_t)r * max_blocks;
    rv_pdl_wait();
    if (!leads) return;
    const int W = G * d;
    const float inv = 1.f / (float)pool;
    auto cached = [&](const T* cache, int j, int at) -> float {
        const int page = table[j / page_size];
        return page >= 0 ? rv_load(cache + ((size_t)page * page_size + j % page_size) * W + at) : 0.f;
    };
    for (int g = warp; g < G; g += 4) {
        const int kc = (H + g) * d, vc = v_is_k ? kc : (H + G + g) * d, at = g * d;
        // pairs that turn, then the dimensions that pass
        for (int i = lane; i < half + (d - rot_dims); i += 32) {
            const bool turns = i < half;
            const int a = turns ? i : rot_dims + (i - half), b = a + half;
            float ka = 0.f, kb = 0.f, va = 0.f, vb = 0.f;
            if (out_slot >= 0)
                for (int j = p0; j < p; ++j) {
                    ka += cached(k_cache, j, at + a);
                    va += cached(v_cache, j, at + a);
                    if (turns) {
                        kb += cached(k_cache, j, at + b);
                        vb += cached(v_cache, j, at + b);
                    }
                }
            const float f = turns ? freq[i] : 0.f;
#pragma unroll 4
            for (int m = 0; m < n; ++m) {
                const T* row = rows + (size_t)(t + m) * stride;
                const int slot = slot_mapping[t + m];
                float u = rv_load(row + kc + a), v = turns ? rv_load(row + kc + b) : 0.f;
                const float x = v_is_k ? u : rv_load(row + vc + a), y = !turns ? 0.f : v_is_k ? v : rv_load(row + vc + b);
                if (turns) {
                    float sn, cs;
                    sincosf((float)(p + m) * f, &sn, &cs);
                    sn *= amplitude;
                    cs *= amplitude;
                    const float u2 = u * cs - v * sn;
                    v = v * cs + u * sn;
                    u = u2;
                }
                T* kd = k_cache + (size_t)slot * W + at;
                T* vd = v_cache + (size_t)slot * W + at;
                rv_store(kd + a, u);
                rv_store(vd + a, x);
                if (turns) {
                    rv_store(kd + b, v);
                    rv_store(vd + b, y);
                }
                ka += rp_round(u, k_cache);
                kb += rp_round(v, k_cache);
                va += x;
                vb += y;
            }
            if (out_slot >= 0) {
                T* ko = pk + (size_t)out_slot * W + at;
                T* vo = pv + (size_t)out_slot * W + at;
                rv_store(ko + a, ka * inv);
                rv_store(vo + a, va * inv);
                if (turns) {
                    rv_store(ko + b, kb * inv);
                    rv_store(vo + b, vb * inv);
                }
            }
        }
    }
}

extern "C" int rv_rope_pool_write(void* rows, int dtype, int stride, int n_tokens, int H, int G, int d,
                                  const float* freq, int rot_dims, float amplitude, int v_is_k,
                                  const int* positions, const int* token_req, const int* q_start,
                                  const int* slot_mapping, const int* block_table, int max_blocks,
                                  int page_size, int pool, const int* pool_slots, void* k_cache,
                                  void* v_cache, void* pk, void* pv, void* stream) {
    if (n_tokens == 0) return 0;
    if (n_tokens < 0 || H < 1 || G < 1 || d < 1 || pool < 1 || page_size < 1) RV_FAIL("rope_pool_write: bad sizes");
    if (!freq) rot_dims = 0;
    if (rot_dims % 2 || rot_dims > d || rot_dims < 0)
        RV_FAIL("rope_pool_write: %d turning dimensions do not fit a head of %d", rot_dims, d);
    if (stride < H * d + G * d * (v_is_k ? 1 : 2)) RV_FAIL("rope_pool_write: rows are too short");
    const int groups = (H + RP_QH - 1) / RP_QH;
    const long long blocks = n_tokens + (freq ? ((long long)n_tokens * groups + 3) / 4 : 0);
    if (blocks > 0x7fffffffLL) RV_FAIL("rope_pool_write: too many rows");
    RV_DISPATCH_DTYPE(dtype, "rope_pool_write",
                      (rv_launch(rope_pool_write_kernel<T>, dim3((unsigned)blocks), dim3(128), 0,
                                 (cudaStream_t)stream, (T*)rows, stride, n_tokens, H, G, d, freq, rot_dims,
                                 amplitude, v_is_k, positions, token_req, q_start, slot_mapping, block_table,
                                 max_blocks, page_size, pool, pool_slots, (T*)k_cache, (T*)v_cache, (T*)pk,
                                 (T*)pv)));
    RV_CHECK_LAUNCH("rope_pool_write");
    return 0;
}
