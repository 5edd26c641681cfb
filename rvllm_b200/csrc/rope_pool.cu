// Rotation, cache write and the rows of pooled blocks, for attention over a window of tokens and the
// blocks before it.  Rows [n, stride] of the storage type:
//   [ q: H heads of d | k: G heads of d | v: G heads of d, unless values are keys ]
// Queries are rotated in place; keys go rotated to the key pages, values as they are (or the keys
// before the rotation) to the value pages: as in rope_partial.cu, which see for the rotation.
//
// A block of `pool` tokens has one row of its own: the means of its cached keys and values.  It is
// formed in the step that brings the block's last token: tokens of earlier steps are read from their
// pages, this step's are formed once more from their rows and rounded as the pages hold them (so
// that nothing waits for the page writes), added in the order of their positions in float32; so
// a block's row does not depend on how its tokens were cut into steps.
//
// Three kinds of thread blocks, which do not wait for one another: [0, n) the pooled blocks (block t
// works if token t completes one; a warp per key/value head), then keys and values (a warp per
// token: a pair's sine and cosine serve all heads), then queries (a warp per token and RP_QH heads).
// Queries are rotated in place; nothing else writes the rows, and only their own warp reads them.
// Plain reference: tests/plain_ops.py rope_pool_write.
#include "common.cuh"

#define RP_QH 4
#define RP_TOK 16

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
    int page_size, int pool, const int* __restrict__ pool_slots, T* k_cache,
    T* v_cache, T* __restrict__ pk, T* __restrict__ pv) {
    rv_pdl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int half = rot_dims >> 1;
    const int W = G * d;
    const int kv_blocks = (n_tokens + 3) / 4;
    if (blockIdx.x >= n_tokens + kv_blocks) {            // queries
        const int groups = (H + RP_QH - 1) / RP_QH;
        const long long w = (long long)(blockIdx.x - n_tokens - kv_blocks) * 4 + warp;
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
    if (blockIdx.x >= n_tokens) {                        // keys and values
        const int t = (blockIdx.x - n_tokens) * 4 + warp;
        const int slot = t < n_tokens ? slot_mapping[t] : -1;
        const float pos = t < n_tokens ? (float)positions[t] : 0.f;
        rv_pdl_wait();
        if (slot < 0) return;
        const T* row = rows + (size_t)t * stride;
        T* kd = k_cache + (size_t)slot * W;
        T* vd = v_cache + (size_t)slot * W;
        for (int i = lane; i < half + (d - rot_dims); i += 32) {
            const bool turns = i < half;
            const int a = turns ? i : rot_dims + (i - half), b = turns ? a + half : a;
            float sn = 0.f, cs = 1.f;
            if (turns) {
                sincosf(pos * freq[i], &sn, &cs);
                sn *= amplitude;
                cs *= amplitude;
            }
#pragma unroll 4
            for (int g = 0; g < G; ++g) {
                const int kc = (H + g) * d, vc = v_is_k ? kc : (H + G + g) * d, at = g * d;
                const float u = rv_load(row + kc + a), v = rv_load(row + kc + b);
                const T x = row[vc + a], y = row[vc + b];
                if (turns) {
                    rv_store(kd + at + a, u * cs - v * sn);
                    rv_store(kd + at + b, v * cs + u * sn);
                    vd[at + b] = y;
                } else {
                    kd[at + a] = row[kc + a];
                }
                vd[at + a] = x;
            }
        }
        return;
    }
    // the pooled block that token t completes
    const int t = blockIdx.x;
    const int out_slot = pool_slots[t];
    const int r = token_req[t], p1 = positions[t];
    const int p0 = p1 - pool + 1;                        // the block's first position
    const int first = max(p0, p1 - (t - q_start[r]));    // its first position in this step
    const int* table = block_table + (size_t)r * max_blocks;
    rv_pdl_wait();
    if (out_slot < 0) return;
    extern __shared__ float2 turn[];                     // [RP_TOK][half]: cosine, sine
    float* sums = (float*)(turn + RP_TOK * half);        // [2 W]: keys, values
    for (int i = threadIdx.x; i < 2 * W; i += 128) {
        const T* src = i < W ? k_cache + i : v_cache + (i - W);
        float sum = 0.f;
#pragma unroll 4
        for (int j = max(p0, 0); j < first; ++j) {
            const int page = table[j / page_size];
            if (page >= 0) sum += rv_load(src + ((size_t)page * page_size + j % page_size) * W);
        }
        sums[i] = sum;
    }
    for (int j0 = first; j0 <= p1; j0 += RP_TOK) {
        const int mn = min(RP_TOK, p1 - j0 + 1);
        __syncthreads();                                 // the sums; the round before has used its sines
        for (int i = threadIdx.x; i < mn * half; i += 128) {
            const int m = i / half, c = i - m * half;
            float sn, cs;
            sincosf((float)(j0 + m) * freq[c], &sn, &cs);
            turn[i] = make_float2(cs * amplitude, sn * amplitude);
        }
        __syncthreads();
        const T* row0 = rows + (size_t)(t - (p1 - j0)) * stride;
        for (int g = warp; g < G; g += 4) {
            const int kc = (H + g) * d, vc = v_is_k ? kc : (H + G + g) * d, at = g * d;
            for (int i = lane; i < half + (d - rot_dims); i += 32) {
                const bool turns = i < half;
                const int a = turns ? i : rot_dims + (i - half), b = turns ? a + half : a;
                float ka = sums[at + a], kb = sums[at + b], va = sums[W + at + a], vb = sums[W + at + b];
#pragma unroll 8
                for (int m = 0; m < mn; ++m) {
                    const T* row = row0 + (size_t)m * stride;
                    const float u = rv_load(row + kc + a), v = rv_load(row + kc + b);
                    const float2 cs = turns ? turn[m * half + i] : make_float2(1.f, 0.f);
                    ka += rp_round(turns ? u * cs.x - v * cs.y : u, rows);
                    kb += rp_round(v * cs.x + u * cs.y, rows);
                    va += v_is_k ? u : rv_load(row + vc + a);
                    vb += v_is_k ? v : rv_load(row + vc + b);
                }
                sums[at + a] = ka;
                sums[W + at + a] = va;
                if (turns) {
                    sums[at + b] = kb;
                    sums[W + at + b] = vb;
                }
            }
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < 2 * W; i += 128)
        rv_store((i < W ? pk + i : pv + (i - W)) + (size_t)out_slot * W, sums[i] / (float)pool);
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
    const size_t smem = (size_t)RP_TOK * (rot_dims / 2) * sizeof(float2) + (size_t)2 * G * d * sizeof(float);
    if (smem > 48 * 1024) RV_FAIL("rope_pool_write: %d heads of %d are too large", G, d);
    const long long blocks = n_tokens + ((long long)n_tokens + 3) / 4 + (freq ? ((long long)n_tokens * groups + 3) / 4 : 0);
    if (blocks > 0x7fffffffLL) RV_FAIL("rope_pool_write: too many rows");
    RV_DISPATCH_DTYPE(dtype, "rope_pool_write",
                      (rv_launch(rope_pool_write_kernel<T>, dim3((unsigned)blocks), dim3(128),
                                 smem,
                                 (cudaStream_t)stream, (T*)rows, stride, n_tokens, H, G, d, freq, rot_dims,
                                 amplitude, v_is_k, positions, token_req, q_start, slot_mapping, block_table,
                                 max_blocks, page_size, pool, pool_slots, (T*)k_cache, (T*)v_cache, (T*)pk,
                                 (T*)pv)));
    RV_CHECK_LAUNCH("rope_pool_write");
    return 0;
}
