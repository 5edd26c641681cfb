// Paged grouped-query attention in float32 arithmetic on CUDA cores, for float32 or
// bfloat16 storage: the true-32-bit path's attention, and the decode attention of the
// bfloat16 path (decode is bound by reading the pages, not by arithmetic).
//
// Two kernels share the inner loop.
//   paged_attention_warp_kernel    one warp per (token, query head); any number of new
//                                  tokens per request.  Keys are taken 32 at a time in
//                                  groups aligned to absolute position 0, so the order
//                                  of every sum depends on the positions only, not on
//                                  how the tokens were cut into steps.
//   paged_attention_decode_kernel  one block per (request, key/value head, split of 256
//                                  keys); the query heads of a group share each key and
//                                  value load; partial results go to scratch and
//                                  paged_attention_merge_kernel combines the splits in
//                                  order.  Split boundaries are fixed multiples of 256.
//
// A key at position j is visible to the query at position p iff j <= p, and with a
// window iff j > p - window; the softmax is the online form (running maximum and sum).
// Two options.  `vd`: the size of a value head when it is not the key size `hd` (the value
// pages are then [slots, kv heads, vd]).  `sinks` (float32, one per query head, or null):
// the softmax's denominator holds one more term exp(sinks[h]) that has no key and no value;
// it enters as the initial running maximum with a sum of 1, in the split form once, in the
// merge.  Key sizes that are no multiple of 8 (bfloat16) or 4 (float32) elements take scalar
// loads.
// A third (template flag EXT): a window of tokens and pooled blocks before it, and capped scores
// (attention_pooled.cuh); the plain instantiations do not carry it.
// Reference counterparts: kv_gather.cu (twice), a batched SGEMM, mask_add_broadcast.cu,
// softmax.cu, a batched SGEMM and transposes (src/cuda/model.rs:528-581).
// Plain reference: tests/plain_ops.py paged_attention.
#include "attention_pooled.cuh"
#include "common.cuh"

#define RV_ATTN_MAX_DPL 16     // head sizes up to 512: up to 16 dimensions per lane
#define RV_ATTN_GT 4           // query heads of a group handled together in decode
#define RV_ATTN_SPLIT 256      // keys per decode split

template <bool kFast>
__device__ __forceinline__ float rv_exp(float x) {
    return kFast ? __expf(x) : expf(x);
}

// cap * tanh(s / cap).  kFast (the result is weighed against bfloat16 values): through one
// exponential and a fast division, whose error is some 1e-7 of the cap.
template <bool kFast>
__device__ __forceinline__ float rv_cap(float s, float cap) {
    if (!kFast) return cap * tanhf(s / cap);
    return cap - 2.f * cap * __fdividef(1.f, 1.f + __expf(2.f * s / cap));
}

// dot product of a float32 vector in shared memory with a stored row
__device__ __forceinline__ float rv_dot_row(const float* __restrict__ q, const float* __restrict__ k,
                                            int hd) {
    float s = 0.f;
    for (int d = 0; d < hd; d += 4) {
        const float4 kv = *(const float4*)(k + d);
        s += q[d] * kv.x + q[d + 1] * kv.y + q[d + 2] * kv.z + q[d + 3] * kv.w;
    }
    return s;
}
__device__ __forceinline__ float rv_dot_row(const float* __restrict__ q,
                                            const __nv_bfloat16* __restrict__ k, int hd) {
    float s = 0.f;
    for (int d = 0; d < hd; d += 8) {
        const uint4 raw = *(const uint4*)(k + d);
        const __nv_bfloat162* h = (const __nv_bfloat162*)&raw;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(h[i]);
            s += q[d + 2 * i] * f.x + q[d + 2 * i + 1] * f.y;
        }
    }
    return s;
}

// any head size: vector loads when the rows allow them, else one element at a time
template <typename T>
__device__ __forceinline__ float rv_dot_any(const float* __restrict__ q, const T* __restrict__ k,
                                            int hd, bool vec) {
    if (vec) return rv_dot_row(q, k, hd);
    float s = 0.f;
    for (int d = 0; d < hd; ++d) s += q[d] * rv_load(k + d);
    return s;
}

// ---------------------------------------------------------------------------------
template <typename T, int DPL, bool EXT>
__global__ void paged_attention_warp_kernel(
    const T* __restrict__ q, int q_stride, const T* __restrict__ k_cache,
    const T* __restrict__ v_cache, const int* __restrict__ block_table, int max_blocks,
    const int* __restrict__ q_start, const int* __restrict__ ctx_lens,
    const int* __restrict__ token_req, T* __restrict__ out, int first_token, int n_tokens,
    int num_heads, int num_kv_heads, int hd, int page_size, float scale, int window, int vd,
    const float* __restrict__ sinks, const RvPooled pl) {
    rv_pdl_prologue();
    constexpr bool kFast = sizeof(T) == 2;
    const bool vec = hd % (16 / (int)sizeof(T)) == 0;
    extern __shared__ float q_smem[];   // [warps per block][hd]
    const int lane = threadIdx.x & 31, wib = threadIdx.x >> 5;
    const long long warp = (long long)blockIdx.x * (blockDim.x >> 5) + wib;
    if (warp >= (long long)n_tokens * num_heads) return;
    const int t = first_token + (int)(warp / num_heads);
    const int h = (int)(warp % num_heads);
    const int g = h / (num_heads / num_kv_heads);
    const int r = token_req[t];
    const int clen = ctx_lens[r];
    T* o = out + (size_t)t * num_heads * vd + (size_t)h * vd;
    if (clen == 0) {
        for (int d = lane; d < vd; d += 32) rv_store(o + d, 0.f);
        return;
    }
    const int qs = q_start[r];
    const int p = clen - (q_start[r + 1] - qs) + (t - qs);
    const int lo = window > 0 ? max(0, p - window + 1) : 0;
    float* qv = q_smem + wib * hd;
    const T* qrow = q + (size_t)t * q_stride + (size_t)h * hd;
    for (int d = lane; d < hd; d += 32) qv[d] = rv_load(qrow + d);
    __syncwarp();

    float m = sinks ? sinks[h] : -INFINITY, l = sinks ? 1.f : 0.f, acc[DPL];
#pragma unroll
    for (int i = 0; i < DPL; ++i) acc[i] = 0.f;
    const size_t row = (size_t)num_kv_heads * hd, vrow_len = (size_t)num_kv_heads * vd;

    // EXT: the pooled blocks first, then the tokens
    for (int part = EXT && pl.pool > 0 ? 0 : 1; part < 2; ++part) {
    const bool blocks = EXT && part == 0;
    const int first = blocks ? 0 : lo, last = blocks ? rv_seen_blocks(p, window, pl.pool, pl.most) - 1 : p;
    const int* table = blocks ? pl.table + (size_t)r * pl.max_blocks : block_table + (size_t)r * max_blocks;
    const T* kc = blocks ? (const T*)pl.k : k_cache;
    const T* vc = blocks ? (const T*)pl.v : v_cache;
    for (int base = first & ~31; base <= last; base += 32) {
        const int j = base + lane;
        const bool valid = j >= first && j <= last;
        int slot = 0;
        float s = -INFINITY;
        if (valid) {
            slot = table[j / page_size] * page_size + j % page_size;
            s = rv_dot_any(qv, kc + (size_t)slot * row + (size_t)g * hd, hd, vec) * scale;
            if (EXT && pl.cap > 0.f) s = rv_cap<kFast>(s, pl.cap);
        }
        const float m_new = fmaxf(m, rv_warp_max(s));
        const float pj = valid ? rv_exp<kFast>(s - m_new) : 0.f;
        const float corr = rv_exp<kFast>(m - m_new);
        l = l * corr + rv_warp_sum(pj);
        m = m_new;
#pragma unroll
        for (int i = 0; i < DPL; ++i) acc[i] *= corr;
        const int count = min(32, last - base + 1);
        for (int jj = 0; jj < count; ++jj) {
            const float pk = __shfl_sync(0xffffffffu, pj, jj);
            const int sk = __shfl_sync(0xffffffffu, slot, jj);
            if (pk != 0.f) {
                const T* vrow = vc + (size_t)sk * vrow_len + (size_t)g * vd;
#pragma unroll
                for (int i = 0; i < DPL; ++i) {
                    const int d = lane + 32 * i;
                    if (d < vd) acc[i] += pk * rv_load(vrow + d);
                }
            }
        }
    }
    }
#pragma unroll
    for (int i = 0; i < DPL; ++i) {
        const int d = lane + 32 * i;
        if (d < vd) rv_store(o + d, acc[i] / l);
    }
}

// ---------------------------------------------------------------------------------
// Decode: requests [0, n_reqs) bring one token each, token index == request index.
// Scratch per (request, head, split): part_o[hd] (unnormalised) and part_ml = (max, sum).
template <typename T, int DPL, bool EXT>
__global__ void __launch_bounds__(128) paged_attention_decode_kernel(
    const T* __restrict__ q, int q_stride, const T* __restrict__ k_cache,
    const T* __restrict__ v_cache, const int* __restrict__ block_table, int max_blocks,
    const int* __restrict__ ctx_lens, float* __restrict__ part_o, float2* __restrict__ part_ml,
    int max_splits, int num_heads, int num_kv_heads, int hd, int page_size, float scale,
    int window, int vd, const RvPooled pl) {
    rv_pdl_prologue();
    constexpr bool kFast = sizeof(T) == 2;
    constexpr int GT = RV_ATTN_GT;
    const bool vec = hd % (16 / (int)sizeof(T)) == 0;
    extern __shared__ float smem[];
    const int G = num_heads / num_kv_heads;
    const int tiles = (G + GT - 1) / GT;
    const int g = blockIdx.x / tiles;                 // key/value head
    const int h0 = g * G + (blockIdx.x % tiles) * GT; // first query head of this block
    const int gcount = min(GT, g * G + G - h0);
    const int r = blockIdx.y;
    const int split = blockIdx.z;
    const int clen = ctx_lens[r];
    if (clen == 0) return;
    const int p = clen - 1;
    const int lo = window > 0 ? max(0, p - window + 1) : 0;
    // EXT: which rows this split covers (attention_pooled.cuh)
    const bool blocks = EXT && split < pl.psplits;
    const int stretch = !EXT || blocks ? split : split - pl.psplits + lo / RV_ATTN_SPLIT;
    const int k0 = max(blocks ? 0 : lo, stretch * RV_ATTN_SPLIT);
    const int k1 = min(blocks ? rv_seen_blocks(p, window, pl.pool, pl.most) - 1 : p,
                       stretch * RV_ATTN_SPLIT + RV_ATTN_SPLIT - 1);   // inclusive
    if ((!EXT && split < lo / RV_ATTN_SPLIT) || k0 > k1) return;

    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
    float* qv = smem;                                // [GT][hd]
    float* ps = qv + GT * hd;                        // [4 warps][32][GT]
    int* ss = (int*)(ps + 4 * 32 * GT);              // [4 warps][32]
    float* red = (float*)(ss + 4 * 32);              // [4 warps][GT][vd + 2]
    for (int i = threadIdx.x; i < GT * hd; i += blockDim.x) {
        const int gi = i / hd, d = i - gi * hd;
        qv[i] = gi < gcount ? rv_load(q + (size_t)r * q_stride + (size_t)(h0 + gi) * hd + d) : 0.f;
    }
    __syncthreads();

    float m[GT], l[GT], acc[GT][DPL];
#pragma unroll
    for (int gi = 0; gi < GT; ++gi) {
        m[gi] = -INFINITY;
        l[gi] = 0.f;
#pragma unroll
        for (int i = 0; i < DPL; ++i) acc[gi][i] = 0.f;
    }
    const int* table = blocks ? pl.table + (size_t)r * pl.max_blocks : block_table + (size_t)r * max_blocks;
    const T* kc = blocks ? (const T*)pl.k : k_cache;
    const T* vc = blocks ? (const T*)pl.v : v_cache;
    const size_t row = (size_t)num_kv_heads * hd, vrow_len = (size_t)num_kv_heads * vd;
    float* my_p = ps + w * 32 * GT;
    int* my_s = ss + w * 32;

    const int split_base = stretch * RV_ATTN_SPLIT;
    for (int base = split_base + w * 32; base <= k1; base += 4 * 32) {
        if (base + 31 < k0) continue;
        const int j = base + lane;
        const bool valid = j >= k0 && j <= k1;
        int slot = 0;
        float s[GT];
#pragma unroll
        for (int gi = 0; gi < GT; ++gi) s[gi] = -INFINITY;
        if (valid) {
            slot = table[j / page_size] * page_size + j % page_size;
            const T* krow = kc + (size_t)slot * row + (size_t)g * hd;
#pragma unroll
            for (int gi = 0; gi < GT; ++gi)
                if (gi < gcount) {
                    s[gi] = rv_dot_any(qv + gi * hd, krow, hd, vec) * scale;
                    if (EXT && pl.cap > 0.f) s[gi] = rv_cap<kFast>(s[gi], pl.cap);
                }
        }
        my_s[lane] = slot;
#pragma unroll
        for (int gi = 0; gi < GT; ++gi) {
            if (gi < gcount) {
                const float m_new = fmaxf(m[gi], rv_warp_max(s[gi]));
                const float pj = valid ? rv_exp<kFast>(s[gi] - m_new) : 0.f;
                const float corr = rv_exp<kFast>(m[gi] - m_new);
                l[gi] = l[gi] * corr + rv_warp_sum(pj);
                m[gi] = m_new;
#pragma unroll
                for (int i = 0; i < DPL; ++i) acc[gi][i] *= corr;
                my_p[lane * GT + gi] = pj;
            } else {
                my_p[lane * GT + gi] = 0.f;
            }
        }
        __syncwarp();
        const int count = min(32, k1 - base + 1);
        for (int jj = max(0, k0 - base); jj < count; ++jj) {
            const T* vrow = vc + (size_t)my_s[jj] * vrow_len + (size_t)g * vd;
            float pk[GT];
#pragma unroll
            for (int gi = 0; gi < GT; ++gi) pk[gi] = my_p[jj * GT + gi];
#pragma unroll
            for (int i = 0; i < DPL; ++i) {
                const int d = lane + 32 * i;
                if (d < vd) {
                    const float v = rv_load(vrow + d);
#pragma unroll
                    for (int gi = 0; gi < GT; ++gi) acc[gi][i] += pk[gi] * v;
                }
            }
        }
        __syncwarp();
    }
    // combine the four warps in warp order
    const int rs = vd + 2;
#pragma unroll
    for (int gi = 0; gi < GT; ++gi) {
        float* mine = red + (size_t)(w * GT + gi) * rs;
#pragma unroll
        for (int i = 0; i < DPL; ++i) {
            const int d = lane + 32 * i;
            if (d < vd) mine[d] = acc[gi][i];
        }
        if (lane == 0) {
            mine[vd] = m[gi];
            mine[vd + 1] = l[gi];
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < gcount * vd; i += blockDim.x) {
        const int gi = i / vd, d = i - gi * vd;
        float M = -INFINITY;
        for (int ww = 0; ww < 4; ++ww) M = fmaxf(M, red[(size_t)(ww * GT + gi) * rs + vd]);
        float L = 0.f, O = 0.f;
        for (int ww = 0; ww < 4; ++ww) {
            const float* src = red + (size_t)(ww * GT + gi) * rs;
            const float f = src[vd] == -INFINITY ? 0.f : rv_exp<kFast>(src[vd] - M);
            L += src[vd + 1] * f;
            O += src[d] * f;
        }
        const size_t slot = ((size_t)r * num_heads + h0 + gi) * max_splits + split;
        part_o[slot * vd + d] = O;
        if (d == 0) part_ml[slot] = make_float2(M, L);
    }
}

template <typename T, bool EXT>
__global__ void paged_attention_merge_kernel(const float* __restrict__ part_o,
                                             const float2* __restrict__ part_ml,
                                             const int* __restrict__ ctx_lens, T* __restrict__ out,
                                             int max_splits, int num_heads, int hd, int window,
                                             int split_keys, const float* __restrict__ sinks,
                                             int psplits, int pool, int most) {
    rv_pdl_launch_dependents();
    constexpr bool kFast = sizeof(T) == 2;
    const int r = blockIdx.y, h = blockIdx.x;
    const int clen = ctx_lens[r];                 // the step's index array: before the wait
    const float sink = sinks ? sinks[h] : -INFINITY;      // a constant of the layer
    rv_pdl_wait();
    T* o = out + ((size_t)r * num_heads + h) * hd;
    if (clen == 0) {
        for (int d = threadIdx.x; d < hd; d += blockDim.x) rv_store(o + d, 0.f);
        return;
    }
    const int p = clen - 1;
    const int lo = window > 0 ? max(0, p - window + 1) : 0;
    // A context longer than the launch's max_ctx_len has keys that no split covered: the row
    // is marked invalid (NaN) and nothing outside this head's slots is read.
    // (EXT: splits that cover blocks, then splits that cover tokens from the window's first on.)
    const int np = EXT ? (rv_seen_blocks(p, window, pool, most) + split_keys - 1) / split_keys : 0;
    const int nt = p / split_keys - lo / split_keys + 1;
    if (EXT ? (np > psplits || nt > max_splits - psplits) : (clen > max_splits * split_keys)) {
        for (int d = threadIdx.x; d < hd; d += blockDim.x) rv_store(o + d, NAN);
        return;
    }
    const int s0 = EXT ? 0 : lo / split_keys, s1 = EXT ? np + nt - 1 : min(p / split_keys, max_splits - 1);
    const size_t base = ((size_t)r * num_heads + h) * max_splits;
    // Splits are combined in order, sixteen at a time: the loads of a group are independent, so
    // a group costs one memory latency, not sixteen.
    constexpr int GROUP = 16;
    for (int d = threadIdx.x; d < hd; d += blockDim.x) {
        float M = sink, L = sinks ? 1.f : 0.f, O = 0.f;     // the sink counts once, here
        for (int sb = s0; sb <= s1; sb += GROUP) {
            float2 ml[GROUP];
            float po[GROUP];
#pragma unroll
            for (int i = 0; i < GROUP; ++i) {
                const bool valid = sb + i <= s1;
                const int sp = EXT && sb + i >= np ? sb + i - np + psplits : sb + i;
                ml[i] = valid ? part_ml[base + sp] : make_float2(-INFINITY, 0.f);
                po[i] = valid ? part_o[(base + sp) * hd + d] : 0.f;
            }
            float mg = M;
#pragma unroll
            for (int i = 0; i < GROUP; ++i) mg = fmaxf(mg, ml[i].x);
            if (mg == -INFINITY) continue;
            const float keep = rv_exp<kFast>(M - mg);          // M = -inf -> 0
            O *= keep;
            L *= keep;
#pragma unroll
            for (int i = 0; i < GROUP; ++i) {
                const float w = ml[i].y > 0.f ? rv_exp<kFast>(ml[i].x - mg) : 0.f;
                O += po[i] * w;
                L += ml[i].y * w;
            }
            M = mg;
        }
        rv_store(o + d, L > 0.f ? O / L : 0.f);
    }
}

// ---------------------------------------------------------------------------------
static int check_attention_sizes(const char* name, int num_heads, int num_kv_heads, int hd, int vd,
                                 int page_size, int dtype) {
    if (num_heads <= 0 || num_kv_heads <= 0 || num_heads % num_kv_heads)
        RV_FAIL("%s: invalid head counts: %d query, %d KV", name, num_heads, num_kv_heads);
    if (hd <= 0 || hd > 32 * RV_ATTN_MAX_DPL || vd <= 0 || vd > 32 * RV_ATTN_MAX_DPL)
        RV_FAIL("%s: head sizes %d and %d are not supported (at most %d)", name, hd, vd,
                32 * RV_ATTN_MAX_DPL);
    if (page_size <= 0) RV_FAIL("%s: bad page size %d", name, page_size);
    (void)dtype;
    return 0;
}

#define RV_DISPATCH_DPL(hd, ...)                                          \
    switch (((hd) + 31) / 32) {                                           \
        case 1: { constexpr int DPL = 1; __VA_ARGS__; break; }            \
        case 2: { constexpr int DPL = 2; __VA_ARGS__; break; }            \
        case 3: { constexpr int DPL = 3; __VA_ARGS__; break; }            \
        case 4: { constexpr int DPL = 4; __VA_ARGS__; break; }            \
        case 5: case 6: { constexpr int DPL = 6; __VA_ARGS__; break; }    \
        case 7: case 8: { constexpr int DPL = 8; __VA_ARGS__; break; }    \
        default: { constexpr int DPL = 16; __VA_ARGS__; break; }          \
    }

// `vd`: size of a value head; `sinks`: float32 [num_heads] or null (see the top of the file).
extern "C" int rv_paged_attention_warp_ex(const void* q, int dtype, int q_stride,
                                          const void* k_cache, const void* v_cache,
                                          const int* block_table, int max_blocks,
                                          const int* q_start, const int* ctx_lens,
                                          const int* token_req, void* out, int first_token,
                                          int n_tokens, int num_heads, int num_kv_heads, int hd,
                                          int page_size, float scale, int window, int vd,
                                          const float* sinks, void* stream) {
    if (n_tokens == 0) return 0;
    if (check_attention_sizes("paged_attention", num_heads, num_kv_heads, hd, vd, page_size, dtype))
        return 1;
    const int wpb = 4;
    const long long warps = (long long)n_tokens * num_heads;
    const long long blocks = (warps + wpb - 1) / wpb;
    if (blocks > 0x7fffffffLL) RV_FAIL("paged_attention: too many rows");
    const size_t smem = (size_t)wpb * hd * sizeof(float);
    cudaStream_t s = (cudaStream_t)stream;
    RV_DISPATCH_DTYPE(dtype, "paged_attention",
        RV_DISPATCH_DPL(vd, (rv_launch(paged_attention_warp_kernel<T, DPL, false>, dim3((int)blocks), dim3(wpb * 32), smem, s, 
            (const T*)q, q_stride, (const T*)k_cache, (const T*)v_cache, block_table, max_blocks,
            q_start, ctx_lens, token_req, (T*)out, first_token, n_tokens, num_heads, num_kv_heads,
            hd, page_size, scale, window, vd, sinks, RvPooled()))));
    RV_CHECK_LAUNCH("paged_attention");
    return 0;
}

extern "C" int rv_paged_attention_warp(const void* q, int dtype, int q_stride, const void* k_cache,
                                       const void* v_cache, const int* block_table, int max_blocks,
                                       const int* q_start, const int* ctx_lens,
                                       const int* token_req, void* out, int first_token,
                                       int n_tokens, int num_heads, int num_kv_heads, int hd,
                                       int page_size, float scale, int window, void* stream) {
    return rv_paged_attention_warp_ex(q, dtype, q_stride, k_cache, v_cache, block_table, max_blocks,
                                      q_start, ctx_lens, token_req, out, first_token, n_tokens,
                                      num_heads, num_kv_heads, hd, page_size, scale, window, hd,
                                      nullptr, stream);
}

// Bytes of part_o for so many (request, head, split) triples, before part_ml's pairs of floats: a
// multiple of 8 (an odd value size times an odd count is not).
static size_t part_bytes(size_t slots, int vd) { return (slots * vd * 4 + 7) & ~(size_t)7; }

// Bytes of scratch rv_paged_attention_decode needs: part_o then part_ml (`hd`: the value size).
extern "C" long long rv_paged_attention_decode_scratch_bytes(int n_reqs, int num_heads, int hd,
                                                             int max_ctx_len) {
    const long long splits = (max_ctx_len + RV_ATTN_SPLIT - 1) / RV_ATTN_SPLIT;
    const long long slots = (long long)n_reqs * num_heads * (splits > 0 ? splits : 1);
    return (long long)part_bytes(slots, hd) + slots * 8;
}

static int merge_threads(int hd) { return hd < 32 ? 32 : (hd > 128 ? 128 : ((hd + 31) / 32) * 32); }

extern "C" int rv_paged_attention_decode_ex(const void* q, int dtype, int q_stride,
                                            const void* k_cache, const void* v_cache,
                                            const int* block_table, int max_blocks,
                                            const int* ctx_lens, void* out, void* scratch,
                                            long long scratch_bytes, int n_reqs, int max_ctx_len,
                                            int num_heads, int num_kv_heads, int hd, int page_size,
                                            float scale, int window, int vd, const float* sinks,
                                            void* stream) {
    if (n_reqs == 0) return 0;
    if (check_attention_sizes("paged_attention_decode", num_heads, num_kv_heads, hd, vd, page_size,
                              dtype))
        return 1;
    int max_splits = (max_ctx_len + RV_ATTN_SPLIT - 1) / RV_ATTN_SPLIT;
    if (max_splits < 1) max_splits = 1;
    if (rv_paged_attention_decode_scratch_bytes(n_reqs, num_heads, vd, max_ctx_len) > scratch_bytes)
        RV_FAIL("paged_attention_decode: scratch of %lld bytes is too small", scratch_bytes);
    if (n_reqs > 65535 || max_splits > 65535) RV_FAIL("paged_attention_decode: batch too large");
    const size_t slots = (size_t)n_reqs * num_heads * max_splits;
    float* part_o = (float*)scratch;
    float2* part_ml = (float2*)((char*)scratch + part_bytes(slots, vd));
    const int G = num_heads / num_kv_heads;
    const int tiles = (G + RV_ATTN_GT - 1) / RV_ATTN_GT;
    dim3 grid(num_kv_heads * tiles, n_reqs, max_splits);
    const size_t smem = (size_t)(RV_ATTN_GT * hd + 4 * 32 * RV_ATTN_GT + 4 * 32 +
                                 4 * RV_ATTN_GT * (vd + 2)) * sizeof(float);
    cudaStream_t s = (cudaStream_t)stream;
    RV_DISPATCH_DTYPE(dtype, "paged_attention_decode",
        RV_DISPATCH_DPL(vd, (rv_launch(paged_attention_decode_kernel<T, DPL, false>, dim3(grid), dim3(128), smem, s, 
            (const T*)q, q_stride, (const T*)k_cache, (const T*)v_cache, block_table, max_blocks,
            ctx_lens, part_o, part_ml, max_splits, num_heads, num_kv_heads, hd, page_size, scale,
            window, vd, RvPooled()))));
    RV_CHECK_LAUNCH("paged_attention_decode");
    dim3 mgrid(num_heads, n_reqs);
    RV_DISPATCH_DTYPE(dtype, "paged_attention_merge",
        (rv_launch(paged_attention_merge_kernel<T, false>, dim3(mgrid), dim3(merge_threads(vd)), 0, s, 
            part_o, part_ml, ctx_lens, (T*)out, max_splits, num_heads, vd, window, RV_ATTN_SPLIT,
            sinks, 0, 0, 0)));
    RV_CHECK_LAUNCH("paged_attention_merge");
    return 0;
}

extern "C" int rv_paged_attention_decode(const void* q, int dtype, int q_stride,
                                         const void* k_cache, const void* v_cache,
                                         const int* block_table, int max_blocks,
                                         const int* ctx_lens, void* out, void* scratch,
                                         long long scratch_bytes, int n_reqs, int max_ctx_len,
                                         int num_heads, int num_kv_heads, int hd, int page_size,
                                         float scale, int window, void* stream) {
    return rv_paged_attention_decode_ex(q, dtype, q_stride, k_cache, v_cache, block_table,
                                        max_blocks, ctx_lens, out, scratch, scratch_bytes, n_reqs,
                                        max_ctx_len, num_heads, num_kv_heads, hd, page_size, scale,
                                        window, hd, nullptr, stream);
}

// The merge step alone, for partial results written by another kernel (attention_mma.cu)
// in the same scratch layout.  `hd`: the value size; `sinks`: float32 [num_heads] or null.
extern "C" int rv_paged_attention_merge_ex(const void* scratch, const int* ctx_lens, void* out,
                                           int dtype, int n_reqs, int max_ctx_len, int num_heads,
                                           int hd, int window, int split_keys, const float* sinks,
                                           void* stream) {
    if (n_reqs == 0) return 0;
    if (split_keys <= 0) RV_FAIL("paged_attention_merge: bad split size");
    int max_splits = (max_ctx_len + split_keys - 1) / split_keys;
    if (max_splits < 1) max_splits = 1;
    if (n_reqs < 0 || n_reqs > 65535 || num_heads <= 0 || hd <= 0)
        RV_FAIL("paged_attention_merge: bad sizes");
    const size_t slots = (size_t)n_reqs * num_heads * max_splits;
    const float* part_o = (const float*)scratch;
    const float2* part_ml = (const float2*)((const char*)scratch + part_bytes(slots, hd));
    dim3 mgrid(num_heads, n_reqs);
    RV_DISPATCH_DTYPE(dtype, "paged_attention_merge",
        (rv_launch(paged_attention_merge_kernel<T, false>, dim3(mgrid), dim3(merge_threads(hd)), 0, (cudaStream_t)stream, 
            part_o, part_ml, ctx_lens, (T*)out, max_splits, num_heads, hd, window, split_keys,
            sinks, 0, 0, 0)));
    RV_CHECK_LAUNCH("paged_attention_merge");
    return 0;
}

extern "C" int rv_paged_attention_merge(const void* scratch, const int* ctx_lens, void* out,
                                        int dtype, int n_reqs, int max_ctx_len, int num_heads,
                                        int hd, int window, int split_keys, void* stream) {
    return rv_paged_attention_merge_ex(scratch, ctx_lens, out, dtype, n_reqs, max_ctx_len,
                                       num_heads, hd, window, split_keys, nullptr, stream);
}

// ---------------------------------------------------------------------------------
// Attention over a window of tokens and the pooled blocks before it (attention_pooled.cuh).
// `window` 0: every token is seen; `pool` 0: no blocks (pk, pv, ptable unused); `most` 0: no bound on
// the blocks seen; `cap` 0: scores are not capped; `vd`: the size of a value head.

// Bytes of scratch of the split form: part_o then part_ml.
extern "C" long long rv_paged_attention_pooled_scratch_bytes(int n_reqs, int num_heads, int vd,
                                                             int max_ctx_len, int window, int pool,
                                                             int most) {
    const long long splits = rv_pooled_psplits(max_ctx_len, window, pool, most, RV_ATTN_SPLIT) +
                             rv_pooled_tsplits(max_ctx_len, window, RV_ATTN_SPLIT);
    const long long slots = (long long)n_reqs * num_heads * splits;
    return (long long)part_bytes(slots, vd) + slots * 8;
}

static int pooled_check(const char* name, int num_heads, int num_kv_heads, int hd, int vd, int page_size,
                        int window, int pool, int most, const void* pk, const void* pv, const int* ptable,
                        int dtype) {
    if (check_attention_sizes(name, num_heads, num_kv_heads, hd, vd, page_size, dtype)) return 1;
    if (window < 0 || pool < 0 || most < 0 || (pool > 0 && (window == 0 || !pk || !pv || !ptable)))
        RV_FAIL("%s: pooled blocks need a window, pages and a block table", name);
    return 0;
}

// One warp per (token, query head), any number of new tokens per request.
extern "C" int rv_paged_attention_pooled_warp(
    const void* q, int dtype, int q_stride, const void* k_cache, const void* v_cache,
    const int* block_table, int max_blocks, const void* pk, const void* pv, const int* ptable,
    int pmax_blocks, int pool, int most, float cap, const int* q_start, const int* ctx_lens,
    const int* token_req, void* out, int first_token, int n_tokens, int num_heads, int num_kv_heads,
    int hd, int page_size, float scale, int window, int vd, const float* sinks, void* stream) {
    if (n_tokens == 0) return 0;
    if (pooled_check("paged_attention_pooled", num_heads, num_kv_heads, hd, vd, page_size, window, pool,
                     most, pk, pv, ptable, dtype))
        return 1;
    const int wpb = 4;
    const long long warps = (long long)n_tokens * num_heads;
    const long long blocks = (warps + wpb - 1) / wpb;
    if (blocks > 0x7fffffffLL) RV_FAIL("paged_attention_pooled: too many rows");
    const size_t smem = (size_t)wpb * hd * sizeof(float);
    const RvPooled pl = {pk, pv, ptable, pmax_blocks, pool, most, cap, 0};
    RV_DISPATCH_DTYPE(dtype, "paged_attention_pooled",
        RV_DISPATCH_DPL(vd, (rv_launch(paged_attention_warp_kernel<T, DPL, true>, dim3((int)blocks),
            dim3(wpb * 32), smem, (cudaStream_t)stream, (const T*)q, q_stride, (const T*)k_cache,
            (const T*)v_cache, block_table, max_blocks, q_start, ctx_lens, token_req, (T*)out,
            first_token, n_tokens, num_heads, num_kv_heads, hd, page_size, scale, window, vd, sinks, pl))));
    RV_CHECK_LAUNCH("paged_attention_pooled");
    return 0;
}

// The merge of split results in the layout above (this file's kernel or attention_mma.cu's).
extern "C" int rv_paged_attention_pooled_merge(const void* scratch, const int* ctx_lens, void* out,
                                               int dtype, int n_reqs, int max_ctx_len, int num_heads,
                                               int hd, int window, int pool, int most,
                                               const float* sinks, void* stream) {
    if (n_reqs == 0) return 0;
    const int psplits = rv_pooled_psplits(max_ctx_len, window, pool, most, RV_ATTN_SPLIT);
    const int max_splits = psplits + rv_pooled_tsplits(max_ctx_len, window, RV_ATTN_SPLIT);
    const size_t slots = (size_t)n_reqs * num_heads * max_splits;
    const float* part_o = (const float*)scratch;
    const float2* part_ml = (const float2*)((const char*)scratch + part_bytes(slots, hd));
    RV_DISPATCH_DTYPE(dtype, "paged_attention_pooled_merge",
        (rv_launch(paged_attention_merge_kernel<T, true>, dim3(num_heads, n_reqs), dim3(merge_threads(hd)),
            0, (cudaStream_t)stream, part_o, part_ml, ctx_lens, (T*)out, max_splits, num_heads, hd,
            window, RV_ATTN_SPLIT, sinks, psplits, pool, most)));
    RV_CHECK_LAUNCH("paged_attention_pooled_merge");
    return 0;
}

// Requests [0, n_reqs) bring one token each: splits, then the merge.
extern "C" int rv_paged_attention_pooled_decode(
    const void* q, int dtype, int q_stride, const void* k_cache, const void* v_cache,
    const int* block_table, int max_blocks, const void* pk, const void* pv, const int* ptable,
    int pmax_blocks, int pool, int most, float cap, const int* ctx_lens, void* out, void* scratch,
    long long scratch_bytes, int n_reqs, int max_ctx_len, int num_heads, int num_kv_heads, int hd,
    int page_size, float scale, int window, int vd, const float* sinks, void* stream) {
    if (n_reqs == 0) return 0;
    if (pooled_check("paged_attention_pooled_decode", num_heads, num_kv_heads, hd, vd, page_size, window,
                     pool, most, pk, pv, ptable, dtype))
        return 1;
    const int psplits = rv_pooled_psplits(max_ctx_len, window, pool, most, RV_ATTN_SPLIT);
    const int max_splits = psplits + rv_pooled_tsplits(max_ctx_len, window, RV_ATTN_SPLIT);
    if (rv_paged_attention_pooled_scratch_bytes(n_reqs, num_heads, vd, max_ctx_len, window, pool, most) >
        scratch_bytes)
        RV_FAIL("paged_attention_pooled_decode: scratch of %lld bytes is too small", scratch_bytes);
    if (n_reqs > 65535 || max_splits > 65535) RV_FAIL("paged_attention_pooled_decode: batch too large");
    const size_t slots = (size_t)n_reqs * num_heads * max_splits;
    float* part_o = (float*)scratch;
    float2* part_ml = (float2*)((char*)scratch + part_bytes(slots, vd));
    const int G = num_heads / num_kv_heads;
    const int tiles = (G + RV_ATTN_GT - 1) / RV_ATTN_GT;
    const size_t smem = (size_t)(RV_ATTN_GT * hd + 4 * 32 * RV_ATTN_GT + 4 * 32 +
                                 4 * RV_ATTN_GT * (vd + 2)) * sizeof(float);
    const RvPooled pl = {pk, pv, ptable, pmax_blocks, pool, most, cap, psplits};
    RV_DISPATCH_DTYPE(dtype, "paged_attention_pooled_decode",
        RV_DISPATCH_DPL(vd, (rv_launch(paged_attention_decode_kernel<T, DPL, true>,
            dim3(num_kv_heads * tiles, n_reqs, max_splits), dim3(128), smem, (cudaStream_t)stream,
            (const T*)q, q_stride, (const T*)k_cache, (const T*)v_cache, block_table, max_blocks,
            ctx_lens, part_o, part_ml, max_splits, num_heads, num_kv_heads, hd, page_size, scale,
            window, vd, pl))));
    RV_CHECK_LAUNCH("paged_attention_pooled_decode");
    return rv_paged_attention_pooled_merge(scratch, ctx_lens, out, dtype, n_reqs, max_ctx_len, num_heads,
                                           vd, window, pool, most, sinks, stream);
}
