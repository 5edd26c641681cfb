// One row per block of `pool` tokens: the means of the block's cached keys and values.
// A token that completes a block has the block's slot in `slots` (-1: it completes none); the
// tokens' rows are read from their pages, those of this step and of earlier ones alike, and added in
// the order of their positions in float32, so a block's row does not depend on how its tokens
// were cut into steps.  Block (token, part of the row), a thread per element.
// Plain reference: tests/plain_ops.py pool_rows.
#include "common.cuh"

template <typename T>
__global__ void pool_rows_kernel(const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                                 const int* __restrict__ block_table, int max_blocks, int page_size,
                                 const int* __restrict__ token_req, const int* __restrict__ positions,
                                 const int* __restrict__ slots, int pool, T* __restrict__ k_out,
                                 T* __restrict__ v_out, int width) {
    rv_pdl_launch_dependents();
    const int t = blockIdx.x;
    const int slot = slots[t];
    const int p1 = positions[t];                     // the block's last position
    const int* table = block_table + (size_t)token_req[t] * max_blocks;
    rv_pdl_wait();                                   // also where nothing is to be done
    if (slot < 0) return;
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < 2 * width; i += gridDim.y * blockDim.x) {
        const T* src = i < width ? k_cache + i : v_cache + (i - width);
        float sum = 0.f;
#pragma unroll 8
        for (int j = max(0, p1 - pool + 1); j <= p1; ++j) {
            const int page = table[j / page_size];
            if (page >= 0) sum += rv_load(src + ((size_t)page * page_size + j % page_size) * width);
        }
        rv_store((i < width ? k_out + i : v_out + (i - width)) + (size_t)slot * width, sum / (float)pool);
    }
}

extern "C" int rv_pool_rows(const void* k_cache, const void* v_cache, int dtype, const int* block_table,
                            int max_blocks, int page_size, const int* token_req, const int* positions,
                            const int* slots, int pool, void* k_out, void* v_out, int n_tokens, int width,
                            void* stream) {
    if (n_tokens == 0) return 0;
    if (n_tokens < 0 || pool < 1 || width < 1 || page_size < 1) RV_FAIL("pool_rows: bad sizes");
    const int parts = (2 * width + 127) / 128;
    RV_DISPATCH_DTYPE(dtype, "pool_rows",
                      (rv_launch(pool_rows_kernel<T>, dim3(n_tokens, parts < 8 ? parts : 8), dim3(128), 0,
                                 (cudaStream_t)stream, (const T*)k_cache, (const T*)v_cache, block_table,
                                 max_blocks, page_size, token_req, positions, slots, pool, (T*)k_out,
                                 (T*)v_out, width)));
    RV_CHECK_LAUNCH("pool_rows");
    return 0;
}
