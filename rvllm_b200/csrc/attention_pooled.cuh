// What attention over a window of tokens and the pooled blocks before it needs beyond plain paged
// attention; shared by the float32-arithmetic kernels (attention_simt.cu) and the tensor-core
// kernels (attention_mma.cu).
//
// The query at position p sees the tokens j with p - window < j <= p and the pooled blocks
// b < rv_seen_blocks(p): stretches of `pool` tokens that have left the window whole.  A block's key
// and value are rows of page tensors of their own with a block table of their own.  Scores may be
// capped, cap * tanh(score / cap).  `most` bounds the blocks a query sees to the first so many: with
// blocks of one token, whose rows are the tokens' own pages, these are first tokens that stay
// visible before the window for good.
//
// Split form (one token a request): splits [0, psplits) cover the blocks, 256 rows each, counted
// from block 0; the others cover the tokens, 256 positions each, in stretches aligned to absolute
// position 0 and counted from the stretch that holds the window's first token.  psplits depends on
// the launch's longest context only, so every kernel of a launch agrees on it.
#pragma once

struct RvPooled {
    const void* k;              // [pages, page_size, kv heads, hd]: one row per block
    const void* v;
    const int* table;           // [requests, max_blocks]
    int max_blocks;
    int pool;                   // tokens a block; 0: no pooled blocks
    int most;                   // 0: no bound on the blocks seen
    float cap;                  // 0: scores are not capped
    int psplits;                // split form: splits that cover blocks
};

__host__ __device__ __forceinline__ int rv_seen_blocks(int p, int window, int pool, int most) {
    const int n = pool > 0 && p - window + 1 > 0 ? (p - window + 1) / pool : 0;
    return most > 0 && n > most ? most : n;
}
// Splits of 256 rows that a launch needs for contexts of up to max_ctx tokens.
static inline int rv_pooled_psplits(int max_ctx, int window, int pool, int most, int split) {
    return (rv_seen_blocks(max_ctx - 1, window, pool, most) + split - 1) / split;
}
static inline int rv_pooled_tsplits(int max_ctx, int window, int split) {
    int n = (max_ctx + split - 1) / split;
    if (n < 1) n = 1;
    if (window > 0 && n > (window - 1) / split + 2) n = (window - 1) / split + 2;
    return n;
}
