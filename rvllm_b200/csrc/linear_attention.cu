// Linear attention with decay: per head a float32 matrix S [d, dv] that starts at zero,
//
//     S <- diag(a_t) S + k_t v_t^T;   o_t = S^T q_t
//     y = o / sqrt(mean(o^2) + eps) * w * gate(g)          the mean over all heads or per head
//
// The decay a_t is a constant per head (log_decay [H]), or made by the token for every key channel,
// log a = logsigmoid(z + bias) / tau, or made by the token for every head (state_space.cuh, whose
// keys and queries are shared by groups of heads and whose keys are weighed by a step size).  q, k
// and v may pass silu; q is multiplied by q_scale.
//
// rows [N, stride] of the compute type: q [H d] | k [H d] | v [H dv] | g [H dv]; z [N, H d] float32.
// A request's record: [H][d][dv] float32.  Everything after the projections is float32, but that an
// activated q, k or v of bfloat16 rows is rounded to bfloat16 again, in every path alike, so
// that the tensor cores can take it (below).
//
// Requests [0, n_decode) bring one token each: la_token reads and writes every state element
// once.  The others' portions are cut into chunks of 64 tokens, counted from the portion's
// start, and a chunk is a few small matrix products instead of 64 dependent steps.  With B_i the
// sum of the log decays of the chunk's tokens 0..i and L its last token:
//
//   state  block per (chunk, head, 64 x 64 tile):   KV = sum_j (k_j e^(B_L - B_j)) v_j^T
//   scan   thread per state element: over the chunks of a request one after another, the state
//          before the chunk replaces KV, S <- e^(B_L) S + KV; the last one is the record
//   out    block per (chunk, head, 64 columns):
//          o_i = sum_(j <= i) <q_i, e^(B_i - B_j) k_j> v_j + S^T (q_i e^(B_i))
//
// No factor is ever above 1, however strong the decays are, so nothing overflows and what underflows
// is nothing: with decays by channel, the tokens of a chunk form eight groups of eight, a pair
// of tokens in different groups I > J splits its factor into e^(B_i - B_(before I)) on q,
// e^(B_(before I) - B_(end of J)) from a table, and e^(B_(end of J) - B_j) on k; a pair inside a
// group takes the exponential of its own difference for every channel.
//   finish  the norm, weight and gate.
//
// bfloat16 rows with d and dv in multiples of 16 (d up to 128) take the tensor-core forms of `state`
// and `out` (with decays by channel, after a kernel that leaves the sums B where z was).  Their float32 operands (the state, the scores, everything multiplied by a decay) go
// through the bfloat16 product without being rounded: x = x1 + x2 + x3, each part the
// bfloat16 nearest to what is left, holds all 24 bits, so x times a bfloat16 is three exact
// products added in float32, and a product of two such sums is the six of its nine products that
// reach a float32's last bits.  There a chunk's pairs take q_i e^(B_i) and k_j e^(-B_j), as long
// as no channel's B_L lies below -40 (then no factor leaves float32's range by far); a chunk with a
// stronger decay takes the exponential of every pair's own difference instead.
// Plain reference: tests/plain_ops.py linear_attention.
#include "common.cuh"
#include "mma_bf16.cuh"
#include "chunks.cuh"

#define LA_T 64             // columns (and rows) of a tile
#define LA_DK 32            // key channels staged at a time in `out`
#define LA_LD 68            // padded row of 64
#define LA_G 8              // tokens a group
#define LA_SCAN_THREADS 64
#define LA_NG 8             // groups a chunk

// how decays are made
#define LA_CONST 0          // a constant per head
#define LA_CHANNEL 1        // by the token, per key channel
#define LA_TOKEN 2          // by the token, per head

// Where a token's row holds q, k and v, and how many heads share a query and key head.
struct LaRows {
    int q, k, v, share;
};
// LA_TOKEN, for tokens of portions: B [n, H], the sum of the log decays of the chunk's tokens up to
// and with this one (float64: differences of sums that large decays have made large stay exact
// enough), and the keys' weights w [n, H].
struct LaToken {
    const double* B;
    const float* w;
};
__device__ __forceinline__ float la_logsigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float la_silu(float x) { return __fdividef(x, 1.f + __expf(-x)); }
// a projection as the recurrence reads it
__device__ __forceinline__ float la_in(const float* p, int act) { return act ? *p / (1.f + expf(-*p)) : *p; }
__device__ __forceinline__ float la_in(const bf16* p, int act) {
    const float x = __bfloat162float(*p);
    return act ? __bfloat162float(__float2bfloat16_rn(la_silu(x))) : x;
}

// ---- single tokens ---------------------------------------------------------------------
// V = 4: 16-byte accesses to the state and sixteen lanes across a tile's 64 columns; V = 1: 64.
// LA_TOKEN: z [n, z_stride] holds the step sizes' pre-activations per head, bias [H] is theirs,
// log_decay [H] the rates' logarithms (state_space.cuh).
template <typename T, int V, bool TOKEN>
__global__ void __launch_bounds__(128) la_token_kernel(
    const T* __restrict__ rows, int stride, const LaRows lr, const float* __restrict__ z, int z_stride,
    const float* __restrict__ log_decay,
    const float* __restrict__ bias, float tau, const int* __restrict__ q_start,
    const int* __restrict__ state_slot, float* __restrict__ state, float* __restrict__ num, int H,
    int d, int dv, int act, float q_scale) {
    rv_pdl_launch_dependents();
    constexpr int LANES = LA_T / V, RG = 128 / LANES;            // row groups
    extern __shared__ float sm[];
    float* qs = sm;                                              // [d]
    float* ks = qs + d;
    float* as = ks + d;
    float* red = as + d;                                         // [RG][64]
    const int h = blockIdx.y, r = blockIdx.z;
    const int slot = state_slot[r];
    const int t = q_start[r];
    rv_pdl_wait();
    if (slot < 0) return;
    const T* row = rows + (size_t)t * stride;
    float ad = log_decay ? expf(log_decay[h]) : 0.f, wk = 1.f;
    if (TOKEN) {
        wk = la_softplus(z[(size_t)t * z_stride + h] + bias[h]);
        ad = expf(-ad * wk);
    }
    const int kh = h / lr.share;
    for (int i = threadIdx.x; i < d; i += 128) {
        qs[i] = la_in(row + lr.q + kh * d + i, act);
        const float k = la_in(row + lr.k + kh * d + i, act);
        ks[i] = TOKEN ? k * wk : k;
        as[i] = log_decay ? ad : expf(la_logsigmoid(z[(size_t)t * H * d + h * d + i] + bias[h * d + i]) / tau);
    }
    const int cl = threadIdx.x % LANES, rg = threadIdx.x / LANES;
    const int col = blockIdx.x * LA_T + cl * V;
    float v[V], o[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
        o[e] = 0.f;
        v[e] = col + e < dv ? la_in(row + lr.v + h * dv + col + e, act) : 0.f;
    }
    __syncthreads();
    float* S = state + ((size_t)slot * H + h) * d * dv;
    if (col < dv) {
#pragma unroll 8
        for (int i = rg; i < d; i += RG) {
            const float a = as[i], k = ks[i], q = qs[i];
            float* p = S + (size_t)i * dv + col;
            if (V == 4) {
                float4 s = *(float4*)p;
                s.x = fmaf(a, s.x, k * v[0]);
                s.y = fmaf(a, s.y, k * v[1 % V]);
                s.z = fmaf(a, s.z, k * v[2 % V]);
                s.w = fmaf(a, s.w, k * v[3 % V]);
                o[0] = fmaf(s.x, q, o[0]);
                o[1 % V] = fmaf(s.y, q, o[1 % V]);
                o[2 % V] = fmaf(s.z, q, o[2 % V]);
                o[3 % V] = fmaf(s.w, q, o[3 % V]);
                *(float4*)p = s;
            } else {
                const float s = fmaf(a, *p, k * v[0]);
                o[0] = fmaf(s, q, o[0]);
                *p = s;
            }
        }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) red[rg * LA_T + cl * V + e] = o[e];
    __syncthreads();
    for (int c = threadIdx.x; c < LA_T; c += 128) {
        if (blockIdx.x * LA_T + c >= dv) break;
        float s = 0.f;
#pragma unroll
        for (int g = 0; g < RG; ++g) s += red[g * LA_T + c];
        num[((size_t)t * H + h) * dv + blockIdx.x * LA_T + c] = s * q_scale;
    }
}

// ---- portions: every chunk's own contribution to the state ----------------------------------
template <typename T, int MODE>
__global__ void __launch_bounds__(256) la_state_kernel(
    const T* __restrict__ rows, int stride, const LaRows lr, const LaToken tk, const float* __restrict__ zr,
    const float* __restrict__ log_decay,
    const float* __restrict__ bias, float tau, const int* __restrict__ q_start,
    const int* __restrict__ state_slot, int first_req, int n_reqs, float* __restrict__ kv,
    float* __restrict__ dec, int H, int d, int dv, int act) {
    constexpr bool CHANNEL = MODE == LA_CHANNEL, TOKEN = MODE == LA_TOKEN;
    rv_pdl_launch_dependents();
    extern __shared__ __align__(16) float sm[];
    float* ks = sm;                                              // [64 tokens][LD]: channels
    float* vs = ks + LA_C * LA_LD;                               // [64 tokens][LD]: columns
    float* lb = vs + LA_C * LA_LD;                               // [64 tokens][LD] (CHANNEL)
    float* tot = lb + (CHANNEL ? LA_C * LA_LD : 0);              // [4][64] segments' sums
    __shared__ int at[2];
    const int tid = threadIdx.x, lane = tid & 31;
    const int item = blockIdx.x, h = blockIdx.y;
    const int tiles_v = (dv + LA_T - 1) / LA_T;
    const int d0 = (blockIdx.z / tiles_v) * LA_T, v0 = (blockIdx.z % tiles_v) * LA_T;
    if (tid < 32) {
        int r = -1, before = 0;
        const bool ok = la_find(q_start, state_slot, first_req, n_reqs, item, lane, r, before);
        if (lane == 0) {
            at[0] = ok ? q_start[r] + (item - before) * LA_C : -1;
            at[1] = ok ? min(LA_C, q_start[r + 1] - at[0]) : 0;
        }
    }
    __syncthreads();
    const int t0 = at[0], L = at[1];
    rv_pdl_wait();
    if (t0 < 0) return;
    const int x = tid & 63, y = tid >> 6;
    const int dn = min(LA_T, d - d0), vn = min(LA_T, dv - v0);
    const T* base = rows + (size_t)t0 * stride;
    const float ld = MODE != LA_CONST ? 0.f : log_decay[h];
    const float bz = CHANNEL && x < dn ? bias[h * d + d0 + x] : 0.f;
    const int kh = h / lr.share;
    const double last = TOKEN ? tk.B[(size_t)(t0 + L - 1) * H + h] : 0.;
    // four values of one column at a time are requested before any is worked on
#pragma unroll 4
    for (int j = y; j < LA_C; j += 4) {
        const T* row = base + (size_t)j * stride;
        const bool tj = j < L;
        float k = tj && x < dn ? la_in(row + lr.k + kh * d + d0 + x, act) : 0.f;
        const float v = tj && x < vn ? la_in(row + lr.v + h * dv + v0 + x, act) : 0.f;
        if (MODE == LA_CONST) k *= expf(ld * (float)(L - 1 - min(j, L - 1)));
        if (TOKEN) {
            const size_t at_j = (size_t)(t0 + min(j, L - 1)) * H + h;
            k *= expf((float)(last - tk.B[at_j])) * tk.w[at_j];
        }
        ks[j * LA_LD + x] = k;
        vs[j * LA_LD + x] = v;
        if (CHANNEL) {
            const float z = tj && x < dn ? zr[(size_t)(t0 + j) * H * d + h * d + d0 + x] : 0.f;
            lb[j * LA_LD + x] = tj && x < dn ? la_logsigmoid(z + bz) / tau : 0.f;
        }
    }
    if (CHANNEL) {
        __syncthreads();
        float s = 0.f;                                           // tokens 16 y .. 16 y + 15
#pragma unroll
        for (int j = 0; j < 16; ++j) {
            s += lb[(16 * y + j) * LA_LD + x];
            lb[(16 * y + j) * LA_LD + x] = s;
        }
        tot[y * 64 + x] = s;
        __syncthreads();
        float after = 0.f;                                       // the segments behind this one
        for (int g = y + 1; g < 4; ++g) after += tot[g * 64 + x];
#pragma unroll
        for (int j = 0; j < 16; ++j)
            ks[(16 * y + j) * LA_LD + x] *= expf(after + (s - lb[(16 * y + j) * LA_LD + x]));
        if (y == 0 && v0 == 0 && x < dn)
            dec[((size_t)item * H + h) * d + d0 + x] = expf(after + s);
    }
    __syncthreads();
    const int ty = tid >> 4, tx = tid & 15;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    const int jn = (L + 3) & ~3;                                 // zeros beyond L
#pragma unroll 4
    for (int j = 0; j < jn; ++j) {
        const float4 a = *(const float4*)(ks + j * LA_LD + 4 * ty), b = *(const float4*)(vs + j * LA_LD + 4 * tx);
        const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[i][e] = fmaf(av[i], bv[e], acc[i][e]);
    }
    float* o = kv + ((size_t)item * H + h) * d * dv;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int dd = 4 * ty + i;
        if (dd >= dn) continue;
        float* p = o + (size_t)(d0 + dd) * dv + v0 + 4 * tx;
        if (dv % 4 == 0) {
            if (4 * tx < vn) *(float4*)p = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (4 * tx + e < vn) p[e] = acc[i][e];
        }
    }
}

// ---- portions: the states between the chunks ---------------------------------------------------
template <int MODE, int V>
__global__ void __launch_bounds__(LA_SCAN_THREADS) la_scan_kernel(
    const float* __restrict__ log_decay, const int* __restrict__ q_start,
    const int* __restrict__ state_slot, int first_req, float* __restrict__ kv,
    const float* __restrict__ dec, float* __restrict__ state, int H, int d, int dv) {
    constexpr bool CHANNEL = MODE == LA_CHANNEL, MADE = MODE != LA_CONST;
    rv_pdl_launch_dependents();
    const int h = blockIdx.y, r = first_req + blockIdx.z;
    const int slot = state_slot[r];
    const int n = slot < 0 ? 0 : (q_start[r + 1] - q_start[r] + LA_C - 1) / LA_C;
    __shared__ int first_item;
    if (threadIdx.x < 32) {
        int before = 0;
        for (int b = first_req + threadIdx.x; b < r; b += 32) before += la_chunks(q_start, state_slot, b);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
        if (threadIdx.x == 0) first_item = before;
    }
    __syncthreads();
    const int last_len = q_start[r + 1] - q_start[r] - (n - 1) * LA_C;
    const float ld = MADE ? 0.f : log_decay[h];
    rv_pdl_wait();
    const long long el = ((long long)blockIdx.x * LA_SCAN_THREADS + threadIdx.x) * V;
    if (n == 0 || el >= (long long)d * dv) return;
    const int ch = (int)(el / dv);
    float* rec = state + ((size_t)slot * H + h) * d * dv + el;
    float* p = kv + ((size_t)first_item * H + h) * d * dv + el;
    const float* dp = CHANNEL ? dec + ((size_t)first_item * H + h) * d + ch
                              : MADE ? dec + (size_t)first_item * H + h : nullptr;
    const size_t step = (size_t)H * d * dv, dstep = CHANNEL ? (size_t)H * d : (size_t)H;
    const float full = MADE ? 0.f : expf(ld * (float)LA_C), rest = MADE ? 0.f : expf(ld * (float)last_len);
    float S[V];
#pragma unroll
    for (int e = 0; e < V; ++e) S[e] = 0.f;
    if (V == 4) {
        const float4 s = *(const float4*)rec;
        S[0] = s.x; S[1 % V] = s.y; S[2 % V] = s.z; S[3 % V] = s.w;
    } else {
        S[0] = *rec;
    }
    constexpr int U = 8;                                         // chunks requested together
    for (int c0 = 0; c0 < n; c0 += U) {
        float in[U][V], a[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (c0 + u >= n) continue;
            const float* s = p + (size_t)(c0 + u) * step;
            if (V == 4) {
                const float4 f = *(const float4*)s;
                in[u][0] = f.x; in[u][1 % V] = f.y; in[u][2 % V] = f.z; in[u][3 % V] = f.w;
            } else {
                in[u][0] = *s;
            }
            a[u] = MADE ? dp[(size_t)(c0 + u) * dstep] : (c0 + u == n - 1 ? rest : full);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (c0 + u >= n) continue;
            float* s = p + (size_t)(c0 + u) * step;
            if (V == 4) *(float4*)s = make_float4(S[0], S[1 % V], S[2 % V], S[3 % V]);
            else *s = S[0];
#pragma unroll
            for (int e = 0; e < V; ++e) S[e] = fmaf(a[u], S[e], in[u][e]);
        }
    }
    if (V == 4) *(float4*)rec = make_float4(S[0], S[1 % V], S[2 % V], S[3 % V]);
    else *rec = S[0];
}

// ---- portions: the outputs -------------------------------------------------------------------
// A thread's share of a 64 x 64 product is rows 4 ty .. + 3 by columns 4 tx .. + 3; a warp's eight
// rows are one group.  Operands lie with the summed index first ([c][64 tokens] and so on), so that
// a thread reads four of its rows and four of its columns with one access each.
template <typename T, int MODE>
__global__ void __launch_bounds__(256) la_out_kernel(
    const T* __restrict__ rows, int stride, const LaRows lr, const LaToken tk, const float* __restrict__ zr,
    const float* __restrict__ log_decay,
    const float* __restrict__ bias, float tau, const int* __restrict__ q_start,
    const int* __restrict__ state_slot, int first_req, int n_reqs, const float* __restrict__ kv,
    float* __restrict__ num, int H, int d, int dv, int act, float q_scale) {
    constexpr bool CHANNEL = MODE == LA_CHANNEL, TOKEN = MODE == LA_TOKEN;
    rv_pdl_launch_dependents();
    extern __shared__ __align__(16) float sm[];
    __shared__ double bt[TOKEN ? LA_C : 1];         // TOKEN: B and the keys' weights
    __shared__ float wt[TOKEN ? LA_C : 1];
    constexpr int SL = LA_DK * LA_LD;
    float* qt = sm;                                 // [DK][LD]: q e^(B_i - B before its group)
    float* kt = qt + SL;                            // [DK][LD]: k e^(B at its group's end - B_j)
    float* ss = kt + SL;                            // [DK][LD]: the state's rows, 64 columns
    float* ps = ss + SL;                            // [64 j][LD i]: scores
    float* vs = ps + LA_C * LA_LD;                  // [64 j][LD]: values
    float* qr = vs + LA_C * LA_LD;                  // CHANNEL: [DK][LD] q as it is
    float* kr = qr + (CHANNEL ? SL : 0);            //          [DK][LD] k as it is
    float* lb = kr + (CHANNEL ? SL : 0);            //          [DK][LD] B_i - B before its group
    float* off = lb + (CHANNEL ? SL : 0);           //          [NG + 1][DK + 1] B before a group
    float* tab = off + (CHANNEL ? (LA_NG + 1) * (LA_DK + 1) : 0);   // [NG][NG][DK + 1]
    __shared__ int at[2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int item = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * LA_T;
    if (tid < 32) {
        int r = -1, before = 0;
        const bool ok = la_find(q_start, state_slot, first_req, n_reqs, item, lane, r, before);
        if (lane == 0) {
            at[0] = ok ? q_start[r] + (item - before) * LA_C : -1;
            at[1] = ok ? min(LA_C, q_start[r + 1] - at[0]) : 0;
        }
    }
    __syncthreads();
    const int t0 = at[0], L = at[1];
    rv_pdl_wait();
    if (t0 < 0) return;
    const T* base = rows + (size_t)t0 * stride;
    const float* Sg = kv + ((size_t)item * H + h) * d * dv;
    const int vn = min(LA_T, dv - v0);
    const int ty = tid >> 4, tx = tid & 15;
    const float ld = MODE != LA_CONST ? 0.f : log_decay[h];
    const int kh = h / lr.share;
    if (TOKEN && tid < LA_C) {
        const size_t at_j = (size_t)(t0 + min(tid, L - 1)) * H + h;
        bt[tid] = tk.B[at_j];
        wt[tid] = tid < L ? tk.w[at_j] : 0.f;
    }
    // values [64 tokens][64 columns]
    {
        const int x = tid & 63, y = tid >> 6;
#pragma unroll 4
        for (int j = y; j < LA_C; j += 4)
            vs[j * LA_LD + x] = j < L && x < vn ? la_in(base + (size_t)j * stride + lr.v + h * dv + v0 + x, act) : 0.f;
    }
    float p[4][4], o[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) p[i][j] = o[i][j] = 0.f;
    // CHANNEL: the pairs (i, j < i) and (i, i) inside groups, 8 x 36 of them, over the threads
    float inner[2] = {0.f, 0.f};
    int pi[2], pj[2];
    if (CHANNEL) {
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int n = tid + 256 * u;            // pair n % 36 of group n / 36
            int a = 0, b = n % 36;
            while (b > a) b -= ++a;                 // row a has a + 1 pairs
            pi[u] = n < 36 * LA_NG ? (n / 36) * LA_G + a : -1;
            pj[u] = (n / 36) * LA_G + b;
        }
    }
    const int I = ty >> 1;                          // the group of this thread's rows
    const int J = tx >> 1;                          // and of its columns
    for (int c0 = 0; c0 < d; c0 += LA_DK) {
        const int cn = min(LA_DK, d - c0);
        __syncthreads();                            // the slice before has been used
        // four tokens by eight channels a warp and access: whole 32-byte pieces of the rows, and
        // 32 different banks of the transposed slice
        {
            const int tl = lane & 3, cl = lane >> 2;
#pragma unroll 4
            for (int u = warp; u < (LA_C / 4) * (LA_DK / 8); u += 8) {
                const int j = (u >> 2) * 4 + tl, c = (u & 3) * 8 + cl;
                const bool in = j < L && c < cn;
                const T* row = base + (size_t)j * stride + kh * d + c0 + c;
                const float q = in ? la_in(row + lr.q, act) : 0.f;
                const float k = in ? la_in(row + lr.k, act) : 0.f;
                if (CHANNEL) {
                    qr[c * LA_LD + j] = q;
                    kr[c * LA_LD + j] = k;
                    lb[c * LA_LD + j] = in ? la_logsigmoid(zr[(size_t)(t0 + j) * H * d + h * d + c0 + c] + bias[h * d + c0 + c]) / tau : 0.f;
                } else {
                    qt[c * LA_LD + j] = q;
                    kt[c * LA_LD + j] = k;
                }
            }
            const int x = tid & 63, y = tid >> 6;
#pragma unroll 4
            for (int c = y; c < LA_DK; c += 4)
                ss[c * LA_LD + x] = c < cn && x < vn ? Sg[(size_t)(c0 + c) * dv + v0 + x] : 0.f;
        }
        if (CHANNEL) {
            __syncthreads();
            {
                // sums inside the groups: thread (channel, group), then the groups' sums before
                const int c = tid >> 3, g = tid & 7;
                float s = 0.f, cum[LA_G];
#pragma unroll
                for (int j = 0; j < LA_G; ++j) {
                    s += lb[c * LA_LD + g * LA_G + j];
                    cum[j] = s;
                }
                float incl = s;
#pragma unroll
                for (int w = 1; w < LA_NG; w <<= 1) {
                    const float up = __shfl_up_sync(0xffffffffu, incl, w, LA_NG);
                    if (g >= w) incl += up;
                }
                // the same sums for whoever asks: B before group g is the sum of the totals before
                off[(g + 1) * (LA_DK + 1) + c] = incl;
                if (g == 0) off[c] = 0.f;
#pragma unroll
                for (int j = 0; j < LA_G; ++j) {
                    const int e = c * LA_LD + g * LA_G + j;
                    lb[e] = cum[j];
                    qt[e] = qr[e] * expf(cum[j]);
                    kt[e] = kr[e] * expf(s - cum[j]);
                }
            }
            __syncthreads();
            // tab[I][J + 1][c] = e^(B before I - B at the end of J), J < I; J = -1: the chunk's start
            for (int n = tid; n < LA_NG * LA_NG * LA_DK; n += 256) {
                const int c = n & (LA_DK - 1), jj = (n / LA_DK) & (LA_NG - 1), ii = n / (LA_DK * LA_NG);
                if (jj <= ii)
                    tab[(ii * LA_NG + jj) * (LA_DK + 1) + c] =
                        expf(off[ii * (LA_DK + 1) + c] - off[jj * (LA_DK + 1) + c]);
            }
#pragma unroll
            for (int u = 0; u < 2; ++u)
                if (pi[u] >= 0) {
                    float s = 0.f;
#pragma unroll 4
                    for (int c = 0; c < cn; ++c)
                        s = fmaf(qr[c * LA_LD + pi[u]] * kr[c * LA_LD + pj[u]],
                                 expf(lb[c * LA_LD + pi[u]] - lb[c * LA_LD + pj[u]]), s);
                    inner[u] += s;
                }
        }
        __syncthreads();
        const float* tij = tab + (I * LA_NG + (J < I ? J + 1 : 0)) * (LA_DK + 1);
        const float* ti0 = tab + I * LA_NG * (LA_DK + 1);
#pragma unroll 4
        for (int c = 0; c < cn; ++c) {
            const float4 a = *(const float4*)(qt + c * LA_LD + 4 * ty), b = *(const float4*)(kt + c * LA_LD + 4 * tx),
                         w = *(const float4*)(ss + c * LA_LD + 4 * tx);
            const float av[4] = {a.x, a.y, a.z, a.w};
            float bv[4] = {b.x, b.y, b.z, b.w}, wv[4] = {w.x, w.y, w.z, w.w};
            if (CHANNEL) {
                const float f = tij[c], f0 = ti0[c];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    bv[e] *= f;
                    wv[e] *= f0;
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    p[i][e] = fmaf(av[i], bv[e], p[i][e]);
                    o[i][e] = fmaf(av[i], wv[e], o[i][e]);
                }
        }
    }
    // scores to shared memory, transposed; zeros above the diagonal
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int ri = 4 * ty + i;
        float row_f = 1.f;
        if (MODE == LA_CONST) row_f = expf(ld * (float)(ri + 1));
        if (TOKEN) row_f = expf((float)bt[ri]);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int cj = 4 * tx + e;
            if (CHANNEL) {
                if (J < I) ps[cj * LA_LD + ri] = p[i][e];
                else if (J > I) ps[cj * LA_LD + ri] = 0.f;
                else if (cj > ri) ps[cj * LA_LD + ri] = 0.f;     // inside a group: the pairs below
            } else {
                const float f = TOKEN ? (cj <= ri ? expf((float)(bt[ri] - bt[cj])) * wt[cj] : 0.f)
                                      : expf(ld * (float)(ri - cj));
                ps[cj * LA_LD + ri] = cj <= ri ? p[i][e] * f : 0.f;
                o[i][e] *= row_f;
            }
        }
    }
    if (CHANNEL) {
#pragma unroll
        for (int u = 0; u < 2; ++u)
            if (pi[u] >= 0) ps[pj[u] * LA_LD + pi[u]] = inner[u];
    }
    __syncthreads();
    // a warp's rows end with its group: later values have no score
    const int jn = min((L + 3) & ~3, 8 * (I + 1));
#pragma unroll 4
    for (int j = 0; j < jn; ++j) {
        const float4 a = *(const float4*)(ps + j * LA_LD + 4 * ty), b = *(const float4*)(vs + j * LA_LD + 4 * tx);
        const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[i][e] = fmaf(av[i], bv[e], o[i][e]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int ri = 4 * ty + i;
        if (ri >= L) continue;
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] *= q_scale;
        float* dst = num + ((size_t)(t0 + ri) * H + h) * dv + v0 + 4 * tx;
        if (dv % 4 == 0) {
            if (4 * tx < vn) *(float4*)dst = make_float4(o[i][0], o[i][1], o[i][2], o[i][3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (4 * tx + e < vn) dst[e] = o[i][e];
        }
    }
}

// ---- norm, weight and gate -----------------------------------------------------------------------
__device__ __forceinline__ float la_gate(float g, int gate) {
    return (gate ? g : 1.f) / (1.f + expf(-g));                  // 0: sigmoid, 1: silu
}

template <typename T, int V>
__device__ __forceinline__ void la_finish_at(const float* nm, const T* g, const float* w, T* o, int c, float inv, int gate) {
    float x[V], y[V], z[V];
    la_load<float, V>(nm + c, x);
    la_load<T, V>(g + c, y);
    la_load<float, V>(w + c, z);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = x[e] * inv * z[e] * la_gate(y[e], gate);
    la_store<T, V>(o + c, x);
}

// One norm over all heads: a block per token.
template <typename T, int V>
__global__ void la_finish_all_kernel(const float* __restrict__ num, const T* __restrict__ rows,
                                     int stride, int g_off, const float* __restrict__ norm_w, float eps,
                                     const int* __restrict__ token_req, const int* __restrict__ state_slot,
                                     T* __restrict__ out, int width, int gate) {
    rv_pdl_launch_dependents();
    __shared__ float scratch[33];
    const int t = blockIdx.x;
    const bool pad = state_slot[token_req[t]] < 0;
    rv_pdl_wait();
    T* o = out + (size_t)t * width;
    if (pad) {
        for (int c = threadIdx.x; c < width; c += blockDim.x) rv_store(o + c, 0.f);
        return;
    }
    const float* nm = num + (size_t)t * width;
    float ss = 0.f;
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
        float x[V];
        la_load<float, V>(nm + c, x);
#pragma unroll
        for (int e = 0; e < V; ++e) ss += x[e] * x[e];
    }
    const float inv = 1.f / sqrtf(rv_block_sum(ss, scratch) / (float)width + eps);
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V)
        la_finish_at<T, V>(nm, rows + (size_t)t * stride + g_off, norm_w, o, c, inv, gate);
}

// A norm per head: a warp per (token, head).
template <typename T, int V>
__global__ void la_finish_head_kernel(const float* __restrict__ num, const T* __restrict__ rows,
                                      int stride, int g_off, const float* __restrict__ norm_w, float eps,
                                      const int* __restrict__ token_req, const int* __restrict__ state_slot,
                                      T* __restrict__ out, int n_tokens, int H, int dv, int gate) {
    rv_pdl_launch_dependents();
    const long long w = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (w >= (long long)n_tokens * H) return;
    const int t = (int)(w / H), h = (int)(w - (long long)t * H);
    const bool pad = state_slot[token_req[t]] < 0;
    rv_pdl_wait();
    T* o = out + (size_t)t * H * dv + (size_t)h * dv;
    if (pad) {
        for (int c = lane; c < dv; c += 32) rv_store(o + c, 0.f);
        return;
    }
    const float* nm = num + ((size_t)t * H + h) * dv;
    float ss = 0.f;
    for (int c = lane * V; c < dv; c += 32 * V) {
        float x[V];
        la_load<float, V>(nm + c, x);
#pragma unroll
        for (int e = 0; e < V; ++e) ss += x[e] * x[e];
    }
    const float inv = 1.f / sqrtf(rv_warp_sum(ss) / (float)dv + eps);
    for (int c = lane * V; c < dv; c += 32 * V)
        la_finish_at<T, V>(nm, rows + (size_t)t * stride + g_off + h * dv, norm_w + h * dv, o, c, inv, gate);
}

#include "linear_attention_mma.cuh"

// ---------------------------------------------------------------------------------
// Floats of scratch: num [n, H, dv]; for portions kv [items, H, d, dv] and dec [items, H, d].
extern "C" long long rv_linear_attention_scratch(int n_tokens, int n_decode, int n_reqs, int H, int d,
                                                 int dv) {
    long long f = ((long long)n_tokens * H * dv + 3) & ~3LL;
    if (n_reqs > n_decode && n_tokens > n_decode)
        f += la_items(n_tokens - n_decode, n_reqs - n_decode) * H * ((long long)d * dv + d);
    return f;
}

struct LaArgs {
    LaRows lr;
    LaToken tk;
    float* z;
    const float *log_decay, *bias, *norm_w;
    float *state, *scratch;
    const int *token_req, *q_start, *state_slot;
    float tau, q_scale, eps;
    int stride, z_stride, n_tokens, n_decode, n_reqs, H, d, dv, act, norm_head, gate, tensor;
};

#define LA_SMEM(kernel, bytes)                                                                       \
    {                                                                                                \
        static size_t have = 40 * 1024;      /* the default 48 KB hold the static arrays too */        \
        if ((bytes) > have) {                                                                        \
            if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,            \
                                     (int)(bytes)) != cudaSuccess)                                   \
                RV_FAIL("linear_attention: %zu bytes of shared memory are not to be had", (size_t)(bytes)); \
            have = (bytes);                                                                          \
        }                                                                                            \
    }

// The tensor-core forms exist for bfloat16 rows.
template <int CH>
static int la_tensor_launch(const float* rows, const LaArgs& a, int what, dim3 grid, float* kv, float* dec,
                            float* num, cudaStream_t s) {
    (void)rows; (void)a; (void)what; (void)grid; (void)kv; (void)dec; (void)num; (void)s;
    RV_FAIL("linear_attention: float32 rows on the tensor cores");
}
template <int CH>
static int la_tensor_launch(const bf16* rows, const LaArgs& a, int what, dim3 grid, float* kv, float* dec,
                            float* num, cudaStream_t s) {
    if (what == 0) {
        const size_t smem = lm_state_smem();
        LA_SMEM(la_state_mma_kernel<CH>, smem)
        rv_launch(la_state_mma_kernel<CH>, grid, dim3(128), smem, s, rows, a.stride, a.lr, a.tk, (const float*)a.z,
                  a.log_decay, a.q_start, a.state_slot, a.n_decode, a.n_reqs, kv, dec, a.H, a.d, a.dv, a.act);
    } else {
        const size_t smem = lm_out_smem(CH == LA_CHANNEL, a.d);
        LA_SMEM(la_out_mma_kernel<CH>, smem)
        rv_launch(la_out_mma_kernel<CH>, grid, dim3(128), smem, s, rows, a.stride, a.lr, a.tk, (const float*)a.z,
                  a.log_decay, a.q_start, a.state_slot, a.n_decode, a.n_reqs, (const float*)kv, num, a.H, a.d, a.dv,
                  a.act, a.q_scale);
    }
    return 0;
}

template <typename T, int CH>
static int la_portions(const T* rows, const LaArgs& a, float* num, float* kv, float* dec, unsigned items,
                       cudaStream_t s) {
    const int tiles_d = (a.d + LA_T - 1) / LA_T, tiles_v = (a.dv + LA_T - 1) / LA_T;
    const dim3 g1(items, a.H, tiles_d * tiles_v), g3(items, a.H, tiles_v);
    if (a.tensor) {
        if (CH == LA_CHANNEL) {
            const int width = a.H * a.d;
            rv_launch(la_decay_kernel, dim3(items, (width + 31) / 32), dim3(256), 0, s, a.z, a.bias,
                      1.4426950408889634f / a.tau, a.q_start, a.state_slot, a.n_decode, a.n_reqs, width);
            RV_CHECK_LAUNCH("linear_attention_decay");
        }
        if (la_tensor_launch<CH>(rows, a, 0, g1, kv, dec, num, s)) return 1;
    } else {
        const size_t smem = (size_t)((CH == LA_CHANNEL ? 3 : 2) * LA_C * LA_LD + 4 * 64) * sizeof(float);
        auto kernel = la_state_kernel<T, CH>;
        LA_SMEM(kernel, smem)
        rv_launch(kernel, g1, dim3(256), smem, s, rows, a.stride, a.lr, a.tk, a.z, a.log_decay, a.bias, a.tau, a.q_start,
                  a.state_slot, a.n_decode, a.n_reqs, kv, dec, a.H, a.d, a.dv, a.act);
    }
    RV_CHECK_LAUNCH("linear_attention_state");
    const bool v4 = a.dv % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    const long long per = LA_SCAN_THREADS * (v4 ? 4 : 1);
    const dim3 g2((unsigned)(((long long)a.d * a.dv + per - 1) / per), a.H, a.n_reqs - a.n_decode);
    if (v4)
        rv_launch(la_scan_kernel<CH, 4>, g2, dim3(LA_SCAN_THREADS), 0, s, a.log_decay, a.q_start, a.state_slot,
                  a.n_decode, kv, dec, a.state, a.H, a.d, a.dv);
    else
        rv_launch(la_scan_kernel<CH, 1>, g2, dim3(LA_SCAN_THREADS), 0, s, a.log_decay, a.q_start, a.state_slot,
                  a.n_decode, kv, dec, a.state, a.H, a.d, a.dv);
    RV_CHECK_LAUNCH("linear_attention_scan");
    if (a.tensor) {
        if (la_tensor_launch<CH>(rows, a, 1, g3, kv, dec, num, s)) return 1;
    } else {
        const size_t smem = (size_t)((CH == LA_CHANNEL ? 6 : 3) * LA_DK * LA_LD + 2 * LA_C * LA_LD +
                                     (CH == LA_CHANNEL ? (LA_NG + 1 + LA_NG * LA_NG) * (LA_DK + 1) : 0)) * sizeof(float);
        auto kernel = la_out_kernel<T, CH>;
        LA_SMEM(kernel, smem)
        rv_launch(kernel, g3, dim3(256), smem, s, rows, a.stride, a.lr, a.tk, a.z, a.log_decay, a.bias, a.tau, a.q_start,
                  a.state_slot, a.n_decode, a.n_reqs, (const float*)kv, num, a.H, a.d, a.dv, a.act, a.q_scale);
    }
    RV_CHECK_LAUNCH("linear_attention_out");
    return 0;
}

// Requests [0, n_decode): one token each.
template <typename T, bool TOKEN>
static int la_tokens(const T* rows, const LaArgs& a, float* num, cudaStream_t s) {
    const bool v4 = a.dv % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    const size_t smem = (size_t)(3 * a.d + (v4 ? 8 : 2) * LA_T) * sizeof(float);
    const dim3 grid((a.dv + LA_T - 1) / LA_T, a.H, a.n_decode);
    if (v4)
        rv_launch(la_token_kernel<T, 4, TOKEN>, grid, dim3(128), smem, s, rows, a.stride, a.lr, a.z, a.z_stride,
                  a.log_decay, a.bias, a.tau, a.q_start, a.state_slot, a.state, num, a.H, a.d, a.dv, a.act, a.q_scale);
    else
        rv_launch(la_token_kernel<T, 1, TOKEN>, grid, dim3(128), smem, s, rows, a.stride, a.lr, a.z, a.z_stride,
                  a.log_decay, a.bias, a.tau, a.q_start, a.state_slot, a.state, num, a.H, a.d, a.dv, a.act, a.q_scale);
    RV_CHECK_LAUNCH("linear_attention_token");
    return 0;
}

template <typename T>
static int la_run(const T* rows, const LaArgs& a, T* out, cudaStream_t s) {
    float* num = a.scratch;
    if (a.n_decode > 0 && la_tokens<T, false>(rows, a, num, s)) return 1;
    if (a.n_tokens > a.n_decode && a.n_reqs > a.n_decode) {
        const long long items = la_items(a.n_tokens - a.n_decode, a.n_reqs - a.n_decode);
        float* kv = a.scratch + (((size_t)a.n_tokens * a.H * a.dv + 3) & ~(size_t)3);
        float* dec = kv + (size_t)items * a.H * a.d * a.dv;
        if (items > 0x7fffffffLL) RV_FAIL("linear_attention: too many tokens");
        if (a.log_decay ? la_portions<T, LA_CONST>(rows, a, num, kv, dec, (unsigned)items, s)
                        : la_portions<T, LA_CHANNEL>(rows, a, num, kv, dec, (unsigned)items, s))
            return 1;
    }
    const int g_off = 2 * a.H * a.d + a.H * a.dv;
    // four values an access: every row, head, weight and gate begins on such a boundary
    const bool vec = a.dv % 4 == 0 && g_off % 4 == 0 && a.stride % 4 == 0 &&
                     (((uintptr_t)rows | (uintptr_t)out | (uintptr_t)a.norm_w) & 15) == 0;
    if (a.norm_head) {
        const long long blocks = ((long long)a.n_tokens * a.H + 3) / 4;
        if (blocks > 0x7fffffffLL) RV_FAIL("linear_attention: too many tokens");
        if (vec)
            rv_launch(la_finish_head_kernel<T, 4>, dim3((int)blocks), dim3(128), 0, s, (const float*)num, rows,
                      a.stride, g_off, a.norm_w, a.eps, a.token_req, a.state_slot, out, a.n_tokens, a.H, a.dv, a.gate);
        else
            rv_launch(la_finish_head_kernel<T, 1>, dim3((int)blocks), dim3(128), 0, s, (const float*)num, rows,
                      a.stride, g_off, a.norm_w, a.eps, a.token_req, a.state_slot, out, a.n_tokens, a.H, a.dv, a.gate);
    } else {
        const int width = a.H * a.dv;
        const dim3 threads(width >= 1024 ? 256 : 128);
        if (vec)
            rv_launch(la_finish_all_kernel<T, 4>, dim3(a.n_tokens), threads, 0, s, (const float*)num, rows,
                      a.stride, g_off, a.norm_w, a.eps, a.token_req, a.state_slot, out, width, a.gate);
        else
            rv_launch(la_finish_all_kernel<T, 1>, dim3(a.n_tokens), threads, 0, s, (const float*)num, rows,
                      a.stride, g_off, a.norm_w, a.eps, a.token_req, a.state_slot, out, width, a.gate);
    }
    RV_CHECK_LAUNCH("linear_attention_finish");
    return 0;
}

// log_decay [H]; or null, then z float32 [n, H d] (used up: the tensor-core forms leave sums of log
// decays there), bias [H d] and tau.  act: 1 silu; norm_head: 0 all
// heads together, 1 per head; gate: 0 sigmoid, 1 silu; norm_w [H dv].  Requests [0, n_decode) bring
// one token each (token r is request r's).  `tensor`: whether portions may take the tensor-core
// forms (where their sizes allow).  rows and out have the type `dtype`.
extern "C" int rv_linear_attention(const void* rows, int dtype, int stride, float* z,
                                   const float* log_decay, const float* bias, float tau,
                                   const float* norm_w, float* state, const int* token_req,
                                   const int* q_start, const int* state_slot, float* scratch, void* out,
                                   int n_tokens, int n_decode, int n_reqs, int H, int d, int dv, int act,
                                   float q_scale, int norm_head, int gate, float eps, int tensor,
                                   void* stream) {
    if (n_tokens == 0 || n_reqs == 0) return 0;
    if (n_tokens < 0 || n_decode < 0 || n_decode > n_reqs || n_decode > n_tokens || H < 1 || d < 1 || dv < 1)
        RV_FAIL("linear_attention: bad sizes");
    if (!log_decay && (!z || !bias || !(tau > 0.f))) RV_FAIL("linear_attention: neither a decay nor z, a bias and tau");
    if (stride < 2 * H * d + 2 * H * dv) RV_FAIL("linear_attention: rows are too short");
    const int tiles_d = (d + LA_T - 1) / LA_T, tiles_v = (dv + LA_T - 1) / LA_T;
    if (n_reqs > 65535 || H > 65535 || d > 2048 || dv > 65535 || tiles_d * tiles_v > 65535)
        RV_FAIL("linear_attention: too many requests or heads, or heads that are too large");
    if ((uintptr_t)scratch & 15) RV_FAIL("linear_attention: the scratch must be 16-byte aligned");
    tensor = tensor && dtype == RV_DTYPE_BF16 && d % 16 == 0 && dv % 16 == 0 && d <= 128 && stride % 8 == 0 &&
             (((uintptr_t)rows | (uintptr_t)z) & 15) == 0;
    const LaArgs a = {{0, H * d, 2 * H * d, 1}, {nullptr, nullptr}, z, log_decay, bias, norm_w, state, scratch, token_req, q_start, state_slot, tau, q_scale, eps,
                      stride, H * d, n_tokens, n_decode, n_reqs, H, d, dv, act, norm_head, gate, tensor};
    RV_DISPATCH_DTYPE(dtype, "linear_attention",
                      return la_run<T>((const T*)rows, a, (T*)out, (cudaStream_t)stream));
    return 0;
}

#include "state_space.cuh"
