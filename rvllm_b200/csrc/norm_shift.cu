// Norms around the residual stream that look at more than one row or more than one source.
//
//   add_rmsnorm_shift  x_t = resid[t] + delta[t] (* dscale) + rows_add[t] + add, written to
//                      `resid_out`;  h_t = x_t / sqrt(mean(x_t^2) + eps) * w;
//                      out_t = h_t + (h_(t-1) - h_t) * shift, h_(t-1) the row of the same
//                      request's token before: of this step, or `state` [slots, hidden]
//                      (float32) for a request's first row of the step.  The request's last h
//                      goes to its state record.  Everything before `out` is float32.
//   normed_sum         out = sa * rms(a) * wa + sb * rms(b) * wb, row by row.
//
// A block of add_rmsnorm_shift takes SHIFT_ROWS consecutive rows; the row before its first is
// normalised once more (a fifth of the work instead of a second pass over the normed rows), which
// is why the stream's rows are read from one buffer and written to another.  A request's record is
// read and then written by the one block that holds the request's first row (it normalises the
// request's last row too), so no block writes what another still reads.
// With few rows (decoding) a block takes one row.
// Plain references: tests/plain_ops.py add_rmsnorm_shift, normed_sum.
#include "common.cuh"

#define SHIFT_ROWS 4

__device__ __forceinline__ float4 ns_load4(const float* p) { return *(const float4*)p; }
__device__ __forceinline__ float4 ns_load4(const __nv_bfloat16* p) {
    const uint2 raw = *(const uint2*)p;
    const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&raw.x);
    const float2 b = __bfloat1622float2(*(const __nv_bfloat162*)&raw.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void ns_store4(float* p, float4 v) { *(float4*)p = v; }
__device__ __forceinline__ void ns_store4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *(const unsigned*)&a;
    raw.y = *(const unsigned*)&b;
    *(uint2*)p = raw;
}
// V values a thread and step: 4 (16-byte float32 accesses) or 1.
template <int V> struct NsVec;
template <> struct NsVec<4> {
    float4 v;
    template <typename T> __device__ __forceinline__ void load(const T* p) { v = ns_load4(p); }
    template <typename T> __device__ __forceinline__ void store(T* p) const { ns_store4(p, v); }
    __device__ __forceinline__ void zero() { v = make_float4(0.f, 0.f, 0.f, 0.f); }
    __device__ __forceinline__ void add(const NsVec& o) { v.x += o.v.x; v.y += o.v.y; v.z += o.v.z; v.w += o.v.w; }
    __device__ __forceinline__ void mul(const NsVec& o) { v.x *= o.v.x; v.y *= o.v.y; v.z *= o.v.z; v.w *= o.v.w; }
    __device__ __forceinline__ void scale(float s) { v.x *= s; v.y *= s; v.z *= s; v.w *= s; }
    __device__ __forceinline__ float sq() const { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
    // this + (before - this) * m
    __device__ __forceinline__ NsVec towards(const NsVec& before, const NsVec& m) const {
        NsVec o;
        o.v = make_float4(v.x + (before.v.x - v.x) * m.v.x, v.y + (before.v.y - v.y) * m.v.y,
                          v.z + (before.v.z - v.z) * m.v.z, v.w + (before.v.w - v.w) * m.v.w);
        return o;
    }
};
template <> struct NsVec<1> {
    float v;
    template <typename T> __device__ __forceinline__ void load(const T* p) { v = rv_load(p); }
    template <typename T> __device__ __forceinline__ void store(T* p) const { rv_store(p, v); }
    __device__ __forceinline__ void zero() { v = 0.f; }
    __device__ __forceinline__ void add(const NsVec& o) { v += o.v; }
    __device__ __forceinline__ void mul(const NsVec& o) { v *= o.v; }
    __device__ __forceinline__ void scale(float s) { v *= s; }
    __device__ __forceinline__ float sq() const { return v * v; }
    __device__ __forceinline__ NsVec towards(const NsVec& before, const NsVec& m) const {
        NsVec o;
        o.v = v + (before.v - v) * m.v;
        return o;
    }
};

// The sums of `n` values each over the block: every thread gets all of them.
template <int N>
__device__ __forceinline__ void ns_block_sums(float (&v)[N], float* scratch /* [32 * N] */) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = rv_warp_sum(v[i]);
    __syncthreads();
    if (lane == 0) {
#pragma unroll
        for (int i = 0; i < N; ++i) scratch[warp * N + i] = v[i];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < N; ++i) {
        float t = 0.f;
        for (int w = 0; w < nwarps; ++w) t += scratch[w * N + i];
        v[i] = t;
    }
}

// ROWS rows a block; CHUNKS * blockDim.x * V >= hidden.  A thread holds its columns of all the
// block's rows (and of the row before them) in registers.
template <typename TD, typename TO, int V, int CHUNKS, int ROWS>
__global__ void add_rmsnorm_shift_kernel(
    const float* resid, float* resid_out, const TD* __restrict__ delta,
    const float* __restrict__ dscale, const float* __restrict__ add,
    const float* __restrict__ rows_add, const float* __restrict__ weight, float eps,
    TO* __restrict__ out, const float* __restrict__ shift, float* __restrict__ state,
    const int* __restrict__ token_req, const int* __restrict__ q_start,
    const int* __restrict__ state_slot, int n_rows, int hidden) {
    rv_pdl_launch_dependents();
    __shared__ float scratch[32 * (ROWS + 1)];
    const int t0 = blockIdx.x * ROWS;
    const int tid = threadIdx.x, nt = blockDim.x;
    // which rows' predecessors lie in this step (index arrays of the step: before the wait)
    bool inside[ROWS];                          // row t0 + i - 1 is the same request's
    int slot_in[ROWS], last_row[ROWS];          // first rows: the record, the request's last row
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        inside[i] = false;
        slot_in[i] = -1;
        last_row[i] = -1;
        if (shift && t0 + i < n_rows) {
            const int r = token_req[t0 + i];
            inside[i] = t0 + i > q_start[r];
            if (!inside[i]) {
                slot_in[i] = state_slot[r];
                last_row[i] = q_start[r + 1] - 1;
            }
        }
    }
    rv_pdl_wait();
    auto load_row = [&](int t, NsVec<V> (&x)[CHUNKS]) -> float {
        const size_t at = (size_t)t * hidden;
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const int i = (tid + c * nt) * V;
            x[c].zero();
            if (i < hidden) {
                x[c].load(resid + at + i);
                NsVec<V> u;
                if (delta) {
                    u.load(delta + at + i);
                    if (dscale) {
                        NsVec<V> g;
                        g.load(dscale + i);
                        u.mul(g);
                    }
                    x[c].add(u);
                }
                if (rows_add) {
                    u.load(rows_add + at + i);
                    x[c].add(u);
                }
                if (add) {
                    u.load(add + i);
                    x[c].add(u);
                }
                ss += x[c].sq();
            }
        }
        return ss;
    };
    NsVec<V> x[ROWS + 1][CHUNKS];               // row 0: the row before the block's first
    float ss[ROWS + 1];
#pragma unroll
    for (int i = 0; i <= ROWS; ++i) ss[i] = 0.f;
    if (inside[0]) ss[0] = load_row(t0 - 1, x[0]);
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
        if (t0 + i < n_rows) ss[i + 1] = load_row(t0 + i, x[i + 1]);
    ns_block_sums<ROWS + 1>(ss, scratch);
    NsVec<V> w[CHUNKS], m[CHUNKS];
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int i = (tid + c * nt) * V;
        w[c].zero();
        m[c].zero();
        if (i < hidden) {
            w[c].load(weight + i);
            if (shift) m[c].load(shift + i);
        }
    }
#pragma unroll
    for (int k = 0; k <= ROWS; ++k) {
        const bool there = k == 0 ? inside[0] : t0 + k - 1 < n_rows;
        if (!there) continue;
        const float inv = 1.f / sqrtf(ss[k] / (float)hidden + eps);
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const int i = (tid + c * nt) * V;
            if (i >= hidden) continue;
            if (k > 0 && resid_out != resid) x[k][c].store(resid_out + (size_t)(t0 + k - 1) * hidden + i);
            else if (k > 0 && (delta || rows_add || add)) x[k][c].store(resid_out + (size_t)(t0 + k - 1) * hidden + i);
            x[k][c].scale(inv);
            x[k][c].mul(w[c]);                                  // h
        }
    }
#pragma unroll
    for (int k = 1; k <= ROWS; ++k) {
        const int t = t0 + k - 1;
        if (t >= n_rows) continue;
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const int i = (tid + c * nt) * V;
            if (i >= hidden) continue;
            NsVec<V> before;
            if (inside[k - 1]) before = x[k - 1][c];
            else if (slot_in[k - 1] >= 0) before.load(state + (size_t)slot_in[k - 1] * hidden + i);
            else before.zero();
            const NsVec<V> y = shift ? x[k][c].towards(before, m[c]) : x[k][c];
            y.store(out + (size_t)t * hidden + i);
        }
    }
    // the records of the requests that begin here: their last rows' h
#pragma unroll
    for (int k = 1; k <= ROWS; ++k) {
        const int s = slot_in[k - 1];
        if (s < 0) continue;                                    // the same for the whole block
        const int last = last_row[k - 1];
        float* rec = state + (size_t)s * hidden;
        if (last >= t0 && last < t0 + ROWS) {
#pragma unroll
            for (int j = 1; j <= ROWS; ++j)
                if (t0 + j - 1 == last)
#pragma unroll
                    for (int c = 0; c < CHUNKS; ++c) {
                        const int i = (tid + c * nt) * V;
                        if (i < hidden) x[j][c].store(rec + i);
                    }
            continue;
        }
        NsVec<V> z[CHUNKS];
        float s1[1] = {load_row(last, z)};
        ns_block_sums<1>(s1, scratch);
        const float inv = 1.f / sqrtf(s1[0] / (float)hidden + eps);
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const int i = (tid + c * nt) * V;
            if (i < hidden) {
                z[c].scale(inv);
                z[c].mul(w[c]);
                z[c].store(rec + i);
            }
        }
    }
}

template <typename TD, typename TO>
static int add_rmsnorm_shift_launch(const float* resid, float* resid_out, const void* delta,
                                    const float* dscale, const float* add, const float* rows_add,
                                    const float* weight, float eps, void* out, const float* shift,
                                    float* state, const int* token_req, const int* q_start,
                                    const int* state_slot, int n_rows, int hidden, cudaStream_t s) {
    const uintptr_t all = (uintptr_t)resid | (uintptr_t)resid_out | (uintptr_t)delta | (uintptr_t)dscale |
                          (uintptr_t)add | (uintptr_t)rows_add | (uintptr_t)weight | (uintptr_t)out |
                          (uintptr_t)shift | (uintptr_t)state;
    const bool vec = hidden % 4 == 0 && all % 16 == 0;
    const int per = vec ? 4 : 1;
    const int need = (hidden + per - 1) / per;                  // positions a row has
    int chunks = 1;
    while (chunks < 8 && (need + chunks - 1) / chunks > 512) chunks *= 2;
    int threads = (((need + chunks - 1) / chunks + 31) / 32) * 32;
    if (threads > 1024) RV_FAIL("add_rmsnorm_shift: width %d is too large", hidden);
    // several rows a block once that leaves every SM work, and while the rows fit the registers
    const bool many = shift && chunks == 1 && n_rows >= 2 * rv_sm_count();
#define NS_GO(V, C, R)                                                                            \
    rv_launch(add_rmsnorm_shift_kernel<TD, TO, V, C, R>, dim3((n_rows + R - 1) / R), dim3(threads), \
              0, s, resid, resid_out, (const TD*)delta, dscale, add, rows_add, weight, eps, (TO*)out, \
              shift, state, token_req, q_start, state_slot, n_rows, hidden)
#define NS_PICK(V)                                  \
    switch (chunks) {                               \
        case 1:                                     \
            if (many) NS_GO(V, 1, SHIFT_ROWS);      \
            else NS_GO(V, 1, 1);                    \
            break;                                  \
        case 2: NS_GO(V, 2, 1); break;              \
        case 4: NS_GO(V, 4, 1); break;              \
        default: NS_GO(V, 8, 1); break;             \
    }
    if (vec) {
        NS_PICK(4)
    } else {
        NS_PICK(1)
    }
#undef NS_PICK
#undef NS_GO
    RV_CHECK_LAUNCH("add_rmsnorm_shift");
    return 0;
}

// `shift` null: no row looks at another, and `resid_out` may be `resid`.
extern "C" int rv_add_rmsnorm_shift(const float* resid, float* resid_out, const void* delta,
                                    int delta_dtype, const float* dscale, const float* add,
                                    const float* rows_add, const float* weight, float eps, void* out,
                                    int out_dtype, const float* shift, float* state,
                                    const int* token_req, const int* q_start, const int* state_slot,
                                    int n_rows, int hidden, void* stream) {
    if (n_rows == 0) return 0;
    if (n_rows < 0 || hidden <= 0) RV_FAIL("add_rmsnorm_shift: bad sizes");
    if (shift && (!state || !token_req || !q_start || !state_slot || resid == resid_out))
        RV_FAIL("add_rmsnorm_shift: a shift needs the records, the step's index arrays and a second "
                "buffer for the stream");
    if (dscale && !delta) RV_FAIL("add_rmsnorm_shift: a scale without rows to scale");
    cudaStream_t s = (cudaStream_t)stream;
#define NS_CALL(TD, TO)                                                                            \
    return add_rmsnorm_shift_launch<TD, TO>(resid, resid_out, delta, dscale, add, rows_add, weight, \
                                            eps, out, shift, state, token_req, q_start, state_slot, \
                                            n_rows, hidden, s)
    if (delta_dtype == RV_DTYPE_F32 && out_dtype == RV_DTYPE_F32) NS_CALL(float, float);
    if (delta_dtype == RV_DTYPE_F32 && out_dtype == RV_DTYPE_BF16) NS_CALL(float, __nv_bfloat16);
    if (delta_dtype == RV_DTYPE_BF16 && out_dtype == RV_DTYPE_F32) NS_CALL(__nv_bfloat16, float);
    if (delta_dtype == RV_DTYPE_BF16 && out_dtype == RV_DTYPE_BF16) NS_CALL(__nv_bfloat16, __nv_bfloat16);
#undef NS_CALL
    RV_FAIL("add_rmsnorm_shift: unknown dtype codes %d, %d", delta_dtype, out_dtype);
}

// ---------------------------------------------------------------------------------
template <typename T, int V, int CHUNKS>
__global__ void normed_sum_kernel(const T* __restrict__ a, const float* __restrict__ wa, float sa,
                                  const T* __restrict__ b, const float* __restrict__ wb, float sb,
                                  float eps, T* __restrict__ out, int hidden) {
    rv_pdl_launch_dependents();
    __shared__ float scratch[64];
    const size_t at = (size_t)blockIdx.x * hidden;
    const int tid = threadIdx.x, nt = blockDim.x;
    NsVec<V> x[CHUNKS], y[CHUNKS], u[CHUNKS], w[CHUNKS];
    float ss[2] = {0.f, 0.f};
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int i = (tid + c * nt) * V;
        if (i < hidden) {                                       // constants: before the wait
            u[c].load(wa + i);
            w[c].load(wb + i);
        }
    }
    rv_pdl_wait();
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int i = (tid + c * nt) * V;
        if (i < hidden) {
            x[c].load(a + at + i);
            y[c].load(b + at + i);
            ss[0] += x[c].sq();
            ss[1] += y[c].sq();
        }
    }
    ns_block_sums<2>(ss, scratch);
    const float ra = sa / sqrtf(ss[0] / (float)hidden + eps), rb = sb / sqrtf(ss[1] / (float)hidden + eps);
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int i = (tid + c * nt) * V;
        if (i < hidden) {
            x[c].mul(u[c]);
            x[c].scale(ra);
            y[c].mul(w[c]);
            y[c].scale(rb);
            x[c].add(y[c]);
            x[c].store(out + at + i);
        }
    }
}

extern "C" int rv_normed_sum(const void* a, const float* wa, float sa, const void* b, const float* wb,
                             float sb, float eps, void* out, int dtype, int n_rows, int hidden,
                             void* stream) {
    if (n_rows == 0) return 0;
    if (n_rows < 0 || hidden <= 0) RV_FAIL("normed_sum: bad sizes");
    const uintptr_t all = (uintptr_t)a | (uintptr_t)b | (uintptr_t)wa | (uintptr_t)wb | (uintptr_t)out;
    const bool vec = hidden % 4 == 0 && all % 16 == 0;
    const int need = (hidden + (vec ? 3 : 0)) / (vec ? 4 : 1);
    int chunks = 1;
    while (chunks < 8 && (need + chunks - 1) / chunks > 512) chunks *= 2;
    const int threads = (((need + chunks - 1) / chunks + 31) / 32) * 32;
    if (threads > 1024) RV_FAIL("normed_sum: width %d is too large", hidden);
    cudaStream_t s = (cudaStream_t)stream;
#define NS_GO(V, C)                                                                            \
    rv_launch(normed_sum_kernel<T, V, C>, dim3(n_rows), dim3(threads), 0, s, (const T*)a, wa, sa, \
              (const T*)b, wb, sb, eps, (T*)out, hidden)
#define NS_PICK(V)                       \
    switch (chunks) {                    \
        case 1: NS_GO(V, 1); break;      \
        case 2: NS_GO(V, 2); break;      \
        case 4: NS_GO(V, 4); break;      \
        default: NS_GO(V, 8); break;     \
    }
    RV_DISPATCH_DTYPE(dtype, "normed_sum", {
        if (vec) { NS_PICK(4) } else { NS_PICK(1) }
    });
#undef NS_PICK
#undef NS_GO
    RV_CHECK_LAUNCH("normed_sum");
    return 0;
}
