// A residual of several streams (hyper-connections) and an embedding that looks at pairs of tokens.
//
// A sublayer f with a norm N in front of it reads ONE row made of the S streams and writes its result back to all of them:
//     u = sum_s a[s] x_s;   y = f(N(u));   x'_t = sum_s M[s, t] x_s + b[t] y          (M is indexed [from, to])
// bl_hyper_step does everything between two sublayers in one pass over a token's streams: the write-back of the sublayer
// before, and the row that the next one reads, normed. A block owns a token; sums are 32-bit, s ascending; a token's
// results depend on its own streams alone.
#include "common.cuh"
#include "api.h"

namespace {

constexpr int MAX_STREAMS = 16;
constexpr int MAX_THREADS = 512;

template <int VEC> struct Lane;
template <> struct Lane<4> {
    float v[4];
    __device__ __forceinline__ void load(const float* p) { const float4 f = *reinterpret_cast<const float4*>(p); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
    __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
    __device__ __forceinline__ void store(__nv_bfloat16* p) const {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
    }
};
template <> struct Lane<1> {
    float v[1];
    __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
    __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
    __device__ __forceinline__ void store(__nv_bfloat16* p) const { *p = __float2bfloat16_rn(v[0]); }
};

struct HyperArgs {
    const float* x; long long x_stride;           // streams [S][rows][d], x_stride floats apart (0: all streams are the same rows)
    float* x_out; long long out_stride;           // where the new streams go (null: they are not written); may be x itself
    const float* write;                           // null: no write-back; else b [S], then M [S, S]
    const float* y; const int* y_pos; const float* y_wts; int top;    // the sublayer's result: see bl_hyper_step
    const float* read;                            // a [S] (null: all ones)
    const void* w; int w_dtype; float eps;        // the norm's weight (null: the row u itself goes to h)
    void* h; int h_dtype;                         // the next sublayer's rows (null: nothing is read)
    const int* row_idx; int n, d;                 // h's row r is token row_idx[r] (null: r)
};

// S > 0: that many streams; S = 0: `n`, up to MAX_STREAMS.
template <int S, int VEC, typename TH>
__global__ void __launch_bounds__(S == 0 ? 256 : MAX_THREADS, S >= 1 && S <= 4 ? 2 : 1)
hyper_step_kernel(const HyperArgs p) {
    bl_pdl_trigger();
    constexpr int NS = S > 0 ? S : MAX_STREAMS;
    const int n = S > 0 ? S : p.n;
    extern __shared__ float sm[];                 // a [NS], b [NS], M [NS * NS], the row u [d] (VEC * 4 bytes aligned)
    float* sa = sm;
    float* sb = sm + MAX_STREAMS;
    float* sM = sb + MAX_STREAMS;
    float* su = sM + MAX_STREAMS * MAX_STREAMS;
    __shared__ float part[MAX_THREADS / 32];
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        sa[i] = p.read ? p.read[i] : 1.f;
        if (p.write) sb[i] = p.write[i];
    }
    if (p.write) for (int i = threadIdx.x; i < n * n; i += blockDim.x) sM[i] = p.write[n + i];
    __syncthreads();
    bl_pdl_wait();
    const int r = blockIdx.x;
    const size_t t = p.row_idx ? (size_t)p.row_idx[r] : (size_t)r;
    const float* y0 = nullptr;
    if (p.write && !p.y_pos && p.top == 1 && !p.y_wts) y0 = p.y + t * p.d;
    float ss = 0.f;
#pragma unroll 1
    for (int c = threadIdx.x * VEC; c < p.d; c += blockDim.x * VEC) {
        Lane<VEC> x[NS], y;
        if (p.x_stride == 0) {
            x[0].load(p.x + t * p.d + c);
#pragma unroll
            for (int s = 1; s < NS; ++s) x[s] = x[0];
        } else {
#pragma unroll
            for (int s = 0; s < NS; ++s) if (s < n) x[s].load(p.x + (size_t)s * p.x_stride + t * p.d + c);
        }
        if (p.write) {
            if (y0) {
                y.load(y0 + c);
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) y.v[e] = 0.f;
                for (int k = 0; k < p.top; ++k) {
                    const long long row = p.y_pos ? (long long)p.y_pos[t * p.top + k] : (long long)(t * p.top + k);
                    if (row < 0) continue;
                    const float wt = p.y_wts ? p.y_wts[t * p.top + k] : 1.f;
                    Lane<VEC> part_y;
                    part_y.load(p.y + (size_t)row * p.d + c);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) y.v[e] = fmaf(wt, part_y.v[e], y.v[e]);
                }
            }
        }
        Lane<VEC> u;
#pragma unroll
        for (int e = 0; e < VEC; ++e) u.v[e] = 0.f;
        if (p.write) {
#pragma unroll
            for (int q = 0; q < NS; ++q) {
                if (q >= n) break;
                Lane<VEC> z;
                const float b = sb[q];
#pragma unroll
                for (int e = 0; e < VEC; ++e) z.v[e] = 0.f;
#pragma unroll
                for (int s = 0; s < NS; ++s) {
                    if (s >= n) break;
                    const float m = sM[s * n + q];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) z.v[e] = fmaf(m, x[s].v[e], z.v[e]);
                }
                const float a = sa[q];
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    z.v[e] = fmaf(b, y.v[e], z.v[e]);
                    u.v[e] = fmaf(a, z.v[e], u.v[e]);
                }
                if (p.x_out) z.store(p.x_out + (size_t)q * p.out_stride + t * p.d + c);
            }
        } else {
#pragma unroll
            for (int s = 0; s < NS; ++s) {
                if (s >= n) break;
                const float a = sa[s];
#pragma unroll
                for (int e = 0; e < VEC; ++e) u.v[e] = fmaf(a, x[s].v[e], u.v[e]);
            }
        }
        if (p.h) {
            u.store(su + c);
#pragma unroll
            for (int e = 0; e < VEC; ++e) ss = fmaf(u.v[e], u.v[e], ss);
        }
    }
    if (!p.h) return;
    float inv = 1.f;
    if (p.w) {
        ss = bl_warp_sum(ss);
        if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
        __syncthreads();
        float total = 0.f;
        for (int i = 0; i < (int)blockDim.x / 32; ++i) total += part[i];
        inv = 1.0f / sqrtf(total / (float)p.d + p.eps);
    }
    TH* h = reinterpret_cast<TH*>(p.h) + (size_t)r * p.d;
    for (int c = threadIdx.x * VEC; c < p.d; c += blockDim.x * VEC) {          // (every thread reads back what it wrote)
        Lane<VEC> u;
        u.load(su + c);
        if (p.w) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) u.v[e] = u.v[e] * inv * bl_load_any(p.w, p.w_dtype, c + e);
        }
        u.store(h + c);
    }
}

template <int S, int VEC>
int launch_hyper(const HyperArgs& a, int rows, cudaStream_t s) {
    int threads = ((a.d + VEC - 1) / VEC + 31) / 32 * 32;
    const int most = S > 0 && rows <= 256 ? MAX_THREADS : 256;                 // few rows: a step waits for one row's way through
    if (threads > most) threads = most;
    const size_t smem = (size_t)(2 * MAX_STREAMS + MAX_STREAMS * MAX_STREAMS + a.d) * sizeof(float);
    if (smem > 200 * 1024) BL_FAIL("bl_hyper_step: rows of %d values do not fit shared memory", a.d);
    if (a.h_dtype == BL_BF16) {
        if (smem > 48 * 1024) BL_CUDA(cudaFuncSetAttribute(hyper_step_kernel<S, VEC, __nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        BL_CUDA(bl_launch_dependent(hyper_step_kernel<S, VEC, __nv_bfloat16>, dim3(rows), dim3(threads), smem, s, a));
    } else {
        if (smem > 48 * 1024) BL_CUDA(cudaFuncSetAttribute(hyper_step_kernel<S, VEC, float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        BL_CUDA(bl_launch_dependent(hyper_step_kernel<S, VEC, float>, dim3(rows), dim3(threads), smem, s, a));
    }
    BL_CHECK_LAUNCH("bl_hyper_step");
    return 0;
}

template <int VEC>
int dispatch_hyper(const HyperArgs& a, int rows, cudaStream_t s) {
    switch (a.n) {
        case 1: return launch_hyper<1, VEC>(a, rows, s);
        case 2: return launch_hyper<2, VEC>(a, rows, s);
        case 3: return launch_hyper<3, VEC>(a, rows, s);
        case 4: return launch_hyper<4, VEC>(a, rows, s);
        case 5: return launch_hyper<5, VEC>(a, rows, s);
        case 6: return launch_hyper<6, VEC>(a, rows, s);
        case 7: return launch_hyper<7, VEC>(a, rows, s);
        case 8: return launch_hyper<8, VEC>(a, rows, s);
        default: return launch_hyper<0, VEC>(a, rows, s);
    }
}

// x[t, :] = table[token, :] + pairs[row, :], row = (previous token * mul_prev + token * mul_cur) mod buckets, or `buckets`
// for a sequence's first token. The previous token of a request's first token in this step comes from the request's slot;
// the same block leaves the request's last token there for the next step.
template <typename TT>
__global__ void embed_pairs_kernel(const TT* __restrict__ table, const TT* __restrict__ pairs, const int* __restrict__ ids,
                                   const int* __restrict__ positions, const int* __restrict__ tok_req, const int* __restrict__ cu_q,
                                   const int* __restrict__ slots, int* prev_tokens, long long mul_prev, long long mul_cur,
                                   long long buckets, float* __restrict__ out, int d) {
    bl_pdl_trigger();
    bl_pdl_wait();
    const int t = blockIdx.x;
    const int r = tok_req[t], first = cu_q[r];
    const long long cur = ids[t];
    long long row = buckets;
    if (positions[t] > 0) {
        const long long prev = t > first ? ids[t - 1] : prev_tokens[slots[r]];
        row = (prev * mul_prev + cur * mul_cur) % buckets;
        if (row < 0) row += buckets;
    }
    if (t == first) {
        __syncthreads();                               // every thread has read the slot
        if (threadIdx.x == 0) prev_tokens[slots[r]] = ids[cu_q[r + 1] - 1];
    }
    const TT* a = table + (size_t)cur * d;
    const TT* b = pairs + (size_t)row * d;
    for (int i = threadIdx.x; i < d; i += blockDim.x) out[(size_t)t * d + i] = bl_load(a + i) + bl_load(b + i);
}

}  // namespace

extern "C" int bl_embed_pairs(const void* table, const void* pairs, int dtype, const int* ids, const int* positions, const int* tok_req,
                              const int* cu_q, const int* slots, int* prev_tokens, long long mul_prev, long long mul_cur,
                              long long buckets, float* out, int T, int d, void* stream) {
    if (T <= 0) return 0;
    if (d <= 0 || buckets <= 0) BL_FAIL("bl_embed_pairs: bad sizes d=%d buckets=%lld", d, buckets);
    cudaStream_t s = (cudaStream_t)stream;
#define BL_GO(TT) BL_CUDA(bl_launch_dependent(embed_pairs_kernel<TT>, dim3(T), dim3(128), 0, s, (const TT*)table, (const TT*)pairs, ids, positions, \
        tok_req, cu_q, slots, prev_tokens, mul_prev, mul_cur, buckets, out, d))
    if (dtype == BL_F32) BL_GO(float);
    else if (dtype == BL_BF16) BL_GO(__nv_bfloat16);
    else BL_FAIL("bl_embed_pairs: unknown table dtype %d", dtype);
#undef BL_GO
    BL_CHECK_LAUNCH("bl_embed_pairs");
    return 0;
}

extern "C" int bl_hyper_step(const float* x, long long x_stride, float* x_out, long long out_stride, int n, const float* write,
                             const float* y, const int* y_pos, const float* y_wts, int top, const float* read, const void* w, int w_dtype,
                             float eps, void* h, int h_dtype, const int* row_idx, int rows, int d, void* stream) {
    if (rows <= 0) return 0;
    if (n < 1 || n > MAX_STREAMS) BL_FAIL("bl_hyper_step: %d streams (1..%d)", n, MAX_STREAMS);
    if (d <= 0 || top < 1) BL_FAIL("bl_hyper_step: bad sizes d=%d top=%d", d, top);
    if (write && !y) BL_FAIL("bl_hyper_step: a write-back needs the sublayer's result");
    if (!write && x_out) BL_FAIL("bl_hyper_step: without a write-back the streams do not change");
    if (h_dtype != BL_F32 && h_dtype != BL_BF16) BL_FAIL("bl_hyper_step: unknown dtype %d", h_dtype);
    HyperArgs a;
    a.x = x; a.x_stride = x_stride; a.x_out = x_out; a.out_stride = out_stride; a.write = write; a.y = y; a.y_pos = y_pos; a.y_wts = y_wts;
    a.top = top; a.read = read; a.w = w; a.w_dtype = w_dtype; a.eps = eps; a.h = h; a.h_dtype = h_dtype; a.row_idx = row_idx; a.n = n; a.d = d;
    const bool vec = d % 4 == 0 && x_stride % 4 == 0 && out_stride % 4 == 0 &&
                     (((uintptr_t)x | (uintptr_t)x_out | (uintptr_t)y | (uintptr_t)h) & 15) == 0;
    return vec ? dispatch_hyper<4>(a, rows, (cudaStream_t)stream) : dispatch_hyper<1>(a, rows, (cudaStream_t)stream);
}
