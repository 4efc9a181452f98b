// Between the joined q/k/v product and the paged cache, for attention whose queries and keys are normed over the WHOLE
// projection (all heads of a token at once, before they are split) and whose values may have another head size than
// its keys: RMS norm of the token's q row and of its k row with plain weights, rotation of the first 2 * rot_half
// dimensions of every head (pairs (2j, 2j + 1) or (j, j + rot_half)), q out, k and v into the pages of the token's
// request. Statistics, angles and the rotation are 32-bit; angle = float(position) * inv_freq[j].
#include "common.cuh"
#include "api.h"

namespace {

constexpr int THREADS = 128;

// Further options. norm_q / norm_k > 0: how many of a row's values the whole-row norms average over (heads that are padded
// with zeros count their own values only). first: values of the same tokens that another layer projected, blended into this
// layer's ones: heads of first_dv values, first_places apart; this layer's heads have dv values of their own (then zeros).
// same: both rows are laid out alike and the other one lies in 16-byte pieces.
struct BlBlendArgs { int norm_q, norm_k; const float* first; int ld_first, first_dv, first_places, dv; const void* lambda; int lambda_dtype; int same; };

__device__ __forceinline__ float block_sum(float v, float* part) {
    v = bl_warp_sum(v);
    __syncthreads();                                   // part may still be read from the call before
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    return (part[0] + part[1]) + (part[2] + part[3]);
}

template <typename TT>
__global__ void __launch_bounds__(THREADS)
qk_norm_rope_write_kernel(const float* proj, int ld, int off_k, int off_v, const void* __restrict__ qw, int qw_dtype,
                          const void* __restrict__ kw, int kw_dtype, float eps, const int* __restrict__ positions,
                          const int* __restrict__ tok_req, const int* __restrict__ block_table, int max_pages,
                          const float* __restrict__ inv_freq, int rot_half, int pair_layout, TT* __restrict__ q_out,
                          TT* __restrict__ k_cache, TT* __restrict__ v_cache, int H, int KV, int dk, int dv, int page_size,
                          int per_head, const float* __restrict__ q_head_scale, BlBlendArgs bl) {
    bl_pdl_trigger();
    bl_pdl_wait();
    extern __shared__ float cs[];                      // cos [rot_half], sin [rot_half], then (per_head) 1 / rms of each of the H + KV heads
    __shared__ float part[4];
    const int t = blockIdx.x;
    const float* row = proj + (size_t)t * ld;
    const int pos = positions[t];
    for (int j = threadIdx.x; j < rot_half; j += THREADS) {
        const float a = (float)pos * inv_freq[j];
        cs[j] = cosf(a);
        cs[rot_half + j] = sinf(a);
    }
    float inv_q = 1.f, inv_k = 1.f;
    float* inv_head = cs + 2 * rot_half;
    if (per_head) {                                    // a norm over each head's dk values; the weights [dk] are shared by the heads
        const int lane = threadIdx.x & 31;
        for (int hh = threadIdx.x >> 5; hh < H + KV; hh += THREADS / 32) {
            const float* hr = row + (hh < H ? hh * dk : off_k + (hh - H) * dk);
            float s = 0.f;
            for (int i = lane; i < dk; i += 32) s += hr[i] * hr[i];
            s = bl_warp_sum(s);
            if (lane == 0) inv_head[hh] = ((hh < H ? qw : kw) != nullptr) ? 1.0f / sqrtf(s / (float)dk + eps) : 1.f;
        }
    } else if (qw) {
        float s = 0.f;
        for (int i = threadIdx.x; i < H * dk; i += THREADS) s += row[i] * row[i];
        inv_q = 1.0f / sqrtf(block_sum(s, part) / (float)(bl.norm_q > 0 ? bl.norm_q : H * dk) + eps);
    }
    if (kw && !per_head) {
        float s = 0.f;
        for (int i = threadIdx.x; i < KV * dk; i += THREADS) s += row[off_k + i] * row[off_k + i];
        inv_k = 1.0f / sqrtf(block_sum(s, part) / (float)(bl.norm_k > 0 ? bl.norm_k : KV * dk) + eps);
    }
    __syncthreads();
    const int r = tok_req[t];
    const int page = k_cache || v_cache ? block_table[(size_t)r * max_pages + pos / page_size] : 0;
    const int in_page = pos % page_size;
    const int n_rot = 2 * rot_half;
    // heads 0 .. H - 1 are q's, H .. H + KV - 1 are k's
    for (int e = threadIdx.x; e < (H + KV) * dk; e += THREADS) {
        const int hh = e / dk, d = e % dk;
        const bool is_q = hh < H;
        const int col = is_q ? hh * dk : off_k + (hh - H) * dk;        // the head's first column in the row
        const int wcol = per_head ? 0 : (is_q ? hh * dk : (hh - H) * dk);
        const void* w = is_q ? qw : kw;
        const int wd = is_q ? qw_dtype : kw_dtype;
        const float inv = per_head ? inv_head[hh] : (is_q ? inv_q : inv_k);
        auto normed = [&](int dd) { return row[col + dd] * inv * (w ? bl_load_any(w, wd, wcol + dd) : 1.f); };
        float val;
        if (d < n_rot) {
            int j, other;
            bool first;
            if (pair_layout == BL_PAIRS_INTERLEAVED) { j = d >> 1; first = (d & 1) == 0; other = first ? d + 1 : d - 1; }
            else { first = d < rot_half; j = first ? d : d - rot_half; other = first ? d + rot_half : d - rot_half; }
            const float c = cs[j], s = cs[rot_half + j];
            const float me = normed(d), ot = normed(other);
            val = first ? me * c - ot * s : me * c + ot * s;
        } else {
            val = normed(d);
        }
        if (is_q) {
            bl_store(q_out + (size_t)t * H * dk + e, q_head_scale ? val * q_head_scale[hh] : val);
        } else if (k_cache) {
            bl_store(k_cache + (((size_t)page * KV + (hh - H)) * page_size + in_page) * dk + d, val);
        }
    }
    if (v_cache) {
        for (int e = threadIdx.x; e < KV * dv; e += THREADS) {
            const int g = e / dv, d = e % dv;
            float v = row[off_v + e];
            if (bl.first) {                            // v <- (1 - lambda) v + lambda first, channel by channel of the flat values
                float f = 0.f;
                if (d < bl.dv) {
                    const int flat = g * bl.dv + d;
                    f = bl.first[(size_t)t * bl.ld_first + (flat / bl.first_dv) * bl.first_places + flat % bl.first_dv];
                }
                const float lam = bl_load_any(bl.lambda, bl.lambda_dtype, 0);
                v = (1.f - lam) * v + lam * f;
            }
            bl_store(v_cache + (((size_t)page * KV + g) * page_size + in_page) * dv + d, v);
        }
    }
}

// The same four values at a time, for rows, heads and rotated parts that are multiples of four and rotation in halves: the
// token's q and k rows are read once, into shared memory, with both sums of squares on the way; positions, angles and page
// numbers are worked out before the kernel's predecessor has finished.
constexpr int FAST_THREADS = 512;

__device__ __forceinline__ void store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&v)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
}
__device__ __forceinline__ float4 weights4(const void* w, int dtype, int i) {
    if (!w) return make_float4(1.f, 1.f, 1.f, 1.f);
    if (dtype == BL_F32) return *reinterpret_cast<const float4*>((const float*)w + i);
    const uint2 u = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)w + i);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

template <typename TT>
__global__ void __launch_bounds__(FAST_THREADS)
qk_norm_rope_write4_kernel(const float* proj, int ld, int off_k, int off_v, const void* __restrict__ qw, int qw_dtype,
                           const void* __restrict__ kw, int kw_dtype, float eps, const int* __restrict__ positions,
                           const int* __restrict__ tok_req, const int* __restrict__ block_table, int max_pages,
                           const float* __restrict__ inv_freq, int rot_half, TT* __restrict__ q_out,
                           TT* __restrict__ k_cache, TT* __restrict__ v_cache, int H, int KV, int dk, int dv, int page_size,
                           int per_head, const float* __restrict__ q_head_scale, BlBlendArgs bl) {
    bl_pdl_trigger();
    extern __shared__ __align__(16) float sm4[];       // cos, sin [rot_half] each, the q and k rows [(H + KV) * dk], 1 / rms per head
    __shared__ float part[2][FAST_THREADS / 32];
    const int t = blockIdx.x, nq = H * dk, nk = KV * dk;
    float* cs = sm4;
    float* sn = cs + rot_half;
    float* x = sn + rot_half;
    float* inv_head = x + nq + nk;
    const int pos = positions[t], r = tok_req[t];
    for (int j = threadIdx.x; j < rot_half; j += blockDim.x) {
        const float a = (float)pos * inv_freq[j];
        cs[j] = cosf(a);
        sn[j] = sinf(a);
    }
    const int page = k_cache || v_cache ? block_table[(size_t)r * max_pages + pos / page_size] : 0;
    const int in_page = pos % page_size;
    const float lam = bl.first ? bl_load_any(bl.lambda, bl.lambda_dtype, 0) : 0.f;
    bl_pdl_wait();
    const float* row = proj + (size_t)t * ld;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x * 4; i < nq + nk; i += blockDim.x * 4) {
        const float4 f = *reinterpret_cast<const float4*>(row + (i < nq ? i : off_k + i - nq));
        *reinterpret_cast<float4*>(x + i) = f;
        const float s = (f.x * f.x + f.y * f.y) + (f.z * f.z + f.w * f.w);
        if (i < nq) sq += s; else sk += s;
    }
    if (v_cache) {                                     // (no norm, no rotation: they need not wait for the sums)
        for (int e = threadIdx.x * 4; e < KV * dv; e += blockDim.x * 4) {
            const int g = e / dv, d = e % dv;
            const float4 f = *reinterpret_cast<const float4*>(row + off_v + e);
            float v[4] = {f.x, f.y, f.z, f.w};
            if (bl.first && bl.same) {
                const float4 o = *reinterpret_cast<const float4*>(bl.first + (size_t)t * bl.ld_first + e);
                v[0] = (1.f - lam) * v[0] + lam * o.x;
                v[1] = (1.f - lam) * v[1] + lam * o.y;
                v[2] = (1.f - lam) * v[2] + lam * o.z;
                v[3] = (1.f - lam) * v[3] + lam * o.w;
            } else if (bl.first) {
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    float o = 0.f;
                    if (d + j < bl.dv) {
                        const int flat = g * bl.dv + d + j;
                        o = bl.first[(size_t)t * bl.ld_first + (flat / bl.first_dv) * bl.first_places + flat % bl.first_dv];
                    }
                    v[j] = (1.f - lam) * v[j] + lam * o;
                }
            }
            store4(v_cache + (((size_t)page * KV + g) * page_size + in_page) * dv + d, v);
        }
    }
    float inv_q = 1.f, inv_k = 1.f;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    if (!per_head) {
        sq = bl_warp_sum(sq);
        sk = bl_warp_sum(sk);
        if (lane == 0) { part[0][warp] = sq; part[1][warp] = sk; }
    }
    __syncthreads();
    if (per_head) {
        for (int hh = warp; hh < H + KV; hh += warps) {
            float s = 0.f;
            for (int i = lane; i < dk; i += 32) s += x[hh * dk + i] * x[hh * dk + i];
            s = bl_warp_sum(s);
            if (lane == 0) inv_head[hh] = ((hh < H ? qw : kw) != nullptr) ? 1.0f / sqrtf(s / (float)dk + eps) : 1.f;
        }
        __syncthreads();
    } else {
        float a = 0.f, b = 0.f;
        for (int i = 0; i < warps; ++i) { a += part[0][i]; b += part[1][i]; }
        if (qw) inv_q = 1.0f / sqrtf(a / (float)(bl.norm_q > 0 ? bl.norm_q : nq) + eps);
        if (kw) inv_k = 1.0f / sqrtf(b / (float)(bl.norm_k > 0 ? bl.norm_k : nk) + eps);
    }
    for (int e = threadIdx.x * 4; e < nq + nk; e += blockDim.x * 4) {
        const bool is_q = e < nq;
        const int hh = e / dk, d = e - hh * dk;
        const int wbase = per_head ? 0 : (is_q ? hh * dk : (hh - H) * dk);
        const void* w = is_q ? qw : kw;
        const int wd = is_q ? qw_dtype : kw_dtype;
        const float inv = per_head ? inv_head[hh] : (is_q ? inv_q : inv_k);
        const float4 m = *reinterpret_cast<const float4*>(x + e);
        const float4 mw = weights4(w, wd, wbase + d);
        float v[4] = {m.x * inv * mw.x, m.y * inv * mw.y, m.z * inv * mw.z, m.w * inv * mw.w};
        if (d < 2 * rot_half) {
            const bool first = d < rot_half;
            const int od = first ? d + rot_half : d - rot_half, j = first ? d : d - rot_half;
            const float4 o = *reinterpret_cast<const float4*>(x + hh * dk + od);
            const float4 ow = weights4(w, wd, wbase + od);
            const float4 c = *reinterpret_cast<const float4*>(cs + j), s4 = *reinterpret_cast<const float4*>(sn + j);
            const float sg = first ? -1.f : 1.f;
            v[0] = v[0] * c.x + sg * (o.x * inv * ow.x) * s4.x;
            v[1] = v[1] * c.y + sg * (o.y * inv * ow.y) * s4.y;
            v[2] = v[2] * c.z + sg * (o.z * inv * ow.z) * s4.z;
            v[3] = v[3] * c.w + sg * (o.w * inv * ow.w) * s4.w;
        }
        if (is_q) {
            if (q_head_scale) {
                const float f = q_head_scale[hh];
#pragma unroll
                for (int j = 0; j < 4; ++j) v[j] *= f;
            }
            store4(q_out + (size_t)t * nq + e, v);
        } else if (k_cache) {
            store4(k_cache + (((size_t)page * KV + (hh - H)) * page_size + in_page) * dk + d, v);
        }
    }
}

}  // namespace

extern "C" int bl_qk_norm_rope_write(const float* proj, int ld, int off_k, int off_v, const void* q_norm_w, int qw_dtype,
                                     const void* k_norm_w, int kw_dtype, float eps, const int* positions, const int* tok_req,
                                     const int* block_table, int max_pages, const float* inv_freq, int rot_half,
                                     int pair_layout, void* q_out, void* k_cache, void* v_cache, int dtype, int T, int H,
                                     int KV, int dk, int dv, int page_size, void* stream) {
    return bl_qk_norm_rope_write_scope(proj, ld, off_k, off_v, q_norm_w, qw_dtype, k_norm_w, kw_dtype, eps, 0, positions, tok_req,
                                       block_table, max_pages, inv_freq, rot_half, pair_layout, q_out, k_cache, v_cache, dtype, T, H,
                                       KV, dk, dv, page_size, nullptr, stream);
}

extern "C" int bl_qk_norm_rope_write_scope(const float* proj, int ld, int off_k, int off_v, const void* q_norm_w, int qw_dtype,
                                           const void* k_norm_w, int kw_dtype, float eps, int per_head, const int* positions,
                                           const int* tok_req, const int* block_table, int max_pages, const float* inv_freq,
                                           int rot_half, int pair_layout, void* q_out, void* k_cache, void* v_cache, int dtype, int T,
                                           int H, int KV, int dk, int dv, int page_size, const float* q_head_scale, void* stream) {
    return bl_qk_norm_rope_write_ext(proj, ld, off_k, off_v, q_norm_w, qw_dtype, k_norm_w, kw_dtype, eps, per_head, positions, tok_req,
                                     block_table, max_pages, inv_freq, rot_half, pair_layout, q_out, k_cache, v_cache, dtype, T, H,
                                     KV, dk, dv, page_size, q_head_scale, 0, 0, nullptr, 0, 0, 0, 0, nullptr, 0, stream);
}

extern "C" int bl_qk_norm_rope_write_ext(const float* proj, int ld, int off_k, int off_v, const void* q_norm_w, int qw_dtype,
                                         const void* k_norm_w, int kw_dtype, float eps, int per_head, const int* positions,
                                         const int* tok_req, const int* block_table, int max_pages, const float* inv_freq,
                                         int rot_half, int pair_layout, void* q_out, void* k_cache, void* v_cache, int dtype, int T,
                                         int H, int KV, int dk, int dv, int page_size, const float* q_head_scale, int norm_q, int norm_k,
                                         const float* v_first, int ld_first, int first_dv, int first_places, int dv_real, const void* lambda,
                                         int lambda_dtype, void* stream) {
    if (T <= 0) return 0;
    if (H <= 0 || KV <= 0 || dk <= 0 || dv <= 0 || rot_half < 0 || 2 * rot_half > dk || page_size <= 0)
        BL_FAIL("bl_qk_norm_rope_write: bad sizes H=%d KV=%d dk=%d dv=%d rotated pairs=%d page=%d", H, KV, dk, dv, rot_half, page_size);
    if (ld < off_v + KV * dv || off_k < H * dk || off_v < off_k + KV * dk)
        BL_FAIL("bl_qk_norm_rope_write: columns q, k (%d), v (%d) do not fit rows of %d", off_k, off_v, ld);
    if (norm_q < 0 || norm_q > H * dk || norm_k < 0 || norm_k > KV * dk)
        BL_FAIL("bl_qk_norm_rope_write: norms over %d and %d values of rows of %d and %d", norm_q, norm_k, H * dk, KV * dk);
    if (v_first && (!lambda || dv_real <= 0 || dv_real > dv || first_dv <= 0 || first_dv > first_places || KV * dv_real % first_dv != 0 ||
                    ld_first < KV * dv_real / first_dv * first_places))
        BL_FAIL("bl_qk_norm_rope_write: values of %d heads of %d cannot be blended with heads of %d in rows of %d", KV, dv_real, first_dv, ld_first);
    const int same = v_first && first_dv == dv_real && first_places == dv && ld_first % 4 == 0 && ((uintptr_t)v_first & 15) == 0;
    const BlBlendArgs bl{norm_q, norm_k, v_first, ld_first, first_dv, first_places, dv_real, lambda, lambda_dtype, same};
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem4 = (size_t)(2 * rot_half + (H + KV) * dk + (per_head ? H + KV : 0)) * sizeof(float);
    const bool fours = (pair_layout == BL_PAIRS_HALVES || rot_half == 0) && dk % 4 == 0 && dv % 4 == 0 && rot_half % 4 == 0 && ld % 4 == 0 &&
                       off_k % 4 == 0 && off_v % 4 == 0 && smem4 <= 48 * 1024 &&
                       (((uintptr_t)proj | (uintptr_t)q_norm_w | (uintptr_t)k_norm_w | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) == 0;
    if (fours) {
        int threads = ((H + KV) * dk / 4 + 31) / 32 * 32;
        const int most = T <= 256 ? FAST_THREADS : 256;
        if (threads > most) threads = most;
#define BL_GO(TT) BL_CUDA(bl_launch_dependent(qk_norm_rope_write4_kernel<TT>, dim3(T), dim3(threads), smem4, s, proj, ld, off_k, off_v, \
        q_norm_w, qw_dtype, k_norm_w, kw_dtype, eps, positions, tok_req, block_table, max_pages, inv_freq, rot_half, \
        (TT*)q_out, (TT*)k_cache, (TT*)v_cache, H, KV, dk, dv, page_size, per_head, q_head_scale, bl))
        if (dtype == BL_F32) BL_GO(float);
        else if (dtype == BL_BF16) BL_GO(__nv_bfloat16);
        else BL_FAIL("bl_qk_norm_rope_write: unknown dtype %d", dtype);
#undef BL_GO
        BL_CHECK_LAUNCH("bl_qk_norm_rope_write");
        return 0;
    }
    const size_t smem = (size_t)(2 * rot_half + 1 + (per_head ? H + KV : 0)) * sizeof(float);
#define BL_GO(TT) BL_CUDA(bl_launch_dependent(qk_norm_rope_write_kernel<TT>, dim3(T), dim3(THREADS), smem, s, proj, ld, off_k, off_v, \
        q_norm_w, qw_dtype, k_norm_w, kw_dtype, eps, positions, tok_req, block_table, max_pages, inv_freq, rot_half, pair_layout, \
        (TT*)q_out, (TT*)k_cache, (TT*)v_cache, H, KV, dk, dv, page_size, per_head, q_head_scale, bl))
    if (dtype == BL_F32) BL_GO(float);
    else if (dtype == BL_BF16) BL_GO(__nv_bfloat16);
    else BL_FAIL("bl_qk_norm_rope_write: unknown dtype %d", dtype);
#undef BL_GO
    BL_CHECK_LAUNCH("bl_qk_norm_rope_write");
    return 0;
}
