// Paged causal attention whose heads' scores are mixed BEFORE the softmax, over keys of unit root mean square whose values
// are the same vectors before that norm:
//   score_g(i, j) = q_g(i) . k_kv(g)(j) * scale - slope_g (i - j),   q and k divided by their root mean square per head
//   score'_h      = sum_g talk[h, g] score_g,   p_h = softmax_j(score'_h),   out_h(i) = sum_j p_h(i, j) v_kv(h)(j)
// The mix is linear in the query and in the slope, so it moves there:
//   score'_h(i, j) = (sum_c Q_h,c(i) . k_c(j)) * scale - slope'_h (i - j),   Q_h,c = sum_{g of key/value head c} talk[h, g] q_g,
//   slope'_h = sum_g talk[h, g] slope_g
// and every head is an ordinary softmax over ONE score per key: a product over the keys of all KV key/value heads side by
// side (KV * dh values a token, the same for every head), and nothing of size heads x heads x keys is ever formed. The cache
// holds a token's normed keys and, per key/value head, the root mean square they were divided by (32-bit): a value is its
// key times that number, which joins the softmax weight in front of the value product, so a token costs one row, not two.
// Scores, bias, softmax, norms and that number are 32-bit. A sigmoid gate per channel may follow (32-bit logits).
//
//   bl_mixed_prep             norms, the mixed queries Q [T, H, KV, dh], keys and their root mean squares into the pages
//   bl_attention_mixed_plain  one warp per (token, head), any dtype: the 32-bit path and the twin of the tensor-core kernels
//   bl_attention_mixed_prefill / _decode   tensor cores (bfloat16 operands, 32-bit sums):
//     prefill: a block is 64 consecutive tokens of one request and one query head, 16 rows a warp; the ring of shared-memory
//              stages takes tiles of 64 keys of ONE key/value head, the head's own last: the scores of a key block are
//              complete when its values (the same tile) are there
//     decode:  a block is one single-token request, up to 16 of its query heads (the MMA rows) and one slice of its keys;
//              each warp streams a page of every key/value head of its own key blocks through a ring of its own; the value
//              product of a key/value head takes the weights with the other heads' rows set to zero, so all rows share one
//              accumulator; slices are the blocks of one cluster and merge through distributed shared memory
#include "common.cuh"
#include "api.h"

namespace {

constexpr int PAGE = 16;
constexpr int KB = 64;                // keys per block (prefill)
constexpr int PAD = 8;                // bfloat16 elements of padding per shared-memory row (keeps ldmatrix conflict-free)
constexpr int MAX_DH = 512;           // the plain kernel's head size
constexpr int PLAIN_WARPS = 4;
constexpr int PREP_THREADS = 128;
constexpr int PREP_FEW_ROWS = 256;    // up to so many tokens a block of bl_mixed_prep makes the mixed queries of four heads, with more of all
constexpr int STAGES = 3;             // prefill ring
constexpr int MAX_DECODE_WARPS = 8;   // warps of a decode block
constexpr int MAX_CLUSTER = 16;       // slices merged through distributed shared memory

// ---- norms, mixed queries, keys into the pages ----------------------------------------------------------------------------
template <typename TT>
__global__ void __launch_bounds__(PREP_THREADS)
mixed_prep_kernel(const float* proj, int ld, int off_k, const float* __restrict__ talk, float eps, const int* __restrict__ positions,
                  const int* __restrict__ tok_req, const int* __restrict__ block_table, int max_pages, TT* __restrict__ q_out,
                  TT* __restrict__ k_cache, float* __restrict__ k_rms, int rms_stride, int H, int KV, int dh, int page_size, int heads_per_block) {
    bl_pdl_trigger();
    extern __shared__ __align__(16) float sm[];
    float* qn = sm;                                    // [H * dh] the token's normed queries
    float* coef = qn + ((H * dh + 3) & ~3);            // this block's rows of the mix, four heads side by side: [heads / 4][H][4]
    const int t = blockIdx.x, h0 = blockIdx.y * heads_per_block, nh = min(heads_per_block, H - h0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int i = threadIdx.x; i < ((nh + 3) & ~3) * H; i += PREP_THREADS) {
        const int hh = (i / (4 * H)) * 4 + (i & 3), g = (i >> 2) % H;
        coef[i] = hh < nh ? talk[(size_t)(h0 + hh) * H + g] : 0.f;
    }
    bl_pdl_wait();
    const float* row = proj + (size_t)t * ld;
    for (int g = warp; g < H; g += PREP_THREADS / 32) {
        const float* z = row + (size_t)g * dh;
        float s = 0.f;
        for (int i = lane; i < dh; i += 32) s += z[i] * z[i];
        const float inv = 1.0f / sqrtf(bl_warp_sum(s) / (float)dh + eps);
        for (int i = lane; i < dh; i += 32) qn[g * dh + i] = z[i] * inv;
    }
    if (blockIdx.y == 0 && k_cache) {                  // the keys, once per token
        const int pos = positions[t];
        const int page = block_table[(size_t)tok_req[t] * max_pages + pos / page_size], at = pos % page_size;
        for (int c = warp; c < KV; c += PREP_THREADS / 32) {
            const float* z = row + off_k + (size_t)c * dh;
            float s = 0.f;
            for (int i = lane; i < dh; i += 32) s += z[i] * z[i];
            const float rms = sqrtf(bl_warp_sum(s) / (float)dh + eps);
            const size_t slot = ((size_t)page * KV + c) * page_size + at;
            for (int i = lane; i < dh; i += 32) bl_store(k_cache + slot * dh + i, z[i] * (1.0f / rms));
            if (lane == 0) k_rms[slot * rms_stride] = rms;
        }
    }
    __syncthreads();
    const int G = H / KV;
    for (int e = threadIdx.x; e < KV * dh; e += PREP_THREADS) {
        const int c = e / dh, d = e - c * dh;
        for (int i0 = 0; i0 < nh; i0 += 4) {
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            const float4* cf = reinterpret_cast<const float4*>(coef + (i0 * H + c * G * 4));
            const float* qg = qn + c * G * dh + d;
            for (int g = 0; g < G; ++g) {
                const float v = qg[g * dh];
                const float4 w = cf[g];
                acc.x = fmaf(w.x, v, acc.x); acc.y = fmaf(w.y, v, acc.y); acc.z = fmaf(w.z, v, acc.z); acc.w = fmaf(w.w, v, acc.w);
            }
            TT* dst = q_out + ((size_t)t * H + h0 + i0) * KV * dh + e;
            const size_t next = (size_t)KV * dh;
            bl_store(dst, acc.x);
            if (i0 + 1 < nh) bl_store(dst + next, acc.y);
            if (i0 + 2 < nh) bl_store(dst + 2 * next, acc.z);
            if (i0 + 3 < nh) bl_store(dst + 3 * next, acc.w);
        }
    }
}

// ---- the plain kernel ------------------------------------------------------------------------------------------------------
template <typename TT>
__global__ void __launch_bounds__(PLAIN_WARPS * 32)
attention_mixed_plain_kernel(const TT* __restrict__ q, const TT* __restrict__ kc, const float* __restrict__ k_rms, int rms_stride,
                             const int* __restrict__ tok_req, const int* __restrict__ cu_q, const int* __restrict__ ctx_len,
                             const int* __restrict__ block_table, int max_pages, const float* __restrict__ slopes, const float* gate,
                             int ld_gate, TT* __restrict__ out, int T, int H, int KV, int dh, int page_size, float scale) {
    bl_pdl_trigger();
    bl_pdl_wait();
    extern __shared__ float qs_all[];                  // [PLAIN_WARPS][KV * dh]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int item = blockIdx.x * PLAIN_WARPS + warp;
    if (item >= T * H) return;                         // whole warps leave together; no block-wide barrier below
    const int width = KV * dh;
    float* qs = qs_all + (size_t)warp * width;
    const int t = item / H, h = item % H, own = h / (H / KV);
    const int r = tok_req[t];
    const int q_len = cu_q[r + 1] - cu_q[r];
    const int pos = ctx_len[r] - q_len + (t - cu_q[r]);
    for (int d = lane; d < width; d += 32) qs[d] = bl_load(q + ((size_t)t * H + h) * width + d);
    __syncwarp();
    const int* bt = block_table + (size_t)r * max_pages;
    const float slope = slopes ? slopes[h] : 0.f;
    float m = -INFINITY, l = 0.f;
    float acc[MAX_DH / 32];
#pragma unroll
    for (int i = 0; i < MAX_DH / 32; ++i) acc[i] = 0.f;
    for (int base = 0; base <= pos; base += 32) {
        const int j = base + lane;
        const bool valid = j <= pos;
        float s = -INFINITY, rms = 0.f;
        if (valid) {
            const size_t page = (size_t)bt[j / page_size];
            const int at = j % page_size;
            float dot = 0.f;
            for (int c = 0; c < KV; ++c) {
                const TT* krow = kc + ((page * KV + c) * page_size + at) * dh;
                for (int d = 0; d < dh; ++d) dot = fmaf(qs[c * dh + d], bl_load(krow + d), dot);
            }
            s = dot * scale - slope * (float)(pos - j);
            rms = k_rms[((page * KV + own) * page_size + at) * rms_stride];
        }
        const float m_new = fmaxf(m, bl_warp_max(s));
        const float p = valid ? expf(s - m_new) : 0.f;
        const float alpha = expf(m - m_new);           // first chunk: exp(-inf) = 0
        l = l * alpha + bl_warp_sum(p);
        const float pr = p * rms;
#pragma unroll
        for (int i = 0; i < MAX_DH / 32; ++i) acc[i] *= alpha;
        const int n = min(32, pos - base + 1);
        for (int jj = 0; jj < n; ++jj) {
            const float pj = __shfl_sync(0xffffffffu, pr, jj);
            const int key = base + jj;
            const TT* vrow = kc + (((size_t)bt[key / page_size] * KV + own) * page_size + key % page_size) * dh;
#pragma unroll
            for (int i = 0; i < MAX_DH / 32; ++i) {
                const int d = lane + 32 * i;
                if (d < dh) acc[i] = fmaf(pj, bl_load(vrow + d), acc[i]);
            }
        }
        m = m_new;
    }
    const float inv = l > 0.f ? 1.0f / l : 0.f;
    TT* orow = out + ((size_t)t * H + h) * dh;
#pragma unroll
    for (int i = 0; i < MAX_DH / 32; ++i) {
        const int d = lane + 32 * i;
        if (d >= dh) continue;
        float v = acc[i] * inv;
        if (gate) v *= 1.0f / (1.0f + expf(-gate[(size_t)t * ld_gate + (size_t)h * dh + d]));
        bl_store(orow + d, v);
    }
}

// ---- tensor cores ----------------------------------------------------------------------------------------------------------
struct MixedParams {
    const __nv_bfloat16* q;       // [tokens, H, KV, dh]
    const __nv_bfloat16* kc;      // [pages, KV, PAGE, dh]
    const float* k_rms;           // [pages, KV, PAGE]
    __nv_bfloat16* out;           // [tokens, H, dh]
    const int* cu_q; const int* ctx_len; const int* block_table; int max_pages;
    const int* work;              // prefill: [n][2] (request, first token of a 64-token tile); decode: [n] requests
    const float* slopes; const float* gate; int ld_gate;
    int H, KV, dh, n_splits;
    float scale_log2;
};

__device__ __forceinline__ void mma_bf16(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4(unsigned (&r)[4], const void* smem) {
    const unsigned addr = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], const void* smem) {
    const unsigned addr = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
    const unsigned addr = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" :: "r"(addr), "l"(gmem));
}
__device__ __forceinline__ void cp_async4(void* smem, const void* gmem) {
    const unsigned addr = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" :: "r"(addr), "l"(gmem));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" :: "n"(N)); }
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<unsigned*>(&v);
}
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// Two neighbouring scores at a time: Blackwell's packed 32-bit operations (each half rounded as its scalar form).
__device__ __forceinline__ unsigned long long pack2(float lo, float hi) {
    unsigned long long r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float2 unpack2(unsigned long long v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
    unsigned long long r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ unsigned long long add2(unsigned long long a, unsigned long long b) {
    unsigned long long r;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ unsigned long long mul2(unsigned long long a, unsigned long long b) {
    unsigned long long r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// The running maximum and sum of two rows (g and g + 8 of a warp's 16) take in NT tiles of 8 keys whose raw scores are s;
// afterwards s holds the weights 2^(score - m). Key n * 8 + 2t + e of the tiles is key `key0` + that.
template <int NT, int NO>
__device__ __forceinline__ void softmax_step(float (&s)[NT][4], float (&o)[NO][4], float (&m)[2], float (&l)[2], const int (&pos)[2],
                                             const float (&slope)[2], int key0, float scale_log2) {
    const int t = threadIdx.x & 3;
    const bool all_seen = key0 + NT * 8 - 1 <= min(pos[0], pos[1]);
    const unsigned long long sc2 = pack2(scale_log2, scale_log2);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const float b0 = -slope[h] * (float)(pos[h] - key0 - 2 * t);       // the bias of this lane's first key; a key on adds a slope
        const unsigned long long first2 = pack2(b0, b0), slope2 = pack2(slope[h], slope[h]);
        float mx = -INFINITY;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            const unsigned long long bias2 = fma2(slope2, pack2((float)(n * 8), (float)(n * 8 + 1)), first2);
            float2 v = unpack2(fma2(pack2(s[n][2 * h], s[n][2 * h + 1]), sc2, bias2));
            if (!all_seen) {
                if (key0 + n * 8 + 2 * t > pos[h]) v.x = -INFINITY;
                if (key0 + n * 8 + 2 * t + 1 > pos[h]) v.y = -INFINITY;
            }
            s[n][2 * h] = v.x; s[n][2 * h + 1] = v.y;
            mx = fmaxf(mx, fmaxf(v.x, v.y));
        }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m[h], mx);
        const float m_use = m_new == -INFINITY ? 0.f : m_new;              // a row that has seen no key yet
        if (m_new != m[h]) {
            const float alpha = ex2(m[h] - m_use);                         // 2^-inf = 0 on the first block
            m[h] = m_new;
            l[h] *= alpha;
#pragma unroll
            for (int n = 0; n < NO; ++n) { o[n][2 * h] *= alpha; o[n][2 * h + 1] *= alpha; }
        }
        const unsigned long long less2 = pack2(-m_use, -m_use);
        unsigned long long sum2 = pack2(0.f, 0.f);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            const float2 d = unpack2(add2(pack2(s[n][2 * h], s[n][2 * h + 1]), less2));
            s[n][2 * h] = ex2(d.x); s[n][2 * h + 1] = ex2(d.y);
            sum2 = add2(sum2, pack2(s[n][2 * h], s[n][2 * h + 1]));
        }
        const float2 sum = unpack2(sum2);
        l[h] += sum.x + sum.y;
    }
}
// The weights of two keys times the keys' root mean squares, as the left operand's word.
__device__ __forceinline__ unsigned weigh(float p0, float p1, unsigned long long rms2) {
    const float2 v = unpack2(mul2(pack2(p0, p1), rms2));
    return pack_bf16(v.x, v.y);
}

// ND: head size in chunks of 16 values (rounded up; the columns past dh are zeros in shared memory).
template <int ND>
struct Sizes {
    static constexpr int DP = ND * 16;
    static constexpr int ROW = DP + PAD;
    static constexpr int TILE = KB * ROW;                                  // elements of a prefill stage's keys
    static int prefill_bytes(int KV) { return (STAGES + KV) * TILE * 2 + STAGES * KB * 4; }
    // decode: a warp's stage is one page of every key/value head (keys, then their root mean squares)
    static int page_bytes(int KV) { return KV * PAGE * (ROW * 2 + 4); }
    static int merge_bytes(int warps) { return (warps * 16 * (DP + 8) + 2 * warps * 16 + 32 + 16 * DP) * 4; }
    static int decode_bytes(int KV, int warps, int stages) {
        const int a = KV * 16 * ROW * 2 + warps * stages * page_bytes(KV), b = merge_bytes(warps);
        return a > b ? a : b;
    }
};

// Keys [key0, key0 + 64) of key/value head c into a stage; with `rms` also their root mean squares. Keys past hi become
// zeros: they are masked anyway, and zeros keep the products finite whatever an earlier request left in a page. Eight threads
// copy a row; the four rows of a thread are the same row of the block's four pages (asked for a tile ahead: `pages`).
template <int ND>
__device__ __forceinline__ void load_tile(__nv_bfloat16* ks, float* rms, const MixedParams& p, const int (&pages)[KB / PAGE], int c, int key0, int hi) {
    constexpr int ROW = Sizes<ND>::ROW;
    const int row = threadIdx.x >> 3, c0 = threadIdx.x & 7, ch = p.dh / 8;
    const size_t in_page = (size_t)(c * PAGE + row) * p.dh + c0 * 8, page_size = (size_t)p.KV * PAGE * p.dh;
    __nv_bfloat16* dst = ks + row * ROW + c0 * 8;
    const bool whole = key0 + KB - 1 <= hi;
#pragma unroll
    for (int q = 0; q < KB / PAGE; ++q) {
        __nv_bfloat16* d = dst + q * PAGE * ROW;
        if (whole || key0 + q * PAGE + row <= hi) {
            const __nv_bfloat16* src = p.kc + (size_t)pages[q] * page_size + in_page;
#pragma unroll
            for (int x = 0; x < (ND + 3) / 4; ++x) if (c0 + 8 * x < ch) cp_async16(d + 64 * x, src + 64 * x);
        } else {
#pragma unroll
            for (int x = 0; x < (ND + 3) / 4; ++x) if (c0 + 8 * x < ch) *reinterpret_cast<uint4*>(d + 64 * x) = make_uint4(0u, 0u, 0u, 0u);
        }
    }
    if (rms && threadIdx.x < KB) {
        if (whole || key0 + (int)threadIdx.x <= hi)
        {
            const int lo_page = (threadIdx.x & 16) ? pages[1] : pages[0], hi_page = (threadIdx.x & 16) ? pages[3] : pages[2];
            cp_async4(rms + threadIdx.x, p.k_rms + ((size_t)((threadIdx.x & 32) ? hi_page : lo_page) * p.KV + c) * PAGE + threadIdx.x % PAGE);
        }
        else rms[threadIdx.x] = 0.f;
    }
}

template <int ND> constexpr int PREFILL_BLOCKS = ND <= 6 ? 3 : 2;          // prefill blocks an SM holds, by registers

template <int ND>
__global__ void __launch_bounds__(128, PREFILL_BLOCKS<ND>)
attention_mixed_prefill_kernel(const MixedParams p) {
    constexpr int ROW = Sizes<ND>::ROW, TILE = Sizes<ND>::TILE, DP = Sizes<ND>::DP;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(smem_raw);        // [STAGES][64][ROW]
    __nv_bfloat16* qs = ks + STAGES * TILE;                                // [KV][64][ROW]
    float* rs = reinterpret_cast<float*>(qs + p.KV * TILE);                // [STAGES][64]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int mi = lane >> 3, ri = lane & 7;                               // ldmatrix: which 8x8 matrix, which row of it
    bl_pdl_trigger();
    // late tiles of a request see the most keys: they go first, the short ones fill the tail
    const int unit = gridDim.x / p.H - 1 - blockIdx.x / p.H;
    const int r = p.work[2 * unit], tok0 = p.work[2 * unit + 1];
    const int head = blockIdx.x % p.H, own = head / (p.H / p.KV);
    const int q_begin = p.cu_q[r], q_len = p.cu_q[r + 1] - q_begin, ctx = p.ctx_len[r];
    const int* table = p.block_table + (size_t)r * p.max_pages;
    if (q_len <= tok0) {                                                   // a filler tile: the whole block leaves together
        bl_pdl_wait();
        return;
    }
    if (DP > p.dh) {                                                       // the columns past dh: zero once and for all
        const int w = DP - p.dh;
        for (int i = threadIdx.x; i < (STAGES + p.KV) * KB * w; i += 128) ks[(i / w) * ROW + p.dh + i % w] = __float2bfloat16_rn(0.f);
    }
    int pos[2], tok[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        tok[h] = tok0 + warp * 16 + g + 8 * h;
        pos[h] = tok[h] < q_len ? ctx - q_len + tok[h] : -1;               // a row that is no token sees nothing
    }
    const int hi = ctx - q_len + min(q_len, tok0 + KB) - 1;
    const int n_tiles = (hi / KB + 1) * p.KV;
    const float sl = p.slopes ? p.slopes[head] * 1.4426950408889634f : 0.f;
    const float slope[2] = {sl, sl};
    bl_pdl_wait();                                                         // queries and the newest keys come from the kernel before
    {
        const int ch = p.dh / 8;
        for (int i = threadIdx.x; i < p.KV * KB * ch; i += 128) {
            const int c = i / (KB * ch), rr = (i / ch) % KB, x = i % ch;
            __nv_bfloat16* dst = qs + c * TILE + rr * ROW + x * 8;
            if (tok0 + rr < q_len) cp_async16(dst, p.q + (((size_t)(q_begin + tok0 + rr) * p.H + head) * p.KV + c) * p.dh + x * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
        }
    }
    // the tiles in their order: key block by key block, the key/value heads in a ring that ends with `own`
    const int c_begin = own + 1 == p.KV ? 0 : own + 1;
    int left = n_tiles, i_key = 0, i_c = c_begin, i_st = 0;                // the next tile to ask for
    int pages[KB / PAGE];                                                  // ... and its pages
    auto find_pages = [&]() {
#pragma unroll
        for (int q = 0; q < KB / PAGE; ++q) pages[q] = i_key + q * PAGE <= hi ? table[i_key / PAGE + q] : 0;
    };
    find_pages();
    auto issue = [&]() {
        if (left > 0) {
            load_tile<ND>(ks + i_st * TILE, i_c == own ? rs + i_st * KB : nullptr, p, pages, i_c, i_key, hi);
            if (i_c == own) { i_key += KB; find_pages(); }
            if (++i_c == p.KV) i_c = 0;
            if (++i_st == STAGES) i_st = 0;
            --left;
        }
        cp_async_commit();
    };
#pragma unroll
    for (int i = 0; i < STAGES - 1; ++i) issue();                          // (the queries belong to the first group)
    float o[2 * ND][4];
#pragma unroll
    for (int n = 0; n < 2 * ND; ++n) { o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f; }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    float s[KB / 8][4];
#pragma unroll
    for (int n = 0; n < KB / 8; ++n) { s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f; }
    int c = c_begin, st = 0, key0 = 0;
    const __nv_bfloat16* q_row = qs + (warp * 16 + (mi & 1) * 8 + ri) * ROW + (mi >> 1) * 8;
    const __nv_bfloat16* k_row = ks + ((mi >> 1) * 8 + ri) * ROW + (mi & 1) * 8;
    const __nv_bfloat16* v_row = ks + ((mi & 1) * 8 + ri) * ROW + (mi >> 1) * 8;
    for (int i = 0; i < n_tiles; ++i) {
        cp_async_wait<STAGES - 2>();
        __syncthreads();                                                   // tile i has landed; everybody is through with tile i - 1
        issue();
        const __nv_bfloat16* kt = k_row + st * TILE;
        const __nv_bfloat16* qt = q_row + c * TILE;
#pragma unroll
        for (int kk = 0; kk < ND; ++kk) {
            unsigned a[4];
            ldmatrix_x4(a, qt + kk * 16);
#pragma unroll
            for (int np = 0; np < KB / 16; ++np) {
                unsigned b[4];
                ldmatrix_x4(b, kt + np * 16 * ROW + kk * 16);
                mma_bf16(s[2 * np], a, b[0], b[1]);
                mma_bf16(s[2 * np + 1], a, b[2], b[3]);
            }
        }
        if (c == own) {                                                    // the block's scores are complete, its values are this tile
            softmax_step<KB / 8, 2 * ND>(s, o, m, l, pos, slope, key0, p.scale_log2);
            const float* rt = rs + st * KB + 2 * t;
            const __nv_bfloat16* vt = v_row + st * TILE;
#pragma unroll
            for (int kk = 0; kk < KB / 16; ++kk) {
                const unsigned long long r0 = *reinterpret_cast<const unsigned long long*>(rt + kk * 16);
                const unsigned long long r1 = *reinterpret_cast<const unsigned long long*>(rt + kk * 16 + 8);
                unsigned a[4];
                a[0] = weigh(s[2 * kk][0], s[2 * kk][1], r0);
                a[1] = weigh(s[2 * kk][2], s[2 * kk][3], r0);
                a[2] = weigh(s[2 * kk + 1][0], s[2 * kk + 1][1], r1);
                a[3] = weigh(s[2 * kk + 1][2], s[2 * kk + 1][3], r1);
#pragma unroll
                for (int np = 0; np < ND; ++np) {
                    unsigned b[4];
                    ldmatrix_x4_trans(b, vt + kk * 16 * ROW + np * 16);
                    mma_bf16(o[2 * np], a, b[0], b[1]);
                    mma_bf16(o[2 * np + 1], a, b[2], b[3]);
                }
            }
            key0 += KB;
#pragma unroll
            for (int n = 0; n < KB / 8; ++n) { s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f; }
        }
        if (++c == p.KV) c = 0;
        if (++st == STAGES) st = 0;
    }
    cp_async_wait<0>();
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
        if (pos[h] < 0) continue;
        const float inv = l[h] > 0.f ? 1.0f / l[h] : 0.f;
        const size_t row = (size_t)(q_begin + tok[h]);
        __nv_bfloat16* op = p.out + (row * p.H + head) * p.dh + 2 * t;
        const float* gp = p.gate ? p.gate + row * p.ld_gate + (size_t)head * p.dh + 2 * t : nullptr;
#pragma unroll
        for (int n = 0; n < 2 * ND; ++n) {
            if (n * 8 >= p.dh) break;
            float a = o[n][2 * h] * inv, b = o[n][2 * h + 1] * inv;
            if (gp) {
                const float2 z = *reinterpret_cast<const float2*>(gp + n * 8);
                a *= sigmoid(z.x); b *= sigmoid(z.y);
            }
            *reinterpret_cast<unsigned*>(op + n * 8) = pack_bf16(a, b);
        }
    }
}

__device__ __forceinline__ void cluster_sync_all() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ uint32_t peer_shared(uint32_t local, uint32_t rank) {
    uint32_t r;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(local), "r"(rank));
    return r;
}
__device__ __forceinline__ float4 ld_cluster_f4(uint32_t a) {
    float4 v;
    asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(a) : "memory");
    return v;
}
__device__ __forceinline__ float2 ld_cluster_f2(uint32_t a) {
    float2 v;
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(a) : "memory");
    return v;
}

// One warp copies the page that holds keys [key0, key0 + 16), of every key/value head, into a stage of its own. Eight lanes
// copy a row; all rows of a page lie together.
template <int ND>
__device__ __forceinline__ void load_page(__nv_bfloat16* ks, float* rms, const MixedParams& p, const int* table, int key0, int hi) {
    constexpr int ROW = Sizes<ND>::ROW;
    const int lane = threadIdx.x & 31, ch = p.dh / 8, c0 = lane & 7;
    const int live = min(PAGE, hi - key0 + 1);                             // keys of the page that exist (may be <= 0)
    const size_t page = live > 0 ? (size_t)table[key0 / PAGE] : 0;
    const int rows = p.KV * PAGE, step = 4 * p.dh;
    const __nv_bfloat16* src = p.kc + (page * rows + (lane >> 3)) * p.dh + c0 * 8;
    __nv_bfloat16* dst = ks + (lane >> 3) * ROW + c0 * 8;
    const float* rsrc = p.k_rms + page * rows;
    if (live == PAGE) {
#pragma unroll 4
        for (int rr = 0; rr < rows; rr += 4, src += step, dst += 4 * ROW) {
#pragma unroll
            for (int x = 0; x < (ND + 3) / 4; ++x) if (c0 + 8 * x < ch) cp_async16(dst + 64 * x, src + 64 * x);
        }
        for (int rr = lane * 4; rr < rows; rr += 128) cp_async16(rms + rr, rsrc + rr);
        return;
    }
    for (int rr = lane >> 3; rr < rows; rr += 4, src += step, dst += 4 * ROW) {
#pragma unroll
        for (int x = 0; x < (ND + 3) / 4; ++x) {
            if (c0 + 8 * x >= ch) continue;
            if (rr % PAGE < live) cp_async16(dst + 64 * x, src + 64 * x);
            else *reinterpret_cast<uint4*>(dst + 64 * x) = make_uint4(0u, 0u, 0u, 0u);
        }
    }
    for (int rr = lane; rr < rows; rr += 32) {
        if (rr % PAGE < live) cp_async4(rms + rr, rsrc + rr);
        else rms[rr] = 0.f;
    }
}

template <int ND, int WSTAGES>
__global__ void __launch_bounds__(MAX_DECODE_WARPS * 32, ND <= 4 ? 2 : 1)
attention_mixed_decode_kernel(const MixedParams p) {
    constexpr int ROW = Sizes<ND>::ROW, DP = Sizes<ND>::DP;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int warps = blockDim.x >> 5;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int mi = lane >> 3, ri = lane & 7;
    const int stage_elems = p.KV * PAGE * ROW, stage_bytes = p.KV * PAGE * (ROW * 2 + 4);
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);        // [KV][16][ROW]
    unsigned char* ring = smem_raw + (size_t)p.KV * 16 * ROW * 2 + (size_t)warp * WSTAGES * stage_bytes;
    auto stage_keys = [&](int i) { return reinterpret_cast<__nv_bfloat16*>(ring + (size_t)i * stage_bytes); };
    auto stage_rms = [&](int i) { return reinterpret_cast<float*>(ring + (size_t)i * stage_bytes + (size_t)stage_elems * 2); };
    bl_pdl_trigger();
    const int r = p.work[blockIdx.z], head0 = blockIdx.y * 16, split = blockIdx.x, G = p.H / p.KV;
    const int q_begin = p.cu_q[r], q_len = p.cu_q[r + 1] - q_begin, ctx = p.ctx_len[r];
    const int* table = p.block_table + (size_t)r * p.max_pages;
    const int hi = ctx - 1, span = warps * PAGE;                           // keys a block takes at a time
    const int rows_here = min(16, p.H - head0);
    int b_begin = 0, b_end = q_len > 0 ? hi / span + 1 : 0;
    {
        const int per = (b_end + p.n_splits - 1) / p.n_splits;
        b_begin = min(split * per, b_end);
        b_end = min(b_end, b_begin + per);
    }
    const int nb = b_end - b_begin;
    if (DP > p.dh) {                                                       // the columns past dh: zero once and for all
        const int w = DP - p.dh;
        for (int i = threadIdx.x; i < p.KV * 16 * w; i += blockDim.x) qs[(i / w) * ROW + p.dh + i % w] = __float2bfloat16_rn(0.f);
        for (int st = 0; st < WSTAGES; ++st)
            for (int i = lane; i < p.KV * PAGE * w; i += 32) stage_keys(st)[(i / w) * ROW + p.dh + i % w] = __float2bfloat16_rn(0.f);
    }
    auto key_of = [&](int i) { return (b_begin + i) * span + warp * PAGE; };
    int issued = 0;
    // pages of earlier tokens do not depend on the kernel before
    while (issued < WSTAGES && issued < nb && key_of(issued) + PAGE <= hi) {
        load_page<ND>(stage_keys(issued), stage_rms(issued), p, table, key_of(issued), hi);
        cp_async_commit();
        ++issued;
    }
    int pos[2];
    float slope[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const bool live = g + 8 * h < rows_here && q_len > 0;
        pos[h] = live ? hi : -1;
        slope[h] = live && p.slopes ? p.slopes[head0 + g + 8 * h] * 1.4426950408889634f : 0.f;
    }
    bl_pdl_wait();                                                         // queries and the newest keys come from the kernel before
    if (q_len > 0) {
        const int ch = p.dh / 8;
        for (int i = threadIdx.x; i < p.KV * 16 * ch; i += blockDim.x) {
            const int c = i / (16 * ch), rr = (i / ch) % 16, x = i % ch;
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (rr < rows_here) v = *reinterpret_cast<const uint4*>(p.q + (((size_t)q_begin * p.H + head0 + rr) * p.KV + c) * p.dh + x * 8);
            *reinterpret_cast<uint4*>(qs + (c * 16 + rr) * ROW + x * 8) = v;
        }
    }
    while (issued < WSTAGES && issued < nb) {
        load_page<ND>(stage_keys(issued), stage_rms(issued), p, table, key_of(issued), hi);
        cp_async_commit();
        ++issued;
    }
    __syncthreads();                                                       // the queries are there
    const int c_first = head0 / G, c_last = (head0 + rows_here - 1) / G;   // the key/value heads whose values these rows take
    const int kv0 = (head0 + g) / G, kv1 = (head0 + g + 8) / G;
    float o[2 * ND][4];
#pragma unroll
    for (int n = 0; n < 2 * ND; ++n) { o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f; }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    const __nv_bfloat16* q_row = qs + ((mi & 1) * 8 + ri) * ROW + (mi >> 1) * 8;
    const __nv_bfloat16* k_row = stage_keys(0) + ((mi >> 1) * 8 + ri) * ROW + (mi & 1) * 8;
    const __nv_bfloat16* v_row = stage_keys(0) + ((mi & 1) * 8 + ri) * ROW + (mi >> 1) * 8;
    for (int i = 0; i < nb; ++i) {
        const int pending = issued - (i + 1);
        if (pending >= 2) cp_async_wait<2>(); else if (pending == 1) cp_async_wait<1>(); else cp_async_wait<0>();
        __syncwarp();
        const float* rt = stage_rms(i % WSTAGES);
        // two sets of sums (even and odd chunks of the head size), so that a product does not wait for the one before it
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}}, s2[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        const __nv_bfloat16* qt = q_row;
        const __nv_bfloat16* kt = k_row + (size_t)(i % WSTAGES) * (stage_bytes / 2);
#pragma unroll 2
        for (int c = 0; c < p.KV; ++c, qt += 16 * ROW, kt += PAGE * ROW) {
#pragma unroll
            for (int kk = 0; kk < ND; ++kk) {
                unsigned a[4], b[4];
                ldmatrix_x4(a, qt + kk * 16);
                ldmatrix_x4(b, kt + kk * 16);
                mma_bf16(kk & 1 ? s2[0] : s[0], a, b[0], b[1]);
                mma_bf16(kk & 1 ? s2[1] : s[1], a, b[2], b[3]);
            }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) { s[0][e] += s2[0][e]; s[1][e] += s2[1][e]; }
        softmax_step<2, 2 * ND>(s, o, m, l, pos, slope, key_of(i), p.scale_log2);
        const __nv_bfloat16* vt = v_row + (size_t)(i % WSTAGES) * (stage_bytes / 2);
        for (int c = c_first; c <= c_last; ++c) {
            const unsigned long long r0 = *reinterpret_cast<const unsigned long long*>(rt + c * PAGE + 2 * t);
            const unsigned long long r1 = *reinterpret_cast<const unsigned long long*>(rt + c * PAGE + 8 + 2 * t);
            unsigned a[4];
            a[0] = kv0 == c ? weigh(s[0][0], s[0][1], r0) : 0u;
            a[1] = kv1 == c ? weigh(s[0][2], s[0][3], r0) : 0u;
            a[2] = kv0 == c ? weigh(s[1][0], s[1][1], r1) : 0u;
            a[3] = kv1 == c ? weigh(s[1][2], s[1][3], r1) : 0u;
#pragma unroll
            for (int np = 0; np < ND; ++np) {
                unsigned b[4];
                ldmatrix_x4_trans(b, vt + c * PAGE * ROW + np * 16);
                mma_bf16(o[2 * np], a, b[0], b[1]);
                mma_bf16(o[2 * np + 1], a, b[2], b[3]);
            }
        }
        __syncwarp();
        if (issued < nb) {                                                 // the stage just used takes the page WSTAGES blocks on
            load_page<ND>(stage_keys(i % WSTAGES), stage_rms(i % WSTAGES), p, table, key_of(issued), hi);
            cp_async_commit();
            ++issued;
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    }
    // merge the warps (same rows, different keys), every sum scaled to the rows' common maximum first
    __syncthreads();
    constexpr int SO = DP + 8;
    float* so = reinterpret_cast<float*>(smem_raw);                        // [warps][16][SO]
    float* sm = so + warps * 16 * SO;                                      // [warps][16]
    float* sl = sm + warps * 16;                                           // [warps][16]
    float* cp_ml = sl + warps * 16;                                        // [16][max, sum] of this slice, for the cluster's merge
    float* cp_o = cp_ml + 32;                                              // [16][DP]
    if (t == 0) {
#pragma unroll
        for (int h = 0; h < 2; ++h) { sm[warp * 16 + g + 8 * h] = m[h]; sl[warp * 16 + g + 8 * h] = l[h]; }
    }
    __syncthreads();
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int row = g + 8 * h;
        float M = -INFINITY;
        for (int w = 0; w < warps; ++w) M = fmaxf(M, sm[w * 16 + row]);
        const float f = m[h] == -INFINITY ? 0.f : exp2f(m[h] - M);
        if (t == 0) sl[warp * 16 + row] = l[h] * f;
        float* dst = so + (warp * 16 + row) * SO + 2 * t;
#pragma unroll
        for (int n = 0; n < 2 * ND; ++n) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[n][2 * h] * f, o[n][2 * h + 1] * f);
    }
    __syncthreads();
    const int d4 = p.dh / 4;
    auto finish = [&](int row, int d, float4 v, float L) {
        const float inv = L > 0.f ? 1.0f / L : 0.f;
        const int hd = head0 + row;
        v.x *= inv; v.y *= inv; v.z *= inv; v.w *= inv;
        if (p.gate) {
            const float* gp = p.gate + (size_t)q_begin * p.ld_gate + (size_t)hd * p.dh + d;
            v.x *= sigmoid(gp[0]); v.y *= sigmoid(gp[1]); v.z *= sigmoid(gp[2]); v.w *= sigmoid(gp[3]);
        }
        *reinterpret_cast<uint2*>(p.out + ((size_t)q_begin * p.H + hd) * p.dh + d) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
    };
    if (q_len > 0) {
        for (int i = threadIdx.x; i < rows_here * d4; i += blockDim.x) {
            const int row = i / d4, d = (i % d4) * 4;
            float M = -INFINITY, L = 0.f;
            float4 O = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int w = 0; w < warps; ++w) {
                M = fmaxf(M, sm[w * 16 + row]);
                L += sl[w * 16 + row];
                const float4 a = *reinterpret_cast<const float4*>(so + (w * 16 + row) * SO + d);
                O.x += a.x; O.y += a.y; O.z += a.z; O.w += a.w;
            }
            if (p.n_splits == 1) {
                finish(row, d, O, L);
            } else {
                *reinterpret_cast<float4*>(cp_o + row * DP + d) = O;
                if (d == 0) *reinterpret_cast<float2*>(cp_ml + row * 2) = make_float2(M, L);
            }
        }
    }
    if (p.n_splits == 1 || q_len <= 0) return;                             // (the blocks of a cluster share a request: they leave together)
    cluster_sync_all();                                                    // every slice's partial result is written
    const uint32_t ml_base = (uint32_t)__cvta_generic_to_shared(cp_ml), o_base = (uint32_t)__cvta_generic_to_shared(cp_o);
    for (int i = split + (int)threadIdx.x * p.n_splits; i < rows_here * d4; i += blockDim.x * p.n_splits) {
        const int row = i / d4, d = (i % d4) * 4;
        float2 ml[MAX_CLUSTER];
        float4 po[MAX_CLUSTER];
#pragma unroll
        for (int q = 0; q < MAX_CLUSTER; ++q) {                            // all loads on their way before any is used
            if (q >= p.n_splits) break;
            ml[q] = ld_cluster_f2(peer_shared(ml_base + (uint32_t)(row * 2) * 4u, (uint32_t)q));
            po[q] = ld_cluster_f4(peer_shared(o_base + (uint32_t)(row * DP + d) * 4u, (uint32_t)q));
        }
        float M = -INFINITY, L = 0.f;
#pragma unroll
        for (int q = 0; q < MAX_CLUSTER; ++q) { if (q >= p.n_splits) break; M = fmaxf(M, ml[q].x); }
        float4 O = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int q = 0; q < MAX_CLUSTER; ++q) {
            if (q >= p.n_splits) break;
            const float f = ml[q].x == -INFINITY ? 0.f : exp2f(ml[q].x - M);
            L += ml[q].y * f;
            O.x += po[q].x * f; O.y += po[q].y * f; O.z += po[q].z * f; O.w += po[q].w * f;
        }
        finish(row, d, O, L);
    }
    cluster_sync_all();                                                    // no block leaves while another may still read its partial result
}

constexpr int SMEM_LIMIT = 227 * 1024;

template <int ND>
bool decode_shape(int KV, int* warps, int* stages) {
    // eight warps with three stages each where two such blocks fit an SM, else what fits
    if (Sizes<ND>::decode_bytes(KV, 8, 3) <= SMEM_LIMIT / 2) { *warps = 8; *stages = 3; return true; }
    const int shapes[6][2] = {{8, 2}, {4, 3}, {4, 2}, {2, 3}, {2, 2}, {1, 2}};
    for (const auto& s : shapes)
        if (Sizes<ND>::decode_bytes(KV, s[0], s[1]) <= SMEM_LIMIT) { *warps = s[0]; *stages = s[1]; return true; }
    return false;
}

template <int ND>
int launch_prefill(const MixedParams& p, int n_tiles, cudaStream_t s) {
    // A launch whose blocks are all resident at once cannot even out its long and short blocks. So a launch of few blocks asks for
    // more shared memory than it uses, which leaves two blocks an SM, and the rest start as places become free (2,048 tokens, 14
    // heads of 64 values: 81 us with two blocks an SM, 101 with three, 110 with four; 4,096 tokens want three).
    int bytes = Sizes<ND>::prefill_bytes(p.KV);
    if ((long long)n_tiles * p.H * 2 < 148LL * 3 * PREFILL_BLOCKS<ND> && bytes < SMEM_LIMIT / 3) bytes = SMEM_LIMIT / 3;
    static thread_local int allowed = 0;
    if (bytes > allowed) {
        BL_CUDA(cudaFuncSetAttribute(attention_mixed_prefill_kernel<ND>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
        allowed = bytes;
    }
    BL_CUDA(bl_launch_dependent(attention_mixed_prefill_kernel<ND>, dim3(n_tiles * p.H), dim3(128), (size_t)bytes, s, p));
    BL_CHECK_LAUNCH("bl_attention_mixed_prefill");
    return 0;
}

template <int ND, int WSTAGES>
int launch_decode(const MixedParams& p, int n, int warps, cudaStream_t s) {
    const int bytes = Sizes<ND>::decode_bytes(p.KV, warps, WSTAGES);
    static thread_local int allowed = 0;
    if (bytes > allowed) {
        BL_CUDA(cudaFuncSetAttribute(attention_mixed_decode_kernel<ND, WSTAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
        BL_CUDA(cudaFuncSetAttribute(attention_mixed_decode_kernel<ND, WSTAGES>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
        allowed = bytes;
    }
    const dim3 grid(p.n_splits, (p.H + 15) / 16, n);
    if (p.n_splits > 1)
        BL_CUDA(bl_launch_dependent_clusters(attention_mixed_decode_kernel<ND, WSTAGES>, grid, dim3(warps * 32), (size_t)bytes, s, (unsigned)p.n_splits, p));
    else
        BL_CUDA(bl_launch_dependent(attention_mixed_decode_kernel<ND, WSTAGES>, grid, dim3(warps * 32), (size_t)bytes, s, p));
    BL_CHECK_LAUNCH("bl_attention_mixed_decode");
    return 0;
}

// Chunks of 16 values of the build that takes head size dh (0: none).
int chunks_of(int dh) {
    if (dh <= 0 || dh % 8 != 0) return 0;
    for (int nd : {1, 2, 3, 4, 6, 8}) if (dh <= nd * 16) return nd;
    return 0;
}

#define BL_BY_CHUNKS(ND_VALUE, OTHERWISE, ...) \
    switch (ND_VALUE) { \
        case 1: { constexpr int ND = 1; __VA_ARGS__; break; } case 2: { constexpr int ND = 2; __VA_ARGS__; break; } \
        case 3: { constexpr int ND = 3; __VA_ARGS__; break; } case 4: { constexpr int ND = 4; __VA_ARGS__; break; } \
        case 6: { constexpr int ND = 6; __VA_ARGS__; break; } case 8: { constexpr int ND = 8; __VA_ARGS__; break; } \
        default: OTHERWISE; }

template <int ND>
int decode_resident(int KV) {
    int warps = 0, stages = 0;
    if (!decode_shape<ND>(KV, &warps, &stages)) return 0;
    const int bytes = Sizes<ND>::decode_bytes(KV, warps, stages);
    int dev = 0, sms = 0;
    if (cudaGetDevice(&dev) != cudaSuccess) return 0;
    if (cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) return 0;
    const int by_smem = SMEM_LIMIT / (bytes + 1024), by_regs = (ND <= 4 ? 16 : 8) / warps;
    const int per_sm = by_smem < by_regs ? by_smem : by_regs;
    return sms * (per_sm < 1 ? 1 : per_sm);
}

int check(const char* who, const MixedParams& p, int page_size) {
    if (p.H <= 0 || p.KV <= 0 || p.H % p.KV != 0) BL_FAIL("%s: %d heads cannot share %d key/value heads", who, p.H, p.KV);
    if (!bl_attention_mixed_supported(p.KV, p.dh, page_size)) BL_FAIL("%s: %d key/value heads of %d values in pages of %d are not built; use the plain kernel", who, p.KV, p.dh, page_size);
    if (p.max_pages <= 0) BL_FAIL("%s: bad table width", who);
    if ((((uintptr_t)p.q | (uintptr_t)p.kc | (uintptr_t)p.out) & 15) != 0) BL_FAIL("%s: queries, keys and output must be 16-byte aligned", who);
    if (p.gate && ((((uintptr_t)p.gate) & 7) != 0 || p.ld_gate % 2 != 0)) BL_FAIL("%s: the gate's rows must be 8-byte aligned", who);
    return 0;
}

MixedParams params(const void* q, const void* k_cache, const float* k_rms, const int* cu_q, const int* ctx_len, const int* block_table,
                   int max_pages, const int* work, void* out, int H, int KV, int dh, float scale, const float* slopes,
                   const float* gate, int ld_gate, int n_splits) {
    MixedParams p;
    p.q = (const __nv_bfloat16*)q; p.kc = (const __nv_bfloat16*)k_cache; p.k_rms = k_rms; p.out = (__nv_bfloat16*)out;
    p.cu_q = cu_q; p.ctx_len = ctx_len; p.block_table = block_table; p.max_pages = max_pages; p.work = work;
    p.slopes = slopes; p.gate = gate; p.ld_gate = ld_gate; p.H = H; p.KV = KV; p.dh = dh; p.n_splits = n_splits;
    p.scale_log2 = scale * 1.4426950408889634f;
    return p;
}

}  // namespace

extern "C" int bl_mixed_prep(const float* proj, int ld, int off_k, const float* talk, float eps, const int* positions, const int* tok_req,
                             const int* block_table, int max_pages, void* q_out, void* k_cache, float* k_rms, int rms_stride, int dtype,
                             int T, int H, int KV, int dh, int page_size, void* stream) {
    if (T <= 0) return 0;
    if (H <= 0 || KV <= 0 || H % KV != 0 || dh <= 0) BL_FAIL("bl_mixed_prep: %d heads of %d values on %d key/value heads", H, dh, KV);
    if (off_k < H * dh || off_k + KV * dh > ld || page_size <= 0 || max_pages <= 0) BL_FAIL("bl_mixed_prep: keys from column %d do not fit rows of %d", off_k, ld);
    if (k_cache && (!k_rms || rms_stride <= 0)) BL_FAIL("bl_mixed_prep: keys without a place for their root mean squares");
    const int per_block = T <= PREP_FEW_ROWS ? 4 : (H + 3) & ~3;
    const size_t smem = (size_t)(((H * dh + 3) & ~3) + per_block * H) * sizeof(float);
    if (smem > 160 * 1024) BL_FAIL("bl_mixed_prep: %d heads of %d values are too many for shared memory", H, dh);
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 grid(T, (H + per_block - 1) / per_block);
#define BL_GO(TT) do { \
        if (smem > 48 * 1024) BL_CUDA(cudaFuncSetAttribute(mixed_prep_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        BL_CUDA(bl_launch_dependent(mixed_prep_kernel<TT>, grid, dim3(PREP_THREADS), smem, s, proj, ld, off_k, talk, eps, positions, tok_req, \
                                    block_table, max_pages, (TT*)q_out, (TT*)k_cache, k_rms, rms_stride, H, KV, dh, page_size, per_block)); } while (0)
    if (dtype == BL_F32) BL_GO(float);
    else if (dtype == BL_BF16) BL_GO(__nv_bfloat16);
    else BL_FAIL("bl_mixed_prep: unknown dtype %d", dtype);
#undef BL_GO
    BL_CHECK_LAUNCH("bl_mixed_prep");
    return 0;
}

extern "C" int bl_attention_mixed_plain(const void* q, const void* k_cache, const float* k_rms, int rms_stride, int dtype, const int* tok_req,
                                        const int* cu_q, const int* ctx_len, const int* block_table, int max_pages, const float* slopes,
                                        const float* gate, int ld_gate, void* out, int T, int H, int KV, int dh, int page_size,
                                        float scale, void* stream) {
    if (T <= 0) return 0;
    if (H <= 0 || KV <= 0 || H % KV != 0 || dh <= 0 || dh > MAX_DH) BL_FAIL("bl_attention_mixed_plain: %d heads of %d values on %d key/value heads (head size up to %d)", H, dh, KV, MAX_DH);
    if (page_size <= 0 || max_pages <= 0) BL_FAIL("bl_attention_mixed_plain: bad page size or table width");
    const size_t smem = (size_t)PLAIN_WARPS * KV * dh * sizeof(float);
    if (smem > SMEM_LIMIT) BL_FAIL("bl_attention_mixed_plain: %d key/value heads of %d values are too many for shared memory", KV, dh);
    cudaStream_t s = (cudaStream_t)stream;
    const int blocks = (T * H + PLAIN_WARPS - 1) / PLAIN_WARPS;
#define BL_GO(TT) do { \
        if (smem > 48 * 1024) BL_CUDA(cudaFuncSetAttribute(attention_mixed_plain_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        BL_CUDA(bl_launch_dependent(attention_mixed_plain_kernel<TT>, dim3(blocks), dim3(PLAIN_WARPS * 32), smem, s, (const TT*)q, (const TT*)k_cache, \
                                    k_rms, rms_stride, tok_req, cu_q, ctx_len, block_table, max_pages, slopes, gate, ld_gate, (TT*)out, T, H, KV, \
                                    dh, page_size, scale)); } while (0)
    if (dtype == BL_F32) BL_GO(float);
    else if (dtype == BL_BF16) BL_GO(__nv_bfloat16);
    else BL_FAIL("bl_attention_mixed_plain: unknown dtype %d", dtype);
#undef BL_GO
    BL_CHECK_LAUNCH("bl_attention_mixed_plain");
    return 0;
}

extern "C" int bl_attention_mixed_supported(int KV, int dh, int page_size) {
    if (page_size != PAGE || KV <= 0) return 0;
    int warps, stages;
    BL_BY_CHUNKS(chunks_of(dh), return 0, return Sizes<ND>::prefill_bytes(KV) <= SMEM_LIMIT && decode_shape<ND>(KV, &warps, &stages))
    return 0;
}

extern "C" int bl_attention_mixed_decode_resident_blocks(int KV, int dh) {
    BL_BY_CHUNKS(chunks_of(dh), return 0, return decode_resident<ND>(KV))
    return 0;
}

extern "C" int bl_attention_mixed_prefill(const void* q, const void* k_cache, const float* k_rms, const int* cu_q, const int* ctx_len,
                                          const int* block_table, int max_pages, const int* tiles, int n_tiles, void* out, int H, int KV,
                                          int dh, int page_size, float scale, const float* slopes, const float* gate, int ld_gate,
                                          void* stream) {
    if (n_tiles <= 0) return 0;
    const MixedParams p = params(q, k_cache, k_rms, cu_q, ctx_len, block_table, max_pages, tiles, out, H, KV, dh, scale, slopes, gate, ld_gate, 1);
    if (check("bl_attention_mixed_prefill", p, page_size)) return 1;
    if ((long long)n_tiles * H > 2147483647LL) BL_FAIL("bl_attention_mixed_prefill: %d tiles x %d heads are more blocks than a launch takes", n_tiles, H);
    BL_BY_CHUNKS(chunks_of(dh), BL_FAIL("bl_attention_mixed_prefill: head size %d", dh), return launch_prefill<ND>(p, n_tiles, (cudaStream_t)stream))
    return 0;
}

extern "C" int bl_attention_mixed_decode(const void* q, const void* k_cache, const float* k_rms, const int* cu_q, const int* ctx_len,
                                         const int* block_table, int max_pages, const int* reqs, int n, int n_splits, void* out, int H,
                                         int KV, int dh, int page_size, float scale, const float* slopes, const float* gate, int ld_gate,
                                         void* stream) {
    if (n <= 0) return 0;
    if (n_splits < 1 || n_splits > MAX_CLUSTER || n > 65535) BL_FAIL("bl_attention_mixed_decode: %d requests in %d slices (up to %d)", n, n_splits, MAX_CLUSTER);
    const MixedParams p = params(q, k_cache, k_rms, cu_q, ctx_len, block_table, max_pages, reqs, out, H, KV, dh, scale, slopes, gate, ld_gate, n_splits);
    if (check("bl_attention_mixed_decode", p, page_size)) return 1;
    int warps = 0, stages = 0;
    BL_BY_CHUNKS(chunks_of(dh), BL_FAIL("bl_attention_mixed_decode: head size %d", dh),
                 decode_shape<ND>(KV, &warps, &stages);
                 return stages == 3 ? launch_decode<ND, 3>(p, n, warps, (cudaStream_t)stream) : launch_decode<ND, 2>(p, n, warps, (cudaStream_t)stream))
    return 0;
}
