// Attention over a latent cache: one normed vector c and one rotated key part per position, shared by all heads (lv_latent_args).
//
// Absorbed form, f32 arithmetic on CUDA cores (decoded tokens, 32-bit caches, short portions, odd sizes).  One token is one launch
// where its sizes fit, latent_step_kernel: a cluster of eight CTAs has one or a few heads, and every CTA an eighth of their rows of
// W_uk (in shared memory before the previous kernel has finished) and W_uv and of the visible cache rows.  The CTAs exchange their parts of W_uk^T q, and later of the weighted sums of c, through distributed shared memory.  Otherwise:
//   latent_query_kernel   per head u = scale * W_uk^T q and the rotated part of q; one more CTA norms, rotates and appends the
//                         token's own cache row
//   latent_decode_kernel  up to eight heads of one token against a share of the visible rows, in chunks of 32 with an online
//                         softmax.  A chunk is fetched to shared memory once and serves as keys (c and rotated part) and as
//                         values (c).  A token's shares are spread over CTAs that leave maximum, sum and weighted sum of c
//   latent_value_kernel   combines a head's shares with its sink and multiplies by W_uv
// Expanded form (prompts with bfloat16 caches): keys and values of the visible rows by lv_gemm_bf16_window, attention by the tensor
// cores (attention_gqa_tc.cu); latent_append_kernel writes the cache rows first.
#include <cuda_bf16.h>
#include <math.h>

#include <algorithm>

#include "attention_gqa.cuh"
#include "common.cuh"
#include "ctx.h"

namespace lv {

constexpr int kLtThreads = 256, kLtWarps = 8;
constexpr int kLtHeads = 8;              // heads of a CTA
constexpr int kLtChunk = 32;             // cache rows of a chunk: a softmax lane each, four per warp
constexpr int kLtQueryCols = 128;        // columns of u that a CTA of latent_query_kernel forms
constexpr int kLtQueryRows = 8;          // rows of W_uk in flight per thread
constexpr int kLtValueRows = 32;         // rows of W_uv per CTA
constexpr uint32_t kLtMaxSplits = 64, kLtMaxRank = 1024;
constexpr int kLtCluster = 8;            // CTAs of a cluster of latent_step_kernel
constexpr int kLtStepThreads = 512, kLtStepWarps = kLtStepThreads / 32, kLtStepChunk = 4 * kLtStepWarps;
constexpr uint32_t kLtStepKeys = 4096;   // most visible rows that a cluster walks; more are spread over more CTAs
constexpr size_t kLtExpandBytes = size_t(512) << 20;      // keys and values expanded at a time; more heads take several passes
constexpr uint32_t kLtAbsorbedBatch = 4;                  // portions up to this size are not worth expanding the window for

struct LatentParams {
    lv_latent_args a;
    uint32_t rank_p, rot_p, ld;          // padded to 8; ld = rank_p + rot_p
    uint32_t head_blocks, splits, part;  // part: floats of one share, {maximum, sum, -, -, c[rank_p]}
    uint32_t col_blocks, buffers;
    uint32_t rows_k, rows_v;             // latent_step_kernel: rows of W_uk and W_uv per CTA
    float* u;                            // [batch][heads][ld]
    float* shares;                       // [batch][heads][splits][part]
    uint32_t out_bf16;
    uint32_t* err;
};

template <typename CT> __device__ __forceinline__ CT lt_cast(float v);
template <> __device__ __forceinline__ float lt_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 lt_cast<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// four consecutive cache values from shared memory
__device__ __forceinline__ void lt_load4(float (&v)[4], const float* p) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void lt_load4(float (&v)[4], const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(u.x << 16); v[1] = __uint_as_float(u.x & 0xffff0000u);
    v[2] = __uint_as_float(u.y << 16); v[3] = __uint_as_float(u.y & 0xffff0000u);
}
__device__ __forceinline__ float2 lt_load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 lt_load2(const __nv_bfloat16* p) {
    const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
    return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
}

// first visible position of position P
__device__ __forceinline__ uint32_t lt_first(uint32_t P, uint32_t window) { return window != 0 && P + 1 > window ? P + 1 - window : 0; }

// value i of the rotated vector v (rot values, the leading 2 * pairs of them turn)
__device__ __forceinline__ float lt_rotated(const float* v, const float* angles, uint32_t i, uint32_t pairs) {
    if (i >= 2 * pairs) return v[i];
    const float2 cs = *reinterpret_cast<const float2*>(angles + (i & ~1u));
    return (i & 1u) ? v[i] * cs.x + v[i - 1] * cs.y : v[i] * cs.x - v[i + 1] * cs.y;
}

// Norms and rotates the cache row of token t (a whole CTA of THREADS): to `dst` and, where given, to `copy`.
template <typename CT, int THREADS>
__device__ __forceinline__ void lt_row(const LatentParams& p, uint32_t t, float* scratch, CT* dst, CT* copy) {
    const lv_latent_args& a = p.a;
    const float* d = a.dkv + size_t(t) * a.dkv_ld;
    constexpr int kPer = kLtMaxRank / THREADS;
    float v[kPer], part = 0.f;
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const uint32_t i = threadIdx.x + k * THREADS;
        v[k] = i < a.kv_rank ? d[i] : 0.f;
        part = fmaf(v[k], v[k], part);
    }
    const float r = 1.f / sqrtf(block_sum(part, scratch) / float(a.kv_rank) + a.eps);
    auto put = [&](uint32_t i, float x) {
        const CT e = lt_cast<CT>(x);
        dst[i] = e;
        if (copy != nullptr) copy[i] = e;
    };
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const uint32_t i = threadIdx.x + k * THREADS;
        if (i < p.rank_p) put(i, i < a.kv_rank ? v[k] * r * a.kv_norm[i] : 0.f);
    }
    for (uint32_t i = threadIdx.x; i < p.rot_p; i += THREADS)
        put(p.rank_p + i, i < a.rot ? lt_rotated(d + a.kv_rank, a.angles + size_t(t) * a.angle_ld, i, a.angle_pairs) : 0.f);
}

template <typename CT>
__device__ __forceinline__ void lt_append(const LatentParams& p, uint32_t t, float* scratch) {
    const uint32_t row = *p.a.pos + t;
    if (row < p.a.ctx_rows) lt_row<CT, kLtThreads>(p, t, scratch, static_cast<CT*>(p.a.cache) + size_t(row) * p.ld, static_cast<CT*>(nullptr));
    else if (threadIdx.x == 0) atomicOr(p.err, ERR_BAD_INDEX);
}

template <typename CT>
__global__ void __launch_bounds__(kLtThreads) latent_append_kernel(const LatentParams p) {
    pdl_launch_dependents();
    __shared__ float scratch[64];
    pdl_wait();
    lt_append<CT>(p, blockIdx.x, scratch);
}

// blockIdx.x: heads * col_blocks CTAs of 128 columns of u, then (with dkv) the CTA that appends; blockIdx.y = token
template <typename CT>
__global__ void __launch_bounds__(kLtThreads) latent_query_kernel(const LatentParams p) {
    pdl_launch_dependents();
    __shared__ float scratch[64], s_q[16 * kLtQueryRows], s_sum[kLtWarps][kLtQueryCols];
    const lv_latent_args& a = p.a;
    const uint32_t t = blockIdx.y;
    if (blockIdx.x == a.heads * p.col_blocks) {
        pdl_wait();
        lt_append<CT>(p, t, scratch);
        return;
    }
    const uint32_t h = blockIdx.x / p.col_blocks, block = blockIdx.x - h * p.col_blocks;
    const uint32_t lane = threadIdx.x & 31u, warp = threadIdx.x >> 5;
    // sixteen lanes hold the columns (eight each), the sixteen half warps take every sixteenth row
    const uint32_t col = block * kLtQueryCols + (lane & 15u) * 8u, first = warp * 2 + (lane >> 4);
    const bool live = col < a.w_ld;
    const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(a.w) + size_t(h) * a.dim * a.w_ld + col;
    uint4 raw[kLtQueryRows];
    auto fetch = [&](uint32_t d0) {
#pragma unroll
        for (int i = 0; i < kLtQueryRows; ++i) {
            const uint32_t d = d0 + first + 16u * i;
            raw[i] = live && d < a.dim ? *reinterpret_cast<const uint4*>(w + size_t(d) * a.w_ld) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    fetch(0);
    pdl_wait();
    const float* q = a.q + size_t(t) * a.q_ld + h * (a.dim + a.rot);
    float acc[8] = {};
    for (uint32_t d0 = 0; d0 < a.dim; d0 += 16u * kLtQueryRows) {
        __syncthreads();
        for (uint32_t i = threadIdx.x; i < 16u * kLtQueryRows; i += kLtThreads) s_q[i] = d0 + i < a.dim ? q[d0 + i] * a.scale : 0.f;
        __syncthreads();
#pragma unroll
        for (int i = 0; i < kLtQueryRows; ++i) {
            const float x = s_q[first + 16u * i];
            const uint32_t u[4] = {raw[i].x, raw[i].y, raw[i].z, raw[i].w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                acc[2 * e] = fmaf(x, __uint_as_float(u[e] << 16), acc[2 * e]);
                acc[2 * e + 1] = fmaf(x, __uint_as_float(u[e] & 0xffff0000u), acc[2 * e + 1]);
            }
        }
        if (d0 + 16u * kLtQueryRows < a.dim) fetch(d0 + 16u * kLtQueryRows);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) {
        acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 16);
        if (lane < 16) s_sum[warp][lane * 8 + e] = acc[e];
    }
    __syncthreads();
    float* dst = p.u + (size_t(t) * a.heads + h) * p.ld;
    for (uint32_t c = threadIdx.x; c < kLtQueryCols; c += kLtThreads) {
        float v = 0.f;
#pragma unroll
        for (int k = 0; k < kLtWarps; ++k) v += s_sum[k][c];
        if (block * kLtQueryCols + c < p.rank_p) dst[block * kLtQueryCols + c] = v;
    }
    if (block == 0)
        for (uint32_t i = threadIdx.x; i < p.rot_p; i += kLtThreads)
            dst[p.rank_p + i] = i < a.rot ? lt_rotated(q + a.dim, a.angles + size_t(t) * a.angle_ld, i, a.angle_pairs) * a.scale : 0.f;
}

// blockIdx: x = heads / 8, y = share, z = token.  NC: pairs of value columns per thread.
template <typename CT, int NC>
__global__ void __launch_bounds__(kLtThreads) latent_decode_kernel(const LatentParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const lv_latent_args& a = p.a;
    const uint32_t h0 = blockIdx.x * kLtHeads, nh = min(uint32_t(kLtHeads), a.heads - h0), t = blockIdx.z;
    const uint32_t lane = threadIdx.x & 31u, warp = threadIdx.x >> 5;
    // groups of threads that share the value columns take every groups-th row of a chunk
    const uint32_t pairs = p.rank_p / 2, group_size = min(uint32_t(kLtThreads), (pairs + 31) / 32 * 32), groups = kLtThreads / group_size;
    const uint32_t group = threadIdx.x / group_size, pair0 = threadIdx.x - group * group_size;
    float* s_q = reinterpret_cast<float*>(smem_raw);       // [8][ld]
    float* s_p = s_q + kLtHeads * p.ld;                    // [chunk][8]
    float* s_f = s_p + kLtChunk * kLtHeads;                // [8] factor of this chunk
    float* s_sum = s_f + kLtHeads;                         // [groups][8][rank_p], groups > 1
    CT* s_rows = reinterpret_cast<CT*>(s_sum + (groups > 1 ? groups * kLtHeads * p.rank_p : 0));      // [buffers][chunk][ld]
    pdl_wait();
    const uint32_t P = *a.pos + t;
    if (P >= a.ctx_rows) {
        if (threadIdx.x == 0) atomicOr(p.err, ERR_BAD_INDEX);
        return;
    }
    const uint32_t first = lt_first(P, a.window), n_keys = P + 1 - first, chunks = (n_keys + kLtChunk - 1) / kLtChunk;
    if (blockIdx.y >= chunks) return;
    const CT* cache = static_cast<const CT*>(a.cache) + size_t(first) * p.ld;
    constexpr uint32_t kPer16 = 16 / sizeof(CT);
    auto fetch = [&](uint32_t chunk, uint32_t buffer) {    // rows behind the last key are left as they are: their weights are masked
        const uint32_t rows = min(uint32_t(kLtChunk), n_keys - chunk * kLtChunk), n16 = rows * (p.ld / kPer16);
        const CT* src = cache + size_t(chunk) * kLtChunk * p.ld;
        const uint32_t dst = smem_u32(s_rows + size_t(buffer) * kLtChunk * p.ld);
        for (uint32_t i = threadIdx.x; i < n16; i += kLtThreads)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + i * 16u), "l"(src + size_t(i) * kPer16) : "memory");
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(blockIdx.y, 0);
    for (uint32_t i = threadIdx.x; i < kLtHeads * p.ld; i += kLtThreads)
        s_q[i] = i < nh * p.ld ? p.u[(size_t(t) * a.heads + h0) * p.ld + i] : 0.f;
    float acc[NC][kLtHeads][2] = {};
    float m = -INFINITY, l = 0.f;                          // warp h: head h
    uint32_t buffer = 0;
    for (uint32_t chunk = blockIdx.y; chunk < chunks; chunk += p.splits) {
        const bool more = chunk + p.splits < chunks;
        if (more && p.buffers == 2) {
            fetch(chunk + p.splits, buffer ^ 1u);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const CT* rows = s_rows + size_t(buffer) * kLtChunk * p.ld;
        const uint32_t live = min(uint32_t(kLtChunk), n_keys - chunk * kLtChunk);
        // scores: a warp takes four rows, lanes across the columns
        float sum[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) sum[i] = 0.f;
        for (uint32_t c = lane * 4; c < p.ld; c += 128) {
            float k[4][4];
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                if (warp * 4 + r < live) lt_load4(k[r], rows + size_t(warp * 4 + r) * p.ld + c);
                else k[r][0] = k[r][1] = k[r][2] = k[r][3] = 0.f;
            }
#pragma unroll
            for (int h = 0; h < kLtHeads; ++h) {
                float q[4];
                lt_load4(q, s_q + h * p.ld + c);
#pragma unroll
                for (int r = 0; r < 4; ++r)
#pragma unroll
                    for (int e = 0; e < 4; ++e) sum[r * 8 + h] = fmaf(q[e], k[r][e], sum[r * 8 + h]);
            }
        }
        // each exchange halves the sums a lane keeps: lane i ends with sum i
#pragma unroll
        for (int n = 16; n > 0; n /= 2) {
            const bool upper = (lane & n) != 0;
#pragma unroll
            for (int i = 0; i < n; ++i) {
                const float keep = upper ? sum[i + n] : sum[i], give = upper ? sum[i] : sum[i + n];
                sum[i] = keep + __shfl_xor_sync(0xffffffffu, give, n);
            }
        }
        s_p[warp * 32 + lane] = warp * 4 + (lane >> 3) < live ? sum[0] : -INFINITY;
        __syncthreads();
        {
            const float s = s_p[lane * kLtHeads + warp];
            const float m_new = fmaxf(m, warp_max(s)), f = expf(m - m_new), e = expf(s - m_new);       // (every chunk has a visible row: m_new is finite)
            s_p[lane * kLtHeads + warp] = e;
            l = l * f + warp_sum(e);
            m = m_new;
            if (lane == 0) s_f[warp] = f;
        }
        __syncthreads();
        if (group < groups) {
            if (chunk != blockIdx.y) {
#pragma unroll
                for (int h = 0; h < kLtHeads; ++h) {
                    const float f = s_f[h];
#pragma unroll
                    for (int n = 0; n < NC; ++n) { acc[n][h][0] *= f; acc[n][h][1] *= f; }
                }
            }
            for (uint32_t j = group; j < live; j += groups) {
                float w[kLtHeads];
                lt_load4(reinterpret_cast<float(&)[4]>(w[0]), s_p + j * kLtHeads);
                lt_load4(reinterpret_cast<float(&)[4]>(w[4]), s_p + j * kLtHeads + 4);
#pragma unroll
                for (int n = 0; n < NC; ++n) {
                    const uint32_t pair = pair0 + n * kLtThreads;
                    if (pair >= pairs) continue;
                    const float2 v = lt_load2(rows + size_t(j) * p.ld + 2 * pair);
#pragma unroll
                    for (int h = 0; h < kLtHeads; ++h) {
                        acc[n][h][0] = fmaf(w[h], v.x, acc[n][h][0]);
                        acc[n][h][1] = fmaf(w[h], v.y, acc[n][h][1]);
                    }
                }
            }
        }
        __syncthreads();
        if (more && p.buffers == 1) fetch(chunk + p.splits, 0);
        if (p.buffers == 2) buffer ^= 1u;
    }
    if (groups > 1) {
        if (group < groups && pair0 < pairs)
#pragma unroll
            for (int h = 0; h < kLtHeads; ++h)
                *reinterpret_cast<float2*>(s_sum + (group * kLtHeads + h) * p.rank_p + 2 * pair0) = make_float2(acc[0][h][0], acc[0][h][1]);
        __syncthreads();
    }
    float* dst = p.shares + ((size_t(t) * a.heads + h0) * p.splits + blockIdx.y) * p.part;
    const size_t per_head = size_t(p.splits) * p.part;
    if (warp < nh && lane == 0) *reinterpret_cast<float2*>(dst + warp * per_head) = make_float2(m, l);
    if (groups > 1) {
        for (uint32_t i = threadIdx.x; i < nh * p.rank_p; i += kLtThreads) {
            const uint32_t h = i / p.rank_p, c = i - h * p.rank_p;
            float v = 0.f;
            for (uint32_t g = 0; g < groups; ++g) v += s_sum[(g * kLtHeads + h) * p.rank_p + c];
            dst[h * per_head + 4 + c] = v;
        }
    } else {
#pragma unroll
        for (int n = 0; n < NC; ++n) {
            const uint32_t pair = pair0 + n * kLtThreads;
            if (group >= groups || pair >= pairs) continue;
#pragma unroll
            for (int h = 0; h < kLtHeads; ++h)
                if (uint32_t(h) < nh) *reinterpret_cast<float2*>(dst + h * per_head + 4 + 2 * pair) = make_float2(acc[n][h][0], acc[n][h][1]);
        }
    }
}

// blockIdx: x = rows of W_uv of a head / 32, y = head, z = token
__global__ void __launch_bounds__(kLtThreads) latent_value_kernel(const LatentParams p) {
    pdl_launch_dependents();
    __shared__ float s_w[kLtMaxSplits];
    __shared__ __align__(16) float s_c[kLtMaxRank];
    const lv_latent_args& a = p.a;
    const uint32_t h = blockIdx.y, t = blockIdx.z, lane = threadIdx.x & 31u, warp = threadIdx.x >> 5;
    constexpr int kRows = kLtValueRows / kLtWarps, kSteps = 2;
    const uint32_t e0 = blockIdx.x * kLtValueRows + warp * kRows;
    const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(a.w) + (size_t(a.heads) * a.dim + size_t(h) * a.vdim) * a.w_ld;
    uint4 raw[kSteps][kRows];
    auto fetch = [&](uint32_t c0) {
#pragma unroll
        for (int s = 0; s < kSteps; ++s)
#pragma unroll
            for (int r = 0; r < kRows; ++r) {
                const uint32_t c = c0 + s * 256 + lane * 8;
                raw[s][r] = e0 + r < a.vdim && c < p.rank_p ? *reinterpret_cast<const uint4*>(w + size_t(e0 + r) * a.w_ld + c) : make_uint4(0u, 0u, 0u, 0u);
            }
    };
    fetch(0);
    const float sink = a.sink ? a.sink[h] : -INFINITY;
    pdl_wait();
    const uint32_t P = *a.pos + t;
    if (P >= a.ctx_rows) return;
    const uint32_t n_keys = P + 1 - lt_first(P, a.window), live = min(p.splits, (n_keys + kLtChunk - 1) / kLtChunk);
    const float* src = p.shares + (size_t(t) * a.heads + h) * p.splits * p.part;
    if (warp == 0) {
        float m[kLtMaxSplits / 32], l[kLtMaxSplits / 32], top = sink, den = 0.f;
#pragma unroll
        for (int i = 0; i < int(kLtMaxSplits / 32); ++i) {
            const uint32_t s = lane + 32 * i;
            m[i] = s < live ? src[s * p.part] : -INFINITY;
            l[i] = s < live ? src[s * p.part + 1] : 0.f;
            top = fmaxf(top, m[i]);
        }
        top = warp_max(top);
#pragma unroll
        for (int i = 0; i < int(kLtMaxSplits / 32); ++i) {
            m[i] = expf(m[i] - top);
            den = fmaf(m[i], l[i], den);
        }
        const float inv = 1.f / (warp_sum(den) + expf(sink - top));
#pragma unroll
        for (int i = 0; i < int(kLtMaxSplits / 32); ++i) s_w[lane + 32 * i] = m[i] * inv;
    }
    __syncthreads();
    for (uint32_t c = threadIdx.x; c < p.rank_p; c += kLtThreads) {
        float v = 0.f;
#pragma unroll 8
        for (uint32_t s = 0; s < live; ++s) v = fmaf(s_w[s], src[s * p.part + 4 + c], v);
        s_c[c] = v;
    }
    __syncthreads();
    float acc[kRows] = {};
    for (uint32_t c0 = 0; c0 < p.rank_p; c0 += 256 * kSteps) {
#pragma unroll
        for (int s = 0; s < kSteps; ++s) {
            const uint32_t c = c0 + s * 256 + lane * 8;
            if (c >= p.rank_p) continue;
            float x[8];
            lt_load4(reinterpret_cast<float(&)[4]>(x[0]), s_c + c);
            lt_load4(reinterpret_cast<float(&)[4]>(x[4]), s_c + c + 4);
#pragma unroll
            for (int r = 0; r < kRows; ++r) {
                const uint32_t u[4] = {raw[s][r].x, raw[s][r].y, raw[s][r].z, raw[s][r].w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc[r] = fmaf(__uint_as_float(u[e] << 16), x[2 * e], acc[r]);
                    acc[r] = fmaf(__uint_as_float(u[e] & 0xffff0000u), x[2 * e + 1], acc[r]);
                }
            }
        }
        if (c0 + 256 * kSteps < p.rank_p) fetch(c0 + 256 * kSteps);
    }
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
        const float v = warp_sum(acc[r]);
        if (lane == 0 && e0 + r < a.vdim) gqa_store_out(a.out, p.out_bf16, size_t(t) * a.out_ld + h * a.vdim + e0 + r, v);
    }
}

template <int HB> static size_t lt_step_floats(const LatentParams& p) {
    return size_t(HB) * (3 * p.rank_p + p.ld) + kLtStepChunk * HB + 3 * HB + HB * kLtCluster + p.ld + p.rows_k;
}

// One token in one launch.  blockIdx: x = heads / HB, y = CTA of the cluster.
template <typename CT, int HB>
__global__ void __launch_bounds__(kLtStepThreads, 1) latent_step_kernel(const LatentParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const lv_latent_args& a = p.a;
    const uint32_t h0 = blockIdx.x * HB, nh = min(uint32_t(HB), a.heads - h0), rank = blockIdx.y;
    const uint32_t lane = threadIdx.x & 31u, warp = threadIdx.x >> 5;
    // value columns: four per thread; groups of threads that share them take every groups-th row of a chunk
    const uint32_t quads = p.rank_p / 4, group_size = (quads + 31) / 32 * 32, groups = kLtStepThreads / group_size;
    const uint32_t group = threadIdx.x / group_size, quad = threadIdx.x - group * group_size;
    const bool values = group < groups && quad < quads;
    // this CTA's rows of the heads' matrices
    const uint32_t k_first = min(rank * p.rows_k, nh * a.dim), k_end = min(k_first + p.rows_k, nh * a.dim);
    const uint32_t v_first = min(rank * p.rows_v, nh * a.vdim), v_end = min(v_first + p.rows_v, nh * a.vdim);
    __nv_bfloat16* s_wm = reinterpret_cast<__nv_bfloat16*>(smem_raw);          // rows of W_uk, later of W_uv
    CT* s_rows = reinterpret_cast<CT*>(s_wm + size_t(max(p.rows_k, p.rows_v)) * a.w_ld);       // [buffers][chunk][ld]
    float* s_up = reinterpret_cast<float*>(s_rows + size_t(p.buffers) * kLtStepChunk * p.ld);  // [HB][rank_p]: this CTA's part of u, read by the cluster
    float* s_op = s_up + HB * p.rank_p;                    // the same of the weighted sums of c
    float* s_o = s_op + HB * p.rank_p;                     // combined sums of the heads of this CTA's rows of W_uv
    float* s_q = s_o + HB * p.rank_p;                      // [HB][ld]
    float* s_p = s_q + HB * p.ld;                          // [chunk][HB]
    float* s_f = s_p + kLtStepChunk * HB;                  // [HB]
    float* s_ml = s_f + HB;                                // [HB][2], read by the cluster
    float* s_w = s_ml + 2 * HB;                            // [HB][cluster] weights of the CTAs' parts
    CT* s_own = reinterpret_cast<CT*>(s_w + HB * kLtCluster);      // [ld] the token's own row
    float* s_x = s_w + HB * kLtCluster + p.ld;             // [rows_k] q of this CTA's rows of W_uk
    __shared__ uint64_t w_full, row_full[2];
    __shared__ float scratch[64];
    const auto* weights = static_cast<const __nv_bfloat16*>(a.w);
    auto fetch_w = [&](size_t row, uint32_t n) {           // by one thread
        const uint32_t bytes = n * a.w_ld * 2;
        mbar_expect_tx(&w_full, bytes);
        if (bytes) bulk_g2s(s_wm, weights + row * a.w_ld, bytes, &w_full);
    };
    if (threadIdx.x == 0) {
        mbar_init(&w_full, 1);
        for (int i = 0; i < 2; ++i) mbar_init(&row_full[i], 1);
        fence_mbar_init();
        fetch_w(size_t(h0) * a.dim + k_first, k_end - k_first);
    }
    const float sink = warp < nh && a.sink ? a.sink[h0 + warp] : -INFINITY;
    pdl_wait();
    __syncthreads();
    const uint32_t P = *a.pos;
    if (P >= a.ctx_rows) {                                 // (the same for every CTA; the copy ends before the CTA does)
        mbar_wait_warp(&w_full, 0, p.err);
        if (threadIdx.x == 0) atomicOr(p.err, ERR_BAD_INDEX);
        return;
    }
    const uint32_t first = lt_first(P, a.window), n_keys = P + 1 - first, chunks = (n_keys + kLtStepChunk - 1) / kLtStepChunk;
    const bool own_row = a.dkv != nullptr && (chunks - 1) % kLtCluster == rank;       // this CTA has the token's own row, which it forms itself
    const CT* cache = static_cast<const CT*>(a.cache) + size_t(first) * p.ld;
    auto fetch = [&](uint32_t chunk, uint32_t buffer) {    // by one thread
        uint32_t rows = min(uint32_t(kLtStepChunk), n_keys - chunk * kLtStepChunk);
        if (a.dkv != nullptr && chunk == chunks - 1) --rows;
        const uint32_t bytes = rows * p.ld * uint32_t(sizeof(CT));
        mbar_expect_tx(&row_full[buffer], bytes);
        if (bytes) bulk_g2s(s_rows + size_t(buffer) * kLtStepChunk * p.ld, cache + size_t(chunk) * kLtStepChunk * p.ld, bytes, &row_full[buffer]);
    };
    if (threadIdx.x == 0) {
        if (rank < chunks) fetch(rank, 0);
        if (p.buffers == 2 && rank + kLtCluster < chunks) fetch(rank + kLtCluster, 1);
    }
#pragma unroll
    for (int h = 0; h < HB; ++h) {
        const float* q = a.q + size_t(h0 + h) * (a.dim + a.rot);
        const bool live = uint32_t(h) < nh;
        if (live) {
            const uint32_t lo = max(k_first, h * a.dim), hi = min(k_end, (h + 1) * a.dim);
            for (uint32_t i = lo + threadIdx.x; i < hi; i += kLtStepThreads) s_x[i - k_first] = q[i - h * a.dim] * a.scale;
        }
        for (uint32_t c = threadIdx.x; c < p.rot_p; c += kLtStepThreads)
            s_q[h * p.ld + p.rank_p + c] = live && c < a.rot ? lt_rotated(q + a.dim, a.angles, c, a.angle_pairs) * a.scale : 0.f;
    }
    if (own_row) lt_row<CT, kLtStepThreads>(p, 0, scratch, s_own, blockIdx.x == 0 ? static_cast<CT*>(a.cache) + size_t(P) * p.ld : static_cast<CT*>(nullptr));
    __syncthreads();
    // this CTA's part of u = scale W_uk^T q
    bool ok = mbar_wait_warp(&w_full, 0, p.err);
#pragma unroll
    for (int h = 0; h < HB; ++h) {
        const uint32_t lo = max(k_first, h * a.dim), hi = min(k_end, (h + 1) * a.dim);
        if (!ok || lo >= hi) continue;
        for (uint32_t pair = threadIdx.x; pair < p.rank_p / 2; pair += kLtStepThreads) {
            const __nv_bfloat16* w = s_wm + size_t(lo - k_first) * a.w_ld + 2 * pair;
            const float* x = s_x + lo - k_first;
            float2 sum = make_float2(0.f, 0.f);
#pragma unroll 8
            for (uint32_t i = 0; i < hi - lo; ++i) {
                const float2 v = lt_load2(w + i * a.w_ld);
                sum.x = fmaf(x[i], v.x, sum.x);
                sum.y = fmaf(x[i], v.y, sum.y);
            }
            *reinterpret_cast<float2*>(s_up + h * p.rank_p + 2 * pair) = sum;
        }
    }
    fence_proxy_async();
    cluster_sync();
    if (threadIdx.x == 0) fetch_w(size_t(a.heads) * a.dim + size_t(h0) * a.vdim + v_first, v_end - v_first);
#pragma unroll
    for (int h = 0; h < HB; ++h) {
        const bool live = uint32_t(h) < nh;
        const uint32_t r0 = h * a.dim / p.rows_k, r1 = ((h + 1) * a.dim - 1) / p.rows_k;       // CTAs with rows of this head
        for (uint32_t c = threadIdx.x; c < p.rank_p; c += kLtStepThreads) {
            float part[kLtCluster], v = 0.f;
#pragma unroll
            for (int r = 0; r < kLtCluster; ++r) part[r] = live && uint32_t(r) >= r0 && uint32_t(r) <= r1 ? cluster_load(s_up + h * p.rank_p + c, r) : 0.f;
#pragma unroll
            for (int r = 0; r < kLtCluster; ++r) v += part[r];
            s_q[h * p.ld + c] = v;
        }
    }
    float acc[HB][4] = {};
    float m = -INFINITY, l = 0.f;                          // warp h: head h
    uint32_t buffer = 0, phase = 0;
    for (uint32_t chunk = rank; chunk < chunks; chunk += kLtCluster) {
        __syncthreads();
        ok = ok && mbar_wait_warp(&row_full[buffer], phase, p.err);
        CT* rows = s_rows + size_t(buffer) * kLtStepChunk * p.ld;
        const uint32_t live = min(uint32_t(kLtStepChunk), n_keys - chunk * kLtStepChunk);
        if (own_row && chunk == chunks - 1) {
            for (uint32_t i = threadIdx.x; i < p.ld; i += kLtStepThreads) rows[size_t(live - 1) * p.ld + i] = s_own[i];
            __syncthreads();
        }
        // scores: a warp takes four rows, lanes across the columns (rows behind the last one count as copies of it)
        float sum[4 * HB];
#pragma unroll
        for (int i = 0; i < 4 * HB; ++i) sum[i] = 0.f;
        const CT* row[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) row[r] = rows + size_t(min(warp * 4 + r, live - 1)) * p.ld;
#pragma unroll 2
        for (uint32_t c = lane * 4; c < p.ld; c += 128) {
            float k[4][4];
#pragma unroll
            for (int r = 0; r < 4; ++r) lt_load4(k[r], row[r] + c);
#pragma unroll
            for (int h = 0; h < HB; ++h) {
                float q[4];
                lt_load4(q, s_q + h * p.ld + c);
#pragma unroll
                for (int r = 0; r < 4; ++r)
#pragma unroll
                    for (int e = 0; e < 4; ++e) sum[r * HB + h] = fmaf(q[e], k[r][e], sum[r * HB + h]);
            }
        }
        lanes_reduce<32, 4 * HB>(sum);
        constexpr uint32_t kLanes = 32 / (4 * HB);         // lanes that end up with the same sum
        const uint32_t at = lane / kLanes;                 // row * HB + head
        if (lane % kLanes == 0) s_p[warp * 4 * HB + at] = warp * 4 + at / HB < live ? sum[0] : -INFINITY;
        __syncthreads();
        if (warp < HB) {
            const float s0 = s_p[lane * HB + warp], s1 = s_p[(lane + 32) * HB + warp];
            const float m_new = fmaxf(m, warp_max(fmaxf(s0, s1))), f = expf(m - m_new), e0 = expf(s0 - m_new), e1 = expf(s1 - m_new);
            s_p[lane * HB + warp] = e0;
            s_p[(lane + 32) * HB + warp] = e1;
            l = l * f + warp_sum(e0 + e1);
            m = m_new;
            if (lane == 0) s_f[warp] = f;
        }
        __syncthreads();
        if (values) {
            if (chunk != rank) {
#pragma unroll
                for (int h = 0; h < HB; ++h) {
                    const float f = s_f[h];
#pragma unroll
                    for (int e = 0; e < 4; ++e) acc[h][e] *= f;
                }
            }
#pragma unroll 4
            for (uint32_t j = group; j < live; j += groups) {
                float v[4];
                lt_load4(v, rows + size_t(j) * p.ld + 4 * quad);
#pragma unroll
                for (int h = 0; h < HB; ++h) {
                    const float w = s_p[j * HB + h];
#pragma unroll
                    for (int e = 0; e < 4; ++e) acc[h][e] = fmaf(w, v[e], acc[h][e]);
                }
            }
        }
        const uint32_t next = chunk + p.buffers * kLtCluster;
        if (next < chunks) {                               // everyone is done with these rows
            fence_proxy_async();
            __syncthreads();
            if (threadIdx.x == 0) fetch(next, buffer);
        }
        if (p.buffers == 2) {
            buffer ^= 1u;
            if (buffer == 0) phase ^= 1u;
        } else {
            phase ^= 1u;
        }
    }
    // sums of the groups, in order; they meet where the rows were
    __syncthreads();
    float* s_sum = reinterpret_cast<float*>(s_rows);       // [groups][HB][rank_p]
    if (values)
#pragma unroll
        for (int h = 0; h < HB; ++h) *reinterpret_cast<float4*>(s_sum + (group * HB + h) * p.rank_p + 4 * quad) = make_float4(acc[h][0], acc[h][1], acc[h][2], acc[h][3]);
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < HB * p.rank_p; i += kLtStepThreads) {
        float v = 0.f;
#pragma unroll 4
        for (uint32_t g = 0; g < groups; ++g) v += s_sum[g * HB * p.rank_p + i];
        s_op[i] = v;
    }
    if (warp < HB && lane == 0) { s_ml[2 * warp] = m; s_ml[2 * warp + 1] = l; }
    cluster_sync();
    // combination for the heads of this CTA's rows of W_uv: warp h weighs the parts of head h
    const uint32_t hv0 = v_first / a.vdim, hv1 = v_end > v_first ? (v_end - 1) / a.vdim + 1 : hv0;
    if (warp < nh && warp >= hv0 && warp < hv1) {
        const float mr = lane < kLtCluster ? cluster_load(s_ml + 2 * warp, lane) : -INFINITY, lr = lane < kLtCluster ? cluster_load(s_ml + 2 * warp + 1, lane) : 0.f;
        const float top = fmaxf(sink, warp_max(mr)), e = expf(mr - top);
        const float inv = 1.f / (warp_sum(e * lr) + expf(sink - top));
        if (lane < kLtCluster) s_w[warp * kLtCluster + lane] = e * inv;
    }
    __syncthreads();
    for (uint32_t h = hv0; h < hv1; ++h) {
        for (uint32_t c = threadIdx.x; c < p.rank_p; c += kLtStepThreads) {
            float part[kLtCluster], v = 0.f;
#pragma unroll
            for (int r = 0; r < kLtCluster; ++r) part[r] = cluster_load(s_op + h * p.rank_p + c, r);
#pragma unroll
            for (int r = 0; r < kLtCluster; ++r) v = fmaf(s_w[h * kLtCluster + r], part[r], v);
            s_o[h * p.rank_p + c] = v;
        }
    }
    __syncthreads();
    ok = mbar_wait_warp(&w_full, 1, p.err) && ok;
    constexpr int kRows = 2;                               // rows of a warp at a time
    for (uint32_t first_row = v_first + warp * kRows; ok && first_row < v_end; first_row += kLtStepWarps * kRows) {
        float dot[kRows] = {};
        const __nv_bfloat16* w[kRows];
        const float* x[kRows];
#pragma unroll
        for (int r = 0; r < kRows; ++r) {
            const uint32_t at = min(first_row + r, v_end - 1);
            w[r] = s_wm + size_t(at - v_first) * a.w_ld;
            x[r] = s_o + at / a.vdim * p.rank_p;
        }
#pragma unroll 2
        for (uint32_t c = lane * 8; c < p.rank_p; c += 256) {
#pragma unroll
            for (int r = 0; r < kRows; ++r) {
                float wv[8], xv[8];
                lt_load4(reinterpret_cast<float(&)[4]>(wv[0]), w[r] + c);
                lt_load4(reinterpret_cast<float(&)[4]>(wv[4]), w[r] + c + 4);
                lt_load4(reinterpret_cast<float(&)[4]>(xv[0]), x[r] + c);
                lt_load4(reinterpret_cast<float(&)[4]>(xv[4]), x[r] + c + 4);
#pragma unroll
                for (int e = 0; e < 8; ++e) dot[r] = fmaf(wv[e], xv[e], dot[r]);
            }
        }
        lanes_reduce<32, kRows>(dot);
        const uint32_t at = first_row + lane / (32 / kRows);
        if (lane % (32 / kRows) == 0 && at < v_end) gqa_store_out(a.out, p.out_bf16, size_t(h0) * a.vdim + at, dot[0]);
    }
    cluster_sync();                                        // no CTA leaves while another reads its shared memory
}

// {cos, sin} of the angles of a step; the angle itself in f64, so that far positions keep their phase
__global__ void __launch_bounds__(128) rotary_table_kernel(float* out, const double* freqs, const float* mults, uint32_t pairs, const uint32_t* pos, uint32_t batch) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= batch * pairs) return;
    const uint32_t t = i / pairs, k = i - t * pairs;
    double s, c;
    sincos(double(*pos + t) * freqs[k], &s, &c);
    *reinterpret_cast<float2*>(out + size_t(i) * 2) = make_float2(float(c) * mults[k], float(s) * mults[k]);
}

static uint32_t lt_pad8(uint32_t n) { return (n + 7) / 8 * 8; }

static int latent_check(const lv_latent_args* a, uint32_t batch) {
    LV_REQUIRE(a && a->q && a->w && a->cache && a->pos && a->out && a->angles && batch && batch <= 65535, "bad latent attention arguments");
    LV_REQUIRE(a->heads && a->heads <= 65535 && a->dim && a->vdim && a->kv_rank && a->kv_rank <= kLtMaxRank && a->angle_pairs * 2 <= a->rot, "latent attention: unsupported sizes");
    LV_REQUIRE(a->q_ld >= a->heads * (a->dim + a->rot) && a->out_ld >= a->heads * a->vdim && a->ctx_rows, "latent attention: bad strides");
    LV_REQUIRE(a->dkv == nullptr || (a->kv_norm && a->dkv_ld >= a->kv_rank + a->rot), "latent attention: bad latent projection");
    LV_REQUIRE(a->w_ld % 8 == 0 && a->w_ld >= a->kv_rank && (reinterpret_cast<uintptr_t>(a->w) & 15u) == 0 && (reinterpret_cast<uintptr_t>(a->cache) & 15u) == 0 &&
               (reinterpret_cast<uintptr_t>(a->angles) & 7u) == 0 && a->angle_ld % 2 == 0, "latent attention: bad alignment");
    LV_REQUIRE((a->cache_type == LV_TYPE_F32 || a->cache_type == LV_TYPE_BF16) && (a->out_type == LV_TYPE_F32 || a->out_type == LV_TYPE_BF16), "latent attention: types");
    return LV_OK;
}

static bool lt_expanded(const lv_latent_args& a, uint32_t batch) {
    if (a.form == LV_LATENT_ABSORBED || batch < 2 || !latent_tc_supported(a)) return false;
    return a.form == LV_LATENT_EXPANDED || batch > kLtAbsorbedBatch;
}

// rows that `batch` tokens can see
static uint32_t lt_rows(const lv_latent_args& a, uint32_t batch, uint32_t capacity) {
    const uint64_t n = a.window ? uint64_t(batch) + a.window - 1 : capacity;
    return uint32_t(std::min<uint64_t>(n, capacity));
}
static uint32_t lt_heads_per_pass(const lv_latent_args& a, uint32_t rows) {
    const size_t per_head = size_t(rows) * (a.dim + a.vdim) * 2;
    return uint32_t(std::max<size_t>(1, std::min<size_t>(a.heads, kLtExpandBytes / per_head)));
}

static uint32_t lt_splits(const lv_ctx* ctx, const lv_latent_args& a, uint32_t batch, uint32_t capacity) {
    const uint32_t ctas = (a.heads + kLtHeads - 1) / kLtHeads * batch, keys = a.window ? std::min(a.window, capacity) : capacity;
    const uint32_t want = (2u * uint32_t(ctx->sm_count) + ctas - 1) / ctas, chunks = (keys + kLtChunk - 1) / kLtChunk;
    return std::max(1u, std::min({want, chunks, kLtMaxSplits}));
}

static size_t lt_scratch(const lv_ctx* ctx, const lv_latent_args& a, uint32_t batch, uint32_t capacity) {
    if (lt_expanded(a, batch)) {
        const uint32_t rows = lt_rows(a, batch, capacity);
        return size_t(rows) * lt_heads_per_pass(a, rows) * (a.dim + a.vdim) * 2;
    }
    const size_t rank_p = lt_pad8(a.kv_rank), ld = rank_p + lt_pad8(a.rot);
    return size_t(batch) * a.heads * 4 * (ld + size_t(lt_splits(ctx, a, batch, capacity)) * (rank_p + 4));
}

// One token in one launch; false when its sizes do not fit.
template <typename CT, int HB>
static bool latent_step(lv_ctx* ctx, LatentParams p, int* rc) {
    const lv_latent_args& a = p.a;
    p.rows_k = (HB * a.dim + kLtCluster - 1) / kLtCluster;
    p.rows_v = (HB * a.vdim + kLtCluster - 1) / kLtCluster;
    const uint32_t quads = p.rank_p / 4, groups = kLtStepThreads / ((quads + 31) / 32 * 32);
    const size_t fixed = size_t(std::max(p.rows_k, p.rows_v)) * a.w_ld * 2 + sizeof(float) * lt_step_floats<HB>(p), rows = size_t(kLtStepChunk) * p.ld * sizeof(CT);
    const size_t limit = size_t(ctx->max_smem_optin) - 1024;
    p.buffers = fixed + 2 * rows <= limit ? 2 : 1;
    if (fixed + p.buffers * rows > limit || sizeof(float) * groups * HB * p.rank_p > p.buffers * rows) return false;
    auto* kernel = latent_step_kernel<CT, HB>;
    auto launch = [&]() -> int {
        LV_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(fixed + p.buffers * rows)));
        LV_CUDA(launch_pdl_cluster(ctx, kernel, dim3((a.heads + HB - 1) / HB, kLtCluster), dim3(kLtStepThreads), dim3(1, kLtCluster), fixed + p.buffers * rows, p));
        return LV_OK;
    };
    *rc = launch();
    return true;
}

template <typename CT>
static int latent_absorbed(lv_ctx* ctx, LatentParams p, uint32_t batch, uint32_t capacity) {
    const lv_latent_args& a = p.a;
    if (batch == 1 && a.form == LV_LATENT_AUTO && (a.window ? std::min(a.window, capacity) : capacity) <= kLtStepKeys) {
        // about as many clusters as fit on the device at a time
        int rc = LV_OK;
        if (a.heads <= 8 ? latent_step<CT, 1>(ctx, p, &rc) : a.heads <= 16 ? latent_step<CT, 2>(ctx, p, &rc) : a.heads <= 32 ? latent_step<CT, 4>(ctx, p, &rc) : latent_step<CT, 8>(ctx, p, &rc))
            return rc;
    }
    LV_CUDA(launch_pdl(ctx, latent_query_kernel<CT>, dim3(a.heads * p.col_blocks + (a.dkv ? 1 : 0), batch), dim3(kLtThreads), 0, p));
    const uint32_t pairs = p.rank_p / 2, group_size = std::min<uint32_t>(kLtThreads, (pairs + 31) / 32 * 32), groups = kLtThreads / group_size;
    const size_t fixed = sizeof(float) * (size_t(kLtHeads) * p.ld + kLtChunk * kLtHeads + kLtHeads + (groups > 1 ? size_t(groups) * kLtHeads * p.rank_p : 0));
    const size_t rows = size_t(kLtChunk) * p.ld * sizeof(CT);
    p.buffers = fixed + 2 * rows <= size_t(ctx->max_smem_optin) ? 2 : 1;
    const size_t smem = fixed + p.buffers * rows;
    LV_REQUIRE(smem <= size_t(ctx->max_smem_optin), "latent attention: sizes need too much shared memory");
    auto* kernel = p.rank_p <= 2 * kLtThreads ? latent_decode_kernel<CT, 1> : latent_decode_kernel<CT, 2>;
    LV_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    LV_CUDA(launch_pdl(ctx, kernel, dim3(p.head_blocks, p.splits, batch), dim3(kLtThreads), smem, p));
    LV_CUDA(launch_pdl(ctx, latent_value_kernel, dim3((a.vdim + kLtValueRows - 1) / kLtValueRows, a.heads, batch), dim3(kLtThreads), 0, p));
    return LV_OK;
}

}  // namespace lv

using namespace lv;

extern "C" int lv_rotary_table(lv_ctx* ctx, float* out, const double* freqs, const float* mults, uint32_t pairs, const uint32_t* pos, uint32_t batch) {
    LV_ENTER(ctx);
    LV_REQUIRE(out && freqs && mults && pairs && pos && batch, "bad rotary_table arguments");
    LV_CUDA(launch_pdl(ctx, rotary_table_kernel, dim3((batch * pairs + 127) / 128), dim3(128), 0, out, freqs, mults, pairs, pos, batch));
    return LV_OK;
}

extern "C" size_t lv_latent_scratch_bytes(lv_ctx* ctx, const lv_latent_args* a, uint32_t batch, uint32_t capacity) {
    if (!ctx || !a || !batch || !capacity || !a->heads) return 0;
    return lt_scratch(ctx, *a, batch, capacity);
}

extern "C" int lv_latent_attention(lv_ctx* ctx, const lv_latent_args* args, void* scratch, size_t scratch_bytes, uint32_t batch, uint32_t capacity) {
    LV_ENTER(ctx);
    if (const int rc = latent_check(args, batch)) return rc;
    lv_latent_args given = *args;
    if (given.window >= given.ctx_rows) given.window = 0;
    const lv_latent_args* a = &given;
    LV_REQUIRE(capacity && capacity <= a->ctx_rows && scratch && scratch_bytes >= lt_scratch(ctx, *a, batch, capacity), "latent attention: scratch too small");
    LV_REQUIRE(a->form != LV_LATENT_EXPANDED || lt_expanded(*a, batch), "latent attention: the expanded form does not take these sizes");
    LatentParams p{};
    p.a = *a;
    p.rank_p = lt_pad8(a->kv_rank);
    p.rot_p = lt_pad8(a->rot);
    p.ld = p.rank_p + p.rot_p;
    p.out_bf16 = a->out_type == LV_TYPE_BF16;
    p.err = ctx->d_err;
    const bool f32 = a->cache_type == LV_TYPE_F32;
    if (lt_expanded(*a, batch)) {
        if (a->dkv) LV_CUDA(launch_pdl(ctx, latent_append_kernel<__nv_bfloat16>, dim3(batch), dim3(kLtThreads), 0, p));
        const uint32_t rows = lt_rows(*a, batch, capacity), per = lt_heads_per_pass(*a, rows), ld = per * (a->dim + a->vdim);
        const auto* w = static_cast<const __nv_bfloat16*>(a->w);
        auto* kv = static_cast<__nv_bfloat16*>(scratch);
        for (uint32_t h = 0; h < a->heads; h += per) {
            const uint32_t n = std::min(per, a->heads - h);
            auto expand = [&](size_t first_row, uint32_t n_rows, uint32_t at) {
                return lv_gemm_bf16_window(ctx, kv + at, LV_TYPE_BF16, ld, w + first_row * a->w_ld, n_rows, a->w_ld, a->kv_rank, a->cache, p.ld, a->ctx_rows, a->pos, batch,
                                           a->window, rows);
            };
            int rc = LV_OK;
            if (n == a->heads) {
                rc = expand(0, n * (a->dim + a->vdim), 0);
            } else {
                rc = expand(size_t(h) * a->dim, n * a->dim, 0);
                if (rc == LV_OK) rc = expand(size_t(a->heads) * a->dim + size_t(h) * a->vdim, n * a->vdim, per * a->dim);
            }
            if (rc == LV_OK) rc = latent_tc_launch(ctx, *a, batch, kv, ld, per * a->dim, rows, h, n);
            if (rc != LV_OK) return rc;
        }
        return LV_OK;
    }
    p.head_blocks = (a->heads + kLtHeads - 1) / kLtHeads;
    p.splits = lt_splits(ctx, *a, batch, capacity);
    p.part = p.rank_p + 4;
    p.col_blocks = (p.rank_p + kLtQueryCols - 1) / kLtQueryCols;
    p.u = static_cast<float*>(scratch);
    p.shares = p.u + size_t(batch) * a->heads * p.ld;
    return f32 ? latent_absorbed<float>(ctx, p, batch, capacity) : latent_absorbed<__nv_bfloat16>(ctx, p, batch, capacity);
}
