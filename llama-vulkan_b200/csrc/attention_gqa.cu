// Causal attention with grouped key/value heads, query/key norm, a distance bias and an optional sink, on CUDA cores in f32.
//
//   q'_h = scale * rmsnorm(q_h) * qw,  k'_g = rmsnorm(k_g) * kw
//   s_ij = q'_i . k'_j - r1_h ln(1 + r2_h (i - j)),  j <= i
//   p_ij = exp(s_ij) / (sink + sum_j exp(s_ij)),     sink = 1 or 0
//
// One CTA serves up to eight query heads of one key/value head for one token and walks its share of the keys in chunks of
// 64 with an online softmax.  A decoded token spreads the chunks over several CTAs: up to 16 form a thread-block cluster and
// combine their partial sums through distributed shared memory; beyond that (long contexts) the last to arrive combines
// them through scratch.  A decoded token's own key and value are normalised and appended to the caches by the same launch;
// tokens of a prompt are appended first (lv_qk_norm_append) and, with bfloat16 caches, go through attention_gqa_tc.cu.  Caches are [kv head][ctx_rows][padded dim], bfloat16 or f32.
#include <cuda_bf16.h>
#include <math.h>

#include <algorithm>

#include "attention_gqa.cuh"
#include "common.cuh"
#include "ctx.h"

namespace lv {

constexpr size_t kGqaCounterBytes = 4096;   // arrival counters at the start of the scratch (kept zero between launches)
constexpr int kGqaThreads = 256, kGqaWarps = 8, kGqaChunk = 64, kGqaHeads = 8, kGqaMaxSplits = 128, kGqaCluster = 16;

struct GqaParams {
    lv_gqa_args a;
    uint32_t dim_p, vdim_p;         // padded to 8
    uint32_t head_blocks;           // CTAs per key/value head
    uint32_t splits;
    uint32_t clustered;             // the splits of a token are one thread-block cluster
    uint32_t out_bf16, append;
    float* scratch;                 // splits > 1: [token][head][split][vdim_p + 2]
    uint32_t* counters;             // [token][kv head * head_blocks]
    uint32_t* err;
};

// eight cache values: as fetched, and widened to f32
template <typename CT> struct Cache8;
template <> struct Cache8<__nv_bfloat16> {
    using raw = uint4;
    static __device__ __forceinline__ raw fetch(const __nv_bfloat16* p) { return *reinterpret_cast<const uint4*>(p); }
    static __device__ __forceinline__ void widen(float (&v)[8], const raw& w) {
        const uint32_t q[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) { v[2 * i] = __uint_as_float(q[i] << 16); v[2 * i + 1] = __uint_as_float(q[i] & 0xffff0000u); }
    }
    static __device__ __forceinline__ __nv_bfloat16 cast(float v) { return __float2bfloat16_rn(v); }
    // (the fast logarithm is good to about 2^-21 here, far below the rounding of the operands)
    static __device__ __forceinline__ float log_one_plus(float v) { return __logf(1.f + v); }
};
template <> struct Cache8<float> {
    struct raw { float4 a, b; };
    static __device__ __forceinline__ raw fetch(const float* p) { return {*reinterpret_cast<const float4*>(p), *reinterpret_cast<const float4*>(p + 4)}; }
    static __device__ __forceinline__ void widen(float (&v)[8], const raw& w) {
        v[0] = w.a.x; v[1] = w.a.y; v[2] = w.a.z; v[3] = w.a.w; v[4] = w.b.x; v[5] = w.b.y; v[6] = w.b.z; v[7] = w.b.w;
    }
    static __device__ __forceinline__ float cast(float v) { return v; }
    static __device__ __forceinline__ float log_one_plus(float v) { return log1pf(v); }
};

// Appends the normalised key and the value of token t (one warp per key/value head).
template <typename CT>
__global__ void __launch_bounds__(128) qk_norm_append_kernel(const GqaParams p, uint32_t n_tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const lv_gqa_args& a = p.a;
    const uint32_t job = blockIdx.x * 4u + (threadIdx.x >> 5), lane = threadIdx.x & 31u;
    if (job >= n_tokens * a.kv_heads) return;
    const uint32_t t = job / a.kv_heads, g = job - t * a.kv_heads;
    const uint32_t row = *a.pos + t;
    if (row >= a.ctx_rows) {
        if (lane == 0) atomicOr(p.err, ERR_BAD_INDEX);
        return;
    }
    const float* k = a.qkv + size_t(t) * a.qkv_ld + a.heads * a.dim + g * a.dim;
    const float* v = a.qkv + size_t(t) * a.qkv_ld + (a.heads + a.kv_heads) * a.dim + g * a.vdim;
    const float r = gqa_rms_factor(k, a.dim, a.eps);
    CT* kd = static_cast<CT*>(a.k_cache) + (size_t(g) * a.ctx_rows + row) * p.dim_p;
    CT* vd = static_cast<CT*>(a.v_cache) + (size_t(g) * a.ctx_rows + row) * p.vdim_p;
    for (uint32_t i = lane; i < p.dim_p; i += 32) kd[i] = Cache8<CT>::cast(i < a.dim ? k[i] * r * a.k_norm[i] : 0.f);
    for (uint32_t i = lane; i < p.vdim_p; i += 32) vd[i] = Cache8<CT>::cast(i < a.vdim ? v[i] : 0.f);
}

// HB: query heads of this CTA, rounded up.  L: lanes that share a key and threads that share a value row (8 values each).
template <typename CT, int HB, int L>
__global__ void __launch_bounds__(kGqaThreads) gqa_kernel(const GqaParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const lv_gqa_args& a = p.a;
    const uint32_t group = a.heads / a.kv_heads;
    const uint32_t g = blockIdx.x / p.head_blocks, hb = blockIdx.x - g * p.head_blocks;
    const uint32_t h0 = g * group + hb * kGqaHeads, nh = min(uint32_t(kGqaHeads), group - hb * kGqaHeads);
    const uint32_t t = blockIdx.z;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    constexpr int kPerWarp = 32 / L, kIters = kGqaChunk / (kGqaWarps * kPerWarp);      // keys of a warp per pass, passes per chunk
    constexpr int kGroups = kGqaThreads / L;                                             // value rows in flight; kIters each
    float* s_q = reinterpret_cast<float*>(smem_raw);      // [HB][dim_p]
    float* s_sc = s_q + HB * p.dim_p;                      // [HB][chunk]
    float* s_red = s_sc + HB * kGqaChunk;                  // [warps][HB][L * 8]; the combination reuses it
    float* s_m = s_red + kGqaWarps * HB * L * 8;           // [HB] running maximum
    float* s_l = s_m + HB;                                 // [HB] running sum
    float* s_c = s_l + HB;                                 // [HB] factor of this chunk
    CT* s_k = reinterpret_cast<CT*>(s_c + 2 * HB);         // append: the token's own key and value as the cache holds them (16-byte aligned)
    CT* s_v = s_k + p.dim_p;
    __shared__ uint32_t s_last;

    const uint32_t sub = lane & (L - 1), key_in_warp = lane / L;
    const uint32_t vcol = (threadIdx.x & (L - 1)) * 8, vgroup = threadIdx.x / L;
    // the lane that ends up with head h's score of a key is lane h * (L / HB) of the key's lanes
    const uint32_t my_head = sub / (L / HB);
    const bool score_lane = sub % (L / HB) == 0;
    const float r1 = my_head < nh ? a.r1[h0 + my_head] : 0.f, r2 = my_head < nh ? a.r2[h0 + my_head] : 0.f;
    // warp h normalises query head h, the last warp the token's own key
    const bool own_key = warp == kGqaWarps - 1;
    float qw[L / 4], kw[L / 4];
    gqa_head_load<L / 4>(qw, a.q_norm, a.dim, warp < int(nh));
    gqa_head_load<L / 4>(kw, a.k_norm, a.dim, own_key);
    pdl_wait();
    CT* kc = static_cast<CT*>(a.k_cache) + size_t(g) * a.ctx_rows * p.dim_p;
    CT* vc = static_cast<CT*>(a.v_cache) + size_t(g) * a.ctx_rows * p.vdim_p;
    const bool append = p.append != 0;
    // a chunk's keys and values are requested before anything waits for them (rows up to `limit`; the position is not known
    // yet when the first chunk is requested, so rows behind it come along and are never used)
    typename Cache8<CT>::raw kr[kIters], vr[kIters];
    auto fetch = [&](uint32_t k0, uint32_t limit) {
#pragma unroll
        for (int i = 0; i < kIters; ++i) {
            const uint32_t j = k0 + (i * kGqaWarps + warp) * kPerWarp + key_in_warp;
            if (sub * 8 < p.dim_p && j < limit) kr[i] = Cache8<CT>::fetch(kc + size_t(j) * p.dim_p + sub * 8);
        }
#pragma unroll
        for (int i = 0; i < kIters; ++i) {
            const uint32_t j = k0 + i * kGroups + vgroup;
            if (vcol < p.vdim_p && j < limit) vr[i] = Cache8<CT>::fetch(vc + size_t(j) * p.vdim_p + vcol);
        }
    };
    const uint32_t P = *a.pos + t;
    const float* raw = a.qkv + size_t(t) * a.qkv_ld;
    float q[L / 4], k[L / 4], v[L / 4];
    gqa_head_load<L / 4>(q, raw + (h0 + warp) * a.dim, a.dim, warp < int(nh));
    gqa_head_load<L / 4>(k, raw + a.heads * a.dim + g * a.dim, a.dim, own_key);
    gqa_head_load<L / 4>(v, raw + (a.heads + a.kv_heads) * a.dim + g * a.vdim, a.vdim, own_key);
    fetch(blockIdx.y * kGqaChunk, a.ctx_rows);
    if (P >= a.ctx_rows) {                                 // (the same for every CTA of a cluster)
        if (threadIdx.x == 0) atomicOr(p.err, ERR_BAD_INDEX);
        return;
    }
    const uint32_t own_chunk = P / kGqaChunk;
    if (warp < HB) {
        const float r = gqa_head_factor<L / 4>(q, a.dim, a.eps) * a.scale;
#pragma unroll
        for (int i = 0; i < L / 4; ++i)
            if (lane + 32 * i < int(p.dim_p)) s_q[warp * p.dim_p + lane + 32 * i] = q[i] * r * qw[i];      // zeros for missing heads and columns
    }
    if (append && own_key && own_chunk % p.splits == blockIdx.y) {
        const float r = gqa_head_factor<L / 4>(k, a.dim, a.eps);
#pragma unroll
        for (int i = 0; i < L / 4; ++i) {
            const uint32_t c = lane + 32 * i;
            if (c < p.dim_p) {
                const CT e = Cache8<CT>::cast(k[i] * r * kw[i]);
                s_k[c] = e;
                if (hb == 0) kc[size_t(P) * p.dim_p + c] = e;
            }
            if (c < p.vdim_p) {
                const CT e = Cache8<CT>::cast(v[i]);
                s_v[c] = e;
                if (hb == 0) vc[size_t(P) * p.vdim_p + c] = e;
            }
        }
    }
    if (threadIdx.x < HB) { s_m[threadIdx.x] = -INFINITY; s_l[threadIdx.x] = 0.f; }
    float acc[HB][8];
#pragma unroll
    for (int h = 0; h < HB; ++h)
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[h][i] = 0.f;
    __syncthreads();

    for (uint32_t c = blockIdx.y; c <= own_chunk; c += p.splits) {
        const uint32_t k0 = c * kGqaChunk;
        if (c != blockIdx.y) fetch(k0, P + 1);
        float bias[kIters];
#pragma unroll
        for (int i = 0; i < kIters; ++i) {
            const uint32_t j = k0 + (i * kGqaWarps + warp) * kPerWarp + key_in_warp;
            bias[i] = j <= P ? r1 * Cache8<CT>::log_one_plus(r2 * float(P - j)) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < kIters; ++i) {
            const uint32_t kk = (i * kGqaWarps + warp) * kPerWarp + key_in_warp, j = k0 + kk;
            const bool live = j <= P && sub * 8 < p.dim_p;
            float kv[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            if (live) {
                if (append && j == P) kr[i] = Cache8<CT>::fetch(s_k + sub * 8);
                Cache8<CT>::widen(kv, kr[i]);
            }
            float sum[HB];
#pragma unroll
            for (int h = 0; h < HB; ++h) {
                sum[h] = 0.f;
                if (live) {
                    float qv[8];
                    Cache8<float>::widen(qv, Cache8<float>::fetch(s_q + h * p.dim_p + sub * 8));
#pragma unroll
                    for (int e = 0; e < 8; ++e) sum[h] = fmaf(qv[e], kv[e], sum[h]);
                }
            }
            // the key's lanes share the sums of all heads: each exchange halves the heads a lane keeps
            int o = L / 2;
#pragma unroll
            for (int n = HB / 2; n > 0; n /= 2, o /= 2) {
                const bool upper = (sub & o) != 0;
#pragma unroll
                for (int h = 0; h < n; ++h) {
                    const float keep = upper ? sum[h + n] : sum[h], give = upper ? sum[h] : sum[h + n];
                    sum[h] = keep + __shfl_xor_sync(0xffffffffu, give, o);
                }
            }
#pragma unroll
            for (; o > 0; o /= 2) sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], o);
            if (score_lane) s_sc[my_head * kGqaChunk + kk] = (j <= P && my_head < nh) ? sum[0] - bias[i] : -INFINITY;
        }
        __syncthreads();
        // online softmax: warp h takes head h
        if (warp < HB) {
            float* sc = s_sc + warp * kGqaChunk;
            const float a0 = sc[lane], a1 = sc[lane + 32];
            const float m_old = s_m[warp], m_new = fmaxf(m_old, warp_max(fmaxf(a0, a1)));
            const float e0 = m_new == -INFINITY ? 0.f : expf(a0 - m_new), e1 = m_new == -INFINITY ? 0.f : expf(a1 - m_new);
            sc[lane] = e0;
            sc[lane + 32] = e1;
            const float l = warp_sum(e0 + e1);
            if (lane == 0) {
                const float f = m_new == -INFINITY ? 1.f : expf(m_old - m_new);
                s_c[warp] = f;
                s_m[warp] = m_new;
                s_l[warp] = s_l[warp] * f + l;
            }
        }
        __syncthreads();
#pragma unroll
        for (int h = 0; h < HB; ++h) {
            const float f = s_c[h];
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[h][i] *= f;
        }
#pragma unroll
        for (int i = 0; i < kIters; ++i) {
            const uint32_t kk = i * kGroups + vgroup, j = k0 + kk;
            if (j > P || vcol >= p.vdim_p) continue;
            if (append && j == P) vr[i] = Cache8<CT>::fetch(s_v + vcol);
            float vv[8];
            Cache8<CT>::widen(vv, vr[i]);
#pragma unroll
            for (int h = 0; h < HB; ++h) {
                const float pr = s_sc[h * kGqaChunk + kk];
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[h][e] = fmaf(pr, vv[e], acc[h][e]);
            }
        }
        __syncthreads();
    }
    // value rows of a warp, then of the CTA, in a fixed order
#pragma unroll
    for (int h = 0; h < HB; ++h)
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            float v = acc[h][i];
#pragma unroll
            for (int o = L; o < 32; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            if (lane < L) s_red[(warp * HB + h) * (L * 8) + vcol + i] = v;
        }
    __syncthreads();
    const uint32_t part = p.vdim_p + 2;
    float* s_part = s_red + kGqaWarps * HB * L * 8 + 4 * HB + (p.dim_p + p.vdim_p) * sizeof(CT) / 4;      // behind s_v: [HB][part]
    for (uint32_t e = threadIdx.x; e < nh * p.vdim_p; e += kGqaThreads) {
        const uint32_t h = e / p.vdim_p, col = e - h * p.vdim_p;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kGqaWarps; ++w) v += s_red[(w * HB + h) * (L * 8) + col];
        const float m = s_m[h], l = s_l[h];
        if (p.splits == 1) {
            if (col < a.vdim) {
                const float M = a.sink ? fmaxf(m, 0.f) : m, f = expf(m - M);
                gqa_store_out(a.out, p.out_bf16, size_t(t) * a.out_ld + (h0 + h) * a.vdim + col, v * f / (l * f + (a.sink ? expf(-M) : 0.f)));
            }
        } else if (p.clustered) {
            s_part[h * part + 2 + col] = v;
            if (col == 0) { s_part[h * part] = m; s_part[h * part + 1] = l; }
        } else {
            float* dst = p.scratch + ((size_t(t) * a.heads + h0 + h) * p.splits + blockIdx.y) * part;
            dst[2 + col] = v;
            if (col == 0) { dst[0] = m; dst[1] = l; }
        }
    }
    if (p.clustered) {
        cluster_sync();                                    // every CTA's partial sums are in its shared memory
        // each CTA combines its slice of the values
        const uint32_t all = nh * a.vdim, slice = (all + p.splits - 1) / p.splits, e_end = min(all, (blockIdx.y + 1) * slice);
        for (uint32_t e = blockIdx.y * slice + threadIdx.x; e < e_end; e += kGqaThreads) {
            const uint32_t h = e / a.vdim, col = e - h * a.vdim;
            const float* mine = s_part + h * part;
            float m[kGqaCluster], l[kGqaCluster], v[kGqaCluster];
#pragma unroll
            for (int s = 0; s < kGqaCluster; ++s) {        // all loads before the first use
                const uint32_t rank = min(uint32_t(s), p.splits - 1);
                m[s] = cluster_load(mine, rank);
                l[s] = cluster_load(mine + 1, rank);
                v[s] = cluster_load(mine + 2 + col, rank);
            }
            float M = a.sink ? 0.f : -INFINITY, num = 0.f;
#pragma unroll
            for (int s = 0; s < kGqaCluster; ++s) M = fmaxf(M, m[s]);
            float den = a.sink ? expf(-M) : 0.f;
#pragma unroll
            for (int s = 0; s < kGqaCluster; ++s) {
                const float f = uint32_t(s) < p.splits ? expf(m[s] - M) : 0.f;
                den = fmaf(f, l[s], den);
                num = fmaf(f, v[s], num);
            }
            gqa_store_out(a.out, p.out_bf16, size_t(t) * a.out_ld + (h0 + h) * a.vdim + col, num / den);
        }
        cluster_sync();                                    // no CTA leaves while another reads its shared memory
        return;
    }
    if (p.splits == 1) return;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        uint32_t* counter = p.counters + size_t(t) * gridDim.x + blockIdx.x;
        s_last = atomicAdd(counter, 1u) == p.splits - 1 ? 1u : 0u;
        if (s_last) *counter = 0u;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    // the last CTA weighs the shares: warp h forms exp(m_s - M) / denominator of head h for every share (splits <= kGqaMaxSplits)
    float* s_w = s_red;                                    // [HB][kGqaMaxSplits]
    if (warp < int(nh)) {
        const float* src = p.scratch + (size_t(t) * a.heads + h0 + warp) * p.splits * part;
        float m[kGqaMaxSplits / 32], l[kGqaMaxSplits / 32], M = a.sink ? 0.f : -INFINITY, den = 0.f;
#pragma unroll
        for (int i = 0; i < kGqaMaxSplits / 32; ++i) {
            const uint32_t s = i * 32 + lane;
            m[i] = s < p.splits ? __ldcg(src + s * part) : -INFINITY;
            l[i] = s < p.splits ? __ldcg(src + s * part + 1) : 0.f;
            M = fmaxf(M, m[i]);
        }
        M = warp_max(M);
#pragma unroll
        for (int i = 0; i < kGqaMaxSplits / 32; ++i) {
            m[i] = expf(m[i] - M);
            den = fmaf(m[i], l[i], den);
        }
        const float inv = 1.f / (warp_sum(den) + (a.sink ? expf(-M) : 0.f));
#pragma unroll
        for (int i = 0; i < kGqaMaxSplits / 32; ++i) s_w[warp * kGqaMaxSplits + i * 32 + lane] = m[i] * inv;
    }
    __syncthreads();
    for (uint32_t e = threadIdx.x; e < nh * a.vdim; e += kGqaThreads) {
        const uint32_t h = e / a.vdim, col = e - h * a.vdim;
        const float* src = p.scratch + (size_t(t) * a.heads + h0 + h) * p.splits * part + 2 + col;
        float v = 0.f;
#pragma unroll 8
        for (uint32_t s = 0; s < p.splits; ++s) v = fmaf(s_w[h * kGqaMaxSplits + s], __ldcg(src + s * part), v);
        gqa_store_out(a.out, p.out_bf16, size_t(t) * a.out_ld + (h0 + h) * a.vdim + col, v);
    }
}

static uint32_t pad8(uint32_t n) { return (n + 7) / 8 * 8; }

static uint32_t gqa_head_blocks(const lv_gqa_args& a) { return (a.heads / a.kv_heads + kGqaHeads - 1) / kGqaHeads; }

// CTAs that share a token's keys: enough to fill the SMs about twice, at most one per chunk of the capacity
static uint32_t gqa_splits(const lv_ctx* ctx, const lv_gqa_args& a, uint32_t batch, uint32_t capacity) {
    const uint32_t ctas = a.kv_heads * gqa_head_blocks(a) * batch, chunks = (capacity + kGqaChunk - 1) / kGqaChunk;
    const uint32_t want = (2u * uint32_t(ctx->sm_count) + ctas - 1) / ctas;
    return std::max(1u, std::min({want, chunks, uint32_t(kGqaMaxSplits)}));
}

static int gqa_check(const lv_gqa_args* a, uint32_t batch) {
    LV_REQUIRE(a && a->qkv && a->q_norm && a->k_norm && a->r1 && a->r2 && a->k_cache && a->v_cache && a->pos && batch && batch <= 65535, "bad attention arguments");
    LV_REQUIRE(a->heads && a->kv_heads && a->heads % a->kv_heads == 0 && a->dim && a->vdim && a->dim <= 256 && a->vdim <= 256, "attention: unsupported head sizes");
    LV_REQUIRE(a->qkv_ld >= (a->heads + a->kv_heads) * a->dim + a->kv_heads * a->vdim && a->ctx_rows, "attention: bad strides");
    LV_REQUIRE(a->cache_type == LV_TYPE_F32 || a->cache_type == LV_TYPE_BF16, "attention: cache type");
    return LV_OK;
}

template <typename CT, int HB, int L>
static int gqa_launch_typed(lv_ctx* ctx, const GqaParams& p, uint32_t batch) {
    const size_t smem = sizeof(float) * (size_t(HB) * p.dim_p + HB * kGqaChunk + size_t(kGqaWarps) * HB * L * 8 + 4 * HB + size_t(HB) * (p.vdim_p + 2)) + sizeof(CT) * (p.dim_p + p.vdim_p) + 16;
    static_assert(kGqaWarps * L * 8 >= kGqaMaxSplits, "the combination's weights reuse the reduction buffer");
    LV_REQUIRE(smem <= size_t(ctx->max_smem_optin), "attention: head sizes need too much shared memory");
    auto* kernel = gqa_kernel<CT, HB, L>;
    if (smem > 48 * 1024) LV_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    const dim3 grid(p.a.kv_heads * p.head_blocks, p.splits, batch);
    if (!p.clustered) {
        LV_CUDA(launch_pdl(ctx, kernel, grid, dim3(kGqaThreads), smem, p));
        return LV_OK;
    }
    if (p.splits > 8) LV_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
    LV_CUDA(launch_pdl_cluster(ctx, kernel, grid, dim3(kGqaThreads), dim3(1, p.splits), smem, p));
    return LV_OK;
}

template <typename CT, int L>
static int gqa_launch_heads(lv_ctx* ctx, const GqaParams& p, uint32_t batch) {
    const uint32_t group = p.a.heads / p.a.kv_heads;
    if (group >= 5) return gqa_launch_typed<CT, 8, L>(ctx, p, batch);
    if (group >= 3) return gqa_launch_typed<CT, 4, L>(ctx, p, batch);
    if (group == 2) return gqa_launch_typed<CT, 2, L>(ctx, p, batch);
    return gqa_launch_typed<CT, 1, L>(ctx, p, batch);
}

template <typename CT>
static int gqa_launch(lv_ctx* ctx, const GqaParams& p, uint32_t batch) {
    const uint32_t widest = std::max(p.dim_p, p.vdim_p);
    if (widest <= 64) return gqa_launch_heads<CT, 8>(ctx, p, batch);
    if (widest <= 128) return gqa_launch_heads<CT, 16>(ctx, p, batch);
    return gqa_launch_heads<CT, 32>(ctx, p, batch);
}

}  // namespace lv

using namespace lv;

extern "C" size_t lv_gqa_scratch_bytes(lv_ctx* ctx, const lv_gqa_args* a, uint32_t batch, uint32_t capacity) {
    if (!ctx || !a || !batch || !capacity || !a->kv_heads) return 0;
    size_t most = 0;
    for (uint32_t n = 1; n <= batch; n *= 2) {             // splits shrink as the batch grows; every size in between needs no more than 2x
        const size_t bytes = 2 * size_t(n) * a->heads * gqa_splits(ctx, *a, n, capacity) * (pad8(a->vdim) + 2) * 4;
        most = bytes > most ? bytes : most;
    }
    return most + kGqaCounterBytes;
}

extern "C" int lv_qk_norm_append(lv_ctx* ctx, const lv_gqa_args* a, uint32_t batch) {
    LV_ENTER(ctx);
    if (const int rc = gqa_check(a, batch)) return rc;
    GqaParams p{};
    p.a = *a;
    p.dim_p = pad8(a->dim);
    p.vdim_p = pad8(a->vdim);
    p.err = ctx->d_err;
    const dim3 grid((batch * a->kv_heads + 3) / 4);
    if (a->cache_type == LV_TYPE_F32) LV_CUDA(launch_pdl(ctx, qk_norm_append_kernel<float>, grid, dim3(128), 0, p, batch));
    else LV_CUDA(launch_pdl(ctx, qk_norm_append_kernel<__nv_bfloat16>, grid, dim3(128), 0, p, batch));
    return LV_OK;
}

extern "C" int lv_attention_gqa(lv_ctx* ctx, const lv_gqa_args* a, void* scratch, size_t scratch_bytes, uint32_t batch, uint32_t capacity, int append) {
    LV_ENTER(ctx);
    if (const int rc = gqa_check(a, batch)) return rc;
    LV_REQUIRE(a->out && a->out_ld >= a->heads * a->vdim && (a->out_type == LV_TYPE_F32 || a->out_type == LV_TYPE_BF16), "attention: bad output");
    LV_REQUIRE(capacity && capacity <= a->ctx_rows && (!append || batch == 1), "attention: bad capacity");
    if (!append && gqa_tc_supported(*a, batch)) return gqa_tc_launch(ctx, *a, batch);
    GqaParams p{};
    p.a = *a;
    p.dim_p = pad8(a->dim);
    p.vdim_p = pad8(a->vdim);
    p.head_blocks = gqa_head_blocks(*a);
    p.splits = gqa_splits(ctx, *a, batch, capacity);
    // up to 64 chunks of keys are shared by a cluster of at most 16 CTAs; longer contexts need more CTAs than a cluster has
    if (p.splits > 1 && capacity <= 64 * kGqaChunk) {
        p.splits = std::min(p.splits, uint32_t(kGqaCluster));
        p.clustered = 1;
    }
    p.out_bf16 = a->out_type == LV_TYPE_BF16;
    p.err = ctx->d_err;
    if (p.splits > 1 && !p.clustered) {
        // fewer than two CTAs per SM would run unsplit, so the counters of a split launch always fit
        LV_REQUIRE(size_t(batch) * a->kv_heads * p.head_blocks * 4 <= kGqaCounterBytes, "attention: too many arrival counters");
        const size_t need = kGqaCounterBytes + size_t(batch) * a->heads * p.splits * (p.vdim_p + 2) * 4;
        LV_REQUIRE(scratch && scratch_bytes >= need, "attention: scratch too small");
        p.counters = static_cast<uint32_t*>(scratch);
        p.scratch = reinterpret_cast<float*>(static_cast<uint8_t*>(scratch) + kGqaCounterBytes);
    }
    p.append = append != 0;
    return a->cache_type == LV_TYPE_F32 ? gqa_launch<float>(ctx, p, batch) : gqa_launch<__nv_bfloat16>(ctx, p, batch);
}
