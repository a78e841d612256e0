// The attention of attention_gqa.cu and attention_latent.cu for the tokens of a prompt, on the tcgen05 tensor cores (bfloat16
// caches).
//
// A CTA takes 128 query rows of one key/value head -- row r is query head r mod group of token r / group, so that grouped
// heads share the keys -- and walks the keys in blocks of 64:
//
//   S = Q K^T      Q normalised, scaled and rounded to bfloat16 in shared memory (128-byte swizzle), K by TMA from the cache
//   P = exp2(S - bias - m)      one row per thread; P goes to tensor memory over the scores it came from
//   O += P V       P is the TMEM operand, V by TMA as an MN-major operand (its rows are keys)
//
// Two threads share a row where tensor memory allows (values of up to 192): each takes one half of every key block, with its
// own running maximum, sum and O, and the halves meet once, at the end.  A prompt has few tiles per SM, so the softmax is
// bound by the latency of a thread's chain, which this halves.
//
// Two score buffers let S of the next block run under the softmax of this one.  The distance bias of a block is a small
// table per head: distances within a block and a tile differ by less than (tokens + 64), so the logarithm is evaluated
// once per (head, distance) instead of once per score.  O stays in tensor memory; it is rescaled only when a row's maximum has grown
// by more than 2^8, which with a sink (maximum >= 0 from the start) is rare.  Everything except the operands is f32.
//
// Latent caches (LATENT): every head has keys and values of its own, expanded from the cache before the launch; a key is the head's
// part from there and the rotated part from the cache itself, side by side in shared memory.  The query is rotated instead of
// normalised, there is no distance bias, a row sees a window of positions (a tile begins at the first row's window), and the
// sink is a logit per head that the running maximum starts from.
//
// Every wait is bounded (common.cuh); a lost wait sets the error word, the CTA drains and frees its tensor memory.
#include <cuda.h>
#include <cuda_bf16.h>
#include <math.h>

#include "attention_gqa.cuh"
#include "common.cuh"
#include "ctx.h"
#include "tcgen05.cuh"
#include "tmap.h"

namespace lv {

// warps: TMA, S products, P V products (each issued by one lane: a single lane would spend longer on the instructions and
// waits of both than the softmax takes), then four softmax warps per half
constexpr int kGtFirstSoftmax = 3;
constexpr int kGtRows = 128, kGtKeys = 64;
constexpr uint32_t kGtQChunk = kGtRows * 128, kGtKChunk = kGtKeys * 128;      // 64 columns of Q / of K or V, bytes
constexpr uint32_t kGtMaxStages = 4;
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kGtRescaleStep = 8.f;        // log2

struct GqaTcParams {
    lv_gqa_args a;
    uint32_t n_tokens, dim_chunks, dim16, v_chunks, vdim16, stages, tmem_cols, tab_stride, tab_tokens;
    uint32_t out_bf16;
    // LATENT (heads == kv_heads: the heads of this launch)
    uint32_t own_chunks, own_steps, steps;       // chunks of the head's own key part; MMA steps of it and of the whole key
    uint32_t rot, angle_ld, angle_pairs, window, v_at;
    const float* angles;
    const float* sinks;
    uint32_t* err;
};

struct GqaTcMaps {
    CUtensorMap k, v, rot;
};

// V: rows are keys (the K of the MMA), 64 columns per 128-byte row; 8-key groups 1024 bytes apart, 64-column blocks kGtKChunk apart
__device__ __forceinline__ uint64_t gt_v_desc(uint32_t smem_addr, uint32_t block_bytes) {
    return uint64_t((smem_addr >> 4) & 0x3fffu) | (uint64_t(block_bytes >> 4) << 16) | (uint64_t(1024 >> 4) << 32) | (uint64_t(1) << 46) | (uint64_t(2) << 61);
}

__device__ __forceinline__ uint32_t gt_pack(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}

__device__ __forceinline__ void gt_store16(uint32_t taddr, const uint32_t (&u)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
        ::"r"(taddr), "r"(u[0]), "r"(u[1]), "r"(u[2]), "r"(u[3]), "r"(u[4]), "r"(u[5]), "r"(u[6]), "r"(u[7]), "r"(u[8]), "r"(u[9]), "r"(u[10]), "r"(u[11]),
          "r"(u[12]), "r"(u[13]), "r"(u[14]), "r"(u[15])
        : "memory");
}
__device__ __forceinline__ void gt_wait_store() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

__device__ __forceinline__ float gt_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// NH: halves a row is split into; PAIRS: 64 PAIRS >= head size (chunks of a key for LATENT)
template <int NH, int PAIRS, bool LATENT>
__global__ void __launch_bounds__(32 * kGtFirstSoftmax + 128 * NH) gqa_tc_kernel(const GqaTcParams p, const __grid_constant__ GqaTcMaps maps) {
    pdl_launch_dependents();
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023u) & ~uintptr_t(1023));
    const lv_gqa_args& a = p.a;
    uint8_t* s_q = smem;
    uint8_t* s_kv = s_q + p.dim_chunks * kGtQChunk;
    const uint32_t k_bytes = p.dim_chunks * kGtKChunk, v_bytes = p.v_chunks * kGtKChunk, stage = k_bytes + v_bytes;
    float* s_tab = reinterpret_cast<float*>(s_kv + p.stages * stage);           // [2][group][tab_stride]
    constexpr int kThreads = 32 * kGtFirstSoftmax + 128 * NH, kHalfKeys = kGtKeys / NH;
    __shared__ float s_ml[2][kGtRows];                           // maximum and sum of the second half
    __shared__ uint64_t k_full[kGtMaxStages], v_full[kGtMaxStages], kv_empty[kGtMaxStages], s_full[2], p_full[2], pv_done[2];
    __shared__ uint32_t s_tmem;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const uint32_t group = a.heads / a.kv_heads, g = blockIdx.y;
    const uint32_t r0 = blockIdx.x * kGtRows, rows_all = p.n_tokens * group;
    const uint32_t t_first = r0 / group, t_last = min(rows_all - 1, r0 + kGtRows - 1) / group;

    if (threadIdx.x == 0) {
        for (uint32_t i = 0; i < kGtMaxStages; ++i) { mbar_init(&k_full[i], 1); mbar_init(&v_full[i], 1); mbar_init(&kv_empty[i], 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_full[i], 4 * NH); mbar_init(&pv_done[i], 1); }
        fence_mbar_init();
    }
    if (warp == 1) tc_alloc(&s_tmem, p.tmem_cols);
    pdl_wait();
    const uint32_t P = *a.pos;
    const bool inside = P + p.n_tokens <= a.ctx_rows;            // (lv_qk_norm_append reports positions beyond the cache)
    // first key of the tile, and of the launch
    const uint32_t tile_first = LATENT && p.window != 0 && P + t_first + 1 > p.window ? P + t_first + 1 - p.window : 0;
    const uint32_t step_first = LATENT && p.window != 0 && P + 1 > p.window ? P + 1 - p.window : 0;
    const uint32_t n_keys = P + t_last + 1 - tile_first, n_blocks = inside ? (n_keys + kGtKeys - 1) / kGtKeys : 0;
    // Q rows: a warp takes several rows at a time, lanes across the head (pairs of columns), all loads before the first sum
    constexpr int kPairs = PAIRS, kBatch = PAIRS <= 2 ? 16 : 8;
    float qw[2 * kPairs];
#pragma unroll
    for (int c2 = 0; c2 < kPairs; ++c2) {
        const uint32_t c = 2 * (uint32_t(lane) + 32 * c2);
        qw[2 * c2] = LATENT ? 1.f : c < a.dim ? a.q_norm[c] : 0.f;
        qw[2 * c2 + 1] = LATENT ? 1.f : c + 1 < a.dim ? a.q_norm[c + 1] : 0.f;
    }
    const uint32_t rot_at = LATENT ? p.own_chunks * 64u : 0;     // column of the rotated part
    for (uint32_t b0 = uint32_t(warp) * kBatch; b0 < uint32_t(kGtRows); b0 += kThreads / 32 * kBatch) {
        float v[kBatch][2 * kPairs], part[kBatch];
#pragma unroll
        for (int i = 0; i < kBatch; ++i) {
            const uint32_t row = r0 + b0 + i, t = row / group, h = g * group + (row - t * group);
            const float* q = a.qkv + size_t(t) * a.qkv_ld + h * (LATENT ? a.dim + p.rot : a.dim);
#pragma unroll
            for (int c2 = 0; c2 < kPairs; ++c2) {
                const uint32_t c = 2 * (uint32_t(lane) + 32 * c2);
                if constexpr (LATENT) {
                    float lo = 0.f, hi = 0.f;
                    if (row < rows_all && c < rot_at) {
                        if (c < a.dim) lo = q[c];
                        if (c + 1 < a.dim) hi = q[c + 1];
                    } else if (row < rows_all && c - rot_at < p.rot) {
                        const uint32_t r = c - rot_at;
                        lo = q[a.dim + r];
                        hi = r + 1 < p.rot ? q[a.dim + r + 1] : 0.f;
                        if (r < 2 * p.angle_pairs) {
                            const float2 cs = *reinterpret_cast<const float2*>(p.angles + size_t(t) * p.angle_ld + r);
                            const float u = lo;
                            lo = u * cs.x - hi * cs.y;
                            hi = hi * cs.x + u * cs.y;
                        }
                    }
                    v[i][2 * c2] = lo;
                    v[i][2 * c2 + 1] = hi;
                    continue;
                }
                v[i][2 * c2] = row < rows_all && c < a.dim ? q[c] : 0.f;
                v[i][2 * c2 + 1] = row < rows_all && c + 1 < a.dim ? q[c + 1] : 0.f;
            }
        }
#pragma unroll
        for (int i = 0; i < kBatch; ++i) {
            part[i] = 0.f;
#pragma unroll
            for (int c = 0; c < 2 * kPairs; ++c) part[i] = fmaf(v[i][c], v[i][c], part[i]);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int i = 0; i < kBatch; ++i) part[i] += __shfl_xor_sync(0xffffffffu, part[i], o);
#pragma unroll
        for (int i = 0; i < kBatch; ++i) {
            const float f = LATENT ? a.scale * kLog2e : a.scale * kLog2e / sqrtf(part[i] / float(a.dim) + a.eps);
            const uint32_t r = b0 + i;
#pragma unroll
            for (int c2 = 0; c2 < kPairs; ++c2) {
                const uint32_t c = 2 * (uint32_t(lane) + 32 * c2);
                if (c >= p.dim_chunks * 64) continue;
                const uint32_t in = c & 63u, off = (r >> 3) * 1024u + (r & 7u) * 128u + (((in >> 3) ^ (r & 7u)) << 4) + (in & 7u) * 2u;
                *reinterpret_cast<uint32_t*>(s_q + (c >> 6) * kGtQChunk + off) = gt_pack(v[i][2 * c2] * f * qw[2 * c2], v[i][2 * c2 + 1] * f * qw[2 * c2 + 1]);
            }
        }
    }
    fence_proxy_async();
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(&s_tmem);
    const uint32_t tmem_o = tmem + 2 * kGtKeys;
    bool ok = true;

    if (warp == 0) {
        if (lane == 0) {
            uint32_t s = 0, phase = 1;                           // the first pass over the ring finds it empty
            for (uint32_t b = 0; b < n_blocks; ++b) {
                if (b >= p.stages && !mbar_wait(&kv_empty[s], phase, p.err)) break;
                const int y = LATENT ? int(tile_first - step_first + b * kGtKeys) : int(g * a.ctx_rows + b * kGtKeys);
                uint8_t* dst = s_kv + s * stage;
                mbar_expect_tx(&k_full[s], k_bytes);
                if constexpr (LATENT) {
                    for (uint32_t c = 0; c < p.own_chunks; ++c) tma_load_2d_plain(dst + c * kGtKChunk, &maps.k, int(g * a.dim + c * 64), y, &k_full[s]);
                    for (uint32_t c = p.own_chunks; c < p.dim_chunks; ++c)
                        tma_load_2d_plain(dst + c * kGtKChunk, &maps.rot, int((c - p.own_chunks) * 64), int(tile_first + b * kGtKeys), &k_full[s]);
                } else {
                    for (uint32_t c = 0; c < p.dim_chunks; ++c) tma_load_2d_plain(dst + c * kGtKChunk, &maps.k, int(c * 64), y, &k_full[s]);
                }
                const int vx = LATENT ? int(p.v_at + g * a.vdim) : 0;
                mbar_expect_tx(&v_full[s], v_bytes);
                for (uint32_t c = 0; c < p.v_chunks; ++c) tma_load_2d_plain(dst + k_bytes + c * kGtKChunk, &maps.v, vx + int(c * 64), y, &v_full[s]);
                if (++s == p.stages) { s = 0; phase ^= 1u; }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | (uint32_t(kGtRows >> 4) << 24) | (uint32_t(kGtKeys >> 3) << 17);
            const uint64_t q_desc = tc_smem_desc(smem_u32(s_q)), k_desc0 = tc_smem_desc(smem_u32(s_kv));
            const uint32_t k_steps = LATENT ? p.steps : p.dim16 / 16;
            uint32_t ks = 0, k_phase = 0;
            for (uint32_t b = 0; b < n_blocks && ok; ++b) {
                // the buffer held P of block b - 2
                ok = mbar_wait(&k_full[ks], k_phase, p.err) && (b < 2 || mbar_wait(&pv_done[b & 1u], ((b >> 1) - 1u) & 1u, p.err));
                if (!ok) break;
                tc_fence_after_sync();
                const uint64_t kd = k_desc0 + ((ks * stage) >> 4);
                for (uint32_t k = 0; k < k_steps; ++k) {
                    const uint32_t at = LATENT && k >= p.own_steps ? p.own_chunks * 4 + k - p.own_steps : k, c = at >> 2, in = (at & 3u) * 2u;
                    tc_mma_f16(tmem + (b & 1u) * kGtKeys, q_desc + ((c * kGtQChunk) >> 4) + in, kd + ((c * kGtKChunk) >> 4) + in, idesc, k != 0 ? 1u : 0u);
                }
                tc_commit(&s_full[b & 1u]);
                if (++ks == p.stages) { ks = 0; k_phase ^= 1u; }
            }
        }
    } else if (warp == 2) {
        if (lane == 0) {
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((p.vdim16 >> 3) << 17) | (uint32_t(kGtRows >> 4) << 24);      // B is MN-major
            const uint64_t v_desc0 = gt_v_desc(smem_u32(s_kv) + k_bytes, p.v_chunks > 1 ? kGtKChunk : 1024u);
            uint32_t vs = 0, v_phase = 0;
            for (uint32_t b = 0; b < n_blocks && ok; ++b) {
                ok = mbar_wait(&p_full[b & 1u], (b >> 1) & 1u, p.err) && mbar_wait(&v_full[vs], v_phase, p.err);
                if (!ok) break;
                tc_fence_after_sync();
                const uint64_t vd = v_desc0 + ((vs * stage) >> 4);
#pragma unroll
                for (uint32_t k = 0; k < kGtKeys / 16; ++k) {    // 16 keys: 8 columns of P, two 8-key groups of V
                    const uint32_t half = k / (kHalfKeys / 16), in = k - half * (kHalfKeys / 16);
                    tc_mma_f16_ta(tmem_o + half * p.vdim16, tmem + (b & 1u) * kGtKeys + half * kHalfKeys + 8u * in, vd + 128u * k, idesc,
                                  (b != 0 || in != 0) ? 1u : 0u);
                }
                tc_commit(&pv_done[b & 1u]);
                tc_commit(&kv_empty[vs]);                        // (the S product of the block is older: its softmax has been here)
                if (++vs == p.stages) { vs = 0; v_phase ^= 1u; }
            }
        }
    } else {
        // ---- softmax: a row (or half of its keys) per thread ---------------------------------------
        const uint32_t quarter = uint32_t(warp) & 3u, tr = quarter * 32u + uint32_t(lane), st = threadIdx.x - 32u * kGtFirstSoftmax;
        const uint32_t half = (uint32_t(warp) - kGtFirstSoftmax) >> 2, key0 = half * kHalfKeys;
        const uint32_t row = r0 + tr, t = min(row, rows_all - 1) / group, hl = min(row, rows_all - 1) - t * group;
        const uint32_t lanes = quarter * 32u << 16, o_half = tmem_o + lanes + half * p.vdim16;
        // the bias table's entries: 32 of one head per warp and job; the first jobs of a warp keep their constants in registers
        constexpr int kJobs = 4;
        const uint32_t tab_jobs = (p.tab_tokens + 31) / 32, all_jobs = group * tab_jobs;
        float job_r1[kJobs], job_r2[kJobs];
        uint32_t job_at[kJobs];
        int job_d[kJobs];
#pragma unroll
        for (int k = 0; k < (LATENT ? 0 : kJobs); ++k) {
            const uint32_t job = uint32_t(warp) - kGtFirstSoftmax + k * 4 * NH, h = job / tab_jobs, i = (job - h * tab_jobs) * 32 + lane;
            const bool live = job < all_jobs && i < p.tab_tokens;
            job_r1[k] = live ? a.r1[g * group + h] : 0.f;
            job_r2[k] = live ? a.r2[g * group + h] : 0.f;
            job_at[k] = live ? h * p.tab_stride + i : ~0u;
            job_d[k] = int(i);
        }
        const float sink = LATENT ? (p.sinks ? p.sinks[g] * kLog2e : -INFINITY) : a.sink ? 0.f : -INFINITY;      // log2 of the sink's share
        float m = sink, l = 0.f;
        uint32_t vs = 0, v_phase = 0;
        // (after a lost wait the warp goes through the remaining blocks without work: the others wait for it at the barrier)
        for (uint32_t b = 0; b < n_blocks; ++b) {
            const uint32_t k0 = tile_first + b * kGtKeys, s_at = tmem + lanes + (b & 1u) * kGtKeys + key0;
            [[maybe_unused]] float* tab = s_tab + (b & 1u) * group * p.tab_stride;
            if constexpr (!LATENT) {
                // bias table of this block: entry i of a head is distance (P + t_first) - (k0 + 63) + i
                const int d0 = int(P + t_first) - int(k0 + kGtKeys - 1);
#pragma unroll
                for (int k = 0; k < kJobs; ++k)
                    if (job_at[k] != ~0u) tab[job_at[k]] = job_r1[k] * __log2f(fmaf(job_r2[k], float(max(d0 + job_d[k], 0)), 1.f));
                for (uint32_t job = uint32_t(warp) - kGtFirstSoftmax + kJobs * 4 * NH; job < all_jobs; job += 4 * NH) {
                    const uint32_t h = job / tab_jobs, i = (job - h * tab_jobs) * 32 + lane;
                    if (i < p.tab_tokens) tab[h * p.tab_stride + i] = a.r1[g * group + h] * __log2f(fmaf(a.r2[g * group + h], float(max(d0 + int(i), 0)), 1.f));
                }
                asm volatile("bar.sync 1, %0;" ::"n"(128 * NH) : "memory");
            }
            ok = ok && mbar_wait_warp(&s_full[b & 1u], (b >> 1) & 1u, p.err);
            if (!ok) continue;
            tc_fence_after_sync();
            float s[kHalfKeys];
            {
                uint32_t u[kHalfKeys / 16][16];
#pragma unroll
                for (int c = 0; c < kHalfKeys / 16; ++c) tc_load16(u[c], s_at + 16 * c);
                tc_wait_load();
#pragma unroll
                for (int c = 0; c < kHalfKeys; ++c) s[c] = __uint_as_float(u[c / 16][c % 16]);
            }
            [[maybe_unused]] const float* bias = tab + hl * p.tab_stride + (t - t_first) + (kGtKeys - 1) - key0;
            const int last = int(P + t) - int(k0 + key0);        // keys 0 .. last of this half are visible
            float tops[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            const int low = LATENT && p.window != 0 ? last + 1 - int(p.window) : -1;      // keys from `low` on
            if (k0 + kGtKeys - 1 <= P + t_first && (!LATENT || p.window == 0 || P + t_last - k0 < p.window)) {
#pragma unroll
                for (int j = 0; j < kHalfKeys; ++j) {
                    if constexpr (!LATENT) s[j] -= bias[-j];
                    tops[j & 3] = fmaxf(tops[j & 3], s[j]);
                }
            } else {
#pragma unroll
                for (int j = 0; j < kHalfKeys; ++j) {
                    if constexpr (LATENT) s[j] = j <= last && j >= low ? s[j] : -INFINITY;
                    else s[j] = j <= last ? s[j] - bias[-j] : -INFINITY;
                    tops[j & 3] = fmaxf(tops[j & 3], s[j]);
                }
            }
            const float top = fmaxf(fmaxf(tops[0], tops[1]), fmaxf(tops[2], tops[3]));
            // a new maximum takes effect when it is far above the old one (or there was none)
            const bool grow = top > m + kGtRescaleStep;
            float f = 1.f;
            if (grow) {
                f = exp2f(m - top);                              // 0 when there was none
                m = top;
                l *= f;
            }
            if (__any_sync(0xffffffffu, grow) && b != 0) {
                ok = mbar_wait_warp(&pv_done[(b - 1) & 1u], ((b - 1) >> 1) & 1u, p.err);
                if (!ok) continue;
                tc_fence_after_sync();
                for (uint32_t c = 0; c < p.vdim16; c += 16) {
                    uint32_t u[16];
                    tc_load16(u, o_half + c);
                    tc_wait_load();
#pragma unroll
                    for (int i = 0; i < 16; ++i) u[i] = __float_as_uint(__uint_as_float(u[i]) * f);
                    gt_store16(o_half + c, u);
                }
                gt_wait_store();
            }
            const float base = m == -INFINITY ? 0.f : m;
            float sums[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int c = 0; c < kHalfKeys; c += 32) {
                uint32_t u[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float p0 = gt_exp2(s[c + 2 * i] - base), p1 = gt_exp2(s[c + 2 * i + 1] - base);
                    sums[(2 * i) & 3] += p0;
                    sums[(2 * i + 1) & 3] += p1;
                    u[i] = gt_pack(p0, p1);
                }
                gt_store16(s_at + c / 2, u);
            }
            l += (sums[0] + sums[1]) + (sums[2] + sums[3]);
            gt_wait_store();
            if (k0 + kGtKeys > P + p.n_tokens) {
                // rows of V behind the last token hold whatever the cache held: their weights are zero, but zero times NaN is not
                ok = mbar_wait_warp(&v_full[vs], v_phase, p.err);
                if (!ok) continue;
                uint8_t* v = s_kv + vs * stage + k_bytes;
                const uint32_t first = P + p.n_tokens - k0, n16 = (kGtKeys - first) * 8;
                for (uint32_t e = st; e < p.v_chunks * n16; e += 128 * NH) {
                    const uint32_t c = e / n16, i = e - c * n16;
                    *reinterpret_cast<uint4*>(v + c * kGtKChunk + first * 128 + i * 16) = make_uint4(0u, 0u, 0u, 0u);
                }
                fence_proxy_async();
            }
            if (++vs == p.stages) { vs = 0; v_phase ^= 1u; }
            tc_fence_before_sync();
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[b & 1u]);
        }
        if (n_blocks != 0) {
            ok = ok && mbar_wait_warp(&pv_done[(n_blocks - 1) & 1u], ((n_blocks - 1) >> 1) & 1u, p.err);
            tc_fence_after_sync();
            float fa = 1.f, fb = 0.f;                            // weights of the two halves' sums
            if constexpr (NH == 2) {
                if (half == 1) { s_ml[0][tr] = m; s_ml[1][tr] = l; }
                asm volatile("bar.sync 1, %0;" ::"n"(128 * NH) : "memory");
                if (half == 0) {
                    const float mb = s_ml[0][tr], lb = s_ml[1][tr], M = fmaxf(m, mb);
                    fa = exp2f(m - M);
                    fb = exp2f(mb - M);
                    l = l * fa + lb * fb;
                    m = M;
                }
            }
            if (ok && half == 0) {
                const float inv = 1.f / (l + exp2f(sink - m));
                fa *= inv;
                fb *= inv;
                const size_t at = size_t(t) * a.out_ld + (g * group + hl) * a.vdim;
                for (uint32_t c = 0; c < p.vdim16; c += 16) {
                    uint32_t u[NH][16];
#pragma unroll
                    for (int h = 0; h < NH; ++h) tc_load16(u[h], o_half + h * p.vdim16 + c);
                    tc_wait_load();
                    if (row >= rows_all) continue;
                    float o[16];
#pragma unroll
                    for (int i = 0; i < 16; ++i)
                        o[i] = NH == 2 ? fmaf(__uint_as_float(u[NH - 1][i]), fb, __uint_as_float(u[0][i]) * fa) : __uint_as_float(u[0][i]) * fa;
                    if (p.out_bf16 && c + 16 <= a.vdim && (at + c) % 8 == 0) {
                        uint4 w[2];
                        uint32_t* ww = reinterpret_cast<uint32_t*>(w);
#pragma unroll
                        for (int i = 0; i < 8; ++i) ww[i] = gt_pack(o[2 * i], o[2 * i + 1]);
                        uint4* dst = reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.out) + at + c);
                        dst[0] = w[0];
                        dst[1] = w[1];
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (c + i < a.vdim) gqa_store_out(a.out, p.out_bf16, at + c + i, o[i]);
                    }
                }
            }
        }
        tc_fence_before_sync();
    }
    __syncthreads();
    if (warp == 1) {
        tc_fence_after_sync();
        tc_free(tmem, p.tmem_cols);
    }
}

bool gqa_tc_supported(const lv_gqa_args& a, uint32_t batch) {
    return a.cache_type == LV_TYPE_BF16 && batch > 1 && a.heads / a.kv_heads <= 64;
}

int gqa_tc_launch(lv_ctx* ctx, const lv_gqa_args& a, uint32_t batch) {
    GqaTcParams p{};
    p.a = a;
    p.n_tokens = batch;
    const uint32_t dim_p = (a.dim + 7) / 8 * 8, vdim_p = (a.vdim + 7) / 8 * 8, group = a.heads / a.kv_heads;
    p.dim_chunks = (dim_p + 63) / 64;
    p.dim16 = (dim_p + 15) / 16 * 16;
    p.v_chunks = (vdim_p + 63) / 64;
    p.vdim16 = (vdim_p + 15) / 16 * 16;
    p.out_bf16 = a.out_type == LV_TYPE_BF16;
    p.err = ctx->d_err;
    const bool halves = 2 * kGtKeys + 2 * p.vdim16 <= 512;
    p.tmem_cols = 2 * kGtKeys + (halves ? 2 : 1) * p.vdim16 <= 256 ? 256 : 512;
    // tokens that a tile of 128 rows can touch, plus the keys of a block; heads 32 / group banks apart
    p.tab_tokens = (kGtRows + group - 1) / group + 1 + kGtKeys;
    const uint32_t want = group < 32 ? 32 / group : 1;
    p.tab_stride = p.tab_tokens;
    while (p.tab_stride % 32 != want % 32) ++p.tab_stride;
    const uint32_t stage = (p.dim_chunks + p.v_chunks) * kGtKChunk, q_bytes = p.dim_chunks * kGtQChunk, tab = 2 * group * p.tab_stride * 4;
    p.stages = 2;
    const uint32_t room = (p.tmem_cols == 512 ? 200 : 110) * 1024;       // two CTAs per SM where their tensor memory fits
    while (p.stages < kGtMaxStages && q_bytes + (p.stages + 1) * stage + tab + 1024 <= room) ++p.stages;
    const size_t smem = 1024 + size_t(q_bytes) + size_t(p.stages) * stage + tab;
    LV_REQUIRE(smem <= size_t(ctx->max_smem_optin), "attention: head sizes need too much shared memory");
    GqaTcMaps maps{};
    const uint64_t rows = uint64_t(a.kv_heads) * a.ctx_rows;
    LV_REQUIRE(rows <= 0x7fffffffu, "attention: cache too long");
    if (int rc = make_bf16_map(&maps.k, a.k_cache, rows, dim_p, dim_p, kGtKeys)) return rc;
    if (int rc = make_bf16_map(&maps.v, a.v_cache, rows, vdim_p, vdim_p, kGtKeys)) return rc;
    auto* kernel = halves ? (a.dim <= 128 ? gqa_tc_kernel<2, 2, false> : gqa_tc_kernel<2, 4, false>) : (a.dim <= 128 ? gqa_tc_kernel<1, 2, false> : gqa_tc_kernel<1, 4, false>);
    LV_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    LV_CUDA(launch_pdl(ctx, kernel, dim3((batch * group + kGtRows - 1) / kGtRows, a.kv_heads), dim3(32 * kGtFirstSoftmax + (halves ? 256 : 128)), smem, p, maps));
    return LV_OK;
}

bool latent_tc_supported(const lv_latent_args& a) {
    return a.cache_type == LV_TYPE_BF16 && a.dim % 8 == 0 && a.vdim % 8 == 0 && (a.dim + 63) / 64 + (a.rot + 63) / 64 <= 4 && a.vdim <= 256;
}

int latent_tc_launch(lv_ctx* ctx, const lv_latent_args& l, uint32_t batch, const void* kv, uint32_t ld, uint32_t v_at, uint32_t rows, uint32_t h0, uint32_t n) {
    GqaTcParams p{};
    lv_gqa_args& a = p.a;
    a.qkv = l.q + size_t(h0) * (l.dim + l.rot);
    a.qkv_ld = l.q_ld;
    a.heads = a.kv_heads = n;
    a.dim = l.dim;
    a.vdim = l.vdim;
    a.scale = l.scale;
    a.ctx_rows = l.ctx_rows;
    a.pos = l.pos;
    a.out = static_cast<uint8_t*>(l.out) + size_t(h0) * l.vdim * (l.out_type == LV_TYPE_BF16 ? 2 : 4);
    a.out_type = l.out_type;
    a.out_ld = l.out_ld;
    p.n_tokens = batch;
    p.own_chunks = (l.dim + 63) / 64;
    p.dim_chunks = p.own_chunks + (l.rot + 63) / 64;
    p.own_steps = (l.dim + 15) / 16;
    p.steps = p.own_steps + (l.rot + 15) / 16;
    p.v_chunks = (l.vdim + 63) / 64;
    p.vdim16 = (l.vdim + 15) / 16 * 16;
    p.out_bf16 = l.out_type == LV_TYPE_BF16;
    p.rot = l.rot;
    p.angles = l.angles;
    p.angle_ld = l.angle_ld;
    p.angle_pairs = l.angle_pairs;
    p.window = l.window;
    p.v_at = v_at;
    p.sinks = l.sink ? l.sink + h0 : nullptr;
    p.err = ctx->d_err;
    const bool halves = 2 * kGtKeys + 2 * p.vdim16 <= 512;
    p.tmem_cols = 2 * kGtKeys + (halves ? 2 : 1) * p.vdim16 <= 256 ? 256 : 512;
    const uint32_t stage = (p.dim_chunks + p.v_chunks) * kGtKChunk, q_bytes = p.dim_chunks * kGtQChunk;
    p.stages = 2;
    const uint32_t room = (p.tmem_cols == 512 ? 200 : 110) * 1024;
    while (p.stages < kGtMaxStages && q_bytes + (p.stages + 1) * stage + 1024 <= room) ++p.stages;
    const size_t smem = 1024 + size_t(q_bytes) + size_t(p.stages) * stage;
    LV_REQUIRE(smem <= size_t(ctx->max_smem_optin), "latent attention: head sizes need too much shared memory");
    LV_REQUIRE(l.ctx_rows <= 0x7fffffffu && n <= 65535, "latent attention: cache too long");
    const uint32_t rank_p = (l.kv_rank + 7) / 8 * 8, rot_p = (l.rot + 7) / 8 * 8;
    GqaTcMaps maps{};
    if (int rc = make_bf16_map(&maps.k, kv, rows, ld, ld, kGtKeys)) return rc;
    maps.v = maps.k;
    maps.rot = maps.k;
    if (l.rot != 0)
        if (int rc = make_bf16_map(&maps.rot, static_cast<const uint8_t*>(l.cache) + rank_p * 2, l.ctx_rows, rot_p, rank_p + rot_p, kGtKeys)) return rc;
    auto* kernel = halves ? (p.dim_chunks <= 2 ? gqa_tc_kernel<2, 2, true> : gqa_tc_kernel<2, 4, true>)
                          : (p.dim_chunks <= 2 ? gqa_tc_kernel<1, 2, true> : gqa_tc_kernel<1, 4, true>);
    LV_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    LV_CUDA(launch_pdl(ctx, kernel, dim3((batch + kGtRows - 1) / kGtRows, n), dim3(32 * kGtFirstSoftmax + (halves ? 256 : 128)), smem, p, maps));
    return LV_OK;
}

}  // namespace lv
