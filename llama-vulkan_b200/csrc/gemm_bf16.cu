// Products of several tokens with bfloat16 matrices on the tcgen05 tensor cores, dense and per expert.
//
//   out[t][r] = act(factor * sum_k W[r][k] x[t][k])        W and x bfloat16, sums f32
//
// A CTA covers 128 rows of W (the M of the MMA) and NT tokens (its N).  Both operands are K-major and come by TMA in boxes of
// 64 columns with the 128-byte swizzle, 4 to 8 stages deep; one lane issues the loads, one lane the MMAs, four warps read the
// accumulator from tensor memory (lane = row, column = token, so a warp stores 32 consecutive features of a token).  The
// first weight tiles are requested before the previous kernel has finished.  Matrices with few tiles are split along K over
// several CTAs: each leaves its partial sums in scratch and the last to arrive adds them in split order (deterministic).
//
// Experts: lv_expert_route sorts the (token, choice) pairs of a step by expert and lists tiles of NT rows; the input rows lie
// in that order (lv_norm_conv scatters them there), a tile multiplies them with its expert's rows of the stacked matrix.
// The gated pair keeps two accumulators, so gate and up of a feature meet in one thread.
//
// Windows (lv_gemm_bf16_window): x is a cache, and the rows to multiply are those that the step's tokens see; where they begin is
// only known on the device, so a tile finds its rows from the position word, and tiles behind the last row leave at once.
//
// Every wait is bounded (common.cuh); a lost wait sets the error word, the CTA drains and frees its tensor memory.
#include <cuda.h>
#include <cuda_bf16.h>

#include <algorithm>

#include "common.cuh"
#include "ctx.h"
#include "tcgen05.cuh"
#include "tmap.h"

namespace lv {

constexpr int kBgThreads = 192;              // TMA warp, MMA warp, four epilogue warps
constexpr int kBgRows = 128, kBgK = 64;
constexpr uint32_t kBgTile = kBgRows * kBgK * 2;
constexpr size_t kBgSmemBudget = 200 * 1024;
constexpr uint32_t kBgMaxStages = 8;
constexpr uint32_t kBgMaxTiles = 4096;       // arrival counters of split launches
constexpr size_t kBgScratchBytes = size_t(32) << 20;

struct GemmBf16Params {
    uint32_t rows, tokens, K, splits, stages;
    void* out;
    uint32_t out_ld, out_bf16;
    float factor;
    float* scratch;
    uint32_t* counters;
    int act;
    const lv_expert_tile* tiles;
    const uint32_t* pos;        // windows: the position word, null otherwise
    uint32_t window, batch;
    uint32_t* err;
};

struct GemmBf16Maps {
    CUtensorMap w, w2, x;
};

__host__ __device__ constexpr uint32_t bg_stage_bytes(int NT, bool pair) { return (pair ? 2 : 1) * kBgTile + NT * kBgK * 2; }
__host__ __device__ constexpr uint32_t bg_tmem_cols(int NT, bool pair) {
    const int need = NT * (pair ? 2 : 1);
    return need <= 32 ? 32 : need <= 64 ? 64 : need <= 128 ? 128 : need <= 256 ? 256 : 512;
}

template <int NT, bool PAIR, bool GROUPED>
__global__ void __launch_bounds__(kBgThreads, 1) gemm_bf16_kernel(const GemmBf16Params p, const __grid_constant__ GemmBf16Maps maps) {
    pdl_launch_dependents();
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023u) & ~uintptr_t(1023));
    constexpr uint32_t kStage = bg_stage_bytes(NT, PAIR), kCols = bg_tmem_cols(NT, PAIR), kXAt = (PAIR ? 2 : 1) * kBgTile;
    __shared__ uint64_t full[kBgMaxStages], empty[kBgMaxStages], acc_full;
    __shared__ uint32_t s_tmem, s_last;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;

    uint32_t row0 = blockIdx.x * kBgRows, tok0 = blockIdx.y * NT, n_tok;
    uint32_t w_row0 = row0, x_row0 = tok0;
    const bool wait_first = GROUPED || p.pos != nullptr;
    if (!GROUPED && p.pos != nullptr) {
        pdl_wait();
        const uint32_t P = *p.pos, first = p.window != 0 && P + 1 > p.window ? P + 1 - p.window : 0, n = min(p.tokens, P + p.batch - first);
        if (tok0 >= n) return;
        n_tok = min(uint32_t(NT), n - tok0);
        x_row0 = first + tok0;
    } else if constexpr (GROUPED) {
        pdl_wait();
        const lv_expert_tile t = p.tiles[blockIdx.y];
        if (t.rows == 0) return;
        tok0 = x_row0 = t.row0;
        n_tok = t.rows;
        w_row0 += t.expert * p.rows;
    } else {
        n_tok = min(uint32_t(NT), p.tokens - tok0);
    }
    const uint32_t chunks_all = (p.K + kBgK - 1) / kBgK;
    const uint32_t c0 = chunks_all * blockIdx.z / p.splits, n_chunks = chunks_all * (blockIdx.z + 1) / p.splits - c0;

    if (threadIdx.x < 2 * kBgMaxStages + 1) {
        const uint32_t i = threadIdx.x;
        mbar_init(i < kBgMaxStages ? &full[i] : i < 2 * kBgMaxStages ? &empty[i - kBgMaxStages] : &acc_full, 1);
        fence_mbar_init();
    }
    if (warp == 1) tc_alloc(&s_tmem, kCols);
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(&s_tmem);
    bool ok = true;

    if (warp == 0) {
        if (lane == 0) {
            auto load_w = [&](uint32_t c, uint32_t s) {
                mbar_expect_tx(&full[s], kStage);
                uint8_t* dst = smem + s * kStage;
                tma_load_2d_plain(dst, &maps.w, int((c0 + c) * kBgK), int(w_row0), &full[s]);
                if constexpr (PAIR) tma_load_2d_plain(dst + kBgTile, &maps.w2, int((c0 + c) * kBgK), int(w_row0), &full[s]);
            };
            auto load_x = [&](uint32_t c, uint32_t s) {
                tma_load_2d_plain(smem + s * kStage + kXAt, &maps.x, int((c0 + c) * kBgK), int(x_row0), &full[s]);
            };
            const uint32_t first = min(p.stages, n_chunks);
            for (uint32_t c = 0; c < first; ++c) load_w(c, c);
            if (!wait_first) pdl_wait();
            for (uint32_t c = 0; c < first; ++c) load_x(c, c);
            uint32_t s = 0, phase = 0;
            for (uint32_t c = first; c < n_chunks; ++c) {
                if (!mbar_wait(&empty[s], phase, p.err)) break;
                load_w(c, s);
                load_x(c, s);
                if (++s == p.stages) { s = 0; phase ^= 1u; }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            // f32 accumulator, bfloat16 operands, both K-major
            constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | (uint32_t(NT >> 3) << 17) | (uint32_t(kBgRows >> 4) << 24);
            const uint64_t base = tc_smem_desc(smem_u32(smem));
            uint32_t s = 0, phase = 0;
            for (uint32_t c = 0; c < n_chunks && ok; ++c) {
                ok = mbar_wait(&full[s], phase, p.err);
                if (!ok) break;
                tc_fence_after_sync();
                const uint64_t a = base + ((s * kStage) >> 4), b = a + (kXAt >> 4);
#pragma unroll
                for (int k = 0; k < kBgK / 16; ++k) {
                    const uint32_t acc = (c != 0 || k != 0) ? 1u : 0u;
                    tc_mma_f16(tmem, a + 2u * k, b + 2u * k, idesc, acc);
                    if constexpr (PAIR) tc_mma_f16(tmem + NT, a + (kBgTile >> 4) + 2u * k, b + 2u * k, idesc, acc);
                }
                tc_commit(&empty[s]);
                if (++s == p.stages) { s = 0; phase ^= 1u; }
            }
            if (ok) tc_commit(&acc_full);
        }
    } else {
        // ---- epilogue: warp w reads lanes 32 (w mod 4) .. + 31 of the accumulator --------------------
        const uint32_t quarter = uint32_t(warp) & 3u, tr = quarter * 32u + uint32_t(lane);
        const uint32_t row = row0 + tr, taddr = tmem + (quarter * 32u << 16);
        ok = mbar_wait_warp(&acc_full, 0, p.err);
        tc_fence_after_sync();
        constexpr int kAcc = PAIR ? 2 : 1;
        const uint32_t tile = blockIdx.y * gridDim.x + blockIdx.x;
        float* partial = p.splits > 1 ? p.scratch + size_t(tile) * p.splits * (kAcc * NT * kBgRows) : nullptr;
        auto finish = [&](const float (&v)[16], const float (&g)[16], uint32_t z0) {
            if (row >= p.rows) return;
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                if (z0 + i >= n_tok) break;
                const float r = PAIR ? silu_f32(v[i]) * g[i] : product_act(v[i] * p.factor, p.act);
                const size_t at = size_t(tok0 + z0 + i) * p.out_ld + row;
                if (p.out_bf16) static_cast<__nv_bfloat16*>(p.out)[at] = __float2bfloat16_rn(r);
                else static_cast<float*>(p.out)[at] = r;
            }
        };
        if (ok) {
            for (uint32_t z0 = 0; z0 < NT; z0 += 16) {
                uint32_t u[kAcc][16];
#pragma unroll
                for (int a = 0; a < kAcc; ++a) tc_load16(u[a], taddr + a * NT + z0);
                tc_wait_load();
                float v[16], g[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) { v[i] = __uint_as_float(u[0][i]); g[i] = __uint_as_float(u[kAcc - 1][i]); }
                if (p.splits == 1) {
                    finish(v, g, z0);
                } else {
                    float* dst = partial + size_t(blockIdx.z) * (kAcc * NT * kBgRows);
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        dst[(z0 + i) * kBgRows + tr] = v[i];
                        if constexpr (PAIR) dst[(NT + z0 + i) * kBgRows + tr] = g[i];
                    }
                }
            }
        }
        if (p.splits > 1) {
            __threadfence();
            asm volatile("bar.sync 1, 128;" ::: "memory");
            if (threadIdx.x == 64) {
                const uint32_t last = atomicAdd(&p.counters[tile], 1u) + 1 == p.splits ? 1u : 0u;
                if (last) p.counters[tile] = 0;
                s_last = last;
            }
            asm volatile("bar.sync 1, 128;" ::: "memory");
            if (*reinterpret_cast<volatile uint32_t*>(&s_last) != 0 && ok) {
                __threadfence();
                for (uint32_t z0 = 0; z0 < NT && z0 < n_tok; z0 += 16) {
                    float v[16] = {}, g[16] = {};
#pragma unroll 2
                    for (uint32_t s = 0; s < p.splits; ++s) {
                        const float* src = partial + size_t(s) * (kAcc * NT * kBgRows);
#pragma unroll
                        for (int i = 0; i < 16; ++i) {
                            v[i] += __ldcg(src + (z0 + i) * kBgRows + tr);
                            if constexpr (PAIR) g[i] += __ldcg(src + (NT + z0 + i) * kBgRows + tr);
                        }
                    }
                    finish(v, g, z0);
                }
            }
        }
        tc_fence_before_sync();
    }
    __syncthreads();
    if (warp == 1) {
        tc_fence_after_sync();
        tc_free(tmem, kCols);
    }
}

// rows of an expert tile: by the rows an expert gets when the ids spread evenly
__host__ __device__ inline uint32_t bg_expert_tile(uint32_t batch, uint32_t top, uint32_t experts) {
    const uint32_t mean = (batch * top + experts - 1) / experts;
    return mean <= 12 ? 16 : mean <= 24 ? 32 : mean <= 56 ? 64 : 128;
}

// Sorts the (token, choice) pairs of a step by expert, one CTA per layer.
__global__ void __launch_bounds__(1024) expert_route_kernel(const lv_route_job* __restrict__ jobs, const uint32_t* __restrict__ token_log,
                                                            const uint32_t* __restrict__ pos, uint32_t vocab, uint32_t batch, uint32_t* err) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ uint32_t s_cursor[];               // [experts]: count, then next free row
    const lv_route_job job = jobs[blockIdx.x];
    const uint32_t pairs = batch * job.top, first = *pos, tile_rows = bg_expert_tile(batch, job.top, job.experts);
    for (uint32_t e = threadIdx.x; e < job.experts; e += blockDim.x) s_cursor[e] = 0;
    __syncthreads();
    auto expert = [&](uint32_t i) {
        const uint32_t id = token_log[first + i / job.top];
        const uint32_t e = id < vocab ? job.table[size_t(id) * job.top + i % job.top] : job.experts;
        if (e < job.experts) return e;
        atomicOr(err, ERR_BAD_INDEX);
        return 0u;
    };
    for (uint32_t i = threadIdx.x; i < pairs; i += blockDim.x) atomicAdd(&s_cursor[expert(i)], 1u);
    __syncthreads();
    if (threadIdx.x < 32) {
        // a lane sums the rows and tiles of consecutive experts, the warp forms the prefix, the lane hands them out
        const uint32_t per = (job.experts + 31) / 32, e0 = min(job.experts, threadIdx.x * per), e1 = min(job.experts, e0 + per);
        uint32_t rows = 0, tiles = 0;
        for (uint32_t e = e0; e < e1; ++e) {
            rows += s_cursor[e];
            tiles += (s_cursor[e] + tile_rows - 1) / tile_rows;
        }
        uint32_t row_at = rows, tile_at = tiles;
        for (int o = 1; o < 32; o <<= 1) {
            const uint32_t r = __shfl_up_sync(0xffffffffu, row_at, o), t = __shfl_up_sync(0xffffffffu, tile_at, o);
            if (threadIdx.x >= uint32_t(o)) { row_at += r; tile_at += t; }
        }
        const uint32_t all_tiles = __shfl_sync(0xffffffffu, tile_at, 31);
        row_at -= rows;
        tile_at -= tiles;
        for (uint32_t e = e0; e < e1; ++e) {
            const uint32_t n = s_cursor[e];
            for (uint32_t r = 0; r < n; r += tile_rows, ++tile_at)
                if (tile_at < job.max_tiles) job.tiles[tile_at] = {e, row_at + r, min(tile_rows, n - r)};
            s_cursor[e] = row_at;
            row_at += n;
        }
        for (uint32_t t = all_tiles + threadIdx.x; t < job.max_tiles; t += 32) job.tiles[t] = {0u, 0u, 0u};
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < pairs; i += blockDim.x) job.index[i] = atomicAdd(&s_cursor[expert(i)], 1u);
}

int gemm_bf16_configure(lv_ctx* ctx) {
    LV_CUDA(cudaMalloc(&ctx->bg_scratch, kBgScratchBytes));
    LV_CUDA(cudaMalloc(&ctx->bg_counters, kBgMaxTiles * sizeof(uint32_t)));
    LV_CUDA(cudaMemset(ctx->bg_counters, 0, kBgMaxTiles * sizeof(uint32_t)));
    return LV_OK;
}

void gemm_bf16_release(lv_ctx* ctx) {
    cudaFree(ctx->bg_scratch);
    cudaFree(ctx->bg_counters);
    ctx->bg_scratch = ctx->bg_counters = nullptr;
}

template <int NT, bool PAIR, bool GROUPED>
static int gemm_bf16_launch(lv_ctx* ctx, GemmBf16Params p, const GemmBf16Maps& maps, uint32_t token_tiles) {
    constexpr uint32_t kStage = bg_stage_bytes(NT, PAIR);
    p.stages = std::min<uint32_t>(kBgMaxStages, kBgSmemBudget / kStage);
    const uint32_t row_tiles = (p.rows + kBgRows - 1) / kBgRows, chunks = (p.K + kBgK - 1) / kBgK, ctas = row_tiles * token_tiles;
    // K splits: as many as fill the SMs once, each with at least four chunks
    p.splits = 1;
    while (ctas * (p.splits + 1) <= uint32_t(ctx->sm_count) && chunks / (p.splits + 1) >= 4 && p.splits < 16) ++p.splits;
    if (ctas > kBgMaxTiles || size_t(ctas) * p.splits * (PAIR ? 2 : 1) * NT * kBgRows * 4 > kBgScratchBytes) p.splits = 1;
    p.scratch = static_cast<float*>(ctx->bg_scratch);
    p.counters = static_cast<uint32_t*>(ctx->bg_counters);
    p.err = ctx->d_err;
    const size_t smem = size_t(p.stages) * kStage + 1024;
    auto* kernel = gemm_bf16_kernel<NT, PAIR, GROUPED>;
    LV_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    LV_REQUIRE(token_tiles <= 65535, "gemm_bf16: too many token tiles");
    LV_CUDA(launch_pdl(ctx, kernel, dim3(row_tiles, token_tiles, p.splits), dim3(kBgThreads), smem, p, maps));
    return LV_OK;
}

template <bool PAIR, bool GROUPED>
static int gemm_bf16_pick(lv_ctx* ctx, const GemmBf16Params& p, const GemmBf16Maps& maps, uint32_t nt, uint32_t token_tiles) {
    switch (nt) {
        case 16: return gemm_bf16_launch<16, PAIR, GROUPED>(ctx, p, maps, token_tiles);
        case 32: return gemm_bf16_launch<32, PAIR, GROUPED>(ctx, p, maps, token_tiles);
        case 64: return gemm_bf16_launch<64, PAIR, GROUPED>(ctx, p, maps, token_tiles);
        default: return gemm_bf16_launch<128, PAIR, GROUPED>(ctx, p, maps, token_tiles);
    }
}

static bool bg_aligned(const void* p) { return p != nullptr && (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

}  // namespace lv

using namespace lv;

extern "C" int lv_gemm_bf16(lv_ctx* ctx, void* out, int out_type, uint32_t out_ld, const void* w, uint32_t rows, uint32_t ld, uint32_t cols,
                            const void* x, uint32_t x_ld, uint32_t batch, float factor, int act) {
    LV_ENTER(ctx);
    LV_REQUIRE(out && bg_aligned(w) && bg_aligned(x) && rows && cols && batch && out_ld >= rows, "bad gemm_bf16 arguments");
    LV_REQUIRE(ld % 8 == 0 && ld >= cols && x_ld % 8 == 0 && x_ld >= cols && (out_type == LV_TYPE_F32 || out_type == LV_TYPE_BF16), "gemm_bf16: bad strides");
    LV_REQUIRE(act == LV_ACT_NONE || act == LV_ACT_RELU2, "gemm_bf16: unknown activation");
    GemmBf16Params p{};
    p.rows = rows; p.tokens = batch; p.K = cols; p.out = out; p.out_ld = out_ld; p.out_bf16 = out_type == LV_TYPE_BF16; p.factor = factor; p.act = act;
    uint32_t nt = batch <= 16 ? 16 : batch <= 32 ? 32 : batch <= 64 ? 64 : 128;
    // narrower token tiles before K splits: partial sums cost more than reading a weight tile twice
    while (nt > 32 && (rows + kBgRows - 1) / kBgRows * ((batch + nt - 1) / nt) * 2 <= uint32_t(ctx->sm_count) && batch > nt / 2) nt /= 2;
    GemmBf16Maps maps{};
    if (int rc = make_bf16_map(&maps.w, w, rows, cols, ld, kBgRows)) return rc;
    if (int rc = make_bf16_map(&maps.x, x, batch, cols, x_ld, nt)) return rc;
    maps.w2 = maps.w;
    return gemm_bf16_pick<false, false>(ctx, p, maps, nt, (batch + nt - 1) / nt);
}

extern "C" int lv_gemm_bf16_window(lv_ctx* ctx, void* out, int out_type, uint32_t out_ld, const void* w, uint32_t rows, uint32_t ld, uint32_t cols,
                                   const void* x, uint32_t x_ld, uint32_t x_rows, const uint32_t* pos, uint32_t batch, uint32_t window, uint32_t max_rows) {
    LV_ENTER(ctx);
    LV_REQUIRE(out && bg_aligned(w) && bg_aligned(x) && rows && cols && batch && pos && max_rows && x_rows && out_ld >= rows, "bad gemm_bf16 arguments");
    LV_REQUIRE(ld % 8 == 0 && ld >= cols && x_ld % 8 == 0 && x_ld >= cols && (out_type == LV_TYPE_F32 || out_type == LV_TYPE_BF16), "gemm_bf16: bad strides");
    GemmBf16Params p{};
    p.rows = rows; p.tokens = max_rows; p.K = cols; p.out = out; p.out_ld = out_ld; p.out_bf16 = out_type == LV_TYPE_BF16; p.factor = 1.0f;
    p.pos = pos; p.window = window; p.batch = batch;
    uint32_t nt = max_rows <= 16 ? 16 : max_rows <= 32 ? 32 : max_rows <= 64 ? 64 : 128;
    while (nt > 32 && (rows + kBgRows - 1) / kBgRows * ((max_rows + nt - 1) / nt) * 2 <= uint32_t(ctx->sm_count)) nt /= 2;
    GemmBf16Maps maps{};
    if (int rc = make_bf16_map(&maps.w, w, rows, cols, ld, kBgRows)) return rc;
    if (int rc = make_bf16_map(&maps.x, x, x_rows, cols, x_ld, nt)) return rc;
    maps.w2 = maps.w;
    return gemm_bf16_pick<false, false>(ctx, p, maps, nt, (max_rows + nt - 1) / nt);
}

extern "C" uint32_t lv_expert_tile_rows(uint32_t batch, uint32_t top, uint32_t experts) {
    return experts ? bg_expert_tile(batch, top, experts) : 0;
}

extern "C" uint32_t lv_expert_max_tiles(uint32_t batch, uint32_t top, uint32_t experts) {
    if (!experts) return 0;
    const uint32_t nt = bg_expert_tile(batch, top, experts), pairs = batch * top;
    return pairs / nt + std::min(experts, pairs);
}

extern "C" int lv_expert_route(lv_ctx* ctx, const lv_route_job* jobs, uint32_t n_jobs, uint32_t max_experts, const uint32_t* token_log,
                               const uint32_t* pos, uint32_t vocab, uint32_t batch) {
    LV_ENTER(ctx);
    LV_REQUIRE(jobs && n_jobs && token_log && pos && vocab && batch, "bad expert_route arguments");
    LV_REQUIRE(max_experts && max_experts <= 8192, "expert_route: more than 8192 experts");
    LV_CUDA(launch_pdl(ctx, expert_route_kernel, dim3(n_jobs), dim3(1024), max_experts * 4, jobs, token_log, pos, vocab, batch, ctx->d_err));
    return LV_OK;
}

static int expert_gemm(lv_ctx* ctx, bool pair, void* out, int out_type, uint32_t out_ld, const lv_expert_args* a, const lv_expert_tile* tiles, const void* x,
                       uint32_t x_ld, uint32_t batch) {
    LV_ENTER(ctx);
    LV_REQUIRE(out && a && tiles && bg_aligned(x) && batch && bg_aligned(a->w0) && (!pair || bg_aligned(a->w1)), "bad expert product arguments");
    LV_REQUIRE(a->ld % 8 == 0 && a->ld >= a->cols && x_ld % 8 == 0 && x_ld >= a->cols && a->rows && a->cols && a->experts && a->top && out_ld >= a->rows &&
               (out_type == LV_TYPE_F32 || out_type == LV_TYPE_BF16), "expert product: bad strides");
    GemmBf16Params p{};
    p.rows = a->rows; p.tokens = batch * a->top; p.K = a->cols; p.out = out; p.out_ld = out_ld; p.out_bf16 = out_type == LV_TYPE_BF16; p.factor = 1.0f;
    p.tiles = tiles;
    const uint32_t nt = lv_expert_tile_rows(batch, a->top, a->experts), n_tiles = lv_expert_max_tiles(batch, a->top, a->experts);
    GemmBf16Maps maps{};
    if (int rc = make_bf16_map(&maps.w, a->w0, uint64_t(a->experts) * a->rows, a->cols, a->ld, kBgRows)) return rc;
    maps.w2 = maps.w;
    if (pair)
        if (int rc = make_bf16_map(&maps.w2, a->w1, uint64_t(a->experts) * a->rows, a->cols, a->ld, kBgRows)) return rc;
    if (int rc = make_bf16_map(&maps.x, x, uint64_t(batch) * a->top, a->cols, x_ld, nt)) return rc;
    return pair ? gemm_bf16_pick<true, true>(ctx, p, maps, nt, n_tiles) : gemm_bf16_pick<false, true>(ctx, p, maps, nt, n_tiles);
}

extern "C" int lv_gemm_bf16_expert_gate_up(lv_ctx* ctx, void* out, uint32_t out_ld, const lv_expert_args* a, const lv_expert_tile* tiles, const void* x,
                                           uint32_t x_ld, uint32_t batch) {
    return expert_gemm(ctx, true, out, LV_TYPE_BF16, out_ld, a, tiles, x, x_ld, batch);
}

extern "C" int lv_gemm_bf16_expert_down(lv_ctx* ctx, float* out, uint32_t out_ld, const lv_expert_args* a, const lv_expert_tile* tiles, const void* x,
                                        uint32_t x_ld, uint32_t batch) {
    return expert_gemm(ctx, false, out, LV_TYPE_F32, out_ld, a, tiles, x, x_ld, batch);
}
