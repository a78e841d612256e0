// Matrix-vector products with bfloat16 weights: the decode-side products of models whose weights are not quantised.
//
//   lv_gemv_bf16                 one matrix (stacked projections that share an input); optional factor and activation
//   lv_gemv_bf16_mingru          three products per channel and the gated recurrence on them in the epilogue
//   lv_gemv_bf16_expert_gate_up  silu(gate x) * (up x) of the experts that a table gives a token
//   lv_gemv_bf16_expert_down     the mean of those experts' down products
//
// Weights are bfloat16 [rows][ld] (ld a multiple of 8, the tail of a row zero), inputs and results f32 and the arithmetic
// f32 throughout: a bfloat16 weight is exact in f32, so the same kernels serve a 32-bit evaluation.  The bound is HBM: two
// bytes per multiply-add, each weight read once.  A warp computes two or three rows, lanes taking 16 bytes of every row per
// step with four steps in flight (up to 6 KB per warp); the first weights are requested before the previous kernel has
// finished.  Lanes are combined by shuffles in a fixed order, so a result does not depend on the launch.  Matrices with few rows
// are cut along K over the warps of a CTA, so that enough loads are in flight.
//
// gridDim.y = tokens: every token has its own pass over the weights.  Prompts use gemm_bf16.cu instead.
#include <cuda_bf16.h>

#include "common.cuh"
#include "ctx.h"

namespace lv {

constexpr int kGbWarps = 8, kGbThreads = kGbWarps * 32;
constexpr int kGbUnroll = 4;

__device__ __forceinline__ uint4 gb_load_w(const __nv_bfloat16* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

// eight consecutive inputs; those at or beyond K are zero
__device__ __forceinline__ void gb_load_x(float (&x)[8], const float* src, uint32_t k, uint32_t K) {
    if (k + 8 <= K) {
        const float4 a = *reinterpret_cast<const float4*>(src + k), b = *reinterpret_cast<const float4*>(src + k + 4);
        x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
    } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] = k + i < K ? src[k + i] : 0.f;
    }
}

__device__ __forceinline__ void gb_fma(float& acc, uint4 w, const float (&x)[8]) {
    const uint32_t q[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        acc = fmaf(__uint_as_float(q[i] << 16), x[2 * i], acc);
        acc = fmaf(__uint_as_float(q[i] & 0xffff0000u), x[2 * i + 1], acc);
    }
}

// Partial dot products of NR rows with x over this lane's share of K.  WAIT: the rows are known before the previous kernel
// has finished and their first elements are requested before waiting for it.
template <int NR, bool WAIT>
__device__ __forceinline__ void gb_dot(float (&acc)[NR], const __nv_bfloat16* const (&row)[NR], const float* x, uint32_t K) {
    const uint32_t lane8 = (threadIdx.x & 31u) * 8u;
    uint4 w[kGbUnroll][NR];
    auto fetch = [&](uint32_t k0) {
#pragma unroll
        for (int u = 0; u < kGbUnroll; ++u) {
            const uint32_t k = k0 + u * 256u + lane8;
#pragma unroll
            for (int r = 0; r < NR; ++r) w[u][r] = k < K ? gb_load_w(row[r] + k) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    fetch(0);
    if constexpr (WAIT) pdl_wait();
    for (uint32_t k0 = 0; k0 < K; k0 += 256u * kGbUnroll) {
#pragma unroll
        for (int u = 0; u < kGbUnroll; ++u) {
            const uint32_t k = k0 + u * 256u + lane8;
            if (k < K) {
                float xv[8];
                gb_load_x(xv, x, k, K);
#pragma unroll
                for (int r = 0; r < NR; ++r) gb_fma(acc[r], w[u][r], xv);
            }
        }
        if (k0 + 256u * kGbUnroll < K) fetch(k0 + 256u * kGbUnroll);
    }
}

struct GemvBf16Params {
    const __nv_bfloat16* w[3];
    uint32_t rows;
    uint32_t ld, K;
    const float* x;
    uint32_t x_ld;
    float* out;
    uint32_t out_ld;
    float factor;
    int act;
};

// SPLIT: warps that share two rows
template <int SPLIT>
__global__ void __launch_bounds__(kGbThreads) gemv_bf16_kernel(const GemvBf16Params p) {
    pdl_launch_dependents();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
    const uint32_t u = 2u * (blockIdx.x * (kGbWarps / SPLIT) + warp / SPLIT);
    float acc[2] = {0.f, 0.f};
    if constexpr (SPLIT == 1) {
        if (u >= p.rows) return;
        const __nv_bfloat16* row[2] = {p.w[0] + size_t(u) * p.ld, p.w[0] + size_t(min(u + 1, p.rows - 1)) * p.ld};
        gb_dot<2, true>(acc, row, p.x + size_t(blockIdx.y) * p.x_ld, p.K);
    } else {
        const uint32_t per = (p.K + SPLIT * 256 - 1) / (SPLIT * 256) * 256, first = warp % SPLIT * per, count = u < p.rows && first < p.K ? min(per, p.K - first) : 0;
        const __nv_bfloat16* row[2] = {p.w[0] + size_t(min(u, p.rows - 1)) * p.ld + first, p.w[0] + size_t(min(u + 1, p.rows - 1)) * p.ld + first};
        gb_dot<2, true>(acc, row, p.x + size_t(blockIdx.y) * p.x_ld + first, count);
    }
    float a0 = warp_sum(acc[0]), a1 = warp_sum(acc[1]);
    if constexpr (SPLIT > 1) {
        __shared__ float s_part[kGbWarps][2];
        if (lane == 0) { s_part[warp][0] = a0; s_part[warp][1] = a1; }
        __syncthreads();
        if (warp % SPLIT != 0) return;
        a0 = a1 = 0.f;
#pragma unroll
        for (int k = 0; k < SPLIT; ++k) { a0 += s_part[warp + k][0]; a1 += s_part[warp + k][1]; }
    }
    if (lane < 2 && u + lane < p.rows) p.out[size_t(blockIdx.y) * p.out_ld + u + lane] = product_act((lane ? a1 : a0) * p.factor, p.act);
}

__global__ void __launch_bounds__(kGbThreads) gemv_bf16_mingru_kernel(const GemvBf16Params p, const float* __restrict__ bz, const float* __restrict__ bx,
                                                                      float* __restrict__ state, const uint32_t* __restrict__ pos) {
    pdl_launch_dependents();
    const uint32_t c = blockIdx.x * kGbWarps + (threadIdx.x >> 5);
    if (c >= p.rows) return;
    const __nv_bfloat16* row[3] = {p.w[0] + size_t(c) * p.ld, p.w[1] + size_t(c) * p.ld, p.w[2] + size_t(c) * p.ld};
    float acc[3] = {0.f, 0.f, 0.f};
    gb_dot<3, true>(acc, row, p.x, p.K);
    const float az = warp_sum(acc[0]), ax = warp_sum(acc[1]), ag = warp_sum(acc[2]);
    if ((threadIdx.x & 31u) == 0) p.out[c] = mingru_step(az + bz[c], ax + bx[c], ag, *pos == 0 ? 0.f : state[c], &state[c]);
}

struct ExpertGemvParams {
    const __nv_bfloat16* gate;      // [experts * ff][ld]; the down matrix [experts * width][ld] in lv_gemv_bf16_expert_down
    const __nv_bfloat16* up;
    uint32_t ld, K, rows, experts, top, vocab;
    const uint32_t* table;          // [vocab][top]
    const uint32_t* token_log;
    const uint32_t* pos;
    const float* x;
    uint32_t x_ld;
    float* out;
    uint32_t out_ld;
    uint32_t* err;
};

__device__ __forceinline__ uint32_t gb_expert(const ExpertGemvParams& p, uint32_t t, uint32_t slot) {
    const uint32_t id = p.token_log[*p.pos + t];
    const uint32_t e = id < p.vocab ? p.table[size_t(id) * p.top + slot] : p.experts;
    if (e < p.experts) return e;
    if (threadIdx.x == 0) atomicOr(p.err, ERR_BAD_INDEX);
    return 0;
}

__global__ void __launch_bounds__(kGbThreads) gemv_bf16_expert_gate_up_kernel(const ExpertGemvParams p) {
    pdl_launch_dependents();
    const uint32_t t = blockIdx.y, slot = blockIdx.z;
    const uint32_t i = blockIdx.x * kGbWarps + (threadIdx.x >> 5);
    pdl_wait();
    const uint32_t e = gb_expert(p, t, slot);
    if (i >= p.rows) return;
    const size_t at = (size_t(e) * p.rows + i) * p.ld;
    const __nv_bfloat16* row[2] = {p.gate + at, p.up + at};
    float acc[2] = {0.f, 0.f};
    gb_dot<2, false>(acc, row, p.x + size_t(t) * p.x_ld, p.K);
    const float g = warp_sum(acc[0]), u = warp_sum(acc[1]);
    if ((threadIdx.x & 31u) == 0) p.out[(size_t(t) * p.top + slot) * p.out_ld + i] = silu_f32(g) * u;
}

__global__ void __launch_bounds__(kGbThreads) gemv_bf16_expert_down_kernel(const ExpertGemvParams p) {
    pdl_launch_dependents();
    const uint32_t t = blockIdx.y;
    const uint32_t r = 2u * (blockIdx.x * kGbWarps + (threadIdx.x >> 5));
    pdl_wait();
    if (r >= p.rows) return;
    float acc[2] = {0.f, 0.f};
    for (uint32_t s = 0; s < p.top; ++s) {
        const size_t first = size_t(gb_expert(p, t, s)) * p.rows;
        const __nv_bfloat16* row[2] = {p.gate + (first + r) * p.ld, p.gate + (first + min(r + 1, p.rows - 1)) * p.ld};
        gb_dot<2, false>(acc, row, p.x + (size_t(t) * p.top + s) * p.x_ld, p.K);
    }
    const float a0 = warp_sum(acc[0]), a1 = warp_sum(acc[1]);
    const uint32_t lane = threadIdx.x & 31u;
    if (lane < 2 && r + lane < p.rows) p.out[size_t(t) * p.out_ld + r + lane] = (lane ? a1 : a0) / float(p.top);
}

static bool gb_aligned(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

}  // namespace lv

using namespace lv;

extern "C" int lv_gemv_bf16(lv_ctx* ctx, float* out, uint32_t out_ld, const void* w, uint32_t rows, uint32_t ld, uint32_t cols, const float* x,
                            uint32_t x_ld, uint32_t batch, float factor, int act) {
    LV_ENTER(ctx);
    LV_REQUIRE(out && w && rows && x && cols && batch && batch <= 65535 && out_ld >= rows, "bad gemv_bf16 arguments");
    LV_REQUIRE(ld % 8 == 0 && ld >= cols && x_ld >= cols && (batch == 1 || x_ld % 4 == 0) && gb_aligned(x) && gb_aligned(w), "gemv_bf16: bad strides");
    LV_REQUIRE(act == LV_ACT_NONE || act == LV_ACT_RELU2, "gemv_bf16: unknown activation");
    GemvBf16Params p{};
    p.w[0] = static_cast<const __nv_bfloat16*>(w);
    p.rows = rows;
    p.ld = ld; p.K = cols; p.x = x; p.x_ld = x_ld; p.out = out; p.out_ld = out_ld; p.factor = factor; p.act = act;
    // three or more CTAs per SM, at least 512 columns per warp
    uint32_t split = 1;
    while (split < 8 && uint64_t(rows) * batch * split < uint64_t(48) * uint32_t(ctx->sm_count) && cols >= 512 * 2 * split) split *= 2;
    const uint32_t per_cta = 2 * kGbWarps / split;
    auto* kernel = split == 1 ? gemv_bf16_kernel<1> : split == 2 ? gemv_bf16_kernel<2> : split == 4 ? gemv_bf16_kernel<4> : gemv_bf16_kernel<8>;
    LV_CUDA(launch_pdl(ctx, kernel, dim3((rows + per_cta - 1) / per_cta, batch), dim3(kGbThreads), 0, p));
    return LV_OK;
}

extern "C" int lv_gemv_bf16_mingru(lv_ctx* ctx, float* out, const void* wz, const void* wx, const void* wg, uint32_t ld, uint32_t channels, uint32_t cols,
                                   const float* bz, const float* bx, const float* x, float* state, const uint32_t* pos) {
    LV_ENTER(ctx);
    LV_REQUIRE(out && wz && wx && wg && bz && bx && x && state && pos && channels && cols, "bad mingru arguments");
    LV_REQUIRE(ld % 8 == 0 && ld >= cols && gb_aligned(x) && gb_aligned(wz) && gb_aligned(wx) && gb_aligned(wg), "mingru: bad strides");
    GemvBf16Params p{};
    p.w[0] = static_cast<const __nv_bfloat16*>(wz);
    p.w[1] = static_cast<const __nv_bfloat16*>(wx);
    p.w[2] = static_cast<const __nv_bfloat16*>(wg);
    p.rows = channels;
    p.ld = ld; p.K = cols; p.x = x; p.out = out;
    LV_CUDA(launch_pdl(ctx, gemv_bf16_mingru_kernel, dim3((channels + kGbWarps - 1) / kGbWarps), dim3(kGbThreads), 0, p, bz, bx, state, pos));
    return LV_OK;
}

static int expert_params(const lv_expert_args* a, ExpertGemvParams* p) {
    LV_REQUIRE(a && a->table && a->token_log && a->pos && a->experts && a->top && a->vocab && a->rows && a->cols, "bad expert arguments");
    LV_REQUIRE(a->ld % 8 == 0 && a->ld >= a->cols && a->w0 && gb_aligned(a->w0) && (!a->w1 || gb_aligned(a->w1)), "experts: bad matrices");
    p->gate = static_cast<const __nv_bfloat16*>(a->w0);
    p->up = static_cast<const __nv_bfloat16*>(a->w1);
    p->ld = a->ld; p->K = a->cols; p->rows = a->rows; p->experts = a->experts; p->top = a->top; p->vocab = a->vocab;
    p->table = a->table; p->token_log = a->token_log; p->pos = a->pos;
    return LV_OK;
}

extern "C" int lv_gemv_bf16_expert_gate_up(lv_ctx* ctx, float* out, uint32_t out_ld, const lv_expert_args* a, const float* x, uint32_t x_ld, uint32_t batch) {
    LV_ENTER(ctx);
    ExpertGemvParams p{};
    if (const int rc = expert_params(a, &p)) return rc;
    LV_REQUIRE(out && x && gb_aligned(x) && batch && batch <= 65535 && a->top <= 65535 && p.up && out_ld >= p.rows && x_ld >= p.K && (batch == 1 || x_ld % 4 == 0), "bad expert_gate_up arguments");
    p.x = x; p.x_ld = x_ld; p.out = out; p.out_ld = out_ld; p.err = ctx->d_err;
    LV_CUDA(launch_pdl(ctx, gemv_bf16_expert_gate_up_kernel, dim3((p.rows + kGbWarps - 1) / kGbWarps, batch, p.top), dim3(kGbThreads), 0, p));
    return LV_OK;
}

extern "C" int lv_gemv_bf16_expert_down(lv_ctx* ctx, float* out, uint32_t out_ld, const lv_expert_args* a, const float* x, uint32_t x_ld, uint32_t batch) {
    LV_ENTER(ctx);
    ExpertGemvParams p{};
    if (const int rc = expert_params(a, &p)) return rc;
    LV_REQUIRE(out && x && gb_aligned(x) && batch && batch <= 65535 && out_ld >= p.rows && x_ld >= p.K && x_ld % 4 == 0, "bad expert_down arguments");
    p.x = x; p.x_ld = x_ld; p.out = out; p.out_ld = out_ld; p.err = ctx->d_err;
    LV_CUDA(launch_pdl(ctx, gemv_bf16_expert_down_kernel, dim3((p.rows + 2 * kGbWarps - 1) / (2 * kGbWarps), batch), dim3(kGbThreads), 0, p));
    return LV_OK;
}
