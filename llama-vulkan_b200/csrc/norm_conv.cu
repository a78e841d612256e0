// The boundary between two sublayers of a pre- and post-normalised decoder: residual add of the finished sublayer (its
// output normalised), an optional vector added to the stream, the norm of the next sublayer and a short causal convolution
// over time on its result.
//
//   y_t   = mean of y_rows rows of the finished sublayer          (experts leave one row per choice)
//   x'_t  = x_t + mult * y_t / rms(y_t) * (1 + post_w)            rms(v) = sqrt(mean(v^2) + eps)
//   x''_t = x'_t + step
//   h_t   = x''_t / rms(x''_t) * (1 + pre_w)
//   out_t = h_t + sum_j conv_w[j] * h_(t - taps + 1 + j)          h before position 0 is zero
//
// plain_w: the weights themselves instead of 1 + w.  pre_w null: no second norm, h_t = x''_t (designs that norm the output of a
// sublayer only).  x may come from the embedding table instead of the stream, with a factor and a second table of pairs of ids.  The last taps - 1 values of h are the state that the next
// step reads; positions before the start of the sequence are masked by the position word, so a state needs no clearing.
//
// A CTA per token holds the token's row in registers (all loads are issued before the first sum).  One token is done in
// that launch.  Several tokens leave x'' and 1 / rms in memory for a second launch that forms h again and convolves: its
// threads own channels and slide over a few tokens, so it has no sum to wait for.
#include <cuda_bf16.h>

#include "common.cuh"
#include "ctx.h"

namespace lv {

constexpr uint32_t kNormConvMaxTaps = 16;

struct NormConvParams {
    lv_norm_conv_args a;
    uint32_t tokens_per_block;
    uint32_t* err;
};

template <int VEC> struct NcVec;
template <> struct NcVec<1> {
    float v[1];
    __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { v[0] = __bfloat162float(*p); }
    __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
    __device__ __forceinline__ void store(__nv_bfloat16* p) const { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct NcVec<4> {
    float v[4];
    __device__ __forceinline__ void load(const float* p) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    }
    __device__ __forceinline__ void load(const __nv_bfloat16* p) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        v[0] = __uint_as_float(u.x << 16); v[1] = __uint_as_float(u.x & 0xffff0000u);
        v[2] = __uint_as_float(u.y << 16); v[3] = __uint_as_float(u.y & 0xffff0000u);
    }
    __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
    __device__ __forceinline__ void store(__nv_bfloat16* p) const {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    }
};

template <int VEC, typename OutT>
__device__ __forceinline__ void nc_store(const lv_norm_conv_args& a, uint32_t t, uint32_t i, const NcVec<VEC>& v) {
    OutT* out = static_cast<OutT*>(a.out);
    if (a.out_index == nullptr) {
        v.store(out + size_t(t - a.first) * a.out_ld + i);
    } else {
        for (uint32_t s = 0; s < a.out_copies; ++s) v.store(out + size_t(a.out_index[t * a.out_copies + s]) * a.out_ld + i);
    }
}

// CTA b: token a.first + b.  A thread holds NV vectors of VEC channels.
template <int VEC, int NV, typename OutT>
__global__ void __launch_bounds__(1024) norm_rows_kernel(const NormConvParams p) {
    pdl_launch_dependents();
    const lv_norm_conv_args& a = p.a;
    __shared__ float scratch[64];
    const uint32_t W = a.width, t = a.first + blockIdx.x, keep = a.taps ? a.taps - 1 : 0;
    const bool finish = a.taps == 0 || a.batch == 1;      // else the second launch forms h
    NcVec<VEC> pre[NV], post[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {                        // weights do not depend on the previous kernel
        const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
        if (i < W) {
            if (finish && a.pre_w != nullptr) pre[k].load(a.pre_w + i);
            if (a.y != nullptr) post[k].load(a.post_w + i);
        }
    }
    const float w0 = a.plain_w ? 0.f : 1.f;
    pdl_wait();
    const uint32_t pos = *a.pos;
    NcVec<VEC> x[NV], y[NV];
    if (a.x == nullptr) {
        uint32_t id = a.token_log[pos + t];
        if (id >= a.vocab) {
            if (threadIdx.x == 0) atomicOr(p.err, ERR_BAD_INDEX);
            id = 0;
        }
        const __nv_bfloat16* row = static_cast<const __nv_bfloat16*>(a.embed) + size_t(id) * a.embed_ld;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
            if (i < W) x[k].load(row + i);
        }
        if (a.embed_scale != 0.f) {
#pragma unroll
            for (int k = 0; k < NV; ++k)
#pragma unroll
                for (int e = 0; e < VEC; ++e) x[k].v[e] *= a.embed_scale;
        }
        if (a.pair_embed != nullptr) {
            uint32_t bucket = a.pair_buckets;             // position 0 has a row of its own
            if (pos + t != 0) {
                const uint64_t n = a.pair_buckets;
                bucket = uint32_t((uint64_t(a.token_log[pos + t - 1]) * a.pair_mul_prev % n + uint64_t(id) * a.pair_mul_cur % n) % n);
            }
            const __nv_bfloat16* pair = static_cast<const __nv_bfloat16*>(a.pair_embed) + size_t(bucket) * a.pair_ld;
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
                NcVec<VEC> v;
                if (i < W) {
                    v.load(pair + i);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) x[k].v[e] += v.v[e];
                }
            }
        }
    } else {
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
            if (i < W) x[k].load(a.x + size_t(t) * W + i);
        }
    }
    if (a.y != nullptr) {
        float part = 0.f;
        if (a.y_index == nullptr) {
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
                if (i < W) y[k].load(a.y + size_t(t) * W + i);
            }
        } else {
#pragma unroll
            for (int k = 0; k < NV; ++k)
#pragma unroll
                for (int e = 0; e < VEC; ++e) y[k].v[e] = 0.f;
            for (uint32_t s = 0; s < a.y_rows; ++s) {
                const float* row = a.y + size_t(a.y_index[t * a.y_rows + s]) * W;
#pragma unroll
                for (int k = 0; k < NV; ++k) {
                    const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
                    NcVec<VEC> v;
                    if (i < W) {
                        v.load(row + i);
#pragma unroll
                        for (int e = 0; e < VEC; ++e) y[k].v[e] += v.v[e];
                    }
                }
            }
            const float n = float(a.y_rows);
#pragma unroll
            for (int k = 0; k < NV; ++k)
#pragma unroll
                for (int e = 0; e < VEC; ++e) y[k].v[e] /= n;
        }
#pragma unroll
        for (int k = 0; k < NV; ++k)
            if ((threadIdx.x + k * blockDim.x) * VEC < W)
#pragma unroll
                for (int e = 0; e < VEC; ++e) part = fmaf(y[k].v[e], y[k].v[e], part);
        const float r = a.mult / sqrtf(block_sum(part, scratch) / float(W) + a.eps);
#pragma unroll
        for (int k = 0; k < NV; ++k)
#pragma unroll
            for (int e = 0; e < VEC; ++e) x[k].v[e] = fmaf(y[k].v[e] * r, w0 + post[k].v[e], x[k].v[e]);
    }
    float part = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
        if (i >= W) continue;
        if (a.trace != nullptr) x[k].store(a.trace + size_t(t) * W + i);
        if (a.step != nullptr) {
            NcVec<VEC> s;
            s.load(a.step + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) x[k].v[e] += s.v[e];
        }
        if (a.x_out != nullptr) x[k].store(a.x_out + size_t(t) * W + i);
#pragma unroll
        for (int e = 0; e < VEC; ++e) part = fmaf(x[k].v[e], x[k].v[e], part);
    }
    if (a.pre_w == nullptr) {
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
            if (i < W) nc_store<VEC, OutT>(a, t, i, x[k]);
        }
        return;
    }
    const float r = 1.f / sqrtf(block_sum(part, scratch) / float(W) + a.eps);
    if (!finish) {
        if (threadIdx.x == 0) a.row_factor[t] = r;
        return;
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
        if (i >= W) continue;
        NcVec<VEC> h, out;
#pragma unroll
        for (int e = 0; e < VEC; ++e) out.v[e] = h.v[e] = x[k].v[e] * r * (w0 + pre[k].v[e]);
        if (a.taps) {
            NcVec<VEC> w, old;
            w.load(a.conv_w + size_t(keep) * W + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) out.v[e] = fmaf(w.v[e], h.v[e], out.v[e]);
            for (uint32_t j = 0; j < keep; ++j) {                   // history oldest first; shifted by one as it is read
                w.load(a.conv_w + size_t(j) * W + i);
                old.load(a.history + size_t(j) * W + i);
                if (pos + j < keep) {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) old.v[e] = 0.f;
                }
#pragma unroll
                for (int e = 0; e < VEC; ++e) out.v[e] = fmaf(w.v[e], old.v[e], out.v[e]);
                if (j > 0) old.store(a.history + size_t(j - 1) * W + i);
            }
            if (keep) h.store(a.history + size_t(keep - 1) * W + i);
        }
        nc_store<VEC, OutT>(a, t, i, out);
    }
}

// Second launch for several tokens: blockIdx.x = channels, blockIdx.y = tokens_per_block tokens.  A thread owns VEC channels
// and slides over its tokens with the last MAXT values of h in registers.  Block row 0 alone reads the state, whose
// successor it writes at its end.
template <int VEC, int MAXT, typename OutT>
__global__ void __launch_bounds__(128) conv_rows_kernel(const NormConvParams p) {
    pdl_launch_dependents();
    const lv_norm_conv_args& a = p.a;
    const uint32_t W = a.width, keep = a.taps - 1, T = a.batch;
    const uint32_t i = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    const uint32_t t0 = blockIdx.y * p.tokens_per_block, t1 = min(T, t0 + p.tokens_per_block);
    if (i >= W) return;
    NcVec<VEC> pre, cw[MAXT], win[MAXT];                  // taps right-aligned: index MAXT - 1 is the current token
    pre.load(a.pre_w + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) pre.v[e] += a.plain_w ? 0.f : 1.f;
#pragma unroll
    for (int j = 0; j < MAXT; ++j) {
        const int s = j - (MAXT - int(a.taps));
        if (s >= 0) cw[j].load(a.conv_w + size_t(s) * W + i);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            if (s < 0) cw[j].v[e] = 0.f;
            win[j].v[e] = 0.f;
        }
    }
    pdl_wait();
    const uint32_t pos = *a.pos;
    auto h_of = [&](uint32_t t) {
        NcVec<VEC> h;
        h.load(a.x_out + size_t(t) * W + i);
        const float r = a.row_factor[t];
#pragma unroll
        for (int e = 0; e < VEC; ++e) h.v[e] = h.v[e] * r * pre.v[e];
        return h;
    };
    // the window before t0: win[j] is h of the token MAXT - j before t0, from this step or from the state
#pragma unroll
    for (int j = 1; j < MAXT; ++j) {
        const uint32_t back = MAXT - j;                   // 1 .. MAXT - 1
        if (back > keep) continue;
        if (t0 >= back) win[j] = h_of(t0 - back);
        else if (blockIdx.y == 0 && pos >= back) win[j].load(a.history + size_t(keep - back) * W + i);
    }
#pragma unroll 2
    for (uint32_t t = t0; t < t1; ++t) {
#pragma unroll
        for (int j = 0; j + 1 < MAXT; ++j) win[j] = win[j + 1];
        win[MAXT - 1] = h_of(t);
        NcVec<VEC> out = win[MAXT - 1];
#pragma unroll
        for (int j = 0; j < MAXT; ++j)
#pragma unroll
            for (int e = 0; e < VEC; ++e) out.v[e] = fmaf(cw[j].v[e], win[j].v[e], out.v[e]);
        nc_store<VEC, OutT>(a, t, i, out);
    }
    if (blockIdx.y != 0) return;
    for (uint32_t j = 0; j < keep; ++j) {                 // ascending: entries that stay move towards lower indexes
        NcVec<VEC> v;
        if (j + T < keep) {
            v.load(a.history + size_t(j + T) * W + i);
            if (pos + j + T < keep) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) v.v[e] = 0.f;
            }
        } else {
            v = h_of(j + T - keep);
        }
        v.store(a.history + size_t(j) * W + i);
    }
}

template <typename OutT>
static int norm_conv_launch(lv_ctx* ctx, const lv_norm_conv_args& a) {
    NormConvParams p{};
    p.a = a;
    p.err = ctx->d_err;
    // four channels per access where every row starts on 16 bytes
    auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15u) == 0; };
    bool vec = a.width % 4 == 0 && a.out_ld % 4 == 0 && a.embed_ld % 4 == 0 && a.pair_ld % 4 == 0;
    for (const void* q : {static_cast<const void*>(a.x), a.embed, a.pair_embed, static_cast<const void*>(a.y), static_cast<const void*>(a.post_w), static_cast<const void*>(a.step),
                          static_cast<const void*>(a.trace), static_cast<const void*>(a.x_out), static_cast<const void*>(a.pre_w),
                          static_cast<const void*>(a.conv_w), static_cast<const void*>(a.history), static_cast<const void*>(a.out)})
        vec = vec && aligned(q);
    const uint32_t count = a.batch - a.first, units = vec ? a.width / 4 : a.width;
    uint32_t nv = vec ? (units <= 1024 ? 1 : units <= 2048 ? 2 : 4) : 16;
    if (vec && units >= 512 && nv == 1) nv = 2;           // fewer warps to sum over
    const uint32_t threads = ((units + nv - 1) / nv + 31) / 32 * 32;
    auto rows = [&](auto kernel) { return launch_pdl(ctx, kernel, dim3(count), dim3(threads), 0, p); };
    if (!vec) LV_CUDA(rows(norm_rows_kernel<1, 16, OutT>));
    else if (nv == 1) LV_CUDA(rows(norm_rows_kernel<4, 1, OutT>));
    else if (nv == 2) LV_CUDA(rows(norm_rows_kernel<4, 2, OutT>));
    else LV_CUDA(rows(norm_rows_kernel<4, 4, OutT>));
    if (a.taps == 0 || a.batch == 1) return LV_OK;
    // the blocks of the first tokens read the state alone: every token that needs it lies in block row 0
    const uint32_t keep = a.taps - 1, cta_columns = (units + 127) / 128;
    p.tokens_per_block = 16;
    while (p.tokens_per_block > 4 && cta_columns * ((count + p.tokens_per_block - 1) / p.tokens_per_block) < 4u * uint32_t(ctx->sm_count)) p.tokens_per_block /= 2;
    if (p.tokens_per_block < keep) p.tokens_per_block = keep;
    const dim3 grid(cta_columns, (count + p.tokens_per_block - 1) / p.tokens_per_block);
    auto conv = [&](auto kernel) { return launch_pdl(ctx, kernel, grid, dim3(128), 0, p); };
    if (vec && a.taps <= 4) LV_CUDA(conv(conv_rows_kernel<4, 4, OutT>));
    else if (a.taps <= 4) LV_CUDA(conv(conv_rows_kernel<1, 4, OutT>));
    else if (vec && a.taps <= 8) LV_CUDA(conv(conv_rows_kernel<4, 8, OutT>));
    else if (vec) LV_CUDA(conv(conv_rows_kernel<4, 16, OutT>));
    else LV_CUDA(conv(conv_rows_kernel<1, 16, OutT>));
    return LV_OK;
}

}  // namespace lv

using namespace lv;

extern "C" int lv_norm_conv(lv_ctx* ctx, const lv_norm_conv_args* args) {
    LV_ENTER(ctx);
    LV_REQUIRE(args != nullptr, "null argument");
    const lv_norm_conv_args& a = *args;
    LV_REQUIRE(a.pos && (a.pre_w || a.taps == 0) && a.out && a.width && a.batch && a.first < a.batch, "bad norm_conv arguments");
    LV_REQUIRE(a.width <= 16384, "norm_conv: width above 16384");
    LV_REQUIRE(a.x != nullptr || (a.embed && a.token_log && a.vocab && a.embed_ld >= a.width), "norm_conv: no input stream");
    LV_REQUIRE(a.pair_embed == nullptr || (a.token_log && a.pair_buckets && a.pair_ld >= a.width), "norm_conv: bad table of pairs");
    LV_REQUIRE(a.y == nullptr || (a.post_w && a.y_rows && (a.y_index || a.y_rows == 1)), "norm_conv: bad sublayer rows");
    LV_REQUIRE(a.taps <= kNormConvMaxTaps && (a.taps == 0 || (a.conv_w && a.first == 0)) && (a.taps < 2 || a.history), "norm_conv: bad taps");
    LV_REQUIRE(a.taps == 0 || a.batch == 1 || (a.x_out && a.row_factor), "norm_conv: several tokens need x_out and row_factor");
    LV_REQUIRE(a.out_index == nullptr || a.out_copies, "norm_conv: bad output rows");
    LV_REQUIRE(a.out_type == LV_TYPE_F32 || a.out_type == LV_TYPE_BF16, "norm_conv: output type");
    return a.out_type == LV_TYPE_F32 ? norm_conv_launch<float>(ctx, a) : norm_conv_launch<__nv_bfloat16>(ctx, a);
}
