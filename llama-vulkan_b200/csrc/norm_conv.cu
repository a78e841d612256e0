// The boundary between two sublayers of a pre- and post-normalised decoder in one launch: residual add of the finished
// sublayer (its output normalised), an optional vector added to the stream, the norm of the next sublayer and a short
// causal convolution over time on its result.
//
//   y_t   = mean of y_rows rows of the finished sublayer          (experts leave one row per choice)
//   x'_t  = x_t + mult * y_t / rms(y_t) * (1 + post_w)            rms(v) = sqrt(mean(v^2) + eps)
//   x''_t = x'_t + step
//   h_t   = x''_t / rms(x''_t) * (1 + pre_w)
//   out_t = h_t + sum_j conv_w[j] * h_(t - taps + 1 + j)          h before position 0 is zero
//
// x may come from the embedding table instead of the stream.  The last taps - 1 values of h are the state that the next
// step reads; positions before the start of the sequence are masked by the position word, so a state needs no clearing.
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

__device__ __forceinline__ float nc_load_x(const lv_norm_conv_args& a, uint32_t t, uint32_t i, uint32_t id) {
    if (a.x != nullptr) return a.x[size_t(t) * a.width + i];
    return __bfloat162float(static_cast<const __nv_bfloat16*>(a.embed)[size_t(id) * a.embed_ld + i]);
}

__device__ __forceinline__ float nc_load_y(const lv_norm_conv_args& a, uint32_t t, uint32_t i) {
    if (a.y_index == nullptr) return a.y[size_t(t) * a.width + i];
    float v = 0.f;
    for (uint32_t s = 0; s < a.y_rows; ++s) v += a.y[size_t(a.y_index[t * a.y_rows + s]) * a.width + i];
    return v / float(a.y_rows);
}

__device__ __forceinline__ uint32_t nc_token(const lv_norm_conv_args& a, uint32_t pos, uint32_t t, uint32_t* err) {
    if (a.x != nullptr) return 0u;
    uint32_t id = a.token_log[pos + t];
    if (id >= a.vocab) {
        if (threadIdx.x == 0) atomicOr(err, ERR_BAD_INDEX);
        id = 0;
    }
    return id;
}

template <typename OutT> __device__ __forceinline__ OutT nc_cast(float v);
template <> __device__ __forceinline__ float nc_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 nc_cast<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

template <typename OutT>
__device__ __forceinline__ void nc_store(const lv_norm_conv_args& a, uint32_t t, uint32_t i, float v) {
    OutT* out = static_cast<OutT*>(a.out);
    if (a.out_index == nullptr) {
        out[size_t(t - a.first) * a.out_ld + i] = nc_cast<OutT>(v);
    } else {
        for (uint32_t s = 0; s < a.out_copies; ++s) out[size_t(a.out_index[t * a.out_copies + s]) * a.out_ld + i] = nc_cast<OutT>(v);
    }
}

// One token: one CTA, a thread keeps its channels in registers.
template <int NV, typename OutT>
__global__ void __launch_bounds__(1024) norm_conv_one_kernel(const NormConvParams p) {
    pdl_launch_dependents();
    const lv_norm_conv_args& a = p.a;
    __shared__ float scratch[64];
    const uint32_t W = a.width, t = a.first, keep = a.taps ? a.taps - 1 : 0;
    float pre[NV], post[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {                        // weights do not depend on the previous kernel
        const uint32_t i = threadIdx.x + k * blockDim.x;
        pre[k] = i < W ? a.pre_w[i] : 0.f;
        post[k] = (a.y != nullptr && i < W) ? a.post_w[i] : 0.f;
    }
    pdl_wait();
    const uint32_t pos = *a.pos;
    const uint32_t id = nc_token(a, pos, t, p.err);
    float x[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const uint32_t i = threadIdx.x + k * blockDim.x;
        x[k] = i < W ? nc_load_x(a, t, i, id) : 0.f;
    }
    if (a.y != nullptr) {
        float y[NV], part = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const uint32_t i = threadIdx.x + k * blockDim.x;
            y[k] = i < W ? nc_load_y(a, t, i) : 0.f;
            part = fmaf(y[k], y[k], part);
        }
        const float r = a.mult / sqrtf(block_sum(part, scratch) / float(W) + a.eps);
#pragma unroll
        for (int k = 0; k < NV; ++k) x[k] = fmaf(y[k] * r, 1.f + post[k], x[k]);
    }
    float part = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const uint32_t i = threadIdx.x + k * blockDim.x;
        if (i < W) {
            if (a.trace != nullptr) a.trace[size_t(t) * W + i] = x[k];
            if (a.step != nullptr) x[k] += a.step[i];
            if (a.x_out != nullptr) a.x_out[size_t(t) * W + i] = x[k];
            part = fmaf(x[k], x[k], part);
        }
    }
    const float r = 1.f / sqrtf(block_sum(part, scratch) / float(W) + a.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const uint32_t i = threadIdx.x + k * blockDim.x;
        if (i >= W) continue;
        const float h = x[k] * r * (1.f + pre[k]);
        float out = h;
        if (a.taps) {
            out = fmaf(a.conv_w[size_t(keep) * W + i], h, out);
            for (uint32_t j = 0; j < keep; ++j) {                   // history oldest first; shifted by one as it is read
                const float old = pos + j >= keep ? a.history[size_t(j) * W + i] : 0.f;
                out = fmaf(a.conv_w[size_t(j) * W + i], old, out);
                if (j > 0) a.history[size_t(j - 1) * W + i] = old;
            }
            if (keep) a.history[size_t(keep - 1) * W + i] = h;
        }
        nc_store<OutT>(a, t, i, out);
    }
}

// Several tokens: a CTA takes tokens_per_block of them and recomputes the h of the taps - 1 tokens before its first
// (x and x_out are different buffers).  Block 0 alone reads the state, whose successor it writes at its end.
template <int MAXT, typename OutT>
__global__ void __launch_bounds__(512) norm_conv_kernel(const NormConvParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const lv_norm_conv_args& a = p.a;
    extern __shared__ float sm[];                        // per row: mult / rms(y), 1 / rms(x''); then token ids
    const uint32_t W = a.width, keep = a.taps ? a.taps - 1 : 0, T = a.batch;
    const uint32_t t0 = a.first + blockIdx.x * p.tokens_per_block, t1 = min(T, t0 + p.tokens_per_block);
    const uint32_t halo = min(keep, t0);                 // rows before t0 that belong to this step
    const uint32_t r_first = t0 - halo;
    const uint32_t n_main = t1 - r_first;
    const bool keeper = blockIdx.x == 0 && keep != 0;
    const uint32_t tail_first = T > keep ? T - keep : 0; // tokens whose h becomes the state
    const uint32_t n_rows = n_main + (keeper ? T - tail_first : 0);
    float* s_ry = sm;
    float* s_rx = sm + n_rows;
    uint32_t* s_id = reinterpret_cast<uint32_t*>(sm + 2 * n_rows);
    const uint32_t pos = *a.pos;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    for (uint32_t r = warp; r < n_rows; r += nwarps) {
        const uint32_t t = r < n_main ? r_first + r : tail_first + (r - n_main);
        uint32_t id = 0;
        if (a.x == nullptr) {
            id = a.token_log[pos + t];
            if (id >= a.vocab) {
                if (lane == 0) atomicOr(p.err, ERR_BAD_INDEX);
                id = 0;
            }
        }
        float ry = 0.f;
        if (a.y != nullptr) {
            float part = 0.f;
            for (uint32_t i = lane; i < W; i += 32) {
                const float y = nc_load_y(a, t, i);
                part = fmaf(y, y, part);
            }
            ry = a.mult / sqrtf(warp_sum(part) / float(W) + a.eps);
        }
        float part = 0.f;
        for (uint32_t i = lane; i < W; i += 32) {
            float x = nc_load_x(a, t, i, id);
            if (a.y != nullptr) x = fmaf(nc_load_y(a, t, i) * ry, 1.f + a.post_w[i], x);
            if (a.step != nullptr) x += a.step[i];
            part = fmaf(x, x, part);
        }
        const float rx = 1.f / sqrtf(warp_sum(part) / float(W) + a.eps);
        if (lane == 0) { s_ry[r] = ry; s_rx[r] = rx; s_id[r] = id; }
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < W; i += blockDim.x) {
        const float pre = 1.f + a.pre_w[i], post = a.y != nullptr ? 1.f + a.post_w[i] : 0.f, step = a.step != nullptr ? a.step[i] : 0.f;
        float cw[MAXT], win[MAXT];                        // taps right-aligned: index MAXT - 1 is the current token
#pragma unroll
        for (int j = 0; j < MAXT; ++j) {
            const int s = j - (MAXT - int(a.taps));
            cw[j] = s >= 0 ? a.conv_w[size_t(s) * W + i] : 0.f;
            win[j] = 0.f;
        }
        // the window before row r_first; positions before this step come from the state
#pragma unroll
        for (int j = 1; j < MAXT; ++j) {
            // win[j] will be h of the token (MAXT - j) before r_first
            const int back = MAXT - j;                    // 1 .. MAXT - 1
            if (blockIdx.x == 0 && back <= int(keep) && pos >= uint32_t(back)) win[j] = a.history[size_t(keep - back) * W + i];
        }
        auto stream = [&](uint32_t r, uint32_t t) {
            float x = nc_load_x(a, t, i, s_id[r]);
            if (a.y != nullptr) x = fmaf(nc_load_y(a, t, i) * s_ry[r], post, x);
            return x;
        };
        for (uint32_t r = 0; r < n_main; ++r) {
            const uint32_t t = r_first + r;
            float x = stream(r, t);
            const bool mine = r >= halo;
            if (mine && a.trace != nullptr) a.trace[size_t(t) * W + i] = x;
            x += step;
            if (mine && a.x_out != nullptr) a.x_out[size_t(t) * W + i] = x;
            const float h = x * s_rx[r] * pre;
#pragma unroll
            for (int j = 0; j + 1 < MAXT; ++j) win[j] = win[j + 1];
            win[MAXT - 1] = h;
            if (mine) {
                float out = h;
#pragma unroll
                for (int j = 0; j < MAXT; ++j) out = fmaf(cw[j], win[j], out);
                nc_store<OutT>(a, t, i, out);
            }
        }
        if (keeper) {
            for (uint32_t j = 0; j < keep; ++j) {         // ascending: entries that stay move towards lower indexes
                float v;
                if (j + T < keep) {
                    v = pos + j + T >= keep ? a.history[size_t(j + T) * W + i] : 0.f;
                } else {
                    const uint32_t t = j + T - keep, r = n_main + (t - tail_first);
                    v = (stream(r, t) + step) * s_rx[r] * pre;
                }
                a.history[size_t(j) * W + i] = v;
            }
        }
    }
}

template <typename OutT>
static int norm_conv_launch(lv_ctx* ctx, const lv_norm_conv_args& a) {
    NormConvParams p{};
    p.a = a;
    p.err = ctx->d_err;
    const uint32_t count = a.batch - a.first;
    if (a.batch == 1 || (count == 1 && a.taps == 0)) {
        const uint32_t threads = a.width >= 1024 ? 1024 : ((a.width + 31) / 32 * 32);
        const uint32_t nv = (a.width + threads - 1) / threads;
        auto go = [&](auto kernel) { return launch_pdl(ctx, kernel, dim3(1), dim3(threads), 0, p); };
        if (nv <= 1) LV_CUDA(go(norm_conv_one_kernel<1, OutT>));
        else if (nv <= 2) LV_CUDA(go(norm_conv_one_kernel<2, OutT>));
        else if (nv <= 4) LV_CUDA(go(norm_conv_one_kernel<4, OutT>));
        else if (nv <= 8) LV_CUDA(go(norm_conv_one_kernel<8, OutT>));
        else LV_CUDA(go(norm_conv_one_kernel<16, OutT>));
        return LV_OK;
    }
    const uint32_t keep = a.taps ? a.taps - 1 : 0;
    p.tokens_per_block = keep > 4 ? keep : 4;            // block 0 holds every token that reads the state
    const uint32_t blocks = (count + p.tokens_per_block - 1) / p.tokens_per_block;
    const size_t smem = size_t(p.tokens_per_block + 2 * keep) * 12;
    auto go = [&](auto kernel) { return launch_pdl(ctx, kernel, dim3(blocks), dim3(512), smem, p); };
    if (a.taps <= 4) LV_CUDA(go(norm_conv_kernel<4, OutT>));
    else if (a.taps <= 8) LV_CUDA(go(norm_conv_kernel<8, OutT>));
    else LV_CUDA(go(norm_conv_kernel<16, OutT>));
    return LV_OK;
}

}  // namespace lv

using namespace lv;

extern "C" int lv_norm_conv(lv_ctx* ctx, const lv_norm_conv_args* args) {
    LV_ENTER(ctx);
    LV_REQUIRE(args != nullptr, "null argument");
    const lv_norm_conv_args& a = *args;
    LV_REQUIRE(a.pos && a.pre_w && a.out && a.width && a.batch && a.first < a.batch, "bad norm_conv arguments");
    LV_REQUIRE(a.width <= 16384, "norm_conv: width above 16384");
    LV_REQUIRE(a.x != nullptr || (a.embed && a.token_log && a.vocab && a.embed_ld >= a.width), "norm_conv: no input stream");
    LV_REQUIRE(a.y == nullptr || (a.post_w && a.y_rows && (a.y_index || a.y_rows == 1)), "norm_conv: bad sublayer rows");
    LV_REQUIRE(a.taps <= kNormConvMaxTaps && (a.taps == 0 || (a.conv_w && a.first == 0)) && (a.taps < 2 || a.history), "norm_conv: bad taps");
    LV_REQUIRE(a.x == nullptr || a.x != a.x_out || a.batch == 1, "norm_conv: the stream cannot be updated in place for several tokens");
    LV_REQUIRE(a.out_index == nullptr || a.out_copies, "norm_conv: bad output rows");
    LV_REQUIRE(a.out_type == LV_TYPE_F32 || a.out_type == LV_TYPE_BF16, "norm_conv: output type");
    return a.out_type == LV_TYPE_F32 ? norm_conv_launch<float>(ctx, a) : norm_conv_launch<__nv_bfloat16>(ctx, a);
}
