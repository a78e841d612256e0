// The gated recurrence of lv_gemv_bf16_mingru for several tokens at once: S_t = (1 - z_t) S_(t-1) + z_t c_t per channel is a
// first-order linear recurrence, so a run of tokens acts on the state as S -> A S + B.  The tokens are cut into 32 segments;
// every (channel, segment) thread forms its A and B, one warp chains the segments of 32 channels, and each thread then
// walks its segment again from the right state.  All of it in f32.
#include <cuda_bf16.h>

#include "common.cuh"
#include "ctx.h"

namespace lv {

constexpr int kScanSegments = 32;

struct MingruScanParams {
    const float* raw;           // [T][raw_ld]: z, x, g products side by side
    uint32_t raw_ld, channels, T;
    const float* bz;
    const float* bx;
    float* state;
    const uint32_t* pos;
    void* out;
    uint32_t out_ld;
};

template <typename OutT> __device__ __forceinline__ void scan_store(void* out, size_t at, float v);
template <> __device__ __forceinline__ void scan_store<float>(void* out, size_t at, float v) { static_cast<float*>(out)[at] = v; }
template <> __device__ __forceinline__ void scan_store<__nv_bfloat16>(void* out, size_t at, float v) { static_cast<__nv_bfloat16*>(out)[at] = __float2bfloat16_rn(v); }

// PER > 0: a segment has at most PER tokens, whose gate and candidate stay in registers between the two walks.
template <int PER, typename OutT>
__global__ void __launch_bounds__(1024) mingru_scan_kernel(const MingruScanParams p) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float s_a[kScanSegments][32], s_b[kScanSegments][32];
    const uint32_t lane = threadIdx.x & 31u, seg = threadIdx.x >> 5;
    const uint32_t c = blockIdx.x * 32u + lane;
    const bool live = c < p.channels;
    const uint32_t per = (p.T + kScanSegments - 1) / kScanSegments, t0 = min(p.T, seg * per), t1 = live ? min(p.T, t0 + per) : t0;
    const float bz = live ? p.bz[c] : 0.f, bx = live ? p.bx[c] : 0.f;
    constexpr int N = PER > 0 ? PER : 1;
    float z[N], u[N], A = 1.f, B = 0.f;
    if constexpr (PER > 0) {
#pragma unroll
        for (int i = 0; i < N; ++i) {                    // all loads before the first use
            if (t0 + i >= t1) continue;
            const float* r = p.raw + size_t(t0 + i) * p.raw_ld + c;
            z[i] = r[0];
            u[i] = r[p.channels];
        }
#pragma unroll
        for (int i = 0; i < N; ++i) {
            if (t0 + i >= t1) continue;
            z[i] = sigmoid_f32(z[i] + bz);
            u[i] = z[i] * mingru_candidate(u[i] + bx);
            A *= 1.f - z[i];
            B = fmaf(1.f - z[i], B, u[i]);
        }
    } else {
#pragma unroll 4
        for (uint32_t t = t0; t < t1; ++t) {
            const float* r = p.raw + size_t(t) * p.raw_ld + c;
            const float k = sigmoid_f32(r[0] + bz), cand = mingru_candidate(r[p.channels] + bx);
            A *= 1.f - k;
            B = fmaf(1.f - k, B, k * cand);
        }
    }
    s_a[seg][lane] = A;
    s_b[seg][lane] = B;
    __syncthreads();
    if (seg == 0 && live) {
        float S = *p.pos == 0 ? 0.f : p.state[c];
        for (int s = 0; s < kScanSegments; ++s) {
            const float a = s_a[s][lane], b = s_b[s][lane];
            s_a[s][lane] = S;                           // the state a segment starts from
            S = fmaf(a, S, b);
        }
    }
    __syncthreads();
    if (t0 >= t1) return;
    float S = s_a[seg][lane];
    if constexpr (PER > 0) {
        float g[N];
#pragma unroll
        for (int i = 0; i < N; ++i) g[i] = t0 + i < t1 ? p.raw[size_t(t0 + i) * p.raw_ld + 2 * p.channels + c] : 0.f;
#pragma unroll
        for (int i = 0; i < N; ++i) {
            if (t0 + i >= t1) continue;
            S = fmaf(1.f - z[i], S, u[i]);
            scan_store<OutT>(p.out, size_t(t0 + i) * p.out_ld + c, S * silu_f32(g[i]));
        }
    } else {
#pragma unroll 4
        for (uint32_t t = t0; t < t1; ++t) {
            const float* r = p.raw + size_t(t) * p.raw_ld + c;
            scan_store<OutT>(p.out, size_t(t) * p.out_ld + c, mingru_step(r[0] + bz, r[p.channels] + bx, r[2 * p.channels], S, &S));
        }
    }
    if (t1 == p.T) p.state[c] = S;                      // the segment that holds the last token
}

template <typename OutT>
static cudaError_t mingru_scan_launch(lv_ctx* ctx, const MingruScanParams& p) {
    const dim3 grid((p.channels + 31) / 32), block(1024);
    if (p.T <= 4 * kScanSegments) return launch_pdl(ctx, mingru_scan_kernel<4, OutT>, grid, block, 0, p);
    if (p.T <= 16 * kScanSegments) return launch_pdl(ctx, mingru_scan_kernel<16, OutT>, grid, block, 0, p);
    return launch_pdl(ctx, mingru_scan_kernel<0, OutT>, grid, block, 0, p);
}

}  // namespace lv

using namespace lv;

extern "C" int lv_mingru_scan(lv_ctx* ctx, void* out, int out_type, uint32_t out_ld, const float* raw, uint32_t raw_ld, uint32_t channels,
                              const float* bz, const float* bx, float* state, const uint32_t* pos, uint32_t batch) {
    LV_ENTER(ctx);
    LV_REQUIRE(out && raw && bz && bx && state && pos && channels && batch, "bad mingru_scan arguments");
    LV_REQUIRE(raw_ld >= 3 * channels && out_ld >= channels && (out_type == LV_TYPE_F32 || out_type == LV_TYPE_BF16), "mingru_scan: bad layout");
    MingruScanParams p{raw, raw_ld, channels, batch, bz, bx, state, pos, out, out_ld};
    LV_CUDA(out_type == LV_TYPE_F32 ? mingru_scan_launch<float>(ctx, p) : mingru_scan_launch<__nv_bfloat16>(ctx, p));
    return LV_OK;
}
