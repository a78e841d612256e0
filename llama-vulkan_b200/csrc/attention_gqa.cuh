// Pieces shared by the attention kernels with bfloat16 or f32 caches.
#pragma once

#include <cuda_bf16.h>

#include "../../include/lv_b200.h"
#include "common.cuh"

namespace lv {

// attention_gqa_tc.cu: the form for several tokens and bfloat16 caches
bool gqa_tc_supported(const lv_gqa_args& a, uint32_t batch);
int gqa_tc_launch(lv_ctx* ctx, const lv_gqa_args& a, uint32_t batch);
// The same for a latent cache: kv holds keys [heads][dim] and, from column v_at on, values [heads][vdim] of the `rows` positions that
// the step sees, expanded for the heads h0 .. h0 + n - 1, bfloat16 with ld elements per position
bool latent_tc_supported(const lv_latent_args& a);
int latent_tc_launch(lv_ctx* ctx, const lv_latent_args& a, uint32_t batch, const void* kv, uint32_t ld, uint32_t v_at, uint32_t rows, uint32_t h0, uint32_t n);

__device__ __forceinline__ void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// a float in the shared memory of another CTA of the cluster
__device__ __forceinline__ float cluster_load(const float* local, uint32_t rank) {
    uint32_t at;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(at) : "r"(smem_u32(local)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(at));
    return v;
}

// 1 / rms of one head's vector, computed by a warp (every lane gets it)
__device__ __forceinline__ float gqa_rms_factor(const float* v, uint32_t dim, float eps) {
    float part = 0.f;
    for (uint32_t i = threadIdx.x & 31u; i < dim; i += 32) part = fmaf(v[i], v[i], part);
    return 1.f / sqrtf(warp_sum(part) / float(dim) + eps);
}

// A head's vector spread over a warp: value lane + 32 i in v[i]; zeros beyond dim and for warps without one
template <int N>
__device__ __forceinline__ void gqa_head_load(float (&v)[N], const float* src, uint32_t dim, bool live) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const uint32_t c = (threadIdx.x & 31u) + 32u * i;
        v[i] = live && c < dim ? src[c] : 0.f;
    }
}
// 1 / rms of such a vector
template <int N>
__device__ __forceinline__ float gqa_head_factor(const float (&v)[N], uint32_t dim, float eps) {
    float part = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) part = fmaf(v[i], v[i], part);
    return 1.f / sqrtf(warp_sum(part) / float(dim) + eps);
}

__device__ __forceinline__ void gqa_store_out(void* out, uint32_t bf16, size_t at, float v) {
    if (bf16) static_cast<__nv_bfloat16*>(out)[at] = __float2bfloat16_rn(v);
    else static_cast<float*>(out)[at] = v;
}

}  // namespace lv
