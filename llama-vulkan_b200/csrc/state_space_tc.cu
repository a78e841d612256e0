// The state-space recurrence of state_space.cu for the prompts of bfloat16 models, as matrix products over chunks of 64 tokens.
//
// With L the running sum of log a from the beginning of a chunk and S the state before it (f32 [state][vdim]),
//
//   G_ij = C_i . B_j                                       M_ij = G_ij dt_j exp(L_i - L_j),  j <= i
//   y_i  = sum_j M_ij x_j + exp(L_i) C_i S                 S'   = exp(L_63) S + sum_j B_j (dt_j exp(L_63 - L_j) x_j)^T
//
// x, B and C are bfloat16 (the convolution's output).  Everything else is f32: M, the weighted x and S enter their products as
// three bfloat16 terms that add up to the f32 value, and sums are f32.  L is summed in f64 and kept as two f32 terms, so that
// differences of large sums stay exact.
//
// A CTA has 32 columns of one head and walks its chunks in order, S in the accumulators of its eight warps (a warp: sixteen state
// rows).  For y a warp has sixteen tokens and sixteen columns.  The tiles are small and the chain from chunk to chunk
// is serial, so the products are warp-level (mma.sync): M goes from accumulators to operands without leaving the warp's registers.
#include <cuda_bf16.h>
#include <math.h>

#include "common.cuh"
#include "ctx.h"
#include "state_space.cuh"

namespace lv {

constexpr int kStThreads = 256, kStTokens = 64, kStCols = 32;
constexpr int kStXLd = kStCols + 8;          // row strides of tiles in shared memory: an odd multiple of 16 bytes

__device__ __forceinline__ void st_ldmatrix(uint32_t (&r)[4], const __nv_bfloat16* at) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(at)) : "memory");
}
__device__ __forceinline__ void st_ldmatrix_t(uint32_t (&r)[4], const __nv_bfloat16* at) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(at)) : "memory");
}
// d (16 x 8, f32) += a (16 x 16) b (16 x 8)
__device__ __forceinline__ void st_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two f32 as three pairs of bfloat16 that add up to them
__device__ __forceinline__ void st_split(uint32_t (&out)[3], float lo, float hi) {
#pragma unroll
    for (int k = 0; k < 3; ++k) {
        const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
        out[k] = *reinterpret_cast<const uint32_t*>(&v);
        lo -= __uint_as_float(out[k] << 16);
        hi -= __uint_as_float(out[k] & 0xffff0000u);
    }
}

template <int NP> constexpr size_t st_smem_bytes() {
    return size_t(3 * kStTokens * (NP + 8) + 2 * kStTokens * kStXLd + 3 * kStTokens * kStXLd + 3 * NP * kStXLd) * 2;
}

// NP: state rows, padded
template <int NP>
__global__ void __launch_bounds__(kStThreads, NP <= 128 ? 2 : 1) ssm_tc_kernel(const SsmParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const lv_ssm_args& a = p.a;
    constexpr uint32_t kLd = NP + 8, kTile = kStTokens * kLd, kXTile = kStTokens * kStXLd, kSTile = NP * kStXLd;
    const uint32_t blocks = (a.vdim + kStCols - 1) / kStCols, h = blockIdx.x / blocks, c0 = (blockIdx.x - h * blocks) * kStCols;
    const uint32_t cols = min(uint32_t(kStCols), a.vdim - c0), g = h / (a.heads / a.groups);
    __nv_bfloat16* s_c = reinterpret_cast<__nv_bfloat16*>(smem_raw);      // [tokens][NP]
    __nv_bfloat16* s_b = s_c + kTile;                                      // [2][tokens][NP]
    __nv_bfloat16* s_x = s_b + 2 * kTile;                                  // [2][tokens][columns]
    __nv_bfloat16* s_wx = s_x + 2 * kXTile;                                // [3][tokens][columns]: terms of the weighted x
    __nv_bfloat16* s_s = s_wx + 3 * kXTile;                                // [3][NP][columns]: terms of S
    __shared__ __align__(16) float s_rate[2][kStTokens][2];                // dt, log a
    __shared__ __align__(16) float s_hi[kStTokens], s_lo[kStTokens], s_dt[kStTokens], s_el[kStTokens], s_w[kStTokens], s_total;
    const uint32_t lane = threadIdx.x & 31u, warp = threadIdx.x >> 5;
    const uint32_t gi = lane >> 2, ti = lane & 3u;                          // row and column pair of an accumulator
    const uint32_t mt = warp >> 1, ph = (warp & 1u) * 16u;                  // tokens 16 mt .., columns ph .. of y
    const float Dh = a.D[h];
    pdl_wait();
    const uint32_t T = p.batch, chunks = (T + kStTokens - 1) / kStTokens;
    const auto* conv = static_cast<const __nv_bfloat16*>(p.conv);
    auto copy16 = [](const void* dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory"); };
    // rows of `width` values (a multiple of 8, `live` of them there) of a chunk's tokens, zero behind the last token and value
    auto fetch = [&](__nv_bfloat16* dst, uint32_t ld, uint32_t width, uint32_t live, uint32_t chunk, uint32_t column) {
        const uint32_t t0 = chunk * kStTokens, units = width / 8;
        for (uint32_t i = threadIdx.x; i < kStTokens * units; i += kStThreads) {
            const uint32_t t = i / units, q = i - t * units;
            if (t0 + t < T && q * 8 < live) copy16(dst + t * ld + q * 8, conv + size_t(t0 + t) * p.conv_ld + column + q * 8);
            else *reinterpret_cast<uint4*>(dst + t * ld + q * 8) = make_uint4(0u, 0u, 0u, 0u);
        }
    };
    auto fetch_bx = [&](uint32_t chunk) {
        const uint32_t into = chunk & 1u, t0 = chunk * kStTokens;
        fetch(s_b + into * kTile, kLd, NP, p.state_p, chunk, p.b_at + g * p.state_p);
        fetch(s_x + into * kXTile, kStXLd, kStCols, cols, chunk, h * a.vdim + c0);
        for (uint32_t i = threadIdx.x; i < kStTokens; i += kStThreads) {
            float2* dst = reinterpret_cast<float2*>(s_rate[into][i]);
            if (t0 + i < T) asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(smem_u32(dst)), "l"(p.rates + (size_t(t0 + i) * a.heads + h) * 2) : "memory");
            else *dst = make_float2(0.f, 0.f);
        }
    };
    fetch_bx(0);
    fetch(s_c, kLd, NP, p.state_p, 0, p.c_at + g * p.state_p);
    // S: sixteen state rows per warp and tile
    constexpr int kTiles = NP / 16, kPer = (kTiles + 7) / 8;
    float S[kPer][4][4];
    float* state = a.S + (size_t(h) * a.vdim + c0) * p.state_p;
    const bool fresh = *a.pos == 0;
    auto element = [&](int m, int n, int e, uint32_t& row, uint32_t& col) {        // of S[m][n][e]
        row = (warp + 8 * m) * 16 + gi + (e >> 1) * 8;
        col = n * 8 + ti * 2 + (e & 1);
    };
#pragma unroll
    for (int m = 0; m < kPer; ++m)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                uint32_t row, col;
                element(m, n, e, row, col);
                S[m][n][e] = !fresh && row < p.state_p && col < cols ? state[size_t(col) * p.state_p + row] : 0.f;
            }
    auto spread = [&]() {                                                   // the terms of S to shared memory
#pragma unroll
        for (int m = 0; m < kPer; ++m) {
            if (warp + 8 * m >= uint32_t(kTiles)) continue;
#pragma unroll
            for (int n = 0; n < 4; ++n)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t row, col, u[3];
                    element(m, n, 2 * half, row, col);
                    st_split(u, S[m][n][2 * half], S[m][n][2 * half + 1]);
#pragma unroll
                    for (int k = 0; k < 3; ++k) *reinterpret_cast<uint32_t*>(s_s + k * kSTile + row * kStXLd + col) = u[k];
                }
        }
    };
    spread();
    // a lane's row and column in the 16 x 16 tile that an ldmatrix.x4 fetches: [row][k] operands, and the two transposed orders
    const uint32_t r_a = lane & 15u, k_a = (lane >> 4) * 8u;                // A from [m][k]; B from [k][n] (transposed)
    const uint32_t r_b = (lane & 7u) + (lane >> 4) * 8u, k_b = ((lane >> 3) & 1u) * 8u;      // B from [n][k]; A from [k][m] (transposed)
    for (uint32_t chunk = 0; chunk < chunks; ++chunk) {
        const uint32_t buffer = chunk & 1u, t0 = chunk * kStTokens;
        const __nv_bfloat16 *b = s_b + buffer * kTile, *x = s_x + buffer * kXTile;
        asm volatile("cp.async.wait_all;" ::: "memory");
        __syncthreads();
        if (chunk + 1 < chunks) fetch_bx(chunk + 1);
        // z of this warp's outputs, requested early
        float z[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t t = t0 + mt * 16 + gi + (e >> 1) * 8, col = ph + n * 8 + ti * 2 + (e & 1);
                z[n][e] = t < T && col < cols ? a.raw[size_t(t) * a.raw_ld + h * a.vdim + c0 + col] : 0.f;
            }
        if (warp == 0) {                                                    // two tokens per lane
            const float4 r = *reinterpret_cast<const float4*>(s_rate[buffer][2 * lane]);
            double sum = double(r.y) + double(r.w);
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double v = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= uint32_t(o)) sum += v;
            }
            const double end = __shfl_sync(0xffffffffu, sum, 31), L[2] = {sum - double(r.w), sum};
            const float dt[2] = {r.x, r.z};
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const float hi = float(L[k]);
                s_hi[2 * lane + k] = hi;
                s_lo[2 * lane + k] = float(L[k] - double(hi));
                s_dt[2 * lane + k] = dt[k];
                s_el[2 * lane + k] = expf(hi);
                s_w[2 * lane + k] = dt[k] * expf(float(end - L[k]));
            }
            if (lane == 0) s_total = expf(float(end));
        }
        // G, without the tiles above the diagonal
        float G[8][4] = {};
#pragma unroll
        for (int k = 0; k < NP / 16; ++k) {
            uint32_t ca[4];
            st_ldmatrix(ca, s_c + (mt * 16 + r_a) * kLd + k * 16 + k_a);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (uint32_t(j) > mt) continue;
                uint32_t bb[4];
                st_ldmatrix(bb, b + (j * 16 + r_b) * kLd + k * 16 + k_b);
                st_mma(G[2 * j], ca, bb[0], bb[1]);
                st_mma(G[2 * j + 1], ca, bb[2], bb[3]);
            }
        }
        __syncthreads();
        // weighted x, for S'
        for (uint32_t i = threadIdx.x; i < kStTokens * kStCols / 2; i += kStThreads) {
            const uint32_t t = i / (kStCols / 2), q = (i - t * (kStCols / 2)) * 2, v = *reinterpret_cast<const uint32_t*>(x + t * kStXLd + q);
            const float w = s_w[t];
            uint32_t u[3];
            st_split(u, __uint_as_float(v << 16) * w, __uint_as_float(v & 0xffff0000u) * w);
#pragma unroll
            for (int k = 0; k < 3; ++k) *reinterpret_cast<uint32_t*>(s_wx + k * kXTile + t * kStXLd + q) = u[k];
        }
        // M x
        float y[2][4] = {};
        const uint32_t i0 = mt * 16 + gi;
        const float hi_i[2] = {s_hi[i0], s_hi[i0 + 8]}, lo_i[2] = {s_lo[i0], s_lo[i0 + 8]};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            if (uint32_t(j) > mt) continue;
            uint32_t m[3][4], xb[4];
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const uint32_t col = j * 16 + n * 8 + ti * 2;
                const float2 hi_j = *reinterpret_cast<const float2*>(s_hi + col), lo_j = *reinterpret_cast<const float2*>(s_lo + col), dt_j = *reinterpret_cast<const float2*>(s_dt + col);
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const uint32_t i = i0 + 8 * r;
                    const float m0 = col <= i ? G[2 * j + n][2 * r] * (expf((hi_i[r] - hi_j.x) + (lo_i[r] - lo_j.x)) * dt_j.x) : 0.f;
                    const float m1 = col + 1 <= i ? G[2 * j + n][2 * r + 1] * (expf((hi_i[r] - hi_j.y) + (lo_i[r] - lo_j.y)) * dt_j.y) : 0.f;
                    uint32_t u[3];
                    st_split(u, m0, m1);
#pragma unroll
                    for (int k = 0; k < 3; ++k) m[k][2 * n + r] = u[k];
                }
            }
            st_ldmatrix_t(xb, x + (j * 16 + r_a) * kStXLd + ph + k_a);
#pragma unroll
            for (int k = 0; k < 3; ++k) {
                st_mma(y[0], m[k], xb[0], xb[1]);
                st_mma(y[1], m[k], xb[2], xb[3]);
            }
        }
        // C S
        float o[2][4] = {};
#pragma unroll
        for (int k = 0; k < NP / 16; ++k) {
            uint32_t ca[4];
            st_ldmatrix(ca, s_c + (mt * 16 + r_a) * kLd + k * 16 + k_a);
#pragma unroll
            for (int s = 0; s < 3; ++s) {
                uint32_t sb[4];
                st_ldmatrix_t(sb, s_s + s * kSTile + (k * 16 + r_a) * kStXLd + ph + k_a);
                st_mma(o[0], ca, sb[0], sb[1]);
                st_mma(o[1], ca, sb[2], sb[3]);
            }
        }
        const float el[2] = {s_el[i0], s_el[i0 + 8]};
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const uint32_t t = t0 + i0 + 8 * r, col = ph + n * 8 + ti * 2;
                const uint32_t v = *reinterpret_cast<const uint32_t*>(x + (i0 + 8 * r) * kStXLd + col);
                const float y0 = fmaf(Dh, __uint_as_float(v << 16), fmaf(el[r], o[n][2 * r], y[n][2 * r]));
                const float y1 = fmaf(Dh, __uint_as_float(v & 0xffff0000u), fmaf(el[r], o[n][2 * r + 1], y[n][2 * r + 1]));
                float* out = p.gated + size_t(t) * p.inner + h * a.vdim + c0 + col;
                if (t < T && col < cols)                                    // (cols is even)
                    *reinterpret_cast<float2*>(out) = make_float2(y0 * silu_f32(z[n][2 * r]), y1 * silu_f32(z[n][2 * r + 1]));
            }
        __syncthreads();
        if (chunk + 1 < chunks) fetch(s_c, kLd, NP, p.state_p, chunk + 1, p.c_at + g * p.state_p);
        // S'
        const float total = s_total;
#pragma unroll
        for (int m = 0; m < kPer; ++m) {
            if (warp + 8 * m >= uint32_t(kTiles)) continue;
#pragma unroll
            for (int n = 0; n < 4; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[m][n][e] *= total;
#pragma unroll
            for (int k = 0; k < kStTokens / 16; ++k) {
                uint32_t ba[4];
                st_ldmatrix_t(ba, b + (k * 16 + r_b) * kLd + (warp + 8 * m) * 16 + k_b);
#pragma unroll
                for (int s = 0; s < 3; ++s)
#pragma unroll
                    for (int n = 0; n < 2; ++n) {
                        uint32_t xb[4];
                        st_ldmatrix_t(xb, s_wx + s * kXTile + (k * 16 + r_a) * kStXLd + n * 16 + k_a);
                        st_mma(S[m][2 * n], ba, xb[0], xb[1]);
                        st_mma(S[m][2 * n + 1], ba, xb[2], xb[3]);
                    }
            }
        }
        spread();
    }
#pragma unroll
    for (int m = 0; m < kPer; ++m)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                uint32_t row, col;
                element(m, n, e, row, col);
                if (warp + 8 * m < uint32_t(kTiles) && row < p.state_p && col < cols) state[size_t(col) * p.state_p + row] = S[m][n][e];
            }
}

bool ssm_tc_supported(const lv_ssm_args& a) { return a.vdim % 8 == 0 && a.state <= kSsMaxState; }

template <int NP>
static int ssm_tc_launch_rows(lv_ctx* ctx, const SsmParams& p) {
    constexpr size_t smem = st_smem_bytes<NP>();
    LV_REQUIRE(smem <= size_t(ctx->max_smem_optin), "ssm: state needs too much shared memory");
    LV_CUDA(cudaFuncSetAttribute(ssm_tc_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    LV_CUDA(launch_pdl(ctx, ssm_tc_kernel<NP>, dim3(p.a.heads * ((p.a.vdim + kStCols - 1) / kStCols)), dim3(kStThreads), smem, p));
    return LV_OK;
}

int ssm_tc_launch(lv_ctx* ctx, const SsmParams& p) {
    if (p.state_p <= 32) return ssm_tc_launch_rows<32>(ctx, p);
    if (p.state_p <= 64) return ssm_tc_launch_rows<64>(ctx, p);
    if (p.state_p <= 128) return ssm_tc_launch_rows<128>(ctx, p);
    return ssm_tc_launch_rows<256>(ctx, p);
}

}  // namespace lv
