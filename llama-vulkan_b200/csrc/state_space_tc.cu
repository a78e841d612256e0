// The state-space recurrence of state_space.cu for the prompts of bfloat16 models, as matrix products over chunks of 64 tokens.
//
// With L the running sum of log a from the beginning of a chunk and S the state before it (f32 [state][vdim]),
//
//   G_ij = C_i . B_j                                       M_ij = G_ij dt_j exp(L_i - L_j),  j <= i
//   y_i  = sum_j M_ij x_j + exp(L_i) C_i S                 S'   = exp(L_63) S + sum_j B_j (dt_j exp(L_63 - L_j) x_j)^T
//
// x, B and C are bfloat16 (the convolution's output).  Everything else is f32, and so is S, which stays in accumulators: the weighted x
// enters S' as three bfloat16 terms that add up to the f32 value, M and S enter y, which ends in bfloat16, as two terms (16 bits).
// L is summed in f64 and kept as two f32 terms, in units of log 2, so that differences of large sums stay exact.
//
// A CTA has 32 or 64 columns of one head and walks its chunks in order, S in the accumulators of its sixteen warps (a warp: sixteen
// state rows, half of the columns).  For y a warp has sixteen tokens and a quarter of the columns.  The tiles are small and the chain from chunk to chunk
// is serial and bound by latency, so the products are warp-level (mma.sync).  A chunk has three phases: {C S, G, L}, {M, weighted x},
// {M x, S'}; the terms of M lie where those of S were.
#include <cuda_bf16.h>
#include <math.h>

#include "common.cuh"
#include "ctx.h"
#include "state_space.cuh"

namespace lv {

constexpr int kStThreads = 512, kStWarps = kStThreads / 32, kStTokens = 64;
constexpr int kStAhead = 8;                 // chunks whose sums of log a are formed together, a warp each

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
// two f32 as N pairs of bfloat16 that add up to them (8 N bits)
template <int N>
__device__ __forceinline__ void st_split(uint32_t (&out)[N], float lo, float hi) {
#pragma unroll
    for (int k = 0; k < N; ++k) {
        const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
        out[k] = *reinterpret_cast<const uint32_t*>(&v);
        if (k + 1 < N) {
            lo -= __uint_as_float(out[k] << 16);
            hi -= __uint_as_float(out[k] & 0xffff0000u);
        }
    }
}
__device__ __forceinline__ float st_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// row strides of tiles in shared memory: odd multiples of 16 bytes
constexpr int kStMLd = kStTokens + 8;
__host__ __device__ constexpr int st_x_ld(int cols) { return cols + 8; }
template <int NP, int COLS> __host__ __device__ constexpr uint32_t st_terms_elems() {
    return 2 * (NP * st_x_ld(COLS) > kStTokens * kStMLd ? NP * st_x_ld(COLS) : kStTokens * kStMLd);
}
template <int NP, int COLS> constexpr size_t st_smem_bytes() {
    return size_t(3 * kStTokens * (NP + 8) + 5 * kStTokens * st_x_ld(COLS) + st_terms_elems<NP, COLS>()) * 2 +
           size_t(kStAhead) * (5 * kStTokens + 4) * 4;
}

// NP: state rows, padded; COLS: columns of a head per CTA
template <int NP, int COLS>
__global__ void __launch_bounds__(kStThreads, 1) ssm_tc_kernel(const SsmParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const lv_ssm_args& a = p.a;
    constexpr uint32_t kStCols = COLS, kStXLd = st_x_ld(COLS);
    constexpr int kYTiles = COLS / 32, kSTiles = COLS / 16;      // column tiles of a warp
    constexpr uint32_t kLd = NP + 8, kTile = kStTokens * kLd, kXTile = kStTokens * kStXLd, kSTile = NP * kStXLd, kMTile = kStTokens * kStMLd;
    const uint32_t blocks = (a.vdim + kStCols - 1) / kStCols, h = blockIdx.x / blocks, c0 = (blockIdx.x - h * blocks) * kStCols;
    const uint32_t cols = min(kStCols, a.vdim - c0), g = h / (a.heads / a.groups);
    __nv_bfloat16* s_c = reinterpret_cast<__nv_bfloat16*>(smem_raw);      // [tokens][NP]
    __nv_bfloat16* s_b = s_c + kTile;                                      // [2][tokens][NP]
    __nv_bfloat16* s_x = s_b + 2 * kTile;                                  // [2][tokens][columns]
    __nv_bfloat16* s_wx = s_x + 2 * kXTile;                                // [3][tokens][columns]: terms of the weighted x
    __nv_bfloat16* s_s = s_wx + 3 * kXTile;                                // [2][NP][columns]: terms of S
    __nv_bfloat16* s_m = s_s;                                              // [2][tokens][tokens]: terms of M, later in a chunk
    float* s_rates = reinterpret_cast<float*>(s_s + st_terms_elems<NP, COLS>());  // [ahead][5][tokens]: see `rates`; then [ahead] exp(L_63)
    const uint32_t lane = threadIdx.x & 31u, warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0);
    const uint32_t gi = lane >> 2, ti = lane & 3u;                          // row and column pair of an accumulator
    const uint32_t mt = warp >> 2, ph = (warp & 3u) * (COLS / 4);           // tokens 16 mt .., columns ph .. of y
    const uint32_t st = warp >> 1, sh = (warp & 1u) * (COLS / 2);           // state rows 16 st .., columns sh .. of S
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
        const uint32_t into = chunk & 1u;
        fetch(s_b + into * kTile, kLd, NP, p.state_p, chunk, p.b_at + g * p.state_p);
        fetch(s_x + into * kXTile, kStXLd, kStCols, cols, chunk, h * a.vdim + c0);
    };
    fetch_bx(0);
    fetch(s_c, kLd, NP, p.state_p, 0, p.c_at + g * p.state_p);
    constexpr int kTiles = NP / 16, kHalf = kStWarps / 2, kPer = (kTiles + kHalf - 1) / kHalf;
    float S[kPer][kSTiles][4];
    float* state = a.S + (size_t(h) * a.vdim + c0) * p.state_p;
    const bool fresh = *a.pos == 0;
    auto element = [&](int m, int n, int e, uint32_t& row, uint32_t& col) {        // of S[m][n][e]
        row = (st + kHalf * m) * 16 + gi + (e >> 1) * 8;
        col = sh + n * 8 + ti * 2 + (e & 1);
    };
#pragma unroll
    for (int m = 0; m < kPer; ++m)
#pragma unroll
        for (int n = 0; n < kSTiles; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                uint32_t row, col;
                element(m, n, e, row, col);
                S[m][n][e] = !fresh && row < p.state_p && col < cols ? state[size_t(col) * p.state_p + row] : 0.f;
            }
    auto spread = [&]() {                                                   // the terms of S to shared memory
#pragma unroll
        for (int m = 0; m < kPer; ++m) {
            if (st + kHalf * m >= uint32_t(kTiles)) continue;
#pragma unroll
            for (int n = 0; n < kSTiles; ++n)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t row, col, u[2];
                    element(m, n, 2 * half, row, col);
                    st_split(u, S[m][n][2 * half], S[m][n][2 * half + 1]);
#pragma unroll
                    for (int k = 0; k < 2; ++k) *reinterpret_cast<uint32_t*>(s_s + k * kSTile + row * kStXLd + col) = u[k];
                }
        }
    };
    spread();
    // a lane's row and column in the 16 x 16 tile that an ldmatrix.x4 fetches: [row][k] operands, and the two transposed orders
    const uint32_t r_a = lane & 15u, k_a = (lane >> 4) * 8u;                // A from [m][k]; B from [k][n] (transposed)
    const uint32_t r_b = (lane & 7u) + (lane >> 4) * 8u, k_b = ((lane >> 3) & 1u) * 8u;      // B from [n][k]; A from [k][m] (transposed)
    // the ten 16 x 16 tiles of M on and below the diagonal: one per warp
    const bool has_tile = warp < 10;
    const uint32_t tile_row = warp < 4 ? 3 : warp < 7 ? 2 : warp < 9 ? 1 : 0, tile_col = warp < 4 ? warp : warp < 7 ? warp - 4 : warp < 9 ? warp - 7 : 0;
    const uint32_t i0 = mt * 16 + gi;
    // per token of a chunk: L in units of log 2 as two terms, dt, exp(L), dt exp(L_63 - L); two tokens per lane
    auto rates = [&](uint32_t chunk) {
        constexpr double kLog2e = 1.4426950408889634;
        float* dst = s_rates + chunk % kStAhead * 5 * kStTokens + 2 * lane;
        float2 r[2];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const uint32_t t = chunk * kStTokens + 2 * lane + k;
            r[k] = t < T ? *reinterpret_cast<const float2*>(p.rates + (size_t(t) * a.heads + h) * 2) : make_float2(0.f, 0.f);
        }
        const double last = double(r[1].y) * kLog2e;
        double sum = double(r[0].y) * kLog2e + last;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double v = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= uint32_t(o)) sum += v;
        }
        const double end = __shfl_sync(0xffffffffu, sum, 31), L[2] = {sum - last, sum};
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const float hi = float(L[k]);
            dst[k] = hi;
            dst[kStTokens + k] = float(L[k] - double(hi));
            dst[2 * kStTokens + k] = r[k].x;
            dst[3 * kStTokens + k] = exp2f(hi);
            dst[4 * kStTokens + k] = r[k].x * exp2f(float(end - L[k]));
        }
        if (lane == 0) s_rates[kStAhead * 5 * kStTokens + chunk % kStAhead] = exp2f(float(end));
    };
    for (uint32_t chunk = 0; chunk < chunks; ++chunk) {
        const uint32_t buffer = chunk & 1u, t0 = chunk * kStTokens;
        const __nv_bfloat16 *b = s_b + buffer * kTile, *x = s_x + buffer * kXTile;
        const float *s_hi = s_rates + chunk % kStAhead * 5 * kStTokens, *s_lo = s_hi + kStTokens, *s_dt = s_lo + kStTokens, *s_el = s_dt + kStTokens, *s_w = s_el + kStTokens;
        if (chunk % kStAhead == 0) {
            if (chunk != 0) __syncthreads();                                // the last ones have been read
            if (warp < uint32_t(kStAhead) && chunk + warp < chunks) rates(chunk + warp);
        }
        asm volatile("cp.async.wait_all;" ::: "memory");
        __syncthreads();
        if (chunk + 1 < chunks) fetch_bx(chunk + 1);
        // z of this warp's outputs, requested early
        float2 z[kYTiles][2];
#pragma unroll
        for (int n = 0; n < kYTiles; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const uint32_t t = t0 + i0 + 8 * r, col = ph + n * 8 + ti * 2;
                const float* at = a.raw + size_t(t) * a.raw_ld + h * a.vdim + c0 + col;
                z[n][r] = t < T && col < cols ? make_float2(at[0], at[1]) : make_float2(0.f, 0.f);
            }
        // C S; a term's two steps of sixteen state rows come with one ldmatrix
        float o[kYTiles][2][4] = {};                                        // a sum per term
#pragma unroll
        for (int k = 0; k < NP / 32; ++k) {
            uint32_t ca[2][4];
#pragma unroll
            for (int i = 0; i < 2; ++i) st_ldmatrix(ca[i], s_c + (mt * 16 + r_a) * kLd + (2 * k + i) * 16 + k_a);
#pragma unroll
            for (int s = 0; s < 2; ++s)
#pragma unroll
                for (int n = 0; n < kYTiles; ++n) {
                    uint32_t sb[4];
                    st_ldmatrix_t(sb, s_s + s * kSTile + (k * 32 + lane) * kStXLd + ph + n * 8);
                    st_mma(o[n][s], ca[0], sb[0], sb[1]);
                    st_mma(o[n][s], ca[1], sb[2], sb[3]);
                }
        }
        // this warp's tile of G
        float G[2][4] = {};
        if (has_tile) {
#pragma unroll
            for (int k = 0; k < NP / 16; ++k) {
                uint32_t ca[4], bb[4];
                st_ldmatrix(ca, s_c + (tile_row * 16 + r_a) * kLd + k * 16 + k_a);
                st_ldmatrix(bb, b + (tile_col * 16 + r_b) * kLd + k * 16 + k_b);
                st_mma(G[0], ca, bb[0], bb[1]);
                st_mma(G[1], ca, bb[2], bb[3]);
            }
        }
        __syncthreads();
        if (chunk + 1 < chunks) fetch(s_c, kLd, NP, p.state_p, chunk + 1, p.c_at + g * p.state_p);
        // terms of M
        if (has_tile) {
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const uint32_t col = tile_col * 16 + n * 8 + ti * 2;
                const float2 hi_j = *reinterpret_cast<const float2*>(s_hi + col), lo_j = *reinterpret_cast<const float2*>(s_lo + col), dt_j = *reinterpret_cast<const float2*>(s_dt + col);
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const uint32_t i = tile_row * 16 + gi + 8 * r;
                    const float hi_i = s_hi[i], lo_i = s_lo[i];
                    const float m0 = col <= i ? G[n][2 * r] * (st_exp2((hi_i - hi_j.x) + (lo_i - lo_j.x)) * dt_j.x) : 0.f;
                    const float m1 = col + 1 <= i ? G[n][2 * r + 1] * (st_exp2((hi_i - hi_j.y) + (lo_i - lo_j.y)) * dt_j.y) : 0.f;
                    uint32_t u[2];
                    st_split(u, m0, m1);
#pragma unroll
                    for (int k = 0; k < 2; ++k) *reinterpret_cast<uint32_t*>(s_m + k * kMTile + i * kStMLd + col) = u[k];
                }
            }
        }
        // terms of the weighted x
#pragma unroll
        for (int k4 = 0; k4 < kStTokens * COLS / 4 / kStThreads; ++k4) {
            const uint32_t i = threadIdx.x + k4 * kStThreads, t = i / (kStCols / 4), q = i % (kStCols / 4) * 4;
            const uint2 v = *reinterpret_cast<const uint2*>(x + t * kStXLd + q);
            const float w = s_w[t];
            uint32_t u0[3], u1[3];
            st_split(u0, __uint_as_float(v.x << 16) * w, __uint_as_float(v.x & 0xffff0000u) * w);
            st_split(u1, __uint_as_float(v.y << 16) * w, __uint_as_float(v.y & 0xffff0000u) * w);
#pragma unroll
            for (int k = 0; k < 3; ++k) *reinterpret_cast<uint2*>(s_wx + k * kXTile + t * kStXLd + q) = make_uint2(u0[k], u1[k]);
        }
        __syncthreads();
        // M x
        float y[kYTiles][2][4] = {};                                        // a sum per term
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            if (uint32_t(2 * j) > mt) continue;
            uint32_t xb[kYTiles][4];
#pragma unroll
            for (int n = 0; n < kYTiles; ++n) st_ldmatrix_t(xb[n], x + (j * 32 + lane) * kStXLd + ph + n * 8);
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                if (uint32_t(2 * j + i) > mt) continue;
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    uint32_t m[4];
                    st_ldmatrix(m, s_m + k * kMTile + (mt * 16 + r_a) * kStMLd + (2 * j + i) * 16 + k_a);
#pragma unroll
                    for (int n = 0; n < kYTiles; ++n) st_mma(y[n][k], m, xb[n][2 * i], xb[n][2 * i + 1]);
                }
            }
        }
        // S'
        const float total = s_rates[kStAhead * 5 * kStTokens + chunk % kStAhead];
#pragma unroll
        for (int m = 0; m < kPer; ++m) {
            if (st + kHalf * m >= uint32_t(kTiles)) continue;
#pragma unroll
            for (int n = 0; n < kSTiles; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[m][n][e] *= total;
#pragma unroll
            for (int k = 0; k < kStTokens / 16; ++k) {
                uint32_t ba[4];
                st_ldmatrix_t(ba, b + (k * 16 + r_b) * kLd + (st + kHalf * m) * 16 + k_b);
#pragma unroll
                for (int s = 0; s < 3; ++s)
#pragma unroll
                    for (int n = 0; n < kSTiles / 2; ++n) {
                        uint32_t xb[4];
                        st_ldmatrix_t(xb, s_wx + s * kXTile + (k * 16 + r_a) * kStXLd + sh + n * 16 + k_a);
                        st_mma(S[m][2 * n], ba, xb[0], xb[1]);
                        st_mma(S[m][2 * n + 1], ba, xb[2], xb[3]);
                    }
            }
        }
#pragma unroll
        for (int n = 0; n < kYTiles; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const uint32_t t = t0 + i0 + 8 * r, col = ph + n * 8 + ti * 2;
                const uint32_t v = *reinterpret_cast<const uint32_t*>(x + (i0 + 8 * r) * kStXLd + col);
                const float el = s_el[i0 + 8 * r];
                const float y0 = fmaf(Dh, __uint_as_float(v << 16), fmaf(el, o[n][0][2 * r] + o[n][1][2 * r], y[n][0][2 * r] + y[n][1][2 * r]));
                const float y1 = fmaf(Dh, __uint_as_float(v & 0xffff0000u), fmaf(el, o[n][0][2 * r + 1] + o[n][1][2 * r + 1], y[n][0][2 * r + 1] + y[n][1][2 * r + 1]));
                float* out = p.gated + size_t(t) * p.inner + h * a.vdim + c0 + col;
                if (t < T && col < cols)                                    // (cols is even)
                    *reinterpret_cast<float2*>(out) = make_float2(y0 * silu_fast(z[n][r].x), y1 * silu_fast(z[n][r].y));
            }
        if (chunk + 1 == chunks) break;
        __syncthreads();                                                    // the terms of M have been read
        spread();
    }
#pragma unroll
    for (int m = 0; m < kPer; ++m)
#pragma unroll
        for (int n = 0; n < kSTiles; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                uint32_t row, col;
                element(m, n, e, row, col);
                if (st + kHalf * m < uint32_t(kTiles) && row < p.state_p && col < cols) state[size_t(col) * p.state_p + row] = S[m][n][e];
            }
}

bool ssm_tc_supported(const lv_ssm_args& a) { return a.vdim % 8 == 0 && a.state <= kSsMaxState; }

template <int NP, int COLS>
static int ssm_tc_launch_sized(lv_ctx* ctx, const SsmParams& p) {
    constexpr size_t smem = st_smem_bytes<NP, COLS>();
    LV_REQUIRE(smem <= size_t(ctx->max_smem_optin), "ssm: state needs too much shared memory");
    LV_CUDA(cudaFuncSetAttribute(ssm_tc_kernel<NP, COLS>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    LV_CUDA(launch_pdl(ctx, ssm_tc_kernel<NP, COLS>, dim3(p.a.heads * ((p.a.vdim + COLS - 1) / COLS)), dim3(kStThreads), smem, p));
    return LV_OK;
}

template <int NP>
static int ssm_tc_launch_rows(lv_ctx* ctx, const SsmParams& p) {
    // narrow CTAs while all of them run at a time
    if constexpr (NP <= 128)
        if (p.a.vdim > 32 && p.a.heads * ((p.a.vdim + 31) / 32) > uint32_t(ctx->sm_count)) return ssm_tc_launch_sized<NP, 64>(ctx, p);
    return ssm_tc_launch_sized<NP, 32>(ctx, p);
}

int ssm_tc_launch(lv_ctx* ctx, const SsmParams& p) {
    if (p.state_p <= 32) return ssm_tc_launch_rows<32>(ctx, p);
    if (p.state_p <= 64) return ssm_tc_launch_rows<64>(ctx, p);
    if (p.state_p <= 128) return ssm_tc_launch_rows<128>(ctx, p);
    return ssm_tc_launch_rows<256>(ctx, p);
}

}  // namespace lv
