// Gated delta rule with one decay per head and key channel (OP_SHORT_CONV, OP_CHANNEL_DELTA, OP_GATED_NORM).
//
//   short_conv_kernel    causal depthwise convolution + silu; the last taps - 1 inputs are kept in the state, two banks:
//                        a run reads the bank of its parity and writes the other, so that no CTA overwrites what
//                        another still reads
//   delta_prep_kernel    unit vectors, decays, step sizes and the products of neighbouring tokens' vectors, fp32
//   delta_scan_kernel    the recurrence, two tokens at a time: S lives in registers, all reductions of both tokens run side
//                        by side
//   gated_norm_kernel    RMS norm of a head's read-out, weight, sigmoid gate
//   delta_step_kernel    all of it for up to 4 rows, with the second halves of the low-rank decay and gate projections
//
// All of it is fp32, token after token: a cut of the prompt changes nothing but roundings.
#include <cooperative_groups.h>
#include "launchers_rows.h"
#include "mma_bf16.cuh"

namespace gehtp {

namespace {

constexpr uint32_t CONV_ROWS = 16;

// value of channel c at row r of the run (r < 0: from the state bank of the run before)
template <class A>
__device__ __forceinline__ float conv_in(const typename A::T* y, const float* bank, int r, uint32_t c, uint32_t ys, uint32_t C, int keep) {
    return r >= 0 ? A::ld(y + (size_t)r * ys + c) : bank[(size_t)(keep + r) * C + c];
}

template <class A>
__global__ void __launch_bounds__(256)
short_conv_kernel(const typename A::T* y, const float* __restrict__ w, float* state, const uint32_t* count, float* out,
                  uint32_t rows, uint32_t C, uint32_t taps, uint32_t ys) {
    pdl_release();
    pdl_wait();
    const uint32_t c = blockIdx.x * 256 + threadIdx.x;
    if (c >= C) return;
    const int keep = (int)taps - 1;
    const uint32_t par = *count & 1u;
    const float* bank = state + (size_t)par * keep * C;
    const float* wc = w + (size_t)c * taps;
    const uint32_t r0 = blockIdx.y * CONV_ROWS, r1 = min(r0 + CONV_ROWS, rows);
    if (taps == 4) {
        const float w0 = __ldg(wc), w1 = __ldg(wc + 1), w2 = __ldg(wc + 2), w3 = __ldg(wc + 3);
        float x0 = conv_in<A>(y, bank, (int)r0 - 3, c, ys, C, 3), x1 = conv_in<A>(y, bank, (int)r0 - 2, c, ys, C, 3),
              x2 = conv_in<A>(y, bank, (int)r0 - 1, c, ys, C, 3);
#pragma unroll 4
        for (uint32_t r = r0; r < r1; r++) {
            const float x3 = A::ld(y + (size_t)r * ys + c);
            out[(size_t)r * C + c] = silu_f(fmaf(w3, x3, fmaf(w2, x2, fmaf(w1, x1, w0 * x0))));
            x0 = x1; x1 = x2; x2 = x3;
        }
    } else {
        for (uint32_t r = r0; r < r1; r++) {
            float s = 0.0f;
            for (int j = 0; j < (int)taps; j++) s = fmaf(__ldg(wc + j), conv_in<A>(y, bank, (int)r - keep + j, c, ys, C, keep), s);
            out[(size_t)r * C + c] = silu_f(s);
        }
    }
    if (r1 == rows) {
        float* next = state + (size_t)(par ^ 1u) * keep * C;
        for (int i = 0; i < keep; i++) next[(size_t)i * C + c] = conv_in<A>(y, bank, (int)rows - keep + i, c, ys, C, keep);
    }
}

__device__ __forceinline__ float softplus_f(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

// work: k [rows][KH][D], q [rows][KH][D], decay [rows][H][D], {step, k . q, (g k') . k, (g k') . q} [rows][H][4] with k' the
// key of the row before (odd rows only)
struct DeltaWork { float *k, *q, *g, *bk; };
__host__ __device__ inline size_t up4(size_t n) { return (n + 3) & ~(size_t)3; }
inline DeltaWork work_of(const DeltaArgs& a, uint32_t rows) {
    DeltaWork w;
    w.k = a.work;
    w.q = w.k + up4((size_t)rows * a.kv_heads * a.dim);
    w.g = w.q + up4((size_t)rows * a.kv_heads * a.dim);
    w.bk = w.g + up4((size_t)rows * a.heads * a.dim);
    return w;
}

// A warp per head and pair of rows (2 p, 2 p + 1), the head's vectors in registers (DR values per lane).
template <class A, int DR>
__global__ void __launch_bounds__(256)
delta_prep_kernel(const DeltaArgs a, const DeltaWork wk, uint32_t rows) {
    pdl_release();
    pdl_wait();
    const uint32_t h = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, D = a.dim, KH = a.kv_heads, H = a.heads;
    if (h >= H) return;
    const uint32_t rep = H / KH, kh = h / rep, r0 = blockIdx.y * 2;
    const float qs = 1.0f / sqrtf((float)D), ea = expf(__ldg(a.a_log + h));
    float kp[DR], k[DR], q[DR], g[DR];
#pragma unroll
    for (int j = 0; j < DR; j++) kp[j] = 0.0f;
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const uint32_t r = r0 + e;
        if (r >= rows) break;
        const float *qx = a.qkv + (size_t)r * a.channels() + kh * D, *kx = qx + KH * D, *ax = a.a + ((size_t)r * H + h) * D;
        float qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
        for (int j = 0; j < DR; j++) {
            const uint32_t i = lane + 32 * j;
            const bool in = i < D;
            q[j] = in ? __ldcg(qx + i) : 0.0f;
            k[j] = in ? __ldcg(kx + i) : 0.0f;
            g[j] = in ? __ldcg(ax + i) + __ldg(a.dt_bias + h * D + i) : 0.0f;
            qq = fmaf(q[j], q[j], qq); kk = fmaf(k[j], k[j], kk); qk = fmaf(q[j], k[j], qk);
        }
        qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
        const float iq = qs / sqrtf(qq + 1e-6f), ik = 1.0f / sqrtf(kk + 1e-6f);
        float m = 0.0f, n = 0.0f;
#pragma unroll
        for (int j = 0; j < DR; j++) {
            const uint32_t i = lane + 32 * j;
            g[j] = expf(-ea * softplus_f(g[j]));
            q[j] *= iq; k[j] *= ik;
            m = fmaf(g[j] * kp[j], k[j], m);
            n = fmaf(g[j] * kp[j], q[j], n);
            if (i < D) {
                wk.g[((size_t)r * H + h) * D + i] = g[j];
                if (h % rep == 0) {
                    wk.q[((size_t)r * KH + kh) * D + i] = q[j];
                    wk.k[((size_t)r * KH + kh) * D + i] = k[j];
                }
            }
            kp[j] = k[j];
        }
        if (e) { m = warp_sum(m); n = warp_sum(n); }
        if (lane == 0) {
            const float b = A::ld((const typename A::T*)a.y + (size_t)r * a.ys + a.b_col + h);
            *(float4*)(wk.bk + ((size_t)r * H + h) * 4) = make_float4(sigmoid_f(b), qk * iq * ik, m, n);
        }
    }
}

// two fp32 values side by side (fma.rn.f32x2): the same roundings as two scalar operations
__device__ __forceinline__ uint64_t pk2(float a, float b) { uint64_t r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b)); return r; }
__device__ __forceinline__ float sum2(uint64_t v) { float a, b; asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); return a + b; }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) { uint64_t r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) { uint64_t r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r; }

// 16 lanes hold 2 neighbouring columns of S, RPL rows each (as RPL / 2 pairs of values); a warp holds 4 columns, a CTA NW
// warps of one head. Tokens are taken two at a time: with P = g1 S, R = g2 P,
//   u1 = b1 (v1 - P^T k1)                 o1 = P^T q1 + u1 (k1 . q1)
//   u2 = b2 (v2 - R^T k2 - u1 m)          o2 = R^T q2 + u1 n + u2 (k2 . q2)       m = (g2 k1) . k2, n = (g2 k1) . q2
//   S  = R + (g2 k1) u1^T + k2 u2^T
// so that the four sums of both tokens are reduced together. The eight sums of a lane (4 per column) are reduced over its
// 16 lanes by halving - an exchange leaves a lane with half of the sums it had - until lane (token, k or q, column, -)
// holds one. Tokens come in chunks of TC through shared memory (cp.async, two stages; VEC = 16-byte copies); a last odd
// token is paired with one that changes nothing (decay 1, key, query and step 0).
constexpr uint32_t TC = 16;
template <int RPL, int NW, bool VEC>
__global__ void __launch_bounds__(NW * 32)
delta_scan_kernel(const DeltaArgs a, const DeltaWork wk, uint32_t rows) {
    constexpr uint32_t DP = 16 * RPL, NC = NW * 4, NT = NW * 32;
    extern __shared__ __align__(16) float sm[];
    float* s_kqg = sm;                                // [2][TC][3][DP]
    float* s_v = s_kqg + 2 * TC * 3 * DP;             // [2][TC][NC]
    float* s_bk = s_v + 2 * TC * NC;                  // [2][TC][4]
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, H = a.heads, D = a.dim, V = a.vdim;
    const uint32_t h = blockIdx.y, kh = h / (H / a.kv_heads), c0 = blockIdx.x * NC;
    const uint32_t l = lane & 15, base = lane & 16, cl = warp * 4 + (lane >> 4) * 2;      // first of this lane's columns, within the CTA
    const uint32_t C = a.channels(), voff = 2 * a.kv_heads * D + h * V;
    for (uint32_t i = tid; i < 2 * TC * 3 * DP; i += NT)
        if (i % DP >= D) s_kqg[i] = 0.0f;             // rows past D: S stays zero there
    for (uint32_t i = tid; i < 2 * TC * NC; i += NT)
        if (c0 + i % NC >= V) s_v[i] = 0.0f;          // columns past V, which no copy writes
    float* Sg = a.S + (size_t)h * D * V;
    auto row_of = [&](int i) -> uint32_t { return (i / 4) * 64 + l * 4 + (i & 3); };
    uint64_t S[RPL / 2][2];
#pragma unroll
    for (int i = 0; i < RPL; i += 2) {
        const uint32_t r = row_of(i);
#pragma unroll
        for (int c = 0; c < 2; c++) {
            const uint32_t col = c0 + cl + c;
            S[i / 2][c] = pk2((r < D && col < V) ? Sg[(size_t)r * V + col] : 0.0f, (r + 1 < D && col < V) ? Sg[(size_t)(r + 1) * V + col] : 0.0f);
        }
    }
    auto fetch = [&](uint32_t t0, uint32_t stg) {
        const uint32_t nt = t0 < rows ? min(TC, rows - t0) : 0;
        float* d = s_kqg + stg * TC * 3 * DP;
        // warp w copies tokens w, w + NW, ...: k, q and g of a token, lanes along the channels
        for (uint32_t t = warp; t < nt; t += NW) {
            const float* sk = wk.k + ((size_t)(t0 + t) * a.kv_heads + kh) * D;
            const float* sq = wk.q + ((size_t)(t0 + t) * a.kv_heads + kh) * D;
            const float* sg = wk.g + ((size_t)(t0 + t) * H + h) * D;
            float* dt = d + t * 3 * DP;
            if (VEC) {
                for (uint32_t c = lane * 4; c < D; c += 128) {
                    cp16(smem_addr(dt + c), sk + c, 16);
                    cp16(smem_addr(dt + DP + c), sq + c, 16);
                    cp16(smem_addr(dt + 2 * DP + c), sg + c, 16);
                }
            } else {
                for (uint32_t c = lane; c < D; c += 32) { dt[c] = __ldcg(sk + c); dt[DP + c] = __ldcg(sq + c); dt[2 * DP + c] = __ldcg(sg + c); }
            }
            if (lane < NC && c0 + lane < V)
                asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_addr(s_v + (stg * TC + t) * NC + lane)),
                             "l"(a.qkv + (size_t)(t0 + t) * C + voff + c0 + lane) : "memory");
            if (lane == 0) cp16(smem_addr(s_bk + (stg * TC + t) * 4), wk.bk + ((size_t)(t0 + t) * H + h) * 4, 16);
        }
        if ((nt & 1u) && warp == (nt % NW)) {         // the idle partner of a last odd token
            for (uint32_t c = lane; c < D; c += 32) { float* dt = d + nt * 3 * DP; dt[c] = 0.0f; dt[DP + c] = 0.0f; dt[2 * DP + c] = 1.0f; }
            if (lane < NC) s_v[(stg * TC + nt) * NC + lane] = 0.0f;
            if (lane < 4) s_bk[(stg * TC + nt) * 4 + lane] = 0.0f;
        }
        cp_commit();
    };
    fetch(0, 0);
    const bool second = l & 8, isq = l & 4, odd = l & 2;      // the sum this lane ends up with: token, S^T q or S^T k, column
    for (uint32_t t0 = 0, stg = 0; t0 < rows; t0 += TC, stg ^= 1) {
        fetch(t0 + TC, stg ^ 1);
        cp_wait<1>();
        __syncthreads();
        const uint32_t nt = min(TC, rows - t0);
        const float* kqg = s_kqg + stg * TC * 3 * DP + l * 4;
        for (uint32_t t = 0; t < nt; t += 2) {
            const float *p1 = kqg + t * 3 * DP, *p2 = p1 + 3 * DP;
            const float4 bk1 = *(const float4*)(s_bk + (stg * TC + t) * 4), bk2 = *(const float4*)(s_bk + (stg * TC + t + 1) * 4);
            const float2 v1 = *(const float2*)(s_v + (stg * TC + t) * NC + cl), v2 = *(const float2*)(s_v + (stg * TC + t + 1) * NC + cl);
            uint64_t ka[RPL / 2], kb[RPL / 2], a1[2], b1[2], a2[2], b2[2];
#pragma unroll
            for (int i = 0; i < RPL; i += 4) {
                const ulonglong2 k1 = *(const ulonglong2*)(p1 + i * 16), q1 = *(const ulonglong2*)(p1 + DP + i * 16), g1 = *(const ulonglong2*)(p1 + 2 * DP + i * 16);
                const ulonglong2 k2 = *(const ulonglong2*)(p2 + i * 16), q2 = *(const ulonglong2*)(p2 + DP + i * 16), g2 = *(const ulonglong2*)(p2 + 2 * DP + i * 16);
                ka[i / 2] = mul2(g2.x, k1.x); ka[i / 2 + 1] = mul2(g2.y, k1.y);
                kb[i / 2] = k2.x; kb[i / 2 + 1] = k2.y;
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    uint64_t x = mul2(S[i / 2][c], g1.x), y = mul2(S[i / 2 + 1][c], g1.y);
                    a1[c] = i == 0 ? mul2(x, k1.x) : fma2(x, k1.x, a1[c]);
                    b1[c] = i == 0 ? mul2(x, q1.x) : fma2(x, q1.x, b1[c]);
                    a1[c] = fma2(y, k1.y, a1[c]);
                    b1[c] = fma2(y, q1.y, b1[c]);
                    x = mul2(x, g2.x); y = mul2(y, g2.y);
                    a2[c] = i == 0 ? mul2(x, k2.x) : fma2(x, k2.x, a2[c]);
                    b2[c] = i == 0 ? mul2(x, q2.x) : fma2(x, q2.x, b2[c]);
                    a2[c] = fma2(y, k2.y, a2[c]);
                    b2[c] = fma2(y, q2.y, b2[c]);
                    S[i / 2][c] = x; S[i / 2 + 1][c] = y;
                }
            }
            float e4[4], e2[2], e;
            {
                const float x0 = sum2(a1[0]), x1 = sum2(a1[1]), x2 = sum2(b1[0]), x3 = sum2(b1[1]);
                const float y0 = sum2(a2[0]), y1 = sum2(a2[1]), y2 = sum2(b2[0]), y3 = sum2(b2[1]);
                e4[0] = (second ? y0 : x0) + __shfl_xor_sync(0xffffffffu, second ? x0 : y0, 8);
                e4[1] = (second ? y1 : x1) + __shfl_xor_sync(0xffffffffu, second ? x1 : y1, 8);
                e4[2] = (second ? y2 : x2) + __shfl_xor_sync(0xffffffffu, second ? x2 : y2, 8);
                e4[3] = (second ? y3 : x3) + __shfl_xor_sync(0xffffffffu, second ? x3 : y3, 8);
            }
            e2[0] = (isq ? e4[2] : e4[0]) + __shfl_xor_sync(0xffffffffu, isq ? e4[0] : e4[2], 4);
            e2[1] = (isq ? e4[3] : e4[1]) + __shfl_xor_sync(0xffffffffu, isq ? e4[1] : e4[3], 4);
            e = (odd ? e2[1] : e2[0]) + __shfl_xor_sync(0xffffffffu, odd ? e2[0] : e2[1], 2);
            e += __shfl_xor_sync(0xffffffffu, e, 1);
            // S^T k of both tokens and columns to every lane
            const float s10 = __shfl_sync(0xffffffffu, e, base), s11 = __shfl_sync(0xffffffffu, e, base | 2);
            const float s20 = __shfl_sync(0xffffffffu, e, base | 8), s21 = __shfl_sync(0xffffffffu, e, base | 10);
            const float u10 = bk1.x * (v1.x - s10), u11 = bk1.x * (v1.y - s11);
            const float u20 = bk2.x * (v2.x - fmaf(u10, bk2.z, s20)), u21 = bk2.x * (v2.y - fmaf(u11, bk2.z, s21));
            const uint64_t w10 = pk2(u10, u10), w11 = pk2(u11, u11), w20 = pk2(u20, u20), w21 = pk2(u21, u21);
#pragma unroll
            for (int i = 0; i < RPL / 2; i++) {
                S[i][0] = fma2(kb[i], w20, fma2(ka[i], w10, S[i][0]));
                S[i][1] = fma2(kb[i], w21, fma2(ka[i], w11, S[i][1]));
            }
            if (isq && !(l & 1) && c0 + cl + odd < V && t + second < nt) {
                const float u1 = odd ? u11 : u10, u2 = odd ? u21 : u20;
                a.o[((size_t)(t0 + t + second) * H + h) * V + c0 + cl + odd] = second ? fmaf(u2, bk2.y, fmaf(u1, bk2.w, e)) : fmaf(u1, bk1.y, e);
            }
        }
        __syncthreads();
    }
    cp_wait<0>();
#pragma unroll
    for (int i = 0; i < RPL; i += 2) {
        const uint32_t r = row_of(i);
#pragma unroll
        for (int c = 0; c < 2; c++) {
            const uint32_t col = c0 + cl + c;
            if (col >= V) continue;
            float lo, hi;
            asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(S[i / 2][c]));
            if (r < D) Sg[(size_t)r * V + col] = lo;
            if (r + 1 < D) Sg[(size_t)(r + 1) * V + col] = hi;
        }
    }
}

template <class A>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const float* o, const float* __restrict__ w, const float* gate, typename A::T* out, uint32_t n, uint32_t V, float eps) {
    pdl_release();
    pdl_wait();
    const uint32_t i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;      // (row, head)
    if (i >= n) return;
    const size_t off = (size_t)i * V;
    float ss = 0.0f;
    for (uint32_t c = lane; c < V; c += 32) { const float v = __ldcg(o + off + c); ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)V + eps);
    for (uint32_t c = lane; c < V; c += 32) A::st(out + off + c, __ldcg(o + off + c) * inv * __ldg(w + c) * sigmoid_f(__ldcg(gate + off + c)));
}

// A cluster of ceil(V / 32) CTAs per head, 32 value columns each: convolution of the head's q, k and its values, unit
// norms, decays and gates from the low-rank vectors, the recurrence, and the gated norm (sum of squares over the cluster).
// Thread (l = warp, c = lane) holds rows l * RPL .. + RPL - 1 of column c of S. What no earlier kernel of the run writes
// (S, the window, weights) is requested before the dependency wait. R: rows of the run, 1 or up to 4.
constexpr uint32_t STEP_ROWS = 4, STEP_COLS = 32;
inline uint32_t step_floats(const DeltaArgs& a, uint32_t dp, uint32_t r) { return r * (3 * dp + ((a.rank_a + 3) & ~3u) + ((a.rank_g + 3) & ~3u)) + 8 * STEP_COLS * 2; }

// elements k .. k + 3 of row `row` of w [.., n], zeros past n
__device__ __forceinline__ float4 low_rank4(const uint16_t* __restrict__ w, size_t row, uint32_t k, uint32_t n) {
    const uint16_t* p = w + row * n + k;
    if ((n & 3u) == 0) {
        if (k >= n) return make_float4(0.f, 0.f, 0.f, 0.f);
        const uint2 q = __ldg((const uint2*)p);
        return make_float4(bf2f((uint16_t)(q.x & 0xffffu)), bf2f((uint16_t)(q.x >> 16)), bf2f((uint16_t)(q.y & 0xffffu)), bf2f((uint16_t)(q.y >> 16)));
    }
    return make_float4(k < n ? bf2f(__ldg(p)) : 0.f, k + 1 < n ? bf2f(__ldg(p + 1)) : 0.f, k + 2 < n ? bf2f(__ldg(p + 2)) : 0.f, k + 3 < n ? bf2f(__ldg(p + 3)) : 0.f);
}

template <class A, int RPL, int R>
__global__ void __launch_bounds__(256, 1)
delta_step_kernel(const DeltaArgs a, uint32_t rows_arg) {
    constexpr uint32_t DP = 8 * RPL, NI = (2 * DP + STEP_COLS + 255) / 256;
    const uint32_t rows = R == 1 ? 1 : rows_arg;
    extern __shared__ __align__(16) float sm[];
    __shared__ float s_v[R][STEP_COLS], s_gate[R][STEP_COLS], s_o[R][STEP_COLS], s_n[R][4], s_ss[8][R];
    cooperative_groups::cluster_group cl = cooperative_groups::this_cluster();
    const uint32_t D = a.dim, V = a.vdim, H = a.heads, KH = a.kv_heads, C = a.channels(), ra4 = (a.rank_a + 3) & ~3u, rg4 = (a.rank_g + 3) & ~3u;
    float *s_k = sm, *s_q = s_k + R * DP, *s_g = s_q + R * DP;        // [R][DP], zero past D
    float *s_a1 = s_g + R * DP, *s_g1 = s_a1 + R * ra4;               // [R][rank rounded up to 4], zero past the rank
    float2* s_part = (float2*)(s_g1 + R * rg4);                       // [8][32]
    cluster_arrive();
    pdl_release();
    const uint32_t tid = threadIdx.x, c = tid & 31, l = tid >> 5, h = blockIdx.y, kh = h / (H / KH), c0 = blockIdx.x * STEP_COLS, col = c0 + c;
    const int keep = (int)a.taps - 1;
    const bool four_taps = a.taps == 4;
    const uint32_t par = *(volatile const uint32_t*)a.conv_count & 1u;      // moves at the end of a run only
    const float* bank = a.conv_state + (size_t)par * keep * C;
    float* next = a.conv_state + (size_t)(par ^ 1u) * keep * C;
    // ---- before the wait
    float* Sg = a.S + (size_t)h * D * V;
    float S[RPL];
#pragma unroll
    for (int i = 0; i < RPL; i++) {
        const uint32_t r = l * RPL + i;
        S[i] = (r < D && col < V) ? __ldcg(Sg + (size_t)r * V + col) : 0.0f;
    }
    // channel of convolution item tid + 256 i: q [DP], k [DP], values [32]; C = none
    uint32_t ch[NI];
    float4 cw[NI];
    float win[NI][3];
#pragma unroll
    for (int i = 0; i < (int)NI; i++) {
        const uint32_t it = tid + 256 * i;
        ch[i] = it < DP ? (it < D ? kh * D + it : C)
              : it < 2 * DP ? (it - DP < D ? (KH + kh) * D + it - DP : C)
              : it < 2 * DP + STEP_COLS && c0 + it - 2 * DP < V ? 2 * KH * D + h * V + c0 + it - 2 * DP : C;
        if (four_taps && ch[i] < C) {
            cw[i] = __ldg((const float4*)a.conv_w + ch[i]);
#pragma unroll
            for (int j = 0; j < 3; j++) win[i][j] = __ldcg(bank + (size_t)j * C + ch[i]);
        }
    }
    constexpr int PRE = RPL < 16 ? RPL : 16;
    float4 wa[PRE], wg[STEP_COLS / 8];
#pragma unroll
    for (int i = 0; i < PRE; i++) wa[i] = l + 8 * i < D ? low_rank4(a.a2, h * D + l + 8 * i, c * 4, a.rank_a) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < (int)STEP_COLS / 8; j++)
        wg[j] = c0 + l + 8 * j < V ? low_rank4(a.g2, h * V + c0 + l + 8 * j, c * 4, a.rank_g) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float ea = expf(__ldg(a.a_log + h)), dtb = tid < D ? __ldg(a.dt_bias + h * D + tid) : 0.0f, nw = col < V ? __ldg(a.norm_w + col) : 0.0f;
    pdl_wait();
    // ---- the joined projection's rows
    const typename A::T* y = (const typename A::T*)a.y;
    const bool qk_keeper = blockIdx.x == 0 && h % (H / KH) == 0;      // one CTA per key head writes the window of q and k
#pragma unroll
    for (int i = 0; i < (int)NI; i++) {
        const uint32_t it = tid + 256 * i;
        if (it >= 2 * DP + STEP_COLS) break;
        float* out = it < DP ? s_q + it : it < 2 * DP ? s_k + it - DP : &s_v[0][it - 2 * DP];
        const uint32_t stride = it < 2 * DP ? DP : STEP_COLS;
        if (ch[i] >= C) {
            for (uint32_t r = 0; r < rows; r++) out[r * stride] = 0.0f;
            continue;
        }
        const bool keeper = it >= 2 * DP || qk_keeper;
        if (four_taps) {
            float x0 = win[i][0], x1 = win[i][1], x2 = win[i][2];
#pragma unroll
            for (int r = 0; r < R; r++) {
                if (R > 1 && r >= (int)rows) break;
                const float x3 = A::ld(y + (size_t)r * a.ys + ch[i]);
                out[r * stride] = silu_f(fmaf(cw[i].w, x3, fmaf(cw[i].z, x2, fmaf(cw[i].y, x1, cw[i].x * x0))));
                x0 = x1; x1 = x2; x2 = x3;
            }
            if (keeper) { next[ch[i]] = x0; next[(size_t)C + ch[i]] = x1; next[2 * (size_t)C + ch[i]] = x2; }
        } else {
            for (uint32_t r = 0; r < rows; r++) {
                float s = 0.0f;
                for (int j = 0; j < (int)a.taps; j++)
                    s = fmaf(__ldg(a.conv_w + (size_t)ch[i] * a.taps + j), conv_in<A>(y, bank, (int)r - keep + j, ch[i], a.ys, C, keep), s);
                out[r * stride] = silu_f(s);
            }
            if (keeper)
                for (int j = 0; j < keep; j++) next[(size_t)j * C + ch[i]] = conv_in<A>(y, bank, (int)rows - keep + j, ch[i], a.ys, C, keep);
        }
    }
    for (uint32_t i = tid; i < rows * (ra4 + rg4); i += 256) {
        const uint32_t r = i / (ra4 + rg4), k = i % (ra4 + rg4);
        const typename A::T* yr = y + (size_t)r * a.ys;
        if (k < ra4) s_a1[r * ra4 + k] = k < a.rank_a ? A::ld(yr + a.a_col + k) : 0.0f;
        else s_g1[r * rg4 + k - ra4] = k - ra4 < a.rank_g ? A::ld(yr + a.g_col + k - ra4) : 0.0f;
    }
    const float blog = l < rows ? A::ld(y + (size_t)l * a.ys + a.b_col + h) : 0.0f;
    __syncthreads();
    // ---- norms (warp r: row r), decays and gates (a warp per output)
    if (l < rows) {
        float qq = 0.0f, kk = 0.0f, qk = 0.0f;
        for (uint32_t i = c; i < D; i += 32) {
            const float qv = s_q[l * DP + i], kv = s_k[l * DP + i];
            qq = fmaf(qv, qv, qq); kk = fmaf(kv, kv, kk); qk = fmaf(qv, kv, qk);
        }
        qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
        if (c == 0) {
            const float iq = 1.0f / sqrtf((float)D) / sqrtf(qq + 1e-6f), ik = 1.0f / sqrtf(kk + 1e-6f);
            s_n[l][0] = iq; s_n[l][1] = ik; s_n[l][2] = qk * iq * ik; s_n[l][3] = sigmoid_f(blog);
        }
    }
    auto dot4 = [&](float4 w, const float* x, uint32_t k, uint32_t n4) -> float {
        if (k >= n4) return 0.0f;
        const float4 v = *(const float4*)(x + k);
        return fmaf(w.w, v.w, fmaf(w.z, v.z, fmaf(w.y, v.y, w.x * v.x)));
    };
#pragma unroll
    for (int r = 0; r < R; r++) {
        if (R > 1 && r >= (int)rows) break;
        float da[RPL], dg[STEP_COLS / 8];
#pragma unroll
        for (int i = 0; i < RPL; i++) {
            const uint32_t d = l + 8 * i;
            da[i] = 0.0f;
            if (d >= D) continue;
            da[i] = dot4(i < PRE ? wa[i < PRE ? i : 0] : low_rank4(a.a2, h * D + d, c * 4, a.rank_a), s_a1 + r * ra4, c * 4, ra4);
            for (uint32_t k = 128 + c * 4; k < ra4; k += 128) da[i] += dot4(low_rank4(a.a2, h * D + d, k, a.rank_a), s_a1 + r * ra4, k, ra4);
        }
#pragma unroll
        for (int j = 0; j < (int)STEP_COLS / 8; j++) {
            const uint32_t v = c0 + l + 8 * j;
            dg[j] = 0.0f;
            if (v >= V) continue;
            dg[j] = dot4(wg[j], s_g1 + r * rg4, c * 4, rg4);
            for (uint32_t k = 128 + c * 4; k < rg4; k += 128) dg[j] += dot4(low_rank4(a.g2, h * V + v, k, a.rank_g), s_g1 + r * rg4, k, rg4);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
            for (int i = 0; i < RPL; i++) da[i] += __shfl_xor_sync(0xffffffffu, da[i], o);
#pragma unroll
            for (int j = 0; j < (int)STEP_COLS / 8; j++) dg[j] += __shfl_xor_sync(0xffffffffu, dg[j], o);
        }
#pragma unroll
        for (int i = 0; i < RPL; i++) if (c == (i & 31)) s_g[r * DP + l + 8 * i] = da[i];
#pragma unroll
        for (int j = 0; j < (int)STEP_COLS / 8; j++) if (c == j) s_gate[r][l + 8 * j] = dg[j];
    }
    __syncthreads();
    for (uint32_t r = 0; r < rows; r++)
        if (tid < DP) {
            const uint32_t i = r * DP + tid;
            s_g[i] = tid < D ? expf(-ea * softplus_f(s_g[i] + dtb)) : 0.0f;
            s_q[i] *= s_n[r][0];
            s_k[i] *= s_n[r][1];
        }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < R; r++) {
        if (R > 1 && r >= (int)rows) break;
        float ak = 0.0f, aq = 0.0f, kreg[RPL];
#pragma unroll
        for (int i = 0; i < RPL; i += 4) {
            const float4 g4 = *(const float4*)(s_g + r * DP + l * RPL + i), k4 = *(const float4*)(s_k + r * DP + l * RPL + i), q4 = *(const float4*)(s_q + r * DP + l * RPL + i);
            kreg[i] = k4.x; kreg[i + 1] = k4.y; kreg[i + 2] = k4.z; kreg[i + 3] = k4.w;
            S[i] *= g4.x; S[i + 1] *= g4.y; S[i + 2] *= g4.z; S[i + 3] *= g4.w;
            ak = fmaf(S[i], k4.x, ak); ak = fmaf(S[i + 1], k4.y, ak); ak = fmaf(S[i + 2], k4.z, ak); ak = fmaf(S[i + 3], k4.w, ak);
            aq = fmaf(S[i], q4.x, aq); aq = fmaf(S[i + 1], q4.y, aq); aq = fmaf(S[i + 2], q4.z, aq); aq = fmaf(S[i + 3], q4.w, aq);
        }
        s_part[l * 32 + c] = make_float2(ak, aq);
        __syncthreads();
        ak = aq = 0.0f;
#pragma unroll
        for (int w = 0; w < 8; w++) { const float2 p = s_part[w * 32 + c]; ak += p.x; aq += p.y; }
        const float u = s_n[r][3] * (s_v[r][c] - ak);
#pragma unroll
        for (int i = 0; i < RPL; i++) S[i] = fmaf(kreg[i], u, S[i]);
        if (l == 0) s_o[r][c] = fmaf(u, s_n[r][2], aq);
        __syncthreads();
    }
    cluster_wait();                                   // every CTA of the cluster has started
    if (l < rows) {
        const float o = col < V ? s_o[l][c] : 0.0f, ss = warp_sum(o * o);
        if (c < gridDim.x) *cl.map_shared_rank(&s_ss[blockIdx.x][l], c) = ss;
    }
    cluster_arrive();
#pragma unroll
    for (int i = 0; i < RPL; i++) {
        const uint32_t r = l * RPL + i;
        if (r < D && col < V) Sg[(size_t)r * V + col] = S[i];
    }
    cluster_wait();
    if (l < rows && col < V) {
        float ss = 0.0f;
        for (uint32_t k = 0; k < gridDim.x; k++) ss += s_ss[k][l];
        const float inv = 1.0f / sqrtf(ss / (float)V + a.eps);
        A::st((typename A::T*)a.out + ((size_t)l * H + h) * V + col, s_o[l][c] * inv * nw * sigmoid_f(s_gate[l][c]));
    }
}

template <class A, int RPL, int R>
bool launch_step_r(cudaStream_t st, const DeltaArgs& a, uint32_t rows) {
    static int have[64] = {};
    const uint32_t vs = (a.vdim + STEP_COLS - 1) / STEP_COLS;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(vs, a.heads); cfg.blockDim = dim3(256); cfg.dynamicSmemBytes = (size_t)step_floats(a, 8 * RPL, R) * 4; cfg.stream = st;
    if (cfg.dynamicSmemBytes > 100 * 1024 || !ensure_dyn_smem(delta_step_kernel<A, RPL, R>, cfg.dynamicSmemBytes, have)) return false;
    if (launch_pdl_cluster(delta_step_kernel<A, RPL, R>, cfg, dim3(vs, 1, 1), a, rows) != cudaSuccess) { cudaGetLastError(); return false; }
    g_launches++;
    return true;
}
template <class A, int RPL>
bool launch_step(cudaStream_t st, const DeltaArgs& a, uint32_t rows) {
    return rows == 1 ? launch_step_r<A, RPL, 1>(st, a, rows) : launch_step_r<A, RPL, (int)STEP_ROWS>(st, a, rows);
}

template <class A>
void launch_prep(cudaStream_t st, const DeltaArgs& a, const DeltaWork& w, uint32_t rows) {
    const dim3 grid((a.heads + 7) / 8, (rows + 1) / 2);
    if (a.dim <= 64) launch_pdl(delta_prep_kernel<A, 2>, grid, dim3(256), 0, st, a, w, rows);
    else if (a.dim <= 128) launch_pdl(delta_prep_kernel<A, 4>, grid, dim3(256), 0, st, a, w, rows);
    else launch_pdl(delta_prep_kernel<A, 16>, grid, dim3(256), 0, st, a, w, rows);
    g_launches++;
}

// Ordinary launch: CTAs that come up while the kernel before still holds SMs pile up on the ones it has left, and the
// recurrence then runs at the pace of the fullest SM.
template <int RPL, int NW, bool VEC>
void launch_scan_t(cudaStream_t st, const DeltaArgs& a, const DeltaWork& w, uint32_t rows) {
    const size_t smem = (size_t)2 * TC * (3 * 16 * RPL + NW * 4 + 4) * 4;
    static int have[64] = {};
    ensure_dyn_smem(delta_scan_kernel<RPL, NW, VEC>, smem, have);
    delta_scan_kernel<RPL, NW, VEC><<<dim3((a.vdim + NW * 4 - 1) / (NW * 4), a.heads), NW * 32, smem, st>>>(a, w, rows);
    g_launches++;
}
template <int RPL>
void launch_scan(cudaStream_t st, const DeltaArgs& a, const DeltaWork& w, uint32_t rows) {
    if (a.dim % 4) { launch_scan_t<RPL, 8, false>(st, a, w, rows); return; }
    // narrower CTAs while those of 8 warps would leave half of the SMs without one
    if ((a.vdim + 31) / 32 * a.heads <= 74) launch_scan_t<RPL, 4, true>(st, a, w, rows);
    else launch_scan_t<RPL, 8, true>(st, a, w, rows);
}

}  // namespace

void k_short_conv(cudaStream_t st, const DeltaArgs& a, uint32_t rows) {
    if (!rows) return;
    const uint32_t C = a.channels();
    const dim3 grid((C + 255) / 256, (rows + CONV_ROWS - 1) / CONV_ROWS);
    if (a.bf16) launch_pdl(short_conv_kernel<ActBf16>, grid, dim3(256), 0, st, (const uint16_t*)a.y, a.conv_w, a.conv_state, a.conv_count, a.qkv, rows, C, a.taps, a.ys);
    else launch_pdl(short_conv_kernel<ActF32>, grid, dim3(256), 0, st, (const float*)a.y, a.conv_w, a.conv_state, a.conv_count, a.qkv, rows, C, a.taps, a.ys);
    g_launches++;
}

size_t delta_work_floats(const DeltaArgs& a, uint32_t rows) {
    return 2 * up4((size_t)rows * a.kv_heads * a.dim) + up4((size_t)rows * a.heads * a.dim) + (size_t)rows * a.heads * 4;
}

void k_channel_delta(cudaStream_t st, const DeltaArgs& a, uint32_t rows) {
    if (!rows) return;
    const DeltaWork w = work_of(a, rows);
    if (a.bf16) launch_prep<ActBf16>(st, a, w, rows);
    else launch_prep<ActF32>(st, a, w, rows);
    if (a.dim <= 64) launch_scan<4>(st, a, w, rows);
    else if (a.dim <= 128) launch_scan<8>(st, a, w, rows);
    else if (a.dim <= 256) launch_scan<16>(st, a, w, rows);
    else launch_scan<32>(st, a, w, rows);
}

bool k_delta_step(cudaStream_t st, const DeltaArgs& a, uint32_t rows) {
    if (!rows || rows > STEP_ROWS || a.dim > 256 || a.vdim > 8 * STEP_COLS) return false;
    if (a.bf16) return a.dim <= 64 ? launch_step<ActBf16, 8>(st, a, rows) : a.dim <= 128 ? launch_step<ActBf16, 16>(st, a, rows) : launch_step<ActBf16, 32>(st, a, rows);
    return a.dim <= 64 ? launch_step<ActF32, 8>(st, a, rows) : a.dim <= 128 ? launch_step<ActF32, 16>(st, a, rows) : launch_step<ActF32, 32>(st, a, rows);
}

void k_gated_norm(cudaStream_t st, const DeltaArgs& a, uint32_t rows) {
    const uint32_t n = rows * a.heads;
    if (!n) return;
    if (a.bf16) launch_pdl(gated_norm_kernel<ActBf16>, dim3((n + 7) / 8), dim3(256), 0, st, (const float*)a.o, a.norm_w, a.gate, (uint16_t*)a.out, n, a.vdim, a.eps);
    else launch_pdl(gated_norm_kernel<ActF32>, dim3((n + 7) / 8), dim3(256), 0, st, (const float*)a.o, a.norm_w, a.gate, (float*)a.out, n, a.vdim, a.eps);
    g_launches++;
}

}  // namespace gehtp
