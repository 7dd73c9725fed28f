// Gated delta rule with one decay per head and key channel (OP_SHORT_CONV, OP_CHANNEL_DELTA, OP_GATED_NORM).
//
//   short_conv_kernel    causal depthwise convolution + silu; the last taps - 1 inputs are kept in the state, two banks:
//                        a run reads the bank of its parity and writes the other, so that no CTA overwrites what
//                        another still reads
//   delta_prep_kernel    unit vectors, decays, step sizes, k . q per token, fp32
//   delta_scan_kernel    the recurrence, token by token: a column of S lives in the registers of 8 (16, 32) lanes, both
//                        reductions of a token (S^T k and S^T q) run side by side; with S' = g S,
//                        u = beta (v - S'^T k), S = S' + k u^T:  S^T q = S'^T q + u (k . q)
//   gated_norm_kernel    RMS norm of a head's read-out, weight, sigmoid gate
//
// The recurrence is the same arithmetic for one token and for a whole prompt, so a cut of the prompt changes nothing.
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

// work: k [rows][KH][D], q [rows][KH][D], decay [rows][H][D], {step, k . q} [rows][H][2]
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

template <class A>
__global__ void __launch_bounds__(256)
delta_prep_kernel(const DeltaArgs a, const DeltaWork wk) {
    extern __shared__ float s_kq[];                   // [kv_heads]
    pdl_release();
    pdl_wait();
    const uint32_t r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, D = a.dim, KH = a.kv_heads, H = a.heads;
    const float* x = a.qkv + (size_t)r * a.channels();
    const float qs = 1.0f / sqrtf((float)D);
    for (uint32_t h = warp; h < KH; h += 8) {
        const float *qx = x + h * D, *kx = x + (KH + h) * D;
        float qq = 0.0f, kk = 0.0f, qk = 0.0f;
        for (uint32_t i = lane; i < D; i += 32) {
            const float qv = __ldcg(qx + i), kv = __ldcg(kx + i);
            qq = fmaf(qv, qv, qq); kk = fmaf(kv, kv, kk); qk = fmaf(qv, kv, qk);
        }
        qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
        const float iq = qs / sqrtf(qq + 1e-6f), ik = 1.0f / sqrtf(kk + 1e-6f);
        for (uint32_t i = lane; i < D; i += 32) {
            wk.q[((size_t)r * KH + h) * D + i] = __ldcg(qx + i) * iq;
            wk.k[((size_t)r * KH + h) * D + i] = __ldcg(kx + i) * ik;
        }
        if (lane == 0) s_kq[h] = qk * iq * ik;
    }
    for (uint32_t i = threadIdx.x; i < H * D; i += 256) {
        const float z = softplus_f(__ldcg(a.a + (size_t)r * H * D + i) + __ldg(a.dt_bias + i));
        wk.g[(size_t)r * H * D + i] = expf(-expf(__ldg(a.a_log + i / D)) * z);
    }
    __syncthreads();
    const typename A::T* b = (const typename A::T*)a.y + (size_t)r * a.ys + a.b_col;
    for (uint32_t h = threadIdx.x; h < H; h += 256) {
        float* d = wk.bk + ((size_t)r * H + h) * 2;
        d[0] = sigmoid_f(A::ld(b + h));
        d[1] = s_kq[h / (H / KH)];
    }
}

// LPC lanes hold a column of S, RPL rows each; a warp holds 32 / LPC columns, a CTA 8 warps of one head. Tokens come in
// chunks of TC through shared memory (cp.async, two stages; VEC = 16-byte copies).
constexpr uint32_t TC = 16;
template <int LPC, int RPL, bool VEC>
__global__ void __launch_bounds__(256)
delta_scan_kernel(const DeltaArgs a, const DeltaWork wk, uint32_t rows) {
    constexpr uint32_t DP = LPC * RPL, CPW = 32 / LPC, NC = 8 * CPW;
    extern __shared__ __align__(16) float sm[];
    float* s_kqg = sm;                                // [2][TC][3][DP]
    float* s_v = s_kqg + 2 * TC * 3 * DP;             // [2][TC][NC]
    float* s_bk = s_v + 2 * TC * NC;                  // [2][TC][2]
    pdl_release();
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, H = a.heads, D = a.dim, V = a.vdim;
    const uint32_t h = blockIdx.y, kh = h / (H / a.kv_heads), c0 = blockIdx.x * NC;
    const uint32_t l = lane % LPC, col = c0 + warp * CPW + lane / LPC;
    const uint32_t C = a.channels(), voff = 2 * a.kv_heads * D + h * V;
    for (uint32_t i = tid; i < 2 * TC * 3 * DP; i += 256)
        if (i % DP >= D) s_kqg[i] = 0.0f;             // rows past D: S stays zero there
    pdl_wait();
    float* Sg = a.S + (size_t)h * D * V;
    auto row_of = [&](int i) -> uint32_t { return (i / 4) * 4 * LPC + l * 4 + (i & 3); };
    float S[RPL];
#pragma unroll
    for (int i = 0; i < RPL; i++) {
        const uint32_t r = row_of(i);
        S[i] = (r < D && col < V) ? Sg[(size_t)r * V + col] : 0.0f;
    }
    auto fetch = [&](uint32_t t0, uint32_t stg) {
        const uint32_t nt = t0 < rows ? min(TC, rows - t0) : 0;
        float* d = s_kqg + stg * TC * 3 * DP;
        if (VEC) {
            const uint32_t ch = D / 4;
            for (uint32_t i = tid; i < nt * 3 * ch; i += 256) {
                const uint32_t t = i / (3 * ch), w = (i / ch) % 3, c = (i % ch) * 4;
                const float* src = w == 2 ? wk.g + ((size_t)(t0 + t) * H + h) * D + c
                                          : (w ? wk.q : wk.k) + ((size_t)(t0 + t) * a.kv_heads + kh) * D + c;
                cp16(smem_addr(d + (t * 3 + w) * DP + c), src, 16);
            }
        } else {
            for (uint32_t i = tid; i < nt * 3 * D; i += 256) {
                const uint32_t t = i / (3 * D), w = (i / D) % 3, c = i % D;
                d[(t * 3 + w) * DP + c] = __ldcg((w == 2 ? wk.g + ((size_t)(t0 + t) * H + h) * D
                                                         : (w ? wk.q : wk.k) + ((size_t)(t0 + t) * a.kv_heads + kh) * D) + c);
            }
        }
        for (uint32_t i = tid; i < nt * NC; i += 256) {
            const uint32_t t = i / NC, c = i % NC;
            const float* src = a.qkv + (size_t)(t0 + t) * C + voff + c0 + c;
            float* dst = s_v + (stg * TC + t) * NC + c;
            if (c0 + c < V) asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
        }
        for (uint32_t i = tid; i < nt * 2; i += 256)
            asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_addr(s_bk + stg * TC * 2 + i)),
                         "l"(wk.bk + ((size_t)(t0 + i / 2) * H + h) * 2 + (i & 1)) : "memory");
        cp_commit();
    };
    fetch(0, 0);
    for (uint32_t t0 = 0, stg = 0; t0 < rows; t0 += TC, stg ^= 1) {
        fetch(t0 + TC, stg ^ 1);
        cp_wait<1>();
        __syncthreads();
        const uint32_t nt = min(TC, rows - t0);
        const float* kqg = s_kqg + stg * TC * 3 * DP + l * 4;
#pragma unroll 2
        for (uint32_t t = 0; t < nt; t++) {
            const float* p = kqg + t * 3 * DP;
            float k[RPL], sk[4] = {0.f, 0.f, 0.f, 0.f}, sq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < RPL; i += 4) {
                const float4 k4 = *(const float4*)(p + i * LPC), q4 = *(const float4*)(p + DP + i * LPC), g4 = *(const float4*)(p + 2 * DP + i * LPC);
                k[i] = k4.x; k[i + 1] = k4.y; k[i + 2] = k4.z; k[i + 3] = k4.w;
                S[i] *= g4.x; S[i + 1] *= g4.y; S[i + 2] *= g4.z; S[i + 3] *= g4.w;
                sk[0] = fmaf(S[i], k4.x, sk[0]); sk[1] = fmaf(S[i + 1], k4.y, sk[1]); sk[2] = fmaf(S[i + 2], k4.z, sk[2]); sk[3] = fmaf(S[i + 3], k4.w, sk[3]);
                sq[0] = fmaf(S[i], q4.x, sq[0]); sq[1] = fmaf(S[i + 1], q4.y, sq[1]); sq[2] = fmaf(S[i + 2], q4.z, sq[2]); sq[3] = fmaf(S[i + 3], q4.w, sq[3]);
            }
            float ak = (sk[0] + sk[1]) + (sk[2] + sk[3]), aq = (sq[0] + sq[1]) + (sq[2] + sq[3]);
#pragma unroll
            for (int o = 1; o < LPC; o <<= 1) {
                ak += __shfl_xor_sync(0xffffffffu, ak, o);
                aq += __shfl_xor_sync(0xffffffffu, aq, o);
            }
            const float2 bk = *(const float2*)(s_bk + (stg * TC + t) * 2);
            const float u = bk.x * (s_v[(stg * TC + t) * NC + warp * CPW + lane / LPC] - ak);
            if (l == 0 && col < V) a.o[((size_t)(t0 + t) * H + h) * V + col] = fmaf(u, bk.y, aq);
#pragma unroll
            for (int i = 0; i < RPL; i++) S[i] = fmaf(k[i], u, S[i]);
        }
        __syncthreads();
    }
    cp_wait<0>();
#pragma unroll
    for (int i = 0; i < RPL; i++) {
        const uint32_t r = row_of(i);
        if (r < D && col < V) Sg[(size_t)r * V + col] = S[i];
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

template <int LPC, int RPL>
void launch_scan(cudaStream_t st, const DeltaArgs& a, const DeltaWork& w, uint32_t rows) {
    constexpr uint32_t DP = LPC * RPL, NC = 8 * (32 / LPC);
    const size_t smem = (size_t)2 * TC * (3 * DP + NC + 2) * 4;
    const dim3 grid((a.vdim + NC - 1) / NC, a.heads);
    static int have_v[64] = {}, have_s[64] = {};
    if (a.dim % 4 == 0) {
        ensure_dyn_smem(delta_scan_kernel<LPC, RPL, true>, smem, have_v);
        launch_pdl(delta_scan_kernel<LPC, RPL, true>, grid, dim3(256), smem, st, a, w, rows);
    } else {
        ensure_dyn_smem(delta_scan_kernel<LPC, RPL, false>, smem, have_s);
        launch_pdl(delta_scan_kernel<LPC, RPL, false>, grid, dim3(256), smem, st, a, w, rows);
    }
    g_launches++;
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
    return 2 * up4((size_t)rows * a.kv_heads * a.dim) + up4((size_t)rows * a.heads * a.dim) + up4((size_t)rows * a.heads * 2);
}

void k_channel_delta(cudaStream_t st, const DeltaArgs& a, uint32_t rows) {
    if (!rows) return;
    const DeltaWork w = work_of(a, rows);
    if (a.bf16) launch_pdl(delta_prep_kernel<ActBf16>, dim3(rows), dim3(256), (size_t)a.kv_heads * 4, st, a, w);
    else launch_pdl(delta_prep_kernel<ActF32>, dim3(rows), dim3(256), (size_t)a.kv_heads * 4, st, a, w);
    g_launches++;
    if (a.dim <= 32) launch_scan<8, 4>(st, a, w, rows);
    else if (a.dim <= 64) launch_scan<8, 8>(st, a, w, rows);
    else if (a.dim <= 128) launch_scan<8, 16>(st, a, w, rows);
    else if (a.dim <= 256) launch_scan<16, 16>(st, a, w, rows);
    else launch_scan<32, 16>(st, a, w, rows);
}

void k_gated_norm(cudaStream_t st, const DeltaArgs& a, uint32_t rows) {
    const uint32_t n = rows * a.heads;
    if (!n) return;
    if (a.bf16) launch_pdl(gated_norm_kernel<ActBf16>, dim3((n + 7) / 8), dim3(256), 0, st, (const float*)a.o, a.norm_w, a.gate, (uint16_t*)a.out, n, a.vdim, a.eps);
    else launch_pdl(gated_norm_kernel<ActF32>, dim3((n + 7) / 8), dim3(256), 0, st, (const float*)a.o, a.norm_w, a.gate, (float*)a.out, n, a.vdim, a.eps);
    g_launches++;
}

}  // namespace gehtp
