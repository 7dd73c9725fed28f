// Projections of the row-count runlists: y[M, N] = act(x[M, K] . w^T) with w bf16 [N, K], fp32 accumulation.
//
//   bf16 x, few rows    streaming product on mma.sync m16n8k16 (lin_stream_kernel): a warp owns 8 output columns and a
//                       share of K, the shares of a column group meet in shared memory
//   bf16 x, more rows   the TMA-fed tcgen05 GEMM (f16_gemm_sm100.cu)
//   fp32 x, shapes whose rows are no multiple of 16 bytes, and the one-kernel-per-op plan: fp32 FMA tiles
#include <type_traits>
#include "launchers_rows.h"
#include "linear_epi.cuh"
#include "mma_bf16.cuh"

namespace gehtp {

namespace {

constexpr int TM = 64, TN = 64, TK = 16;

// fp32 FMA tiles, k ascending per output element; any shape and stride
template <class X, class E>
__global__ void __launch_bounds__(256)
lin_fma_kernel(const typename X::T* x, const uint16_t* __restrict__ w, const E epi, uint32_t M, uint32_t K, uint32_t N, uint32_t xs) {
    __shared__ float As[TK][TM + 4];
    __shared__ float Ws[TK][TN + 4];
    pdl_release();
    pdl_wait();
    const uint32_t m0 = blockIdx.y * TM, c0 = blockIdx.x * TN;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < K; k0 += TK) {
        for (int e = threadIdx.x; e < TM * TK; e += 256) {
            const int k = e % TK, m = e / TK;
            As[k][m] = (m0 + m < M && k0 + k < K) ? X::ld(x + (size_t)(m0 + m) * xs + k0 + k) : 0.0f;
        }
        for (int e = threadIdx.x; e < TN * TK; e += 256) {
            const int k = e % TK, n = e / TK;
            Ws[k][n] = (c0 + n < N && k0 + k < K) ? bf2f(__ldg(w + (size_t)(c0 + n) * K + k0 + k)) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < TK; k++) {
            const float4 a4 = *(const float4*)&As[k][ty * 4], w4 = *(const float4*)&Ws[k][tx * 4];
            const float av[4] = {a4.x, a4.y, a4.z, a4.w}, wv[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const uint32_t m = m0 + ty * 4 + i;
        if (m < M && c0 + tx * 4 < N) epi.quad(m, c0 + tx * 4, acc[i], N);
    }
}

// fp32 FMA, up to 4 rows per pass: a warp per pair of output columns, lanes along K
template <class X, class E>
__global__ void __launch_bounds__(256)
lin_fma_rows_kernel(const typename X::T* x, const uint16_t* __restrict__ w, const E epi, uint32_t M, uint32_t K, uint32_t N, uint32_t xs) {
    pdl_release();
    pdl_wait();
    const uint32_t n = (blockIdx.x * 8 + (threadIdx.x >> 5)) * 2, lane = threadIdx.x & 31, m0 = blockIdx.y * 4;
    if (n >= N) return;
    const uint16_t *w0 = w + (size_t)n * K, *w1 = w + (size_t)min(n + 1, N - 1) * K;
    float acc[4][2] = {};
    for (uint32_t k = lane; k < K; k += 32) {
        const float a = bf2f(__ldg(w0 + k)), b = bf2f(__ldg(w1 + k));
#pragma unroll
        for (int r = 0; r < 4; r++)
            if (m0 + r < M) {
                const float v = X::ld(x + (size_t)(m0 + r) * xs + k);
                acc[r][0] = fmaf(v, a, acc[r][0]);
                acc[r][1] = fmaf(v, b, acc[r][1]);
            }
    }
#pragma unroll
    for (int r = 0; r < 4; r++) {
        const float s0 = warp_sum(acc[r][0]), s1 = warp_sum(acc[r][1]);
        if (lane == 0 && m0 + r < M) epi.pair(m0 + r, n, s0, s1, N);
    }
}

// Few bf16 rows. A CTA of 8 warps owns 8 * (8 / KS) output columns: KS warps share a group of 8 columns and split K in
// chunks of 32. Lane (g, t) loads 16 bytes of weight row n0 + g and the 16 bytes at the same k of activation row g;
// the two halves feed two MMAs (which k slot a value takes does not matter as long as both operands agree). The first
// batch of weights is requested before the dependency wait. Activation rows are staged in shared memory.
template <int KS, int UNR, class E>
__global__ void __launch_bounds__(256)
lin_stream_kernel(const uint16_t* x, const uint16_t* __restrict__ w, const E epi, uint32_t M, uint32_t K, uint32_t N, uint32_t xs) {
    extern __shared__ __align__(16) unsigned char smem_a[];      // [rows of this CTA][RS] bytes
    __shared__ float part[8][64];
    pdl_release();
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const uint32_t ks = warp % KS, cg = warp / KS;
    const uint32_t m0 = blockIdx.y * 8, rows = min(8u, M - m0), n0 = (blockIdx.x * (8 / KS) + cg) * 8;
    const uint32_t KC = (K + 31) / 32, RS = KC * 64 + 64;          // rows 16 banks apart, zero-filled past K
    const bool active = n0 < N;
    const uint16_t* wr = w + (size_t)min(n0 + g, N - 1) * K + t * 8;
    auto load = [&](uint32_t kc) -> uint4 {
        const uint32_t k = kc * 32;
        return (active && kc < KC && k + t * 8 < K) ? __ldcs((const uint4*)(wr + k)) : make_uint4(0, 0, 0, 0);
    };
    uint4 wq[UNR];
#pragma unroll
    for (int u = 0; u < UNR; u++) wq[u] = load(ks + u * KS);
    pdl_wait();
    for (uint32_t i = threadIdx.x; i < rows * KC * 4; i += 256) {
        const uint32_t r = i / (KC * 4), c = i % (KC * 4);
        *(uint4*)(smem_a + r * RS + c * 16) = c * 8 < K ? __ldcg((const uint4*)(x + (size_t)(m0 + r) * xs + c * 8)) : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    const unsigned char* arow = smem_a + min(g, rows - 1) * RS + t * 16;       // rows past the last repeat it; never stored
    for (uint32_t kc0 = ks; kc0 < KC; kc0 += UNR * KS) {
        uint4 nx[UNR];
#pragma unroll
        for (int u = 0; u < UNR; u++) nx[u] = load(kc0 + (UNR + u) * KS);
#pragma unroll
        for (int u = 0; u < UNR; u++) {
            const uint32_t kc = kc0 + u * KS;
            if (kc >= KC) break;
            const uint4 av = *(const uint4*)(arow + kc * 64);
            const uint32_t a1[4] = {av.x, 0u, av.y, 0u}, a2[4] = {av.z, 0u, av.w, 0u};
            mma_bf16(acc, a1, wq[u].x, wq[u].y);
            mma_bf16(acc, a2, wq[u].z, wq[u].w);
        }
#pragma unroll
        for (int u = 0; u < UNR; u++) wq[u] = nx[u];
    }
    if (KS > 1) {
        part[warp][g * 8 + 2 * t] = acc[0];
        part[warp][g * 8 + 2 * t + 1] = acc[1];
        __syncthreads();
        if (ks != 0) return;
#pragma unroll
        for (int s = 1; s < KS; s++) { acc[0] += part[warp + s][g * 8 + 2 * t]; acc[1] += part[warp + s][g * 8 + 2 * t + 1]; }
    }
    const uint32_t n = n0 + 2 * t;
    if (g < rows && n < N) epi.pair(m0 + g, n, acc[0], acc[1], N);
}

template <int KS, class E>
bool launch_stream(cudaStream_t st, const LinearArgs& a, const E& epi, uint32_t M) {
    const uint32_t KC = (a.K + 31) / 32;
    const size_t smem = (size_t)(M < 8 ? M : 8) * (KC * 64 + 64);
    if (smem > 200 * 1024) return false;
    const dim3 grid((a.N + 8 * (8 / KS) - 1) / (8 * (8 / KS)), (M + 7) / 8);
    static int have[64] = {};
    if (smem > 40 * 1024 && !ensure_dyn_smem(lin_stream_kernel<KS, 8, E>, smem, have)) return false;
    if (launch_pdl(lin_stream_kernel<KS, 8, E>, grid, dim3(256), smem, st, (const uint16_t*)a.x, a.w, epi, M, a.K, a.N, a.xs) != cudaSuccess) {
        cudaGetLastError();
        return false;
    }
    g_launches++;
    return true;
}

// K shares per column group: enough CTAs for two per SM, a share of at least one batch of chunks
template <class E>
bool launch_stream_any(cudaStream_t st, const LinearArgs& a, const E& epi, uint32_t M) {
    const uint32_t KC = (a.K + 31) / 32, groups = (a.N + 7) / 8;
    if (groups >= 8 * 296 || KC < 16) return launch_stream<1>(st, a, epi, M);
    if (groups >= 4 * 296 || KC < 32) return launch_stream<2>(st, a, epi, M);
    if (groups >= 2 * 296 || KC < 64) return launch_stream<4>(st, a, epi, M);
    return launch_stream<8>(st, a, epi, M);
}

template <class X, class E>
void launch_fma(cudaStream_t st, const LinearArgs& a, const E& epi, uint32_t M) {
    const typename X::T* x = (const typename X::T*)a.x;
    if (M <= 16) launch_pdl(lin_fma_rows_kernel<X, E>, dim3((a.N + 15) / 16, (M + 3) / 4), dim3(256), 0, st, x, a.w, epi, M, a.K, a.N, a.xs);
    else launch_pdl(lin_fma_kernel<X, E>, dim3((a.N + TN - 1) / TN, (M + TM - 1) / TM), dim3(256), 0, st, x, a.w, epi, M, a.K, a.N, a.xs);
    g_launches++;
}

// the epilogue of `a`, outputs in the activation type of YB
template <bool YB, class F>
void with_epilogue(const LinearArgs& a, F&& f) {
    if (a.tanh) f(make_epi_tanh<typename std::conditional<YB, ActBf16, ActF32>::type>(a.p, a.res, a.next, a.x_out, a.act, a.N, a.act_ld));
    else if (a.gelu_gate) f(EpiGelu<YB>{a.y, a.ys});
    else if (YB && a.y_bf16) { if (a.relu2) f(EpiPlain<YB, true>{a.y, a.ys, a.bias}); else f(EpiPlain<YB, false>{a.y, a.ys, a.bias}); }
    else { if (a.relu2) f(EpiPlain<false, true>{a.y, a.ys, a.bias}); else f(EpiPlain<false, false>{a.y, a.ys, a.bias}); }
}

}  // namespace

void k_linear(cudaStream_t st, const LinearArgs& a, uint32_t M, bool exact, unsigned int* status) {
    if (!M) return;
    if (!a.x_bf16) { with_epilogue<false>(a, [&](const auto& epi) { launch_fma<ActF32>(st, a, epi, M); }); return; }
    const bool vec = a.K % 8 == 0 && a.xs % 8 == 0 && (((uintptr_t)a.x | (uintptr_t)a.w) & 15u) == 0;
    with_epilogue<true>(a, [&](const auto& epi) {
        if (!exact && vec) {
            if (M < 32 && launch_stream_any(st, a, epi, M)) return;
            if (k_linear_sm100(st, a, M, status)) return;
            if (launch_stream_any(st, a, epi, M)) return;
        }
        launch_fma<ActBf16>(st, a, epi, M);
    });
}

}  // namespace gehtp
