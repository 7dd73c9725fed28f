// Row-wise pieces of the row-count runlists: embedding rows, RMS norm or element-wise tanh norm added to the residual
// stream, picked rows, greedy choice, position counters. The residual stream and every norm are fp32.
#include "launchers_rows.h"
#include "linear_epi.cuh"

namespace gehtp {

namespace {

template <class A>
__global__ void __launch_bounds__(256)
embed_rows_kernel(const uint16_t* __restrict__ table, const int32_t* ids, float* x, typename A::T* act, uint32_t act_ld, uint32_t width,
                  uint32_t vocab, float scale) {
    pdl_release();
    pdl_wait();
    const uint32_t r = blockIdx.x;
    const int32_t id = ids[r];
    const bool ok = id >= 0 && (uint32_t)id < vocab;             // the host checks ids; a stray one reads nothing
    const uint16_t* src = table + (size_t)(ok ? id : 0) * width;
    for (uint32_t i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = ok ? bf2f(__ldg(src + i)) * scale : 0.0f;
        x[(size_t)r * width + i] = v;
        if (act) A::st(act + (size_t)r * act_ld + i, v);
    }
}

// One CTA per row: x_out = x + y / sqrt(mean(y^2) + eps) * (base + w), act = x_out in the activation type. A thread
// keeps up to KEEP values of the row in registers between the two passes; longer rows are read twice.
template <class Y, class A, int VEC>
__global__ void __launch_bounds__(256)
norm_resid_kernel(const typename Y::T* y, const float* __restrict__ w, const float* x, float* x_out, typename A::T* act,
                  uint32_t width, float eps, float base) {
    __shared__ float part[8];
    constexpr int KEEP = 16;
    pdl_release();
    const size_t off = (size_t)blockIdx.x * width;
    const uint32_t tid = threadIdx.x, step = 256 * VEC;
    pdl_wait();
    float keep[KEEP], res[KEEP];
    float ss = 0.0f;
#pragma unroll
    for (int u = 0; u < KEEP / VEC; u++) {
        const uint32_t i = tid * VEC + u * step;
#pragma unroll
        for (int k = 0; k < VEC; k++) { keep[u * VEC + k] = 0.0f; res[u * VEC + k] = 0.0f; }
        if (i >= width) continue;
        if constexpr (VEC == 4 && sizeof(typename Y::T) == 4) {
            const float4 q = __ldcg((const float4*)(y + off + i));
            keep[u * 4] = q.x; keep[u * 4 + 1] = q.y; keep[u * 4 + 2] = q.z; keep[u * 4 + 3] = q.w;
            if (x) {
                const float4 xr = __ldcg((const float4*)(x + off + i));
                res[u * 4] = xr.x; res[u * 4 + 1] = xr.y; res[u * 4 + 2] = xr.z; res[u * 4 + 3] = xr.w;
            }
        } else {
#pragma unroll
            for (int k = 0; k < VEC; k++)
                if (i + k < width) { keep[u * VEC + k] = Y::ld(y + off + i + k); if (x) res[u * VEC + k] = __ldcg(x + off + i + k); }
        }
#pragma unroll
        for (int k = 0; k < VEC; k++) ss = fmaf(keep[u * VEC + k], keep[u * VEC + k], ss);
    }
    for (uint32_t i = tid + 256 * KEEP; i < width; i += 256) { const float v = Y::ld(y + off + i); ss = fmaf(v, v, ss); }
    ss = block_sum(ss, part);
    const float inv = 1.0f / sqrtf(ss / (float)width + eps);
#pragma unroll
    for (int u = 0; u < KEEP / VEC; u++) {
        const uint32_t i = tid * VEC + u * step;
        if (i >= width) continue;
        float o[VEC];
#pragma unroll
        for (int k = 0; k < VEC; k++) o[k] = (i + k < width) ? res[u * VEC + k] + keep[u * VEC + k] * inv * (base + __ldg(w + i + k)) : 0.0f;
        if constexpr (VEC == 4) {
            if (x_out) *(float4*)(x_out + off + i) = make_float4(o[0], o[1], o[2], o[3]);
            if (act) {
                if constexpr (sizeof(typename A::T) == 2) *(uint2*)(act + off + i) = make_uint2(pack_bf2(o[0], o[1]), pack_bf2(o[2], o[3]));
                else *(float4*)(act + off + i) = make_float4(o[0], o[1], o[2], o[3]);
            }
        } else {
#pragma unroll
            for (int k = 0; k < VEC; k++) {
                if (i + k >= width) break;
                if (x_out) x_out[off + i + k] = o[k];
                if (act) A::st(act + off + i + k, o[k]);
            }
        }
    }
    for (uint32_t i = tid + 256 * KEEP; i < width; i += 256) {
        const float o = (x ? __ldcg(x + off + i) : 0.0f) + Y::ld(y + off + i) * inv * (base + __ldg(w + i));
        if (x_out) x_out[off + i] = o;
        if (act) A::st(act + off + i, o);
    }
}

// Rows of y (or, with idx, the rows idx picks of it) through the epilogue of linear_epi.cuh, 4 columns per thread
template <class Y, class A>
__global__ void __launch_bounds__(256)
tanh_resid_kernel(const typename Y::T* y, const int32_t* idx, uint32_t y_rows, const EpiTanh<A> epi, uint32_t width) {
    pdl_release();
    pdl_wait();
    const uint32_t r = blockIdx.y, n = (blockIdx.x * 256 + threadIdx.x) * 4;
    if (n >= width) return;
    uint32_t src = r;
    bool ok = true;
    if (idx) { const int32_t s = idx[r]; ok = s >= 0 && (uint32_t)s < y_rows; src = ok ? (uint32_t)s : 0u; }
    const typename Y::T* p = y + (size_t)src * width + n;
    float v[4];
    if (sizeof(typename Y::T) == 4 && width % 4 == 0) {
        const float4 q = __ldcg((const float4*)p);
        v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    } else {
#pragma unroll
        for (uint32_t k = 0; k < 4; k++) v[k] = n + k < width ? Y::ld(p + k) : 0.0f;
    }
#pragma unroll
    for (uint32_t k = 0; k < 4; k++) v[k] = ok ? v[k] : 0.0f;
    epi.quad(r, n, v, width);
}

__global__ void __launch_bounds__(256)
pick_rows_kernel(const float* x, const int32_t* idx, float* out, uint32_t width, uint32_t x_rows) {
    pdl_release();
    pdl_wait();
    const int32_t s = idx[blockIdx.x];
    const bool ok = s >= 0 && (uint32_t)s < x_rows;
    for (uint32_t i = threadIdx.x; i < width; i += blockDim.x)
        out[(size_t)blockIdx.x * width + i] = ok ? __ldcg(x + (size_t)s * width + i) : 0.0f;
}

// first index of the largest value (a NaN never wins)
__global__ void __launch_bounds__(1024)
argmax_rows_f32_kernel(const float* x, int32_t* out, uint32_t n) {
    __shared__ float bv[32];
    __shared__ uint32_t bi[32];
    pdl_release();
    pdl_wait();
    const float* row = x + (size_t)blockIdx.x * n;
    float best = -INFINITY;
    uint32_t at = 0xFFFFFFFFu;
    for (uint32_t i = threadIdx.x; i < n; i += blockDim.x) {
        const float v = __ldcg(row + i);
        if (v > best || (v == best && i < at)) { best = v; at = i; }
    }
    for (int o = 16; o > 0; o >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, best, o);
        const uint32_t i = __shfl_xor_sync(0xffffffffu, at, o);
        if (v > best || (v == best && i < at)) { best = v; at = i; }
    }
    if ((threadIdx.x & 31) == 0) { bv[threadIdx.x >> 5] = best; bi[threadIdx.x >> 5] = at; }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (uint32_t w = 1; w < blockDim.x / 32; w++)
            if (bv[w] > best || (bv[w] == best && bi[w] < at)) { best = bv[w]; at = bi[w]; }
        out[blockIdx.x] = at == 0xFFFFFFFFu ? 0 : (int32_t)at;
    }
}

__global__ void state_advance_kernel(uint32_t* counters, uint32_t n, uint32_t rows) {
    for (uint32_t i = threadIdx.x; i < n; i += blockDim.x) counters[i] += rows;
}

template <class Y, class A>
void launch_tanh(cudaStream_t st, const TanhResidArgs& a, uint32_t rows) {
    launch_pdl(tanh_resid_kernel<Y, A>, dim3((a.width + 1023) / 1024, rows), dim3(256), 0, st, (const typename Y::T*)a.y, a.idx, a.y_rows,
               make_epi_tanh<A>(a.p, a.x, a.next, a.x_out, a.act, a.width, a.act_ld), a.width);
}

template <class Y, class A>
void launch_norm(cudaStream_t st, const NormResidArgs& a, uint32_t rows) {
    const uintptr_t al = (uintptr_t)a.y | (uintptr_t)a.x | (uintptr_t)a.x_out | (uintptr_t)a.act;
    const typename Y::T* y = (const typename Y::T*)a.y;
    typename A::T* act = (typename A::T*)a.act;
    if (a.width % 4 == 0 && a.width <= 4096 && (al & 15u) == 0)
        launch_pdl(norm_resid_kernel<Y, A, 4>, dim3(rows), dim3(256), 0, st, y, a.w, a.x, a.x_out, act, a.width, a.eps, a.base);
    else
        launch_pdl(norm_resid_kernel<Y, A, 1>, dim3(rows), dim3(256), 0, st, y, a.w, a.x, a.x_out, act, a.width, a.eps, a.base);
}

}  // namespace

void k_embed_rows(cudaStream_t st, const uint16_t* table, const int32_t* ids, float* x, void* act, uint32_t act_ld, uint32_t rows, uint32_t width,
                  uint32_t vocab, float scale, bool bf16) {
    if (!rows) return;
    // ordinary launch: the first kernel of a run starts after everything of the run before
    if (bf16) embed_rows_kernel<ActBf16><<<rows, 256, 0, st>>>(table, ids, x, (uint16_t*)act, act_ld, width, vocab, scale);
    else embed_rows_kernel<ActF32><<<rows, 256, 0, st>>>(table, ids, x, (float*)act, act_ld, width, vocab, scale);
    g_launches++;
}

void k_norm_resid(cudaStream_t st, const NormResidArgs& a, uint32_t rows) {
    if (!rows) return;
    if (a.y_bf16) { if (a.act_bf16) launch_norm<ActBf16, ActBf16>(st, a, rows); else launch_norm<ActBf16, ActF32>(st, a, rows); }
    else { if (a.act_bf16) launch_norm<ActF32, ActBf16>(st, a, rows); else launch_norm<ActF32, ActF32>(st, a, rows); }
    g_launches++;
}

void k_tanh_resid(cudaStream_t st, const TanhResidArgs& a, uint32_t rows) {
    if (!rows) return;
    if (a.y_bf16) { if (a.act_bf16) launch_tanh<ActBf16, ActBf16>(st, a, rows); else launch_tanh<ActBf16, ActF32>(st, a, rows); }
    else { if (a.act_bf16) launch_tanh<ActF32, ActBf16>(st, a, rows); else launch_tanh<ActF32, ActF32>(st, a, rows); }
    g_launches++;
}

void k_pick_rows(cudaStream_t st, const float* x, const int32_t* idx, float* out, uint32_t rows, uint32_t width, uint32_t x_rows) {
    if (!rows) return;
    launch_pdl(pick_rows_kernel, dim3(rows), dim3(256), 0, st, x, idx, out, width, x_rows);
    g_launches++;
}

void k_argmax_rows_f32(cudaStream_t st, const float* x, int32_t* out, uint32_t rows, uint32_t n) {
    if (!rows) return;
    launch_pdl(argmax_rows_f32_kernel, dim3(rows), dim3(1024), 0, st, x, out, n);
    g_launches++;
}

void k_state_advance(cudaStream_t st, uint32_t* counters, uint32_t n, uint32_t rows) {
    if (!rows) return;
    state_advance_kernel<<<1, 64, 0, st>>>(counters, n, rows);
    g_launches++;
}

}  // namespace gehtp
