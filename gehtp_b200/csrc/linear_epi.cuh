// What a projection of a row-count runlist does with its fp32 sums before they leave the kernel. Every kernel behind
// k_linear (streaming product, tcgen05 GEMM, split-K reduction, FMA tiles) takes one of these by value:
//   pair(m, n, v0, v1, N)   columns n, n + 1 of row m (n even)
//   quad(m, n, v, N)        columns n .. n + 3 (n a multiple of 4)
//   chunk(m, n, f, N)       columns n .. n + 31 (n a multiple of 32)
// Columns at or past N are left out.
#pragma once
#include <type_traits>
#include "rows_common.cuh"

namespace gehtp {

// y = v + bias, or max(v + bias, 0)^2
template <bool YB, bool RELU2>
struct EpiPlain {
    void* y;
    uint32_t ldy;
    const float* bias;
    __device__ __forceinline__ float val(float v, uint32_t n) const {
        if (bias) v += __ldg(bias + n);
        if (RELU2) { v = fmaxf(v, 0.0f); v = v * v; }
        return v;
    }
    __device__ __forceinline__ void one(uint32_t m, uint32_t n, float v) const {
        const size_t i = (size_t)m * ldy + n;
        if (YB) ((uint16_t*)y)[i] = f2bf(val(v, n)); else ((float*)y)[i] = val(v, n);
    }
    __device__ __forceinline__ void pair(uint32_t m, uint32_t n, float v0, float v1, uint32_t N) const {
        if (n < N) one(m, n, v0);
        if (n + 1 < N) one(m, n + 1, v1);
    }
    __device__ __forceinline__ void quad(uint32_t m, uint32_t n, const float* v, uint32_t N) const {
        const size_t i = (size_t)m * ldy + n;
        if (n + 4 <= N && (((uintptr_t)y + i * (YB ? 2 : 4)) & (YB ? 7u : 15u)) == 0) {
            const float a = val(v[0], n), b = val(v[1], n + 1), c = val(v[2], n + 2), d = val(v[3], n + 3);
            if (YB) *(uint2*)((uint16_t*)y + i) = make_uint2(pack_bf2(a, b), pack_bf2(c, d));
            else *(float4*)((float*)y + i) = make_float4(a, b, c, d);
            return;
        }
#pragma unroll
        for (uint32_t k = 0; k < 4; k++) if (n + k < N) one(m, n + k, v[k]);
    }
    __device__ __forceinline__ void chunk(uint32_t m, uint32_t n, const float (&f)[32], uint32_t N) const {
        if (YB && !RELU2 && bias && n + 32 <= N && ((uintptr_t)(bias + n) & 15u) == 0 && (((uintptr_t)y + ((size_t)m * ldy + n) * 2) & 15u) == 0) {
            uint4* d = (uint4*)((uint16_t*)y + (size_t)m * ldy + n);
#pragma unroll
            for (uint32_t q = 0; q < 4; q++) {
                const float4 a = __ldg((const float4*)(bias + n) + 2 * q), b = __ldg((const float4*)(bias + n) + 2 * q + 1);
                const float* v = f + 8 * q;
                d[q] = make_uint4(pack_bf2(v[0] + a.x, v[1] + a.y), pack_bf2(v[2] + a.z, v[3] + a.w), pack_bf2(v[4] + b.x, v[5] + b.y),
                                  pack_bf2(v[6] + b.z, v[7] + b.w));
            }
            return;
        }
#pragma unroll
        for (uint32_t q = 0; q < 4; q++) {
            const uint32_t c = n + 8 * q;
            if (c >= N) break;
            const size_t i = (size_t)m * ldy + c;
            if (YB && c + 8 <= N && (((uintptr_t)y + i * 2) & 15u) == 0) {
                uint32_t w[4];
#pragma unroll
                for (uint32_t k = 0; k < 4; k++) w[k] = pack_bf2(val(f[8 * q + 2 * k], c + 2 * k), val(f[8 * q + 2 * k + 1], c + 2 * k + 1));
                *(uint4*)((uint16_t*)y + i) = make_uint4(w[0], w[1], w[2], w[3]);
            } else {
                quad(m, c, f + 8 * q, N);
                if (c + 4 < N) quad(m, c + 4, f + 8 * q + 4, N);
            }
        }
    }
};

// tanh and 1 / (1 + e^-z) by output type: the library functions where fp32 comes out; beside bf16 outputs forms on the
// hardware exponential and reciprocal, whose absolute error stays within a few 2^-23.
template <class A> struct Curve {
    static __device__ __forceinline__ float tanh_(float z) { return tanhf(z); }
    static __device__ __forceinline__ float sigmoid(float z) { return sigmoid_f(z); }
};
template <> struct Curve<ActBf16> {
    static __device__ __forceinline__ float tanh_(float z) { return fmaf(-2.0f, sigmoid_fast(-2.0f * z), 1.0f); }
    static __device__ __forceinline__ float sigmoid(float z) { return sigmoid_fast(z); }
};

// Columns are (gate, up) pairs: y[m][n / 2] = gelu(gate) * up. The tanh form of gelu, z (1 + tanh u) / 2, is z sigmoid(2u).
template <bool YB>
struct EpiGelu {
    void* y;
    uint32_t ldy;
    static __device__ __forceinline__ float val(float z, float up) {
        const float u = 0.79788456080286535588f * fmaf(0.044715f * z * z, z, z);      // sqrt(2 / pi)
        return z * Curve<typename std::conditional<YB, ActBf16, ActF32>::type>::sigmoid(2.0f * u) * up;
    }
    __device__ __forceinline__ void pair(uint32_t m, uint32_t n, float v0, float v1, uint32_t N) const {
        if (n + 1 >= N) return;
        const size_t i = (size_t)m * ldy + n / 2;
        if (YB) ((uint16_t*)y)[i] = f2bf(val(v0, v1)); else ((float*)y)[i] = val(v0, v1);
    }
    __device__ __forceinline__ void quad(uint32_t m, uint32_t n, const float* v, uint32_t N) const {
        pair(m, n, v[0], v[1], N);
        pair(m, n + 2, v[2], v[3], N);
    }
    __device__ __forceinline__ void chunk(uint32_t m, uint32_t n, const float (&f)[32], uint32_t N) const {
#pragma unroll
        for (uint32_t q = 0; q < 2; q++) {
            const uint32_t c = n + 16 * q;
            const size_t i = (size_t)m * ldy + c / 2;
            if (YB && c + 16 <= N && (((uintptr_t)y + i * 2) & 15u) == 0) {
                uint32_t w[4];
#pragma unroll
                for (uint32_t k = 0; k < 4; k++) {
                    const float* p = f + 16 * q + 4 * k;
                    w[k] = pack_bf2(val(p[0], p[1]), val(p[2], p[3]));
                }
                *(uint4*)((uint16_t*)y + i) = make_uint4(w[0], w[1], w[2], w[3]);
            } else {
#pragma unroll
                for (uint32_t k = 0; k < 8; k++) pair(m, c + 2 * k, f[16 * q + 2 * k], f[16 * q + 2 * k + 1], N);
            }
        }
    }
};

// t(z, p) = tanh(alpha z) w + b of one column; p = [alpha, 0, 0, 0 | w: width | b: width], none: z
template <class A>
__device__ __forceinline__ float tanh_norm(const float* p, uint32_t width, uint32_t n, float z) {
    return p ? fmaf(Curve<A>::tanh_(__ldg(p) * z), __ldg(p + 4 + n), __ldg(p + 4 + width + n)) : z;
}

// x_out = x + t(v, p), act = t(x_out, next): the element-wise norm behind a sublayer, the residual sum and the norm in
// front of the next one. x and x_out may be the same rows.
template <class A>
struct EpiTanh {
    const float *p, *x, *next;
    float* x_out;
    typename A::T* act;
    uint32_t width, act_ld;
    bool vec;                          // rows of 16-byte quads (fp32) and 8- or 16-byte quads (act)
    __device__ __forceinline__ void one(uint32_t m, uint32_t n, float v) const {
        const size_t i = (size_t)m * width + n;
        const float s = (x ? __ldcg(x + i) : 0.0f) + tanh_norm<A>(p, width, n, v);
        if (x_out) x_out[i] = s;
        if (act) A::st(act + (size_t)m * act_ld + n, tanh_norm<A>(next, width, n, s));
    }
    __device__ __forceinline__ void pair(uint32_t m, uint32_t n, float v0, float v1, uint32_t N) const {
        if (n < N) one(m, n, v0);
        if (n + 1 < N) one(m, n + 1, v1);
    }
    // t of four columns
    __device__ __forceinline__ float4 t4(const float* q, uint32_t n, float4 z) const {
        if (!q) return z;
        const float a = __ldg(q);
        const float4 w = __ldg((const float4*)(q + 4 + n)), b = __ldg((const float4*)(q + 4 + width + n));
        return make_float4(fmaf(Curve<A>::tanh_(a * z.x), w.x, b.x), fmaf(Curve<A>::tanh_(a * z.y), w.y, b.y),
                           fmaf(Curve<A>::tanh_(a * z.z), w.z, b.z), fmaf(Curve<A>::tanh_(a * z.w), w.w, b.w));
    }
    __device__ __forceinline__ float4 res4(uint32_t m, uint32_t n) const {
        return x ? __ldcg((const float4*)(x + (size_t)m * width + n)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    __device__ __forceinline__ void put4(uint32_t m, uint32_t n, const float* v, float4 r) const {
        const float4 t = t4(p, n, make_float4(v[0], v[1], v[2], v[3]));
        r.x += t.x; r.y += t.y; r.z += t.z; r.w += t.w;
        if (x_out) *(float4*)(x_out + (size_t)m * width + n) = r;
        if (!act) return;
        const float4 o = t4(next, n, r);
        typename A::T* d = act + (size_t)m * act_ld + n;
        if constexpr (sizeof(typename A::T) == 2) *(uint2*)d = make_uint2(pack_bf2(o.x, o.y), pack_bf2(o.z, o.w));
        else *(float4*)d = o;
    }
    __device__ __forceinline__ void quad(uint32_t m, uint32_t n, const float* v, uint32_t N) const {
        if (vec) { put4(m, n, v, res4(m, n)); return; }
#pragma unroll
        for (uint32_t k = 0; k < 4; k++) if (n + k < N) one(m, n + k, v[k]);
    }
    __device__ __forceinline__ void chunk(uint32_t m, uint32_t n, const float (&f)[32], uint32_t N) const {
        if (!vec) {
#pragma unroll
            for (uint32_t k = 0; k < 32; k++) if (n + k < N) one(m, n + k, f[k]);
            return;
        }
        float4 r[8];                   // the residual is requested ahead: its stores may not be reordered with the loads
#pragma unroll
        for (uint32_t q = 0; q < 8; q++) r[q] = n + 4 * q < N ? res4(m, n + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (uint32_t q = 0; q < 8; q++) if (n + 4 * q < N) put4(m, n + 4 * q, f + 4 * q, r[q]);
    }
};

// host: `p`, `x` etc. as planned, rows aligned for four columns at a time?
template <class A>
inline EpiTanh<A> make_epi_tanh(const float* p, const float* x, const float* next, float* x_out, void* act, uint32_t width, uint32_t act_ld) {
    EpiTanh<A> e;
    e.p = p; e.x = x; e.next = next; e.x_out = x_out; e.act = (typename A::T*)act; e.width = width; e.act_ld = act_ld;
    const uintptr_t al = (uintptr_t)p | (uintptr_t)x | (uintptr_t)next | (uintptr_t)x_out;
    e.vec = width % 4 == 0 && act_ld % 4 == 0 && (al & 15u) == 0 && ((uintptr_t)act & (sizeof(typename A::T) == 2 ? 7u : 15u)) == 0;
    return e;
}

}  // namespace gehtp
