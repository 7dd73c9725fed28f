// Window attention over many rows (bf16) for any head sizes: a flash kernel on mma.sync. 128 query rows of one head per
// CTA, tiles of 64 positions by cp.async in two stages, of which only those a row of the CTA can see are visited. Scores
// and weights are fp32; the weights enter the value product as hi + lo bf16 pairs.
#include "launchers_rows.h"
#include "mma_bf16.cuh"

namespace gehtp {

namespace {

constexpr uint32_t BM = 128, BN = 64;

// Rows [j0, j0 + n) of `len` elements, row j at src + (j mod ring) * stride, to rows of `rs` elements; rows at or past
// `limit` are zero-filled. VEC: 16-byte copies, and no wrap inside the n rows; else one element at a time.
template <bool VEC>
__device__ __forceinline__ void load_ring(uint16_t* dst, uint32_t rs, const uint16_t* src, size_t stride, uint32_t j0, uint32_t n,
                                          uint32_t ring, uint32_t limit, uint32_t len) {
    if (VEC) {
        const uint32_t ch = len / 8, base = j0 % ring;
        for (uint32_t i = threadIdx.x; i < n * ch; i += 256) {
            const uint32_t r = i / ch, c = i % ch;
            cp16(smem_addr(dst + r * rs + c * 8), src + (size_t)(base + r) * stride + c * 8, j0 + r < limit ? 16 : 0);
        }
    } else {
        for (uint32_t i = threadIdx.x; i < n * len; i += 256) {
            const uint32_t r = i / len, c = i % len, j = j0 + r;
            dst[r * rs + c] = j < limit ? __ldcg(src + (size_t)(j % ring) * stride + c) : (uint16_t)0;
        }
    }
}

__device__ __forceinline__ void zero_tail(uint16_t* dst, uint32_t rs, uint32_t n, uint32_t c0, uint32_t c1) {
    if (c1 <= c0) return;
    const uint32_t w = c1 - c0;
    for (uint32_t i = threadIdx.x; i < n * w; i += 256) dst[(i / w) * rs + c0 + i % w] = 0;
}

template <int VT, bool VEC>
__global__ void __launch_bounds__(256)
window_flash_kernel(const WindowArgs a, uint32_t rows) {
    extern __shared__ __align__(16) unsigned char smem[];
    const uint32_t dp = (a.dim + 15u) & ~15u, vp = (a.vdim + 15u) & ~15u, rk = dp + 8, rv = vp + 8, row = a.row();
    uint16_t* sq = (uint16_t*)smem;                       // [BM][rk]
    uint16_t* sk = sq + BM * rk;                          // [2][BN][rk]
    uint16_t* sv = sk + 2 * BN * rk;                      // [2][BN][rv]
    pdl_release();
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
    const uint32_t h = blockIdx.x, g = h / (a.heads / a.kv_heads), q0 = (gridDim.y - 1 - blockIdx.y) * BM;
    zero_tail(sq, rk, BM, a.dim, dp);
    zero_tail(sk, rk, 2 * BN, a.dim, dp);
    zero_tail(sv, rv, 2 * BN, a.vdim, vp);
    pdl_wait();
    const uint32_t past = *a.counter, n = past + rows, p0 = past + q0;
    const uint32_t first = p0 + 1 > a.window ? p0 + 1 - a.window : 0, last = min(p0 + BM, n);      // positions [first, last) matter
    const uint32_t tb = first / BN, te = (last + BN - 1) / BN;
    const uint16_t *keys = (const uint16_t*)a.state + g * a.dim, *vals = (const uint16_t*)a.state + a.kv_heads * a.dim + g * a.vdim;
    auto fetch = [&](uint32_t t) {
        if (t < te) {
            load_ring<VEC>(sk + (t & 1) * BN * rk, rk, keys, row, t * BN, BN, a.ring, n, a.dim);
            load_ring<VEC>(sv + (t & 1) * BN * rv, rv, vals, row, t * BN, BN, a.ring, n, a.vdim);
        }
        if (VEC) cp_commit();
    };
    load_ring<VEC>(sq, rk, (const uint16_t*)a.q + (size_t)h * a.dim, (size_t)a.heads * a.dim, q0, BM, 0xFFFFFFFFu, rows, a.dim);
    fetch(tb);
    float o[VT][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < VT; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const float sc = a.scale * 1.44269504088896340736f;                         // scores in powers of two
    const uint32_t qaddr = smem_addr(sq + (warp * 16 + (lane & 15)) * rk + (lane >> 4) * 8);
    const uint32_t w0 = p0 + warp * 16, w1 = w0 + 15, row_lo = w0 + g4;         // positions of this warp's rows, of this lane's first
    for (uint32_t t = tb; t < te; t++) {
        if (VEC) cp_wait<0>();
        __syncthreads();
        fetch(t + 1);
        const uint32_t j0 = t * BN, j1 = j0 + BN - 1;
        if (j0 > w1 || j1 + a.window <= w0) continue;                           // nothing of the tile is visible to this warp
        const uint16_t *k = sk + (t & 1) * BN * rk, *v = sv + (t & 1) * BN * rv;
        float s[BN / 8][4];
#pragma unroll
        for (int i = 0; i < (int)BN / 8; i++) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
        const uint32_t kaddr = smem_addr(k + ((lane & 7) + (lane >> 4) * 8) * rk + ((lane >> 3) & 1) * 8);
#pragma unroll 4
        for (uint32_t ks = 0; ks < dp / 16; ks++) {
            uint32_t qa[4];
            ldsm4(qa, qaddr + ks * 32);
#pragma unroll
            for (int i = 0; i < (int)BN / 16; i++) {
                uint32_t b[4];
                ldsm4(b, kaddr + (i * 16 * rk) * 2 + ks * 32);
                mma_bf16(s[2 * i], qa, b[0], b[1]);
                mma_bf16(s[2 * i + 1], qa, b[2], b[3]);
            }
        }
        const bool edge = j1 > w0 || j0 + a.window <= w1;                       // some key of the tile is hidden from some row
        float mx[2] = {m[0], m[1]};
#pragma unroll
        for (int i = 0; i < (int)BN / 8; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                float x = s[i][e] * sc;
                if (edge) {
                    const uint32_t j = j0 + i * 8 + 2 * t4 + (e & 1), p = row_lo + (e >> 1) * 8;
                    if (j > p || j + a.window <= p) x = -INFINITY;
                }
                s[i][e] = x;
                mx[e >> 1] = fmaxf(mx[e >> 1], x);
            }
        float base[2];
#pragma unroll
        for (int r = 0; r < 2; r++) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            base[r] = mx[r] == -INFINITY ? 0.0f : mx[r];                        // a row that has seen no key yet
            const float corr = exp2f(m[r] - base[r]);
            m[r] = mx[r];
            l[r] *= corr;
#pragma unroll
            for (int i = 0; i < VT; i++) { o[i][2 * r] *= corr; o[i][2 * r + 1] *= corr; }
        }
#pragma unroll
        for (int i = 0; i < (int)BN / 8; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const float p = exp2f(s[i][e] - base[e >> 1]);
                s[i][e] = p;
                l[e >> 1] += p;
            }
        const uint32_t vaddr = smem_addr(v + (lane & 15) * rv + (lane >> 4) * 8);
#pragma unroll
        for (int ks = 0; ks < (int)BN / 16; ks++) {
            uint32_t ph[4], pl[4];
            split_bf2(s[2 * ks][0], s[2 * ks][1], ph[0], pl[0]);
            split_bf2(s[2 * ks][2], s[2 * ks][3], ph[1], pl[1]);
            split_bf2(s[2 * ks + 1][0], s[2 * ks + 1][1], ph[2], pl[2]);
            split_bf2(s[2 * ks + 1][2], s[2 * ks + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int i = 0; i < VT; i += 2) {
                if (i * 8 >= (int)vp) break;
                uint32_t b[4];
                ldsm4_t(b, vaddr + (ks * 16 * rv + i * 8) * 2);
                mma_bf16(o[i], ph, b[0], b[1]);
                mma_bf16(o[i], pl, b[0], b[1]);
                mma_bf16(o[i + 1], ph, b[2], b[3]);
                mma_bf16(o[i + 1], pl, b[2], b[3]);
            }
        }
    }
    if (VEC) cp_wait<0>();
    const bool gate = a.gate_col != 0xFFFFFFFFu;
#pragma unroll
    for (int r = 0; r < 2; r++) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        const uint32_t qr = q0 + warp * 16 + g4 + r * 8;
        if (qr >= rows) continue;
        const float f = 1.0f / l[r];
        const uint16_t* yg = (const uint16_t*)a.y + (size_t)qr * a.y_cols + a.gate_col + h * a.vdim;
        uint16_t* out = (uint16_t*)a.out + ((size_t)qr * a.heads + h) * a.vdim;
#pragma unroll
        for (int i = 0; i < VT; i++) {
            const uint32_t c = i * 8 + 2 * t4;
            if (c >= a.vdim) break;
            const float u = o[i][2 * r] * f * (gate ? sigmoid_fast(bf2f(__ldcg(yg + c))) : 1.0f);
            if (c + 1 >= a.vdim) { out[c] = f2bf(u); break; }
            const float w = o[i][2 * r + 1] * f * (gate ? sigmoid_fast(bf2f(__ldcg(yg + c + 1))) : 1.0f);
            if (VEC) *(uint32_t*)(out + c) = pack_bf2(u, w);
            else { out[c] = f2bf(u); out[c + 1] = f2bf(w); }
        }
    }
}

size_t flash_smem(const WindowArgs& a) {
    const size_t dp = (a.dim + 15u) & ~15u, vp = (a.vdim + 15u) & ~15u;
    return ((BM + 2 * BN) * (dp + 8) + 2 * BN * (vp + 8)) * 2;
}

template <int VT, bool VEC>
bool launch_flash(cudaStream_t st, const WindowArgs& a, uint32_t rows) {
    static int have[64] = {};
    const size_t smem = flash_smem(a);
    if (!ensure_dyn_smem(window_flash_kernel<VT, VEC>, smem, have)) return false;
    launch_pdl(window_flash_kernel<VT, VEC>, dim3(a.heads, (rows + BM - 1) / BM), dim3(256), smem, st, a, rows);
    g_launches++;
    return true;
}

}  // namespace

// false: sizes outside what the kernel takes, nothing launched
bool k_window_flash(cudaStream_t st, const WindowArgs& a, uint32_t rows) {
    if (!a.bf16 || a.vdim > 256 || flash_smem(a) > 220 * 1024) return false;
    const uint32_t vt = (a.vdim + 15) / 16 * 2;
    if (a.dim % 8 == 0 && a.vdim % 8 == 0 && a.ring % BN == 0) {
        if (vt <= 4) return launch_flash<4, true>(st, a, rows);
        if (vt <= 8) return launch_flash<8, true>(st, a, rows);
        if (vt <= 16) return launch_flash<16, true>(st, a, rows);
        return launch_flash<32, true>(st, a, rows);
    }
    if (vt <= 8) return launch_flash<8, false>(st, a, rows);
    if (vt <= 16) return launch_flash<16, false>(st, a, rows);
    return launch_flash<32, false>(st, a, rows);
}

}  // namespace gehtp
