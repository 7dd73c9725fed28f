// Latent attention over many rows (bf16): keys and values of every cached position are expanded by one projection of
// the state rows (all heads' key and value up-projections side by side), then a flash kernel on mma.sync runs per head:
// 128 query rows, tiles of 64 positions by cp.async in two stages, the rotated key part read from the state row that
// all heads share. Scores and weights are fp32; the weights enter the value product as hi + lo bf16 pairs.
#include "launchers_rows.h"
#include "mma_bf16.cuh"

namespace gehtp {

namespace {

constexpr uint32_t BM = 128, BN = 64;

__device__ __forceinline__ uint32_t up16(uint32_t v) { return (v + 15u) & ~15u; }

// Loads rows [j0, j0 + n) of a tile: `len` elements per row at src + j * stride, to dst rows of `rs` elements; rows at
// or past `limit` are zero-filled. VEC: 16-byte copies (everything a multiple of 8 elements), else one element at a time.
template <bool VEC>
__device__ __forceinline__ void load_rows(uint16_t* dst, uint32_t rs, const uint16_t* src, size_t stride, uint32_t j0, uint32_t n,
                                          uint32_t limit, uint32_t len) {
    if (VEC) {
        const uint32_t ch = len / 8;
        for (uint32_t i = threadIdx.x; i < n * ch; i += 256) {
            const uint32_t r = i / ch, c = i % ch, j = j0 + r;
            cp16(smem_addr(dst + r * rs + c * 8), src + (size_t)min(j, limit - 1) * stride + c * 8, j < limit ? 16 : 0);
        }
    } else {
        for (uint32_t i = threadIdx.x; i < n * len; i += 256) {
            const uint32_t r = i / len, c = i % len, j = j0 + r;
            dst[r * rs + c] = j < limit ? __ldcg(src + (size_t)j * stride + c) : (uint16_t)0;
        }
    }
}

__device__ __forceinline__ void zero_cols(uint16_t* dst, uint32_t rs, uint32_t n, uint32_t c0, uint32_t c1) {
    if (c1 <= c0) return;
    const uint32_t w = c1 - c0;
    for (uint32_t i = threadIdx.x; i < n * w; i += 256) dst[(i / w) * rs + c0 + i % w] = 0;
}

// VT: 8-column tiles of a head's value, an even number >= vdim / 8
template <int VT, bool VEC>
__global__ void __launch_bounds__(256)
latent_flash_kernel(const LatentArgs a, const uint16_t* kv, uint32_t rows, uint32_t past) {
    extern __shared__ __align__(16) unsigned char smem[];
    const uint32_t hd = a.dim + a.rot, dp = up16(hd), vp = up16(a.vdim), rk = dp + 8, rv = vp + 8, ls = a.ls();
    const uint32_t kvs = a.heads * (a.dim + a.vdim);
    uint16_t* sq = (uint16_t*)smem;                       // [BM][rk]
    uint16_t* sk = sq + BM * rk;                          // [2][BN][rk]
    uint16_t* sv = sk + 2 * BN * rk;                      // [2][BN][rv]
    pdl_release();
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const uint32_t h = blockIdx.x, q0 = (gridDim.y - 1 - blockIdx.y) * BM;       // longest rows of all heads first
    // columns no copy writes: padding of a head to 16
    zero_cols(sq, rk, BM, hd, dp);
    zero_cols(sk, rk, 2 * BN, hd, dp);
    zero_cols(sv, rv, 2 * BN, a.vdim, vp);
    pdl_wait();
    const uint32_t n = past + rows, last = min(past + q0 + BM, n);              // positions [0, last) matter to this block
    const uint32_t tiles = (last + BN - 1) / BN;
    const uint16_t* state = (const uint16_t*)a.state;
    auto fetch = [&](uint32_t t) {
        if (t < tiles) {
            uint16_t *k = sk + (t & 1) * BN * rk, *v = sv + (t & 1) * BN * rv;
            load_rows<VEC>(k, rk, kv + h * a.dim, kvs, t * BN, BN, n, a.dim);
            if (a.rot) load_rows<VEC>(k + a.dim, rk, state + a.rank, ls, t * BN, BN, n, a.rot);
            load_rows<VEC>(v, rv, kv + a.heads * a.dim + h * a.vdim, kvs, t * BN, BN, n, a.vdim);
        }
        if (VEC) cp_commit();
    };
    load_rows<VEC>(sq, rk, (const uint16_t*)a.q + (size_t)h * hd, (size_t)a.heads * hd, q0, BM, rows, hd);
    fetch(0);
    float o[VT][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < VT; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const float sc = a.scale * 1.44269504088896340736f;                         // scores in powers of two
    const uint32_t a_row = lane & 15, a_col = (lane >> 4) * 8;
    const uint32_t qaddr = smem_addr(sq + (warp * 16 + a_row) * rk + a_col);
    const uint32_t row_lo = past + q0 + warp * 16 + g;                          // position of this lane's first row
    const uint32_t warp_last = past + q0 + warp * 16 + 15;
    for (uint32_t t = 0; t < tiles; t++) {
        if (VEC) cp_wait<0>();
        __syncthreads();
        fetch(t + 1);
        if (t * BN > warp_last) continue;                                       // entirely in this warp's future
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
        const bool edge = t * BN + BN - 1 > past + q0 + warp * 16;              // some key of the tile is hidden from some row
        float mx[2] = {m[0], m[1]};
#pragma unroll
        for (int i = 0; i < (int)BN / 8; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                float x = s[i][e] * sc;
                if (edge && t * BN + i * 8 + 2 * t4 + (e & 1) > row_lo + (e >> 1) * 8) x = -INFINITY;
                s[i][e] = x;
                mx[e >> 1] = fmaxf(mx[e >> 1], x);
            }
#pragma unroll
        for (int r = 0; r < 2; r++) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            const float corr = exp2f(m[r] - mx[r]);                             // key 0 is visible to every row: mx is finite
            m[r] = mx[r];
            l[r] *= corr;
#pragma unroll
            for (int i = 0; i < VT; i++) { o[i][2 * r] *= corr; o[i][2 * r + 1] *= corr; }
        }
#pragma unroll
        for (int i = 0; i < (int)BN / 8; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const float p = exp2f(s[i][e] - m[e >> 1]);
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
#pragma unroll
    for (int r = 0; r < 2; r++) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        const uint32_t row = q0 + warp * 16 + g + r * 8;
        if (row >= rows) continue;
        const float f = a.gate[(size_t)row * a.heads + h] / l[r];
        uint16_t* out = (uint16_t*)a.out + ((size_t)row * a.heads + h) * a.vdim;
#pragma unroll
        for (int i = 0; i < VT; i++) {
            const uint32_t c = i * 8 + 2 * t4;
            if (VEC) { if (c < a.vdim) *(uint32_t*)(out + c) = pack_bf2(o[i][2 * r] * f, o[i][2 * r + 1] * f); }
            else {
                if (c < a.vdim) out[c] = f2bf(o[i][2 * r] * f);
                if (c + 1 < a.vdim) out[c + 1] = f2bf(o[i][2 * r + 1] * f);
            }
        }
    }
}

size_t flash_smem(const LatentArgs& a) {
    const size_t dp = (a.dim + a.rot + 15u) & ~15u, vp = (a.vdim + 15u) & ~15u;
    return ((BM + 2 * BN) * (dp + 8) + 2 * BN * (vp + 8)) * 2;
}

template <int VT, bool VEC>
bool launch_flash(cudaStream_t st, const LatentArgs& a, const uint16_t* kv, uint32_t rows, uint32_t past) {
    static int have[64] = {};
    const size_t smem = flash_smem(a);
    if (!ensure_dyn_smem(latent_flash_kernel<VT, VEC>, smem, have)) return false;
    launch_pdl(latent_flash_kernel<VT, VEC>, dim3(a.heads, (rows + BM - 1) / BM), dim3(256), smem, st, a, kv, rows, past);
    g_launches++;
    return true;
}

bool takes(const LatentArgs& a) { return a.bf16 && a.vdim <= 256 && flash_smem(a) <= 220 * 1024; }

}  // namespace

size_t latent_prefill_floats(const LatentArgs& a, uint32_t) {
    return takes(a) ? ((size_t)a.nslots * a.heads * (a.dim + a.vdim) + 1) / 2 : 0;
}

// false: sizes outside what the kernel takes, nothing launched
bool k_latent_prefill(cudaStream_t st, const LatentArgs& a, uint32_t rows, uint32_t n_past) {
    if (!takes(a) || n_past + rows > a.nslots) return false;
    LinearArgs lin{};
    lin.x = a.state; lin.w = a.w_kv; lin.y = a.work;
    lin.K = a.rank; lin.N = a.heads * (a.dim + a.vdim); lin.xs = a.ls(); lin.ys = lin.N;
    lin.x_bf16 = lin.y_bf16 = true;
    k_linear(st, lin, n_past + rows, false, a.status);
    const uint16_t* kv = (const uint16_t*)a.work;
    const bool vec = a.dim % 8 == 0 && a.rot % 8 == 0 && a.vdim % 8 == 0 && a.rank % 8 == 0;
    const uint32_t vt = (a.vdim + 15) / 16 * 2;
    if (vec) {
        if (vt <= 4) return launch_flash<4, true>(st, a, kv, rows, n_past);
        if (vt <= 8) return launch_flash<8, true>(st, a, kv, rows, n_past);
        if (vt <= 16) return launch_flash<16, true>(st, a, kv, rows, n_past);
        return launch_flash<32, true>(st, a, kv, rows, n_past);
    }
    if (vt <= 8) return launch_flash<8, false>(st, a, kv, rows, n_past);
    if (vt <= 16) return launch_flash<16, false>(st, a, kv, rows, n_past);
    return launch_flash<32, false>(st, a, kv, rows, n_past);
}

}  // namespace gehtp
