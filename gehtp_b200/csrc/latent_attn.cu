// Latent attention: the cache holds one normed latent and one rotated key part per position, shared by all heads
// (OP_LATENT_APPEND, OP_LATENT_ATTEND).
//
//   latent_append_kernel   rotary on q and the key part, RMS norm of the latent, gate, append to the state
//   latent_exact_kernel    plain form, fp32 throughout: one CTA per (head, row), any size
//   few bf16 rows          latent_absorb_kernel (append + q taken through the key up-projection into latent space),
//                          latent_split_kernel (all heads against slices of the cached rows: every row is read once,
//                          as key and as value), latent_merge_kernel (slices combined, value up-projection, gate)
//   more bf16 rows         latent_prefill.cu
#include <cooperative_groups.h>
#include "launchers_rows.h"
#include "mma_bf16.cuh"

namespace gehtp {

namespace {

constexpr uint32_t kAbsorbRows = 16;      // rows up to which the absorbed chain runs
constexpr uint32_t kMaxSplit = 148;       // slices of the cached rows, at most one CTA per SM and query group

// one row's latent, key part and gates, by the whole block: [norm(latent) * w | rotated part | zeros] to the state
template <class A>
__device__ __forceinline__ void append_row(const LatentArgs& a, uint32_t r, uint32_t pos, float* part) {
    typedef typename A::T T;
    const T* y = (const T*)a.y + (size_t)r * a.y_cols();
    const T* lat = y + a.col_lat();
    float ss = 0.0f;
    for (uint32_t i = threadIdx.x; i < a.rank; i += blockDim.x) { const float v = A::ld(lat + i); ss = fmaf(v, v, ss); }
    ss = block_sum(ss, part);
    const float inv = 1.0f / sqrtf(ss / (float)a.rank + a.eps);
    T* dst = (T*)a.state + (size_t)pos * a.ls();
    for (uint32_t i = threadIdx.x; i < a.rank; i += blockDim.x) A::st(dst + i, A::ld(lat + i) * inv * __ldg(a.norm_w + i));
    const float2* tab = (const float2*)a.rope + (size_t)pos * (a.rot / 2);
    for (uint32_t i = threadIdx.x; i < a.rot / 2; i += blockDim.x) {
        const float2 cs = __ldg(tab + i);
        const float u = A::ld(lat + a.rank + 2 * i), v = A::ld(lat + a.rank + 2 * i + 1);
        A::st(dst + a.rank + 2 * i, u * cs.x - v * cs.y);
        A::st(dst + a.rank + 2 * i + 1, v * cs.x + u * cs.y);
    }
    for (uint32_t i = a.rank + a.rot + threadIdx.x; i < a.ls(); i += blockDim.x) A::st(dst + i, 0.0f);
    for (uint32_t h = threadIdx.x; h < a.heads; h += blockDim.x) a.gate[(size_t)r * a.heads + h] = sigmoid_f(A::ld(y + a.col_gate() + h));
}

template <class A>
__global__ void __launch_bounds__(256)
latent_append_kernel(const LatentArgs a) {
    __shared__ float part[8];
    typedef typename A::T T;
    pdl_release();
    pdl_wait();
    const uint32_t r = blockIdx.x, pos = *a.counter + r;
    if (pos >= a.nslots) return;                    // the host has checked the room
    append_row<A>(a, r, pos, part);
    const T* y = (const T*)a.y + (size_t)r * a.y_cols();
    const uint32_t hd = a.dim + a.rot, half = a.rot / 2;
    T* q = (T*)a.q + (size_t)r * a.heads * hd;
    for (uint32_t i = threadIdx.x; i < a.heads * a.dim; i += 256) {
        const uint32_t h = i / a.dim, d = i % a.dim;
        q[h * hd + d] = __ldcg(y + h * hd + d);
    }
    const float2* tab = (const float2*)a.rope + (size_t)pos * half;
    for (uint32_t i = threadIdx.x; i < a.heads * half; i += 256) {
        const uint32_t h = i / half, p = i % half, at = h * hd + a.dim + 2 * p;
        const float2 cs = __ldg(tab + p);
        const float u = A::ld(y + at), v = A::ld(y + at + 1);
        A::st(q + at, u * cs.x - v * cs.y);
        A::st(q + at + 1, v * cs.x + u * cs.y);
    }
}

// Plain attention of one (row, head): the query through the key up-projection, scores against the cached rows, running
// softmax over blocks of 128 keys, the weighted latent through the value up-projection. Dynamic shared memory:
// [rank + rot] query, [rank] latent, fp32.
template <class A>
__global__ void __launch_bounds__(128)
latent_exact_kernel(const LatentArgs a) {
    extern __shared__ float sm[];
    __shared__ float p[128], part[4];
    typedef typename A::T T;
    pdl_release();
    pdl_wait();
    const uint32_t h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x;
    const uint32_t n = *a.counter + r + 1, hd = a.dim + a.rot, ls = a.ls();
    float *qa = sm, *ctx = sm + a.rank + a.rot;
    const T* q = (const T*)a.q + ((size_t)r * a.heads + h) * hd;
    for (uint32_t c = tid; c < a.rank; c += 128) {
        float s = 0.0f;
        const uint16_t* w = a.w_kv + (size_t)h * a.dim * a.rank + c;
        for (uint32_t d = 0; d < a.dim; d++) s = fmaf(A::ld(q + d), bf2f(__ldg(w + (size_t)d * a.rank)), s);
        qa[c] = s;
        ctx[c] = 0.0f;
    }
    for (uint32_t c = tid; c < a.rot; c += 128) qa[a.rank + c] = A::ld(q + a.dim + c);
    __syncthreads();
    float m = -INFINITY, l = 0.0f;
    for (uint32_t j0 = 0; j0 < n; j0 += 128) {
        const uint32_t j = j0 + tid;
        float s = -INFINITY;
        if (j < n) {
            const T* row = (const T*)a.state + (size_t)j * ls;
            float acc = 0.0f;
            for (uint32_t c = 0; c < a.rank + a.rot; c++) acc = fmaf(qa[c], A::ld(row + c), acc);
            s = acc * a.scale;
        }
        float bm = warp_max(s);
        __syncthreads();
        if ((tid & 31) == 0) part[tid >> 5] = bm;
        __syncthreads();
        bm = fmaxf(fmaxf(part[0], part[1]), fmaxf(part[2], part[3]));
        const float mn = fmaxf(m, bm), corr = expf(m - mn), e = expf(s - mn);
        p[tid] = e;
        l = l * corr + block_sum(e, part);
        m = mn;
        const uint32_t cnt = min(128u, n - j0);
        for (uint32_t c = tid; c < a.rank; c += 128) {
            float o = ctx[c] * corr;
            const T* col = (const T*)a.state + (size_t)j0 * ls + c;
            for (uint32_t k = 0; k < cnt; k++) o = fmaf(p[k], A::ld(col + (size_t)k * ls), o);
            ctx[c] = o;
        }
    }
    __syncthreads();
    const float g = a.gate[(size_t)r * a.heads + h] / l;
    const uint32_t warp = tid >> 5, lane = tid & 31;
    T* out = (T*)a.out + ((size_t)r * a.heads + h) * a.vdim;
    for (uint32_t v = warp; v < a.vdim; v += 4) {
        const uint16_t* w = a.w_kv + ((size_t)a.heads * a.dim + (size_t)h * a.vdim + v) * a.rank;
        float s = 0.0f;
        for (uint32_t c = lane; c < a.rank; c += 32) s = fmaf(ctx[c], bf2f(__ldg(w + c)), s);
        s = warp_sum(s);
        if (lane == 0) A::st(out + v, s * g);
    }
}

// Few rows: q of every head into latent space, times the score scale, stored as hi + lo bf16 rows like the cached ones.
// Grid (heads + 1, ceil(rank / 64), ceil(rows / AR)), AR = 1 or 8; the CTAs of column block 0 add the rotated q part (and the zero
// tail), the CTAs of x = heads append the latents.
constexpr int kAbsorbTile = 8;
template <int AR>
__global__ void __launch_bounds__(256)
latent_absorb_kernel(const LatentArgs a, uint16_t* __restrict__ qh, uint16_t* __restrict__ ql, uint32_t rows) {
    extern __shared__ float sq[];                  // [AR][dim]
    __shared__ float red[8][AR][64 + 2];
    __shared__ float part[8];
    pdl_release();
    const uint32_t tid = threadIdx.x, h = blockIdx.x, r0 = blockIdx.z * AR, nr = AR == 1 ? 1u : min((uint32_t)AR, rows - r0);
    const uint16_t* yb = (const uint16_t*)a.y;
    if (h == a.heads) {
        pdl_wait();
        if (blockIdx.y) return;
        const uint32_t base = *a.counter;
        for (uint32_t r = 0; r < nr; r++)
            if (base + r0 + r < a.nslots) append_row<ActBf16>(a, r0 + r, base + r0 + r, part);
        return;
    }
    const uint32_t hd = a.dim + a.rot, ls = a.ls(), yc = a.y_cols();
    const uint32_t c0 = blockIdx.y * 64, cp = tid & 31, ds = tid >> 5;      // column pair, share of dim
    const uint32_t c = c0 + 2 * cp;
    const uint16_t* w = a.w_kv + (size_t)h * a.dim * a.rank + c;
    const bool pair = (a.rank & 1u) == 0;
    auto put = [&](size_t i, float v) {
        v *= a.scale;
        const uint16_t hi = f2bf(v);
        qh[i] = hi;
        ql[i] = f2bf(v - bf2f(hi));
    };
    // this thread's first weights are requested before the wait
    uint32_t wv[16];
    auto loadw = [&](uint32_t d) -> uint32_t {
        if (d >= a.dim || c >= a.rank) return 0u;
        const uint16_t* s = w + (size_t)d * a.rank;
        if (pair) return __ldg((const uint32_t*)s);
        return (uint32_t)__ldg(s) | (c + 1 < a.rank ? (uint32_t)__ldg(s + 1) << 16 : 0u);
    };
#pragma unroll
    for (int u = 0; u < 16; u++) wv[u] = loadw(ds + 8 * u);
    pdl_wait();
    for (uint32_t i = tid; i < nr * a.dim; i += 256) sq[i] = bf2f(__ldcg(yb + (size_t)(r0 + i / a.dim) * yc + h * hd + i % a.dim));
    if (blockIdx.y == 0) {
        const uint32_t base = *a.counter, half = a.rot / 2;
        for (uint32_t i = tid; i < nr * half; i += 256) {
            const uint32_t r = i / half, p = i % half;
            if (base + r0 + r >= a.nslots) continue;
            const float2 cs = __ldg((const float2*)a.rope + (size_t)(base + r0 + r) * half + p);
            const uint16_t* s = yb + (size_t)(r0 + r) * yc + h * hd + a.dim + 2 * p;
            const float u = bf2f(__ldcg(s)), v = bf2f(__ldcg(s + 1));
            put(((size_t)(r0 + r) * a.heads + h) * ls + a.rank + 2 * p, u * cs.x - v * cs.y);
            put(((size_t)(r0 + r) * a.heads + h) * ls + a.rank + 2 * p + 1, v * cs.x + u * cs.y);
        }
        const uint32_t tail = ls - a.rank - a.rot;
        for (uint32_t i = tid; i < nr * tail; i += 256)
            put(((size_t)(r0 + i / tail) * a.heads + h) * ls + a.rank + a.rot + i % tail, 0.0f);
    }
    __syncthreads();
    float acc[AR][2];
#pragma unroll
    for (int r = 0; r < AR; r++) acc[r][0] = acc[r][1] = 0.0f;
    for (uint32_t d0 = ds; d0 < a.dim; d0 += 128) {
        if (d0 != ds) {
#pragma unroll
            for (int u = 0; u < 16; u++) wv[u] = loadw(d0 + 8 * u);
        }
#pragma unroll
        for (int u = 0; u < 16; u++) {
            const uint32_t d = d0 + 8 * u;
            if (d >= a.dim) break;
            const float w0 = bf2f((uint16_t)(wv[u] & 0xffffu)), w1 = bf2f((uint16_t)(wv[u] >> 16));
#pragma unroll
            for (int r = 0; r < AR; r++) {
                if (AR > 1 && r >= (int)nr) break;
                const float q = sq[r * a.dim + d];
                acc[r][0] = fmaf(q, w0, acc[r][0]);
                acc[r][1] = fmaf(q, w1, acc[r][1]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < AR; r++) { red[ds][r][2 * cp] = acc[r][0]; red[ds][r][2 * cp + 1] = acc[r][1]; }
    __syncthreads();
    for (uint32_t i = tid; i < nr * 64; i += 256) {
        const uint32_t r = i / 64, k = i % 64;
        if (c0 + k >= a.rank) continue;
        float s = 0.0f;
#pragma unroll
        for (int j = 0; j < 8; j++) s += red[j][r][k];
        put(((size_t)(r0 + r) * a.heads + h) * ls + c0 + k, s);
    }
}

// Attention of 16 * QT (row, head) pairs against one slice of the cached rows. Tiles of 32 positions, two stages.
//   scores   every warp takes an eighth of the latent for all pairs and positions of the tile, so that each operand
//            fragment is read from shared memory once; q as hi + lo bf16
//   softmax  the eight shares added, a warp per 2 * QT pairs, lane = position; weights to shared memory as hi + lo bf16
//   values   each warp 8 * NT latent columns, accumulators in registers
// Partial result per pair and slice: latent [rank], maximum, sum.
constexpr int TP = 32, STG = 2;
template <int NT, int QT>
__global__ void __launch_bounds__(256)
latent_split_kernel(const LatentArgs a, const uint16_t* qh, const uint16_t* ql, float* part_o, float* part_ml, uint32_t rows) {
    extern __shared__ __align__(16) unsigned char smem[];
    constexpr int M = 16 * QT;
    const uint32_t ls = a.ls(), rs = ls + 8;                          // padded rows: 16-byte chunks of 8 rows fall into different banks
    uint16_t* sk = (uint16_t*)smem;                                   // [STG][TP][rs]
    uint16_t* sqh = sk + STG * TP * rs;                               // [M][rs] hi, then lo
    uint16_t* sql = sqh + M * rs;
    float* ss = (float*)(sql + M * rs);                               // [8][M][TP + 1] scores by share of the latent
    uint16_t* sph = (uint16_t*)(ss + 8 * M * (TP + 1));               // [M][TP + 8] weights hi, then lo
    uint16_t* spl = sph + M * (TP + 8);
    float* sm_m = (float*)(spl + M * (TP + 8));                       // [M] maximum, sum, correction
    float* sm_l = sm_m + M;
    float* sm_c = sm_l + M;
    pdl_release();
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t pairs = rows * a.heads, p0 = blockIdx.y * M, nsplit = gridDim.x;
    // The position counter moves at the end of a run only, and rows below it were written by earlier runs: tiles that
    // hold none of this run's rows are requested before the dependency wait.
    const uint32_t past = *(volatile const uint32_t*)a.counter, n = min(past + rows, a.nslots);
    const uint32_t tiles = (n + TP - 1) / TP, per = (tiles + nsplit - 1) / nsplit;
    const uint32_t t0 = min(blockIdx.x * per, tiles), t1 = min(t0 + per, tiles);
    const uint16_t* st = (const uint16_t*)a.state;
    const uint32_t ch = ls / 8;
    auto fetch = [&](uint32_t t) {
        if (t >= t1) return;
        uint16_t* d = sk + (t % STG) * TP * rs;
        for (uint32_t r = warp; r < TP; r += 8) {
            const uint32_t pos = t * TP + r;
            const uint16_t* src = st + (size_t)min(pos, n - 1) * ls;
            for (uint32_t c = lane; c < ch; c += 32) cp16(smem_addr(d + r * rs + c * 8), src + c * 8, pos < n ? 16 : 0);
        }
    };
    const bool early0 = (t0 + 1) * TP <= past, early1 = (t0 + 2) * TP <= past;
    if (early0) fetch(t0);
    if (early1) fetch(t0 + 1);
    pdl_wait();
    for (uint32_t r = warp; r < M; r += 8) {
        const bool live = p0 + r < pairs;
        const size_t src = (size_t)(live ? p0 + r : 0) * ls;
        for (uint32_t c = lane; c < ch; c += 32) {
            cp16(smem_addr(sqh + r * rs + c * 8), qh + src + c * 8, live ? 16 : 0);
            cp16(smem_addr(sql + r * rs + c * 8), ql + src + c * 8, live ? 16 : 0);
        }
    }
    if (!early0) fetch(t0);
    cp_commit();
    if (!early1) fetch(t0 + 1);
    cp_commit();
    cp_wait<1>();
    if (tid < M) { sm_m[tid] = -INFINITY; sm_l[tid] = 0.0f; }
    float o[QT][NT][4];
#pragma unroll
    for (int q = 0; q < QT; q++)
#pragma unroll
        for (int i = 0; i < NT; i++)
#pragma unroll
            for (int k = 0; k < 4; k++) o[q][i][k] = 0.0f;
    const uint32_t g = lane >> 2, t4 = lane & 3;
    const uint32_t KS = ls / 16, k_lo = KS * warp / 8, k_hi = KS * (warp + 1) / 8;      // this warp's k steps
    const uint32_t a_row = lane & 15, a_col = (lane >> 4) * 8;        // ldmatrix addresses of an A tile
    for (uint32_t t = t0; t < t1; t++) {
        if (t > t0) cp_wait<0>();
        __syncthreads();                                              // tile t is here; everyone is done with tile t - 1
        if (t > t0) { fetch(t + 1); cp_commit(); }
        const uint16_t* kt = sk + (t % STG) * TP * rs;
        {
            float acc[QT][TP / 8][4] = {};
            const uint32_t kb = smem_addr(kt + ((lane & 7) + (lane >> 4) * 8) * rs + ((lane >> 3) & 1) * 8);
            for (uint32_t ks = k_lo; ks < k_hi; ks++) {
                uint32_t b[TP / 16][4];
#pragma unroll
                for (int j = 0; j < TP / 16; j++) ldsm4(b[j], kb + j * 16 * rs * 2 + ks * 32);        // 16 positions each
#pragma unroll
                for (int q = 0; q < QT; q++) {
                    uint32_t ah[4], al[4];
                    ldsm4(ah, smem_addr(sqh + (q * 16 + a_row) * rs + a_col) + ks * 32);
                    ldsm4(al, smem_addr(sql + (q * 16 + a_row) * rs + a_col) + ks * 32);
#pragma unroll
                    for (int j = 0; j < TP / 16; j++) {
                        mma_bf16(acc[q][2 * j], ah, b[j][0], b[j][1]);
                        mma_bf16(acc[q][2 * j + 1], ah, b[j][2], b[j][3]);
                        mma_bf16(acc[q][2 * j], al, b[j][0], b[j][1]);
                        mma_bf16(acc[q][2 * j + 1], al, b[j][2], b[j][3]);
                    }
                }
            }
#pragma unroll
            for (int q = 0; q < QT; q++)
#pragma unroll
                for (int j = 0; j < TP / 8; j++) {
                    float* d = ss + warp * M * (TP + 1) + (q * 16 + g) * (TP + 1) + j * 8 + 2 * t4;
                    d[0] = acc[q][j][0]; d[1] = acc[q][j][1];
                    d[8 * (TP + 1)] = acc[q][j][2]; d[8 * (TP + 1) + 1] = acc[q][j][3];
                }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2 * QT; i++) {
            const uint32_t r = warp * 2 * QT + i, pos = t * TP + lane;
            const uint32_t row = (p0 + r) / a.heads;
            float s = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; w++) s += ss[w * M * (TP + 1) + r * (TP + 1) + lane];
            if (pos >= n || pos > past + row) s = -INFINITY;
            const float mo = sm_m[r], mn = fmaxf(mo, warp_max(s));
            const float e = mn == -INFINITY ? 0.0f : expf(s - mn);
            const float sum = warp_sum(e);
            const uint16_t hi = f2bf(e);
            sph[r * (TP + 8) + lane] = hi;
            spl[r * (TP + 8) + lane] = f2bf(e - bf2f(hi));
            __syncwarp();
            if (lane == 0) {
                const float corr = mo == -INFINITY ? 0.0f : expf(mo - mn);
                sm_c[r] = corr; sm_m[r] = mn; sm_l[r] = sm_l[r] * corr + sum;
            }
        }
        __syncthreads();
#pragma unroll
        for (int q = 0; q < QT; q++) {
            const float c_lo = sm_c[q * 16 + g], c_hi = sm_c[q * 16 + g + 8];
#pragma unroll
            for (int i = 0; i < NT; i++) { o[q][i][0] *= c_lo; o[q][i][1] *= c_lo; o[q][i][2] *= c_hi; o[q][i][3] *= c_hi; }
        }
#pragma unroll
        for (int ks = 0; ks < TP / 16; ks++) {
            uint32_t ph[QT][4], pl[QT][4];
#pragma unroll
            for (int q = 0; q < QT; q++) {
                ldsm4(ph[q], smem_addr(sph + (q * 16 + a_row) * (TP + 8) + ks * 16 + a_col));
                ldsm4(pl[q], smem_addr(spl + (q * 16 + a_row) * (TP + 8) + ks * 16 + a_col));
            }
#pragma unroll
            for (int i = 0; i < NT; i += 2) {
                const uint32_t c = warp * 8 * NT + i * 8;
                if (c >= a.rank) continue;
                uint32_t b[4];
                ldsm4_t(b, smem_addr(kt + (ks * 16 + (lane & 15)) * rs + c + (lane >> 4) * 8));
#pragma unroll
                for (int q = 0; q < QT; q++) {
                    mma_bf16(o[q][i], ph[q], b[0], b[1]);
                    mma_bf16(o[q][i], pl[q], b[0], b[1]);
                    mma_bf16(o[q][i + 1], ph[q], b[2], b[3]);
                    mma_bf16(o[q][i + 1], pl[q], b[2], b[3]);
                }
            }
        }
    }
    cp_wait<0>();
    __syncthreads();
#pragma unroll
    for (int q = 0; q < QT; q++) {
#pragma unroll
        for (int hf = 0; hf < 2; hf++) {
            const uint32_t pr = p0 + q * 16 + g + hf * 8;
            if (pr >= pairs) continue;
            float* d = part_o + ((size_t)pr * nsplit + blockIdx.x) * a.rank;
#pragma unroll
            for (int i = 0; i < NT; i++) {
                const uint32_t c = warp * 8 * NT + i * 8 + 2 * t4;
                if (c < a.rank) d[c] = o[q][i][2 * hf];
                if (c + 1 < a.rank) d[c + 1] = o[q][i][2 * hf + 1];
            }
        }
    }
    if (tid < M && p0 + tid < pairs) {
        float* d = part_ml + ((size_t)(p0 + tid) * nsplit + blockIdx.x) * 2;
        d[0] = sm_m[tid]; d[1] = sm_l[tid];
    }
}

// Slices of one (row, head) pair combined, value up-projection, gate. A cluster of 8 CTAs per pair: each combines an
// eighth of the latent columns (a column by 4 threads, a quarter of the slices each), the pieces meet through
// distributed shared memory, then each CTA computes an eighth of the values.
constexpr uint32_t MC = 8, MCOLS = 64;
__global__ void __launch_bounds__(256)
latent_merge_kernel(const LatentArgs a, const float* part_o, const float* part_ml, uint32_t nsplit) {
    __shared__ float sw[kMaxSplit], red[8], quarter[4][MCOLS], ctx[MC * MCOLS];
    cooperative_groups::cluster_group cl = cooperative_groups::this_cluster();
    cluster_arrive();                                  // paired with the wait in front of the first remote store
    const uint32_t pr = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = pr % a.heads, part = blockIdx.y;
    // the weights of this CTA's first 8 values (one per warp) are requested before the wait
    const uint32_t vper = (a.vdim + MC - 1) / MC, v0 = part * vper, v1 = min(v0 + vper, a.vdim);
    const bool vec = (a.rank & 7u) == 0;
    auto wrow = [&](uint32_t v) { return a.w_kv + ((size_t)a.heads * a.dim + (size_t)h * a.vdim + v) * a.rank; };
    uint4 w0[2];
#pragma unroll
    for (int u = 0; u < 2; u++) {
        const uint32_t c = lane * 8 + u * 256;
        w0[u] = vec && v0 + warp < v1 && c < a.rank ? __ldg((const uint4*)(wrow(v0 + warp) + c)) : make_uint4(0, 0, 0, 0);
    }
    pdl_wait();
    pdl_release();          // after the wait, like the merge of the KV-ring attention
    // nsplit <= kMaxSplit: one slice per thread here, at most kMaxSplit / 4 slices of a column per thread below; the
    // partial latents are requested before the weights are known
    const float2 ml = tid < nsplit ? __ldcg((const float2*)part_ml + (size_t)pr * nsplit + tid) : make_float2(-INFINITY, 0.0f);
    const uint32_t cper = (a.rank + MC - 1) / MC, c = part * cper + tid % MCOLS, q = tid / MCOLS;     // cper <= MCOLS
    const bool live = tid % MCOLS < cper && c < a.rank;
    const float* po = part_o + (size_t)pr * nsplit * a.rank + c;
    float v[kMaxSplit / 4];
#pragma unroll
    for (int i = 0; i < (int)kMaxSplit / 4; i++) {
        const uint32_t s = q + 4 * i;
        v[i] = live && s < nsplit ? __ldcg(po + (size_t)s * a.rank) : 0.0f;
    }
    float m = warp_max(ml.x);
    if (lane == 0) red[warp] = m;
    __syncthreads();
#pragma unroll
    for (int w = 0; w < 8; w++) m = fmaxf(m, red[w]);
    const float wt = ml.y > 0.0f ? expf(ml.x - m) : 0.0f;          // an empty slice has sum 0 (and a zero latent)
    if (tid < kMaxSplit) sw[tid] = wt;
    const float l = block_sum(wt * ml.y, red);
    {
        float o = 0.0f;
#pragma unroll
        for (int i = 0; i < (int)kMaxSplit / 4; i++) o = fmaf(sw[q + 4 * i], v[i], o);
        quarter[q][tid % MCOLS] = o;
        __syncthreads();
        cluster_wait();                                // every CTA of the cluster has started
        if (tid < cper && part * cper + tid < a.rank) {
            const float sum = (quarter[0][tid] + quarter[1][tid]) + (quarter[2][tid] + quarter[3][tid]);
            for (uint32_t k = 0; k < MC; k++) *cl.map_shared_rank(ctx + part * cper + tid, k) = sum;
        }
    }
    cl.sync();
    const float gt = a.gate[pr] / l;
    uint16_t* out = (uint16_t*)a.out + (size_t)pr * a.vdim;
    for (uint32_t v = v0 + warp; v < v1; v += 8) {
        const uint16_t* w = wrow(v);
        float s = 0.0f;
        if (vec) {
#pragma unroll
            for (int u = 0; u < 2; u++) {
                const uint32_t c = lane * 8 + u * 256;
                if (c >= a.rank) break;
                const uint4 q = v == v0 + warp ? w0[u] : __ldg((const uint4*)(w + c));
                const uint32_t x[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                for (int k = 0; k < 4; k++) {
                    s = fmaf(ctx[c + 2 * k], bf2f((uint16_t)(x[k] & 0xffffu)), s);
                    s = fmaf(ctx[c + 2 * k + 1], bf2f((uint16_t)(x[k] >> 16)), s);
                }
            }
        } else {
            for (uint32_t c = lane; c < a.rank; c += 32) s = fmaf(ctx[c], bf2f(__ldg(w + c)), s);
        }
        s = warp_sum(s);
        if (lane == 0) out[v] = f2bf(s * gt);
    }
}

size_t split_smem(uint32_t ls, int qt) {
    const size_t M = 16 * qt, rs = ls + 8;
    return STG * TP * rs * 2 + 2 * M * rs * 2 + 8 * M * (TP + 1) * 4 + 2 * M * (TP + 8) * 2 + 3 * M * 4;
}

struct SplitPlan { uint32_t nt, qt, groups, nsplit; };
// false: a latent the split kernel does not take
bool split_plan(const LatentArgs& a, uint32_t rows, SplitPlan& s) {
    const uint32_t pairs = rows * a.heads;
    if (!a.bf16 || a.rank > 512 || a.dim > 512) return false;
    s.nt = a.rank <= 128 ? 2 : a.rank <= 256 ? 4 : 8;
    s.qt = pairs > 16 && split_smem(a.ls(), 2) <= 220 * 1024 ? 2 : 1;
    if (split_smem(a.ls(), (int)s.qt) > 220 * 1024) return false;
    s.groups = (pairs + 16 * s.qt - 1) / (16 * s.qt);
    const uint32_t tiles = (a.nslots + TP - 1) / TP;
    s.nsplit = kMaxSplit / s.groups;
    if (s.nsplit > (tiles + 1) / 2) s.nsplit = (tiles + 1) / 2;
    if (s.nsplit < 1) s.nsplit = 1;
    return true;
}

template <int NT, int QT>
bool launch_split(cudaStream_t st, const LatentArgs& a, const uint16_t* qh, const uint16_t* ql, float* po, float* pml, uint32_t rows, const SplitPlan& s) {
    static int have[64] = {};
    const size_t smem = split_smem(a.ls(), QT);
    if (!ensure_dyn_smem(latent_split_kernel<NT, QT>, smem, have)) return false;
    launch_pdl(latent_split_kernel<NT, QT>, dim3(s.nsplit, s.groups), dim3(256), smem, st, a, qh, ql, po, pml, rows);
    g_launches++;
    return true;
}

// floats: absorbed queries, partial latents, maxima and sums
size_t step_floats(const LatentArgs& a, uint32_t rows) {
    SplitPlan s;
    if (!split_plan(a, rows, s)) return 0;
    const size_t pairs = (size_t)rows * a.heads;
    return pairs * a.ls() + ((pairs * s.nsplit * a.rank + 3) & ~(size_t)3) + pairs * s.nsplit * 2;
}

}  // namespace

size_t latent_prefill_floats(const LatentArgs& a, uint32_t max_rows);
bool k_latent_prefill(cudaStream_t st, const LatentArgs& a, uint32_t rows, uint32_t n_past);

size_t latent_work_floats(const LatentArgs& a, uint32_t max_rows) {
    size_t n = 4;
    for (uint32_t r = 1; r <= kAbsorbRows && r <= max_rows; r++) { const size_t f = step_floats(a, r); n = f > n ? f : n; }
    const size_t p = latent_prefill_floats(a, max_rows);
    return p > n ? p : n;
}

void k_latent_append(cudaStream_t st, const LatentArgs& a, uint32_t rows) {
    if (!rows) return;
    if (a.bf16) launch_pdl(latent_append_kernel<ActBf16>, dim3(rows), dim3(256), 0, st, a);
    else launch_pdl(latent_append_kernel<ActF32>, dim3(rows), dim3(256), 0, st, a);
    g_launches++;
}

void k_latent_attend(cudaStream_t st, const LatentArgs& a, uint32_t rows, uint32_t n_past, bool exact) {
    if (!rows) return;
    if (a.bf16 && !exact && k_latent_prefill(st, a, rows, n_past)) return;
    const size_t smem = (size_t)(2 * a.rank + a.rot) * 4;
    static int have_b[64] = {}, have_f[64] = {};
    if (a.bf16) {
        if (smem > 40 * 1024) ensure_dyn_smem(latent_exact_kernel<ActBf16>, smem, have_b);
        launch_pdl(latent_exact_kernel<ActBf16>, dim3(a.heads, rows), dim3(128), smem, st, a);
    } else {
        if (smem > 40 * 1024) ensure_dyn_smem(latent_exact_kernel<ActF32>, smem, have_f);
        launch_pdl(latent_exact_kernel<ActF32>, dim3(a.heads, rows), dim3(128), smem, st, a);
    }
    g_launches++;
}

bool k_latent_step(cudaStream_t st, const LatentArgs& a, uint32_t rows) {
    SplitPlan s;
    if (!rows || rows > kAbsorbRows || !split_plan(a, rows, s)) return false;
    const size_t pairs = (size_t)rows * a.heads;
    uint16_t *qh = (uint16_t*)a.work, *ql = qh + pairs * a.ls();      // rows of a multiple of 16 elements
    float* po = a.work + pairs * a.ls();
    float* pml = po + ((pairs * s.nsplit * a.rank + 3) & ~(size_t)3);
    const dim3 ag(a.heads + 1, (a.rank + 63) / 64, rows == 1 ? 1 : (rows + kAbsorbTile - 1) / kAbsorbTile);
    if (rows == 1) launch_pdl(latent_absorb_kernel<1>, ag, dim3(256), (size_t)a.dim * 4, st, a, qh, ql, rows);
    else launch_pdl(latent_absorb_kernel<kAbsorbTile>, ag, dim3(256), (size_t)kAbsorbTile * a.dim * 4, st, a, qh, ql, rows);
    g_launches++;
    bool ok;
    switch (s.nt * 10 + s.qt) {
    case 21: ok = launch_split<2, 1>(st, a, qh, ql, po, pml, rows, s); break;
    case 22: ok = launch_split<2, 2>(st, a, qh, ql, po, pml, rows, s); break;
    case 41: ok = launch_split<4, 1>(st, a, qh, ql, po, pml, rows, s); break;
    case 42: ok = launch_split<4, 2>(st, a, qh, ql, po, pml, rows, s); break;
    case 81: ok = launch_split<8, 1>(st, a, qh, ql, po, pml, rows, s); break;
    default: ok = launch_split<8, 2>(st, a, qh, ql, po, pml, rows, s); break;
    }
    if (!ok) return false;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((uint32_t)pairs, MC); cfg.blockDim = dim3(256); cfg.stream = st;
    if (launch_pdl_cluster(latent_merge_kernel, cfg, dim3(1, MC, 1), a, (const float*)po, (const float*)pml, s.nsplit) != cudaSuccess) { cudaGetLastError(); return false; }
    g_launches++;
    return true;
}

}  // namespace gehtp
