// Grouped-query attention over a window of positions (OP_HEADS_APPEND, OP_WINDOW_ATTEND). A state row holds the keys,
// then the values, of one position for every key head; the state is a ring of rows, position p in row p mod ring.
//
//   heads_append_kernel   norm and rotation of q and k per head, k | v to the ring
//   window_exact_kernel   plain attention, fp32 throughout: one CTA per (head, row), any size
//   window_step_kernel    few bf16 rows: a cluster of CTAs per (key head, row) shares the window out, the partial results
//                         meet through distributed shared memory; for one row the append is part of it
//   more bf16 rows        window_attn_sm100.cu, window_prefill.cu
#include <cooperative_groups.h>
#include "launchers_rows.h"
#include "mma_bf16.cuh"

namespace gehtp {

namespace {

constexpr uint32_t kStepRows = 8;

// One head of one row by one warp: RMS norm (nw = 0: none), then the first `rot` components turned, i with i + rot / 2.
// The result goes to out(i, value of i, value of i + 1) for even i (the second value past an odd dim is to be ignored);
// buf: dim + 1 floats of shared memory of this warp.
template <class A, class F>
__device__ __forceinline__ void head_row(const typename A::T* src, uint32_t dim, const float* nw, const float2* rope, uint32_t rot, float eps,
                                         float* buf, F&& out) {
    const uint32_t lane = threadIdx.x & 31, half = rot / 2;
    float ss = 0.0f;
    float2 early[2];                               // constants, on their way while the row is summed
#pragma unroll
    for (int u = 0; u < 2; u++) early[u] = lane + 32 * u < half ? __ldg(rope + lane + 32 * u) : make_float2(0.f, 0.f);
    if (sizeof(typename A::T) == 2 && ((dim | (uint32_t)((uintptr_t)src >> 1)) & 1u) == 0) {
        for (uint32_t i = 2 * lane; i < dim; i += 64) {
            const uint32_t w = __ldcg((const uint32_t*)(src + i));
            const float a = __uint_as_float(w << 16), b = __uint_as_float(w & 0xffff0000u);
            buf[i] = a;
            buf[i + 1] = b;
            ss = fmaf(a, a, fmaf(b, b, ss));
        }
    } else {
        for (uint32_t i = lane; i < dim; i += 32) {
            const float a = A::ld(src + i);
            buf[i] = a;
            ss = fmaf(a, a, ss);
        }
    }
    const float inv = nw ? 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps) : 1.0f;
    __syncwarp();
    auto val = [&](uint32_t i) { return nw ? buf[i] * inv * __ldg(nw + i) : buf[i]; };
    for (uint32_t i = lane; i < half; i += 32) {
        const float2 cs = i < 32 ? early[0] : i < 64 ? early[1] : __ldg(rope + i);
        const float u = val(i), v = val(i + half);
        buf[i] = u * cs.x - v * cs.y;
        buf[i + half] = v * cs.x + u * cs.y;
    }
    for (uint32_t i = rot + lane; i < dim; i += 32) buf[i] = val(i);
    __syncwarp();
    for (uint32_t i = 2 * lane; i < dim; i += 64) out(i, buf[i], buf[i + 1]);
    __syncwarp();
}

template <class A>
__device__ __forceinline__ void put_pair(typename A::T* dst, uint32_t i, uint32_t dim, float a, float b) {
    if (sizeof(typename A::T) == 2 && i + 1 < dim && ((uintptr_t)(dst + i) & 3u) == 0) *(uint32_t*)(dst + i) = pack_bf2(a, b);
    else {
        A::st(dst + i, a);
        if (i + 1 < dim) A::st(dst + i + 1, b);
    }
}

// a warp per row and head (queries, then keys, then values); dynamic shared memory: [8][dim + 1] floats
template <class A>
__global__ void __launch_bounds__(256)
heads_append_kernel(const WindowArgs a) {
    extern __shared__ float sm[];
    typedef typename A::T T;
    pdl_release();
    const uint32_t r = blockIdx.x, pos = *(volatile const uint32_t*)a.counter + r, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t h = blockIdx.y * 8 + warp;
    pdl_wait();
    if (pos >= a.positions || h >= a.heads + 2 * a.kv_heads) return;            // the host has checked the room
    const T* y = (const T*)a.y + (size_t)r * a.y_cols;
    T* dst = (T*)a.state + (size_t)(pos % a.ring) * a.row();
    if (h >= a.heads + a.kv_heads) {
        const uint32_t g = h - a.heads - a.kv_heads;
        const T* v = y + a.col_v() + g * a.vdim;
        T* to = dst + a.kv_heads * a.dim + g * a.vdim;
        if (a.vdim % 8 == 0 && (((uintptr_t)v | (uintptr_t)to) & 15u) == 0)
            for (uint32_t i = lane; i < a.vdim * sizeof(T) / 16; i += 32) ((uint4*)to)[i] = __ldcg((const uint4*)v + i);
        else
            for (uint32_t i = lane; i < a.vdim; i += 32) to[i] = __ldcg(v + i);
        return;
    }
    const bool key = h >= a.heads;
    const uint32_t k = h - a.heads;
    T* to = key ? dst + k * a.dim : (T*)a.q + ((size_t)r * a.heads + h) * a.dim;
    head_row<A>(key ? y + a.col_k() + k * a.dim : y + h * a.dim, a.dim, a.norms ? a.norms + (key ? a.dim : 0) : nullptr,
                (const float2*)a.rope + (size_t)pos * (a.rot / 2), a.rot, a.eps, sm + warp * (a.dim + 1),
                [&](uint32_t i, float u, float v) { put_pair<A>(to, i, a.dim, u, v); });
}

// Eight neighbouring components of one head of LP * 8, a lane each: norm, then the first `rot` components turned; rotation
// partners lie rot / 16 lanes apart. The constants are fetched on construction, ahead of the data.
template <int LP>
struct HeadVec {
    float nw[8], cs[8], sn[8];
    uint32_t mate;
    bool norm;
    __device__ __forceinline__ HeadVec(bool live, uint32_t c, const float* norms, const float* rope, uint32_t pos, uint32_t rot) {
        const uint32_t hl = rot / 16, lane = threadIdx.x & 31;
        norm = norms != nullptr;
        mate = c < hl ? lane + hl : c < 2 * hl ? lane - hl : lane;
#pragma unroll
        for (int i = 0; i < 8; i++) { nw[i] = 1.0f; cs[i] = 1.0f; sn[i] = 0.0f; }
        if (!live) return;
        if (norms) {
            const float4* n = (const float4*)(norms + c * 8);
            const float4 n0 = __ldg(n), n1 = __ldg(n + 1);
            nw[0] = n0.x; nw[1] = n0.y; nw[2] = n0.z; nw[3] = n0.w; nw[4] = n1.x; nw[5] = n1.y; nw[6] = n1.z; nw[7] = n1.w;
        }
        if (c < 2 * hl) {                          // the second half of the pairs turns with the other sign
            const float4* t = (const float4*)((const float2*)rope + (size_t)pos * (rot / 2) + (c < hl ? c : c - hl) * 8);
            const float f = c < hl ? -1.0f : 1.0f;
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const float4 q = __ldg(t + i);
                cs[2 * i] = q.x; sn[2 * i] = f * q.y; cs[2 * i + 1] = q.z; sn[2 * i + 1] = f * q.w;
            }
        }
    }
    // every lane of the warp takes part
    __device__ __forceinline__ uint4 turn(uint4 w, float eps) const {
        const uint32_t ww[4] = {w.x, w.y, w.z, w.w};
        float x[8], o[8], ss = 0.0f;
#pragma unroll
        for (int i = 0; i < 4; i++) { x[2 * i] = __uint_as_float(ww[i] << 16); x[2 * i + 1] = __uint_as_float(ww[i] & 0xffff0000u); }
#pragma unroll
        for (int i = 0; i < 8; i++) ss = fmaf(x[i], x[i], ss);
#pragma unroll
        for (int d = LP / 2; d > 0; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
        const float inv = norm ? 1.0f / sqrtf(ss / (float)(LP * 8) + eps) : 1.0f;
#pragma unroll
        for (int i = 0; i < 8; i++) {
            x[i] = x[i] * inv * nw[i];
            o[i] = fmaf(__shfl_sync(0xffffffffu, x[i], mate), sn[i], x[i] * cs[i]);
        }
        return make_uint4(pack_bf2(o[0], o[1]), pack_bf2(o[2], o[3]), pack_bf2(o[4], o[5]), pack_bf2(o[6], o[7]));
    }
};

// sizes and alignment the 8-component form takes
bool head_vec(const WindowArgs& a) {
    const uint32_t lp = a.dim / 8;
    const uintptr_t al = (uintptr_t)a.y | (uintptr_t)a.q | (uintptr_t)a.state | (uintptr_t)a.norms | (uintptr_t)a.rope;
    return a.bf16 && a.dim % 8 == 0 && (lp == 8 || lp == 16 || lp == 32) && a.rot % 16 == 0 && a.vdim % 8 == 0 && a.y_cols % 8 == 0 && (al & 15u) == 0;
}

// heads_append_kernel for such heads: a thread per 8 components; grid (rows, items / 256)
template <int LP>
__global__ void __launch_bounds__(256)
heads_append_vec_kernel(const WindowArgs a) {
    pdl_release();
    const uint32_t r = blockIdx.x, pos = *(volatile const uint32_t*)a.counter + r, item = blockIdx.y * 256 + threadIdx.x;
    const uint32_t nq = (a.heads + a.kv_heads) * LP, nv = a.kv_heads * (a.vdim / 8), h = item / LP, c = item % LP;
    const bool head = item < nq, key = h >= a.heads, live = item < nq + nv && pos < a.positions;
    const uint32_t v = item - nq;
    const uint16_t* y = (const uint16_t*)a.y + (size_t)r * a.y_cols;
    uint16_t* dst = (uint16_t*)a.state + (size_t)(pos % a.ring) * a.row();
    const uint16_t* src = !head ? y + a.col_v() + v * 8 : key ? y + a.col_k() + (h - a.heads) * LP * 8 + c * 8 : y + h * LP * 8 + c * 8;
    uint16_t* to = !head ? dst + a.kv_heads * LP * 8 + v * 8 : key ? dst + (h - a.heads) * LP * 8 + c * 8 : (uint16_t*)a.q + ((size_t)r * a.heads + h) * LP * 8 + c * 8;
    const HeadVec<LP> hv(live && head, c, a.norms ? a.norms + (key ? LP * 8 : 0) : nullptr, a.rope, pos, a.rot);
    pdl_wait();
    const uint4 w = live ? __ldcg((const uint4*)src) : make_uint4(0, 0, 0, 0);
    const uint4 o = hv.turn(w, a.eps);
    if (live) *(uint4*)to = head ? o : w;
}

// Attention of one (head, row): running softmax over blocks of 128 keys. Dynamic shared memory: [dim] query, [vdim] sums.
template <class A>
__global__ void __launch_bounds__(128)
window_exact_kernel(const WindowArgs a) {
    extern __shared__ float sm[];
    __shared__ float p[128], part[4];
    typedef typename A::T T;
    pdl_release();
    pdl_wait();
    const uint32_t h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x, g = h / (a.heads / a.kv_heads);
    const uint32_t pos = *a.counter + r, first = pos + 1 > a.window ? pos + 1 - a.window : 0, row = a.row();
    float *q = sm, *ctx = sm + a.dim;
    const T* qs = (const T*)a.q + ((size_t)r * a.heads + h) * a.dim;
    for (uint32_t c = tid; c < a.dim; c += 128) q[c] = A::ld(qs + c);
    for (uint32_t c = tid; c < a.vdim; c += 128) ctx[c] = 0.0f;
    __syncthreads();
    const T *keys = (const T*)a.state + g * a.dim, *vals = (const T*)a.state + a.kv_heads * a.dim + g * a.vdim;
    float m = -INFINITY, l = 0.0f;
    for (uint32_t j0 = first; j0 <= pos; j0 += 128) {
        const uint32_t j = j0 + tid;
        float s = -INFINITY;
        if (j <= pos) {
            const T* k = keys + (size_t)(j % a.ring) * row;
            float acc = 0.0f;
            for (uint32_t c = 0; c < a.dim; c++) acc = fmaf(q[c], A::ld(k + c), acc);
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
        const uint32_t cnt = min(128u, pos + 1 - j0);
        for (uint32_t c = tid; c < a.vdim; c += 128) {
            float o = ctx[c] * corr;
            for (uint32_t k = 0; k < cnt; k++) o = fmaf(p[k], A::ld(vals + (size_t)((j0 + k) % a.ring) * row + c), o);
            ctx[c] = o;
        }
    }
    const bool gate = a.gate_col != 0xFFFFFFFFu;
    const T* yg = (const T*)a.y + (size_t)r * a.y_cols + a.gate_col + h * a.vdim;
    T* out = (T*)a.out + ((size_t)r * a.heads + h) * a.vdim;
    for (uint32_t c = tid; c < a.vdim; c += 128) A::st(out + c, ctx[c] / l * (gate ? sigmoid_f(A::ld(yg + c)) : 1.0f));
}

// Up to 16 query heads of one key head and one row against the window. A cluster of CTAs takes one (head group, row);
// tiles of 16 positions go round the warps of the cluster, each warp with two stages of its own in shared memory and a
// running softmax in registers; warps meet in shared memory, CTAs in distributed shared memory. Queries are rows of one
// 16-row MMA tile. APPEND: the row's own key and value come from the projection and are stored to the ring by one CTA.
// Positions below the counter were written by earlier runs and the counter moves at the end of a run only: tiles of such
// positions are requested before the dependency wait.
constexpr uint32_t SP = 16, SW = 8, MAXC = 16;    // positions per tile, warps, CTAs of a cluster at most
template <int VT, bool VEC, bool APPEND, int LP>
__global__ void __launch_bounds__(256)
window_step_kernel(const WindowArgs a, uint32_t stages) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float wm[SW][16], wl[SW][16], cm[16], cl[16];
    cooperative_groups::cluster_group cluster = cooperative_groups::this_cluster();
    const uint32_t dp = (a.dim + 15u) & ~15u, vp = (a.vdim + 15u) & ~15u, rk = dp + 8, rv = vp + 8, row = a.row();
    uint16_t* sq = (uint16_t*)smem;                               // [16][rk]
    uint16_t* snew = sq + 16 * rk;                                // [dp + vp]: this row's key and value
    float* scr = (float*)(snew + dp + vp);                        // [SW][dim + 2]
    uint16_t* tiles = (uint16_t*)(scr + (LP ? 0 : SW * (((a.dim + 2) + 3u) & ~3u)));
    const uint32_t tile_el = SP * (rk + rv);
    float* acc = (float*)tiles;                                   // [SW][16][vp], after the last tile
    pdl_release();
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
    const uint32_t C = gridDim.x, rep = a.heads / a.kv_heads, parts = (rep + 15) / 16;
    const uint32_t g = blockIdx.y / parts, h0 = g * rep + (blockIdx.y % parts) * 16, nh = min(16u, (g + 1) * rep - h0), r = blockIdx.z;
    const uint32_t past = *(volatile const uint32_t*)a.counter, pos = past + r;
    const uint32_t first = pos + 1 > a.window ? pos + 1 - a.window : 0;
    const uint32_t known = APPEND ? pos : pos + 1;                // positions whose rows are in the ring for this row
    const uint32_t t_end = pos / SP + 1, stride = C * SW;
    uint16_t* my = tiles + warp * stages * tile_el;
    const uint16_t *keys = (const uint16_t*)a.state + g * a.dim, *vals = (const uint16_t*)a.state + a.kv_heads * a.dim + g * a.vdim;
    auto fetch = [&](uint32_t t, uint32_t stage) {
        if (t < t_end) {
            uint16_t *k = my + stage * tile_el, *v = k + SP * rk;
            if (VEC) {
                const uint32_t ck = a.dim / 8, cv = a.vdim / 8, j0 = t * SP;
                const size_t src0 = (size_t)(j0 % a.ring) * row;      // a tile does not wrap: the ring is a multiple of it
                for (uint32_t c = lane; c < ck + cv; c += 32) {
                    const uint16_t* src = (c < ck ? keys + c * 8 : vals + (c - ck) * 8) + src0;
                    const uint32_t dst = c < ck ? smem_addr(k + c * 8) : smem_addr(v + (c - ck) * 8), rs = (c < ck ? rk : rv) * 2;
#pragma unroll
                    for (uint32_t p = 0; p < SP; p++) cp16(dst + p * rs, src + (size_t)p * row, j0 + p < known ? 16 : 0);
                }
            } else {
                for (uint32_t i = lane; i < SP * (a.dim + a.vdim); i += 32) {
                    const uint32_t p = i / (a.dim + a.vdim), c = i % (a.dim + a.vdim), j = t * SP + p;
                    const size_t src = (size_t)(j % a.ring) * row;
                    if (c < a.dim) k[p * rk + c] = j < known ? __ldcg(keys + src + c) : (uint16_t)0;
                    else v[p * rv + c - a.dim] = j < known ? __ldcg(vals + src + c - a.dim) : (uint16_t)0;
                }
            }
        }
        if (VEC) cp_commit();
    };
    // columns no copy writes: padding of a head to 16
    if (dp > a.dim || vp > a.vdim) {
        for (uint32_t i = lane; i < stages * SP * (dp - a.dim); i += 32) {
            const uint32_t p = i / (dp - a.dim);
            my[(p / SP) * tile_el + (p % SP) * rk + a.dim + i % (dp - a.dim)] = 0;
        }
        for (uint32_t i = lane; i < stages * SP * (vp - a.vdim); i += 32) {
            const uint32_t p = i / (vp - a.vdim);
            my[(p / SP) * tile_el + SP * rk + (p % SP) * rv + a.vdim + i % (vp - a.vdim)] = 0;
        }
    }
    // the first tiles, one a stage; those of earlier runs' positions ahead of the dependency wait
    const uint32_t t0 = first / SP + blockIdx.x * SW + warp;
    uint32_t ahead = 0;
    if (VEC) for (; ahead < stages && (t0 + ahead * stride + 1) * SP <= past; ahead++) fetch(t0 + ahead * stride, ahead);
    // LP: the heads of this group, then its key, LP lanes each; what needs no projection is fetched ahead as well
    constexpr int LQ = LP ? LP : 8;
    const uint32_t item_h = tid / LQ, item_c = tid % LQ;
    const HeadVec<LQ> hv(LP && APPEND && item_h <= nh, item_c, a.norms ? a.norms + (item_h == nh ? a.dim : 0) : nullptr, a.rope, pos, a.rot);
    pdl_wait();
    if (nh < 16) for (uint32_t i = nh * rk + tid; i < 16 * rk; i += 256) sq[i] = 0;
    if (dp > a.dim) for (uint32_t i = tid; i < nh * (dp - a.dim); i += 256) sq[(i / (dp - a.dim)) * rk + a.dim + i % (dp - a.dim)] = 0;
    if (APPEND) {
        const uint16_t* y = (const uint16_t*)a.y + (size_t)r * a.y_cols;
        if (LP) {
            // 256 threads take 256 / LP heads at a time; the constants of the second round on are not fetched ahead
            for (uint32_t h = item_h; h - item_h <= nh; h += 256 / LQ) {
                const bool live = h <= nh, key = h == nh;
                const uint4 w = live ? __ldcg((const uint4*)(y + (key ? a.col_k() + g * a.dim : (h0 + h) * a.dim) + item_c * 8)) : make_uint4(0, 0, 0, 0);
                uint4 o;
                if (h == item_h) o = hv.turn(w, a.eps);
                else o = HeadVec<LQ>(live, item_c, a.norms ? a.norms + (key ? a.dim : 0) : nullptr, a.rope, pos, a.rot).turn(w, a.eps);
                if (live) *(uint4*)((key ? snew : sq + h * rk) + item_c * 8) = o;
            }
        } else {
            const float2* rope = (const float2*)a.rope + (size_t)pos * (a.rot / 2);
            float* buf = scr + warp * (((a.dim + 2) + 3u) & ~3u);
            for (uint32_t h = warp; h <= nh; h += SW) {
                const bool key = h == nh;
                uint16_t* to = key ? snew : sq + h * rk;
                head_row<ActBf16>(key ? y + a.col_k() + g * a.dim : y + (h0 + h) * a.dim, a.dim, a.norms ? a.norms + (key ? a.dim : 0) : nullptr,
                                  rope, a.rot, a.eps, buf, [&](uint32_t i, float u, float v) { put_pair<ActBf16>(to, i, a.dim, u, v); });
            }
        }
        for (uint32_t i = tid; i < a.vdim; i += 256) snew[dp + i] = __ldcg(y + a.col_v() + g * a.vdim + i);
    } else {
        const uint16_t* q = (const uint16_t*)a.q + ((size_t)r * a.heads + h0) * a.dim;
        for (uint32_t i = tid; i < nh * a.dim; i += 256) sq[(i / a.dim) * rk + i % a.dim] = __ldcg(q + i);
    }
    for (uint32_t u = ahead; u < stages; u++) fetch(t0 + u * stride, u);
    __syncthreads();
    if (APPEND && blockIdx.x == 0 && h0 == g * rep && pos < a.positions) {
        uint16_t *dk = (uint16_t*)a.state + (size_t)(pos % a.ring) * row + g * a.dim;
        uint16_t *dv = (uint16_t*)a.state + (size_t)(pos % a.ring) * row + a.kv_heads * a.dim + g * a.vdim;
        for (uint32_t i = tid; i < a.dim; i += 256) dk[i] = snew[i];
        for (uint32_t i = tid; i < a.vdim; i += 256) dv[i] = snew[dp + i];
    }
    float o[VT][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < VT; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const float sc = a.scale * 1.44269504088896340736f;           // scores in powers of two
    const uint32_t qaddr = smem_addr(sq + (lane & 15) * rk + (lane >> 4) * 8);
    uint32_t stage = 0;
    for (uint32_t t = t0; t < t_end; t += stride) {
        if (VEC) { if (stages == 2) cp_wait<1>(); else if (stages == 3) cp_wait<2>(); else cp_wait<3>(); }
        uint16_t *k = my + stage * tile_el, *v = k + SP * rk;
        if (APPEND && t + 1 == t_end) {                           // this row's own key and value
            const uint32_t p = pos % SP;
            __syncwarp();
            for (uint32_t i = lane; i < a.dim; i += 32) k[p * rk + i] = snew[i];
            for (uint32_t i = lane; i < a.vdim; i += 32) v[p * rv + i] = snew[dp + i];
        }
        __syncwarp();
        float s[2][4] = {}, s2[2][4] = {};                        // even and odd k steps: two chains of products
        const uint32_t kaddr = smem_addr(k + ((lane & 7) + (lane >> 4) * 8) * rk + ((lane >> 3) & 1) * 8);
#pragma unroll 4
        for (uint32_t ks = 0; ks < dp / 16; ks += 2) {
            uint32_t qa[4], b[4];
            ldsm4(qa, qaddr + ks * 32);
            ldsm4(b, kaddr + ks * 32);
            mma_bf16(s[0], qa, b[0], b[1]);
            mma_bf16(s[1], qa, b[2], b[3]);
            if (ks + 1 < dp / 16) {
                ldsm4(qa, qaddr + ks * 32 + 32);
                ldsm4(b, kaddr + ks * 32 + 32);
                mma_bf16(s2[0], qa, b[0], b[1]);
                mma_bf16(s2[1], qa, b[2], b[3]);
            }
        }
        float mx[2] = {m[0], m[1]};
#pragma unroll
        for (int i = 0; i < 2; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const uint32_t j = t * SP + i * 8 + 2 * t4 + (e & 1);
                const float x = j >= first && j <= pos ? (s[i][e] + s2[i][e]) * sc : -INFINITY;
                s[i][e] = x;
                mx[e >> 1] = fmaxf(mx[e >> 1], x);
            }
#pragma unroll
        for (int q = 0; q < 2; q++) {                             // every tile has a visible position: mx is finite
            mx[q] = fmaxf(mx[q], __shfl_xor_sync(0xffffffffu, mx[q], 1));
            mx[q] = fmaxf(mx[q], __shfl_xor_sync(0xffffffffu, mx[q], 2));
            const float corr = exp2f(m[q] - mx[q]);
            m[q] = mx[q];
            l[q] *= corr;
#pragma unroll
            for (int i = 0; i < VT; i++) { o[i][2 * q] *= corr; o[i][2 * q + 1] *= corr; }
        }
#pragma unroll
        for (int i = 0; i < 2; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const float x = exp2f(s[i][e] - m[e >> 1]);
                s[i][e] = x;
                l[e >> 1] += x;
            }
        uint32_t ph[4], pl[4];
        split_bf2(s[0][0], s[0][1], ph[0], pl[0]);
        split_bf2(s[0][2], s[0][3], ph[1], pl[1]);
        split_bf2(s[1][0], s[1][1], ph[2], pl[2]);
        split_bf2(s[1][2], s[1][3], ph[3], pl[3]);
        const uint32_t vaddr = smem_addr(v + (lane & 15) * rv + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < VT; i += 2) {
            if (i * 8 >= (int)vp) break;
            uint32_t b[4];
            ldsm4_t(b, vaddr + i * 16);
            mma_bf16(o[i], ph, b[0], b[1]);
            mma_bf16(o[i + 1], ph, b[2], b[3]);
            mma_bf16(o[i], pl, b[0], b[1]);
            mma_bf16(o[i + 1], pl, b[2], b[3]);
        }
        __syncwarp();
        fetch(t + stages * stride, stage);
        stage = stage + 1 == stages ? 0 : stage + 1;
    }
    if (VEC) cp_wait<0>();
    __syncthreads();
    // the warps' partial results: maximum, sum, values of the group's heads
#pragma unroll
    for (int q = 0; q < 2; q++) {
        l[q] += __shfl_xor_sync(0xffffffffu, l[q], 1);
        l[q] += __shfl_xor_sync(0xffffffffu, l[q], 2);
        const uint32_t h = g4 + 8 * q;
        if (t4 == 0) { wm[warp][h] = m[q]; wl[warp][h] = l[q]; }
        if (h >= nh) continue;
        float* d = acc + ((size_t)warp * 16 + h) * vp + 2 * t4;
#pragma unroll
        for (int i = 0; i < VT; i++) if (i * 8 < (int)vp) *(float2*)(d + i * 8) = make_float2(o[i][2 * q], o[i][2 * q + 1]);
    }
    // this CTA's share of the output, and its gates
    const uint32_t per = (nh * a.vdim + C - 1) / C, e0 = blockIdx.x * per, e1 = min(e0 + per, nh * a.vdim);
    const uint16_t* yg = a.gate_col == 0xFFFFFFFFu ? nullptr : (const uint16_t*)a.y + (size_t)r * a.y_cols + a.gate_col + h0 * a.vdim;
    const float gate0 = yg && e0 + tid < e1 ? bf2f(__ldcg(yg + e0 + tid)) : 0.0f;
    __syncthreads();
    for (uint32_t i = tid; i < nh * vp; i += 256) {
        const uint32_t h = i / vp;
        float f[SW], mx = -INFINITY, sum = 0.0f, s = 0.0f;
#pragma unroll
        for (uint32_t w = 0; w < SW; w++) { f[w] = wm[w][h]; mx = fmaxf(mx, f[w]); }
#pragma unroll
        for (uint32_t w = 0; w < SW; w++) {
            f[w] = f[w] > -INFINITY ? exp2f(f[w] - mx) : 0.0f;    // a warp without tiles has sum 0
            sum = fmaf(f[w], wl[w][h], sum);
            s = fmaf(f[w], acc[(size_t)w * 16 * vp + i], s);
        }
        acc[i] = s;                                               // only this thread reads element i of any warp
        if (i % vp == 0) { cm[h] = mx; cl[h] = sum; }
    }
    if (C > 1) cluster.sync(); else __syncthreads();
    uint16_t* out = (uint16_t*)a.out + ((size_t)r * a.heads + h0) * a.vdim;
    for (uint32_t i = e0 + tid; i < e1; i += 256) {
        const uint32_t h = i / a.vdim, c = i % a.vdim;
        float pm[MAXC], pl[MAXC], pv[MAXC], mx = -INFINITY, num = 0.0f, den = 0.0f;
#pragma unroll
        for (uint32_t k = 0; k < MAXC; k++) {
            const uint32_t from = k < C ? k : 0;
            pm[k] = *cluster.map_shared_rank(cm + h, from);
            pl[k] = *cluster.map_shared_rank(cl + h, from);
            pv[k] = *cluster.map_shared_rank(acc + h * vp + c, from);
        }
#pragma unroll
        for (uint32_t k = 0; k < MAXC; k++) mx = fmaxf(mx, pm[k]);
#pragma unroll
        for (uint32_t k = 0; k < MAXC; k++) {
            const float f = k < C && pl[k] > 0.0f ? exp2f(pm[k] - mx) : 0.0f;
            num = fmaf(f, pv[k], num);
            den = fmaf(f, pl[k], den);
        }
        const float gt = !yg ? 1.0f : sigmoid_fast(i == e0 + tid ? gate0 : bf2f(__ldcg(yg + i)));
        out[i] = f2bf(num / den * gt);
    }
    if (C > 1) cluster.sync();                                    // nobody leaves while its results are being read
}

size_t step_smem(const WindowArgs& a, uint32_t stages, bool lp) {
    const size_t dp = (a.dim + 15u) & ~15u, vp = (a.vdim + 15u) & ~15u, rk = dp + 8, rv = vp + 8;
    return (16 * rk + dp + vp) * 2 + (lp ? 0 : SW * (((a.dim + 2) + 3u) & ~3u) * 4) + SW * stages * SP * (rk + rv) * 2;
}

bool vec_rows(const WindowArgs& a) { return a.dim % 8 == 0 && a.vdim % 8 == 0 && a.ring % SP == 0; }

constexpr size_t kStepSmem = 224 * 1024;

template <int VT, bool VEC, bool APPEND, int LP>
bool launch_step(cudaStream_t st, const WindowArgs& a, uint32_t rows) {
    static int have[64] = {}, wide[64] = {};       // wide: clusters of 16 CTAs the device can hold at once, + 1
    const uint32_t tiles = (a.window < a.ring ? a.window : a.ring) / SP + 1, rep = a.heads / a.kv_heads;
    const uint32_t clusters = a.kv_heads * ((rep + 15) / 16) * rows;
    // two tiles per warp before another CTA helps, as many stages as fit (and as a warp has tiles)
    uint32_t C = 1, stages = 4;
    while (C < 8 && C * SW * 2 < tiles) C *= 2;
    while (stages > 2 && step_smem(a, stages, LP) > kStepSmem) stages--;
    const size_t smem = step_smem(a, stages, LP);
    auto kernel = window_step_kernel<VT, VEC, APPEND, LP>;
    if (!ensure_dyn_smem(kernel, smem, have)) return false;
    cudaLaunchConfig_t cfg = {};
    cfg.blockDim = dim3(256); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    int dev = 0;
    if (C == 8 && tiles >= 16 * SW * 2 && cudaGetDevice(&dev) == cudaSuccess && dev >= 0 && dev < 64) {
        if (!wide[dev]) {
            int n = 0;
            cudaLaunchAttribute at;
            at.id = cudaLaunchAttributeClusterDimension;
            at.val.clusterDim.x = 16; at.val.clusterDim.y = 1; at.val.clusterDim.z = 1;
            cudaLaunchConfig_t q = cfg;
            q.gridDim = dim3(16); q.attrs = &at; q.numAttrs = 1;
            if (cudaFuncSetAttribute(kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1) != cudaSuccess ||
                cudaOccupancyMaxActiveClusters(&n, kernel, &q) != cudaSuccess) { cudaGetLastError(); n = 0; }
            wide[dev] = n + 1;
        }
        if ((uint32_t)(wide[dev] - 1) >= clusters) C = 16;
    }
    cfg.gridDim = dim3(C, a.kv_heads * ((rep + 15) / 16), rows);
    if (launch_pdl_cluster(kernel, cfg, dim3(C, 1, 1), a, stages) != cudaSuccess) { cudaGetLastError(); return false; }
    g_launches++;
    return true;
}

template <bool APPEND>
bool step(cudaStream_t st, const WindowArgs& a, uint32_t rows) {
    if (!a.bf16 || a.vdim > 256 || step_smem(a, 2, false) > kStepSmem) return false;
    const uint32_t vt = (a.vdim + 15) / 16 * 2;
    if (vec_rows(a)) {
        if (APPEND && head_vec(a) && vt <= 16) {
            if (a.dim == 64) return vt <= 8 ? launch_step<8, true, APPEND, 8>(st, a, rows) : launch_step<16, true, APPEND, 8>(st, a, rows);
            if (a.dim == 128) return vt <= 8 ? launch_step<8, true, APPEND, 16>(st, a, rows) : launch_step<16, true, APPEND, 16>(st, a, rows);
        }
        if (vt <= 8) return launch_step<8, true, APPEND, 0>(st, a, rows);
        if (vt <= 16) return launch_step<16, true, APPEND, 0>(st, a, rows);
        return launch_step<32, true, APPEND, 0>(st, a, rows);
    }
    if (vt <= 8) return launch_step<8, false, APPEND, 0>(st, a, rows);
    if (vt <= 16) return launch_step<16, false, APPEND, 0>(st, a, rows);
    return launch_step<32, false, APPEND, 0>(st, a, rows);
}

}  // namespace

bool k_window_sm100(cudaStream_t st, const WindowArgs& a, uint32_t rows);
bool k_window_flash(cudaStream_t st, const WindowArgs& a, uint32_t rows);

void k_heads_append(cudaStream_t st, const WindowArgs& a, uint32_t rows) {
    if (!rows) return;
    const uint32_t lp = a.dim / 8;
    if (head_vec(a)) {
        const dim3 grid(rows, ((a.heads + a.kv_heads) * lp + a.kv_heads * (a.vdim / 8) + 255) / 256);
        if (lp == 8) launch_pdl(heads_append_vec_kernel<8>, grid, dim3(256), 0, st, a);
        else if (lp == 16) launch_pdl(heads_append_vec_kernel<16>, grid, dim3(256), 0, st, a);
        else launch_pdl(heads_append_vec_kernel<32>, grid, dim3(256), 0, st, a);
        g_launches++;
        return;
    }
    const size_t smem = 8 * (size_t)(a.dim + 1) * 4;
    const dim3 grid(rows, (a.heads + 2 * a.kv_heads + 7) / 8);
    static int have_b[64] = {}, have_f[64] = {};
    if (a.bf16) {
        if (smem > 40 * 1024) ensure_dyn_smem(heads_append_kernel<ActBf16>, smem, have_b);
        launch_pdl(heads_append_kernel<ActBf16>, grid, dim3(256), smem, st, a);
    } else {
        if (smem > 40 * 1024) ensure_dyn_smem(heads_append_kernel<ActF32>, smem, have_f);
        launch_pdl(heads_append_kernel<ActF32>, grid, dim3(256), smem, st, a);
    }
    g_launches++;
}

void k_window_attend(cudaStream_t st, const WindowArgs& a, uint32_t rows, bool exact) {
    if (!rows) return;
    if (a.bf16 && !exact) {
        if (rows <= kStepRows && step<false>(st, a, rows)) return;
        if (k_window_sm100(st, a, rows) || k_window_flash(st, a, rows)) return;
    }
    const size_t smem = (size_t)(a.dim + a.vdim) * 4;
    static int have_b[64] = {}, have_f[64] = {};
    if (a.bf16) {
        if (smem > 40 * 1024) ensure_dyn_smem(window_exact_kernel<ActBf16>, smem, have_b);
        launch_pdl(window_exact_kernel<ActBf16>, dim3(a.heads, rows), dim3(128), smem, st, a);
    } else {
        if (smem > 40 * 1024) ensure_dyn_smem(window_exact_kernel<ActF32>, smem, have_f);
        launch_pdl(window_exact_kernel<ActF32>, dim3(a.heads, rows), dim3(128), smem, st, a);
    }
    g_launches++;
}

bool k_window_step(cudaStream_t st, const WindowArgs& a, uint32_t rows) { return rows == 1 && step<true>(st, a, rows); }

}  // namespace gehtp
