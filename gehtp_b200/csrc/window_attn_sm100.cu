// Window attention over many rows on tcgen05 / TMEM (bf16, key and value sizes 64 or 128).
//
// One CTA = two tiles of 128 query rows that share key and value tiles: the same rows of two heads of a key head or, when
// the query heads of a key head are odd in number, two neighbouring row tiles of one head. Key / value tiles of 128
// positions, position-aligned, straight from the ring by TMA (the ring is a multiple of the tile, so a tile never wraps);
// only tiles a row of the CTA can see are visited.
//
//   S = Q K^T       tcgen05.mma into TMEM (128 columns per query tile)
//   P               one thread per row: running maximum, 2^(s - m), split into hi + lo bf16 and written over S: the 32
//                   columns of 32 positions become 16 columns of hi and 16 of lo pairs
//   O += P V        tcgen05.mma with P as the A operand from TMEM, V as it lies in memory (MN-major B operand)
//
// The maximum a row is referred to is raised - and its O rescaled - only when a tile exceeds it by more than 2^8.
// Products of one query tile run while the softmax warps work on the other.
//
//   warp 0     TMA: both Q tiles once, K and V tiles in two stages
//   warp 1     one lane issues tcgen05.mma / tcgen05.commit
//   warp 2     owns the TMEM allocation (512 columns: S/P of both tiles, O of both tiles)
//   warps 4-7  softmax and output of the first tile, warps 8-11 of the second
// Every mbarrier wait is bounded; on a timeout the CTA raises the engine's status word and winds down.
#include <cuda.h>
#include <cuda_runtime.h>
#include "launchers_rows.h"
#include "rows_common.cuh"
#include "sm100_umma.cuh"

namespace gehtp {

using namespace sm100;

namespace {

constexpr uint32_t BQ = 128, BKV = 128, BOX = 64 * 64 * 2;      // bytes of a box of 64 rows x 64 elements
constexpr int NTHREADS = 384;
constexpr float kRaise = 8.0f;

struct __align__(8) WBars {
    uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[2], p_full[2], o_full;
    uint32_t tmem_base, abort_flag;
};

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}


__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t (&v)[32]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
        : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]),
          "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]),
          "=r"(v[16]), "=r"(v[17]), "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), "=r"(v[23]),
          "=r"(v[24]), "=r"(v[25]), "=r"(v[26]), "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
        : "r"(taddr));
}
// waits for the loads in flight; the registers of the last one pass through, so that nothing reads them ahead of it
__device__ __forceinline__ void tmem_ld_wait(uint32_t (&v)[32]) {
    asm volatile("tcgen05.wait::ld.sync.aligned;"
        : "+r"(v[0]), "+r"(v[1]), "+r"(v[2]), "+r"(v[3]), "+r"(v[4]), "+r"(v[5]), "+r"(v[6]), "+r"(v[7]),
          "+r"(v[8]), "+r"(v[9]), "+r"(v[10]), "+r"(v[11]), "+r"(v[12]), "+r"(v[13]), "+r"(v[14]), "+r"(v[15]),
          "+r"(v[16]), "+r"(v[17]), "+r"(v[18]), "+r"(v[19]), "+r"(v[20]), "+r"(v[21]), "+r"(v[22]), "+r"(v[23]),
          "+r"(v[24]), "+r"(v[25]), "+r"(v[26]), "+r"(v[27]), "+r"(v[28]), "+r"(v[29]), "+r"(v[30]), "+r"(v[31])
        :: "memory");
}
__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t (&v)[32]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%32], "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31};"
        ::"r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]),
          "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]),
          "r"(v[16]), "r"(v[17]), "r"(v[18]), "r"(v[19]), "r"(v[20]), "r"(v[21]), "r"(v[22]), "r"(v[23]),
          "r"(v[24]), "r"(v[25]), "r"(v[26]), "r"(v[27]), "r"(v[28]), "r"(v[29]), "r"(v[30]), "r"(v[31]), "r"(taddr)
        : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// two fp32 operations in one instruction
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("{\n .reg .b64 a, b, c, d;\n mov.b64 a, {%2, %3};\n mov.b64 b, {%4, %5};\n mov.b64 c, {%6, %7};\n"
        " fma.rn.f32x2 d, a, b, c;\n mov.b64 {%0, %1}, d;\n}"
        : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
    return d;
}
__device__ __forceinline__ float2 add2(float2 a, float2 b) {
    float2 d;
    asm("{\n .reg .b64 a, b, d;\n mov.b64 a, {%2, %3};\n mov.b64 b, {%4, %5};\n add.rn.f32x2 d, a, b;\n mov.b64 {%0, %1}, d;\n}"
        : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
    return d;
}

// bit i: column c0 + i lies in [lo, hi]
__device__ __forceinline__ uint32_t visible32(int c0, int lo, int hi) {
    const int a = lo - c0, b = hi - c0;
    const uint32_t from = a <= 0 ? 0xFFFFFFFFu : a > 31 ? 0u : 0xFFFFFFFFu << a, to = b < 0 ? 0u : b >= 31 ? 0xFFFFFFFFu : 0xFFFFFFFFu >> (31 - b);
    return from & to;
}

// largest of 32 scores, EDGE: of those whose bit is set
template <bool EDGE>
__device__ __forceinline__ float max32(const uint32_t (&v)[32], uint32_t see) {
    float m[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
    for (int i = 0; i < 32; i++) m[i & 3] = fmaxf(m[i & 3], !EDGE || ((see >> i) & 1u) ? __uint_as_float(v[i]) : -INFINITY);
    return fmaxf(fmaxf(m[0], m[1]), fmaxf(m[2], m[3]));
}

// 2^(s sc + off) of 32 scores (EDGE: 0 where the bit is not set), as 16 words of hi and 16 of lo bf16 pairs; adds the
// values to l
template <bool EDGE>
__device__ __forceinline__ void probs32(const uint32_t (&v)[32], uint32_t (&w)[32], float sc, float off, uint32_t see, float2 (&l)[2]) {
#pragma unroll
    for (int i = 0; i < 16; i++) {
        const float2 x = fma2(make_float2(__uint_as_float(v[2 * i]), __uint_as_float(v[2 * i + 1])), make_float2(sc, sc), make_float2(off, off));
        float2 e = make_float2(ex2(x.x), ex2(x.y));
        if (EDGE) {
            e.x = (see >> (2 * i)) & 1u ? e.x : 0.0f;
            e.y = (see >> (2 * i + 1)) & 1u ? e.y : 0.0f;
        }
        l[i & 1] = add2(l[i & 1], e);
        const uint32_t p = pack_bf2(e.x, e.y);
        w[i] = p;
        const float2 r = fma2(make_float2(__uint_as_float(p << 16), __uint_as_float(p & 0xffff0000u)), make_float2(-1.0f, -1.0f), e);
        w[16 + i] = pack_bf2(r.x, r.y);
    }
}

// D[tmem] (+)= A[tmem] B[smem]
__device__ __forceinline__ void umma_f16_ta(uint32_t tmem_d, uint32_t tmem_a, uint64_t db, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n"
        " tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n}\n"
        ::"r"(tmem_d), "r"(tmem_a), "l"(db), "r"(idesc), "r"(accumulate) : "memory");
}

// B operand of a value tile as it lies in memory ([position][value], value contiguous): boxes of 64 positions x 64 values
// with the 128-byte swizzle, 8-position groups 1024 bytes apart, the second 64 values one box further
__device__ __forceinline__ uint64_t umma_desc_v(uint32_t saddr) {
    uint64_t d = 0;
    d |= (uint64_t)((saddr & 0x3FFFFu) >> 4);
    d |= (uint64_t)(BOX >> 4) << 16;
    d |= (uint64_t)(1024 >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}

constexpr uint32_t IDESC_BF16 = (1u << 7) | (1u << 10);          // A and B are bf16

// DB, VB: key and value size in units of 64
template <int DB, int VB>
__global__ void __launch_bounds__(NTHREADS, 1)
window_attn_sm100_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_kv, const WindowArgs A, uint32_t rows) {
    extern __shared__ unsigned char smem_raw[];
    constexpr uint32_t Q_BYTES = DB * 2 * BOX, K_BYTES = DB * 2 * BOX, V_BYTES = VB * 2 * BOX;
    unsigned char* smem = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    unsigned char* sQ = smem;                                    // two tiles
    unsigned char* sK = sQ + 2 * Q_BYTES;                        // two stages
    unsigned char* sV = sK + 2 * K_BYTES;                        // two stages: [position half][64 values][64 positions x 128 bytes]
    WBars* bars = (WBars*)(sV + 2 * V_BYTES);
    volatile uint32_t* abort_flag = &bars->abort_flag;
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t rep = A.heads / A.kv_heads;
    const bool by_head = (rep & 1u) == 0;                        // the pair: two heads, or two row tiles
    const uint32_t qt = gridDim.y - 1 - blockIdx.y;              // the longest rows of all heads first
    const uint32_t h0 = by_head ? 2 * blockIdx.x : blockIdx.x, kvh = h0 / rep;
    const uint32_t q0 = by_head ? qt * BQ : 2 * qt * BQ;
    // the counter moves at the end of a run only: it may be read before the dependency wait
    const uint32_t past = *(volatile const uint32_t*)A.counter, n = past + rows;
    const uint32_t p0 = past + q0, span = by_head ? BQ : 2 * BQ;
    const uint32_t first = p0 + 1 > A.window ? p0 + 1 - A.window : 0, last = min(p0 + span, n);
    const uint32_t kt0 = first / BKV, n_kt = (last + BKV - 1) / BKV - kt0;

    if (threadIdx.x == 0) {
        mbar_init(&bars->q_full, 1); mbar_init(&bars->o_full, 1);
        for (int s = 0; s < 2; s++) {
            mbar_init(&bars->k_full[s], 1); mbar_init(&bars->k_empty[s], 1);
            mbar_init(&bars->v_full[s], 1); mbar_init(&bars->v_empty[s], 1);
            mbar_init(&bars->s_full[s], 1); mbar_init(&bars->p_full[s], 4);
        }
        bars->abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 2) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&bars->tmem_base)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = bars->tmem_base;

    if (warp == 0) {
        // ------------------------------------------------------------ TMA producer
        if (lane == 0) {
            asm volatile("griddepcontrol.wait;" ::: "memory");
            mbar_expect_tx(&bars->q_full, 2 * Q_BYTES);
#pragma unroll
            for (uint32_t t = 0; t < 2; t++)
#pragma unroll
                for (uint32_t d = 0; d < DB; d++)
#pragma unroll
                    for (uint32_t r = 0; r < 2; r++)
                        tma_load_2d(sQ + t * Q_BYTES + (d * 2 + r) * BOX, &tmap_q, (int)((h0 + (by_head ? t : 0)) * DB * 64 + d * 64),
                                    (int)(q0 + (by_head ? 0 : t * BQ) + r * 64), &bars->q_full);
            uint32_t kn = 0, vn = 0;
            for (uint32_t j = 0; j < n_kt && !*abort_flag; j++) {
                const uint32_t s = j & 1, ph = (j >> 1) & 1;
                const int y = (int)(((kt0 + j) * BKV) % A.ring);
                if (!mbar_wait_or_abort(&bars->k_empty[s], ph ^ 1, abort_flag)) { *abort_flag = 1; break; }
                mbar_expect_tx(&bars->k_full[s], K_BYTES);
#pragma unroll
                for (uint32_t d = 0; d < DB; d++)
#pragma unroll
                    for (uint32_t r = 0; r < 2; r++)
                        tma_load_2d(sK + s * K_BYTES + (d * 2 + r) * BOX, &tmap_kv, (int)(kvh * DB * 64 + d * 64), y + (int)r * 64, &bars->k_full[s]);
                kn++;
                if (!mbar_wait_or_abort(&bars->v_empty[s], ph ^ 1, abort_flag)) { *abort_flag = 1; break; }
                mbar_expect_tx(&bars->v_full[s], V_BYTES);
#pragma unroll
                for (uint32_t r = 0; r < 2; r++)
#pragma unroll
                    for (uint32_t d = 0; d < VB; d++)
                        tma_load_2d(sV + s * V_BYTES + (r * VB + d) * BOX, &tmap_kv, (int)(A.kv_heads * DB * 64 + kvh * VB * 64 + d * 64), y + (int)r * 64, &bars->v_full[s]);
                vn++;
            }
            if (*abort_flag) {   // copies already requested must land before the CTA may go away
                mbar_wait(&bars->q_full, 0);
                for (uint32_t j = kn > 2 ? kn - 2 : 0; j < kn; j++) mbar_wait(&bars->k_full[j & 1], (j >> 1) & 1);
                for (uint32_t j = vn > 2 ? vn - 2 : 0; j < vn; j++) mbar_wait(&bars->v_full[j & 1], (j >> 1) & 1);
            }
        }
    } else if (warp == 1) {
        // ------------------------------------------------------------ MMA issuer
        if (lane == 0) {
            const uint32_t q_base = smem_u32(sQ), k_base = smem_u32(sK), v_base = smem_u32(sV);
            bool ok = true;
            auto wait = [&](uint64_t* bar, uint32_t parity) {
                if (ok) ok = mbar_wait_or_abort(bar, parity, abort_flag);
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                return ok;
            };
            auto issue_s = [&](uint32_t t, uint32_t j) {
#pragma unroll
                for (uint32_t d = 0; d < DB; d++)
#pragma unroll
                    for (uint32_t k4 = 0; k4 < 4; k4++)
                        umma_f16(tmem + t * 128, umma_desc(q_base + t * Q_BYTES + d * 2 * BOX) + (uint64_t)(k4 * 2),
                                 umma_desc(k_base + (j & 1) * K_BYTES + d * 2 * BOX) + (uint64_t)(k4 * 2), idesc_f16(128) | IDESC_BF16, (d | k4) ? 1u : 0u);
                umma_commit(&bars->s_full[t]);
            };
            auto issue_o = [&](uint32_t t, uint32_t j) {
#pragma unroll
                for (uint32_t part = 0; part < 2; part++)
#pragma unroll
                    for (uint32_t k = 0; k < 8; k++)             // 16 positions = two 8-position groups = 2048 bytes per step
                        umma_f16_ta(tmem + 256 + t * 128, tmem + t * 128 + (k >> 1) * 32 + part * 16 + (k & 1) * 8,
                                    umma_desc_v(v_base + (j & 1) * V_BYTES + (k >> 2) * (VB * BOX) + (k & 3) * 2048),
                                    idesc_f16(VB * 64) | IDESC_BF16 | (1u << 16), (j | part | k) ? 1u : 0u);
            };
            if (wait(&bars->q_full, 0) && wait(&bars->k_full[0], 0)) {
                issue_s(0, 0);
                issue_s(1, 0);
                umma_commit(&bars->k_empty[0]);
            }
            for (uint32_t j = 0; ok && j < n_kt; j++) {
                const uint32_t s = j & 1, ph = (j >> 1) & 1, s1 = (j + 1) & 1, ph1 = ((j + 1) >> 1) & 1;
                const bool more = j + 1 < n_kt;
                if (!wait(&bars->v_full[s], ph) || !wait(&bars->p_full[0], j & 1)) break;
                issue_o(0, j);
                if (more) {
                    if (!wait(&bars->k_full[s1], ph1)) break;
                    issue_s(0, j + 1);
                }
                if (!wait(&bars->p_full[1], j & 1)) break;
                issue_o(1, j);
                umma_commit(&bars->v_empty[s]);
                if (more) {
                    issue_s(1, j + 1);
                    umma_commit(&bars->k_empty[s1]);
                }
            }
            if (ok) umma_commit(&bars->o_full);
            else *abort_flag = 1;
        }
    } else if (warp >= 4) {
        // ------------------------------------------------------------ softmax and output: one thread per query row
        const uint32_t t = (warp - 4) >> 2, quarter = warp & 3, row = quarter * 32 + lane;
        const uint32_t qrow = q0 + (by_head ? 0 : t * BQ) + row, h = h0 + (by_head ? t : 0);
        const uint32_t pos = past + qrow, w_first = pos - lane, w_last = w_first + 31;
        const uint32_t ts = tmem + ((quarter * 32) << 16) + t * 128, to = ts + 256;
        const float sc = A.scale * 1.44269504088896340736f;      // scores in powers of two
        float m = -INFINITY;
        float2 l2[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
        bool ok = true;
        asm volatile("griddepcontrol.wait;" ::: "memory");
        for (uint32_t j = 0; j < n_kt; j++) {
            ok = !__any_sync(0xffffffffu, *abort_flag != 0) && __all_sync(0xffffffffu, mbar_wait_or_abort(&bars->s_full[t], j & 1, abort_flag));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t j0 = (kt0 + j) * BKV;
            const bool edge = j0 + BKV - 1 > w_first || j0 + A.window <= w_last;      // some key of the tile is hidden from some row
            // columns [lo, hi] of the tile are visible to this row
            const int hi = (int)(pos - j0), lo = (int)(pos + 1 - A.window - j0);
            // the next 32 columns are on their way while 32 are worked on
            uint32_t va[32], vb[32];
            auto largest = [&](const uint32_t (&v)[32], int c) { return edge ? max32<true>(v, visible32(c * 32, lo, hi)) : max32<false>(v, 0u); };
            tmem_ld32(ts, va);
            tmem_ld_wait(va);
            tmem_ld32(ts + 32, vb);
            float mt = largest(va, 0);
            tmem_ld_wait(vb);
            tmem_ld32(ts + 64, va);
            mt = fmaxf(mt, largest(vb, 1));
            tmem_ld_wait(va);
            tmem_ld32(ts + 96, vb);
            mt = fmaxf(mt, largest(va, 2));
            tmem_ld_wait(vb);
            mt = fmaxf(mt, largest(vb, 3)) * sc;
            // s_full of this tile came after the products of the tile before: O is at rest
            const bool raise = mt > m + kRaise;
            if (__any_sync(0xffffffffu, raise)) {
                const float f = raise ? (m == -INFINITY ? 0.0f : ex2(m - mt)) : 1.0f;
                if (raise) m = mt;
#pragma unroll
                for (int i = 0; i < 2; i++) { l2[i].x *= f; l2[i].y *= f; }
                if (j) {
#pragma unroll 1
                    for (int c = 0; c < VB * 2; c++) {
                        uint32_t v[32];
                        tmem_ld32(to + c * 32, v);
                        tmem_ld_wait(v);
#pragma unroll
                        for (int i = 0; i < 32; i++) v[i] = __float_as_uint(__uint_as_float(v[i]) * f);
                        tmem_st32(to + c * 32, v);
                    }
                    tmem_st_wait();
                }
            }
            const float off = m == -INFINITY ? 0.0f : -m;        // a row that has seen no key yet: zeros
            auto weigh = [&](const uint32_t (&v)[32], int c) {
                uint32_t w[32];
                if (edge) probs32<true>(v, w, sc, off, visible32(c * 32, lo, hi), l2);
                else probs32<false>(v, w, sc, off, 0u, l2);
                tmem_st32(ts + c * 32, w);
            };
            tmem_ld32(ts, va);
            tmem_ld_wait(va);
            tmem_ld32(ts + 32, vb);
            weigh(va, 0);
            tmem_ld_wait(vb);
            tmem_ld32(ts + 64, va);
            weigh(vb, 1);
            tmem_ld_wait(va);
            tmem_ld32(ts + 96, vb);
            weigh(va, 2);
            tmem_ld_wait(vb);
            weigh(vb, 3);
            tmem_st_wait();
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&bars->p_full[t]);
        }
        // the gates come in while the last products run
        const bool gate = A.gate_col != 0xFFFFFFFFu, live = qrow < rows;
        const uint4* yg = (const uint4*)((const uint16_t*)A.y + (size_t)qrow * A.y_cols + A.gate_col + h * (VB * 64));
        uint4 g[VB * 8];
#pragma unroll
        for (int q = 0; q < VB * 8; q++) g[q] = live && gate ? __ldcg(yg + q) : make_uint4(0, 0, 0, 0);
        if (ok) ok = __all_sync(0xffffffffu, mbar_wait_or_abort(&bars->o_full, 0, abort_flag));
        if (ok) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const float inv = 1.0f / ((l2[0].x + l2[0].y) + (l2[1].x + l2[1].y));
            uint4* out = (uint4*)((uint16_t*)A.out + ((size_t)qrow * A.heads + h) * (VB * 64));
#pragma unroll
            for (int c = 0; c < VB * 2; c++) {
                uint32_t v[32];
                tmem_ld32(to + c * 32, v);
                tmem_ld_wait(v);
                if (!live) continue;
#pragma unroll
                for (int q = 0; q < 4; q++) {
                    const uint4 gq = g[c * 4 + q];
                    const uint32_t gw[4] = {gq.x, gq.y, gq.z, gq.w};
                    uint32_t w[4];
#pragma unroll
                    for (int i = 0; i < 4; i++) {
                        float a = __uint_as_float(v[8 * q + 2 * i]) * inv, b = __uint_as_float(v[8 * q + 2 * i + 1]) * inv;
                        if (gate) { a *= sigmoid_fast(__uint_as_float(gw[i] << 16)); b *= sigmoid_fast(__uint_as_float(gw[i] & 0xffff0000u)); }
                        w[i] = pack_bf2(a, b);
                    }
                    out[c * 4 + q] = make_uint4(w[0], w[1], w[2], w[3]);
                }
            }
        } else {
            *abort_flag = 1;
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 2) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
        if (lane == 0 && *abort_flag) raise_status(A.status, kStatusAttnTimeout);
    }
}

bool make_map(CUtensorMap* tm, const void* base, uint64_t inner, uint64_t rows, uint64_t row_elems) {
    EncodeTiledFn enc = encode_fn();
    if (!enc) return false;
    cuuint64_t dims[2] = {inner, rows};
    cuuint64_t strides[1] = {row_elems * 2};
    cuuint32_t box[2] = {64, 64};
    cuuint32_t estr[2] = {1, 1};
    return enc(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (void*)base, dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
               CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int DB, int VB>
bool launch(cudaStream_t st, const WindowArgs& a, uint32_t rows) {
    CUtensorMap tq, tkv;
    if (!make_map(&tq, a.q, (uint64_t)a.heads * a.dim, rows, (uint64_t)a.heads * a.dim) || !make_map(&tkv, a.state, a.row(), a.ring, a.row())) return false;
    const size_t smem = 1024 + (size_t)(DB * 8 + VB * 4) * BOX + sizeof(WBars) + 16;
    static int have[64] = {};
    if (!ensure_dyn_smem(window_attn_sm100_kernel<DB, VB>, smem, have)) return false;
    const uint32_t tiles = (rows + BQ - 1) / BQ;
    const bool by_head = (a.heads / a.kv_heads) % 2 == 0;
    const dim3 grid(by_head ? a.heads / 2 : a.heads, by_head ? tiles : (tiles + 1) / 2);
    if (launch_pdl(window_attn_sm100_kernel<DB, VB>, grid, dim3(NTHREADS), smem, st, tq, tkv, a, rows) != cudaSuccess) { cudaGetLastError(); return false; }
    g_launches++;
    return true;
}

}  // namespace

// false: sizes or alignment not taken, nothing launched
bool k_window_sm100(cudaStream_t st, const WindowArgs& a, uint32_t rows) {
    const bool gate = a.gate_col != 0xFFFFFFFFu;
    if (!a.bf16 || !rows || a.dim % 64 || a.vdim % 64 || a.dim > 128 || a.vdim > 128 || a.ring % BKV || a.scale <= 0.0f) return false;
    if ((((uintptr_t)a.q | (uintptr_t)a.state | (uintptr_t)a.out) & 15u) || (gate && ((a.y_cols | a.gate_col) & 7u || (uintptr_t)a.y & 15u))) return false;
    if (a.dim == 64) return a.vdim == 64 ? launch<1, 1>(st, a, rows) : launch<1, 2>(st, a, rows);
    return a.vdim == 64 ? launch<2, 1>(st, a, rows) : launch<2, 2>(st, a, rows);
}

}  // namespace gehtp
