// The walk over an op list that sizes temps and bakes launches, shared by the per-op planners
// (plan.cu: the reference's opcodes, plan_rows.cu: the row-count opcodes).
#pragma once
#include <cstdio>
#include <cstring>
#include "engine.h"

namespace gehtp {

struct LiveRange { uint32_t w, r; };  // written at op w, last read at op r

struct Planner {
    const wt_blob* b;
    bool build;
    uint32_t opi = 0;
    bool written[kMaxTemps];
    // 64-bit: a temp that only exists inside a fused chain may exceed the 4 GB a
    // materialised temp is limited to (e.g. the GQA-expanded K/V faces at batch 64)
    uint64_t cap[kMaxTemps], last[kMaxTemps];
    // measuring walk results
    uint64_t maxb[kMaxTemps];
    bool oversize[kMaxTemps];
    std::vector<LiveRange> live[kMaxTemps];
    // building walk inputs
    uint8_t* addr[kMaxTemps];
    bool in_static[kMaxTemps], in_vtcm[kMaxTemps];
    bool internal[kMaxTemps];   // exists only inside fused chains: no memory
    PlanOp* cur = nullptr;

    uint8_t* dummy() const { return (uint8_t*)(uintptr_t)256; }

    const uint8_t* slot_ptr(uint32_t s) const {
        if (s >= b->n_slots) return nullptr;
        const wt_slot& sl = b->slots[s];
        if (sl.addr == WT_SLOT_EXT_IN || sl.addr == WT_SLOT_EXT_WGT) {
            if (sl.addr == WT_SLOT_EXT_WGT && !g.ext_wgt) return nullptr;
            if (!build) return dummy();
            auto it = g.d_ext.find(s);
            return it == g.d_ext.end() ? nullptr : it->second;
        }
        return build ? g.d_weights + sl.offset : dummy();
    }

    // ref_ptr, oplist_exec.c:189-203
    const uint8_t* ref(uint32_t arg) {
        if (arg & 0x8000u) return slot_ptr(arg & 0x7FFFu);
        if ((arg & 0xE000u) == WT_REF_STATE_FLAG) {
            uint32_t s = arg & 0x1FFFu;
            return s < g.n_states ? g.st_buf[s] : nullptr;
        }
        uint32_t t;
        if (arg & 0x4000u) {
            t = arg & 0x3FFFu;
            if (t >= kMaxTemps || g.vtcm_off[t] == kNoOff) return nullptr;
            if (!build) { touch(t); return dummy(); }
            return g.d_arena + g.vtcm_base + g.vtcm_off[t];
        }
        t = arg;
        if (t >= kMaxTemps || !written[t]) return nullptr;
        touch(t);
        if (build && internal[t]) { if (cur) cur->uses_internal = true; return dummy(); }
        return build ? addr[t] : dummy();
    }
    void touch(uint32_t t) {
        if (!build && !live[t].empty()) live[t].back().r = opi;
    }
    // ref_elem_count, oplist_exec.c:209-213
    uint32_t ref_count(uint32_t arg) const {
        if (arg & 0x8000u) { uint32_t s = arg & 0x7FFFu; return s < b->n_slots ? b->slots[s].count : 0; }
        if (arg & 0x4000u) return 0;
        return arg < kMaxTemps ? (uint32_t)(last[arg] / 2u) : 0;
    }
    // temp_get, oplist_exec.c:257-335
    uint8_t* temp_get(uint32_t id, uint64_t bytes64, PlanOp& p) {
        if (id >= kMaxTemps || bytes64 > (1ull << 40)) return nullptr;
        // Above 4 GB (the reference's temp sizes are 32-bit) only as a temp that fusion removes.
        if (bytes64 > 0xFFFFFFFFull) {
            if (!build) oversize[id] = true;
            else if (!internal[id]) return nullptr;
        }
        const uint64_t bytes = bytes64;
        bool vt = g.vtcm_off[id] != kNoOff, stc = !vt && g.have_static && g.static_off[id] != kNoOff;
        if (vt && (uint64_t)g.vtcm_off[id] + bytes > g.vtcm_cap) return nullptr;
        if (stc && (!build || in_static[id]) && (uint64_t)g.static_off[id] + bytes > g.static_cap) return nullptr;
        if (vt || stc) cap[id] = bytes;
        else if (!written[id] || cap[id] < bytes) cap[id] = bytes;
        last[id] = bytes;
        written[id] = true;
        for (int k = 0; k < 2; k++)
            if (p.out_id[k] == kNoOff || p.out_id[k] == id) { p.out_id[k] = id; p.out_bytes[k] = (uint32_t)(bytes > 0xFFFFFFFFull ? 0xFFFFFFFFull : bytes); break; }
        if (!build) {
            if (bytes > maxb[id]) maxb[id] = bytes;
            live[id].push_back({opi, opi});
            return dummy();
        }
        if (internal[id]) { p.uses_internal = true; return dummy(); }
        return addr[id];
    }
};

#define FAIL(...)                                            \
    do {                                                     \
        char _m[160];                                        \
        std::snprintf(_m, sizeof _m, __VA_ARGS__);           \
        p.rc = -1; p.err = _m; return;                       \
    } while (0)

// plan_rows.cu: opcodes OP_EMBED_ROWS .. OP_WINDOW_ATTEND
void plan_rows_op(Planner& P, const wt_op& op, PlanOp& p);

}  // namespace gehtp
