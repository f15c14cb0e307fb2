// Decode attention on tensor cores: one query position per row, split over
// the keys.
//
// A CTA serves one (row, kv head, tile of up to 8 query heads of that kv
// head's group, split of the key range).  The keys are the rows of the MMA
// tiles and the query heads that share the kv head its 8 columns
// (attn_mma.cuh: attend_keys16), so each K/V page is read once for the whole
// group (the reference's decode kernel does the same with CUDA cores:
// src/kernels_cuda/attention_decode.cuh:34-176).  Pages of 64 keys stream
// through a three-stage ring of shared-memory tiles; warp w takes keys
// [16 w, 16 w + 16) of every page with its own running (max, sum, acc), and
// the four warps are merged at the end.  With more than one split the splits
// either form a thread-block cluster that merges its partials over distributed
// shared memory, or write unnormalised partials (acc, max, sum) to scratch for
// a second kernel that combines them in split order
// (src/kernels_cuda/attention_online.cu:51-78).  Softmax runs in 32-bit on
// base-2 exponentials: p = 2^((s - m) * scale * log2 e).
//
// A page's key and value tiles come by TMA where the head size is a multiple
// of 64 and the caller says how many pages the store has: one thread issues
// D / 64 box loads per tile (128-byte swizzle, which the fragment loads undo)
// and a barrier counts the bytes.  Copying the same page in 16-byte pieces from
// all threads (the general form, any head size) costs about as many issue
// cycles as the page's tile code itself.
#include "attention_decode.cuh"
#include "noalloc.h"

namespace {

int decode_entry(const void* q, const void* k_pages, const void* v_pages, const int* page_table,
                 int max_pages, int page_size, const int* row_pos, const int* row_slot, void* out,
                 float* partial, int R, int nq, int nkv, int head_dim, int n_splits, int window,
                 int keep_first, float scale, const float* sink, const float* slopes, float softcap, int cluster_merge,
                 long long pool_pages, int* err, void* stream, rfx::RowGate gate = rfx::RowGate{nullptr, 0, 0, 0}) {
    if (R <= 0) return 0;
    if (page_size != PAGE || nkv <= 0 || nq % nkv != 0 || n_splits < 1) return RFX_ERR_BAD_ARG;
    if (softcap < 0.0f || (softcap > 0.0f && slopes)) return RFX_ERR_UNSUPPORTED;  // one or the other
    if (n_splits > 1 && !partial && !cluster_merge) return RFX_ERR_BAD_ARG;
    if (cluster_merge && n_splits != 2 && n_splits != 4 && n_splits != 8 && n_splits != 16) return RFX_ERR_UNSUPPORTED;
    if (n_splits > MAX_SPLITS) return RFX_ERR_UNSUPPORTED;
    if (n_splits > 65535 || (long long)nkv * ((nq / nkv + 7) / 8) > 65535) return RFX_ERR_UNSUPPORTED;
    PagedKV cache{page_table, max_pages, page_size, nkv, head_dim};
    cudaStream_t s = (cudaStream_t)stream;
    // page tiles by TMA: head sizes that are whole 64-column boxes, a store whose
    // size the caller gave, 16-byte aligned (REFLEX_B200_DECODE_TMA=0: a tuning aid)
    static const bool tma_on = [] {
        const char* e = getenv("REFLEX_B200_DECODE_TMA");
        return !(e && e[0] == '0');
    }();
    const bool tma = tma_on && pool_pages > 0 && head_dim % 64 == 0 &&
                     ((reinterpret_cast<uintptr_t>(k_pages) | reinterpret_cast<uintptr_t>(v_pages)) & 15) == 0 &&
                     pool_pages * nkv * PAGE < 2147483647LL;
    // with slopes or a cap: the kernel's form that has that term
#define RFX_FORM(DD, T, M)                                                                                  \
    launch_decode<DD, T, M>(q, k_pages, v_pages, pool_pages, cache, row_pos, row_slot, out, partial, R, nq, \
                            n_splits, window, keep_first, scale, sink, slopes, softcap, cluster_merge, 1, err, s, \
                            gate)
#define RFX_GO(DD, T) (slopes ? RFX_FORM(DD, T, 1) : softcap > 0.0f ? RFX_FORM(DD, T, 2) : RFX_FORM(DD, T, 0))
#define RFX_CASE(DD)                                        \
    case DD:                                                \
        if (DD % 64 == 0 && tma) {                          \
            const int st = RFX_GO(DD, (DD % 64 == 0));      \
            if (st != RFX_ERR_UNSUPPORTED) return st;       \
        }                                                   \
        return RFX_GO(DD, false);
    switch (head_dim) {
        RFX_CASE(16) RFX_CASE(32) RFX_CASE(48) RFX_CASE(64) RFX_CASE(80) RFX_CASE(96)
        RFX_CASE(112) RFX_CASE(128) RFX_CASE(144) RFX_CASE(160) RFX_CASE(176) RFX_CASE(192)
        RFX_CASE(208) RFX_CASE(224) RFX_CASE(240) RFX_CASE(256)
        default:
            return RFX_ERR_UNSUPPORTED;
    }
#undef RFX_CASE
#undef RFX_GO
#undef RFX_FORM
}

}  // namespace

// bfloat16 q [R, nq, D], paged K/V, one query position per row.  `partial` is
// scratch of R * nq * n_splits * (D + 2) floats, needed when n_splits > 1.
// head_dim: multiples of 16 up to 256; the page size must be 64.
// `pool_pages`: pages of the key (and value) store that `k_pages` points to, if the
// caller knows (else 0): with it, head sizes 64, 128, 192 and 256 take their pages by
// TMA.  `err` (may be null): a device word that receives a non-zero code if a bounded
// wait ran out.  `sink`, `slopes` (one float per query head each, or null): exp(sink)
// joins the softmax's denominator; slope * (query position - key position) is taken
// off every score.
extern "C" int rfx_attention_decode(const void* q, const void* k_pages, const void* v_pages,
                                    const int* page_table, int max_pages, int page_size,
                                    const int* row_pos, const int* row_slot, void* out,
                                    float* partial, int R, int nq, int nkv, int head_dim,
                                    int n_splits, int window, float scale, const float* sink,
                                    const float* slopes, long long pool_pages, int* err, void* stream) {
    return decode_entry(q, k_pages, v_pages, page_table, max_pages, page_size, row_pos, row_slot, out,
                        partial, R, nq, nkv, head_dim, n_splits, window, 0, scale, sink, slopes, 0.0f, 0, pool_pages,
                        err, stream);
}

// The same with `keep_first` (the first so many positions of a sequence stay
// visible beyond the window) and `softcap` (> 0: a score s becomes softcap * tanh(s / softcap)
// before the softmax; not together with slopes).  `gate_z` (or null): rows of `gate_ld` elements;
// sigmoid(gate_z[r, gate_col + h]) scales what head h of row r gives.
extern "C" int rfx_attention_decode_kf(const void* q, const void* k_pages, const void* v_pages,
                                       const int* page_table, int max_pages, int page_size,
                                       const int* row_pos, const int* row_slot, void* out,
                                       float* partial, int R, int nq, int nkv, int head_dim,
                                       int n_splits, int window, int keep_first, float scale, const float* sink,
                                       const float* slopes, float softcap, long long pool_pages, int cluster,
                                       const void* gate_z, int gate_dt, int gate_ld, int gate_col, int* err,
                                       void* stream) {
    rfx::RowGate gate;
    if (keep_first < 0 || !rfx::row_gate(&gate, gate_z, gate_dt, gate_ld, gate_col, nq)) return RFX_ERR_BAD_ARG;
    return decode_entry(q, k_pages, v_pages, page_table, max_pages, page_size, row_pos, row_slot, out,
                        cluster ? nullptr : partial, R, nq, nkv, head_dim, n_splits, window, keep_first, scale,
                        sink, slopes, softcap, cluster ? 1 : 0, pool_pages, err, stream, gate);
}

// The same with 2, 4, 8 or (where the device places such a cluster) 16 splits that
// form a thread-block cluster: every rank
// sends its partial to the rank that owns that slice of the output over
// distributed shared memory, one cluster barrier, and the owners merge in rank
// order with the combine kernel's arithmetic.  No scratch, no second kernel.
// RFX_ERR_UNSUPPORTED for other split counts or sizes that leave no shared
// memory for the exchange: the caller then takes the entry point above.
extern "C" int rfx_attention_decode_cluster(const void* q, const void* k_pages, const void* v_pages,
                                            const int* page_table, int max_pages, int page_size,
                                            const int* row_pos, const int* row_slot, void* out, int R,
                                            int nq, int nkv, int head_dim, int n_splits, int window,
                                            float scale, const float* sink, const float* slopes,
                                            long long pool_pages, int* err, void* stream) {
    return decode_entry(q, k_pages, v_pages, page_table, max_pages, page_size, row_pos, row_slot, out,
                        nullptr, R, nq, nkv, head_dim, n_splits, window, 0, scale, sink, slopes, 0.0f, 1, pool_pages,
                        err, stream);
}

// ---------------------------------------------------------------------------
// The same kernel behind an entry point that allocates nothing (noalloc.h).
// Its split partials live in this file-scope device array instead of a buffer
// the caller allocates.  In host code the array's name is only a stand-in for
// the device symbol, never a device address, so the address is asked for once
// per device, with that device current, and that pointer is what the kernel
// gets.
namespace {

static __device__ __align__(256) float g_noalloc_partial[RFX_NOALLOC_SCRATCH_FLOATS];

constexpr int NOALLOC_MAX_DEVICES = 64;
float* g_noalloc_ptr[NOALLOC_MAX_DEVICES] = {};
std::mutex g_noalloc_mu;

// Device address of the array on the current device; looked up on the first
// call per device.
int noalloc_scratch(float** out) {
    int dev = -1;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return (int)e;
    if (dev < 0 || dev >= NOALLOC_MAX_DEVICES) return RFX_ERR_UNSUPPORTED;
    std::lock_guard<std::mutex> lock(g_noalloc_mu);
    if (!g_noalloc_ptr[dev]) {
        float* p = nullptr;
        e = cudaGetSymbolAddress((void**)&p, g_noalloc_partial);
        if (e != cudaSuccess) return (int)e;
        g_noalloc_ptr[dev] = p;
    }
    *out = g_noalloc_ptr[dev];
    return 0;
}

}  // namespace

// Tuning aid: give the decode attention kernel a device buffer of launches * ctas
// records of twelve 64-bit words (time stamps and cycle counts); the next launch writes record 0.  Null turns
// it off.
extern "C" int rfx_attention_decode_trace(void* buffer, int launches, int ctas) {
    g_dtrace_next = 0;
    DecTraceRec* p = (DecTraceRec*)buffer;
    cudaError_t e = cudaMemcpyToSymbol(g_dtrace, &p, sizeof(p));
    if (e == cudaSuccess) e = cudaMemcpyToSymbol(g_dtrace_ctas, &ctas, sizeof(int));
    if (e == cudaSuccess) e = cudaMemcpyToSymbol(g_dtrace_launches, &launches, sizeof(int));
    return (int)e;
}

extern "C" long long rfx_attention_decode_noalloc_capacity(void) {
    return (long long)RFX_NOALLOC_SCRATCH_FLOATS;
}

extern "C" int rfx_attention_decode_noalloc(const void* q, const void* k_pages, const void* v_pages,
                                            const int* page_table, int max_pages, int page_size,
                                            const int* row_pos, const int* row_slot, void* out, int R,
                                            int nq, int nkv, int head_dim, int n_splits, int window,
                                            float scale, void* stream) {
    if (R <= 0) return 0;
    if (n_splits < 1 || nq <= 0 || head_dim <= 0) return RFX_ERR_BAD_ARG;
    const long long need = (long long)R * nq * n_splits * (head_dim + 2);
    if (n_splits > 1 && need > (long long)RFX_NOALLOC_SCRATCH_FLOATS) return RFX_ERR_SCRATCH;
    float* scratch = nullptr;
    const int st = noalloc_scratch(&scratch);
    if (st != 0) return st;
    // every split writes its whole partial (empty splits write max = -inf, sum = 0)
    // before the combine reads it, so nothing in the array has to start at zero
    return rfx_attention_decode(q, k_pages, v_pages, page_table, max_pages, page_size, row_pos,
                                row_slot, out, scratch, R, nq, nkv, head_dim, n_splits, window, scale,
                                nullptr, nullptr, 0, nullptr, stream);
}
