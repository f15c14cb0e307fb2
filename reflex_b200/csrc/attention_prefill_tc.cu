// Prefill attention on the 5th-generation tensor cores (tcgen05 + TMEM + TMA).
//
// Same problem as attention_prefill.cu (causal, optionally windowed
// grouped-query attention of a packed batch over the paged cache; a CTA =
// one sequence, one kv head, 128 rows that are (position, head of the group)
// pairs), for head sizes 64 and 128.  Per page of 64 keys:
//   S = Q K^T      tcgen05.mma, Q [128 x D] and the K page [64 x D] in shared
//                  memory (TMA, 128-byte swizzle), S [128 x 64] float32 in TMEM;
//   softmax        four warps, one thread per row: tcgen05.ld its row of S,
//                  mask, running max and sum in 32-bit, P as bfloat16 back into
//                  TMEM over the columns S came from (tcgen05.st);
//   O += P V       tcgen05.mma with P from TMEM and the V page as the MN-major
//                  shared-memory operand, O [128 x D] accumulating in TMEM.
// The running maximum is a reference, not the exact maximum: it is raised (and
// the row of O rescaled through tcgen05.ld / tcgen05.st) only when a page's
// maximum passes it by more than 2^8, so rescaling is rare; probabilities are
// 2^(s - reference) <= 2^8 and the final division by the sum, taken with the
// same reference, gives the exact softmax.  S and P are double-buffered so the
// tensor core works on page j + 1 while the softmax warps are on page j.  Warp 0 issues TMA loads, warp 1 issues
// MMAs, warps 2..5 are the softmax rows.  Every mbarrier wait is bounded; on a
// timeout the kernel records it, stops, frees its tensor memory and returns.
// The reference's tiled kernel is the CUDA-core ancestor
// (src/kernels_cuda/attention_tiled.cuh:73-296).
#include <map>
#include <mutex>
#include <tuple>

#include "attn_mma.cuh"
#include "common.cuh"
#include "paged.cuh"
#include "sm100.cuh"
#include "tma_host.cuh"

namespace {

// Optional timeline for tuning: when a buffer is set (rfx_attention_prefill_tc_trace),
// chosen threads store %globaltimer at a few places of a CTA's life (32 slots per
// CTA); the last launch wins.
static __device__ unsigned long long* g_trace = nullptr;
static __device__ int g_trace_ctas = 0;
__device__ __forceinline__ void trace_mark(int which) {
    if (g_trace == nullptr) return;
    const int cta = (blockIdx.z * gridDim.y + blockIdx.y) * gridDim.x + blockIdx.x;
    if (cta >= g_trace_ctas) return;
    unsigned long long t;
    asm volatile("mov.u64 %0, %globaltimer;" : "=l"(t));
    g_trace[(size_t)cta * 32 + which] = t;
}

// a raw value (cycles spent in a wait, summed) instead of a timestamp
__device__ __forceinline__ void trace_value(int which, long long v) {
    if (g_trace == nullptr) return;
    const int cta = (blockIdx.z * gridDim.y + blockIdx.y) * gridDim.x + blockIdx.x;
    if (cta >= g_trace_ctas) return;
    g_trace[(size_t)cta * 32 + which] = (unsigned long long)v;
}

using namespace sm100;
using rfx::PagedKV;

constexpr int PAGE = 64;
constexpr int ROWS = 128;
constexpr int THREADS = 192;
constexpr int KV_STAGES = 2;  // with 97 KB of shared memory two CTAs share an SM

// 3-D tile load (x innermost)
__device__ __forceinline__ void tma_load_3d(void* smem_dst, const CUtensorMap* map, uint64_t* bar,
                                            int x, int y, int z) {
    asm volatile(
        "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes"
        " [%0], [%1, {%3, %4, %5}], [%2];"
        ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(map)), "r"(smem_u32(bar)),
          "r"(x), "r"(y), "r"(z)
        : "memory");
}
// 2^x, hardware approximation (about 2 ulp; the result is rounded to bfloat16)
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void fence_async_proxy() {
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}
// MN-major operand, 128-byte swizzle: 64 elements contiguous per k-row, k-rows
// 128 bytes apart, groups of 8 k-rows `sbo` bytes apart, blocks of 64 elements
// along MN `lbo` bytes apart.
__device__ __forceinline__ uint64_t umma_desc_mn_sw128(uint32_t smem_addr, uint32_t lbo, uint32_t sbo) {
    uint64_t d = 0;
    d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
    d |= (uint64_t)(lbo >> 4) << 16;
    d |= (uint64_t)(sbo >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
// kind::f16, A bfloat16 K-major, B bfloat16 MN-major, D float32
__host__ __device__ constexpr uint32_t idesc_b_mn(int M, int N) {
    return umma_idesc_bf16(M, N) | (1u << 16);
}

struct Bars {
    uint64_t q_full, k_full[KV_STAGES], k_empty[KV_STAGES], v_full[KV_STAGES], v_empty[KV_STAGES], s_full[2], p_full[2],
        o_full;
    uint32_t tmem_base;
    int abort_flag;
};

// Value tiles in flight: two, or one where keys wider than values would otherwise keep a second
// CTA off the SM.
constexpr int v_stages(int DK, int DV) { return DK > DV ? 1 : KV_STAGES; }

struct Smem {
    // all tiles 1024-byte aligned
    static constexpr int tiles(int DK, int DV) {
        return ROWS * DK * 2 + KV_STAGES * PAGE * DK * 2 + v_stages(DK, DV) * PAGE * DV * 2;
    }
    // paged: slack to align the tiles (the barriers are static); contiguous: the barriers lie
    // behind the tiles and the block's shared memory is all dynamic, so it starts aligned
    static constexpr int total(int DK, int DV, bool contig) {
        return tiles(DK, DV) + (contig ? (int)sizeof(Bars) : 1024);
    }
};

// 16 neighbouring gate logits; the place is a multiple of 16 bytes
__device__ __forceinline__ void load_logits16(const rfx::RowGate& gate, size_t at, float (&z)[16]) {
    if (gate.bf16) {
        const __nv_bfloat16* p = reinterpret_cast<const __nv_bfloat16*>(gate.z) + at;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const uint4 u = reinterpret_cast<const uint4*>(p)[i];
            const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float2 f = __bfloat1622float2(h[j]);
                z[8 * i + 2 * j] = f.x;
                z[8 * i + 2 * j + 1] = f.y;
            }
        }
    } else {
        const float4* p = reinterpret_cast<const float4*>(reinterpret_cast<const float*>(gate.z) + at);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float4 f = p[i];
            z[4 * i] = f.x, z[4 * i + 1] = f.y, z[4 * i + 2] = f.z, z[4 * i + 3] = f.w;
        }
    }
}

// SLOPES: a linear distance bias, slope_h * (query position - key position) off
// every score of head h; taken off the raw score as (slope / scale) * distance,
// so that the scale's multiply-add in the exponent covers it.  Without it the
// kernel's instructions are what they were.
// MODE 1: slopes.  MODE 2, 3: capped scores, cap * tanh(s scale / cap): the tanh of s * `in_scale`
// takes the raw score's place and `scale_log2` is cap * log2(e), so the rest of the page's code
// is the same.  MODE 2 takes any argument; MODE 3 the polynomial for |s in_scale| <= 1/2, which
// leaves the special-function unit to the softmax's exponentials.
// CONTIG: keys and values are not pages but the rows of one matrix (a latent's keys and
// values made for this step): position p of sequence i is row seq_base[i] + p, head h's key its
// columns h DK .., its value its columns v_col + h DV .. (map_k and map_v then are the same
// matrix).  `dv` columns of a value are written out (DV without CONTIG).
// `gate`: a head's output times one number a row and head, or (CONTIG) element by element.
template <int DK, int DV, int MODE, bool CONTIG>
__global__ void __launch_bounds__(THREADS)
attention_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q,
                            const __grid_constant__ CUtensorMap map_k,
                            const __grid_constant__ CUtensorMap map_v, PagedKV cache,
                            const int* __restrict__ seq_slot, const int* __restrict__ seq_start,
                            const int* __restrict__ seq_new, const int* __restrict__ seq_row0,
                            __nv_bfloat16* __restrict__ out, int nq, int bq, int window, int keep_first,
                            float scale_log2, float in_scale, const float* __restrict__ sink,
                            const float* __restrict__ slopes, const int* __restrict__ seq_base, int v_col, int dv,
                            rfx::RowGate gate, int* __restrict__ err) {
    constexpr bool SLOPES = MODE == 1;
    static_assert(DK % 64 == 0 && DK <= 192 && (DV == 64 || DV == 128), "keys up to 192, values 64 or 128");
    constexpr int KB = DK / 64, VB = DV / 64;  // 64-column blocks of a row
    constexpr int K_BYTES = PAGE * DK * 2, V_BYTES = PAGE * DV * 2;
    constexpr int VS = v_stages(DK, DV);
    constexpr uint32_t TMEM_COLS = 256;
    // S: 2 x 64 columns (P_b, 32 columns of packed bfloat16, overwrites the start
    // of S_b once the row has read it), then O: DV columns
    constexpr uint32_t S_COL = 0, O_COL = 128;

    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    Bars* bars;
    if constexpr (CONTIG) {
        if (base != smem_raw) {  // every thread alike: nothing has been set up yet
            rfx::pdl_prologue();
            if (threadIdx.x == 0) atomicExch(err, 26);
            return;
        }
        bars = reinterpret_cast<Bars*>(base + Smem::tiles(DK, DV));
    } else {
        __shared__ __align__(8) Bars bars_static;
        bars = &bars_static;
    }
    uint64_t &q_full = bars->q_full, &o_full = bars->o_full;
    uint64_t *k_full = bars->k_full, *k_empty = bars->k_empty, *v_full = bars->v_full, *v_empty = bars->v_empty,
             *s_full = bars->s_full, *p_full = bars->p_full;
    uint32_t& tmem_base_smem = bars->tmem_base;
    int& abort_flag = bars->abort_flag;
    uint8_t* q_tile = base;
    uint8_t* k_ring = q_tile + ROWS * DK * 2;
    uint8_t* v_ring = k_ring + KV_STAGES * K_BYTES;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) trace_mark(0);  // 0 entry, 1 set up, 2 first scores, 3 last page done, 4 output written, 5 exit
    // CTAs are handed out with x fastest: kv heads and sequences vary fastest and
    // the tile slowest, so that the longest tiles of every head start first
    const int kvh = blockIdx.x, seq = blockIdx.y;
    const int n_new = seq_new[seq];
    const int q0 = (gridDim.z - 1 - blockIdx.z) * bq;  // the longest tiles first
    const bool active = q0 < n_new;
    const int g = nq / cache.n_kv_heads;
    const int slot = seq_slot[seq], start = seq_start[seq], row0 = seq_row0[seq];
    const int n_pos = active ? min(bq, n_new - q0) : 0;
    const int n_rows = n_pos * g;
    const int pos_first = start + q0, pos_last = pos_first + n_pos - 1;
    const int lo_tile = (window > 0 && pos_first + 1 > window) ? pos_first + 1 - window : 0;
    const int pg0 = lo_tile / PAGE, pg1 = active ? pos_last / PAGE + 1 : 0;
    // The first `keep_first` positions stay visible beyond the window: the pages that hold
    // such positions and lie before the window's first page are walked first, then the
    // window's; entry j of that list is page `logical(j)` of the sequence.
    const int kp = min((min(keep_first, lo_tile) + PAGE - 1) / PAGE, pg0);
    auto logical = [&](int j) { return j < kp ? j : pg0 + j - kp; };
    const int n_pages = active ? kp + pg1 - pg0 : 0;

    if (threadIdx.x == 0) {
        mbar_init(&q_full, 1);
        for (int i = 0; i < KV_STAGES; ++i) {
            mbar_init(&k_full[i], 1);
            mbar_init(&k_empty[i], 1);
            mbar_init(&v_full[i], 1);
            mbar_init(&v_empty[i], 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(&s_full[i], 1);
            mbar_init(&p_full[i], 4);
        }
        mbar_init(&o_full, 1);
        abort_flag = 0;
        fence_barrier_init();
    }
    if (warp == 1) {
        tmem_alloc(&tmem_base_smem, TMEM_COLS);
        tmem_relinquish();
    }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = tmem_base_smem;
    rfx::pdl_prologue();  // q and this step's keys and values come from the kernel before
    if (threadIdx.x == 0) trace_mark(1);

    if (!active) {
        // nothing to do for this tile; fall through to the teardown
    } else if (warp == 0) {
        if (elect_one()) {
            const int* table = cache.page_table + (size_t)slot * cache.max_pages;
            mbar_expect_tx(&q_full, (uint32_t)(bq * g * 128 * KB));
            for (int kb = 0; kb < KB; ++kb)
                tma_load_3d(q_tile + kb * ROWS * 128, &map_q, &q_full, kb * 64, kvh * g, row0 + q0);
            // the tile's first row in the store (or in the matrix), and its first columns
            const int row_base = CONTIG ? seq_base[seq] : 0;
            auto y_of = [&](int j) {
                return CONTIG ? row_base + logical(j) * PAGE : (table[logical(j)] * cache.n_kv_heads + kvh) * PAGE;
            };
            const int kx = CONTIG ? kvh * DK : 0, vx = CONTIG ? v_col + kvh * DV : 0;
            auto load_k = [&](int j, int y) -> bool {
                const int s = j % KV_STAGES;
                if (!mbar_wait(&k_empty[s], ((j / KV_STAGES) & 1) ^ 1)) { atomicExch(err, 11); return false; }
                mbar_expect_tx(&k_full[s], K_BYTES);
                for (int kb = 0; kb < KB; ++kb)
                    tma_load_2d(k_ring + s * K_BYTES + kb * PAGE * 128, &map_k, &k_full[s], kx + kb * 64, y);
                return true;
            };
            auto load_v = [&](int j, int y) -> bool {
                const int s = j % VS;
                if (!mbar_wait(&v_empty[s], ((j / VS) & 1) ^ 1)) { atomicExch(err, 12); return false; }
                mbar_expect_tx(&v_full[s], V_BYTES);
                for (int kb = 0; kb < VB; ++kb)
                    tma_load_2d(v_ring + s * V_BYTES + kb * PAGE * 128, &map_v, &v_full[s], vx + kb * 64, y);
                return true;
            };
            bool ok = true;
            if constexpr (VS == 1) {
                // one value tile: the next page's keys are asked for before this page's values, whose
                // tile comes free late
                int y_next = y_of(0);
                ok = load_k(0, y_next);
                for (int j = 0; j < n_pages && ok; ++j) {
                    const int y = y_next;
                    if (j + 1 < n_pages) {
                        y_next = y_of(j + 1);
                        ok = load_k(j + 1, y_next);
                    }
                    ok = ok && load_v(j, y);
                }
            } else {
                for (int j = 0; j < n_pages && ok; ++j) {
                    const int y = y_of(j);
                    ok = load_k(j, y) && load_v(j, y);
                }
            }
            if (!ok) abort_flag = 1;
        }
        __syncwarp();
    } else if (warp == 1) {
        if (elect_one()) {
            constexpr uint32_t idesc_s = umma_idesc_bf16(ROWS, PAGE);  // S: N = 64 keys
            constexpr uint32_t idesc_o = idesc_b_mn(ROWS, DV);         // O: N = DV, V is MN-major
            const bool tracing = g_trace != nullptr;
            long long wait_k = 0, wait_p = 0, wait_v = 0, c0 = 0;
            bool ok = mbar_wait(&q_full, 0);
            if (!ok) { atomicExch(err, 13); abort_flag = 1; }
            auto pv = [&](int i) -> bool {
                const int b = i & 1, s = i % VS;
                const uint32_t ph2 = (i >> 1) & 1, phs = (i / VS) & 1;
                // P_i is delivered after any rescaling of O that page i asked for
                if (tracing) c0 = clock64();
                if (!mbar_wait(&p_full[b], ph2)) { atomicExch(err, 14); return false; }
                if (tracing) { const long long c1 = clock64(); wait_p += c1 - c0; c0 = c1; }
                if (!mbar_wait(&v_full[s], phs)) { atomicExch(err, 15); return false; }
                if (tracing) wait_v += clock64() - c0;
                tc_fence_after_sync();
                const uint32_t va = smem_u32(v_ring + s * V_BYTES);
#pragma unroll
                for (int k = 0; k < PAGE / 16; ++k) {  // 16 keys per MMA: 8 packed columns of P
                    const uint64_t db = umma_desc_mn_sw128(va + k * 16 * 128, PAGE * 128, 1024);
                    umma_bf16_ts(tmem + O_COL, tmem + S_COL + b * PAGE + k * 8, db, idesc_o,
                                 (i > 0 || k > 0) ? 1u : 0u);
                }
                umma_commit(&v_empty[s]);
                umma_commit(&o_full);
                return true;
            };
            for (int j = 0; j < n_pages && ok; ++j) {
                const int b = j & 1, s = j % KV_STAGES;
                const uint32_t phs = (j / KV_STAGES) & 1;
                // S_j reuses the columns of S_{j-2} and P_{j-2}: PV_{j-2} was issued
                // before this and the tensor core runs MMAs in issue order
                if (tracing) c0 = clock64();
                if (!mbar_wait(&k_full[s], phs)) { atomicExch(err, 18); ok = false; break; }
                if (tracing) wait_k += clock64() - c0;
                tc_fence_after_sync();
                const uint32_t qa = smem_u32(q_tile), ka = smem_u32(k_ring + s * K_BYTES);
#pragma unroll
                for (int kb = 0; kb < KB; ++kb)
#pragma unroll
                    for (int k = 0; k < 4; ++k) {
                        const uint64_t da = umma_desc_k_sw128(qa + kb * ROWS * 128) + 2 * k;
                        const uint64_t db = umma_desc_k_sw128(ka + kb * PAGE * 128) + 2 * k;
                        umma_bf16(tmem + S_COL + b * PAGE, da, db, idesc_s, (kb > 0 || k > 0) ? 1u : 0u);
                    }
                umma_commit(&k_empty[s]);
                umma_commit(&s_full[b]);
                if (j > 0) ok = pv(j - 1);
            }
            if (ok && n_pages > 0) ok = pv(n_pages - 1);
            if (!ok) abort_flag = 1;
            if (tracing) {
                trace_value(8, wait_k);
                trace_value(9, wait_p);
                trace_value(10, wait_v);
            }
        }
        __syncwarp();
    } else {
        // softmax rows: this thread owns row t (TMEM lane t) of the tile
        const int qd = warp & 3;
        const int t = qd * 32 + lane;
        const uint32_t lane_addr = (uint32_t)(qd * 32) << 16;
        const bool row_valid = t < n_rows;
        const int row_p = t / g, row_h = t % g;
        const int row_pos = row_valid ? pos_first + row_p : -1;
        const int row_lo = (window > 0 && row_pos + 1 > window) ? row_pos + 1 - window : 0;
        const int lo_last = (window > 0 && pos_last + 1 > window) ? pos_last + 1 - window : 0;
        // the row's head's slope in units of the raw score (a weight: read before any wait)
        float slope_raw = 0.0f;
        if constexpr (SLOPES) slope_raw = slopes[kvh * g + min(row_h, g - 1)] * 1.4426950408889634f / scale_log2;
        constexpr float RAISE = 8.0f;  // raise the reference maximum only past 2^8
        float m = -INFINITY, l = 0.0f;
        bool ok = true;
        const bool tracing = g_trace != nullptr && t == 0;
        long long wait_s = 0, c0 = 0;

        for (int j = 0; j < n_pages && ok; ++j) {
            const int b = j & 1;
            const uint32_t ph2 = (j >> 1) & 1;
            if (tracing) c0 = clock64();
            if (!mbar_wait(&s_full[b], ph2)) { atomicExch(err, 22); ok = false; break; }
            if (tracing) wait_s += clock64() - c0;
            tc_fence_after_sync();
            if (t == 0 && j == 0) trace_mark(2);
            uint32_t sr[PAGE];
#pragma unroll
            for (int c = 0; c < PAGE / 16; ++c)
                tmem_ld_16_nowait(tmem + lane_addr + S_COL + b * PAGE + c * 16, sr + c * 16);
            tmem_ld_wait();

            const int basej = logical(j) * PAGE;
            // every key of the page visible to every valid row of the tile: no compares
            const bool all_visible = basej + PAGE - 1 <= pos_first && (basej >= lo_last || basej + PAGE <= keep_first) &&
                                     n_rows == ROWS;
            // four independent chains each for the maximum and the sum: one warp per
            // scheduler has nothing else to hide a dependent chain's latency with
            float s[PAGE];  // raw scores; the scale (positive) goes into the exponent's multiply-add
            float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            if constexpr (SLOPES) {
                const float d0 = (float)(row_pos - basej);  // distance of the page's first key
#pragma unroll
                for (int c = 0; c < PAGE; ++c)
                    sr[c] = __float_as_uint(fmaf(-slope_raw, d0 - (float)c, __uint_as_float(sr[c])));
            }
            if constexpr (MODE == 2) {
#pragma unroll
                for (int c = 0; c < PAGE; ++c)
                    sr[c] = __float_as_uint(
                        attn::capped_log2(__uint_as_float(sr[c]), 2.0f * 1.4426950408889634f * in_scale, 1.0f));
            }
            if constexpr (MODE == 3) {
#pragma unroll
                for (int c = 0; c < PAGE; ++c)
                    sr[c] = __float_as_uint(attn::tanh_small(__uint_as_float(sr[c]) * in_scale));
            }
            if (all_visible) {
#pragma unroll
                for (int c = 0; c < PAGE; ++c) s[c] = __uint_as_float(sr[c]);
#pragma unroll
                for (int c = 0; c < PAGE; c += 8)  // two new values per maximum: a three-input instruction
#pragma unroll
                    for (int k = 0; k < 4; ++k) mx4[k] = fmaxf(fmaxf(mx4[k], s[c + 2 * k]), s[c + 2 * k + 1]);
            } else {
#pragma unroll
                for (int c = 0; c < PAGE; ++c) {
                    const int key = basej + c;
                    s[c] = (key <= row_pos && (key >= row_lo || key < keep_first)) ? __uint_as_float(sr[c]) : -INFINITY;
                    mx4[c & 3] = fmaxf(mx4[c & 3], s[c]);
                }
            }
            const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * scale_log2;
            // the reference maximum moves only when it must
            float corr = 1.0f;
            const bool raise = mx > m + RAISE || (m == -INFINITY && mx != -INFINITY);
            if (raise) {
                corr = (m == -INFINITY) ? 0.0f : ex2(m - mx);
                m = mx;
                l *= corr;
            }
            // rows that have seen no key yet: every s is -inf, shift by 0 gives p = 0
            const float shift = (m == -INFINITY) ? 0.0f : m;
            float rs4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            uint32_t packed[PAGE / 2];
#pragma unroll
            for (int c = 0; c < PAGE; c += 2) {
                const float e0 = ex2(fmaf(s[c], scale_log2, -shift));
                const float e1 = ex2(fmaf(s[c + 1], scale_log2, -shift));
                rs4[(c >> 1) & 3] += e0 + e1;
                __nv_bfloat162 h = __floats2bfloat162_rn(e0, e1);
                packed[c / 2] = *reinterpret_cast<uint32_t*>(&h);
            }
            l += (rs4[0] + rs4[1]) + (rs4[2] + rs4[3]);

            // rescale this row of O if its reference moved (whole warp together:
            // the TMEM accesses are warp-wide; lanes that did not move scale by 1)
            if (j > 0 && __any_sync(0xffffffffu, raise)) {
                if (!mbar_wait(&o_full, (uint32_t)((j - 1) & 1))) { atomicExch(err, 21); ok = false; break; }
                tc_fence_after_sync();
#pragma unroll
                for (int c = 0; c < DV / 16; ++c) {
                    uint32_t o[16];
                    tmem_ld_16_nowait(tmem + lane_addr + O_COL + c * 16, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * corr);
                    tmem_st_16(tmem + lane_addr + O_COL + c * 16, o);
                }
                tmem_st_wait();
                tc_fence_before_sync();
            }

            // row t of P into TMEM, over the columns its S came from
            tmem_st_16(tmem + lane_addr + S_COL + b * PAGE, packed);
            tmem_st_16(tmem + lane_addr + S_COL + b * PAGE + 16, packed + 16);
            tmem_st_wait();
            // the last page may hold keys past this tile's last position whose
            // value rows were never written: zero them, 0 * NaN would not be 0 (a matrix has no such
            // rows: what lies behind a sequence is the next one's, and zeros behind the last)
            const int valid_keys = CONTIG ? PAGE : pos_last + 1 - basej;
            if (valid_keys < PAGE) {
                const int sidx = j % VS;
                if (!mbar_wait(&v_full[sidx], (j / VS) & 1)) { atomicExch(err, 24); ok = false; break; }
                uint8_t* vt = v_ring + sidx * V_BYTES;
                for (int i = t; i < (PAGE - valid_keys) * VB * 8; i += ROWS) {
                    const int rrow = valid_keys + i / (VB * 8), rem = i % (VB * 8);
                    *reinterpret_cast<uint4*>(vt + (rem / 8) * PAGE * 128 + rrow * 128 + (rem % 8) * 16) =
                        make_uint4(0, 0, 0, 0);
                }
            }
            if (valid_keys < PAGE) fence_async_proxy();
            tc_fence_before_sync();
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[b]);
        }
        if (t == 0) trace_mark(3);
        if (tracing) trace_value(11, wait_s);
        if (ok && n_pages > 0) {
            if (!mbar_wait(&o_full, (uint32_t)((n_pages - 1) & 1))) { atomicExch(err, 25); ok = false; }
        }
        if (ok && n_pages > 0) {
            tc_fence_after_sync();
            // a sink adds exp(sink - reference) to the denominator, once, with no value
            float inv = 1.0f / (sink ? l + ex2(fmaf(sink[kvh * g + row_h], 1.4426950408889634f, -m)) : l);
            if (!CONTIG && gate.z && row_valid) inv *= gate.factor(row0 + q0 + row_p, kvh * g + row_h);
            const int ow = CONTIG ? dv : DV;  // columns of an output head
            __nv_bfloat16* o = out + ((size_t)(row0 + q0 + row_p) * nq + kvh * g + row_h) * ow;
            // two loads of 16 columns in flight: the next one travels while this one is stored
            uint32_t rr[2][16];
            tmem_ld_16_nowait(tmem + lane_addr + O_COL, rr[0]);
            // an element gate's next 16 logits travel likewise, 16 bytes an access
            const bool element_gate = CONTIG && gate.z != nullptr;
            const size_t gate_at = (size_t)(row0 + q0 + row_p) * gate.ld + gate.col + (size_t)(kvh * g + row_h) * ow;
            float zz[2][16];
            if (element_gate && row_valid) load_logits16(gate, gate_at, zz[0]);
#pragma unroll
            for (int c = 0; c < DV / 16; ++c) {
                tmem_ld_wait_16(rr[c & 1]);
                if (c + 1 < DV / 16) tmem_ld_16_nowait(tmem + lane_addr + O_COL + (c + 1) * 16, rr[(c + 1) & 1]);
                uint32_t(&r)[16] = rr[c & 1];
                if (row_valid && (!CONTIG || c * 16 < ow)) {
                    if (element_gate) {
                        if ((c + 1) * 16 < ow) load_logits16(gate, gate_at + (c + 1) * 16, zz[(c + 1) & 1]);
#pragma unroll
                        for (int e = 0; e < 16; ++e)
                            r[e] = __float_as_uint(__fdividef(__uint_as_float(r[e]), 1.0f + __expf(-zz[c & 1][e])));
                    }
                    uint4 v[2];
                    __nv_bfloat162* pv2 = reinterpret_cast<__nv_bfloat162*>(v);
#pragma unroll
                    for (int e = 0; e < 8; ++e)
                        pv2[e] = __floats2bfloat162_rn(__uint_as_float(r[2 * e]) * inv, __uint_as_float(r[2 * e + 1]) * inv);
                    *reinterpret_cast<uint4*>(o + c * 16) = v[0];
                    *reinterpret_cast<uint4*>(o + c * 16 + 8) = v[1];
                }
            }
        }
        if (t == 0) trace_mark(4);
        tc_fence_before_sync();
    }

    __syncthreads();
    if (threadIdx.x == 0) trace_mark(5);
    if (warp == 1) {
        tc_fence_after_sync();
        tmem_dealloc(tmem, TMEM_COLS);
    }
}

// ---- host ---------------------------------------------------------------------
using rfx::tma::encode_fn;
using rfx::tma::EncodeTiledFn;

// q [R, nq, D]: dims (D, nq, R), a box of 64 columns x g heads x bq positions
bool make_map_q(CUtensorMap* map, const void* base, int R, int nq, int D, int g, int bq) {
    EncodeTiledFn fn = encode_fn();
    if (!fn) return false;
    cuuint64_t dims[3] = {(cuuint64_t)D, (cuuint64_t)nq, (cuuint64_t)R};
    cuuint64_t strides[2] = {(cuuint64_t)D * 2, (cuuint64_t)nq * D * 2};
    cuuint32_t box[3] = {64, (cuuint32_t)g, (cuuint32_t)bq};
    cuuint32_t estr[3] = {1, 1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int D, int MODE>
int launch_tc(const void* q, const void* k_pages, const void* v_pages, long long n_pages_total,
              const PagedKV& cache, const int* seq_slot, const int* seq_start, const int* seq_new,
              const int* seq_row0, void* out, int S, int max_new, int R, int nq, int window, int keep_first,
              float scale, const float* sink, const float* slopes, float softcap, rfx::RowGate gate, int* err,
              cudaStream_t s) {
    const int g = nq / cache.n_kv_heads;
    if (g > ROWS) return RFX_ERR_UNSUPPORTED;
    const int bq = ROWS / g;
    CUtensorMap mq, mk, mv;
    const long long kv_rows = n_pages_total * cache.n_kv_heads * PAGE;
    if (!make_map_q(&mq, q, R, nq, D, g, bq) || !rfx::tma::make_map_rows64(&mk, k_pages, kv_rows, D, PAGE) ||
        !rfx::tma::make_map_rows64(&mv, v_pages, kv_rows, D, PAGE))
        return RFX_ERR_UNSUPPORTED;
    const size_t smem = Smem::total(D, D, false);
    auto kernel = attention_prefill_tc_kernel<D, D, MODE, false>;
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    if ((max_new + bq - 1) / bq > 65535 || S > 65535) return RFX_ERR_UNSUPPORTED;
    dim3 grid(cache.n_kv_heads, S, (max_new + bq - 1) / bq);
    if (grid.y > 65535 || grid.z > 65535) return RFX_ERR_UNSUPPORTED;
    RFX_LAUNCH(kernel, grid, THREADS, smem, s, mq, mk, mv, cache, seq_slot, seq_start, seq_new, seq_row0,
               (__nv_bfloat16*)out, nq, bq, window, keep_first,
               (MODE >= 2 ? softcap : scale) * 1.4426950408889634f, MODE >= 2 ? scale / softcap : 1.0f, sink, slopes,
               (const int*)nullptr, 0, D, gate, err);
    return 0;
}

// [rows, cols] bfloat16, row-major: boxes of 64 columns x 64 rows (rows beyond: zeros)
bool make_map_matrix(CUtensorMap* map, const void* base, long long rows, long long cols) {
    EncodeTiledFn fn = encode_fn();
    if (!fn) return false;
    cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    cuuint64_t strides[1] = {(cuuint64_t)cols * 2};
    cuuint32_t box[2] = {64, PAGE};
    cuuint32_t estr[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int DK, int DV>
int launch_contig(const void* q, const void* kv, long long kv_rows, const int* seq_base, const int* seq_slot,
                  const int* seq_start, const int* seq_new, const int* seq_row0, void* out, int S, int max_new, int R,
                  int heads, int dv, int window, float scale, const float* sink, rfx::RowGate gate, int* err,
                  cudaStream_t s) {
    CUtensorMap mq, mkv;
    if (!make_map_q(&mq, q, R, heads, DK, 1, ROWS) ||
        !make_map_matrix(&mkv, kv, kv_rows, (long long)heads * (DK + DV)))
        return RFX_ERR_UNSUPPORTED;
    const size_t smem = Smem::total(DK, DV, true);
    auto kernel = attention_prefill_tc_kernel<DK, DV, 0, true>;
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    dim3 grid(heads, S, (max_new + ROWS - 1) / ROWS);
    if (grid.y > 65535 || grid.z > 65535) return RFX_ERR_UNSUPPORTED;
    PagedKV cache{nullptr, 0, PAGE, heads, DK};
    RFX_LAUNCH(kernel, grid, THREADS, smem, s, mq, mkv, mkv, cache, seq_slot, seq_start, seq_new, seq_row0,
               (__nv_bfloat16*)out, heads, ROWS, window, 0, scale * 1.4426950408889634f, 1.0f, sink,
               (const float*)nullptr, seq_base, heads * DK, dv, gate, err);
    return 0;
}

}  // namespace

// As rfx_attention_prefill, for head_dim 64 or 128.  `n_pages_total` is the
// number of pages of the K/V store (for the TMA maps), R the number of rows of
// q.  `err` is a device word that receives a code if a bounded wait ran out.
// `slopes` (one float per query head, or null): slope * (query position - key
// position) is taken off every score; needs scale > 0.
// Tuning aid: 32 64-bit timestamps per CTA of the launches that follow (null
// switches it off).
extern "C" int rfx_attention_prefill_tc_trace(void* buffer, int ctas) {
    unsigned long long* p = (unsigned long long*)buffer;
    cudaError_t e = cudaMemcpyToSymbol(g_trace, &p, sizeof(p));
    if (e == cudaSuccess) e = cudaMemcpyToSymbol(g_trace_ctas, &ctas, sizeof(int));
    return (int)e;
}

// `keep_first`: with a window, the first so many positions of a sequence stay visible
// beyond it.  `softcap` > 0: a score s becomes softcap * tanh(s / softcap) (not with slopes);
// `score_bound` > 0: the caller's word that no |s| is larger.  `gate_z` (or null): rows of
// `gate_ld` elements; sigmoid(gate_z[r, gate_col + h]) scales what head h of row r gives.
extern "C" int rfx_attention_prefill_tc_kf(const void* q, const void* k_pages, const void* v_pages,
                                           long long n_pages_total, const int* page_table, int max_pages,
                                           int page_size, const int* seq_slot, const int* seq_start,
                                           const int* seq_new, const int* seq_row0, void* out, int S,
                                           int max_new, int R, int nq, int nkv, int head_dim, int window,
                                           int keep_first, float scale, const float* sink, const float* slopes,
                                           float softcap, float score_bound, const void* gate_z, int gate_dt,
                                           int gate_ld, int gate_col, int* err, void* stream) {
    if (S <= 0 || max_new <= 0 || R <= 0) return 0;
    rfx::RowGate gate;
    if (!rfx::row_gate(&gate, gate_z, gate_dt, gate_ld, gate_col, nq)) return RFX_ERR_BAD_ARG;
    if (keep_first < 0 || !(scale > 0.0f)) return RFX_ERR_UNSUPPORTED;  // the maximum is taken before the scale
    if (page_size != PAGE || nkv <= 0 || nq % nkv != 0) return RFX_ERR_BAD_ARG;
    if (softcap < 0.0f || (softcap > 0.0f && slopes)) return RFX_ERR_UNSUPPORTED;
    if (slopes && !(scale > 0.0f)) return RFX_ERR_UNSUPPORTED;  // the slopes ride on the scale's multiply-add
    if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_pages) |
         reinterpret_cast<uintptr_t>(v_pages)) & 15)
        return RFX_ERR_BAD_ARG;
    PagedKV cache{page_table, max_pages, page_size, nkv, head_dim};
    cudaStream_t s = (cudaStream_t)stream;
#define RFX_GO(DD, M)                                                                                   \
    launch_tc<DD, M>(q, k_pages, v_pages, n_pages_total, cache, seq_slot, seq_start, seq_new, seq_row0, \
                      out, S, max_new, R, nq, window, keep_first, scale, sink, slopes, softcap, gate, err, s)
    const int mode = slopes ? 1 : !(softcap > 0.0f) ? 0 : (score_bound > 0.0f && score_bound <= attn::TANH_SMALL * softcap) ? 3 : 2;
#define RFX_D(DD)                             \
    if (head_dim == DD) {                     \
        if (mode == 0) return RFX_GO(DD, 0);  \
        if (mode == 1) return RFX_GO(DD, 1);  \
        if (mode == 2) return RFX_GO(DD, 2);  \
        return RFX_GO(DD, 3);                 \
    }
    RFX_D(64)
    RFX_D(128)
#undef RFX_D
#undef RFX_GO
    return RFX_ERR_UNSUPPORTED;
}

extern "C" int rfx_attention_prefill_tc(const void* q, const void* k_pages, const void* v_pages,
                                        long long n_pages_total, const int* page_table, int max_pages,
                                        int page_size, const int* seq_slot, const int* seq_start,
                                        const int* seq_new, const int* seq_row0, void* out, int S,
                                        int max_new, int R, int nq, int nkv, int head_dim, int window,
                                        float scale, const float* sink, const float* slopes, int* err,
                                        void* stream) {
    return rfx_attention_prefill_tc_kf(q, k_pages, v_pages, n_pages_total, page_table, max_pages, page_size,
                                       seq_slot, seq_start, seq_new, seq_row0, out, S, max_new, R, nq, nkv,
                                       head_dim, window, 0, scale, sink, slopes, 0.0f, 0.0f, nullptr, 0, 0, 0, err, stream);
}

// Attention over keys and values that lie as rows of one matrix, one key and value per head
// and position (a latent's, made for this step): `kv` bfloat16 [kv_rows, heads * (dk + dvp)], a
// row's keys head by head, dk elements each, then its values, dvp each (dv of them used); position
// p of sequence i is row seq_base[i] + p.  q [R, heads, dk], out [R, heads, dv].  dk: 64, 128 or
// 192; dvp: 64 or 128, at most dk; dv a multiple of 16; scale > 0.  `gate_z` (or null): out[r, h, i]
// is multiplied by sigmoid(gate_z[r, gate_col + h dv + i]); gate_ld and gate_col multiples of 8.
extern "C" int rfx_attention_prefill_tc_rows(const void* q, const void* kv, long long kv_rows, const int* seq_base,
                                             const int* seq_slot, const int* seq_start, const int* seq_new,
                                             const int* seq_row0, void* out, int S, int max_new, int R, int heads,
                                             int dk, int dvp, int dv, int window, float scale, const float* sink,
                                             const void* gate_z, int gate_dt, int gate_ld, int gate_col, int* err,
                                             void* stream) {
    if (S <= 0 || max_new <= 0 || R <= 0) return 0;
    rfx::RowGate gate;
    if (!rfx::row_gate(&gate, gate_z, gate_dt, gate_ld, gate_col, heads * dv)) return RFX_ERR_BAD_ARG;
    // the logits come 16 bytes an access
    if (gate_z && (gate_ld % 8 || gate_col % 8 || (reinterpret_cast<uintptr_t>(gate_z) & 15))) return RFX_ERR_UNSUPPORTED;
    if (!(scale > 0.0f) || dv <= 0 || dv % 16 || dv > dvp || heads <= 0 || kv_rows <= 0) return RFX_ERR_UNSUPPORTED;
    if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(out)) & 15)
        return RFX_ERR_BAD_ARG;
#define RFX_CASE(A, B)                                                                                              \
    if (dk == A && dvp == B)                                                                                        \
        return launch_contig<A, B>(q, kv, kv_rows, seq_base, seq_slot, seq_start, seq_new, seq_row0, out, S,        \
                                   max_new, R, heads, dv, window, scale, sink, gate, err, (cudaStream_t)stream);
    RFX_CASE(64, 64) RFX_CASE(128, 64) RFX_CASE(128, 128) RFX_CASE(192, 64) RFX_CASE(192, 128)
#undef RFX_CASE
    return RFX_ERR_UNSUPPORTED;
}
