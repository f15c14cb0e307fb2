// The gated delta rule: a matrix memory per head, one decay and one write rate a head.
//
// Per head, with d key channels and dv value channels, and for every row
//     S <- g S                                  g in (0, 1), one number a head and row
//     u  = beta (v - S^T k)                     beta in (0, 1), likewise
//     S <- S + k u^T
//     o  = S^T q                                the read-out sees this row's write
// A head reads the q and k of head h / (heads / kv_heads).  Everything is 32-bit.
//
//  * rfx_gated_delta_prep: from the rows of a stacked product [q | k | v | ..] the short
//    causal convolution of every q, k and v channel (short_conv.cuh) and its silu; q and k
//    then become unit vectors per head, x / sqrt(sum(x^2) + unit_eps), q also times a
//    factor; and from the columns of the two gates
//        beta = sigmoid(b),   g = exp(A softplus(a + dt_bias))        (A negative)
//    A warp a head of a row.  In a step of one row a sequence the launch also moves the
//    convolution's last inputs on.
//  * rfx_gated_delta_scan: the recurrence over the step's rows, sequence by sequence.  A
//    block owns (sequence, head, some of the value columns) and walks the rows in tiles of
//    TT, copied into shared memory a tile ahead (cp.async).  Each warp walks the tile's
//    rows on its own columns with no barrier between them: KG lanes share a column, lane
//    (g, c) holds its key channels 4 (g + KG m) .. + 3 in registers (NC groups of four); the
//    KG partial sums of S^T k and of S^T q meet by shuffles.  The state lies
//    [heads][value column][key channel padded to a multiple of four].  Which block and
//    warp walks a column changes nothing of its arithmetic.
//    gated_delta_chunk.cu has the form for steps that bring a sequence many rows.
#include "attn_mma.cuh"
#include "common.cuh"
#include "short_conv.cuh"

namespace {

using namespace rfx;
using namespace rfx::conv;

__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }

constexpr int PREP_THREADS = 256;

// y / (1 + e^-y) with the hardware's exponential and reciprocal (about 2^-21 off)
__device__ __forceinline__ float silu_fast(float y) { return __fdividef(y, 1.0f + __expf(-y)); }

// NV: a head's elements in 128s, four a lane (up to 512), 0: heads whose size is no multiple of four.
// TAPS: the filters' length where it is known here (all taps' loads go out together), 0: `taps_any`.
// `fast`: the activation with the hardware's approximations (rows of the bfloat16 path).
template <int NV, int TAPS>
__global__ void __launch_bounds__(PREP_THREADS, NV <= 1 ? 5 : 2)
gated_delta_prep_kernel(const float* __restrict__ proj, int ld, int b_off, int a_off,
                        const float* __restrict__ filters, int taps_any, float* state, long long slot_stride,
                        const int* __restrict__ row_slot, const float* __restrict__ dt_bias,
                        const float* __restrict__ A, float unit_eps, float q_scale, float* __restrict__ out,
                        float* __restrict__ gates, int H, int G, int d, int dv, int update, int fast) {
    pdl_prologue();
    const int taps = TAPS ? TAPS : taps_any;
    const int r = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int unit = blockIdx.y * (PREP_THREADS / 32) + warp;
    const int C = 2 * G * d + H * dv;
    if (unit == 2 * G + H) {  // the two gates of every head: [decay | write rate]
        for (int h = lane; h < H; h += 32) {
            const float* pr = proj + (size_t)r * ld;
            gates[(size_t)r * 2 * H + h] = expf(A[h] * softplus_f(pr[a_off + h] + dt_bias[h]));
            gates[(size_t)r * 2 * H + H + h] = 1.0f / (1.0f + expf(-pr[b_off + h]));
        }
        return;
    }
    if (unit > 2 * G + H) return;
    const int width = unit < 2 * G ? d : dv;
    const int c0 = unit < 2 * G ? unit * d : 2 * G * d + (unit - 2 * G) * dv;
    const int before = rows_before(row_slot, r, taps - 1);
    float* tail = taps > 1 ? state + (size_t)row_slot[r] * slot_stride : nullptr;
    const int T = taps - 1;
    float* orow = out + (size_t)r * C + c0;
    float ss = 0.0f;
    if constexpr (NV > 0) {
        float4 y[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int e = 4 * (lane + 32 * i);
            if (e < width) {
                float4 t = conv4_at(proj, ld, 0, c0 + e, nullptr, filters, taps, tail, C, r, before);
                if (fast) { t.x = silu_fast(t.x); t.y = silu_fast(t.y); t.z = silu_fast(t.z); t.w = silu_fast(t.w); }
                else { t.x = silu_of(t.x); t.y = silu_of(t.y); t.z = silu_of(t.z); t.w = silu_of(t.w); }
                ss = fmaf(t.x, t.x, fmaf(t.y, t.y, fmaf(t.z, t.z, fmaf(t.w, t.w, ss))));
                y[i] = t;
                if (update && T > 0) {
                    for (int j = 0; j + 1 < T; ++j)
                        store4(tail + (size_t)j * C + c0 + e,
                               *reinterpret_cast<const float4*>(tail + (size_t)(j + 1) * C + c0 + e));
                    store4(tail + (size_t)(T - 1) * C + c0 + e,
                           *reinterpret_cast<const float4*>(proj + (size_t)r * ld + c0 + e));
                }
            }
        }
        float f = 1.0f;
        if (unit < 2 * G) f = (unit < G ? q_scale : 1.0f) / sqrtf(warp_sum(ss) + unit_eps);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int e = 4 * (lane + 32 * i);
            if (e < width) store4(orow + e, make_float4(y[i].x * f, y[i].y * f, y[i].z * f, y[i].w * f));
        }
    } else {
        for (int e = lane; e < width; e += 32) {
            const float t = silu_of(conv_at(proj, ld, 0, c0 + e, nullptr, filters, taps, tail, C, r, before));
            ss = fmaf(t, t, ss);
            orow[e] = t;
            if (update && T > 0) {
                for (int j = 0; j + 1 < T; ++j) tail[(size_t)j * C + c0 + e] = tail[(size_t)(j + 1) * C + c0 + e];
                tail[(size_t)(T - 1) * C + c0 + e] = proj[(size_t)r * ld + c0 + e];
            }
        }
        if (unit >= 2 * G) return;
        const float f = (unit < G ? q_scale : 1.0f) / sqrtf(warp_sum(ss) + unit_eps);
        for (int e = lane; e < width; e += 32) orow[e] *= f;  // each lane its own elements
    }
}

__device__ __forceinline__ void cp_async_4(void* smem, const void* gmem) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(attn::smem_u32(smem)), "l"(gmem) : "memory");
}

// A row of a staged tile: k [dp] | q [dp] | v [cols padded] | decay, write rate, 0, 0
template <int NC, int KG, bool V16, typename TO>
__global__ void __launch_bounds__(512)
gated_delta_scan_kernel(const float* __restrict__ qkv, const float* __restrict__ gates, float* __restrict__ state,
                        long long state_stride, long long state_off, const int* __restrict__ seq_slot,
                        const int* __restrict__ seq_row0, TO* __restrict__ out, int H, int G, int d, int dv,
                        int cols, int TT) {
    extern __shared__ __align__(16) float sm[];
    pdl_prologue();
    constexpr int CW = 32 / KG;  // columns a warp walks; KG lanes share a column
    const int seq = blockIdx.x, h = blockIdx.y, c_first = blockIdx.z * cols;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane / CW, cl = warp * CW + (lane % CW), col = c_first + cl;
    const int d4 = (d + 3) / 4, dp = 4 * d4, colsp = (cols + 3) / 4 * 4;
    const int stride = 2 * dp + colsp + 4;
    const int C = 2 * G * d + H * dv, kvh = h / (H / G);
    const int row0 = seq_row0[seq], row1 = seq_row0[seq + 1];
    const bool live = col < dv;
    float* Sg = state + (size_t)seq_slot[seq] * state_stride + state_off + ((size_t)h * dv + (live ? col : 0)) * dp;
    float S[NC][4];
#pragma unroll
    for (int m = 0; m < NC; ++m) {
        float4 s = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (live && g + KG * m < d4) s = *reinterpret_cast<const float4*>(Sg + 4 * (g + KG * m));
        S[m][0] = s.x; S[m][1] = s.y; S[m][2] = s.z; S[m][3] = s.w;
    }
    const int v_cols = min(cols, dv - c_first);
    const int q_src = kvh * d, k_src = G * d + kvh * d, v_src = 2 * G * d + h * dv + c_first;
    auto stage = [&](int t0, int buf) {
        const int nt = min(TT, row1 - t0);
        float* base = sm + (size_t)buf * TT * stride;
        if constexpr (V16) {
            const int v4 = v_cols / 4, per = 2 * d4 + v4;
            for (int e = threadIdx.x; e < nt * per; e += blockDim.x) {
                const int t = e / per, c = e - t * per;
                const float* src = qkv + (size_t)(t0 + t) * C;
                float* dst = base + (size_t)t * stride + 4 * c;
                if (c < d4) src += k_src + 4 * c;
                else if (c < 2 * d4) src += q_src + 4 * (c - d4);
                else src += v_src + 4 * (c - 2 * d4);
                attn::cp_async_16(dst, src, true);
            }
        } else {
            const int per = 2 * d + v_cols;
            for (int e = threadIdx.x; e < nt * per; e += blockDim.x) {
                const int t = e / per, c = e - t * per;
                const float* src = qkv + (size_t)(t0 + t) * C;
                float* dst = base + (size_t)t * stride;
                if (c < d) { src += k_src + c; dst += c; }
                else if (c < 2 * d) { src += q_src + (c - d); dst += dp + (c - d); }
                else { src += v_src + (c - 2 * d); dst += 2 * dp + (c - 2 * d); }
                cp_async_4(dst, src);
            }
        }
        for (int e = threadIdx.x; e < 2 * nt; e += blockDim.x) {
            const int t = e >> 1, w = e & 1;
            cp_async_4(base + (size_t)t * stride + 2 * dp + colsp + w, gates + (size_t)(t0 + t) * 2 * H + w * H + h);
        }
        attn::cp_async_commit();
    };
    if constexpr (!V16) {  // the key channels' padding stays zero: nothing copies over it
        if (dp != d) {
            for (int t = threadIdx.x; t < 2 * TT; t += blockDim.x)
                for (int e = d; e < dp; ++e) sm[(size_t)t * stride + e] = sm[(size_t)t * stride + dp + e] = 0.0f;
        }
    }
    if (row0 < row1) stage(row0, 0);
    int buf = 0;
    for (int t0 = row0; t0 < row1; t0 += TT, buf ^= 1) {
        const int nt = min(TT, row1 - t0);
        if (t0 + TT < row1) {
            stage(t0 + TT, buf ^ 1);
            attn::cp_async_wait<1>();
        } else {
            attn::cp_async_wait<0>();
        }
        __syncthreads();
        const float* base = sm + (size_t)buf * TT * stride;
        // one row: S^T k must meet before the state's step (a chain of shuffles); the rows' partial
        // sums of S^T q meet afterwards, four rows' chains side by side
        auto row = [&](int t) -> float {
            const float* tile = base + (size_t)t * stride;
            const float4* k4 = reinterpret_cast<const float4*>(tile);
            const float4* q4 = reinterpret_cast<const float4*>(tile + dp);
            const float2 gb = *reinterpret_cast<const float2*>(tile + 2 * dp + colsp);
            const float vj = tile[2 * dp + cl];
            float4 k[NC];
            float acc = 0.0f, acc1 = 0.0f;
#pragma unroll
            for (int m = 0; m < NC; ++m) {
                const int c = g + KG * m;
                k[m] = c < d4 ? k4[c] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                acc = fmaf(k[m].x, S[m][0], fmaf(k[m].y, S[m][1], acc));
                acc1 = fmaf(k[m].z, S[m][2], fmaf(k[m].w, S[m][3], acc1));
            }
            acc += acc1;
#pragma unroll
            for (int off = CW; off < 32; off <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, off);
            const float u = gb.y * fmaf(-gb.x, acc, vj);  // S^T k after the decay is g times the one before it
            float o = 0.0f, o1 = 0.0f;
#pragma unroll
            for (int m = 0; m < NC; ++m) {
                const int c = g + KG * m;
                const float4 q = c < d4 ? q4[c] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                S[m][0] = fmaf(k[m].x, u, gb.x * S[m][0]);
                S[m][1] = fmaf(k[m].y, u, gb.x * S[m][1]);
                S[m][2] = fmaf(k[m].z, u, gb.x * S[m][2]);
                S[m][3] = fmaf(k[m].w, u, gb.x * S[m][3]);
                o = fmaf(S[m][0], q.x, fmaf(S[m][1], q.y, o));
                o1 = fmaf(S[m][2], q.z, fmaf(S[m][3], q.w, o1));
            }
            return o + o1;
        };
        int t = 0;
        for (; t + 4 <= nt; t += 4) {
            float ov[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) ov[i] = row(t + i);
#pragma unroll
            for (int off = CW; off < 32; off <<= 1)
#pragma unroll
                for (int i = 0; i < 4; ++i) ov[i] += __shfl_xor_sync(0xffffffffu, ov[i], off);
            if (g == 0 && live) {
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    st<TO>(out, (size_t)(t0 + t + i) * H * dv + (size_t)h * dv + col, ov[i]);
            }
        }
        for (; t < nt; ++t) {
            float o = row(t);
#pragma unroll
            for (int off = CW; off < 32; off <<= 1) o += __shfl_xor_sync(0xffffffffu, o, off);
            if (g == 0 && live) st<TO>(out, (size_t)(t0 + t) * H * dv + (size_t)h * dv + col, o);
        }
        __syncthreads();  // this buffer is copied into again two tiles on
    }
    if (!live) return;
#pragma unroll
    for (int m = 0; m < NC; ++m)
        if (g + KG * m < d4)
            *reinterpret_cast<float4*>(Sg + 4 * (g + KG * m)) = make_float4(S[m][0], S[m][1], S[m][2], S[m][3]);
}

template <int NC, int KG>
int launch_scan(const float* qkv, const float* gates, float* state, long long state_stride, long long state_off,
                const int* seq_slot, const int* seq_row0, int n_seq, float* out, int H, int G, int d, int dv,
                int max_rows, cudaStream_t s) {
    constexpr int CW = 32 / KG;
    // value columns a block owns, whole warps of them, at most sixteen warps: fewer while the
    // blocks do not fill the SMs
    int cols = (dv + CW - 1) / CW * CW;
    if (cols > 16 * CW) {
        const int n = (dv + 16 * CW - 1) / (16 * CW);
        cols = ((dv + n - 1) / n + CW - 1) / CW * CW;
    }
    while (cols > 4 * CW && cols % (2 * CW) == 0 &&
           (long long)n_seq * H * ((dv + cols - 1) / cols) < 2 * (long long)sm_count())
        cols /= 2;
    const int blocks_z = (dv + cols - 1) / cols;
    const int dp = (d + 3) / 4 * 4, colsp = (cols + 3) / 4 * 4, stride = 2 * dp + colsp + 4;
    int TT = (40 * 1024) / (stride * (int)sizeof(float));
    if (TT > 32) TT = 32;
    if (TT >= 4) TT = TT / 4 * 4;
    if (TT > max_rows) TT = max_rows;
    if (TT < 1) TT = 1;
    const size_t smem = (size_t)2 * TT * stride * sizeof(float);
    if (smem > 200 * 1024 || blocks_z > 65535 || H > 65535) return RFX_ERR_UNSUPPORTED;
    const bool v16 = d % 4 == 0 && dv % 4 == 0 && cols % 4 == 0 &&
                     (reinterpret_cast<uintptr_t>(qkv) & 15) == 0;
    dim3 grid(n_seq, H, blocks_z);
    const int threads = cols / CW * 32;
#define RFX_GO(V)                                                                                             \
    do {                                                                                                      \
        auto kernel = gated_delta_scan_kernel<NC, KG, V, float>;                                              \
        if (smem > 48 * 1024) {                                                                               \
            cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                              \
        }                                                                                                     \
        RFX_LAUNCH(kernel, grid, threads, smem, s, qkv, gates, state, state_stride, state_off, seq_slot,      \
                   seq_row0, out, H, G, d, dv, cols, TT);                                                     \
    } while (0)
    if (v16) RFX_GO(true);
    else RFX_GO(false);
#undef RFX_GO
    return 0;
}

}  // namespace

// `proj` float32 rows whose first columns are q [G d], k [G d], v [H dv], with the write rates'
// and the decays' pre-activations at `b_off` and `a_off` (H each).  `filters` transposed,
// [taps][2 G d + H dv]; `state` the slots' last taps - 1 inputs (the vector's start).  Out:
// `out` float32 [R, 2 G d + H dv] and `gates` float32 [R, 2 H] (decays, write rates).
// `update` 1: every sequence has exactly one of the R rows, and its last inputs move on.  `fast`:
// the filters' activation with the hardware's exponential.
extern "C" int rfx_gated_delta_prep(const float* proj, int ld, int b_off, int a_off, const float* filters, int taps,
                                    float* state, long long slot_stride, const int* row_slot,
                                    const float* dt_bias, const float* A, float unit_eps, float q_scale, float* out,
                                    float* gates, int R, int H, int G, int d, int dv, int update, int fast,
                                    void* stream) {
    if (R <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || d <= 0 || dv <= 0 || taps < 1 || taps > MAX_TAPS) return RFX_ERR_BAD_ARG;
    if (taps > 1 && !state) return RFX_ERR_BAD_ARG;
    const int units = 2 * G + H + 1, per = PREP_THREADS / 32;
    dim3 grid(R, (units + per - 1) / per);
    if (grid.y > 65535) return RFX_ERR_UNSUPPORTED;
    const bool by4 = d % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && slot_stride % 4 == 0 && d <= 512 && dv <= 512 &&
                     ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(filters) |
                       reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    cudaStream_t s = (cudaStream_t)stream;
#define RFX_PREP(N, T)                                                                                              \
    RFX_LAUNCH((gated_delta_prep_kernel<N, T>), grid, PREP_THREADS, 0, s, proj, ld, b_off, a_off, filters, taps, state, \
               slot_stride, row_slot, dt_bias, A, unit_eps, q_scale, out, gates, H, G, d, dv, update, fast)
    if (!by4) RFX_PREP(0, 0);
    else if (d > 128 || dv > 128) RFX_PREP(4, 0);
    else if (taps == 2) RFX_PREP(1, 2);
    else if (taps == 3) RFX_PREP(1, 3);
    else if (taps == 4) RFX_PREP(1, 4);
    else RFX_PREP(1, 0);
#undef RFX_PREP
    return 0;
}

// `qkv` and `gates` as rfx_gated_delta_prep leaves them; the running state is
// state[slot * state_stride + state_off ..], [H][dv][d rounded up to 4] float32, 16-byte
// aligned.  Out: o float32 [R, H dv].  `max_rows`: the most rows any sequence brings.
extern "C" int rfx_gated_delta_scan(const float* qkv, const float* gates, float* state, long long state_stride,
                                    long long state_off, const int* seq_slot, const int* seq_row0, int n_seq,
                                    float* out, int H, int G, int d, int dv, int max_rows, void* stream) {
    if (n_seq <= 0 || max_rows <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || d <= 0 || dv <= 0) return RFX_ERR_BAD_ARG;
    if ((state_stride | state_off) & 3 || (reinterpret_cast<uintptr_t>(state) & 15)) return RFX_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
#define RFX_SCAN(N, K)                                                                                        \
    return launch_scan<N, K>(qkv, gates, state, state_stride, state_off, seq_slot, seq_row0, n_seq, out, H, G, d, \
                             dv, max_rows, s)
    if (d <= 32) RFX_SCAN(1, 8);
    if (d <= 64) RFX_SCAN(2, 8);
    if (d <= 128) RFX_SCAN(4, 8);
    if (d <= 256) RFX_SCAN(4, 16);
    if (d <= 512) RFX_SCAN(4, 32);
#undef RFX_SCAN
    return RFX_ERR_UNSUPPORTED;
}
