// The gated delta rule (gated_delta.cu) for steps that bring a sequence many rows: sixteen
// rows at a time, as products on the tensor cores.
//
// With S0 the memory before a chunk of rows, c_i the product of the chunk's decays up to
// row i, r_ij that of the rows after j up to i, and L_ij = r_ij (k_i.k_j) for j < i,
//     u = T (v - c * (K S0)),     T = (I + diag(beta) L)^-1 diag(beta)
//     o = c * (Q S0) + M u,       M_ij = r_ij (q_i.k_j) for j <= i
//     S0 <- c_last S0 + K^T (r_last * u)
// which is the row-by-row rule with the rows' dependence on one another solved once per
// chunk and head (T, by forward substitution), independently of the memory and of every other
// chunk: rfx_gated_delta_chunk_prep does that for all chunks side by side, and
// rfx_gated_delta_chunk walks the chunks with the products.
//
// The memory stays 32-bit (the products' accumulators are the memory itself).  Products run as
// three tensor-core products of operands split into a leading and a trailing part of 11 bits
// (x = hi + lo exactly up to 2^-22; hi hi + hi lo + lo hi, 32-bit sums): 32-bit products up
// to about 2^-21 of their size.  The true 32-bit path takes the row-by-row kernel instead.
//
// S^T [16 columns x channels] of a warp is an accumulator tile row of mma.sync m16n8k8, and,
// with the channels of every eight taken in the order (0, 2, 4, 6, 1, 3, 5, 7), the same
// registers are the left operand of the next chunk's products; likewise u^T.
#include "attn_mma.cuh"
#include "common.cuh"
#include "sm100.cuh"

namespace {

constexpr int CH = 16;            // rows of a chunk
constexpr int MAX_STAGES = 4;     // chunks in flight of a block
constexpr int TLD = 24;           // row stride of T and M: a fragment's 8-byte loads meet all banks
// per chunk and head: T [16][TLD], M [16][TLD], c [16], r_last [16], c_last and padding
constexpr int COEF = 2 * CH * TLD + 2 * CH + 4;

struct Split {
    uint32_t hi, lo;
};
__device__ __forceinline__ Split split(float x) {
    const uint32_t h = __float_as_uint(x) & 0xffffe000u;
    return {h, __float_as_uint(x - __uint_as_float(h))};
}
__device__ __forceinline__ void mma_tf32(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm(
        "mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
        "{%0, %1, %2, %3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// The left operand of a k-step from an accumulator tile (columns 2 j and 2 j + 1 are the k
// places j and j + 4), split.
struct Left {
    uint32_t hi[4], lo[4];
};
__device__ __forceinline__ Left left_of(const float (&t)[4]) {
    Left l;
    const int order[4] = {0, 2, 1, 3};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const Split s = split(t[order[i]]);
        l.hi[i] = s.hi;
        l.lo[i] = s.lo;
    }
    return l;
}
// d[n] += a b[n]^T for N right operands, pass by pass so that the products of different n
// follow one another, not those of one sum.
template <int N>
__device__ __forceinline__ void product3(float (&d)[N][4], const Left& a, const float2 (&b)[N]) {
    Split x[N], y[N];
#pragma unroll
    for (int n = 0; n < N; ++n) {
        x[n] = split(b[n].x);
        y[n] = split(b[n].y);
    }
#pragma unroll
    for (int n = 0; n < N; ++n) mma_tf32(d[n], a.lo, x[n].hi, y[n].hi);
#pragma unroll
    for (int n = 0; n < N; ++n) mma_tf32(d[n], a.hi, x[n].lo, y[n].lo);
#pragma unroll
    for (int n = 0; n < N; ++n) mma_tf32(d[n], a.hi, x[n].hi, y[n].hi);
}

// `bytes` (a multiple of 16, both addresses 16-byte aligned) into shared memory, counted on `bar`.
__device__ __forceinline__ void bulk_load(void* dst, const void* src, int bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                     sm100::smem_u32(dst)),
                 "l"(src), "r"(bytes), "r"(sm100::smem_u32(bar))
                 : "memory");
}

// Chunk c of sequence `seq`, whose first row of the step is row0: its place among all chunks
// (a sequence of n rows has ceil(n / 16), so no two places meet; at most R / 16 + sequences).
__device__ __forceinline__ size_t chunk_place(int row0, int seq, int c) { return (size_t)row0 / CH + seq + c; }

// A block a (chunk, query/key head): the products between the chunk's rows once, then per value
// head of the group T, M and the decays' products.
__global__ void __launch_bounds__(CH * CH)
gated_delta_chunk_prep_kernel(const float* __restrict__ qkv, const float* __restrict__ gates,
                              const int* __restrict__ seq_row0, float* __restrict__ coef, int H, int G, int d, int dv) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float L[CH][CH + 1], gs[CH], bs[CH];
    rfx::pdl_prologue();
    const int seq = blockIdx.y, kvh = blockIdx.z;
    const int row0 = seq_row0[seq], row1 = seq_row0[seq + 1];
    const int first = row0 + blockIdx.x * CH, n = min(CH, row1 - first);
    if (n <= 0) return;
    const int C = 2 * G * d + H * dv, LD = d + 4, d4 = d / 4;
    float *ks = sm, *qs = sm + CH * LD;
    const int tid = threadIdx.x, i = tid / CH, j = tid % CH;
    for (int e = tid; e < CH * d4; e += CH * CH) {
        const int r = e / d4, c = 4 * (e - r * d4);
        float4 k = make_float4(0.0f, 0.0f, 0.0f, 0.0f), q = k;
        if (r < n) {
            const float* src = qkv + (size_t)(first + r) * C + kvh * d + c;
            q = *reinterpret_cast<const float4*>(src);
            k = *reinterpret_cast<const float4*>(src + G * d);
        }
        *reinterpret_cast<float4*>(ks + r * LD + c) = k;
        *reinterpret_cast<float4*>(qs + r * LD + c) = q;
    }
    __syncthreads();
    float kk = 0.0f, qk = 0.0f;
    for (int c = 0; c < d; c += 4) {
        const float4 kj = *reinterpret_cast<const float4*>(ks + j * LD + c);
        const float4 ki = *reinterpret_cast<const float4*>(ks + i * LD + c);
        const float4 qi = *reinterpret_cast<const float4*>(qs + i * LD + c);
        kk = fmaf(ki.x, kj.x, fmaf(ki.y, kj.y, fmaf(ki.z, kj.z, fmaf(ki.w, kj.w, kk))));
        qk = fmaf(qi.x, kj.x, fmaf(qi.y, kj.y, fmaf(qi.z, kj.z, fmaf(qi.w, kj.w, qk))));
    }
    for (int h = kvh * (H / G); h < (kvh + 1) * (H / G); ++h) {
        __syncthreads();  // L, gs and bs of the head before have been read
        if (tid < CH) {
            gs[tid] = tid < n ? gates[(size_t)(first + tid) * 2 * H + h] : 1.0f;
            bs[tid] = tid < n ? gates[(size_t)(first + tid) * 2 * H + H + h] : 0.0f;
        }
        __syncthreads();
        float* out = coef + (chunk_place(row0, seq, blockIdx.x) * H + h) * COEF;
        float r = 1.0f;
        for (int l = j + 1; l <= i; ++l) r *= gs[l];
        L[i][j] = j < i ? bs[i] * (r * kk) : 0.0f;
        out[CH * TLD + i * TLD + j] = j <= i ? r * qk : 0.0f;
        if (i == 0) {
            float c = gs[0], last = 1.0f;
            for (int l = 1; l <= j; ++l) c *= gs[l];
            for (int l = j + 1; l < CH; ++l) last *= gs[l];
            out[2 * CH * TLD + j] = c;
            out[2 * CH * TLD + CH + j] = last;
            if (j == CH - 1) out[2 * CH * TLD + 2 * CH] = c;
        }
        __syncthreads();
        if (tid < CH) {  // column `tid` of T, row by row
            float t[CH];
#pragma unroll
            for (int a = 0; a < CH; ++a) {
                float s = a == tid ? bs[a] : 0.0f;
#pragma unroll
                for (int l = 0; l < a; ++l) s = fmaf(-L[a][l], t[l], s);
                t[a] = s;
                out[a * TLD + tid] = s;
            }
        }
    }
}

// Four warps own sixteen value columns, a quarter of the key channels each (NT eights; channels
// beyond d are zeros); a block has up to four such groups and one more warp that only brings the
// chunks: rows, values and coefficients by bulk copies, `stages` chunks in flight, a barrier per
// buffer for the bytes and one for the warps that are done with it.  The four quarters'
// partial sums of K S0 and Q S0 meet in shared memory in their order; u is solved by every
// warp of the group (each needs it for its channels), o by one of them in turn.
template <int NT>
__global__ void __launch_bounds__(544)
gated_delta_chunk_kernel(const float* __restrict__ qkv, const float* __restrict__ coef, float* __restrict__ state,
                         long long state_stride, long long state_off, const int* __restrict__ seq_slot,
                         const int* __restrict__ seq_row0, float* __restrict__ out, int H, int G, int d, int dv,
                         int cols, int stages, int* __restrict__ err) {
    constexpr int DP = 32 * NT, LDK = DP + 8;
    extern __shared__ __align__(16) float sm[];
    __shared__ __align__(8) uint64_t full[MAX_STAGES], empty[MAX_STAGES];
    __shared__ volatile int gave_up;
    const int seq = blockIdx.x, h = blockIdx.y, c_first = blockIdx.z * cols;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n_warps = cols / 16 * 4;  // the walking warps
    const int l4 = lane >> 2, j = lane & 3;
    const int VLD = cols + 4, buf_floats = 2 * CH * LDK + COEF + CH * VLD;
    const int C = 2 * G * d + H * dv, kvh = h / (H / G);
    const int grp = warp >> 2, quarter = warp & 3;
    // partial sums: [parity][group][tile of D][quarter][lane] four floats
    float4* red = reinterpret_cast<float4*>(sm + stages * buf_floats);
    // everything a copy does not reach stays zero: channels beyond d, rows beyond the first chunks'
    for (int e = threadIdx.x; e < stages * buf_floats; e += blockDim.x) sm[e] = 0.0f;
    if (threadIdx.x == 0) {
        for (int i = 0; i < stages; ++i) {
            sm100::mbar_init(&full[i], 1);
            sm100::mbar_init(&empty[i], n_warps);
        }
        sm100::fence_barrier_init();
        gave_up = 0;
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    __syncthreads();
    rfx::pdl_prologue();
    const int row0 = seq_row0[seq], row1 = seq_row0[seq + 1];
    const int n_chunks = (row1 - row0 + CH - 1) / CH;
    if (warp == n_warps) {
        const int v_bytes = min(cols, dv - c_first) * 4;
        int buf = 0, round = 0;  // chunk c is the round-th use of its buffer
        for (int c = 0; c < n_chunks; ++c) {
            const int first = row0 + c * CH, n = min(CH, row1 - first);
            if (round > 0 && !gave_up && !sm100::mbar_wait(&empty[buf], (round - 1) & 1)) {
                if (lane == 0) atomicExch(err, 41);
                gave_up = 1;
            }
            __syncwarp();
            if (gave_up) break;
            float* base = sm + (size_t)buf * buf_floats;
            if (lane == 0) sm100::mbar_expect_tx(&full[buf], n * (8 * d + v_bytes) + COEF * 4);
            __syncwarp();
            if (lane < n) {
                const float* src = qkv + (size_t)(first + lane) * C;
                bulk_load(base + lane * LDK, src + G * d + kvh * d, 4 * d, &full[buf]);
                bulk_load(base + (CH + lane) * LDK, src + kvh * d, 4 * d, &full[buf]);
                bulk_load(base + 2 * CH * LDK + COEF + lane * VLD, src + 2 * G * d + h * dv + c_first, v_bytes, &full[buf]);
            }
            if (lane == 31)
                bulk_load(base + 2 * CH * LDK, coef + (chunk_place(row0, seq, c) * H + h) * COEF, COEF * 4, &full[buf]);
            if (++buf == stages) {
                buf = 0;
                ++round;
            }
        }
        return;
    }
    const int cl = grp * 16, col = c_first + cl;
    const bool live = col < dv;  // dv is a multiple of sixteen: a group's columns all or none
    const int ch0 = quarter * 8 * NT;  // the warp's first channel
    float* Sg = state + (size_t)seq_slot[seq] * state_stride + state_off + ((size_t)h * dv + (live ? col : 0)) * d + ch0;
    float S[NT][4];
#pragma unroll
    for (int s = 0; s < NT; ++s) {
        float2 x = make_float2(0.0f, 0.0f), y = x;
        if (live && ch0 + 8 * s < d) {
            x = *reinterpret_cast<const float2*>(Sg + (size_t)l4 * d + 8 * s + 2 * j);
            y = *reinterpret_cast<const float2*>(Sg + (size_t)(l4 + 8) * d + 8 * s + 2 * j);
        }
        S[s][0] = x.x; S[s][1] = x.y; S[s][2] = y.x; S[s][3] = y.y;
    }
    int buf = 0, round = 0;
    for (int c = 0; c < n_chunks; ++c) {
        const int par = c & 1;  // of the partial sums' two places
        if (!gave_up && !sm100::mbar_wait(&full[buf], round & 1)) {  // reported; the walk ends without waiting on
            if (lane == 0) atomicExch(err, 42);
            gave_up = 1;
        }
        const float* base = sm + (size_t)buf * buf_floats;
        const float *ks = base + ch0, *cf = base + 2 * CH * LDK, *vs = cf + COEF;
        // this quarter's K S0 and Q S0, transposed: [0], [1] the k rows 0..7 and 8..15, [2], [3] the q rows
        float D[4][4] = {};
#pragma unroll
        for (int s = 0; s < NT; ++s) {
            const Left a = left_of(S[s]);
            float2 b[4];
#pragma unroll
            for (int n = 0; n < 4; ++n)
                b[n] = *reinterpret_cast<const float2*>(ks + (8 * n + l4) * LDK + 8 * s + 2 * j);
            product3<4>(D, a, b);
        }
        float4* mine = red + ((size_t)(par * (n_warps >> 2) + grp) * 4 * 4 + quarter) * 32 + lane;
#pragma unroll
        for (int n = 0; n < 4; ++n) mine[n * 4 * 32] = make_float4(D[n][0], D[n][1], D[n][2], D[n][3]);
        asm volatile("bar.sync %0, 128;" ::"r"(1 + grp) : "memory");  // the group's four warps
        const float4* all4 = red + (size_t)(par * (n_warps >> 2) + grp) * 4 * 4 * 32 + lane;
        auto total = [&](int n, float (&t)[4]) {
            const float4 p0 = all4[n * 128], p1 = all4[n * 128 + 32], p2 = all4[n * 128 + 64], p3 = all4[n * 128 + 96];
            t[0] = (p0.x + p1.x) + (p2.x + p3.x);
            t[1] = (p0.y + p1.y) + (p2.y + p3.y);
            t[2] = (p0.z + p1.z) + (p2.z + p3.z);
            t[3] = (p0.w + p1.w) + (p2.w + p3.w);
        };
        // v - c * (K S0), then u = T of it; a tile holds rows 8 t + 2 j and + 1 of columns l4 and l4 + 8
        float U[2][4] = {};
        float2 ci[2];
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            ci[t] = *reinterpret_cast<const float2*>(cf + 2 * CH * TLD + 8 * t + 2 * j);
            const float* v = vs + (8 * t + 2 * j) * VLD + cl + l4;
            float x[4];
            total(t, x);
            x[0] = fmaf(-ci[t].x, x[0], v[0]);
            x[1] = fmaf(-ci[t].y, x[1], v[VLD]);
            x[2] = fmaf(-ci[t].x, x[2], v[8]);
            x[3] = fmaf(-ci[t].y, x[3], v[VLD + 8]);
            const Left a = left_of(x);
            float2 b[2];
#pragma unroll
            for (int n = 0; n < 2; ++n)
                b[n] = *reinterpret_cast<const float2*>(cf + (8 * n + l4) * TLD + 8 * t + 2 * j);
            // T is lower triangular: rows 8..15 of its right side meet rows 8..15 alone
            if (t == 0) product3<2>(U, a, b);
            else product3<1>(*reinterpret_cast<float(*)[1][4]>(&U[1]), a, *reinterpret_cast<const float2(*)[1]>(&b[1]));
        }
        // the memory's step: K^T (r_last * u)
        const float all = cf[2 * CH * TLD + 2 * CH];
#pragma unroll
        for (int s = 0; s < NT; ++s)
#pragma unroll
            for (int i = 0; i < 4; ++i) S[s][i] *= all;
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            const float2 rl = *reinterpret_cast<const float2*>(cf + 2 * CH * TLD + CH + 8 * t + 2 * j);
            const float w[4] = {U[t][0] * rl.x, U[t][1] * rl.y, U[t][2] * rl.x, U[t][3] * rl.y};
            const Left a = left_of(w);
            const float* k = ks + (8 * t + 2 * j) * LDK + l4;
            float2 b[NT];
#pragma unroll
            for (int s = 0; s < NT; ++s) b[s] = make_float2(k[8 * s], k[LDK + 8 * s]);
            product3<NT>(S, a, b);
        }
        if (quarter == (c & 3)) {
            float O[2][4];
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                total(2 + t, O[t]);
                O[t][0] *= ci[t].x;
                O[t][1] *= ci[t].y;
                O[t][2] *= ci[t].x;
                O[t][3] *= ci[t].y;
            }
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                const Left a = left_of(U[t]);
                float2 b[2];
#pragma unroll
                for (int n = 0; n < 2; ++n)
                    b[n] = *reinterpret_cast<const float2*>(cf + CH * TLD + (8 * n + l4) * TLD + 8 * t + 2 * j);
                if (t == 0) product3<2>(O, a, b);
                else product3<1>(*reinterpret_cast<float(*)[1][4]>(&O[1]), a, *reinterpret_cast<const float2(*)[1]>(&b[1]));
            }
            if (live) {
                const int left = row1 - row0 - c * CH;
                const size_t ld = (size_t)H * dv;
                float* o = out + (size_t)(row0 + c * CH) * ld + (size_t)h * dv + col + l4;
#pragma unroll
                for (int t = 0; t < 2; ++t) {
                    const int r = 8 * t + 2 * j;
                    if (r < left) {
                        o[r * ld] = O[t][0];
                        o[r * ld + 8] = O[t][2];
                    }
                    if (r + 1 < left) {
                        o[(r + 1) * ld] = O[t][1];
                        o[(r + 1) * ld + 8] = O[t][3];
                    }
                }
            }
        }
        __syncwarp();
        if (lane == 0) sm100::mbar_arrive(&empty[buf]);  // this warp is done with the chunk
        if (++buf == stages) {
            buf = 0;
            ++round;
        }
    }
    if (!live) return;
#pragma unroll
    for (int s = 0; s < NT; ++s)
        if (ch0 + 8 * s < d) {
            *reinterpret_cast<float2*>(Sg + (size_t)l4 * d + 8 * s + 2 * j) = make_float2(S[s][0], S[s][1]);
            *reinterpret_cast<float2*>(Sg + (size_t)(l4 + 8) * d + 8 * s + 2 * j) = make_float2(S[s][2], S[s][3]);
        }
}

template <int NT>
int launch_chunk(const float* qkv, const float* coef, float* state, long long state_stride, long long state_off,
                 const int* seq_slot, const int* seq_row0, int n_seq, float* out, int H, int G, int d, int dv,
                 int* err, cudaStream_t s) {
    // value columns a block owns, sixteen a group of four warps; fewer while the blocks do not fill the SMs
    int cols = 64;
    while (cols > 16 && (cols / 2 >= dv ||
                         (long long)n_seq * H * ((dv + cols - 1) / cols) < rfx::sm_count() * 3LL / 4))
        cols /= 2;
    const size_t stage = (size_t)(2 * CH * (32 * NT + 8) + COEF + CH * (cols + 4)) * sizeof(float);
    const size_t red = (size_t)2 * (cols / 16) * 4 * 4 * 32 * sizeof(float4);
    // one block an SM: as many chunks in flight as fit, up to four; more blocks: two chunks each
    int stages = (long long)n_seq * H * ((dv + cols - 1) / cols) <= rfx::sm_count() ? MAX_STAGES : 2;
    while (stages > 2 && stages * stage + red > 220 * 1024) --stages;
    const size_t smem = stages * stage + red;
    if (smem > 220 * 1024) return RFX_ERR_UNSUPPORTED;
    auto kernel = gated_delta_chunk_kernel<NT>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    dim3 grid(n_seq, H, (dv + cols - 1) / cols);
    RFX_LAUNCH(kernel, grid, cols / 16 * 128 + 32, smem, s, qkv, coef, state, state_stride, state_off, seq_slot,
               seq_row0, out, H, G, d, dv, cols, stages, err);
    return 0;
}

}  // namespace

// Floats of `coef` that steps of R rows in n_seq sequences need.
extern "C" long long rfx_gated_delta_chunk_floats(int R, int n_seq, int H) {
    return (long long)(R / CH + n_seq) * H * COEF;
}

// T, M and the decays' products of every chunk (chunks counted from each sequence's first row of the
// step).  `max_rows`: the most rows any sequence brings.  d a multiple of 4, `qkv` 16-byte aligned.
extern "C" int rfx_gated_delta_chunk_prep(const float* qkv, const float* gates, const int* seq_row0, int n_seq,
                                          float* coef, int H, int G, int d, int dv, int max_rows, void* stream) {
    if (n_seq <= 0 || max_rows <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || d <= 0 || dv <= 0) return RFX_ERR_BAD_ARG;
    const size_t smem = (size_t)2 * CH * (d + 4) * sizeof(float);
    if (d % 4 || dv % 4 || smem > 48 * 1024 || n_seq > 65535 || G > 65535) return RFX_ERR_UNSUPPORTED;
    dim3 grid((max_rows + CH - 1) / CH, n_seq, G);
    RFX_LAUNCH(gated_delta_chunk_prep_kernel, grid, CH * CH, smem, (cudaStream_t)stream, qkv, gates, seq_row0, coef, H,
               G, d, dv);
    return 0;
}

// The recurrence over the step's rows, chunk by chunk.  d a multiple of 8 up to 256, dv of 16;
// the running state as rfx_gated_delta_scan keeps it.  `err`: a device word that receives a
// non-zero code if a bounded wait ran out.
extern "C" int rfx_gated_delta_chunk(const float* qkv, const float* coef, float* state, long long state_stride,
                                     long long state_off, const int* seq_slot, const int* seq_row0, int n_seq,
                                     float* out, int H, int G, int d, int dv, int* err, void* stream) {
    if (n_seq <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || d <= 0 || dv <= 0) return RFX_ERR_BAD_ARG;
    if ((state_stride | state_off) & 3 || (reinterpret_cast<uintptr_t>(state) & 15)) return RFX_ERR_BAD_ARG;
    if (d % 8 || dv % 16 || d > 256 || H > 65535 ||
        ((reinterpret_cast<uintptr_t>(qkv) | reinterpret_cast<uintptr_t>(coef)) & 15))
        return RFX_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
#define RFX_CHUNK(N)                                                                                              \
    return launch_chunk<N>(qkv, coef, state, state_stride, state_off, seq_slot, seq_row0, n_seq, out, H, G, d, dv, \
                           err, s)
    if (d <= 32) RFX_CHUNK(1);
    if (d <= 64) RFX_CHUNK(2);
    if (d <= 96) RFX_CHUNK(3);
    if (d <= 128) RFX_CHUNK(4);
    if (d <= 192) RFX_CHUNK(6);
    RFX_CHUNK(8);
#undef RFX_CHUNK
}
