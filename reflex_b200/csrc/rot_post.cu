// What lies between a stacked first product and the attention kernel, for mixers that
// rotate before they norm and for latents with a rotated key part.
//
//  * rfx_rot_qkv_post: rows [q | k | v] (+ a bias a column): the first `rot_dims`
//    dimensions of every q and k head turn in half-split pairs (i with i + rot_dims / 2) by
//    the angle position / denom[i]; then, with `unit`, q and k are divided by their
//    root mean square over the head, x / sqrt(mean(x^2) + eps); or (`unit` 2) they are normed
//    first, with a weight per dimension, and turned after it; cosine and sine may have a
//    magnitude; q goes out, k and v go
//    into their pages at the row's position, heads `pad` wide (zeros beyond the key and
//    the value size).  Value mixing: with `v_out` the row's values are also kept
//    (32-bit); with `v_first` and `lambda` they become (1 - lambda) v + lambda v_first
//    before they are cached.
//  * rfx_latent_low_post: rows [query latent | latent | shared key part | ...]: the query
//    latent over its root mean square and times a weight goes out (for the query
//    up-projection); the latent, likewise, and the turned key part go into the page of the
//    row's position as one row [latent | key part | zeros].
//  * rfx_rotate_tails: the last `rot` elements of every head turn where they stand.
//  * rfx_latent_rot_post: rows [q | latent | shared key part]: per head the unrotated
//    part of q and the turned rotated part with zeros behind it go to places of the caller's
//    (apart, where the product with W_uk follows; side by side as one query); the latent, over its root
//    mean square and times a weight, and the turned key part go into the page of the
//    row's position as one row [latent | key part | zeros].
//
// A warp a head of a row; everything is 32-bit; sine and cosine are taken once a row and
// block into shared memory, by `exact_sincosf` (whose range reduction runs in double precision,
// at a small fraction of this GPU's 32-bit rate) for 32-bit results, by sincosf for rounded ones.
#include "common.cuh"
#include "exact_math.cuh"
#include "paged.cuh"

namespace {

using namespace rfx;

constexpr int RP_THREADS = 256;
constexpr int RP_WARPS = RP_THREADS / 32;

// cos and sin of a row's angles into cs[0 .. half) and cs[half .. 2 half)
template <typename TO>
__device__ __forceinline__ void angles(float* cs, const float* denom, int half, int pos, float magnitude = 1.0f) {
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float s, c;
        if constexpr (sizeof(TO) == 2) sincosf((float)pos / denom[i], &s, &c);
        else exact_sincosf((float)pos / denom[i], &s, &c);
        cs[i] = c * magnitude;
        cs[half + i] = s * magnitude;
    }
    __syncthreads();
}

// (u, v) -> (u cos - v sin, v cos + u sin): element `x` at i of the rotated part, its partner
// at the other half
__device__ __forceinline__ float turned(float x, float partner, int i, const float* cs, int half) {
    const int f = i < half ? i : i - half;
    return fmaf(partner, i < half ? -cs[half + f] : cs[half + f], __fmul_rn(x, cs[f]));
}

struct QkvPost {
    const float* bias;   // [nq d + nkv d + nkv dv] or null
    const float* denom;  // [rot_dims / 2]
    int rot_dims;
    float magnitude;
    int unit;            // 0 no norm, 1 unit root mean square after the rotation, 2 norm with a weight before it
    float eps;
    const float *q_w, *k_w;  // unit 2: norm weights [d], applied as w_offset + w
    float w_offset;
    const float* lambda;   // one number, or null
    const float* v_first;  // [R, nkv dv] float32, or null
    float* v_out;          // [R, nkv dv] float32, or null
    int nq, nkv, d, dv, pad, writes_cache;
};

// NV: a head's elements in 128s, four a lane (up to 512), 0: sizes that are no multiples of four
template <typename TI, typename TO, int NV>
__global__ void __launch_bounds__(RP_THREADS)
rot_qkv_post_kernel(const TI* __restrict__ proj, int ldp, QkvPost a, const int* __restrict__ row_pos,
                    const int* __restrict__ row_slot, TO* __restrict__ q_out, TO* __restrict__ k_pages,
                    TO* __restrict__ v_pages, PagedKV cache) {
    extern __shared__ float cs[];
    pdl_prologue();
    const int r = blockIdx.x;
    const int pos = row_pos[r], slot = row_slot[r];
    const int half = a.rot_dims / 2;
    angles<TO>(cs, a.denom, half, pos, a.magnitude);
    const int lane = threadIdx.x & 31;
    const int units = a.nq + (a.writes_cache ? 2 * a.nkv : 0);
    for (int u = blockIdx.y * RP_WARPS + (threadIdx.x >> 5); u < units; u += gridDim.y * RP_WARPS) {
        const bool is_v = u >= a.nq + a.nkv;
        const int vh = u - a.nq - a.nkv;
        const int col = is_v ? (a.nq + a.nkv) * a.d + vh * a.dv : u * a.d;
        const int width = is_v ? a.dv : a.d;
        const TI* x = proj + (size_t)r * ldp + col;
        const float* b = a.bias ? a.bias + col : nullptr;
        TO* dst;
        if (u < a.nq) dst = q_out + ((size_t)r * a.nq + u) * a.pad;
        else if (!is_v) dst = k_pages + kv_offset(cache, slot, pos, u - a.nq);
        else dst = v_pages + kv_offset(cache, slot, pos, vh);
        const float lam = a.lambda ? *a.lambda : 0.0f;
        const size_t vrow = ((size_t)r * a.nkv + vh) * a.dv;
        const float* nw = a.unit == 2 && !is_v ? (u < a.nq ? a.q_w : a.k_w) : nullptr;
        if (nw) {
            // norm, weight, rotation; a head's elements and their partners' are read once more than
            // they are summed (the row's products are in the cache)
            if constexpr (NV > 0) {
                float4 y[NV];
                float ss = 0.0f;
#pragma unroll
                for (int i = 0; i < NV; ++i) {
                    const int e = 4 * (lane + 32 * i);
                    if (e >= width) continue;
                    float4 t = load4(x + e);
                    if (b) {
                        const float4 bb = load4(b + e);
                        t.x += bb.x; t.y += bb.y; t.z += bb.z; t.w += bb.w;
                    }
                    ss = fmaf(t.x, t.x, fmaf(t.y, t.y, fmaf(t.z, t.z, fmaf(t.w, t.w, ss))));
                    y[i] = t;
                }
                const float f = 1.0f / sqrtf(warp_sum(ss) / (float)a.d + a.eps);
                auto weighted = [&](float4 t, int e) {
                    const float4 w = load4(nw + e);
                    return make_float4((t.x * f) * (a.w_offset + w.x), (t.y * f) * (a.w_offset + w.y),
                                       (t.z * f) * (a.w_offset + w.z), (t.w * f) * (a.w_offset + w.w));
                };
#pragma unroll
                for (int i = 0; i < NV; ++i) {
                    const int e = 4 * (lane + 32 * i);
                    if (e < width) {
                        float4 t = weighted(y[i], e);
                        if (e < a.rot_dims) {
                            const int pe = e < half ? e + half : e - half;
                            float4 p = load4(x + pe);
                            if (b) {
                                const float4 bb = load4(b + pe);
                                p.x += bb.x; p.y += bb.y; p.z += bb.z; p.w += bb.w;
                            }
                            p = weighted(p, pe);
                            t.x = turned(t.x, p.x, e, cs, half);
                            t.y = turned(t.y, p.y, e + 1, cs, half);
                            t.z = turned(t.z, p.z, e + 2, cs, half);
                            t.w = turned(t.w, p.w, e + 3, cs, half);
                        }
                        store4(dst + e, t);
                    } else if (e < a.pad) {
                        store4(dst + e, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
                    }
                }
            } else {
                auto raw = [&](int e) { return ld<TI>(x, e) + (b ? b[e] : 0.0f); };
                float ss = 0.0f;
                for (int e = lane; e < width; e += 32) ss = fmaf(raw(e), raw(e), ss);
                const float f = 1.0f / sqrtf(warp_sum(ss) / (float)a.d + a.eps);
                auto normed = [&](int e) { return (raw(e) * f) * (a.w_offset + nw[e]); };
                for (int e = lane; e < a.pad; e += 32) {
                    float t = 0.0f;
                    if (e < width) {
                        t = normed(e);
                        if (e < a.rot_dims) t = turned(t, normed(e < half ? e + half : e - half), e, cs, half);
                    }
                    st<TO>(dst, e, t);
                }
            }
            continue;
        }
        if constexpr (NV > 0) {
            float4 y[NV];
            float ss = 0.0f;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int e = 4 * (lane + 32 * i);
                if (e >= width) continue;
                float4 t = load4(x + e);
                if (b) {
                    const float4 bb = load4(b + e);
                    t.x += bb.x; t.y += bb.y; t.z += bb.z; t.w += bb.w;
                }
                if (is_v) {
                    if (a.v_out) store4(a.v_out + vrow + e, t);
                    if (a.v_first) {
                        const float4 f = load4(a.v_first + vrow + e);
                        t.x = fmaf(1.0f - lam, t.x, lam * f.x);
                        t.y = fmaf(1.0f - lam, t.y, lam * f.y);
                        t.z = fmaf(1.0f - lam, t.z, lam * f.z);
                        t.w = fmaf(1.0f - lam, t.w, lam * f.w);
                    }
                } else if (e < a.rot_dims) {
                    const int pe = e < half ? e + half : e - half;
                    float4 p = load4(x + pe);
                    if (b) {
                        const float4 bb = load4(b + pe);
                        p.x += bb.x; p.y += bb.y; p.z += bb.z; p.w += bb.w;
                    }
                    t.x = turned(t.x, p.x, e, cs, half);
                    t.y = turned(t.y, p.y, e + 1, cs, half);
                    t.z = turned(t.z, p.z, e + 2, cs, half);
                    t.w = turned(t.w, p.w, e + 3, cs, half);
                }
                ss = fmaf(t.x, t.x, fmaf(t.y, t.y, fmaf(t.z, t.z, fmaf(t.w, t.w, ss))));
                y[i] = t;
            }
            float f = 1.0f;
            if (!is_v && a.unit == 1) f = 1.0f / sqrtf(warp_sum(ss) / (float)a.d + a.eps);
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int e = 4 * (lane + 32 * i);
                if (e < width) store4(dst + e, make_float4(y[i].x * f, y[i].y * f, y[i].z * f, y[i].w * f));
                else if (e < a.pad) store4(dst + e, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
            }
        } else {
            auto value = [&](int e) -> float {
                float t = ld<TI>(x, e) + (b ? b[e] : 0.0f);
                if (is_v) {
                    if (a.v_out) a.v_out[vrow + e] = t;
                    if (a.v_first) t = fmaf(1.0f - lam, t, lam * a.v_first[vrow + e]);
                } else if (e < a.rot_dims) {
                    const int pe = e < half ? e + half : e - half;
                    t = turned(t, ld<TI>(x, pe) + (b ? b[pe] : 0.0f), e, cs, half);
                }
                return t;
            };
            float f = 1.0f;
            if (!is_v && a.unit == 1) {
                float ss = 0.0f;
                for (int e = lane; e < width; e += 32) {
                    const float t = value(e);
                    ss = fmaf(t, t, ss);
                }
                f = 1.0f / sqrtf(warp_sum(ss) / (float)a.d + a.eps);
            }
            for (int e = lane; e < a.pad; e += 32) st<TO>(dst, e, e < width ? value(e) * f : 0.0f);
        }
    }
}

template <typename TI, typename TO, bool BY4>
__global__ void __launch_bounds__(RP_THREADS)
latent_rot_post_kernel(const TI* __restrict__ proj, int ldp, const float* __restrict__ kv_w, float eps,
                       const float* __restrict__ denom, const int* __restrict__ row_pos,
                       const int* __restrict__ row_slot, TO* __restrict__ q_flat, int flat_h,
                       TO* __restrict__ q_rot, int rot_h, int rot_w, TO* __restrict__ pages, PagedKV cache, int H,
                       int d, int rot, int rank, int width, int writes_cache) {
    extern __shared__ float cs[];
    pdl_prologue();
    const int r = blockIdx.x;
    const int pos = row_pos[r], slot = row_slot[r];
    const int half = rot / 2;
    angles<TO>(cs, denom, half, pos);
    const int lane = threadIdx.x & 31;
    const TI* row = proj + (size_t)r * ldp;
    auto turn_into = [&](TO* dst, const TI* x, int n) {  // the rotated part and the zeros behind it
        for (int e = lane; e < n; e += 32)
            st<TO>(dst, e, e < rot ? turned(ld<TI>(x, e), ld<TI>(x, e < half ? e + half : e - half), e, cs, half) : 0.0f);
    };
    const int units = H + (writes_cache ? 1 : 0);
    for (int u = blockIdx.y * RP_WARPS + (threadIdx.x >> 5); u < units; u += gridDim.y * RP_WARPS) {
        if (u < H) {
            const TI* x = row + (size_t)u * (d + rot);
            TO* flat = q_flat + ((size_t)r * H + u) * flat_h;
            if constexpr (BY4)
                for (int e = 4 * lane; e < d; e += 128) store4(flat + e, load4(x + e));
            else
                for (int e = lane; e < d; e += 32) st<TO>(flat, e, ld<TI>(x, e));
            turn_into(q_rot + ((size_t)r * H + u) * rot_h, x + d, rot_w);
        } else {
            const TI* x = row + (size_t)H * (d + rot);
            TO* dst = pages + kv_offset(cache, slot, pos, 0);
            float ss = 0.0f;
            if constexpr (BY4) {
                for (int e = 4 * lane; e < rank; e += 128) {
                    const float4 t = load4(x + e);
                    ss = fmaf(t.x, t.x, fmaf(t.y, t.y, fmaf(t.z, t.z, fmaf(t.w, t.w, ss))));
                }
            } else {
                for (int e = lane; e < rank; e += 32) {
                    const float t = ld<TI>(x, e);
                    ss = fmaf(t, t, ss);
                }
            }
            const float f = 1.0f / sqrtf(warp_sum(ss) / (float)rank + eps);
            if constexpr (BY4) {
                for (int e = 4 * lane; e < rank; e += 128) {
                    const float4 t = load4(x + e), w = load4(kv_w + e);
                    store4(dst + e, make_float4((t.x * f) * w.x, (t.y * f) * w.y, (t.z * f) * w.z, (t.w * f) * w.w));
                }
            } else {
                for (int e = lane; e < rank; e += 32) st<TO>(dst, e, (ld<TI>(x, e) * f) * kv_w[e]);
            }
            turn_into(dst + rank, x + rank, width - rank);
        }
    }
}

// One block a (row, latent): block 0 of a row the query latent, block 1 the cached latent and
// the shared key part.
template <typename TI, typename TO, bool BY4>
__global__ void __launch_bounds__(128)
latent_low_post_kernel(const TI* __restrict__ proj, int ldp, const float* __restrict__ q_w,
                       const float* __restrict__ kv_w, float eps, const float* __restrict__ denom,
                       const int* __restrict__ row_pos, const int* __restrict__ row_slot, TO* __restrict__ q_out,
                       TO* __restrict__ pages, PagedKV cache, int q_rank, int rank, int rot, int width) {
    extern __shared__ float cs[];
    __shared__ float scratch[32];
    const bool cached = blockIdx.y == 1;
    const int r = blockIdx.x, half = rot / 2, n = cached ? rank : q_rank;
    const float* w = cached ? kv_w : q_w;
    TO* dst = q_out + (size_t)r * q_rank;
    pdl_launch_dependents();
    if (cached) {  // positions are the step's inputs: none of this waits for the kernel before
        const int pos = row_pos[r];
        angles<TO>(cs, denom, half, pos);
        dst = pages + kv_offset(cache, row_slot[r], pos, 0);
    }
    pdl_wait();
    const TI* x = proj + (size_t)r * ldp + (cached ? q_rank : 0);
    float ss = 0.0f;
    if constexpr (BY4) {
        for (int e = 4 * threadIdx.x; e < n; e += 4 * blockDim.x) {
            const float4 t = load4(x + e);
            ss = fmaf(t.x, t.x, fmaf(t.y, t.y, fmaf(t.z, t.z, fmaf(t.w, t.w, ss))));
        }
    } else {
        for (int e = threadIdx.x; e < n; e += blockDim.x) {
            const float t = ld<TI>(x, e);
            ss = fmaf(t, t, ss);
        }
    }
    const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
    if constexpr (BY4) {
        for (int e = 4 * threadIdx.x; e < n; e += 4 * blockDim.x) {
            const float4 t = load4(x + e), g = load4(w + e);
            store4(dst + e, make_float4((t.x * f) * g.x, (t.y * f) * g.y, (t.z * f) * g.z, (t.w * f) * g.w));
        }
    } else {
        for (int e = threadIdx.x; e < n; e += blockDim.x) st<TO>(dst, e, (ld<TI>(x, e) * f) * w[e]);
    }
    if (!cached) return;
    x += rank;
    for (int e = threadIdx.x; e < width - rank; e += blockDim.x)
        st<TO>(dst + rank, e,
               e < rot ? turned(ld<TI>(x, e), ld<TI>(x, e < half ? e + half : e - half), e, cs, half) : 0.0f);
}

// x [R, H, n]: of every head the last `rot` elements, half-split pairs, in place; a thread two
// neighbouring pairs (rot a multiple of 4)
template <typename T>
__global__ void __launch_bounds__(RP_THREADS)
rotate_tails_kernel(T* __restrict__ x, const float* __restrict__ denom, const int* __restrict__ row_pos, int H, int n,
                    int rot) {
    extern __shared__ float cs[];
    pdl_launch_dependents();
    const int r = blockIdx.x, half = rot / 2, quads = half / 2;
    angles<T>(cs, denom, half, row_pos[r]);  // positions are the step's inputs
    pdl_wait();
    T* row = x + (size_t)r * H * n + (n - rot);
    for (int u = threadIdx.x; u < H * quads; u += blockDim.x) {
        const int i = 2 * (u % quads);
        T* p = row + (size_t)(u / quads) * n + i;
        const float a0 = ld<T>(p, 0), a1 = ld<T>(p, 1), b0 = ld<T>(p, half), b1 = ld<T>(p, half + 1);
        store2(p, fmaf(b0, -cs[half + i], __fmul_rn(a0, cs[i])), fmaf(b1, -cs[half + i + 1], __fmul_rn(a1, cs[i + 1])));
        store2(p + half, fmaf(a0, cs[half + i], __fmul_rn(b0, cs[i])), fmaf(a1, cs[half + i + 1], __fmul_rn(b1, cs[i + 1])));
    }
}

// blocks of a row: few rows spread their heads over blocks, many rows keep a row's angles in one
int rows_blocks(int R, int units) {
    int y = (units + RP_WARPS - 1) / RP_WARPS;
    const int want = (4 * sm_count() + R - 1) / R;
    return y < want ? y : (want < 1 ? 1 : want);
}

bool aligned(const void* p, uintptr_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

}  // namespace

extern "C" int rfx_rot_qkv_post(const void* proj, int in_dt, int ld, const float* bias, const float* denom,
                                int rot_dims, float magnitude, int unit, float eps, const float* q_w, const float* k_w,
                                float w_offset, const float* lambda, const float* v_first,
                                float* v_out, const int* row_pos, const int* row_slot, void* q_out, void* k_pages,
                                void* v_pages, int out_dt, const int* page_table, int max_pages, int page_size,
                                int R, int nq, int nkv, int d, int dv, int pad, int writes_cache, void* stream) {
    if (R <= 0) return 0;
    if (nkv <= 0 || nq <= 0 || d <= 0 || dv <= 0 || pad < d || pad < dv || rot_dims < 0 || rot_dims % 2 ||
        rot_dims > d || (v_first && !lambda) || unit < 0 || unit > 2 ||
        (unit == 2 && (!q_w || (writes_cache && !k_w))))
        return RFX_ERR_BAD_ARG;
    QkvPost a{bias, denom, rot_dims, magnitude, unit, eps, q_w, k_w, w_offset, lambda, v_first, v_out, nq, nkv, d, dv, pad, writes_cache};
    PagedKV cache{page_table, max_pages, page_size, nkv, pad};
    cudaStream_t s = (cudaStream_t)stream;
    const uintptr_t in_al = in_dt == RFX_DT_F32 ? 16 : 8, out_al = out_dt == RFX_DT_F32 ? 16 : 8;
    const bool by4 = d % 4 == 0 && dv % 4 == 0 && pad % 4 == 0 && ld % 4 == 0 && (rot_dims / 2) % 4 == 0 &&
                     pad <= 512 && aligned(proj, in_al) && aligned(bias, 16) && aligned(q_w, 16) && aligned(k_w, 16) && aligned(v_first, 16) &&
                     aligned(v_out, 16) && aligned(q_out, out_al) && aligned(k_pages, out_al) &&
                     aligned(v_pages, out_al);
    dim3 grid(R, rows_blocks(R, nq + 2 * nkv));
    const size_t smem = (size_t)(rot_dims > 0 ? rot_dims : 1) * sizeof(float);
#define RFX_N(TI, TO, N)                                                                                          \
    RFX_LAUNCH((rot_qkv_post_kernel<TI, TO, N>), grid, RP_THREADS, smem, s, (const TI*)proj, ld, a, row_pos,      \
               row_slot, (TO*)q_out, (TO*)k_pages, (TO*)v_pages, cache)
#define RFX_GO(TI, TO)                   \
    do {                                 \
        if (!by4) RFX_N(TI, TO, 0);      \
        else if (pad <= 128) RFX_N(TI, TO, 1); \
        else RFX_N(TI, TO, 4);           \
    } while (0)
    if (in_dt == RFX_DT_F32 && out_dt == RFX_DT_F32) RFX_GO(float, float);
    else if (in_dt == RFX_DT_F32 && out_dt == RFX_DT_BF16) RFX_GO(float, __nv_bfloat16);
    else if (in_dt == RFX_DT_BF16 && out_dt == RFX_DT_BF16) RFX_GO(__nv_bfloat16, __nv_bfloat16);
    else return RFX_ERR_BAD_ARG;
#undef RFX_GO
#undef RFX_N
    return 0;
}

// `width`: elements of a cached row (at least rank + rot; zeros behind them).  Of head h of row r
// the unrotated d elements go to q_flat + (r H + h) flat_h, the turned ones and zeros, rot_w in all,
// to q_rot + (r H + h) rot_h.
extern "C" int rfx_latent_rot_post(const void* proj, int in_dt, int ld, const float* kv_w, float eps,
                                   const float* denom, const int* row_pos, const int* row_slot, void* q_flat,
                                   int flat_h, void* q_rot, int rot_h, int rot_w, void* pages, int out_dt, const int* page_table, int max_pages,
                                   int page_size, int R, int H, int d, int rot, int rank, int width,
                                   int writes_cache, void* stream) {
    if (R <= 0) return 0;
    if (H <= 0 || d <= 0 || rank <= 0 || rot < 0 || rot % 2 || width < rank + rot || flat_h < d || rot_h < rot_w ||
        rot_w < rot ||
        ld < H * (d + rot) + (writes_cache ? rank + rot : 0))
        return RFX_ERR_BAD_ARG;
    PagedKV cache{page_table, max_pages, page_size, 1, width};
    cudaStream_t s = (cudaStream_t)stream;
    const uintptr_t in_al = in_dt == RFX_DT_F32 ? 16 : 8, out_al = out_dt == RFX_DT_F32 ? 16 : 8;
    const bool by4 = d % 4 == 0 && rot % 4 == 0 && rank % 4 == 0 && width % 4 == 0 && ld % 4 == 0 && flat_h % 4 == 0 &&
                     aligned(proj, in_al) && aligned(kv_w, 16) && aligned(q_flat, out_al) && aligned(pages, out_al);
    dim3 grid(R, rows_blocks(R, H + 1));
    const size_t smem = (size_t)(rot > 0 ? rot : 1) * sizeof(float);
#define RFX_GO(TI, TO)                                                                                              \
    do {                                                                                                            \
        if (by4)                                                                                                    \
            RFX_LAUNCH((latent_rot_post_kernel<TI, TO, true>), grid, RP_THREADS, smem, s, (const TI*)proj, ld,      \
                       kv_w, eps, denom, row_pos, row_slot, (TO*)q_flat, flat_h, (TO*)q_rot, rot_h, rot_w, (TO*)pages, cache, H, d, rot,  \
                       rank, width, writes_cache);                                                                  \
        else                                                                                                        \
            RFX_LAUNCH((latent_rot_post_kernel<TI, TO, false>), grid, RP_THREADS, smem, s, (const TI*)proj, ld,     \
                       kv_w, eps, denom, row_pos, row_slot, (TO*)q_flat, flat_h, (TO*)q_rot, rot_h, rot_w, (TO*)pages, cache, H, d, rot,  \
                       rank, width, writes_cache);                                                                  \
    } while (0)
    if (in_dt == RFX_DT_F32 && out_dt == RFX_DT_F32) RFX_GO(float, float);
    else if (in_dt == RFX_DT_F32 && out_dt == RFX_DT_BF16) RFX_GO(float, __nv_bfloat16);
    else if (in_dt == RFX_DT_BF16 && out_dt == RFX_DT_BF16) RFX_GO(__nv_bfloat16, __nv_bfloat16);
    else return RFX_ERR_BAD_ARG;
#undef RFX_GO
    return 0;
}

// proj rows [q_rank | rank | rot | ...]; `width`: elements of a cached row (at least rank + rot)
extern "C" int rfx_latent_low_post(const void* proj, int in_dt, int ld, const float* q_w, const float* kv_w, float eps,
                                   const float* denom, const int* row_pos, const int* row_slot, void* q_out, void* pages,
                                   int out_dt, const int* page_table, int max_pages, int page_size, int R, int q_rank,
                                   int rank, int rot, int width, int writes_cache, void* stream) {
    if (R <= 0) return 0;
    if (q_rank <= 0 || rank <= 0 || rot < 0 || rot % 2 || width < rank + rot || ld < q_rank + rank + rot)
        return RFX_ERR_BAD_ARG;
    PagedKV cache{page_table, max_pages, page_size, 1, width};
    cudaStream_t s = (cudaStream_t)stream;
    const uintptr_t in_al = in_dt == RFX_DT_F32 ? 16 : 8, out_al = out_dt == RFX_DT_F32 ? 16 : 8;
    const bool by4 = q_rank % 4 == 0 && rank % 4 == 0 && width % 4 == 0 && ld % 4 == 0 && aligned(proj, in_al) &&
                     aligned(q_w, 16) && aligned(kv_w, 16) && aligned(q_out, out_al) && aligned(pages, out_al);
    dim3 grid(R, writes_cache ? 2 : 1);
    const size_t smem = (size_t)(rot > 0 ? rot : 1) * sizeof(float);
#define RFX_N(TI, TO, B)                                                                                           \
    RFX_LAUNCH((latent_low_post_kernel<TI, TO, B>), grid, 128, smem, s, (const TI*)proj, ld, q_w, kv_w, eps, denom, \
               row_pos, row_slot, (TO*)q_out, (TO*)pages, cache, q_rank, rank, rot, width)
#define RFX_GO(TI, TO)              \
    do {                            \
        if (by4) RFX_N(TI, TO, true); \
        else RFX_N(TI, TO, false);  \
    } while (0)
    if (in_dt == RFX_DT_F32 && out_dt == RFX_DT_F32) RFX_GO(float, float);
    else if (in_dt == RFX_DT_F32 && out_dt == RFX_DT_BF16) RFX_GO(float, __nv_bfloat16);
    else if (in_dt == RFX_DT_BF16 && out_dt == RFX_DT_BF16) RFX_GO(__nv_bfloat16, __nv_bfloat16);
    else return RFX_ERR_BAD_ARG;
#undef RFX_GO
#undef RFX_N
    return 0;
}

// x [R, H, n], n - rot and rot / 2 even
extern "C" int rfx_rotate_tails(void* x, int dt, const float* denom, const int* row_pos, int R, int H, int n, int rot,
                                void* stream) {
    if (R <= 0 || H <= 0) return 0;
    if (rot <= 0 || rot > n || rot % 4 || n % 2 || !aligned(x, 8)) return RFX_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem = (size_t)rot * sizeof(float);
    if (dt == RFX_DT_F32) RFX_LAUNCH(rotate_tails_kernel<float>, R, RP_THREADS, smem, s, (float*)x, denom, row_pos, H, n, rot);
    else if (dt == RFX_DT_BF16)
        RFX_LAUNCH(rotate_tails_kernel<__nv_bfloat16>, R, RP_THREADS, smem, s, (__nv_bfloat16*)x, denom, row_pos, H, n, rot);
    else return RFX_ERR_BAD_ARG;
    return 0;
}
