// Row-wise kernels of layers that norm a sublayer's result before it joins the
// residual (a norm on both sides of every sublayer), and a few small companions.
//
// sandwich_norm: with y a sublayer's 32-bit result [R, H], the residual x [R, H]
// (32-bit, updated in place) and two weights,
//     x <- x + mult * y * rsqrt(mean(y^2) + eps) * w_post
//     out = x * rsqrt(mean(x^2) + eps) * w_next        (when w_next is given)
// so the norm after one sublayer and the norm before the next are one pass over
// the row.  Weights stored around zero come with an offset (w_post and w_next are taken
// as offset + w).  Without w_next `out`, where given, is the new x itself in the product's
// type (layers that norm only what a sublayer gives); with `fresh` x <- mult * norm(y) alone
// (a normed embedding; y may be x).  A block a row; the row lives in shared memory between the sums of
// squares and the outputs.
//
// sum_norm: x <- rms_norm(alpha * x + y) * (offset + w), and the new x in the product's type
// where `out` is given: layers that norm the sum of the stream and a sublayer's result.  y is
// 32-bit rows, or a mixture's expert rows in place order, whose weighted sum (in the order of
// rank) is then made on the way.
//
// group_norm_gate: x [R, C] 32-bit in `groups` equal parts, each over its own
// root mean square, times w[c] (or a weight the parts share, `shared`), times
// sigmoid(z[r, col + c]) or silu of it (`act` 1) when a gate is given.
//
// xielu: z > 0: ap z^2 + z / 2; else an (e^z - 1 - z) + z / 2, with ap and an given
// (the softplus of the stored numbers is taken once, when the weights are bound).
//
// loop_input: x[r, :] += x0[r, :] (when given) + vec[:], the start of a pass over
// a repeated stretch of layers.  tanh_cols: out[r, j] = tanh(in[r, col + j]).
// scaled_sum: a <- sa * a + sb * b.
#include "common.cuh"

namespace {

using namespace rfx;

template <typename TO>
__global__ void __launch_bounds__(256)
sandwich_norm_kernel(const float* y, float* x, const float* __restrict__ w_post,
                     float post_offset, float mult, float eps, const float* __restrict__ w_next,
                     float next_offset, float eps_next, TO* __restrict__ out, int fresh, int H) {
    extern __shared__ __align__(16) float row[];  // [H]
    __shared__ float scratch[32];
    pdl_prologue();
    const size_t base = (size_t)blockIdx.x * H;
    float ss = 0.0f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float v = y[base + c];
        row[c] = v;
        ss = fmaf(v, v, ss);
    }
    const float r1 = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + eps);
    ss = 0.0f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float v = fmaf(mult, (row[c] * r1) * (post_offset + w_post[c]), fresh ? 0.0f : x[base + c]);
        x[base + c] = v;
        row[c] = v;
        ss = fmaf(v, v, ss);
        if (w_next == nullptr && out) st<TO>(out, base + c, v);
    }
    if (w_next == nullptr) return;
    const float r2 = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + eps_next);
    for (int c = threadIdx.x; c < H; c += blockDim.x) st<TO>(out, base + c, (row[c] * r2) * (next_offset + w_next[c]));
}

// The same with 16-byte accesses, for widths that are a multiple of four: the row stays in
// registers (up to V groups of four a thread) between the sums of squares and the outputs.
template <typename TO, int V>
__global__ void __launch_bounds__(512)
sandwich_norm4_kernel(const float* y, float* x, const float* __restrict__ w_post,
                      float post_offset, float mult, float eps, const float* __restrict__ w_next,
                      float next_offset, float eps_next, TO* __restrict__ out, int fresh, int H) {
    __shared__ float scratch[32];
    pdl_prologue();
    const size_t base = (size_t)blockIdx.x * H;
    const int H4 = H / 4;
    const float4* y4 = reinterpret_cast<const float4*>(y + base);
    float4* x4 = reinterpret_cast<float4*>(x + base);
    const float4* wp4 = reinterpret_cast<const float4*>(w_post);
    float4 v[V], xv[V], wp[V];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < H4) {
            v[i] = y4[c];
            xv[i] = fresh ? make_float4(0.0f, 0.0f, 0.0f, 0.0f) : x4[c];
            wp[i] = wp4[c];
            ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
        }
    }
    const float r1 = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + eps);
    ss = 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < H4) {
            v[i].x = fmaf(mult, (v[i].x * r1) * (post_offset + wp[i].x), xv[i].x);
            v[i].y = fmaf(mult, (v[i].y * r1) * (post_offset + wp[i].y), xv[i].y);
            v[i].z = fmaf(mult, (v[i].z * r1) * (post_offset + wp[i].z), xv[i].z);
            v[i].w = fmaf(mult, (v[i].w * r1) * (post_offset + wp[i].w), xv[i].w);
            x4[c] = v[i];
            if (w_next == nullptr && out) store4(out + base + 4 * (size_t)c, v[i]);
            ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
        }
    }
    if (w_next == nullptr) return;
    const float r2 = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + eps_next);
    const float4* wn4 = reinterpret_cast<const float4*>(w_next);
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < H4) {
            const float4 wn = wn4[c];
            store4(out + base + 4 * (size_t)c,
                   make_float4((v[i].x * r2) * (next_offset + wn.x), (v[i].y * r2) * (next_offset + wn.y),
                               (v[i].z * r2) * (next_offset + wn.z), (v[i].w * r2) * (next_offset + wn.w)));
        }
    }
}

// A sublayer's result: rows as they are, or (EXPERTS) sum_k wts[r, k] y[place[r top + k]].
template <typename TY>
struct SubResult {
    const TY* y;
    const int* place;
    const float* wts;  // null: every weight is one
    int top;
};

template <typename TY, typename TO, bool EXPERTS>
__global__ void __launch_bounds__(256)
sum_norm_kernel(SubResult<TY> s, float* __restrict__ x, float alpha, const float* __restrict__ w, float offset, float eps,
                TO* __restrict__ out, int H) {
    extern __shared__ __align__(16) float row[];  // [H]
    __shared__ float scratch[32];
    pdl_prologue();
    const int r = blockIdx.x;
    const size_t base = (size_t)r * H;
    float ss = 0.0f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float y = 0.0f;
        if constexpr (EXPERTS)
            for (int k = 0; k < s.top; ++k)
                y = fmaf(s.wts ? s.wts[(size_t)r * s.top + k] : 1.0f, ld<TY>(s.y, (size_t)s.place[(size_t)r * s.top + k] * H + c), y);
        else
            y = ld<TY>(s.y, base + c);
        const float v = fmaf(alpha, x[base + c], y);
        row[c] = v;
        ss = fmaf(v, v, ss);
    }
    const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float v = (row[c] * f) * (offset + w[c]);
        x[base + c] = v;
        if (out) st<TO>(out, base + c, v);
    }
}

// the same with four elements an access, the row in registers (up to V groups of four a thread)
template <typename TY, typename TO, bool EXPERTS, int V>
__global__ void __launch_bounds__(512)
sum_norm4_kernel(SubResult<TY> s, float* __restrict__ x, float alpha, const float* __restrict__ w, float offset, float eps,
                 TO* __restrict__ out, int H) {
    __shared__ float scratch[32];
    const int H4 = H / 4;
    const int r = blockIdx.x;
    const size_t base = (size_t)r * H;
    const float4* w4 = reinterpret_cast<const float4*>(w);
    float4* x4 = reinterpret_cast<float4*>(x + base);
    float4 wv[V], v[V];
    pdl_launch_dependents();
#pragma unroll
    for (int i = 0; i < V; ++i) {  // the weights are no kernel's output: they come before the wait
        const int c = threadIdx.x + i * blockDim.x;
        if (c < H4) wv[i] = w4[c];
    }
    pdl_wait();
    float ss = 0.0f;
    float4 y[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < H4) {
            v[i] = x4[c];
            y[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if constexpr (!EXPERTS) y[i] = load4(s.y + base + 4 * (size_t)c);
        }
    }
    if constexpr (EXPERTS) {
        for (int k = 0; k < s.top; ++k) {
            const TY* src = s.y + (size_t)s.place[(size_t)r * s.top + k] * H;
            const float f = s.wts ? s.wts[(size_t)r * s.top + k] : 1.0f;
#pragma unroll
            for (int i = 0; i < V; ++i) {
                const int c = threadIdx.x + i * blockDim.x;
                if (c >= H4) continue;
                const float4 t = load4(src + 4 * (size_t)c);
                y[i].x = fmaf(f, t.x, y[i].x);
                y[i].y = fmaf(f, t.y, y[i].y);
                y[i].z = fmaf(f, t.z, y[i].z);
                y[i].w = fmaf(f, t.w, y[i].w);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < H4) {
            v[i].x = fmaf(alpha, v[i].x, y[i].x);
            v[i].y = fmaf(alpha, v[i].y, y[i].y);
            v[i].z = fmaf(alpha, v[i].z, y[i].z);
            v[i].w = fmaf(alpha, v[i].w, y[i].w);
            ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
        }
    }
    const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + eps);
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < H4) {
            const float4 t = make_float4((v[i].x * f) * (offset + wv[i].x), (v[i].y * f) * (offset + wv[i].y),
                                         (v[i].z * f) * (offset + wv[i].z), (v[i].w * f) * (offset + wv[i].w));
            x4[c] = t;
            if (out) store4(out + base + 4 * (size_t)c, t);
        }
    }
}

template <typename TY, typename TO, bool EXPERTS>
int launch_sum_norm(const SubResult<TY>& y, float* x, float alpha, const float* w, float offset, float eps, TO* out, int R,
                    int H, cudaStream_t s) {
    const bool al = ((reinterpret_cast<uintptr_t>(y.y) | reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) |
                      reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    if (H % 4 == 0 && H <= 4 * 512 * 4 && al) {
        const int H4 = H / 4;
        const int threads = H4 <= 128 ? 128 : H4 <= 256 ? 256 : 512;
#define RFX_V(V) RFX_LAUNCH((sum_norm4_kernel<TY, TO, EXPERTS, V>), R, threads, 0, s, y, x, alpha, w, offset, eps, out, H)
        if (H4 <= threads) RFX_V(1);
        else if (H4 <= 2 * threads) RFX_V(2);
        else RFX_V(4);
#undef RFX_V
        return 0;
    }
    const size_t smem = (size_t)H * sizeof(float);
    if (smem > 200 * 1024) return RFX_ERR_UNSUPPORTED;
    auto kernel = sum_norm_kernel<TY, TO, EXPERTS>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    RFX_LAUNCH(kernel, R, 256, smem, s, y, x, alpha, w, offset, eps, out, H);
    return 0;
}

// sigmoid(t), or (act 1) silu(t)
__device__ __forceinline__ float gate_of(float t, int act) {
    const float s = 1.0f / (1.0f + exact_expf(-t));
    return act ? t * s : s;
}
// the same for a result that is rounded to bfloat16: the hardware's exponential and division
template <typename TO>
__device__ __forceinline__ float gate_for(float t, int act) {
    if constexpr (sizeof(TO) == 2) return __fdividef(act ? t : 1.0f, 1.0f + __expf(-t));
    else return gate_of(t, act);
}

// One block a (row, part), 16 bytes an access: parts of many elements (a norm in a few equal
// parts of a wide row), where a warp a part would leave a row to a warp or two.
template <typename TO>
__global__ void __launch_bounds__(256)
group_norm_gate_wide_kernel(const float* __restrict__ x, const float* __restrict__ w, float eps,
                            const float* __restrict__ z, int ldz, int zcol, int act, int shared,
                            TO* __restrict__ out, int C, int gs) {
    __shared__ float scratch[32];
    pdl_prologue();
    const int r = blockIdx.x, g = blockIdx.y;
    const size_t base = (size_t)r * C + (size_t)g * gs;
    const float4* x4 = reinterpret_cast<const float4*>(x + base);
    const float4* w4 = reinterpret_cast<const float4*>(shared ? w : w + (size_t)g * gs);
    float ss = 0.0f;
    for (int c = threadIdx.x; c < gs / 4; c += blockDim.x) {
        const float4 v = x4[c];
        ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
    const float rs = 1.0f / sqrtf(block_sum(ss, scratch) / (float)gs + eps);
    for (int c = threadIdx.x; c < gs / 4; c += blockDim.x) {
        const float4 v = x4[c], wv = w4[c];
        float4 o = make_float4((v.x * rs) * wv.x, (v.y * rs) * wv.y, (v.z * rs) * wv.z, (v.w * rs) * wv.w);
        if (z) {
            const float* zp = z + (size_t)r * ldz + zcol + (size_t)g * gs + 4 * c;
            o.x *= gate_of(zp[0], act);
            o.y *= gate_of(zp[1], act);
            o.z *= gate_of(zp[2], act);
            o.w *= gate_of(zp[3], act);
        }
        store4(out + base + 4 * (size_t)c, o);
    }
}

// Parts of up to 512 elements, a multiple of four: a warp a part, the part in registers between
// its sum of squares and the outputs, 16 bytes an access, the gate's loads beside the row's.
template <typename TO>
__global__ void __launch_bounds__(256)
group_norm_gate4_kernel(const float* __restrict__ x, const float* __restrict__ w, float eps,
                        const float* __restrict__ z, int ldz, int zcol, int act, int shared, TO* __restrict__ out,
                        long long parts, int groups, int gs) {
    pdl_prologue();
    const long long part = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (part >= parts) return;
    const int lane = threadIdx.x & 31, g = (int)(part % groups);
    const size_t r = (size_t)(part / groups), base = (size_t)part * gs;
    constexpr int V = 4;
    float4 v[V], t[V];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int c = 4 * (lane + 32 * i);
        if (c < gs) {
            v[i] = *reinterpret_cast<const float4*>(x + base + c);
            if (z) t[i] = *reinterpret_cast<const float4*>(z + r * ldz + zcol + (size_t)g * gs + c);
            ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
        }
    }
    const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)gs + eps);
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int c = 4 * (lane + 32 * i);
        if (c < gs) {
            const float4 ww = *reinterpret_cast<const float4*>(w + (shared ? 0 : (size_t)g * gs) + c);
            float4 o = make_float4((v[i].x * rs) * ww.x, (v[i].y * rs) * ww.y, (v[i].z * rs) * ww.z, (v[i].w * rs) * ww.w);
            if (z) {
                o.x *= gate_for<TO>(t[i].x, act);
                o.y *= gate_for<TO>(t[i].y, act);
                o.z *= gate_for<TO>(t[i].z, act);
                o.w *= gate_for<TO>(t[i].w, act);
            }
            store4(out + base + c, o);
        }
    }
}

template <typename TO>
__global__ void __launch_bounds__(256)
group_norm_gate_kernel(const float* __restrict__ x, const float* __restrict__ w, float eps,
                       const float* __restrict__ z, int ldz, int zcol, int act, int shared, TO* __restrict__ out,
                       int C, int groups) {
    pdl_prologue();
    const int r = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    const int gs = C / groups;
    // a warp a part; a row's parts spread over the blocks of its grid row
    for (int g = blockIdx.y * nwarps + warp; g < groups; g += gridDim.y * nwarps) {
        const float* xr = x + (size_t)r * C + (size_t)g * gs;
        float ss = 0.0f;
        for (int c = lane; c < gs; c += 32) ss = fmaf(xr[c], xr[c], ss);
        const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)gs + eps);
        for (int c = lane; c < gs; c += 32) {
            float v = (xr[c] * rs) * w[shared ? c : g * gs + c];
            if (z) {
                const float t = z[(size_t)r * ldz + zcol + g * gs + c];
                v *= gate_of(t, act);
            }
            st<TO>(out, (size_t)r * C + (size_t)g * gs + c, v);
        }
    }
}

template <typename T>
__global__ void xielu_kernel(T* __restrict__ a, size_t n, float ap, float an) {
    pdl_prologue();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const float z = ld<T>(a, i);
        float v;
        if (z > 0.0f) v = fmaf(ap * z, z, 0.5f * z);
        else v = fmaf(an, expm1f(z) - z, 0.5f * z);
        st<T>(a, i, v);
    }
}

__global__ void loop_input_kernel(float* __restrict__ x, const float* __restrict__ x0,
                                  const float* __restrict__ vec, size_t n, int H) {
    pdl_prologue();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        float v = x[i];
        if (x0) v += x0[i];
        x[i] = v + vec[i % H];
    }
}

template <typename TO>
__global__ void tanh_cols_kernel(const float* __restrict__ in, int ld, int col, TO* __restrict__ out, int R, int n) {
    pdl_prologue();
    const size_t total = (size_t)R * n;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x)
        st<TO>(out, i, tanhf(in[(i / n) * ld + col + (i % n)]));
}

__global__ void scaled_sum_kernel(float* __restrict__ a, const float* __restrict__ b, float sa, float sb, size_t n) {
    pdl_prologue();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        a[i] = fmaf(sa, a[i], sb * b[i]);
}

inline int blocks_for(size_t n, int threads) {
    size_t b = (n + threads - 1) / threads;
    const size_t cap = (size_t)sm_count() * 8;
    return (int)(b < 1 ? 1 : (b > cap ? cap : b));
}

}  // namespace

extern "C" int rfx_sandwich_norm(const float* y, float* x, const float* w_post, float post_offset, float mult,
                                 float eps, const float* w_next, float next_offset, float eps_next, void* out,
                                 int out_dt, int fresh, int R, int H, void* stream) {
    if (R <= 0) return 0;
    const size_t smem = (size_t)H * sizeof(float);
    if (smem > 200 * 1024) return RFX_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const bool al = ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w_post) |
                      reinterpret_cast<uintptr_t>(w_next) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    if (H % 4 == 0 && H <= 4 * 512 * 4 && al) {
        // the row in registers, 16 bytes an access; threads so that a thread holds one to four groups
        const int H4 = H / 4;
        const int threads = H4 <= 128 ? 128 : H4 <= 256 ? 256 : 512;
#define RFX_V(TO, V)                                                                                           \
    RFX_LAUNCH((sandwich_norm4_kernel<TO, V>), R, threads, 0, s, y, x, w_post, post_offset, mult, eps, w_next, \
               next_offset, eps_next, (TO*)out, fresh, H)
#define RFX_PICK(TO)                                      \
    do {                                                  \
        if (H4 <= threads) RFX_V(TO, 1);                  \
        else if (H4 <= 2 * threads) RFX_V(TO, 2);         \
        else RFX_V(TO, 4);                                \
    } while (0)
        if (out_dt == RFX_DT_F32) RFX_PICK(float);
        else if (out_dt == RFX_DT_BF16) RFX_PICK(__nv_bfloat16);
        else return RFX_ERR_BAD_ARG;
#undef RFX_PICK
#undef RFX_V
        return 0;
    }
#define RFX_GO(TO)                                                                                          \
    do {                                                                                                    \
        if (smem > 48 * 1024) {                                                                             \
            cudaError_t e = cudaFuncSetAttribute(sandwich_norm_kernel<TO>,                                  \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);   \
            if (e != cudaSuccess) return (int)e;                                                            \
        }                                                                                                   \
        RFX_LAUNCH(sandwich_norm_kernel<TO>, R, 256, smem, s, y, x, w_post, post_offset, mult, eps, w_next, \
                   next_offset, eps_next, (TO*)out, fresh, H);                                                                           \
    } while (0)
    if (out_dt == RFX_DT_F32) RFX_GO(float);
    else if (out_dt == RFX_DT_BF16) RFX_GO(__nv_bfloat16);
    else return RFX_ERR_BAD_ARG;
#undef RFX_GO
    return 0;
}

// y: [R, H] (32-bit), or with `place` the expert rows that row r's `top` places name
extern "C" int rfx_sum_norm(const void* y, int y_dt, const int* place, const float* wts, int top, float* x, float alpha,
                            const float* w, float offset, float eps, void* out, int out_dt, int R, int H, void* stream) {
    if (R <= 0) return 0;
    if (H <= 0 || !w || (place && top <= 0)) return RFX_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
#define RFX_GO(TY, TO, EX)                                                                                              \
    return launch_sum_norm<TY, TO, EX>(SubResult<TY>{(const TY*)y, place, wts, top}, x, alpha, w, offset, eps, (TO*)out, \
                                       R, H, s)
#define RFX_OUT(TY, EX)                                     \
    do {                                                    \
        if (out_dt == RFX_DT_F32) RFX_GO(TY, float, EX);    \
        if (out_dt == RFX_DT_BF16) RFX_GO(TY, __nv_bfloat16, EX); \
        return RFX_ERR_BAD_ARG;                             \
    } while (0)
    if (place) {
        if (y_dt == RFX_DT_F32) RFX_OUT(float, true);
        if (y_dt == RFX_DT_BF16) RFX_OUT(__nv_bfloat16, true);
    } else if (y_dt == RFX_DT_F32) {
        RFX_OUT(float, false);
    }
#undef RFX_OUT
#undef RFX_GO
    return RFX_ERR_BAD_ARG;
}

extern "C" int rfx_group_norm_gate(const float* x, const float* w, float eps, const float* z, int ldz, int zcol,
                                   int act, int shared, void* out, int out_dt, int R, int C, int groups,
                                   void* stream) {
    if (R <= 0) return 0;
    if (groups <= 0 || C % groups) return RFX_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const int gs = C / groups;
    const bool al = ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    if (gs >= 512 && gs % 4 == 0 && C % 4 == 0 && al && groups <= 65535) {
        dim3 grid(R, groups);
        if (out_dt == RFX_DT_F32)
            RFX_LAUNCH(group_norm_gate_wide_kernel<float>, grid, 256, 0, s, x, w, eps, z, ldz, zcol, act, shared,
                       (float*)out, C, gs);
        else if (out_dt == RFX_DT_BF16)
            RFX_LAUNCH(group_norm_gate_wide_kernel<__nv_bfloat16>, grid, 256, 0, s, x, w, eps, z, ldz, zcol, act, shared,
                       (__nv_bfloat16*)out, C, gs);
        else return RFX_ERR_BAD_ARG;
        return 0;
    }
    const long long parts = (long long)R * groups;
    if (gs % 4 == 0 && gs <= 512 && al && (!z || (ldz % 4 == 0 && zcol % 4 == 0 && (reinterpret_cast<uintptr_t>(z) & 15) == 0)) &&
        (parts + 7) / 8 <= 2147483647LL) {
        const int blocks = (int)((parts + 7) / 8);
        if (out_dt == RFX_DT_F32)
            RFX_LAUNCH(group_norm_gate4_kernel<float>, blocks, 256, 0, s, x, w, eps, z, ldz, zcol, act, shared,
                       (float*)out, parts, groups, gs);
        else if (out_dt == RFX_DT_BF16)
            RFX_LAUNCH(group_norm_gate4_kernel<__nv_bfloat16>, blocks, 256, 0, s, x, w, eps, z, ldz, zcol, act, shared,
                       (__nv_bfloat16*)out, parts, groups, gs);
        else return RFX_ERR_BAD_ARG;
        return 0;
    }
    const int threads = groups >= 4 ? 128 : 32 * groups;
    int gy = (groups + 3) / 4;
    if (gy > 65535) gy = 65535;
    dim3 grid(R, gy);
    if (out_dt == RFX_DT_F32)
        RFX_LAUNCH(group_norm_gate_kernel<float>, grid, threads, 0, s, x, w, eps, z, ldz, zcol, act, shared,
                   (float*)out, C, groups);
    else if (out_dt == RFX_DT_BF16)
        RFX_LAUNCH(group_norm_gate_kernel<__nv_bfloat16>, grid, threads, 0, s, x, w, eps, z, ldz, zcol, act, shared,
                   (__nv_bfloat16*)out, C, groups);
    else return RFX_ERR_BAD_ARG;
    return 0;
}

extern "C" int rfx_xielu(void* a, int dt, long long n, float ap, float an, void* stream) {
    if (n <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const int blocks = blocks_for((size_t)n, 256);
    if (dt == RFX_DT_F32) RFX_LAUNCH(xielu_kernel<float>, blocks, 256, 0, s, (float*)a, (size_t)n, ap, an);
    else if (dt == RFX_DT_BF16)
        RFX_LAUNCH(xielu_kernel<__nv_bfloat16>, blocks, 256, 0, s, (__nv_bfloat16*)a, (size_t)n, ap, an);
    else return RFX_ERR_BAD_ARG;
    return 0;
}

extern "C" int rfx_loop_input(float* x, const float* x0, const float* vec, int R, int H, void* stream) {
    if (R <= 0) return 0;
    const size_t n = (size_t)R * H;
    RFX_LAUNCH(loop_input_kernel, blocks_for(n, 256), 256, 0, (cudaStream_t)stream, x, x0, vec, n, H);
    return 0;
}

extern "C" int rfx_tanh_cols(const float* in, int ld, int col, void* out, int out_dt, int R, int n, void* stream) {
    if (R <= 0 || n <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const int blocks = blocks_for((size_t)R * n, 256);
    if (out_dt == RFX_DT_F32) RFX_LAUNCH(tanh_cols_kernel<float>, blocks, 256, 0, s, in, ld, col, (float*)out, R, n);
    else if (out_dt == RFX_DT_BF16)
        RFX_LAUNCH(tanh_cols_kernel<__nv_bfloat16>, blocks, 256, 0, s, in, ld, col, (__nv_bfloat16*)out, R, n);
    else return RFX_ERR_BAD_ARG;
    return 0;
}

extern "C" int rfx_scaled_sum(float* a, const float* b, float sa, float sb, long long n, void* stream) {
    if (n <= 0) return 0;
    RFX_LAUNCH(scaled_sum_kernel, blocks_for((size_t)n, 256), 256, 0, (cudaStream_t)stream, a, b, sa, sb, (size_t)n);
    return 0;
}
