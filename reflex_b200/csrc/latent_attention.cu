// Attention of all heads over one cached row a position that is key and value at once: a
// latent [c | rotated key part | zeros], `width` elements, of which the first are the value.
//
//  * rfx_latent_decode: split-KV attention for rows that each stand at one position
//    (attention_decode.cuh with one tile a page for keys and values): the query heads
//    come folded through the latent's key matrix, the weighted latents go out, and
//    the latent's value matrix follows.  Widths in steps of 64 up to 640.
//  * rfx_latent_gather: the cached rows of a step's sequences, positions 0 up to each
//    sequence's last row of the step, one sequence after another as the rows of a matrix,
//    and where each sequence begins: what a product needs to make every head's keys and
//    values of a prompt at once.
#include "attention_decode.cuh"

namespace {

__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ pages, const int* __restrict__ page_table, int max_pages,
                     const int* __restrict__ seq_slot, const int* __restrict__ seq_start,
                     const int* __restrict__ seq_new, uint4* __restrict__ rows, int* __restrict__ seq_base, int w16) {
    rfx::pdl_prologue();
    const int seq = blockIdx.y;
    int base = 0;
    for (int i = 0; i < seq; ++i) base += seq_start[i] + seq_new[i];
    if (blockIdx.x == 0 && threadIdx.x == 0) seq_base[seq] = base;
    const int n = seq_start[seq] + seq_new[seq];
    // a block a quarter of a page
    constexpr int PART = PAGE / 4;
    const int first = blockIdx.x * PART, count = min(PART, n - first);
    if (count <= 0) return;
    const int page = page_table[(size_t)seq_slot[seq] * max_pages + blockIdx.x / 4];
    const uint4* src = pages + ((size_t)page * PAGE + first % PAGE) * w16;
    uint4* dst = rows + (size_t)(base + first) * w16;
    for (int i = threadIdx.x; i < count * w16; i += blockDim.x) dst[i] = src[i];
}

}  // namespace

// bfloat16 q [R, nq, width], pages [n][64][width] of one key head, out [R, nq, value columns];
// `rank`: how many of a row's first columns are the value; out has the value columns
// rfx_latent_value_columns(width, rank) of a head (columns from `rank` on hold nothing of use).
// `early`: the pages before each row's own were written by earlier steps (a row a sequence).
extern "C" int rfx_latent_value_columns(int width, int rank) {
    return width > 64 && rank <= width - 64 ? width - 64 : width;
}

extern "C" int rfx_latent_decode(const void* q, const void* pages, const int* page_table, int max_pages, int page_size,
                                 const int* row_pos, const int* row_slot, void* out, float* partial, int R, int nq,
                                 int width, int rank, int n_splits, int window, float scale, const float* sink,
                                 long long pool_pages, int cluster, int early, int* err, void* stream) {
    if (R <= 0) return 0;
    if (page_size != PAGE || nq <= 0 || n_splits < 1 || rank <= 0 || rank > width) return RFX_ERR_BAD_ARG;
    if (n_splits > 1 && !partial && !cluster) return RFX_ERR_BAD_ARG;
    if (cluster && n_splits != 2 && n_splits != 4 && n_splits != 8 && n_splits != 16) return RFX_ERR_UNSUPPORTED;
    if (n_splits > MAX_SPLITS || pool_pages <= 0 || pool_pages * PAGE >= 2147483647LL || (nq + 7) / 8 > 65535 ||
        (reinterpret_cast<uintptr_t>(pages) & 15))
        return RFX_ERR_UNSUPPORTED;
    PagedKV cache{page_table, max_pages, page_size, 1, width};
    cudaStream_t s = (cudaStream_t)stream;
    const int dv = rfx_latent_value_columns(width, rank);
#define RFX_GO(D, V)                                                                                                  \
    return launch_decode<D, true, 0, V, true, (D <= 256 ? 3 : 2)>(q, pages, pages, pool_pages, cache, row_pos,        \
                                                                  row_slot, out, partial, R, nq, n_splits, window, 0, \
                                                                  scale, sink, nullptr, 0.0f, cluster, early, err, s);
#define RFX_CASE(D)                  \
    case D:                          \
        if (dv == D) RFX_GO(D, D)    \
        else RFX_GO(D, (D - 64))
    switch (width) {
        case 64:
            RFX_GO(64, 64)
        RFX_CASE(128) RFX_CASE(192) RFX_CASE(256) RFX_CASE(320) RFX_CASE(384) RFX_CASE(448) RFX_CASE(512)
        RFX_CASE(576) RFX_CASE(640)
        default:
            return RFX_ERR_UNSUPPORTED;
    }
#undef RFX_CASE
#undef RFX_GO
}

// rows [sum over sequences of start + new, width] (16-bit elements, width a multiple of 8),
// seq_base [S]; `max_context`: the largest start + new.
extern "C" int rfx_latent_gather(const void* pages, const int* page_table, int max_pages, int page_size,
                                 const int* seq_slot, const int* seq_start, const int* seq_new, void* rows,
                                 int* seq_base, int S, int max_context, int width, void* stream) {
    if (S <= 0 || max_context <= 0) return 0;
    if (page_size != PAGE || width % 8 || S > 65535) return RFX_ERR_BAD_ARG;
    dim3 grid((max_context + PAGE / 4 - 1) / (PAGE / 4), S);
    RFX_LAUNCH(latent_gather_kernel, grid, 256, 0, (cudaStream_t)stream, (const uint4*)pages, page_table, max_pages,
               seq_slot, seq_start, seq_new, (uint4*)rows, seq_base, width / 8);
    return 0;
}
