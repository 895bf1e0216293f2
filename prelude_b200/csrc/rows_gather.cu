// Cached rows out of their pages, in order, one below the other: what a product over a request's whole context reads
// (attention through a latent makes keys and values per head of them for a long prompt portion).
//
// out block b (128 rows) holds positions block_pos0[b] .. + 127 of request block_seq[b] of the step; rows behind the request's
// last cached token are zeros, and so are those that a window has passed before the request's first token of the step.  A row is one key/value head's `width` bfloat16 elements of pages [num_pages, 1, page_size,
// width]; 16 bytes per access.
#include "common.cuh"

namespace {

#define RG_BLOCK 128
#define RG_PART 16                                            // rows of a thread block

__global__ void __launch_bounds__(256) rows_gather_kernel(const __nv_bfloat16* __restrict__ pages, __nv_bfloat16* __restrict__ out,
                                                          const int32_t* __restrict__ block_seq, const int32_t* __restrict__ block_pos0,
                                                          const int32_t* __restrict__ kv_len, const int32_t* __restrict__ cu_q,
                                                          const int32_t* __restrict__ table_row, const int32_t* __restrict__ block_table,
                                                          int table_stride, int page_size, int num_pages, int width,
                                                          const int32_t* __restrict__ q_start, int window, int* __restrict__ status) {
    pb_grid_dep_launch();
    pb_grid_dep_wait();
    const int seq = block_seq[blockIdx.x], pos0 = block_pos0[blockIdx.x] + blockIdx.y * RG_PART;
    const int32_t* table = block_table + (size_t)table_row[cu_q[seq]] * table_stride;
    const int first = window > 0 ? q_start[seq] - window + 1 : 0;    // the first position that a token of the step sees
    const int end = kv_len[seq], pieces = width >> 3;
    __nv_bfloat16* dst = out + ((size_t)blockIdx.x * RG_BLOCK + blockIdx.y * RG_PART) * width;
    for (int i = threadIdx.x; i < RG_PART * pieces; i += blockDim.x) {
        const int r = i / pieces, c = (i - r * pieces) * 8, pos = pos0 + r;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (pos >= first && pos < end) {
            const int page = table[pos / page_size];
            if (page < 0 || page >= num_pages) { if (status) atomicExch(status, 2); }
            else v = *reinterpret_cast<const uint4*>(pages + ((size_t)page * page_size + pos % page_size) * width + c);
        }
        *reinterpret_cast<uint4*>(dst + (size_t)r * width + c) = v;
    }
}

}  // namespace

// pages bfloat16 [num_pages, 1, page_size, width]; out [n_blocks * 128, width]; block_seq, block_pos0 [n_blocks]; kv_len [requests],
// cu_q [requests + 1], table_row [tokens], block_table [rows, table_stride], q_start [requests]: the step's; window 0: none.
PB_API int pb_rows_gather_bf16(const void* pages, void* out, const int32_t* block_seq, const int32_t* block_pos0, int n_blocks,
                               const int32_t* kv_len, const int32_t* cu_q, const int32_t* table_row, const int32_t* block_table, int table_stride,
                               int page_size, int num_pages, int width, const int32_t* q_start, int window, int* status, cudaStream_t stream) {
    PB_REQUIRE(n_blocks >= 0 && width > 0 && width % 8 == 0 && page_size > 0 && num_pages > 0 && table_stride > 0, "rows_gather: bad sizes (rows of %d)", width);
    PB_REQUIRE(pages && out && q_start && window >= 0 && block_seq && block_pos0 && kv_len && cu_q && table_row && block_table && pb_aligned(pages, 16) && pb_aligned(out, 16),
               "rows_gather: null or unaligned pointer");
    if (n_blocks == 0) return 0;
    pb_launch(rows_gather_kernel, dim3(n_blocks, RG_BLOCK / RG_PART), dim3(256), 0, stream, (const __nv_bfloat16*)pages, (__nv_bfloat16*)out, block_seq,
              block_pos0, kv_len, cu_q, table_row, block_table, table_stride, page_size, num_pages, width, q_start, window, status);
    PB_CHECK_LAUNCH("rows_gather");
    return 0;
}
