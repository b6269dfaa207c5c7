// Token embedding: out[t, :] = float(table[ids[t], :]) * scale.  The residual stream
// that it starts is float32 in both precisions.
// Formula: src/HyMT2Sharp/HunyuanDenseModel.cs:494-537 (row gather; that model has no scale, so its
// scale is 1; architectures that multiply their embeddings by a constant give it here).
#include "common.cuh"

template <typename T>
__global__ void embed_kernel(float* __restrict__ out, const T* __restrict__ table,
                             const int* __restrict__ ids, int hidden, int vocab, float scale, int* status) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    int id = ids[t];
    if (id < 0 || id >= vocab) {  // never read outside the table: flag it and give zeros
        if (threadIdx.x == 0) atomicExch(status, 1);
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) out[(size_t)t * hidden + i] = 0.f;
        return;
    }
    const T* row = table + (size_t)id * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) out[(size_t)t * hidden + i] = scale == 1.0f ? to_float(row[i]) : to_float(row[i]) * scale;
}

HYMT2_API int hymt2_embed(float* out, const void* table, int table_dtype, const int* ids, int tokens,
                          int hidden, int vocab, float scale, int* status, cudaStream_t stream) {
    if (tokens == 0) return HYMT2_OK;
    HYMT2_REQUIRE(tokens > 0 && hidden > 0 && vocab > 0, "embed: bad sizes tokens=%d hidden=%d vocab=%d", tokens, hidden, vocab);
    HYMT2_DISPATCH_DTYPE(table_dtype, T,
        launch_pdl(embed_kernel<T>, dim3(tokens), dim3(256), 0, stream, out, (const T*)table, ids, hidden, vocab, scale, status));
    return hymt2_check_launch("embed");
}

// The same with a stored vector per position: out[t] = table[id] * scale + positions[pos[t]] (not scaled), written a second time to
// `copy` where one is given (a model that needs the embedding's output again further up).  A position outside the table gives
// status 3 and zeros.
template <typename T>
__global__ void embed_positions_kernel(float* __restrict__ out, float* __restrict__ copy, const T* __restrict__ table, const T* __restrict__ positions,
                                       const int* __restrict__ ids, const int* __restrict__ token_pos, int hidden, int vocab, int max_positions,
                                       float scale, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    const size_t t = blockIdx.x;
    const int id = ids[t], pos = token_pos[t];
    const bool ok = id >= 0 && id < vocab && pos >= 0 && pos < max_positions;
    if (!ok && threadIdx.x == 0) atomicExch(status, id < 0 || id >= vocab ? 1 : 3);
    const T* row = table + (size_t)(ok ? id : 0) * hidden;
    const T* at = positions + (size_t)(ok ? pos : 0) * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = ok ? fmaf(to_float(row[i]), scale, to_float(at[i])) : 0.f;
        out[t * hidden + i] = v;
        if (copy) copy[t * hidden + i] = v;
    }
}

HYMT2_API int hymt2_embed_positions(float* out, float* copy, const void* table, const void* positions, int table_dtype, const int* ids,
                                    const int* token_pos, int tokens, int hidden, int vocab, int max_positions, float scale, int* status,
                                    cudaStream_t stream) {
    if (tokens == 0) return HYMT2_OK;
    HYMT2_REQUIRE(tokens > 0 && hidden > 0 && vocab > 0 && max_positions > 0 && positions, "embed_positions: bad sizes tokens=%d hidden=%d vocab=%d positions=%d",
                  tokens, hidden, vocab, max_positions);
    HYMT2_DISPATCH_DTYPE(table_dtype, T,
        launch_pdl(embed_positions_kernel<T>, dim3(tokens), dim3(256), 0, stream, out, copy, (const T*)table, (const T*)positions, ids, token_pos,
                   hidden, vocab, max_positions, scale, status));
    return hymt2_check_launch("embed_positions");
}

// The same with a second table: out[t] = table[id] * scale + pairs[row], row = (previous token * mul_prev + id * mul_cur) mod
// buckets, and row `buckets` for a sequence's first token (position 0).  The token in front of a step's first one is the
// int32 at `state_offset` of the sequence's state row, which then receives the step's last token: the block of a sequence's
// first token reads it and writes it, so nothing is read after it was overwritten.  Rows without a slot touch no state.
template <typename T>
__global__ void embed_pairs_kernel(float* __restrict__ out, const T* __restrict__ table, const T* __restrict__ pairs,
                                   const int* __restrict__ ids, const int* __restrict__ token_seq, const int* __restrict__ token_pos,
                                   const int* __restrict__ cu_seqlens, const int* __restrict__ slot_ids, uint8_t* state, long state_offset,
                                   long state_stride, int hidden, int vocab, float scale, int buckets, long long mul_prev,
                                   long long mul_cur, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ int row_s;
    const int t = blockIdx.x;
    const int id = ids[t];
    if (threadIdx.x == 0) {
        const int seq = token_seq[t], slot = slot_ids[seq], first = cu_seqlens[seq];
        int* kept = slot >= 0 ? reinterpret_cast<int*>(state + (size_t)slot * state_stride + state_offset) : nullptr;
        long long row = buckets;
        if (token_pos[t] > 0 && slot >= 0) {
            const long long prev = t == first ? *kept : ids[t - 1];
            row = (prev * mul_prev + (long long)id * mul_cur) % buckets;
            if (row < 0) row += buckets;
        }
        if (t == first && kept) *kept = ids[cu_seqlens[seq + 1] - 1];
        row_s = (int)row;
    }
    __syncthreads();
    if (id < 0 || id >= vocab) {  // never read outside the table: flag it and give zeros
        if (threadIdx.x == 0) atomicExch(status, 1);
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) out[(size_t)t * hidden + i] = 0.f;
        return;
    }
    const T* row = table + (size_t)id * hidden;
    const T* pair = pairs + (size_t)row_s * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x)
        out[(size_t)t * hidden + i] = fmaf(to_float(row[i]), scale, to_float(pair[i]));
}

HYMT2_API int hymt2_embed_pairs(float* out, const void* table, const void* pairs, int table_dtype, const int* ids, const int* token_seq,
                                const int* token_pos, const int* cu_seqlens, const int* slot_ids, void* state, long state_offset,
                                long state_stride, int tokens, int hidden, int vocab, float scale, int buckets, long long mul_prev,
                                long long mul_cur, int* status, cudaStream_t stream) {
    if (tokens == 0) return HYMT2_OK;
    HYMT2_REQUIRE(tokens > 0 && hidden > 0 && vocab > 0 && buckets > 0, "embed_pairs: bad sizes tokens=%d hidden=%d vocab=%d buckets=%d", tokens,
                  hidden, vocab, buckets);
    HYMT2_REQUIRE(state && state_offset % 4 == 0 && state_stride % 4 == 0, "embed_pairs: the state rows are not aligned");
    HYMT2_DISPATCH_DTYPE(table_dtype, T,
        launch_pdl(embed_pairs_kernel<T>, dim3(tokens), dim3(256), 0, stream, out, (const T*)table, (const T*)pairs, ids, token_seq, token_pos,
                   cu_seqlens, slot_ids, (uint8_t*)state, state_offset, state_stride, hidden, vocab, scale, buckets, mul_prev, mul_cur, status));
    return hymt2_check_launch("embed_pairs");
}

// After a decode step: every live row of the batch is one token longer.
__global__ void advance_decode_kernel(int* token_pos, int* kv_lens, const int* slot_ids, int rows) {
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b >= rows || slot_ids[b] < 0) return;
    token_pos[b] += 1;
    kv_lens[b] += 1;
}

HYMT2_API int hymt2_advance_decode(int* token_pos, int* kv_lens, const int* slot_ids, int rows, cudaStream_t stream) {
    if (rows == 0) return HYMT2_OK;
    launch_pdl(advance_decode_kernel, dim3((rows + 127) / 128), dim3(128), 0, stream, token_pos, kv_lens, slot_ids, rows);
    return hymt2_check_launch("advance_decode");
}

// Asks for `bytes` from `ptr` on to be brought into L2 (cp.async.bulk.prefetch.L2 in pieces of 16 KB), for a stream
// beside the one that computes: a decode step leaves the memory idle most of the time, and the next large product's
// weights can come in meanwhile.  Nothing is written anywhere.
__global__ void l2_prefetch_kernel(const uint8_t* ptr, long bytes) {
    constexpr long PIECE = 16384;
    const long pieces = (bytes + PIECE - 1) / PIECE;
    for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < pieces; i += (long)gridDim.x * blockDim.x) {
        const long off = i * PIECE;
        const uint32_t n = (uint32_t)min(PIECE, bytes - off);
        asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(ptr + off), "r"(n) : "memory");
    }
}

HYMT2_API int hymt2_l2_prefetch(const void* ptr, long bytes, cudaStream_t stream) {
    bytes &= ~15L;
    if (bytes <= 0) return HYMT2_OK;
    HYMT2_REQUIRE(ptr != nullptr && (uintptr_t)ptr % 16 == 0, "l2_prefetch: the address must be 16-byte aligned");
    const long pieces = (bytes + 16383) / 16384;
    const unsigned blocks = (unsigned)(pieces < 128 * 32 ? (pieces + 31) / 32 : 128);
    l2_prefetch_kernel<<<blocks, 32, 0, stream>>>((const uint8_t*)ptr, bytes);
    return hymt2_check_launch("l2_prefetch");
}

// The device's clock (nanoseconds of %globaltimer) into out[0]: launched between the kernels of a captured step while
// kernels are being timed, since a graph can hold this where the host cannot look.  Launched without programmatic
// overlap, so a stamp is taken when everything in front of it on the stream is complete.
__global__ void stamp_kernel(unsigned long long* out) {
    unsigned long long t;
    asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
    *out = t;
}

HYMT2_API int hymt2_stamp(unsigned long long* out, cudaStream_t stream) {
    HYMT2_REQUIRE(out != nullptr, "stamp: no place to write");
    stamp_kernel<<<1, 1, 0, stream>>>(out);
    return hymt2_check_launch("stamp");
}
