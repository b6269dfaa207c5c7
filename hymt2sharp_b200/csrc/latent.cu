// Low-rank (latent) key/value attention: what happens between the fused projection and the attention itself.
//
// The projection of a token holds, side by side, the queries of all heads (per head `dim` entries that meet the
// keys made from the latent vector, then `rot` entries that meet the rotated key part) and the compressed row
// (`rank` entries of the latent vector, then `rot` entries of the one rotated key part that all heads share).
// This kernel, one block per token, all arithmetic in float32:
//   * divides the latent vector by its root mean square (eps inside the root), multiplies it by its gain and
//     writes it to the token's row of the cache, entries [0, rank);
//   * rotates the shared key part by the token's position and writes it behind it, entries [rank, rank + rot);
//   * rotates the `rot` part of every head's query and writes it to q_out[t, h, rank .. rank + rot): the place
//     behind the head's `rank` entries, which the product with the key up-projection fills.
// Where the queries come out of a latent vector of their own, the projection starts with that vector instead: it is normed
// with its gain into cq_out, and the heads' queries, once a product has made them, come through this kernel in a second
// call, as a projection without a compressed row.
// Rotation: of the first `rot_dims` entries, (2i, 2i+1) are a pair that turns by angle = position * inv_freq[i]
// (a float32 product); cosine and sine are multiplied by `amplitude`; entries from rot_dims on pass unchanged.
// Cache plane: [block][token in block][rank + rot]; block_table[slot * table_stride + pos / block_tokens] names
// the block.  A token of a padding row (slot < 0) writes its query part and nothing else.
#include "common.cuh"

namespace {

struct LatentPrepParams {
    const void* proj;     // [T, ldp]
    void* q_out;          // [T, heads * (rank + rot)], or null: the rotated query parts go back into proj, in place
    void* rows_out;       // [T, rank + rot] or null: the compressed rows once more, side by side for all tokens
    void* cache;          // plane base, or null: nothing is written (a run that reads another run's cache)
    const int* block_table;
    const int* token_seq;
    const int* token_pos;
    const int* slot_ids;
    const float* gain;      // [rank]
    const float* inv_freq;  // [rot_dims / 2]
    long ldp;
    int q_cols;             // where the compressed row starts inside a projection row: behind the queries (heads * (dim + rot)), or
                            // behind a compressed query of q_rank entries
    const float* q_gain;    // [q_rank]: the projection starts with a compressed query, which is normed into cq_out; null: with the queries
    void* cq_out;           // [T, q_rank]
    int q_rank;
    int table_stride, block_tokens, heads, dim, rot, rank, rot_dims;
    float eps, amplitude;
};

template <typename T>
__global__ void __launch_bounds__(512)
latent_prep_kernel(LatentPrepParams p) {
    extern __shared__ float smem[];   // [rot_dims / 2][2] cosine, sine; then 33 floats for the sum
    float* cs = smem;
    float* scratch = smem + p.rot_dims;
    pdl_wait();   // everything in front is complete before anything is read; then the next kernel may be set up meanwhile
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int pos = p.token_pos[t];
    const int slot = p.slot_ids[p.token_seq[t]];
    const T* row = (const T*)p.proj + (size_t)t * p.ldp;
    const int half = p.rot_dims / 2;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float angle = (float)pos * p.inv_freq[i];
        float sn, c;
        sincosf(angle, &sn, &c);
        cs[2 * i] = c * p.amplitude;
        cs[2 * i + 1] = sn * p.amplitude;
    }
    // the latent vectors' sums of squares (block_sum synchronises, which also publishes cs)
    const T* lat = row + p.q_cols;
    float ss = 0.f, qs = 0.f;
    if (p.cq_out)
        for (int i = threadIdx.x; i < p.q_rank; i += blockDim.x) {
            const float v = to_float(row[i]);
            qs = fmaf(v, v, qs);
        }
    if (p.cache || p.rows_out)      // (a projection without a compressed row of its own is never read behind its queries)
        for (int i = threadIdx.x; i < p.rank; i += blockDim.x) {
            const float v = to_float(lat[i]);
            ss = fmaf(v, v, ss);
        }
    ss = block_sum(ss, scratch);
    if (p.cq_out) {   // the compressed query: normed as the latent vector is; there are no heads' queries yet
        const float scale = 1.0f / sqrtf(block_sum(qs, scratch) / (float)p.q_rank + p.eps);
        T* o = (T*)p.cq_out + (size_t)t * p.q_rank;
        for (int i = threadIdx.x; i < p.q_rank; i += blockDim.x) o[i] = from_float<T>(to_float(row[i]) * scale * p.q_gain[i]);
    }
    const int dl = p.rank + p.rot;
    T* dst = nullptr;    // the token's cache row
    if (p.cache && slot >= 0) {
        const int block = p.block_table[(size_t)slot * p.table_stride + pos / p.block_tokens];
        dst = (T*)p.cache + ((size_t)block * p.block_tokens + (pos % p.block_tokens)) * dl;
    }
    T* dst2 = p.rows_out ? (T*)p.rows_out + (size_t)t * dl : nullptr;
    if (dst || dst2) {
        const float scale = 1.0f / sqrtf(ss / (float)p.rank + p.eps);
        for (int i = threadIdx.x; i < p.rank; i += blockDim.x) {
            const T v = from_float<T>(to_float(lat[i]) * scale * p.gain[i]);
            if (dst) dst[i] = v;
            if (dst2) dst2[i] = v;
        }
        const T* kr = lat + p.rank;
        for (int i = threadIdx.x; i < half; i += blockDim.x) {
            const float a = to_float(kr[2 * i]), b = to_float(kr[2 * i + 1]);
            const T v0 = from_float<T>(a * cs[2 * i] - b * cs[2 * i + 1]), v1 = from_float<T>(b * cs[2 * i] + a * cs[2 * i + 1]);
            if (dst) { dst[p.rank + 2 * i] = v0; dst[p.rank + 2 * i + 1] = v1; }
            if (dst2) { dst2[p.rank + 2 * i] = v0; dst2[p.rank + 2 * i + 1] = v1; }
        }
        for (int i = p.rot_dims + threadIdx.x; i < p.rot; i += blockDim.x) {
            if (dst) dst[p.rank + i] = kr[i];
            if (dst2) dst2[p.rank + i] = kr[i];
        }
    }
    // the heads' rotated query parts
    const int per_head = half + (p.rot - p.rot_dims);
    for (int item = threadIdx.x; item < p.heads * per_head; item += blockDim.x) {
        const int h = item / per_head, i = item - h * per_head;
        const T* q = row + (size_t)h * (p.dim + p.rot) + p.dim;
        T* o = p.q_out ? (T*)p.q_out + (size_t)t * p.heads * dl + (size_t)h * dl + p.rank : const_cast<T*>(q);
        if (i < half) {
            const float a = to_float(q[2 * i]), b = to_float(q[2 * i + 1]);
            o[2 * i] = from_float<T>(a * cs[2 * i] - b * cs[2 * i + 1]);
            o[2 * i + 1] = from_float<T>(b * cs[2 * i] + a * cs[2 * i + 1]);
        } else {
            const int x = p.rot_dims + (i - half);
            o[x] = q[x];
        }
    }
}

// Whole prompts from position 0 for the paged prompt attention: every head's queries, keys and values in the layout that kernel
// reads, with heads of D and DV entries (D: dim + rot and zeros behind them).  One block per token, 16 bytes a thread and access:
//   q_out[t, h] = [query entries | rotated query entries | zeros]
//   k_out[block][h][place] = [own key entries | shared rotated key entries | zeros],  v_out[block][h][place] = values
// A sequence's tokens fill blocks of BLOCK_TOKENS of its own, numbered through the step; table[slot][i] names its i-th block.
constexpr int BLOCK_TOKENS = 64;

struct LatentPlaceParams {
    const __nv_bfloat16* q;       // [T, ldq], not rotated
    const __nv_bfloat16* kv;      // [T, ld_kv]: heads' own key entries (dim each), then heads' values (dv each)
    const __nv_bfloat16* shared;  // [T, ld_shared]: the shared key entries, rotated
    long ldq, ld_kv, ld_shared;
    __nv_bfloat16 *q_out, *k_out, *v_out;
    int* table;
    const int *token_seq, *token_pos, *cu_seqlens, *slot_ids;
    const float* inv_freq;
    int table_stride, heads, dim, rot, dv, D, rot_dims, max_blocks;
    float amplitude;
};

__global__ void __launch_bounds__(256)
latent_place_kernel(LatentPlaceParams p) {
    extern __shared__ float smem[];   // [rot_dims / 2][2] cosine, sine
    __shared__ int block_s;
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x, seq = p.token_seq[t], pos = p.token_pos[t];
    const int place = t - p.cu_seqlens[seq];
    if (threadIdx.x == 0) {
        int block = place / BLOCK_TOKENS;
        for (int b = 0; b < seq; b++) block += (p.cu_seqlens[b + 1] - p.cu_seqlens[b] + BLOCK_TOKENS - 1) / BLOCK_TOKENS;
        block_s = block;
        const int slot = p.slot_ids[seq];
        if (place % BLOCK_TOKENS == 0 && slot >= 0) p.table[(size_t)slot * p.table_stride + place / BLOCK_TOKENS] = block;
    }
    for (int i = threadIdx.x; i < p.rot_dims / 2; i += blockDim.x) {
        float sn, c;
        sincosf((float)pos * p.inv_freq[i], &sn, &c);
        smem[2 * i] = c * p.amplitude;
        smem[2 * i + 1] = sn * p.amplitude;
    }
    __syncthreads();
    const int block = block_s;
    if (block >= p.max_blocks) return;    // (never: the host makes room for every sequence's last block)
    const int d8 = p.D / 8, dim8 = p.dim / 8, rot8 = p.rot / 8, dv8 = p.dv / 8;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    const uint4* q = reinterpret_cast<const uint4*>(p.q + (size_t)t * p.ldq);
    const uint4* kv = reinterpret_cast<const uint4*>(p.kv + (size_t)t * p.ld_kv);
    const uint4* sh = reinterpret_cast<const uint4*>(p.shared + (size_t)t * p.ld_shared);
    uint4* qo = reinterpret_cast<uint4*>(p.q_out) + (size_t)t * p.heads * d8;
    const size_t row0 = (size_t)block * p.heads * BLOCK_TOKENS + place % BLOCK_TOKENS;
    for (int i = threadIdx.x; i < p.heads * d8; i += blockDim.x) {
        const int h = i / d8, c = i - h * d8;
        uint4 k = zero, v = zero;
        if (c < dim8) {
            v = q[h * (dim8 + rot8) + c];
            k = kv[h * dim8 + c];
        } else if (c < dim8 + rot8) {
            v = q[h * (dim8 + rot8) + c];
            k = sh[c - dim8];
            __nv_bfloat162* pair = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int at = (c - dim8) * 4 + j;
                if (2 * at >= p.rot_dims) continue;
                const float a = __low2float(pair[j]), b = __high2float(pair[j]), cs = smem[2 * at], sn = smem[2 * at + 1];
                pair[j] = __floats2bfloat162_rn(a * cs - b * sn, b * cs + a * sn);
            }
        }
        qo[i] = v;
        reinterpret_cast<uint4*>(p.k_out)[(row0 + (size_t)h * BLOCK_TOKENS) * d8 + c] = k;
    }
    for (int i = threadIdx.x; i < p.heads * dv8; i += blockDim.x) {
        const int h = i / dv8, c = i - h * dv8;
        reinterpret_cast<uint4*>(p.v_out)[(row0 + (size_t)h * BLOCK_TOKENS) * dv8 + c] = kv[p.heads * dim8 + i];
    }
}

// A few tokens' queries (a decode step) into the compressed space, and their rotation:
//   q_out[t, h, n] = sum_k uk_t[h, n, k] * q[t, h, k] for n < rank, k < dim;   q_out[t, h, rank ..] = the head's rotated part, turned
// One launch, 16 tokens a block.  L lanes hold a weight row of `dim` entries, 16 bytes each, and take every token's entries past it; the weights are
// asked for before the kernel in front is waited for.  A head's last block does its rotation.
constexpr int ABSORB_THREADS = 256, ABSORB_COLS = 2, ABSORB_TOKENS = 16, ABSORB_MAX_TOKENS = 128;   // of a block; of a launch

struct LatentAbsorbParams {
    const void* q;       // [T, ldq]: head h's dim + rot entries at column h * (dim + rot)
    const void* uk_t;    // [heads, rank, dim]
    void* q_out;         // [T, heads * (rank + rot)]
    const int* token_pos;
    const float* inv_freq;
    long ldq;
    int tokens, heads, dim, rot, rank, rot_dims;
    float amplitude;
};

template <typename T, int L>
__global__ void __launch_bounds__(ABSORB_THREADS)
latent_absorb_kernel(LatentAbsorbParams p) {
    constexpr int V = 16 / sizeof(T), GROUPS = ABSORB_THREADS / L;
    const int h = blockIdx.y, dl = p.rank + p.rot;
    const T* q = (const T*)p.q + (size_t)h * (p.dim + p.rot);
    T* out = (T*)p.q_out + (size_t)h * dl;
    const size_t out_ld = (size_t)p.heads * dl;
    const int t0 = blockIdx.z * ABSORB_TOKENS, t1 = min(p.tokens, t0 + ABSORB_TOKENS);
    if (blockIdx.x == gridDim.x - 1) {
        pdl_wait();
        pdl_launch_dependents();
        const int half = p.rot_dims / 2, per = half + (p.rot - p.rot_dims);
        for (int item = threadIdx.x; item < (t1 - t0) * per; item += blockDim.x) {
            const int t = t0 + item / per, i = item % per;
            const T* src = q + (size_t)t * p.ldq + p.dim;
            T* dst = out + (size_t)t * out_ld + p.rank;
            if (i < half) {
                float sn, c;
                sincosf((float)p.token_pos[t] * p.inv_freq[i], &sn, &c);
                c *= p.amplitude;
                sn *= p.amplitude;
                const float a = to_float(src[2 * i]), b = to_float(src[2 * i + 1]);
                dst[2 * i] = from_float<T>(a * c - b * sn);
                dst[2 * i + 1] = from_float<T>(b * c + a * sn);
            } else {
                const int e = p.rot_dims + (i - half);
                dst[e] = src[e];
            }
        }
        return;
    }
    const int lane = threadIdx.x % L, group = threadIdx.x / L, k = lane * V;
    const bool k_ok = k < p.dim;
    int n[ABSORB_COLS];
    float wv[ABSORB_COLS][V];
#pragma unroll
    for (int c = 0; c < ABSORB_COLS; c++) {
        n[c] = (blockIdx.x * ABSORB_COLS + c) * GROUPS + group;
        uint4 raw = make_uint4(0, 0, 0, 0);
        if (k_ok && n[c] < p.rank) raw = __ldg(reinterpret_cast<const uint4*>((const T*)p.uk_t + ((size_t)h * p.rank + n[c]) * p.dim + k));
        const T* wt = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int i = 0; i < V; i++) wv[c][i] = to_float(wt[i]);
    }
    pdl_wait();
    pdl_launch_dependents();
#pragma unroll 4
    for (int t = t0; t < t1; t++) {
        uint4 raw = make_uint4(0, 0, 0, 0);
        if (k_ok) raw = *reinterpret_cast<const uint4*>(q + (size_t)t * p.ldq + k);
        const T* qt = reinterpret_cast<const T*>(&raw);
        float acc[ABSORB_COLS];
#pragma unroll
        for (int c = 0; c < ABSORB_COLS; c++) {
            acc[c] = 0.f;
#pragma unroll
            for (int i = 0; i < V; i++) acc[c] = fmaf(to_float(qt[i]), wv[c][i], acc[c]);
#pragma unroll
            for (int o = L / 2; o > 0; o >>= 1) acc[c] += __shfl_xor_sync(0xffffffffu, acc[c], o);
            if (lane == 0 && n[c] < p.rank) out[(size_t)t * out_ld + n[c]] = from_float<T>(acc[c]);
        }
    }
}

}  // namespace

HYMT2_API int hymt2_latent_prep(const void* proj, long ldp, int q_cols, void* q_out, void* rows_out, void* cache, int dtype,
                                const int* block_table, int table_stride, int block_tokens, const int* token_seq,
                                const int* token_pos, const int* slot_ids, const float* gain, const float* q_gain, void* cq_out, int q_rank,
                                const float* inv_freq,
                                int rot_dims, float amplitude, float eps, int tokens, int heads, int dim, int rot, int rank,
                                cudaStream_t stream) {
    if (tokens == 0) return HYMT2_OK;
    HYMT2_REQUIRE(tokens > 0 && heads >= 0 && dim >= 0 && rot >= 0 && rank > 0, "latent_prep: bad sizes");
    HYMT2_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= rot, "latent_prep: %d rotated entries of %d", rot_dims, rot);
    HYMT2_REQUIRE(rot_dims == 0 || inv_freq != nullptr, "latent_prep: no frequencies");
    HYMT2_REQUIRE(!cq_out || (q_gain && q_rank > 0 && q_rank <= q_cols && heads == 0), "latent_prep: a compressed query of %d entries", q_rank);
    LatentPrepParams p;
    p.q_gain = q_gain; p.cq_out = cq_out; p.q_rank = q_rank;
    p.proj = proj; p.q_out = q_out; p.rows_out = rows_out; p.cache = cache; p.block_table = block_table; p.token_seq = token_seq;
    p.token_pos = token_pos; p.slot_ids = slot_ids; p.gain = gain; p.inv_freq = inv_freq; p.ldp = ldp; p.q_cols = q_cols;
    p.table_stride = table_stride; p.block_tokens = block_tokens; p.heads = heads; p.dim = dim; p.rot = rot; p.rank = rank;
    p.rot_dims = rot_dims; p.eps = eps; p.amplitude = amplitude;
    const size_t smem = sizeof(float) * ((size_t)rot_dims + 33);
    const int threads = tokens <= 64 ? 512 : 128;   // (few tokens: the time is one block's chain of passes)
    HYMT2_DISPATCH_DTYPE(dtype, T, launch_pdl(latent_prep_kernel<T>, dim3(tokens), dim3(threads), smem, stream, p));
    return hymt2_check_launch("latent_prep");
}

// See latent_place_kernel; k_out holds max_blocks * heads * 64 rows of D entries, v_out as many of dv, table a row per cache slot.
HYMT2_API int hymt2_latent_place(const void* q, long ldq, const void* kv, long ld_kv, const void* shared, long ld_shared, void* q_out, void* k_out,
                                 void* v_out, int* table, int table_stride, int max_blocks, const int* token_seq, const int* token_pos,
                                 const int* cu_seqlens, const int* slot_ids, const float* inv_freq, int rot_dims, float amplitude, int tokens,
                                 int heads, int dim, int rot, int dv, int D, cudaStream_t stream) {
    if (tokens == 0) return HYMT2_OK;
    HYMT2_REQUIRE(tokens > 0 && heads > 0 && dim > 0 && rot >= 0 && dv > 0 && dim + rot <= D && max_blocks > 0, "latent_place: bad sizes");
    HYMT2_REQUIRE(dim % 8 == 0 && rot % 8 == 0 && dv % 8 == 0 && D % 8 == 0 && ldq % 8 == 0 && ld_kv % 8 == 0 && ld_shared % 8 == 0, "latent_place: rows come in pieces of 8 entries");
    HYMT2_REQUIRE(((uintptr_t)q | (uintptr_t)kv | (uintptr_t)shared | (uintptr_t)q_out | (uintptr_t)k_out | (uintptr_t)v_out) % 16 == 0, "latent_place: matrices must be 16-byte aligned");
    HYMT2_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= rot && (rot_dims == 0 || inv_freq), "latent_place: %d rotated entries of %d", rot_dims, rot);
    LatentPlaceParams p;
    p.q = (const __nv_bfloat16*)q; p.kv = (const __nv_bfloat16*)kv; p.shared = (const __nv_bfloat16*)shared;
    p.ldq = ldq; p.ld_kv = ld_kv; p.ld_shared = ld_shared;
    p.q_out = (__nv_bfloat16*)q_out; p.k_out = (__nv_bfloat16*)k_out; p.v_out = (__nv_bfloat16*)v_out; p.table = table;
    p.token_seq = token_seq; p.token_pos = token_pos; p.cu_seqlens = cu_seqlens; p.slot_ids = slot_ids; p.inv_freq = inv_freq;
    p.table_stride = table_stride; p.heads = heads; p.dim = dim; p.rot = rot; p.dv = dv; p.D = D; p.rot_dims = rot_dims; p.max_blocks = max_blocks;
    p.amplitude = amplitude;
    launch_pdl(latent_place_kernel, dim3(tokens), dim3(256), sizeof(float) * (size_t)rot_dims, stream, p);
    return hymt2_check_launch("latent_place");
}

// Whether latent_absorb takes heads of `dim` unrotated entries (they fill at most a warp's 16-byte pieces) for this many tokens.
HYMT2_API int hymt2_latent_absorb_supported(int dtype, int tokens, int dim, int rot) {
    const int v = dtype == HYMT2_BF16 ? 8 : 4;
    return tokens <= ABSORB_MAX_TOKENS && dim > 0 && dim <= 32 * v && dim % v == 0 && rot % v == 0;
}

HYMT2_API int hymt2_latent_absorb(void* q_out, const void* q, long ldq, const void* uk_t, int dtype, const int* token_pos, const float* inv_freq,
                                  int rot_dims, float amplitude, int tokens, int heads, int dim, int rot, int rank, cudaStream_t stream) {
    if (tokens == 0) return HYMT2_OK;
    HYMT2_REQUIRE(hymt2_latent_absorb_supported(dtype, tokens, dim, rot) && heads > 0 && heads <= 65535 && rank > 0, "latent_absorb: %d tokens with heads of %d + %d entries are not taken", tokens, dim, rot);
    HYMT2_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= rot && (rot_dims == 0 || inv_freq), "latent_absorb: %d rotated entries of %d", rot_dims, rot);
    HYMT2_DISPATCH_DTYPE(dtype, T, {
        constexpr int v = 16 / sizeof(T);
        HYMT2_REQUIRE(ldq % v == 0 && ((uintptr_t)q | (uintptr_t)uk_t) % 16 == 0, "latent_absorb: operands must be 16-byte aligned");
        LatentAbsorbParams p{q, uk_t, q_out, token_pos, inv_freq, ldq, tokens, heads, dim, rot, rank, rot_dims, amplitude};
        auto run = [&](auto kernel, int lanes) {
            const int cols = ABSORB_THREADS / lanes * ABSORB_COLS;
            launch_pdl(kernel, dim3((rank + cols - 1) / cols + 1, heads, (tokens + ABSORB_TOKENS - 1) / ABSORB_TOKENS), dim3(ABSORB_THREADS), 0, stream, p);
        };
        if (dim <= 4 * v) run(latent_absorb_kernel<T, 4>, 4);
        else if (dim <= 8 * v) run(latent_absorb_kernel<T, 8>, 8);
        else if (dim <= 16 * v) run(latent_absorb_kernel<T, 16>, 16);
        else run(latent_absorb_kernel<T, 32>, 32);
    });
    return hymt2_check_launch("latent_absorb");
}
