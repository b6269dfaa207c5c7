// Decode-step attention over a cache of ONE vector per token that all heads share (the key of every head is the whole row of d
// entries, its value the first dv of them), bfloat16: the products on warp-level matrix instructions (m16n8k16, float32 sums), the
// keys streamed through a ring of stages.
//
// A block owns one sequence's token, up to 16 * RF heads and one chunk of `split_keys` keys (or all keys), which it walks in tiles
// of 64, one cache block each.  Per tile: warp w takes the scores of keys 8w .. 8w + 7 for all of the block's heads (Q and K
// fragments from shared memory); the rows' maxima meet through shared memory; P goes to shared memory in bfloat16; every
// warp adds P V for its own columns of the output, whose fragments it keeps in registers throughout.  All warps follow the same
// running maximum, so a row's sum is kept per warp and added up once, in warp order, at the end.
// The query at position p sees keys max(0, p - window + 1) .. p.  With split_keys > 0 unnormalised partials are left for the merge
// kernel of the CUDA-core attention (which brings a sink in); without, the sink is added here: one more term exp(sink_h) in the
// head's denominator.
#include "common.cuh"

int hymt2_attention_merge_launch(void* out, int dtype, const int* cu_seqlens, const int* slot_ids, const int* kv_lens,
                                 float* part_acc, float* part_ml, int tokens, int nh, int d, int window, int split_keys,
                                 int max_splits, cudaStream_t stream, int* status, const float* sink_scores);

namespace {

typedef __nv_bfloat16 bf16;
constexpr int KEYS = 64, WARPS = 8, THREADS = WARPS * 32, P_LD = KEYS + 8;

struct LatentDecodeParams {
    const bf16* q;        // [rows * nh, d]
    bf16* out;            // [rows * nh, dv]
    const bf16* cache;    // plane base, [block][64][d]
    const int* block_table;
    const int* slot_ids;
    const int* kv_lens;
    float* part_acc;      // [rows * nh, splits, dv]
    float* part_ml;       // [rows * nh, splits, 2]
    const float* sink;    // [nh] or null
    int table_stride, nh, d, dv, window, split_keys, max_splits, stages;
    int grid_splits;      // chunks that blocks are launched for: all, or with a window as many as it can touch
    float scale;
};

__device__ __forceinline__ uint32_t smem_at(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
// c += A (16 x 16, rows) * B (16 x 8, columns)
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 16 bytes from global to shared memory; `valid` false: zeros (the address only has to exist)
__device__ __forceinline__ void copy16(uint32_t smem, const void* gmem, bool valid) {
    const int bytes = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem), "l"(gmem), "r"(bytes) : "memory");
}

// bytes of shared memory of a block with `stages` key tiles
size_t smem_bytes(int rows, int d, int stages) {
    return (size_t)(rows + stages * KEYS) * (d + 8) * sizeof(bf16) + 2 * (size_t)rows * P_LD * sizeof(bf16) + 2 * (size_t)WARPS * rows * sizeof(float);
}

// PAIRS: 16-column pieces of the output that a warp takes at most (warp, warp + 8, ...)
template <int RF, int PAIRS>
__global__ void __launch_bounds__(THREADS)
latent_decode_kernel(LatentDecodeParams p) {
    extern __shared__ __align__(128) unsigned char smem_raw[];
    constexpr int ROWS = 16 * RF;
    const int d = p.d, dv = p.dv, ld = d + 8;
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);                     // [ROWS][ld]
    bf16* Ks = Qs + ROWS * ld;                                        // [stages][KEYS][ld]
    bf16* Ps = Ks + (size_t)p.stages * KEYS * ld;                     // [2][ROWS][P_LD]
    float* red = reinterpret_cast<float*>(Ps + 2 * ROWS * P_LD);      // [2][WARPS][ROWS]

    const int b = blockIdx.y / p.grid_splits, h0 = blockIdx.x * ROWS;
    const int slot = p.slot_ids[b];
    if (slot < 0) return;
    const int kv_len = p.kv_lens[b], pos = kv_len - 1;
    const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    int begin = lo, end = kv_len, split = 0;
    if (p.split_keys > 0) {
        split = lo / p.split_keys + blockIdx.y % p.grid_splits;
        if (split >= p.max_splits) return;
        begin = max(begin, split * p.split_keys);
        end = min(end, (split + 1) * p.split_keys);
    }
    if (begin >= end) return;      // (no key of this chunk is seen; the merge never asks for it)
    const int heads = min(ROWS, p.nh - h0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int* table = p.block_table + (size_t)slot * p.table_stride;
    const int tile0 = begin / KEYS, tiles = (end - 1) / KEYS - tile0 + 1;
    const size_t row0 = (size_t)b * p.nh + h0;

    // a thread's 16-byte pieces of a [rows][d] tile are THREADS * 8 entries apart: row and column move on by fixed steps
    const int step_r = (THREADS * 8) / d, step_c = THREADS * 8 - step_r * d, first_r = tid * 8 / d, first_c = tid * 8 - first_r * d;
    auto load_tile = [&](int i) {
        const int k0 = (tile0 + i) * KEYS;
        const int block = table[tile0 + i];
        const bf16* src = p.cache + (size_t)(block < 0 ? 0 : block) * KEYS * d;
        const int keys_here = block < 0 ? 0 : min(KEYS, kv_len - k0);      // rows past the sequence's end hold anything: they are zeroed
        bf16* dst = Ks + (size_t)(i % p.stages) * KEYS * ld;
        for (int r = first_r, c = first_c; r < KEYS;) {
            const bool ok = r < keys_here;
            copy16(smem_at(dst + r * ld + c), src + (ok ? (size_t)r * d + c : 0), ok);
            r += step_r; c += step_c;
            if (c >= d) { c -= d; r++; }
        }
    };
    for (int r = first_r, c = first_c; r < ROWS;) {
        const bool ok = r < heads;
        copy16(smem_at(Qs + r * ld + c), p.q + (row0 + (ok ? r : 0)) * d + c, ok);
        r += step_r; c += step_c;
        if (c >= d) { c -= d; r++; }
    }
    for (int i = 0; i < p.stages - 1; i++) {     // (a group a tile, empty ones included, so that counting groups counts tiles)
        if (i < tiles) load_tile(i);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }

    const int g = lane >> 2, t4 = lane & 3;      // the fragments' row and column pair of this lane
    float m[RF][2], l[RF][2], acc[RF][PAIRS][2][4];
#pragma unroll
    for (int f = 0; f < RF; f++) {
        m[f][0] = m[f][1] = -INFINITY;
        l[f][0] = l[f][1] = 0.f;
#pragma unroll
        for (int i = 0; i < PAIRS; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) acc[f][i][0][e] = acc[f][i][1][e] = 0.f;
    }
    const int pairs = dv >> 4;
    const uint32_t q_addr = smem_at(Qs + (lane & 15) * ld + (lane >> 4) * 8);

    for (int i = 0; i < tiles; i++) {
        // tile i has landed (of the groups asked for, only the stages - 2 behind it may be open), and every warp is through with
        // tile i - 1, whose stage the tile stages - 1 ahead takes
        if (p.stages == 2) asm volatile("cp.async.wait_group 0;" ::: "memory");
        else if (p.stages == 3) asm volatile("cp.async.wait_group 1;" ::: "memory");
        else asm volatile("cp.async.wait_group 2;" ::: "memory");
        __syncthreads();
        if (i + p.stages - 1 < tiles) load_tile(i + p.stages - 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        const bf16* K = Ks + (size_t)(i % p.stages) * KEYS * ld;

        // scores of this warp's eight keys
        float s[RF][4];
#pragma unroll
        for (int f = 0; f < RF; f++)
#pragma unroll
            for (int e = 0; e < 4; e++) s[f][e] = 0.f;
        const uint32_t k_addr = smem_at(K + (warp * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8);
#pragma unroll 4
        for (int kk = 0; kk < d; kk += 16) {
            uint32_t b0, b1;
            ldsm2(k_addr + kk * 2, b0, b1);
#pragma unroll
            for (int f = 0; f < RF; f++) {
                uint32_t a[4];
                ldsm4(q_addr + (f * 16 * ld + kk) * 2, a);
                mma_bf16(s[f], a, b0, b1);
            }
        }
        const int key = (tile0 + i) * KEYS + warp * 8 + 2 * t4;
        const bool see0 = key >= begin && key < end, see1 = key + 1 >= begin && key + 1 < end;
        float* red_i = red + (i & 1) * WARPS * ROWS;
        float top[RF][2];
#pragma unroll
        for (int f = 0; f < RF; f++) {
#pragma unroll
            for (int e = 0; e < 4; e++) s[f][e] = ((e & 1) ? see1 : see0) ? s[f][e] * p.scale : -INFINITY;
#pragma unroll
            for (int x = 0; x < 2; x++) {
                float v = fmaxf(s[f][2 * x], s[f][2 * x + 1]);
                v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
                v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
                if (t4 == 0) red_i[warp * ROWS + f * 16 + x * 8 + g] = v;
            }
        }
        __syncthreads();
        bf16* P = Ps + (i & 1) * ROWS * P_LD;
#pragma unroll
        for (int f = 0; f < RF; f++)
#pragma unroll
            for (int x = 0; x < 2; x++) {
                float v = m[f][x];
#pragma unroll
                for (int w = 0; w < WARPS; w++) v = fmaxf(v, red_i[w * ROWS + f * 16 + x * 8 + g]);
                // (a tile holds at least one key that the token sees, so v is finite from the first tile on)
                const float corr = expf(m[f][x] - v), p0 = expf(s[f][2 * x] - v), p1 = expf(s[f][2 * x + 1] - v);
                m[f][x] = v;
                top[f][x] = corr;
                l[f][x] = l[f][x] * corr + (p0 + p1);
                *reinterpret_cast<__nv_bfloat162*>(P + (f * 16 + x * 8 + g) * P_LD + warp * 8 + 2 * t4) = __floats2bfloat162_rn(p0, p1);
            }
        __syncthreads();

        // O = O * corr + P V: this warp's columns
#pragma unroll
        for (int f = 0; f < RF; f++)
#pragma unroll
            for (int j = 0; j < PAIRS; j++)
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int e = 0; e < 4; e++) acc[f][j][n][e] *= top[f][e >> 1];
        const uint32_t p_addr = smem_at(P + (lane & 15) * P_LD + (lane >> 4) * 8);
        const uint32_t v_addr = smem_at(K + (lane & 15) * ld + (lane >> 4) * 8);
#pragma unroll
        for (int kk = 0; kk < KEYS; kk += 16) {
            uint32_t a[RF][4];
#pragma unroll
            for (int f = 0; f < RF; f++) ldsm4(p_addr + (f * 16 * P_LD + kk) * 2, a[f]);
#pragma unroll
            for (int j = 0; j < PAIRS; j++) {
                const int pair = warp + j * WARPS;
                if (pair < pairs) {
                    uint32_t v[4];
                    ldsm4_trans(v_addr + (kk * ld + pair * 16) * 2, v);
#pragma unroll
                    for (int f = 0; f < RF; f++) {
                        mma_bf16(acc[f][j][0], a[f], v[0], v[1]);
                        mma_bf16(acc[f][j][1], a[f], v[2], v[3]);
                    }
                }
            }
        }
    }

    // the rows' sums: over the lanes of a row, then over the warps in their order
    float* red_end = red + (tiles & 1) * WARPS * ROWS;
#pragma unroll
    for (int f = 0; f < RF; f++)
#pragma unroll
        for (int x = 0; x < 2; x++) {
            float v = l[f][x];
            v += __shfl_xor_sync(0xffffffffu, v, 1);
            v += __shfl_xor_sync(0xffffffffu, v, 2);
            if (t4 == 0) red_end[warp * ROWS + f * 16 + x * 8 + g] = v;
        }
    __syncthreads();
    const bool partial = p.split_keys > 0;
#pragma unroll
    for (int f = 0; f < RF; f++)
#pragma unroll
        for (int x = 0; x < 2; x++) {
            const int r = f * 16 + x * 8 + g;
            if (r >= heads) continue;
            float sum = 0.f;
#pragma unroll
            for (int w = 0; w < WARPS; w++) sum += red_end[w * ROWS + r];
            float factor = 1.f;
            if (partial) {
                if (warp == 0 && t4 == 0) {
                    float* ml = p.part_ml + ((row0 + r) * p.max_splits + split) * 2;
                    ml[0] = m[f][x];
                    ml[1] = sum;
                }
            } else {
                float up = 1.f;
                if (p.sink) {
                    const float z = p.sink[h0 + r], M = fmaxf(m[f][x], z);
                    up = expf(m[f][x] - M);
                    sum = sum * up + expf(z - M);
                }
                factor = up / sum;
            }
#pragma unroll
            for (int j = 0; j < PAIRS; j++) {
                const int pair = warp + j * WARPS;
                if (pair >= pairs) continue;
#pragma unroll
                for (int n = 0; n < 2; n++) {
                    const int col = pair * 16 + n * 8 + 2 * t4;
                    const float a = acc[f][j][n][2 * x] * factor, c = acc[f][j][n][2 * x + 1] * factor;
                    if (partial) *reinterpret_cast<float2*>(p.part_acc + ((row0 + r) * p.max_splits + split) * dv + col) = make_float2(a, c);
                    else *reinterpret_cast<__nv_bfloat162*>(p.out + (row0 + r) * dv + col) = __floats2bfloat162_rn(a, c);
                }
            }
        }
}

constexpr size_t SMEM_LIMIT = 220 * 1024;

}  // namespace

// Whether the kernel takes these sizes: rows in pieces of 16 entries, cache blocks of 64 tokens, room for two tiles.
HYMT2_API int hymt2_latent_decode_supported(int d, int dv, int block_tokens) {
    return d > 0 && dv > 0 && d % 16 == 0 && dv % 16 == 0 && dv <= d && dv <= 512 && block_tokens == KEYS && smem_bytes(32, d, 2) <= SMEM_LIMIT;
}

// A decode step: row b of the batch brings one token, q [rows, nh * d], out [rows, nh * dv].
HYMT2_API int hymt2_latent_decode(void* out, const void* q, const void* cache, const int* block_table, int table_stride, int block_tokens,
                                  const int* cu_seqlens, const int* slot_ids, const int* kv_lens, int rows, int nh, int d, int dv, float scale,
                                  int window, const float* sink, int split_keys, int max_splits, float* part_acc, float* part_ml, int* status,
                                  cudaStream_t stream) {
    if (rows == 0) return HYMT2_OK;
    HYMT2_REQUIRE(hymt2_latent_decode_supported(d, dv, block_tokens), "latent_decode: keys of %d, values of %d, blocks of %d are not taken", d, dv, block_tokens);
    HYMT2_REQUIRE(rows > 0 && nh > 0, "latent_decode: bad sizes");
    HYMT2_REQUIRE(((uintptr_t)q | (uintptr_t)out | (uintptr_t)cache) % 16 == 0, "latent_decode: operands must be 16-byte aligned");
    HYMT2_REQUIRE(split_keys == 0 || (split_keys % KEYS == 0 && max_splits > 0 && part_acc && part_ml), "latent_decode: a split comes in whole tiles and with scratch");
    LatentDecodeParams p;
    p.q = (const bf16*)q; p.out = (bf16*)out; p.cache = (const bf16*)cache; p.block_table = block_table; p.slot_ids = slot_ids; p.kv_lens = kv_lens;
    p.part_acc = part_acc; p.part_ml = part_ml; p.sink = sink; p.table_stride = table_stride; p.nh = nh; p.d = d; p.dv = dv; p.window = window;
    p.split_keys = split_keys; p.max_splits = split_keys > 0 ? max_splits : 1; p.scale = scale;
    p.grid_splits = p.max_splits;
    if (split_keys > 0 && window > 0 && (window - 1) / split_keys + 2 < p.grid_splits) p.grid_splits = (window - 1) / split_keys + 2;
    HYMT2_REQUIRE((long)rows * p.grid_splits <= 65535, "latent_decode: grid too large (%d rows x %d splits)", rows, p.max_splits);
    const int block_rows = nh <= 16 ? 16 : 32;
    p.stages = 2;
    // as many stages as leave room for a second block beside this one; else as many as fit
    while (p.stages < 4 && (smem_bytes(block_rows, d, p.stages + 1) <= SMEM_LIMIT / 2 || (smem_bytes(block_rows, d, p.stages) > SMEM_LIMIT / 2 &&
           smem_bytes(block_rows, d, p.stages + 1) <= SMEM_LIMIT))) p.stages++;
    const size_t smem = smem_bytes(block_rows, d, p.stages);
    const dim3 grid((nh + block_rows - 1) / block_rows, rows * p.grid_splits);
    auto launch = [&](auto kernel) -> int {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) { hymt2_set_error("latent_decode: %s", cudaGetErrorString(e)); return HYMT2_ERR_LAUNCH; }
        kernel<<<grid, THREADS, smem, stream>>>(p);
        return hymt2_check_launch("latent_decode");
    };
    int rc;
    if (block_rows == 16) rc = dv <= 128 ? launch(latent_decode_kernel<1, 1>) : dv <= 256 ? launch(latent_decode_kernel<1, 2>) : launch(latent_decode_kernel<1, 4>);
    else rc = dv <= 128 ? launch(latent_decode_kernel<2, 1>) : dv <= 256 ? launch(latent_decode_kernel<2, 2>) : launch(latent_decode_kernel<2, 4>);
    if (rc == HYMT2_OK && split_keys > 0)
        rc = hymt2_attention_merge_launch(out, HYMT2_BF16, cu_seqlens, slot_ids, kv_lens, part_acc, part_ml, rows, nh, dv, window, split_keys,
                                          max_splits, stream, status, sink);
    return rc;
}
