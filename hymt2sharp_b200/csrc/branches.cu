// The end of a block whose sublayers read the same rows: their outputs join the residual together, each multiplied entry by
// entry by a stored vector where it has one, and the norm that reads the residual next is computed on the way.  One block of
// threads a token:
//
//     v = x + sum_b gain_b * (y_b + bias_b)                            (up to MAX_BRANCHES plain branches; gain and bias may be absent)
//           + gain_r * (sum_k weight[k] * routed[pair_row[k]] + sigmoid(z) * shared)      (a mixture's pieces, if there is one)
//     x <- v;   h = v / sqrt(mean(v^2) + eps) * norm_gain              (if the next reader's norm is known)
//
// All arithmetic is float32 and every sum has a fixed order.  The mixture is added up here, from the experts' rows of the
// grouped product, so that no buffer of its own is written and read for it.
#include "common.cuh"

namespace {

constexpr int MAX_BRANCHES = 3, MAX_TOP = 32;

struct JoinParams {
    float* x;                        // [T, width]
    const float* y[MAX_BRANCHES];    // [T, width]
    const float* gain[MAX_BRANCHES]; // [width] or null
    const float* bias[MAX_BRANCHES]; // [width] or null
    int branches, width;
    const float* routed;             // sorted rows [rows, width], or null
    const int* pair_row;             // [T, top]
    const float* weight;             // [T, top]
    const float* routed_gain;        // [width] or null
    int top;
    const float* shared;             // [T, width] or null
    const float* z;                  // the shared branch's gate in front of its sigmoid, one a token (row stride ldz), or null: 1
    long ldz;
    void* h;                         // [T, width] or null
    const void* norm_gain;
    float eps;
};

// IT > 0: a thread's IT pieces of V entries stay in registers between the sum of squares and the scaling; IT 0: rows of any
// width, read again (a thread meets its own entries only)
template <typename TW, typename TH, int V, int IT>
__global__ void __launch_bounds__(256)
join_branches_kernel(JoinParams p) {
    __shared__ float scratch[33];
    __shared__ int row_s[MAX_TOP];
    __shared__ float weight_s[MAX_TOP];
    pdl_wait();
    pdl_launch_dependents();
    const size_t t = blockIdx.x;
    const int width = p.width;
    if (p.routed && threadIdx.x < p.top) {
        row_s[threadIdx.x] = p.pair_row[t * p.top + threadIdx.x];
        weight_s[threadIdx.x] = p.weight[t * p.top + threadIdx.x];
    }
    float share = 1.f;
    if (p.shared && p.z) share = 1.0f / (1.0f + expf(-p.z[t * p.ldz]));
    __syncthreads();
    float ss = 0.f;
    auto piece = [&](int c) {
        Pack<float, V> v = load_pack<float, V>(p.x + t * width + c);
        for (int b = 0; b < p.branches; b++) {
            Pack<float, V> y = load_pack<float, V>(p.y[b] + t * width + c);
            if (p.bias[b]) {
                const Pack<float, V> z = load_pack<float, V>(p.bias[b] + c);
#pragma unroll
                for (int k = 0; k < V; k++) y.v[k] += z.v[k];
            }
            if (p.gain[b]) {
                const Pack<float, V> g = load_pack<float, V>(p.gain[b] + c);
#pragma unroll
                for (int k = 0; k < V; k++) v.v[k] = fmaf(y.v[k], g.v[k], v.v[k]);
            } else {
#pragma unroll
                for (int k = 0; k < V; k++) v.v[k] += y.v[k];
            }
        }
        if (p.routed) {
            float m[V];
#pragma unroll
            for (int k = 0; k < V; k++) m[k] = 0.f;
#pragma unroll 4
            for (int e = 0; e < p.top; e++) {
                const Pack<float, V> y = load_pack<float, V>(p.routed + (size_t)row_s[e] * width + c);
#pragma unroll
                for (int k = 0; k < V; k++) m[k] = fmaf(weight_s[e], y.v[k], m[k]);
            }
            if (p.shared) {
                const Pack<float, V> y = load_pack<float, V>(p.shared + t * width + c);
#pragma unroll
                for (int k = 0; k < V; k++) m[k] = fmaf(share, y.v[k], m[k]);
            }
            if (p.routed_gain) {
                const Pack<float, V> g = load_pack<float, V>(p.routed_gain + c);
#pragma unroll
                for (int k = 0; k < V; k++) v.v[k] = fmaf(m[k], g.v[k], v.v[k]);
            } else {
#pragma unroll
                for (int k = 0; k < V; k++) v.v[k] += m[k];
            }
        }
        store_pack<float, V>(p.x + t * width + c, v);
#pragma unroll
        for (int k = 0; k < V; k++) ss = fmaf(v.v[k], v.v[k], ss);
        return v;
    };
    const TW* gain = (const TW*)p.norm_gain;
    TH* h = (TH*)p.h + t * width;
    auto scaled = [&](const Pack<float, V>& v, float scale, int c) {
        const Pack<TW, V> g = load_pack<TW, V>(gain + c);
        Pack<TH, V> o;
#pragma unroll
        for (int k = 0; k < V; k++) o.v[k] = from_float<TH>(v.v[k] * scale * to_float(g.v[k]));
        store_pack<TH, V>(h + c, o);
    };
    if constexpr (IT > 0) {
        Pack<float, V> v[IT];
#pragma unroll
        for (int i = 0; i < IT; i++) {
            const int c = (threadIdx.x + i * blockDim.x) * V;
            if (c < width) v[i] = piece(c);
        }
        if (!p.h) return;
        const float scale = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + p.eps);
#pragma unroll
        for (int i = 0; i < IT; i++) {
            const int c = (threadIdx.x + i * blockDim.x) * V;
            if (c < width) scaled(v[i], scale, c);
        }
    } else {
        for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) piece(c);
        if (!p.h) return;
        const float scale = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + p.eps);
        for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) scaled(load_pack<float, V>(p.x + t * width + c), scale, c);
    }
}

template <typename TW, typename TH>
void launch_join(const JoinParams& p, int tokens, bool vec, cudaStream_t stream) {
    if (vec) {
        const int pieces = p.width / 4;
        const int threads = pieces >= 256 ? 256 : (pieces + 31) / 32 * 32;
        const int it = (pieces + threads - 1) / threads;
        if (it <= 1) { launch_pdl(join_branches_kernel<TW, TH, 4, 1>, dim3(tokens), dim3(threads), 0, stream, p); return; }
        if (it <= 2) { launch_pdl(join_branches_kernel<TW, TH, 4, 2>, dim3(tokens), dim3(threads), 0, stream, p); return; }
        if (it <= 4) { launch_pdl(join_branches_kernel<TW, TH, 4, 4>, dim3(tokens), dim3(threads), 0, stream, p); return; }
        launch_pdl(join_branches_kernel<TW, TH, 4, 0>, dim3(tokens), dim3(threads), 0, stream, p);
        return;
    }
    const int threads = p.width >= 256 ? 256 : (p.width + 31) / 32 * 32;
    launch_pdl(join_branches_kernel<TW, TH, 1, 0>, dim3(tokens), dim3(threads), 0, stream, p);
}

}  // namespace

// `branches` plain branches: y, gain and bias are host arrays of that many device pointers (a gain or a bias may be null).
// `routed` null: no mixture; `h` null: no norm.  Gains and biases of branches are float32; the norm's gain has a type of its own.
HYMT2_API int hymt2_join_branches(float* x, const float* const* y, const float* const* gain, const float* const* bias, int branches,
                                  const float* routed, const int* pair_row, const float* weight, int top, const float* routed_gain,
                                  const float* shared, const float* z, long ldz, void* h, int h_dtype, const void* norm_gain,
                                  int norm_gain_dtype, float eps, int tokens, int width, cudaStream_t stream) {
    if (tokens == 0) return HYMT2_OK;
    HYMT2_REQUIRE(tokens > 0 && width > 0 && x, "join_branches: bad sizes");
    HYMT2_REQUIRE(branches >= 0 && branches <= MAX_BRANCHES, "join_branches: %d plain branches (at most %d)", branches, MAX_BRANCHES);
    HYMT2_REQUIRE(!routed || (pair_row && weight && top > 0 && top <= MAX_TOP), "join_branches: at most %d chosen experts are taken", MAX_TOP);
    HYMT2_REQUIRE(!shared || routed, "join_branches: a shared expert stands beside routed ones");
    HYMT2_REQUIRE(!h || norm_gain, "join_branches: a norm needs its gain");
    JoinParams p = {};
    p.x = x; p.branches = branches; p.width = width; p.routed = routed; p.pair_row = pair_row; p.weight = weight; p.routed_gain = routed_gain;
    p.top = top; p.shared = shared; p.z = z; p.ldz = ldz; p.h = h; p.norm_gain = norm_gain; p.eps = eps;
    uintptr_t bits = (uintptr_t)x | (uintptr_t)routed | (uintptr_t)routed_gain | (uintptr_t)shared | (uintptr_t)h | (uintptr_t)norm_gain;
    for (int b = 0; b < branches; b++) {
        HYMT2_REQUIRE(y[b], "join_branches: branch %d is missing", b);
        p.y[b] = y[b]; p.gain[b] = gain[b]; p.bias[b] = bias[b];
        bits |= (uintptr_t)y[b] | (uintptr_t)gain[b] | (uintptr_t)bias[b];
    }
    const bool vec = width % 4 == 0 && bits % 16 == 0;
    HYMT2_DISPATCH_DTYPE(norm_gain_dtype, TW, HYMT2_DISPATCH_DTYPE(h_dtype, TH, (launch_join<TW, TH>(p, tokens, vec, stream))));
    return hymt2_check_launch("join_branches");
}
