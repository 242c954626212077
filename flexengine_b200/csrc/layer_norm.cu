// The layer norm of a stream that is settled in the same pass:
//   y' = scale (w_b (y + bias - mean) / sqrt(var + eps) + b_b)     the branch before, through a norm of its own (or y as it is)
//   x += y' (+ plus);   out = w (x - mean) / sqrt(var + eps) + b
// Variances are means of squared deviations (two passes over the row, which stays in registers); all arithmetic is float.
#define FE_PDL_CLASS 4
#include "common.cuh"

using namespace fe;

namespace {

template <typename T, int V> struct Piece;        // V (1 or 4) consecutive elements as floats
template <typename T> struct Piece<T, 1> {
    static __device__ __forceinline__ void load(const T* p, float* v) { v[0] = to_float(p[0]); }
    static __device__ __forceinline__ void store(T* p, const float* v) { p[0] = from_float<T>(v[0]); }
};
template <> struct Piece<float, 4> {
    static __device__ __forceinline__ void load(const float* p, float* v) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    }
    static __device__ __forceinline__ void store(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct Piece<bf16, 4> {
    static __device__ __forceinline__ void load(const bf16* p, float* v) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        v[0] = __uint_as_float(raw.x << 16); v[1] = __uint_as_float(raw.x & 0xffff0000u);
        v[2] = __uint_as_float(raw.y << 16); v[3] = __uint_as_float(raw.y & 0xffff0000u);
    }
    static __device__ __forceinline__ void store(bf16* p, const float* v) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<const unsigned*>(&a);
        raw.y = *reinterpret_cast<const unsigned*>(&b);
        *reinterpret_cast<uint2*>(p) = raw;
    }
};

// Sum over the block with one barrier: ``part`` (32 floats) is used by this call alone.
__device__ __forceinline__ float block_sum_once(float v, float* part) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    if (warps == 1) return v;
    if (lane == 0) part[warp] = v;
    __syncthreads();
    return warp_sum(lane < warps ? part[lane] : 0.f);
}

// mean and 1 / sqrt(variance + eps) of the row that the block's threads hold
template <int V, int N>
__device__ __forceinline__ void statistics(const float (&row)[N][V], int H, float eps, float (*part)[32], float& mean, float& inv) {
    float s = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
        for (int e = 0; e < V; ++e) s += row[n][e];              // entries beyond the row are zeros
    mean = block_sum_once(s, part[0]) / (float)H;
    float q = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n) {
        if ((n * (int)blockDim.x + (int)threadIdx.x) * V >= H) continue;
#pragma unroll
        for (int e = 0; e < V; ++e) {
            const float d = row[n][e] - mean;
            q = fmaf(d, d, q);
        }
    }
    inv = rsqrtf(block_sum_once(q, part[1]) / (float)H + eps);
}

}  // namespace

// One block per output row.  V = 4: H is a multiple of 4 and every row starts on a 16-byte boundary (8 for bfloat16 rows).
// A thread holds N pieces of V entries; block N V >= H.
template <typename T, typename TD, int V, int N>
__global__ void layer_norm_kernel(float* __restrict__ residual, const TD* __restrict__ delta, const float* __restrict__ y_bias,
                                  const float* __restrict__ post_w, const float* __restrict__ post_b, float post_eps, float post_scale,
                                  const float* __restrict__ plus, const float* __restrict__ w, const float* __restrict__ b, float eps,
                                  T* __restrict__ out, const int* __restrict__ rows, int H, int T_tokens) {
    griddep_wait();
    griddep_launch_dependents();
    __shared__ float part[4][32];
    const int r = rows ? rows[blockIdx.x] : blockIdx.x;
    if (r < 0 || r >= T_tokens) return;
    float* x = residual + (size_t)r * H;
    float xs[N][V], ys[N][V];
    // everything the row needs is asked for before any of it is used
#pragma unroll
    for (int n = 0; n < N; ++n) {
        const int j = (n * blockDim.x + threadIdx.x) * V;
        const bool in = j < H;
#pragma unroll
        for (int e = 0; e < V; ++e) xs[n][e] = ys[n][e] = 0.f;
        if (in) Piece<float, V>::load(x + j, xs[n]);
        if (in && delta) Piece<TD, V>::load(delta + (size_t)r * H + j, ys[n]);
    }
    if (delta && y_bias) {
#pragma unroll
        for (int n = 0; n < N; ++n) {
            const int j = (n * blockDim.x + threadIdx.x) * V;
            if (j >= H) continue;
#pragma unroll
            for (int e = 0; e < V; ++e) ys[n][e] += y_bias[j + e];
        }
    }
    float mean, inv;
    if (delta && post_w) {
        statistics<V, N>(ys, H, post_eps, part, mean, inv);
#pragma unroll
        for (int n = 0; n < N; ++n) {
            const int j = (n * blockDim.x + threadIdx.x) * V;
            if (j >= H) continue;
            float pw[V], pb[V];
            Piece<float, V>::load(post_w + j, pw);
            Piece<float, V>::load(post_b + j, pb);
#pragma unroll
            for (int e = 0; e < V; ++e) ys[n][e] = fmaf((ys[n][e] - mean) * inv, pw[e], pb[e]);
        }
    }
    if (delta || plus) {
#pragma unroll
        for (int n = 0; n < N; ++n) {
            const int j = (n * blockDim.x + threadIdx.x) * V;
            if (j >= H) continue;
#pragma unroll
            for (int e = 0; e < V; ++e) xs[n][e] = fmaf(post_scale, ys[n][e], xs[n][e]);
            if (plus) {
                float p[V];
                Piece<float, V>::load(plus + (size_t)r * H + j, p);
#pragma unroll
                for (int e = 0; e < V; ++e) xs[n][e] += p[e];
            }
            if (!rows) Piece<float, V>::store(x + j, xs[n]);
        }
    }
    statistics<V, N>(xs, H, eps, part + 2, mean, inv);
    T* o = out + (size_t)blockIdx.x * H;
#pragma unroll
    for (int n = 0; n < N; ++n) {
        const int j = (n * blockDim.x + threadIdx.x) * V;
        if (j >= H) continue;
        float wv[V], bv[V], v[V];
        Piece<float, V>::load(w + j, wv);
        Piece<float, V>::load(b + j, bv);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = fmaf((xs[n][e] - mean) * inv, wv[e], bv[e]);
        Piece<T, V>::store(o + j, v);
    }
}

template <typename T, typename TD>
static int launch_layer_norm(float* residual, const void* delta, const float* y_bias, const float* post_w, const float* post_b,
                             float post_eps, float post_scale, const float* plus, const float* w, const float* b, float eps, void* out,
                             const int* rows, int n_out, int H, int T_tokens, cudaStream_t stream) {
    const bool vec = H % 4 == 0 && (((size_t)residual | (size_t)delta | (size_t)out | (size_t)post_w | (size_t)post_b | (size_t)plus |
                                     (size_t)w | (size_t)b) & 15) == 0;
    const int pieces = vec ? H / 4 : H;
    // one or two pieces a thread: short rows in few warps, long rows in many
    int per = pieces <= 512 ? 1 : (pieces <= 1024 ? 2 : (pieces <= 2048 ? 4 : 8));
    int threads = (pieces + per - 1) / per;
    threads = (threads + 31) / 32 * 32;
    FE_REQUIRE(threads <= 1024, "layer_norm: rows of %d columns (up to %d)", H, vec ? 32768 : 8192);
#define FE_LAYER_NORM(V, N)                                                                                                            \
    fe::launch(layer_norm_kernel<T, TD, V, N>, n_out, threads, 0, stream, residual, (const TD*)delta, y_bias, post_w, post_b, post_eps, \
               post_scale, plus, w, b, eps, (T*)out, rows, H, T_tokens)
    if (vec) {
        if (per == 1) FE_LAYER_NORM(4, 1);
        else if (per == 2) FE_LAYER_NORM(4, 2);
        else if (per == 4) FE_LAYER_NORM(4, 4);
        else FE_LAYER_NORM(4, 8);
    } else {
        if (per == 1) FE_LAYER_NORM(1, 1);
        else if (per == 2) FE_LAYER_NORM(1, 2);
        else if (per == 4) FE_LAYER_NORM(1, 4);
        else FE_LAYER_NORM(1, 8);
    }
#undef FE_LAYER_NORM
    return fe_check_launch("layer_norm");
}

// delta (may be null) [T, H] in delta_dtype, y_bias (may be null) added to it; post_w, post_b (both or neither): the branch's own
// norm, its result times post_scale (post_scale multiplies a plain branch as well); plus (may be null) float [T, H]; rows (may be
// null): only these rows are read and nothing is written back to the stream.  out [n_out, H] in dtype.
extern "C" int fe_layer_norm(float* residual, const void* delta, int delta_dtype, const float* y_bias, const float* post_w,
                             const float* post_b, float post_eps, float post_scale, const float* plus, const float* w, const float* b,
                             float eps, void* out, const int* rows, int n_out, int H, int T, int dtype, cudaStream_t stream) {
    FE_REQUIRE(n_out >= 0 && H > 0 && T >= 0, "layer_norm: bad sizes (H %d)", H);
    FE_REQUIRE((dtype == FE_F32 || dtype == FE_BF16) && (delta_dtype == FE_F32 || delta_dtype == FE_BF16), "layer_norm: unknown dtype");
    FE_REQUIRE(!(dtype == FE_F32 && delta_dtype == FE_BF16), "layer_norm: a bfloat16 branch beside float rows");
    FE_REQUIRE((post_w == nullptr) == (post_b == nullptr) && w && b, "layer_norm: weights and biases come in pairs");
    if (n_out == 0) return 0;
    if (dtype == FE_F32)
        return launch_layer_norm<float, float>(residual, delta, y_bias, post_w, post_b, post_eps, post_scale, plus, w, b, eps, out, rows, n_out, H, T, stream);
    if (delta_dtype == FE_F32)
        return launch_layer_norm<bf16, float>(residual, delta, y_bias, post_w, post_b, post_eps, post_scale, plus, w, b, eps, out, rows, n_out, H, T, stream);
    return launch_layer_norm<bf16, bf16>(residual, delta, y_bias, post_w, post_b, post_eps, post_scale, plus, w, b, eps, out, rows, n_out, H, T, stream);
}
