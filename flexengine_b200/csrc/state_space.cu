// What state-space layers do besides the scan of a head's matrix (head_scan.cu):
//   conv_silu            a causal convolution over time per channel (with a bias and a kept history) and silu; beside it the
//                        steps of the heads: dt = softplus(row + bias) and the decays' logarithms minus_a * dt
//   gated_group_rmsnorm  rows times silu(z), then every one of ``groups`` equal parts divided by its root mean square, times a weight
//   selective_scan       a recurrence with a decay per channel, state entry and token, token by token, the state in registers:
//                          S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n ;   y_c = sum_n S[c, n] C_n + D_c x_c
//                        with dt = softplus(row + bias); out = y silu(z) times a factor
//   selective_decode     the same for a step of one token a request, the step sizes' projection W_dt low in the same kernel
// Arithmetic is float throughout; rows come in float or bfloat16.
#define FE_PDL_CLASS 128
#include "common.cuh"

using namespace fe;

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }
// The same with the hardware's division (two units in the last place; a z so far down that the divisor overflows gives 0, as it should).
__device__ __forceinline__ float silu_near(float z) { return __fdividef(z, 1.f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <typename T, int V> __device__ __forceinline__ void load_v(const T* p, float* out);
template <> __device__ __forceinline__ void load_v<float, 1>(const float* p, float* out) { out[0] = *p; }
template <> __device__ __forceinline__ void load_v<bf16, 1>(const bf16* p, float* out) { out[0] = __bfloat162float(*p); }
template <> __device__ __forceinline__ void load_v<float, 4>(const float* p, float* out) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    out[0] = v.x, out[1] = v.y, out[2] = v.z, out[3] = v.w;
}
template <> __device__ __forceinline__ void load_v<bf16, 4>(const bf16* p, float* out) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    out[0] = __uint_as_float(raw.x << 16), out[1] = __uint_as_float(raw.x & 0xffff0000u);
    out[2] = __uint_as_float(raw.y << 16), out[3] = __uint_as_float(raw.y & 0xffff0000u);
}
template <typename T, int V> __device__ __forceinline__ void store_v(T* p, const float* v);
template <> __device__ __forceinline__ void store_v<float, 1>(float* p, const float* v) { *p = v[0]; }
template <> __device__ __forceinline__ void store_v<bf16, 1>(bf16* p, const float* v) { *p = __float2bfloat16_rn(v[0]); }
template <> __device__ __forceinline__ void store_v<float, 4>(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
template <> __device__ __forceinline__ void store_v<bf16, 4>(bf16* p, const float* v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned*>(&a), raw.y = *reinterpret_cast<const unsigned*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
}

// ---------------------------------------------------------------------------------------------
// Grid (tiles of CONV_TILE tokens, requests, stretches of channels [+ 1 for the steps]); a thread has V channels of the tile.  The
// blocks of a portion's first tile bring their channels' history up to date after their reads; nobody else touches it.
constexpr int CONV_TILE = 8;
constexpr int CONV_THREADS = 128;

struct Steps {
    const float* rows;           // [T, >= heads], rows ld entries long; null: no steps
    long long ld;
    const float* bias;           // [heads]
    const float* minus_a;        // [heads]
    float* gates;                // [2][plane]: minus_a dt, dt
    long long plane;
    int heads;
};

template <typename TI, typename TO, int TAPS, int V>
__global__ void __launch_bounds__(CONV_THREADS)
conv_silu_kernel(const TI* __restrict__ u, long long ld, const float* __restrict__ conv, const float* __restrict__ bias, int taps, float* state,
                 long long state_stride, long long history_at, const int* __restrict__ seats, const int* __restrict__ cu_q,
                 TO* __restrict__ out, int C, int n_seats, int stretches, Steps steps) {
    griddep_wait();
    griddep_launch_dependents();
    const int r = blockIdx.y;
    const int first = cu_q[r], n = cu_q[r + 1] - first;
    const int i0 = blockIdx.x * CONV_TILE;
    if (i0 >= n) return;
    if ((int)blockIdx.z >= stretches) {
        const int count = min(CONV_TILE, n - i0) * steps.heads;
        for (int e = threadIdx.x; e < count; e += CONV_THREADS) {
            const int t = first + i0 + e / steps.heads, h = e % steps.heads;
            const float dt = softplus(steps.rows[(size_t)t * steps.ld + h] + steps.bias[h]);
            const size_t at = (size_t)t * steps.heads + h;
            steps.gates[at] = steps.minus_a[h] * dt;
            steps.gates[steps.plane + at] = dt;
        }
        return;
    }
    const int ch = ((int)blockIdx.z * CONV_THREADS + threadIdx.x) * V;
    if (ch >= C) return;
    const int seat = seats[r];
    float* hist = (taps > 1 && seat >= 0 && seat < n_seats) ? state + (size_t)seat * state_stride + history_at + ch : nullptr;
    const TI* rows = u + (size_t)first * ld + ch;
    TO* to = out + (size_t)(first + i0) * C + ch;
    float b[V];
    load_v<float, V>(bias + ch, b);
    if (TAPS > 0) {
        constexpr int K = TAPS > 0 ? TAPS : 1;
        float x[K - 1 + CONV_TILE][V], w[K][V];
#pragma unroll
        for (int j = 0; j < K; ++j) load_v<float, V>(conv + (size_t)j * C + ch, w[j]);
#pragma unroll
        for (int y = 0; y < K - 1 + CONV_TILE; ++y) {           // every row asked for once and before any is used
            const int from = i0 - (K - 1) + y;
#pragma unroll
            for (int c = 0; c < V; ++c) x[y][c] = 0.f;
            if (from >= 0) {
                if (from < n) load_v<TI, V>(rows + (size_t)from * ld, x[y]);
            } else if (hist) load_v<float, V>(hist + (size_t)(K - 1 + from) * C, x[y]);
        }
#pragma unroll
        for (int y = 0; y < CONV_TILE; ++y) {
            if (i0 + y >= n) break;
            float acc[V];
#pragma unroll
            for (int c = 0; c < V; ++c) {
                acc[c] = b[c];
#pragma unroll
                for (int j = 0; j < K; ++j) acc[c] = fmaf(w[j][c], x[y + j][c], acc[c]);
                acc[c] = silu_near(acc[c]);
            }
            store_v<TO, V>(to + (size_t)y * C, acc);
        }
    } else {
        for (int y = 0; y < CONV_TILE && i0 + y < n; ++y) {
            float acc[V];
#pragma unroll
            for (int c = 0; c < V; ++c) acc[c] = b[c];
            for (int j = 0; j < taps; ++j) {
                const int from = i0 + y - (taps - 1 - j);
                float x[V] = {}, w[V];
                load_v<float, V>(conv + (size_t)j * C + ch, w);
                if (from >= 0) load_v<TI, V>(rows + (size_t)from * ld, x);
                else if (hist) load_v<float, V>(hist + (size_t)(taps - 1 + from) * C, x);
#pragma unroll
                for (int c = 0; c < V; ++c) acc[c] = fmaf(w[c], x[c], acc[c]);
            }
#pragma unroll
            for (int c = 0; c < V; ++c) acc[c] = silu_near(acc[c]);
            store_v<TO, V>(to + (size_t)y * C, acc);
        }
    }
    if (hist && i0 == 0) {
        // the last taps - 1 inputs, oldest first: what was kept moves up, the portion's rows follow
        const int back = taps - 1;
        for (int m = 0; m < back; ++m) {
            const int from = m + n;
            float x[V];
            if (from < back) load_v<float, V>(hist + (size_t)from * C, x);
            else load_v<TI, V>(rows + (size_t)(from - back) * ld, x);
            store_v<float, V>(hist + (size_t)m * C, x);
        }
    }
}

// ---------------------------------------------------------------------------------------------
// Block per (token, part).
template <typename T, int V>
__global__ void gated_group_rmsnorm_kernel(const float* __restrict__ y, const float* __restrict__ z, long long ldz, const float* __restrict__ weight,
                                           float eps, T* __restrict__ out, int inner, int width) {
    griddep_wait();
    griddep_launch_dependents();
    extern __shared__ __align__(16) float row[];
    __shared__ float scratch[33];
    const size_t t = blockIdx.x;
    const int first = blockIdx.y * width;
    const float* ys = y + t * inner + first;
    const float* zs = z + t * ldz + first;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float a[V], g[V];
        load_v<float, V>(ys + i, a);
        load_v<float, V>(zs + i, g);
#pragma unroll
        for (int c = 0; c < V; ++c) {
            a[c] *= silu(g[c]);
            ss = fmaf(a[c], a[c], ss);
        }
        store_v<float, V>(row + i, a);
    }
    const float inv = rsqrtf(block_sum(ss, scratch) / (float)width + eps);
    T* to = out + t * inner + first;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {      // a thread reads back what it wrote
        float a[V], w[V];
        load_v<float, V>(row + i, a);
        load_v<float, V>(weight + first + i, w);
#pragma unroll
        for (int c = 0; c < V; ++c) a[c] *= inv * w[c];
        store_v<T, V>(to + i, a);
    }
}

// ---------------------------------------------------------------------------------------------
// The selective scan.  LANES neighbouring lanes share a channel, each with NPT neighbouring entries of its state in registers
// (entries beyond N have B = C = 0 and stay zero); the true 32-bit path takes the decays from exp_decay, the other one
// with the hardware's 2^x; a block has 128 / LANES channels of one request and walks its tokens in tiles of TT staged in shared
// memory; the rows of the next tile are on their way (in registers, as they lie in memory) while one is walked.  Four tokens at a
// time share the rounds of the sum over the lanes.
// A long portion of few channels would leave most of the device idle: it is cut into segments that are walked side by side.  MODE
// WALK: a portion from its seat to its seat.  Else three launches: FOLD walks every segment from a state of zero, without outputs,
// and leaves the state it ends with and the sum of its step sizes (and, in place of the step sizes' rows, the step sizes);
// the chain makes of them the state before every segment, S <- exp(A sum) S + fold; OUT walks every segment from there.  Segment
// s of request r has row cu_q[r] / SEGMENT + r + s of ``folds`` and ``sums``.
constexpr int SCAN_THREADS = 128;
constexpr int SEGMENT = 128;
enum ScanMode { WALK, FOLD, OUT };

__device__ __forceinline__ size_t segment_row(const int* __restrict__ cu_q, int r) { return (size_t)(cu_q[r] / SEGMENT + r); }

struct SelectiveScan {
    float* dt;                  // [T, inner]: before bias and softplus; FOLD leaves the step sizes there
    const float* dt_bias;
    const float* minus_a;       // [inner, N]
    const float* skip;
    float* state;
    long long state_stride;
    const int* seats;
    const int* cu_q;
    float* folds;               // [rows][inner N]
    float* sums;                // [rows][inner]
    float scale;
    int inner, N, n_seats;
};

template <typename TX, ScanMode MODE, int LANES, int NPT, int TT>
__global__ void __launch_bounds__(SCAN_THREADS)
selective_scan_kernel(const TX* __restrict__ x, const TX* __restrict__ bc, long long ldbc, const TX* __restrict__ z, long long ldz,
                      TX* __restrict__ out, long long ldo, SelectiveScan sc) {
    griddep_wait();
    griddep_launch_dependents();
    constexpr bool EXACT = sizeof(TX) == 4;        // the true 32-bit path
    constexpr int CH = SCAN_THREADS / LANES, NP = LANES * NPT, KEYS = MODE == FOLD ? NP : 2 * NP;       // B, or B and C
    constexpr int PER_X = (TT * CH + SCAN_THREADS - 1) / SCAN_THREADS, PER_B = (TT * KEYS + SCAN_THREADS - 1) / SCAN_THREADS;
    extern __shared__ __align__(16) float smem[];
    float* dts = smem;                              // [TT][CH] step sizes
    float* dxs = dts + TT * CH;                     // [TT][CH] step size times input
    float* bs = dxs + TT * CH;                      // [TT][NP]
    float* cs = bs + TT * NP;                       // [TT][NP]
    float* xs = cs + TT * NP;                       // [TT][CH] inputs
    float* ys = xs + TT * CH;                       // [TT][CH]
    const int inner = sc.inner, N = sc.N;
    const int tid = threadIdx.x, r = blockIdx.y, c0 = blockIdx.x * CH;
    const int l = tid % LANES, cl = tid / LANES, ch = c0 + cl;
    const int first = sc.cu_q[r], last = sc.cu_q[r + 1];
    const int begin = MODE == WALK ? first : first + (int)blockIdx.z * SEGMENT;
    const int end = MODE == WALK ? last : min(last, begin + SEGMENT);
    if (begin >= end) return;
    const size_t seg_row = MODE == WALK ? 0 : segment_row(sc.cu_q, r) + blockIdx.z;
    const int seat = sc.seats[r];
    float* mine = (seat >= 0 && seat < sc.n_seats && ch < inner) ? sc.state + (size_t)seat * sc.state_stride + (size_t)ch * N : nullptr;
    float* fold = (MODE != WALK && ch < inner) ? sc.folds + seg_row * ((size_t)inner * N) + (size_t)ch * N : nullptr;
    const float* from = MODE == WALK ? mine : MODE == OUT ? fold : nullptr;
    float S[NPT], A[NPT];
#pragma unroll
    for (int e = 0; e < NPT; ++e) {
        const int i = l * NPT + e;
        S[e] = (from && i < N) ? from[i] : 0.f;
        A[e] = (ch < inner && i < N) ? sc.minus_a[(size_t)ch * N + i] * (EXACT ? 1.f : LOG2E) : 0.f;
    }
    // element e of a tile's [TT][CH] rows belongs to thread e % 128; a thread's channel is the same in all of them
    const int my_c = tid % CH, my_t = tid / CH;
    const bool in_c = c0 + my_c < inner;
    const float my_bias = in_c ? sc.dt_bias[c0 + my_c] : 0.f, my_skip = in_c ? sc.skip[c0 + my_c] : 0.f;
    TX px[PER_X], pz[PER_X], pb[PER_B];
    float pd[PER_X];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int i = 0; i < PER_X; ++i) {
            const int t = t0 + my_t + i * (SCAN_THREADS / CH);
            const bool in = in_c && my_t + i * (SCAN_THREADS / CH) < TT && t < end;
            px[i] = TX(0.f);
            pd[i] = 0.f;
            if (in) {
                px[i] = x[(size_t)t * inner + c0 + my_c];
                pd[i] = sc.dt[(size_t)t * inner + c0 + my_c];
            }
        }
#pragma unroll
        for (int i = 0; i < PER_B; ++i) {
            const int e = tid + i * SCAN_THREADS, tt = e / KEYS, n = e % KEYS, at = n % NP;
            pb[i] = TX(0.f);
            if (tt < TT && t0 + tt < end && at < N) pb[i] = bc[(size_t)(t0 + tt) * ldbc + (n < NP ? at : N + at)];
        }
    };
    float dt_sum = 0.f;
    fetch(begin);
    for (int t0 = begin; t0 < end; t0 += TT) {
        const int count = min(TT, end - t0);
#pragma unroll
        for (int i = 0; i < PER_X; ++i) {
            const int tt = my_t + i * (SCAN_THREADS / CH);
            if (tt >= TT) break;
            // tokens beyond the end have a step size of zero: the state stays as it is
            const bool in = in_c && tt < count;
            const float d = in ? (MODE == OUT ? pd[i] : softplus(pd[i] + my_bias)) : 0.f;
            const float xv = to_float(px[i]);
            dts[tt * CH + my_c] = d;
            dxs[tt * CH + my_c] = d * xv;
            if (MODE == FOLD) {
                if (in) sc.dt[(size_t)(t0 + tt) * inner + c0 + my_c] = d;
            } else {
                xs[tt * CH + my_c] = xv;
            }
        }
#pragma unroll
        for (int i = 0; i < PER_B; ++i) {
            const int e = tid + i * SCAN_THREADS, tt = e / KEYS, n = e % KEYS;
            if (tt < TT) (n < NP ? bs : cs)[tt * NP + n % NP] = to_float(pb[i]);
        }
        __syncthreads();
        // the gates of this tile and the rows of the next one
        if (MODE != FOLD) {
#pragma unroll
            for (int i = 0; i < PER_X; ++i) {
                const int tt = my_t + i * (SCAN_THREADS / CH);
                pz[i] = TX(0.f);
                if (in_c && tt < count) pz[i] = z[(size_t)(t0 + tt) * ldz + c0 + my_c];
            }
        }
        if (t0 + TT < end) fetch(t0 + TT);
#pragma unroll 1
        for (int tq = 0; tq < count; tq += 4) {
            float y4[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const int tt = tq + q;
                const float d = dts[tt * CH + cl], dx = dxs[tt * CH + cl];
                float y = 0.f;
#pragma unroll
                for (int e = 0; e < NPT; e += 4) {
                    const float4 b4 = *reinterpret_cast<const float4*>(bs + tt * NP + l * NPT + e);
                    const float bb[4] = {b4.x, b4.y, b4.z, b4.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) S[e + i] = fmaf(EXACT ? exp_decay(d * A[e + i]) : exp2f(d * A[e + i]), S[e + i], dx * bb[i]);
                    if (MODE != FOLD) {
                        const float4 q4 = *reinterpret_cast<const float4*>(cs + tt * NP + l * NPT + e);
                        const float qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                        for (int i = 0; i < 4; ++i) y = fmaf(S[e + i], qq[i], y);
                    }
                }
                y4[q] = y;
                if (MODE == FOLD) dt_sum += d;
            }
            if constexpr (MODE != FOLD) {
                // the sums over the lanes: two rounds in which a lane gives half of its tokens away, then plain rounds; the lane
                // ends with token (l & 1) * 2 + ((l >> 1) & 1)
                float y2[2];
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const float keep = l & 1 ? y4[2 + i] : y4[i], give = l & 1 ? y4[i] : y4[2 + i];
                    y2[i] = keep + __shfl_xor_sync(0xffffffffu, give, 1);
                }
                const float keep = l & 2 ? y2[1] : y2[0], give = l & 2 ? y2[0] : y2[1];
                float y = keep + __shfl_xor_sync(0xffffffffu, give, 2);
#pragma unroll
                for (int o = 4; o < LANES; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
                if (l < 4) ys[(tq + (l & 1) * 2 + ((l >> 1) & 1)) * CH + cl] = y;
            }
        }
        __syncthreads();
        if (MODE != FOLD) {
#pragma unroll
            for (int i = 0; i < PER_X; ++i) {
                const int tt = my_t + i * (SCAN_THREADS / CH);
                if (in_c && tt < count)
                    out[(size_t)(t0 + tt) * ldo + c0 + my_c] =
                        from_float<TX>(fmaf(my_skip, xs[tt * CH + my_c], ys[tt * CH + my_c]) * silu(to_float(pz[i])) * sc.scale);
            }
            __syncthreads();                        // everyone is done with this tile before it is filled again
        }
    }
    float* to = MODE == FOLD ? fold : (MODE == WALK || end == last) ? mine : nullptr;
    if (to) {
#pragma unroll
        for (int e = 0; e < NPT; ++e) {
            const int i = l * NPT + e;
            if (i < N) to[i] = S[e];
        }
    }
    if (MODE == FOLD && l == 0 && ch < inner) sc.sums[seg_row * inner + ch] = dt_sum;
}

// One thread an entry of the state: from the seat over the portion's segments, leaving in each one's fold the state before it.
__global__ void __launch_bounds__(256)
selective_chain_kernel(SelectiveScan sc) {
    griddep_wait();
    griddep_launch_dependents();
    const int r = blockIdx.x;
    const size_t per = (size_t)sc.inner * sc.N, e = (size_t)blockIdx.y * 256 + threadIdx.x;
    const int n = sc.cu_q[r + 1] - sc.cu_q[r];
    if (e >= per || n <= 0) return;
    const int segments = (n + SEGMENT - 1) / SEGMENT, seat = sc.seats[r];
    const size_t row = segment_row(sc.cu_q, r);
    float S = (seat >= 0 && seat < sc.n_seats) ? sc.state[(size_t)seat * sc.state_stride + e] : 0.f;
    const float a = sc.minus_a[e];
    float* p = sc.folds + row * per + e;
    const float* sum = sc.sums + row * sc.inner + e / sc.N;
    constexpr int AHEAD = 8;                      // the folds of so many segments are asked for at once: the chain waits on memory
    for (int s0 = 0; s0 < segments; s0 += AHEAD, p += AHEAD * per, sum += (size_t)AHEAD * sc.inner) {
        float u[AHEAD], d[AHEAD];
#pragma unroll
        for (int x = 0; x < AHEAD; ++x) {
            const bool in = s0 + x < segments;
            u[x] = in ? p[x * per] : 0.f;
            d[x] = in ? sum[(size_t)x * sc.inner] : 0.f;
        }
#pragma unroll
        for (int x = 0; x < AHEAD; ++x) {
            if (s0 + x >= segments) break;
            p[x * per] = S;
            S = fmaf(exp_decay(a * d[x]), S, u[x]);
        }
    }
}

template <typename TX, int LANES, int NPT, int TT>
int launch_selective(const void* x, const void* bc, long long ldbc, const void* z, long long ldz, void* out, long long ldo, SelectiveScan sc,
                     int requests, int segments, cudaStream_t stream) {
    constexpr int CH = SCAN_THREADS / LANES, NP = LANES * NPT;
    constexpr size_t smem = (size_t)(4 * TT * CH + 2 * TT * NP) * sizeof(float);
    static_assert(smem <= 48 * 1024, "a tile of the selective scan fits the shared memory every block has");
    const int blocks = (sc.inner + CH - 1) / CH;
#define FE_SELECTIVE_LAUNCH(MODE, SEGMENTS)                                                                                            \
    fe::launch(selective_scan_kernel<TX, MODE, LANES, NPT, TT>, dim3(blocks, requests, SEGMENTS), SCAN_THREADS, smem, stream, (const TX*)x, \
               (const TX*)bc, ldbc, (const TX*)z, ldz, (TX*)out, ldo, sc)
    if (segments <= 1) {
        FE_SELECTIVE_LAUNCH(WALK, 1);
    } else {
        FE_SELECTIVE_LAUNCH(FOLD, segments);
        fe::launch(selective_chain_kernel, dim3(requests, (unsigned)(((long long)sc.inner * sc.N + 255) / 256)), 256, 0, stream, sc);
        FE_SELECTIVE_LAUNCH(OUT, segments);
    }
#undef FE_SELECTIVE_LAUNCH
    return fe_check_launch("selective_scan");
}

template <typename TX>
int dispatch_selective(const void* x, const void* bc, long long ldbc, const void* z, long long ldz, void* out, long long ldo, SelectiveScan sc,
                       int requests, int segments, cudaStream_t stream) {
#define FE_SELECTIVE(LANES, NPT, TT) return launch_selective<TX, LANES, NPT, TT>(x, bc, ldbc, z, ldz, out, ldo, sc, requests, segments, stream)
    if (sc.N <= 16) FE_SELECTIVE(4, 4, 32);
    if (sc.N <= 32) FE_SELECTIVE(8, 4, 32);
    if (sc.N <= 64) FE_SELECTIVE(16, 4, 32);
    if (sc.N <= 128) FE_SELECTIVE(32, 4, 16);
    FE_SELECTIVE(32, 16, 8);
#undef FE_SELECTIVE
}

// ---------------------------------------------------------------------------------------------
// One token a request: LANES lanes share a channel, first its step size's dot product over the rank, then its state.
template <typename TX, int LANES>
__global__ void __launch_bounds__(SCAN_THREADS)
selective_decode_kernel(const TX* __restrict__ x, const TX* __restrict__ low, long long ldl, const TX* __restrict__ dt_weight,
                        const float* __restrict__ dt_bias, const float* __restrict__ minus_a, const float* __restrict__ skip,
                        const TX* __restrict__ z, long long ldz, float* state, long long state_stride, const int* __restrict__ seats,
                        TX* __restrict__ out, long long ldo, float scale, int inner, int N, int rank, int n_seats) {
    griddep_wait();
    griddep_launch_dependents();
    constexpr int CH = SCAN_THREADS / LANES;
    extern __shared__ __align__(16) float lows[];          // [rank + 2 N]: low | B | C
    const int tid = threadIdx.x, r = blockIdx.y;
    const int l = tid % LANES, ch = blockIdx.x * CH + tid / LANES;
    const bool in = ch < inner;
    for (int i = tid; i < rank + 2 * N; i += SCAN_THREADS) lows[i] = to_float(low[(size_t)r * ldl + i]);
    __syncthreads();
    float sum = 0.f;
    if (in) {
        const TX* w = dt_weight + (size_t)ch * rank;
        if (rank % 8 == 0) {
            for (int i = l * 8; i < rank; i += LANES * 8) {
                float v[8];
                load8<TX>(w + i, v);
#pragma unroll
                for (int e = 0; e < 8; ++e) sum = fmaf(v[e], lows[i + e], sum);
            }
        } else {
            for (int i = l; i < rank; i += LANES) sum = fmaf(to_float(w[i]), lows[i], sum);
        }
    }
#pragma unroll
    for (int o = 1; o < LANES; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    const float d = in ? softplus(sum + dt_bias[ch]) : 0.f;
    const float xc = in ? to_float(x[(size_t)r * inner + ch]) : 0.f, dx = d * xc;
    const int seat = seats[r];
    float* mine = (in && seat >= 0 && seat < n_seats) ? state + (size_t)seat * state_stride + (size_t)ch * N : nullptr;
    const float* a = minus_a + (size_t)ch * N;
    const float *B = lows + rank, *C = B + N;
    float y = 0.f;
    if (in) {
        if (N % 4 == 0) {
            for (int n = l * 4; n < N; n += LANES * 4) {
                const float4 a4 = *reinterpret_cast<const float4*>(a + n);
                const float4 s4 = mine ? *reinterpret_cast<const float4*>(mine + n) : make_float4(0.f, 0.f, 0.f, 0.f);
                const float aa[4] = {a4.x, a4.y, a4.z, a4.w};
                float ss[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    ss[e] = fmaf(exp_decay(d * aa[e]), ss[e], dx * B[n + e]);
                    y = fmaf(ss[e], C[n + e], y);
                }
                if (mine) *reinterpret_cast<float4*>(mine + n) = make_float4(ss[0], ss[1], ss[2], ss[3]);
            }
        } else {
            for (int n = l; n < N; n += LANES) {
                const float s = fmaf(exp_decay(d * a[n]), mine ? mine[n] : 0.f, dx * B[n]);
                y = fmaf(s, C[n], y);
                if (mine) mine[n] = s;
            }
        }
    }
#pragma unroll
    for (int o = 1; o < LANES; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (in && l == 0)
        out[(size_t)r * ldo + ch] = from_float<TX>(fmaf(skip[ch], xc, y) * silu(to_float(z[(size_t)r * ldz + ch])) * scale);
}

}  // namespace

// u [T, >= C] in in_dtype (rows ld entries long); conv float [taps, C], bias float [C]; the last taps - 1 inputs of a seat lie at
// state[seat][history_at] (float, oldest first); out [T, C] in out_dtype.  step_rows (may be null) float [T, >= heads]: gates
// [2][plane] gets minus_a softplus(row + step_bias) and softplus(row + step_bias).  most_tokens: the longest portion or more.
extern "C" int fe_conv_silu(const void* u, long long ld, int in_dtype, const float* conv, const float* bias, int taps, float* state,
                            long long state_stride, long long history_at, const int* seats, const int* cu_q, void* out, int out_dtype,
                            int requests, int most_tokens, int C, int n_seats, const float* step_rows, long long step_ld,
                            const float* step_bias, const float* minus_a, float* gates, long long plane, int heads, cudaStream_t stream) {
    FE_REQUIRE(requests >= 0 && requests <= 65535 && most_tokens >= 0 && C > 0 && taps >= 1 && ld >= C && n_seats >= 0 && history_at >= 0 &&
                   history_at + (long long)(taps - 1) * C <= state_stride && (step_rows == nullptr || (heads > 0 && step_ld >= heads)),
               "conv_silu: bad sizes (%d channels, %d taps)", C, taps);
    FE_REQUIRE(taps - 1 <= CONV_TILE, "conv_silu: %d taps; only a portion's first %d tokens may read the history", taps, CONV_TILE);
    FE_REQUIRE((in_dtype == FE_F32 && out_dtype == FE_F32) || (in_dtype == FE_BF16 && out_dtype == FE_BF16), "conv_silu: dtypes %d -> %d", in_dtype, out_dtype);
    if (requests == 0 || most_tokens == 0) return 0;
    const size_t align = in_dtype == FE_F32 ? 16 : 8;
    const bool vec = C % 4 == 0 && ld % 4 == 0 && ((size_t)u % align) == 0 && ((size_t)out % align) == 0 && state_stride % 4 == 0 && history_at % 4 == 0 &&
                     (((size_t)state | (size_t)conv | (size_t)bias) & 15) == 0;
    const int per_block = CONV_THREADS * (vec ? 4 : 1), stretches = (C + per_block - 1) / per_block;
    FE_REQUIRE(stretches < 65535, "conv_silu: %d channels", C);
    const Steps steps{step_rows, step_ld, step_bias, minus_a, gates, plane, heads};
    const dim3 grid((most_tokens + CONV_TILE - 1) / CONV_TILE, requests, stretches + (step_rows ? 1 : 0));
#define FE_CONV(T, TAPS, V)                                                                                                             \
    fe::launch(conv_silu_kernel<T, T, TAPS, V>, grid, CONV_THREADS, 0, stream, (const T*)u, ld, conv, bias, taps, state, state_stride,   \
               history_at, seats, cu_q, (T*)out, C, n_seats, stretches, steps)
#define FE_CONV_TAPS(T, V)                     \
    do {                                       \
        if (taps == 2) FE_CONV(T, 2, V);       \
        else if (taps == 3) FE_CONV(T, 3, V);  \
        else if (taps == 4) FE_CONV(T, 4, V);  \
        else FE_CONV(T, 0, V);                 \
    } while (0)
    if (in_dtype == FE_F32) {
        if (vec) FE_CONV_TAPS(float, 4);
        else FE_CONV_TAPS(float, 1);
    } else {
        if (vec) FE_CONV_TAPS(bf16, 4);
        else FE_CONV_TAPS(bf16, 1);
    }
#undef FE_CONV_TAPS
#undef FE_CONV
    return fe_check_launch("conv_silu");
}

// y float [T, inner], z float [T, >= inner] (rows ldz entries long), weight float [inner]; out [T, inner] in ``dtype``.
extern "C" int fe_gated_group_rmsnorm(const float* y, const float* z, long long ldz, const float* weight, float eps, void* out, int T, int inner,
                                      int groups, int dtype, cudaStream_t stream) {
    FE_REQUIRE(T >= 0 && inner > 0 && groups > 0 && inner % groups == 0 && groups <= 65535 && ldz >= inner, "gated_group_rmsnorm: bad sizes (%d in %d parts)", inner, groups);
    FE_REQUIRE(dtype == FE_F32 || dtype == FE_BF16, "gated_group_rmsnorm: unknown dtype %d", dtype);
    if (T == 0) return 0;
    const int width = inner / groups;
    const size_t smem = (size_t)width * sizeof(float);
    FE_REQUIRE(smem <= 200 * 1024, "gated_group_rmsnorm: a part of %d entries needs more shared memory than a block has", width);
    const bool vec = width % 4 == 0 && ldz % 4 == 0 && (((size_t)y | (size_t)z | (size_t)weight | (size_t)out) & 15) == 0;
    const int work = vec ? width / 4 : width;
    const int threads = work >= 1024 ? 512 : work >= 192 ? 256 : work >= 96 ? 128 : work >= 48 ? 64 : 32;
#define FE_GATED_NORM(TYPE, V)                                                                                                           \
    do {                                                                                                                                 \
        if (smem > 48 * 1024) {                                                                                                          \
            const cudaError_t err = cudaFuncSetAttribute(gated_group_rmsnorm_kernel<TYPE, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            FE_REQUIRE(err == cudaSuccess, "gated_group_rmsnorm: %s", cudaGetErrorString(err));                                           \
        }                                                                                                                                \
        fe::launch(gated_group_rmsnorm_kernel<TYPE, V>, dim3(T, groups), threads, smem, stream, y, z, ldz, weight, eps, (TYPE*)out, inner, width); \
    } while (0)
    if (dtype == FE_F32) {
        if (vec) FE_GATED_NORM(float, 4);
        else FE_GATED_NORM(float, 1);
    } else {
        if (vec) FE_GATED_NORM(bf16, 4);
        else FE_GATED_NORM(bf16, 1);
    }
#undef FE_GATED_NORM
    return fe_check_launch("gated_group_rmsnorm");
}

// How many tokens a segment has; a step's ``folds`` and ``sums`` have tokens / that + requests rows.
extern "C" int fe_selective_segment_tokens() { return SEGMENT; }

// x [T, inner] in ``dtype``; dt float [T, inner] before its bias and softplus (overwritten where ``segments`` is above 1); minus_a float
// [inner, N]; bc [T, >= 2 N] = B | C in ``dtype`` (rows ldbc entries long); z, out [T, >= inner] in ``dtype`` (rows ldz, ldo); state float
// [n_seats, >= inner N].  segments: how many the longest portion has, or 1 to walk every portion as a whole (folds and sums may then
// be null; else float [rows, inner N] and [rows, inner]).
extern "C" int fe_selective_scan(const void* x, float* dt, const float* dt_bias, const float* minus_a, const void* bc, long long ldbc,
                                 const float* skip, const void* z, long long ldz, float* state, long long state_stride, const int* seats,
                                 const int* cu_q, void* out, long long ldo, float scale, float* folds, float* sums, int segments, int requests,
                                 int inner, int N, int n_seats, int dtype, cudaStream_t stream) {
    FE_REQUIRE(requests >= 0 && requests <= 65535 && inner > 0 && N > 0 && N <= 512 && ldbc >= 2LL * N && ldz >= inner && ldo >= inner && n_seats >= 0 &&
                   (long long)inner * N <= state_stride && ((long long)inner * N + 255) / 256 <= 65535,
               "selective_scan: bad sizes (%d channels, %d state entries of at most 512)", inner, N);
    FE_REQUIRE(dtype == FE_F32 || dtype == FE_BF16, "selective_scan: unknown dtype %d", dtype);
    FE_REQUIRE(segments <= 65535 && (segments <= 1 || (folds && sums)), "selective_scan: segments need their scratch");
    if (requests == 0) return 0;
    const SelectiveScan sc{dt, dt_bias, minus_a, skip, state, state_stride, seats, cu_q, folds, sums, scale, inner, N, n_seats};
    if (dtype == FE_F32) return dispatch_selective<float>(x, bc, ldbc, z, ldz, out, ldo, sc, requests, segments, stream);
    return dispatch_selective<bf16>(x, bc, ldbc, z, ldz, out, ldo, sc, requests, segments, stream);
}

// One token a request: low [requests, >= rank + 2 N] = low | B | C (rows ldl), dt_weight [inner, rank] in ``dtype``.
extern "C" int fe_selective_decode(const void* x, const void* low, long long ldl, const void* dt_weight, const float* dt_bias, const float* minus_a,
                                   const float* skip, const void* z, long long ldz, float* state, long long state_stride, const int* seats,
                                   void* out, long long ldo, float scale, int requests, int inner, int N, int rank, int n_seats, int dtype,
                                   cudaStream_t stream) {
    FE_REQUIRE(requests >= 0 && requests <= 65535 && inner > 0 && N > 0 && rank > 0 && ldl >= rank + 2LL * N && ldz >= inner && ldo >= inner && n_seats >= 0 &&
                   (long long)inner * N <= state_stride,
               "selective_decode: bad sizes (%d channels, %d state entries, rank %d)", inner, N, rank);
    FE_REQUIRE(dtype == FE_F32 || dtype == FE_BF16, "selective_decode: unknown dtype %d", dtype);
    FE_REQUIRE(N % 4 != 0 || (state_stride % 4 == 0 && (((size_t)state | (size_t)minus_a) & 15) == 0), "selective_decode: states start on 16-byte boundaries");
    FE_REQUIRE(rank % 8 != 0 || ((size_t)dt_weight & 15) == 0, "selective_decode: the projection's rows start on 16-byte boundaries");
    if (requests == 0) return 0;
    const size_t smem = ((size_t)rank + 2 * N) * sizeof(float);
    FE_REQUIRE(smem <= 48 * 1024, "selective_decode: rank %d and %d state entries need more shared memory than a block has", rank, N);
#define FE_SELECTIVE_DECODE(TYPE, LANES)                                                                                                \
    fe::launch(selective_decode_kernel<TYPE, LANES>, dim3((inner + SCAN_THREADS / LANES - 1) / (SCAN_THREADS / LANES), requests),        \
               SCAN_THREADS, smem, stream, (const TYPE*)x, (const TYPE*)low, ldl, (const TYPE*)dt_weight, dt_bias, minus_a, skip,         \
               (const TYPE*)z, ldz, state, state_stride, seats, (TYPE*)out, ldo, scale, inner, N, rank, n_seats)
    if (dtype == FE_F32) {
        if (N <= 32) FE_SELECTIVE_DECODE(float, 4);
        else FE_SELECTIVE_DECODE(float, 16);
    } else {
        if (N <= 32) FE_SELECTIVE_DECODE(bf16, 4);
        else FE_SELECTIVE_DECODE(bf16, 16);
    }
#undef FE_SELECTIVE_DECODE
    return fe_check_launch("selective_decode");
}
