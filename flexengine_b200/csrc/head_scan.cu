// Linear attention whose decay and weight are a head's own for every token:
//   S_t = exp(l_t) S_(t-1) + w_t k_t v_t^T ;   o_t = S_t^T q_t (+ skip v_t)          S [d, dv] float per request and head
// with l_t <= 0 the logarithm of the decay; head h reads the query/key group h / (heads / groups).  Divided: a memory n [d] of
// the keys alone, n_t = exp(l_t) n_(t-1) + w_t k_t, and o_t / (max(|n_t . q_t|, e_t) + floor) with a number e_t per token.
// State-space layers with one decay per head (k, q, v = B, C, x; w the step size) and matrix memories with exponential gates
// (w = exp(i - m), l = f + m' - m, e = exp(-m) against a running maximum m) are both this.
// Kernels (all arithmetic float; logarithms are summed up in double, so that a decay between two tokens is as exact as its terms):
//   memory_gates   l, w and e of a matrix memory from its two gates' rows, the running maximum kept in the state
//   head_scan      the scan over the step's portions in blocks of C = 64 tokens.  With L_n = l_1 + .. + l_n inside a block,
//                    o_n = exp(L_n) S_0^T q_n + sum_(b <= n) exp(L_n - L_b) w_b (q_n . k_b) v_b
//                    S_C = exp(L_C) S_0 + sum_b exp(L_C - L_b) w_b k_b v_b^T
//                  so three launches (four where heads share queries and keys) do a step: every block's own sum of k v^T (independent of the others), the chain S_0 -> S_C -> ...
//                  over a portion's blocks (elementwise), and every block's outputs from the state before it (independent again)
//   head_step      a step of one token a request; with MEMORY everything of a matrix memory between its two products: gates,
//                  running maximum, recurrence, divisor, head norm and output gate
#define FE_PDL_CLASS 128
#include <math_constants.h>

#include "common.cuh"

using namespace fe;

namespace {

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }

// ---------------------------------------------------------------------------------------------
// Blocks of CHUNK tokens.  Block c of request r has row cu_q[r] / CHUNK + r + c of ``sums`` and ``totals``: the rows of different
// requests never meet, and T / CHUNK + requests rows hold a step.  A row of sums is a seat's layout: [heads][d][dv], then with a
// divisor [heads][d]; a row of totals the blocks' decays exp(L_C) [heads].
constexpr int CHUNK = 64;                // tokens a block
constexpr int TILE = 64;                 // key channels or value channels a tile
constexpr int PITCH = CHUNK + 4;         // a transposed tile's row: float4 reads stay aligned, stores spread over banks
static_assert(CHUNK == TILE, "a block of tokens and a tile of channels are loaded by the same loops");

__device__ __forceinline__ size_t chunk_row(const int* __restrict__ cu_q, int r) { return (size_t)(cu_q[r] / CHUNK + r); }

// ---------------------------------------------------------------------------------------------
// The gates of a matrix memory, in blocks of CHUNK tokens.  Over a block the running maximum goes from m to max(m + F, G) with F the
// sum of the block's f and G what it comes to from minus infinity.  The first kernel makes the gates and F and G; the second one
// folds the blocks before its own and walks its tokens one after the other.  A block's last token takes the folded value, which the
// next block (and the seat) starts from.  Planes 0 and 1 of ``gates`` hold f and i in between.  Grid (block of tokens, request).
constexpr int GATE_THREADS = 256;

__global__ void __launch_bounds__(GATE_THREADS)
memory_gates_local_kernel(const float* __restrict__ rows, long long ld, const float* __restrict__ bias, float cap, const float* __restrict__ state,
                          long long state_stride, long long maxima_at, const int* __restrict__ seats, const int* __restrict__ cu_q,
                          float* __restrict__ gates, long long plane, float* __restrict__ totals, float* __restrict__ starts, int heads,
                          int n_seats) {
    griddep_wait();
    griddep_launch_dependents();
    extern __shared__ float smem[];
    float *is = smem, *fs = smem + CHUNK * heads;          // [CHUNK][heads]
    const int c = blockIdx.x, r = blockIdx.y;
    const int begin = cu_q[r] + c * CHUNK, end = cu_q[r + 1];
    if (begin >= end) return;
    const int len = min(CHUNK, end - begin);
    for (int e = threadIdx.x; e < len * 2 * heads; e += GATE_THREADS) {
        const int t = e / (2 * heads), col = e - t * 2 * heads;
        const float z = capped(rows[(size_t)(begin + t) * ld + col] + bias[col], cap);
        if (col < heads) {
            is[t * heads + col] = z;
            gates[plane + (size_t)(begin + t) * heads + col] = z;
        } else {
            const float f = log_sigmoid(z);
            fs[t * heads + col - heads] = f;
            gates[(size_t)(begin + t) * heads + col - heads] = f;
        }
    }
    __syncthreads();
    const size_t row = chunk_row(cu_q, r) + c;
    const int seat = seats[r];
    for (int h = threadIdx.x; h < heads; h += GATE_THREADS) {
        float F = 0.f, G = -CUDART_INF_F;
#pragma unroll 8
        for (int t = 0; t < len; ++t) {
            const float f = fs[t * heads + h];
            G = fmaxf(G + f, is[t * heads + h]);
            F += f;
        }
        totals[(2 * row) * heads + h] = F;
        totals[(2 * row + 1) * heads + h] = G;
        if (c == 0) starts[(size_t)r * heads + h] = (seat >= 0 && seat < n_seats) ? state[(size_t)seat * state_stride + maxima_at + h] : 0.f;
    }
}

__global__ void __launch_bounds__(GATE_THREADS)
memory_gates_walk_kernel(float* state, long long state_stride, long long maxima_at, const int* __restrict__ seats, const int* __restrict__ cu_q,
                         float* __restrict__ gates, long long plane, const float* __restrict__ totals, const float* __restrict__ starts, int heads,
                         int n_seats) {
    griddep_wait();
    griddep_launch_dependents();
    extern __shared__ float smem[];
    float *is = smem, *fs = smem + CHUNK * heads, *ms = fs + CHUNK * heads;        // [CHUNK][heads] twice, the maxima [CHUNK + 1][heads]
    const int c = blockIdx.x, r = blockIdx.y;
    const int begin = cu_q[r] + c * CHUNK, end = cu_q[r + 1];
    if (begin >= end) return;
    const int len = min(CHUNK, end - begin), count = len * heads;
    float *decays = gates + (size_t)begin * heads, *weights = decays + plane, *floors = weights + plane;
    for (int e = threadIdx.x; e < count; e += GATE_THREADS) {
        fs[e] = decays[e];
        is[e] = weights[e];
    }
    __syncthreads();
    const size_t row0 = chunk_row(cu_q, r);
    const int seat = seats[r];
    for (int h = threadIdx.x; h < heads; h += GATE_THREADS) {
        float m = starts[(size_t)r * heads + h];
#pragma unroll 8
        for (int b = 0; b < c; ++b) m = fmaxf(m + totals[2 * (row0 + b) * heads + h], totals[(2 * (row0 + b) + 1) * heads + h]);
        const float after = fmaxf(m + totals[2 * (row0 + c) * heads + h], totals[(2 * (row0 + c) + 1) * heads + h]);
        ms[h] = m;
#pragma unroll 8
        for (int t = 0; t < len - 1; ++t) {
            m = fmaxf(fs[t * heads + h] + m, is[t * heads + h]);
            ms[(t + 1) * heads + h] = m;
        }
        ms[len * heads + h] = after;
        if (begin + len == end && seat >= 0 && seat < n_seats) state[(size_t)seat * state_stride + maxima_at + h] = after;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < count; e += GATE_THREADS) {
        const float next = ms[e + heads];
        decays[e] = (fs[e] + ms[e]) - next;
        weights[e] = expf(is[e] - next);
        floors[e] = expf(-next);
    }
}

// ---------------------------------------------------------------------------------------------
// cum[n] = l_0 + .. + l_n of the block's tokens (tokens from len on repeat the last sum); the first CHUNK threads work.
__device__ __forceinline__ void cumulate(const float* __restrict__ gates, int begin, int len, int heads, int head, double* cum, double* half) {
    const int tid = threadIdx.x;
    double x = 0.0;
    if (tid < CHUNK) {
        x = tid < len ? (double)gates[(size_t)(begin + tid) * heads + head] : 0.0;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double y = __shfl_up_sync(0xffffffffu, x, o);
            if ((tid & 31) >= o) x += y;
        }
        if (tid == 31) *half = x;
    }
    __syncthreads();
    if (tid < CHUNK) cum[tid] = tid < 32 ? x : x + *half;
    __syncthreads();
}

// sums[row][head] <- sum_b exp(L_last - L_b) w_b k_b v_b^T over the block's tokens (and the same of the keys alone).  Grid (block of
// tokens, request, head x tile of key channels x tile of value channels), 256 threads as 16 x 16, a thread 4 key x 4 value channels.
__global__ void __launch_bounds__(256)
head_scan_sums_kernel(const float* __restrict__ k, long long ldk, const float* __restrict__ v, long long ldv, const float* __restrict__ gates,
                      long long plane, const int* __restrict__ cu_q, float* __restrict__ sums, float* __restrict__ totals, long long per,
                      int heads, int groups, int d, int dv, int nd, int nv, int divided) {
    griddep_wait();
    griddep_launch_dependents();
    __shared__ __align__(16) float ks[CHUNK * TILE];
    __shared__ __align__(16) float vs[CHUNK * TILE];
    __shared__ double cum[CHUNK], half;
    __shared__ float pw[CHUNK];
    const int c = blockIdx.x, r = blockIdx.y;
    int z = blockIdx.z;
    const int vt = z % nv;
    z /= nv;
    const int dt = z % nd, head = z / nd;
    const int begin = cu_q[r] + c * CHUNK, end = cu_q[r + 1];
    if (begin >= end) return;
    const int len = min(CHUNK, end - begin);
    const int tid = threadIdx.x;
    const size_t row = chunk_row(cu_q, r) + c;
    cumulate(gates, begin, len, heads, head, cum, &half);
    if (tid < CHUNK) pw[tid] = tid < len ? expf((float)(cum[len - 1] - cum[tid])) * gates[plane + (size_t)(begin + tid) * heads + head] : 0.f;
    if (tid == 0 && dt == 0 && vt == 0) totals[row * heads + head] = exp_decay((float)cum[len - 1]);
    __syncthreads();
    const int group = head / (heads / groups);
    for (int e = tid; e < CHUNK * TILE; e += 256) {
        const int b = e / TILE, i = e - b * TILE;
        const int gi = dt * TILE + i, gj = vt * TILE + i;
        const bool in = b < len;
        ks[e] = (in && gi < d) ? pw[b] * k[(size_t)(begin + b) * ldk + (size_t)group * d + gi] : 0.f;
        vs[e] = (in && gj < dv) ? v[(size_t)(begin + b) * ldv + (size_t)head * dv + gj] : 0.f;
    }
    __syncthreads();
    const int ty = tid >> 4, tx = tid & 15;
    float acc[4][4] = {};
#pragma unroll 4
    for (int b = 0; b < len; ++b) {
        const float4 k4 = *reinterpret_cast<const float4*>(ks + b * TILE + ty * 4);
        const float4 v4 = *reinterpret_cast<const float4*>(vs + b * TILE + tx * 4);
        const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(kk[x], vv[y], acc[x][y]);
    }
    float* to = sums + row * per + (size_t)head * d * dv;
#pragma unroll
    for (int x = 0; x < 4; ++x) {
        const int gi = dt * TILE + ty * 4 + x;
        if (gi >= d) continue;
#pragma unroll
        for (int y = 0; y < 4; ++y) {
            const int gj = vt * TILE + tx * 4 + y;
            if (gj < dv) to[(size_t)gi * dv + gj] = acc[x][y];
        }
    }
    if (divided && vt == 0 && tid < TILE && dt * TILE + tid < d) {
        float sum = 0.f;
        for (int b = 0; b < len; ++b) sum += ks[b * TILE + tid];
        sums[row * per + (size_t)heads * d * dv + (size_t)head * d + dt * TILE + tid] = sum;
    }
}

// One thread an entry of the seat: S walks the portion's blocks, leaving in each block's row what S was BEFORE that block in
// place of the block's sum, and ends in the seat.
__global__ void __launch_bounds__(256)
head_scan_chain_kernel(const float* __restrict__ totals, float* state, long long state_stride, const int* __restrict__ seats,
                       const int* __restrict__ cu_q, float* sums, long long per, int heads, int d, int dv, int n_seats) {
    griddep_wait();
    griddep_launch_dependents();
    const int r = blockIdx.x;
    const long long e = (long long)blockIdx.y * blockDim.x + threadIdx.x;
    const int n = cu_q[r + 1] - cu_q[r];
    if (e >= per || n <= 0) return;
    const long long matrices = (long long)heads * d * dv;
    const int head = e < matrices ? (int)(e / ((long long)d * dv)) : (int)((e - matrices) / d);
    const int blocks = (n + CHUNK - 1) / CHUNK;
    const int seat = seats[r];
    float* mine = (seat >= 0 && seat < n_seats) ? state + (size_t)seat * state_stride + e : nullptr;
    float S = mine ? *mine : 0.f;
    const size_t row = chunk_row(cu_q, r);
    float* p = sums + row * per + e;
    const float* decay = totals + row * heads + head;
    constexpr int AHEAD = 8;                      // the sums of so many blocks are asked for at once: the chain waits on memory
    for (int c0 = 0; c0 < blocks; c0 += AHEAD, p += AHEAD * per, decay += (size_t)AHEAD * heads) {
        float u[AHEAD], a[AHEAD];
#pragma unroll
        for (int x = 0; x < AHEAD; ++x) {
            const bool in = c0 + x < blocks;
            u[x] = in ? __ldcs(p + x * per) : 0.f;
            a[x] = in ? decay[(size_t)x * heads] : 0.f;
        }
#pragma unroll
        for (int x = 0; x < AHEAD; ++x) {
            if (c0 + x >= blocks) break;
            p[x * per] = S;
            S = fmaf(a[x], S, u[x]);
        }
    }
    if (mine) *mine = S;
}

// The products of a block's queries and keys where several heads read one group of them: qk[row][group] [b][n] = query_scale q_n . k_b.
// Grid (block of tokens, request, group), 256 threads as 16 x 16.
__global__ void __launch_bounds__(256)
head_scan_products_kernel(const float* __restrict__ q, long long ldq, float query_scale, const float* __restrict__ k, long long ldk,
                          const int* __restrict__ cu_q, float* __restrict__ qk, int groups, int d, int nd) {
    griddep_wait();
    griddep_launch_dependents();
    __shared__ __align__(16) float qT[TILE * PITCH];
    __shared__ __align__(16) float kT[TILE * PITCH];
    const int c = blockIdx.x, r = blockIdx.y, group = blockIdx.z;
    const int begin = cu_q[r] + c * CHUNK, end = cu_q[r + 1];
    if (begin >= end) return;
    const int len = min(CHUNK, end - begin);
    const int tid = threadIdx.x, ty = tid >> 4, tx = tid & 15;
    float W[4][4] = {};
    for (int dt = 0; dt < nd; ++dt) {
        __syncthreads();
        for (int e = tid; e < CHUNK * TILE; e += 256) {
            const int n = e / TILE, i = e - n * TILE, gi = dt * TILE + i;
            const bool in = n < len && gi < d;
            qT[i * PITCH + n] = in ? query_scale * q[(size_t)(begin + n) * ldq + (size_t)group * d + gi] : 0.f;
            kT[i * PITCH + n] = in ? k[(size_t)(begin + n) * ldk + (size_t)group * d + gi] : 0.f;
        }
        __syncthreads();
#pragma unroll 4
        for (int i = 0; i < TILE; ++i) {
            const float4 q4 = *reinterpret_cast<const float4*>(qT + i * PITCH + ty * 4);
            const float4 k4 = *reinterpret_cast<const float4*>(kT + i * PITCH + tx * 4);
            const float qq[4] = {q4.x, q4.y, q4.z, q4.w}, kk[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
            for (int x = 0; x < 4; ++x)
#pragma unroll
                for (int y = 0; y < 4; ++y) W[x][y] = fmaf(qq[x], kk[y], W[x][y]);
        }
    }
    float* to = qk + ((chunk_row(cu_q, r) + c) * groups + group) * (size_t)(CHUNK * CHUNK);
#pragma unroll
    for (int y = 0; y < 4; ++y) *reinterpret_cast<float4*>(to + (tx * 4 + y) * CHUNK + ty * 4) = make_float4(W[0][y], W[1][y], W[2][y], W[3][y]);
}

// A block's outputs for a tile of value channels: W = (Q K^T) with entry (n, b) times exp(L_n - L_b) w_b where b <= n, else 0, and
// ``skip`` added on the diagonal; out = diag(exp(L_n)) Q S_0 + W V.  Q, K and S_0 pass through shared memory in tiles of key
// channels; W takes the keys' place.  Grid (block of tokens, request, head x tile of value channels), 256 threads as 16 x 16, a
// thread 4 tokens x 4 columns.  SHARED: Q K^T comes from head_scan_products (``qk``) instead.
constexpr size_t CHUNK_OUT_SMEM = ((size_t)2 * TILE * PITCH + (size_t)TILE * TILE + (size_t)CHUNK * TILE + 5 * CHUNK + 4) * sizeof(float) +
                                  CHUNK * sizeof(double);

template <bool SHARED>
__global__ void __launch_bounds__(256)
head_scan_out_kernel(const float* __restrict__ q, long long ldq, float query_scale, const float* __restrict__ k, long long ldk,
                     const float* __restrict__ v, long long ldv, const float* __restrict__ gates, long long plane,
                     const float* __restrict__ skip, const float* __restrict__ qk, const int* __restrict__ cu_q,
                     const float* __restrict__ sums, long long per,
                     float* __restrict__ out, int heads, int groups, int d, int dv, int nd, int nv, int divided, float floor) {
    griddep_wait();
    griddep_launch_dependents();
    extern __shared__ __align__(16) float smem[];
    double* cum = reinterpret_cast<double*>(smem);              // [CHUNK]
    float* qT = smem + 2 * CHUNK;                // [TILE][PITCH]: key channel i of token n at i * PITCH + n
    float* kT = qT + TILE * PITCH;               // the same of the keys; later W as [b][n]
    float* sS = kT + TILE * PITCH;               // [TILE][TILE] the state before the block, key channel x value channel
    float* vS = sS + TILE * TILE;                // [CHUNK][TILE]
    float* wb = vS + CHUNK * TILE;               // [CHUNK] the tokens' weights
    float* below = wb + CHUNK;                   // [CHUNK] n_t . q_t, then the factor of the output
    float* nS = below + CHUNK;                   // [TILE] the keys' memory before the block
    __shared__ double half;
    const int c = blockIdx.x, r = blockIdx.y;
    const int vt = blockIdx.z % nv, head = blockIdx.z / nv, group = head / (heads / groups);
    const int begin = cu_q[r] + c * CHUNK, end = cu_q[r + 1];
    if (begin >= end) return;
    const int len = min(CHUNK, end - begin);
    const int tid = threadIdx.x, ty = tid >> 4, tx = tid & 15;
    cumulate(gates, begin, len, heads, head, cum, &half);
    if (tid < CHUNK) wb[tid] = tid < len ? gates[plane + (size_t)(begin + tid) * heads + head] : 0.f;
    for (int e = tid; e < CHUNK * TILE; e += 256) {
        const int b = e / TILE, j = e - b * TILE, gj = vt * TILE + j;
        vS[e] = (b < len && gj < dv) ? v[(size_t)(begin + b) * ldv + (size_t)head * dv + gj] : 0.f;
    }
    const float* before = sums + (chunk_row(cu_q, r) + c) * per + (size_t)head * d * dv;
    const float* keys_before = sums + (chunk_row(cu_q, r) + c) * per + (size_t)heads * d * dv + (size_t)head * d;
    float W[4][4] = {}, O[4][4] = {};
    const int mine = tid >> 2, part = tid & 3;   // four threads a token for its product with the keys' memory
    float nq = 0.f;
    for (int dt = 0; dt < nd; ++dt) {
        __syncthreads();
        for (int e = tid; e < CHUNK * TILE; e += 256) {
            const int n = e / TILE, i = e - n * TILE, gi = dt * TILE + i;
            const bool in = n < len && gi < d;
            qT[i * PITCH + n] = in ? query_scale * q[(size_t)(begin + n) * ldq + (size_t)group * d + gi] : 0.f;
            if (!SHARED) kT[i * PITCH + n] = in ? k[(size_t)(begin + n) * ldk + (size_t)group * d + gi] : 0.f;
            const int gj = vt * TILE + i;                                       // here n walks key channels, i value channels
            sS[e] = (dt * TILE + n < d && gj < dv) ? before[(size_t)(dt * TILE + n) * dv + gj] : 0.f;
        }
        if (divided && tid < TILE) nS[tid] = dt * TILE + tid < d ? keys_before[dt * TILE + tid] : 0.f;
        __syncthreads();
#pragma unroll 4
        for (int i = 0; i < TILE; ++i) {
            const float4 q4 = *reinterpret_cast<const float4*>(qT + i * PITCH + ty * 4);
            const float4 k4 = SHARED ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(kT + i * PITCH + tx * 4);
            const float4 s4 = *reinterpret_cast<const float4*>(sS + i * TILE + tx * 4);
            const float qq[4] = {q4.x, q4.y, q4.z, q4.w}, kk[4] = {k4.x, k4.y, k4.z, k4.w}, ss[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
            for (int x = 0; x < 4; ++x)
#pragma unroll
                for (int y = 0; y < 4; ++y) {
                    if (!SHARED) W[x][y] = fmaf(qq[x], kk[y], W[x][y]);
                    O[x][y] = fmaf(qq[x], ss[y], O[x][y]);
                }
        }
        if (divided)
            for (int i = part; i < TILE; i += 4) nq = fmaf(qT[i * PITCH + mine], nS[i], nq);
    }
    __syncthreads();
    if (SHARED) {
        const float* from = qk + ((chunk_row(cu_q, r) + c) * groups + group) * (size_t)(CHUNK * CHUNK);
#pragma unroll
        for (int y = 0; y < 4; ++y) {
            const float4 w4 = *reinterpret_cast<const float4*>(from + (tx * 4 + y) * CHUNK + ty * 4);
            W[0][y] = w4.x, W[1][y] = w4.y, W[2][y] = w4.z, W[3][y] = w4.w;
        }
    }
    const float skip_of = skip ? skip[head] : 0.f;
#pragma unroll
    for (int y = 0; y < 4; ++y) {
        const int b = tx * 4 + y;
        float w[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int n = ty * 4 + x;
            w[x] = b < n ? W[x][y] * (expf((float)(cum[n] - cum[b])) * wb[b]) : b == n ? fmaf(W[x][y], wb[b], skip_of) : 0.f;
        }
        *reinterpret_cast<float4*>(kT + b * PITCH + ty * 4) = make_float4(w[0], w[1], w[2], w[3]);
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) {
        const float a = expf((float)cum[ty * 4 + x]);
#pragma unroll
        for (int y = 0; y < 4; ++y) O[x][y] *= a;
    }
    __syncthreads();
    if (divided) {
        nq *= expf((float)cum[mine]);
        for (int b = part; b <= mine; b += 4) nq += kT[b * PITCH + mine];
        nq += __shfl_xor_sync(0xffffffffu, nq, 1);
        nq += __shfl_xor_sync(0xffffffffu, nq, 2);
        if (part == 0) {
            const float e = mine < len ? gates[2 * plane + (size_t)(begin + mine) * heads + head] : 1.f;
            below[mine] = fmaxf(fabsf(nq), e) + floor;
        }
    }
    const int seen = min(len, ty * 4 + 4);                                       // tokens after a thread's last one weigh nothing
#pragma unroll 4
    for (int b = 0; b < seen; ++b) {
        const float4 w4 = *reinterpret_cast<const float4*>(kT + b * PITCH + ty * 4);
        const float4 v4 = *reinterpret_cast<const float4*>(vS + b * TILE + tx * 4);
        const float ww[4] = {w4.x, w4.y, w4.z, w4.w}, vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int y = 0; y < 4; ++y) O[x][y] = fmaf(ww[x], vv[y], O[x][y]);
    }
    if (divided) __syncthreads();
#pragma unroll
    for (int x = 0; x < 4; ++x) {
        const int n = ty * 4 + x;
        if (n >= len) continue;
        const float under = divided ? below[n] : 1.f;
#pragma unroll
        for (int y = 0; y < 4; ++y) {
            const int gj = vt * TILE + tx * 4 + y;
            if (gj < dv) out[(size_t)(begin + n) * heads * dv + (size_t)head * dv + gj] = divided ? O[x][y] / under : O[x][y];
        }
    }
}

// ---------------------------------------------------------------------------------------------
// A step of ONE token a request.  Block per (request, head); its threads are ``step_groups`` runs of key channels x ``columns``
// value channels, so that the state's rows are read and written side by side and many of them are in flight; the runs' shares of
// S^T q meet in shared memory.  MEMORY: the row holds q | k | v | g | i | f of a matrix memory; gates, running maximum, the memory
// of the keys, the divisor, the head's norm with its weight and the sigmoid gate are done here too and ``out`` is T; else
// ``out`` is float and the decay's logarithm and the weight come from ``gates``.
struct MemoryStep {
    const float* bias;           // [2 heads]: of i, then of f
    const float* norm_weight;    // [heads dv]
    float cap, floor, eps;
};

template <typename T, bool MEMORY>
__global__ void __launch_bounds__(1024)
head_step_kernel(const float* __restrict__ q, long long ldq, float query_scale, const float* __restrict__ k, long long ldk,
                 const float* __restrict__ v, long long ldv, const float* __restrict__ gates, long long plane, const float* __restrict__ skip,
                 float* state, long long state_stride, const int* __restrict__ seats, T* __restrict__ out, int heads, int groups, int d,
                 int dv, int n_seats, int step_groups, MemoryStep ms) {
    griddep_wait();
    griddep_launch_dependents();
    extern __shared__ __align__(16) float smem[];
    const int columns = blockDim.x / step_groups;
    float* qs = smem;                               // [d]
    float* ks = qs + d;                             // [d] the key times the weight
    float* os = ks + d;                             // [dv]
    float* part = os + dv;                          // [step_groups][columns]
    float* red = part + step_groups * columns;      // [33]
    float* gate = red + 33;                         // decay, weight, exp(-m)
    const int r = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, group = head / (heads / groups);
    const int seat = seats[r];
    float* base = (seat >= 0 && seat < n_seats) ? state + (size_t)seat * state_stride : nullptr;
    float* mine = base ? base + (size_t)head * d * dv : nullptr;
    if (tid == 0) {
        if (MEMORY) {
            const float* row = q + (size_t)r * ldq + 2 * (size_t)heads * d + 2 * (size_t)heads * dv;
            float* kept = base ? base + (size_t)heads * d * dv + (size_t)heads * d + head : nullptr;
            const float i = capped(row[head] + ms.bias[head], ms.cap), f = log_sigmoid(capped(row[heads + head] + ms.bias[heads + head], ms.cap));
            const float m = kept ? *kept : 0.f, next = fmaxf(f + m, i);
            gate[0] = exp_decay((f + m) - next);
            gate[1] = expf(i - next);
            gate[2] = expf(-next);
            if (kept) *kept = next;
        } else {
            gate[0] = exp_decay(gates[(size_t)r * heads + head]);
            gate[1] = gates[plane + (size_t)r * heads + head];
        }
    }
    for (int i = tid; i < d; i += blockDim.x) {
        qs[i] = query_scale * q[(size_t)r * ldq + (size_t)group * d + i];
        ks[i] = k[(size_t)r * ldk + (size_t)group * d + i];
    }
    __syncthreads();
    const float a = gate[0], w = gate[1];
    float dot = 0.f, nq = 0.f;
    for (int i = tid; i < d; i += blockDim.x) {
        dot = fmaf(qs[i], ks[i], dot);
        if (MEMORY) {
            float* n = base ? base + (size_t)heads * d * dv + (size_t)head * d + i : nullptr;
            const float next = fmaf(w, ks[i], n ? a * *n : 0.f);
            nq = fmaf(next, qs[i], nq);
            if (n) *n = next;
        }
    }
    dot = w * block_sum(dot, red);
    if (MEMORY) nq = fmaxf(fabsf(block_sum(nq, red)), gate[2]) + ms.floor;
    const int g = tid / columns, jj = tid - g * columns;
    const int per = (d + step_groups - 1) / step_groups;
    const int i0 = g * per, i1 = min(d, i0 + per);
    const float* vrow = v + (size_t)r * ldv + (size_t)head * dv;
    const float skip_of = (!MEMORY && skip) ? skip[head] : 0.f;
    float ss = 0.f;
    for (int j0 = 0; j0 < dv; j0 += columns) {
        const int j = j0 + jj;
        const bool own = g < step_groups && j < dv;
        const float vj = own ? vrow[j] : 0.f, wv = w * vj;
        float acc = 0.f;
        if (own && mine) {
            float* col = mine + j;
            for (int i = i0; i < i1; i += 8) {          // eight rows asked for before any is written
                float sv[8];
#pragma unroll
                for (int x = 0; x < 8; ++x) sv[x] = i + x < i1 ? col[(size_t)(i + x) * dv] : 0.f;
#pragma unroll
                for (int x = 0; x < 8; ++x) {
                    if (i + x >= i1) break;
                    acc = fmaf(qs[i + x], sv[x], acc);
                    col[(size_t)(i + x) * dv] = fmaf(a, sv[x], ks[i + x] * wv);
                }
            }
        }
        if (g < step_groups) part[g * columns + jj] = acc;
        __syncthreads();
        if (g == 0 && j < dv) {
            float sum = 0.f;
            for (int x = 0; x < step_groups; ++x) sum += part[x * columns + jj];
            float o = fmaf(a, sum, (dot + skip_of) * vj);
            if (MEMORY) {
                o /= nq;
                os[j] = o;
                ss = fmaf(o, o, ss);
            } else {
                out[((size_t)r * heads + head) * dv + j] = from_float<T>(o);
            }
        }
        __syncthreads();
    }
    if (!MEMORY) return;
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)dv + ms.eps);
    const float* grow = vrow + (size_t)heads * dv;
    for (int j = tid; j < dv; j += blockDim.x)
        out[((size_t)r * heads + head) * dv + j] = from_float<T>(os[j] * inv * ms.norm_weight[(size_t)head * dv + j] / (1.f + expf(-grow[j])));
}

template <typename T, bool MEMORY>
int launch_step(const float* q, long long ldq, float query_scale, const float* k, long long ldk, const float* v, long long ldv,
                const float* gates, long long plane, const float* skip, float* state, long long state_stride, const int* seats, void* out,
                int requests, int heads, int groups, int d, int dv, int n_seats, MemoryStep ms, cudaStream_t stream) {
    int columns = ((dv < 256 ? dv : 256) + 31) / 32 * 32;
    int step_groups = 512 / columns;
    step_groups = step_groups < 1 ? 1 : (step_groups > d ? d : step_groups);
    const size_t smem = ((size_t)2 * d + dv + (size_t)step_groups * columns + 33 + 3) * sizeof(float);
    FE_REQUIRE(smem <= 48 * 1024, "head_step: key size %d and value size %d need more shared memory than a block has", d, dv);
    fe::launch(head_step_kernel<T, MEMORY>, dim3(requests, heads), step_groups * columns, smem, stream, q, ldq, query_scale, k, ldk, v, ldv,
               gates, plane, skip, state, state_stride, seats, (T*)out, heads, groups, d, dv, n_seats, step_groups, ms);
    return fe_check_launch("head_step");
}

}  // namespace

// rows float [T, >= 2 heads] (i, then f; rows ld entries long); bias float [2 heads]; gates float [3][plane] with plane >= T heads: the
// decays' logarithms, the weights, exp(-m); the running maxima [heads] of a seat lie at state[seat][maxima_at].  totals float [tokens /
// 64 + requests, 2, heads] and starts float [requests, heads] are scratch; most_tokens: the longest portion of the step or more.
extern "C" int fe_memory_gates(const float* rows, long long ld, const float* bias, float cap, float* state, long long state_stride,
                               long long maxima_at, const int* seats, const int* cu_q, float* gates, long long plane, float* totals, float* starts,
                               int requests, int most_tokens, int heads, int n_seats, cudaStream_t stream) {
    FE_REQUIRE(requests >= 0 && heads > 0 && ld >= 2 * heads && cap > 0.f && n_seats >= 0 && maxima_at >= 0 && maxima_at + heads <= state_stride,
               "memory_gates: bad sizes (%d heads)", heads);
    if (requests == 0 || most_tokens == 0) return 0;
    FE_REQUIRE(requests <= 65535 && heads <= 256, "memory_gates: %d requests or %d heads (up to 256)", requests, heads);
    const dim3 grid((most_tokens + CHUNK - 1) / CHUNK, requests);
    const size_t local = (size_t)2 * CHUNK * heads * sizeof(float), walk = (size_t)(3 * CHUNK + 1) * heads * sizeof(float);
    if (walk > 48 * 1024) {
        cudaError_t err = cudaFuncSetAttribute(memory_gates_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)local);
        if (err == cudaSuccess) err = cudaFuncSetAttribute(memory_gates_walk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)walk);
        FE_REQUIRE(err == cudaSuccess, "memory_gates: %s", cudaGetErrorString(err));
    }
    fe::launch(memory_gates_local_kernel, grid, GATE_THREADS, local, stream, rows, ld, bias, cap, (const float*)state, state_stride, maxima_at,
               seats, cu_q, gates, plane, totals, starts, heads, n_seats);
    fe::launch(memory_gates_walk_kernel, grid, GATE_THREADS, walk, stream, state, state_stride, maxima_at, seats, cu_q, gates, plane,
               (const float*)totals, (const float*)starts, heads, n_seats);
    return fe_check_launch("memory_gates");
}

extern "C" int fe_head_scan_chunk_tokens() { return CHUNK; }

// q, k float [T, >= groups d], v float [T, >= heads dv] (rows ldq, ldk, ldv entries long); gates float [2 or 3][plane] ([T, heads] each:
// logarithms of the decays, weights, with ``divided`` the numbers e_t); skip float [heads] or null (not with ``divided``); state
// float [n_seats, >= per] with per = heads d dv (+ heads d with ``divided``); sums float [tokens / 64 + requests, per] and totals
// [the same, heads] are scratch, and where several heads read a group (heads > groups) products [the same, groups, 64, 64]; out float [T, heads dv]; most_tokens: the longest portion of the step or more.
extern "C" int fe_head_scan(const float* q, long long ldq, float query_scale, const float* k, long long ldk, const float* v, long long ldv,
                            const float* gates, long long plane, const float* skip, float* state, long long state_stride, const int* seats,
                            const int* cu_q, float* out, float* sums, float* totals, float* products, int requests, int most_tokens, int heads, int groups, int d,
                            int dv, int n_seats, int divided, float floor, cudaStream_t stream) {
    const int nd = (d + TILE - 1) / TILE, nv = (dv + TILE - 1) / TILE;
    const long long per = (long long)heads * d * dv + (divided ? (long long)heads * d : 0);
    FE_REQUIRE(requests >= 0 && requests <= 65535 && heads > 0 && groups > 0 && heads % groups == 0 && d > 0 && dv > 0 && n_seats >= 0 && most_tokens >= 0 &&
                   per <= state_stride && ldq >= (long long)groups * d && ldk >= (long long)groups * d && ldv >= (long long)heads * dv &&
                   (long long)heads * nd * nv <= 65535 && (per + 255) / 256 <= 65535,
               "head_scan: bad sizes (heads %d over %d, key size %d, value size %d, %d requests)", heads, groups, d, dv, requests);
    FE_REQUIRE(!(divided && skip), "head_scan: a skip does not go with a divisor");
    if (requests == 0 || most_tokens == 0) return 0;
    static bool opted = false;
    if (!opted) {
        cudaError_t err = cudaFuncSetAttribute(head_scan_out_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)CHUNK_OUT_SMEM);
        if (err == cudaSuccess) err = cudaFuncSetAttribute(head_scan_out_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)CHUNK_OUT_SMEM);
        FE_REQUIRE(err == cudaSuccess, "head_scan: %s", cudaGetErrorString(err));
        opted = true;
    }
    const int most_blocks = (most_tokens + CHUNK - 1) / CHUNK;
    fe::launch(head_scan_sums_kernel, dim3(most_blocks, requests, heads * nd * nv), 256, 0, stream, k, ldk, v, ldv, gates, plane, cu_q, sums,
               totals, per, heads, groups, d, dv, nd, nv, divided);
    fe::launch(head_scan_chain_kernel, dim3(requests, (unsigned)((per + 255) / 256)), 256, 0, stream, (const float*)totals, state, state_stride,
               seats, cu_q, sums, per, heads, d, dv, n_seats);
    const bool shared = heads > groups && products != nullptr;
    if (shared)
        fe::launch(head_scan_products_kernel, dim3(most_blocks, requests, groups), 256, 0, stream, q, ldq, query_scale, k, ldk, cu_q, products,
                   groups, d, nd);
    fe::launch(shared ? head_scan_out_kernel<true> : head_scan_out_kernel<false>, dim3(most_blocks, requests, heads * nv), 256, CHUNK_OUT_SMEM,
               stream, q, ldq, query_scale, k, ldk, v, ldv, gates, plane, skip, (const float*)products, cu_q, (const float*)sums, per, out, heads,
               groups, d, dv, nd, nv, divided, floor);
    return fe_check_launch("head_scan");
}

// The same for a step of one token a request (row r is request r's token), without a divisor: one kernel.
extern "C" int fe_head_step(const float* q, long long ldq, float query_scale, const float* k, long long ldk, const float* v, long long ldv,
                            const float* gates, long long plane, const float* skip, float* state, long long state_stride, const int* seats,
                            float* out, int requests, int heads, int groups, int d, int dv, int n_seats, cudaStream_t stream) {
    FE_REQUIRE(requests >= 0 && heads > 0 && heads <= 65535 && groups > 0 && heads % groups == 0 && d > 0 && dv > 0 && n_seats >= 0 &&
                   (long long)heads * d * dv <= state_stride && ldq >= (long long)groups * d && ldk >= (long long)groups * d && ldv >= (long long)heads * dv,
               "head_step: bad sizes (heads %d over %d, key size %d, value size %d)", heads, groups, d, dv);
    if (requests == 0) return 0;
    return launch_step<float, false>(q, ldq, query_scale, k, ldk, v, ldv, gates, plane, skip, state, state_stride, seats, out, requests, heads,
                                     groups, d, dv, n_seats, MemoryStep{}, stream);
}

// A step of one token a request of a matrix memory: proj float [requests, >= 2 heads d + 2 heads dv + 2 heads] = q | k | v | g | i | f with
// rows ld entries long; a seat holds S of every head, the heads' memories of the keys, their maxima; out [requests, heads dv].
extern "C" int fe_memory_decode(const float* proj, long long ld, const float* bias, float cap, float query_scale, float floor, float* state,
                                long long state_stride, const int* seats, const float* norm_weight, float eps, void* out, int requests,
                                int heads, int d, int dv, int n_seats, int dtype, cudaStream_t stream) {
    FE_REQUIRE(requests >= 0 && heads > 0 && heads <= 65535 && d > 0 && dv > 0 && n_seats >= 0 && cap > 0.f &&
                   (long long)heads * ((long long)d * dv + d + 1) <= state_stride && ld >= 2LL * heads * d + 2LL * heads * dv + 2 * heads,
               "memory_decode: bad sizes (heads %d, key size %d, value size %d)", heads, d, dv);
    FE_REQUIRE(dtype == FE_F32 || dtype == FE_BF16, "memory_decode: unknown dtype %d", dtype);
    if (requests == 0) return 0;
    const MemoryStep ms{bias, norm_weight, cap, floor, eps};
    const float* k = proj + (size_t)heads * d;
    const float* v = k + (size_t)heads * d;
    if (dtype == FE_F32)
        return launch_step<float, true>(proj, ld, query_scale, k, ld, v, ld, nullptr, 0, nullptr, state, state_stride, seats, out, requests,
                                        heads, heads, d, dv, n_seats, ms, stream);
    return launch_step<bf16, true>(proj, ld, query_scale, k, ld, v, ld, nullptr, 0, nullptr, state, state_stride, seats, out, requests, heads,
                                   heads, d, dv, n_seats, ms, stream);
}
