// The gated delta rule: per request and head a float state S [d, dv] that a token lets decay, corrects and reads,
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q .
// Kernels (all arithmetic float; everything comes from one float projection, rows q | k | v | g | b | a):
//   delta_prepare  short causal convolutions over time with a kept history, silu, unit vectors, decays and step sizes
//   delta_scan     the recurrence over the step's portions
//   delta_decode   a step of one token a request: everything between the projection and the output product in one kernel
//
// The recurrence takes B = 4 tokens at a time.  With P_i = g_1 .. g_i, D_ij = g_(j+1) .. g_i and S the state before the four,
//   u_i = beta_i (v_i - P_i S^T k_i - sum_(j<i) D_ij (k_i . k_j) u_j)
//   o_i = P_i S^T q_i + sum_(j<=i) D_ij (q_i . k_j) u_j
//   S  <- P_4 S + sum_j D_4j k_j u_j^T
// so the eight products with S are independent of one another and are added up over the warp together, and the numbers that
// do not depend on S (32 a block of four and head: ``coefs``) are made by delta_prepare.  Blocks are counted from the portion's
// start; tokens beyond its end have beta = 0, g = 1 and zero vectors, which change nothing.
#define FE_PDL_CLASS 128
#include "common.cuh"

using namespace fe;

namespace {

constexpr int B = 4;                     // tokens of a block
constexpr int COEFS = 32;                // its numbers: beta[4], beta P[4], P[4], E[4] = D_4j, beta M[6], N[10]
constexpr int C_BETA = 0, C_BP = 4, C_P = 8, C_E = 12, C_M = 16, C_N = 22;

__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float decay_of(float a, float dt_bias, float a_log) { return expf(-expf(a_log) * softplus(a + dt_bias)); }
__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// Block c of request r has row cu_q[r] / B + r + c of ``coefs``: the rows of different requests never meet.
__device__ __forceinline__ size_t coef_row(const int* __restrict__ cu_q, int r) { return (size_t)(cu_q[r] / B + r); }

// The convolution of channel ``ch`` at the portion's tokens i .. i + N - 1: rows before the portion come from the history (oldest
// first), tokens from n on count as zeros.  TAPS > 0: that many taps, every row asked for once and before any is used.
template <int TAPS, int N>
__device__ __forceinline__ void convolved(const float* __restrict__ first_row, long long ld, const float* __restrict__ conv, int taps, int C,
                                          const float* hist, int ch, int i, int n, float* acc) {
    if (TAPS > 0) {
        constexpr int K = TAPS > 0 ? TAPS : 1;
        float u[K - 1 + N], w[K];
#pragma unroll
        for (int j = 0; j < K; ++j) w[j] = conv[(size_t)j * C + ch];
#pragma unroll
        for (int x = 0; x < K - 1 + N; ++x) {
            const int from = i - (K - 1) + x;
            u[x] = 0.f;
            if (from >= 0) {
                if (from < n) u[x] = first_row[(size_t)from * ld + ch];
            } else if (hist) u[x] = hist[(size_t)(K - 1 + from) * C + ch];
        }
#pragma unroll
        for (int y = 0; y < N; ++y) {
            acc[y] = 0.f;
#pragma unroll
            for (int j = 0; j < K; ++j) acc[y] = fmaf(w[j], u[y + j], acc[y]);
        }
    } else {
        for (int y = 0; y < N; ++y) {
            acc[y] = 0.f;
            for (int j = 0; j < taps; ++j) {
                const int from = i + y - (taps - 1 - j);
                float u = 0.f;
                if (from >= 0) {
                    if (from < n) u = first_row[(size_t)from * ld + ch];
                } else if (hist) u = hist[(size_t)(taps - 1 + from) * C + ch];
                acc[y] = fmaf(conv[(size_t)j * C + ch], u, acc[y]);
            }
        }
    }
}

// The last taps - 1 projected rows of channel ``ch``, oldest first: what was kept moves up, the portion's n rows follow.
__device__ __forceinline__ void keep_history(const float* __restrict__ first_row, long long ld, int taps, int C, float* hist, int ch, int n) {
    const int back = taps - 1;
    for (int m = 0; m < back; ++m) {
        const int from = m + n;
        hist[(size_t)m * C + ch] = from < back ? hist[(size_t)from * C + ch] : first_row[(size_t)(from - back) * ld + ch];
    }
}

// ---------------------------------------------------------------------------------------------
// A warp per (tile of PREP_TILE tokens, unit): units 0 .. kv_heads - 1 are query/key heads (with the gates and the block numbers of
// the value heads that read them), the others value heads.  The warp of a portion's first tile brings its channels' history up
// to date after its reads; no other warp touches those channels' history.
constexpr int PREP_TILE = 8;
constexpr int PREP_WARPS = 4;

template <int TAPS>
__global__ void __launch_bounds__(PREP_WARPS * 32)
delta_prepare_kernel(const float* __restrict__ proj, long long ld, const float* __restrict__ conv, int taps, float* state,
                     long long state_stride, long long history_at, const int* __restrict__ seats, const int* __restrict__ cu_q,
                     const float* __restrict__ a_log, const float* __restrict__ dt_bias, float unit_eps, float query_scale,
                     float* __restrict__ out, float* __restrict__ coefs, int heads, int kv_heads, int d, int dv, int n_seats) {
    griddep_wait();
    griddep_launch_dependents();
    extern __shared__ float smem[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int r = blockIdx.y;
    const int first = cu_q[r], n = cu_q[r + 1] - first;
    const int i0 = blockIdx.x * PREP_TILE;
    if (i0 >= n) return;
    const int unit = blockIdx.z * PREP_WARPS + warp;
    if (unit >= kv_heads + heads) return;
    const int i1 = min(n, i0 + PREP_TILE);
    const int C = 2 * kv_heads * d + heads * dv;
    const int seat = seats[r];
    float* hist = (taps > 1 && seat >= 0 && seat < n_seats) ? state + (size_t)seat * state_stride + history_at : nullptr;
    const float* rows = proj + (size_t)first * ld;
    if (unit >= kv_heads) {                              // a value head: convolution and silu
        const int ch0 = 2 * kv_heads * d + (unit - kv_heads) * dv;
        for (int c = lane; c < dv; c += 32) {
            float acc[PREP_TILE];
            convolved<TAPS, PREP_TILE>(rows, ld, conv, taps, C, hist, ch0 + c, i0, n, acc);
#pragma unroll
            for (int y = 0; y < PREP_TILE; ++y)
                if (i0 + y < i1) out[(size_t)(first + i0 + y) * C + ch0 + c] = silu(acc[y]);
        }
        if (hist && i0 == 0)
            for (int c = lane; c < dv; c += 32) keep_history(rows, ld, taps, C, hist, ch0 + c, n);
        return;
    }
    float* qs = smem + (size_t)warp * 2 * B * d;         // [B][d] of the block at hand
    float* ks = qs + B * d;
    const int q0 = unit * d, k0 = (kv_heads + unit) * d, ratio = heads / kv_heads;
    for (int b0 = i0; b0 < i1; b0 += B) {
        float sq[B], sk[B];
#pragma unroll
        for (int i = 0; i < B; ++i) sq[i] = sk[i] = 0.f;
        for (int c = lane; c < d; c += 32) {             // a lane reads back what it wrote: its own channels
            float q[B], k[B];
            convolved<TAPS, B>(rows, ld, conv, taps, C, hist, q0 + c, b0, n, q);
            convolved<TAPS, B>(rows, ld, conv, taps, C, hist, k0 + c, b0, n, k);
#pragma unroll
            for (int i = 0; i < B; ++i) {
                const bool in = b0 + i < n;
                q[i] = in ? silu(q[i]) : 0.f;
                k[i] = in ? silu(k[i]) : 0.f;
                qs[i * d + c] = q[i];
                ks[i * d + c] = k[i];
                sq[i] = fmaf(q[i], q[i], sq[i]);
                sk[i] = fmaf(k[i], k[i], sk[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < B; ++i) {
            sq[i] = query_scale * rsqrtf(warp_sum(sq[i]) + unit_eps);
            sk[i] = rsqrtf(warp_sum(sk[i]) + unit_eps);
        }
        for (int c = lane; c < d; c += 32) {
#pragma unroll
            for (int i = 0; i < B; ++i) {
                const float q = qs[i * d + c] *= sq[i], k = ks[i * d + c] *= sk[i];
                if (b0 + i < n) {
                    out[(size_t)(first + b0 + i) * C + q0 + c] = q;
                    out[(size_t)(first + b0 + i) * C + k0 + c] = k;
                }
            }
        }
        __syncwarp();
        float kk[6], qk[10];
#pragma unroll
        for (int x = 0; x < 6; ++x) kk[x] = 0.f;
#pragma unroll
        for (int x = 0; x < 10; ++x) qk[x] = 0.f;
        for (int c = lane; c < d; c += 32) {
            float kc[B], qc[B];
#pragma unroll
            for (int i = 0; i < B; ++i) kc[i] = ks[i * d + c], qc[i] = qs[i * d + c];
#pragma unroll
            for (int i = 0; i < B; ++i)
#pragma unroll
                for (int j = 0; j <= i; ++j) {
                    qk[i * (i + 1) / 2 + j] = fmaf(qc[i], kc[j], qk[i * (i + 1) / 2 + j]);
                    if (j < i) kk[i * (i - 1) / 2 + j] = fmaf(kc[i], kc[j], kk[i * (i - 1) / 2 + j]);
                }
        }
#pragma unroll
        for (int x = 0; x < 6; ++x) kk[x] = warp_sum(kk[x]);
#pragma unroll
        for (int x = 0; x < 10; ++x) qk[x] = warp_sum(qk[x]);
        for (int hh = lane; hh < ratio; hh += 32) {
            const int head = unit * ratio + hh;
            float g[B], beta[B];
#pragma unroll
            for (int i = 0; i < B; ++i) {
                g[i] = 1.f;
                beta[i] = 0.f;
                if (b0 + i < n) {
                    const float* row = rows + (size_t)(b0 + i) * ld + C + (size_t)heads * dv;
                    beta[i] = sigmoid(row[head]);
                    g[i] = decay_of(row[heads + head], dt_bias[head], a_log[head]);
                }
            }
            float* to = coefs + ((coef_row(cu_q, r) + b0 / B) * heads + head) * COEFS;
            float P = 1.f;
#pragma unroll
            for (int i = 0; i < B; ++i) {
                P *= g[i];
                to[C_BETA + i] = beta[i];
                to[C_BP + i] = beta[i] * P;
                to[C_P + i] = P;
                float D = 1.f;                            // D_ij from j = i downwards
#pragma unroll
                for (int j = i; j >= 0; --j) {
                    to[C_N + i * (i + 1) / 2 + j] = D * qk[i * (i + 1) / 2 + j];
                    if (j < i) to[C_M + i * (i - 1) / 2 + j] = beta[i] * D * kk[i * (i - 1) / 2 + j];
                    if (i == B - 1) to[C_E + j] = D;
                    D *= g[j];
                }
            }
        }
        __syncwarp();
    }
    if (hist && i0 == 0) {
        for (int c = lane; c < d; c += 32) {
            keep_history(rows, ld, taps, C, hist, q0 + c, n);
            keep_history(rows, ld, taps, C, hist, k0 + c, n);
        }
    }
}

// ---------------------------------------------------------------------------------------------
// The recurrence.  A block owns a slice of the value channels of one (request, head); the lanes of a warp are 16 groups of key
// channels x 2 pairs of value channels, and a thread keeps 4 NX key channels (four neighbours in each stretch of 64) of two value
// channels of the state in registers (d <= 64 NX; channels beyond d are zeros), so that the queries and keys it reads from shared
// memory serve two columns.  Odd groups take the pair's columns in the other order, so that the first round of the sums over the
// groups gives away every lane's second column.  The products with the queries are added up after the corrections u are on their
// way: nothing but the outputs waits for them.  The keys and queries of the next four tokens are read from shared memory while
// these four are worked on.  Tiles of SCAN_BLOCKS blocks of four tokens are copied into the other half of shared memory (cp.async)
// while this one is walked.
constexpr int SCAN_BLOCKS = 8;
constexpr int SCAN_TILE = SCAN_BLOCKS * B;

template <int BYTES> __device__ __forceinline__ void copy_async(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    if (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

// Multiply-adds of two floats at once.
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) { return __ffma2_rn(a, b, c); }
__device__ __forceinline__ float2 both(float x) { return make_float2(x, x); }

template <int NX, bool VEC>
__global__ void __launch_bounds__(128)
delta_scan_kernel(const float* __restrict__ qkv, const float* __restrict__ coefs, float* state, long long state_stride,
                  const int* __restrict__ seats, const int* __restrict__ cu_q, float* __restrict__ out, int heads, int kv_heads, int d,
                  int dv, int n_seats) {
    griddep_wait();
    griddep_launch_dependents();
    constexpr int ROW = 64 * NX;
    constexpr int STEP = VEC ? 4 : 1;
    extern __shared__ __align__(16) float smem[];
    const int columns = (blockDim.x >> 5) * 4;
    const int stage_floats = SCAN_TILE * (2 * ROW + columns) + SCAN_BLOCKS * COEFS;
    const int req = blockIdx.x, head = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int group = lane & 15, odd = group & 1;
    const int la = warp * 4 + (lane >> 4) * 2 + odd, lb = la + 1 - 2 * odd;      // this lane's first and second column
    const int j0 = blockIdx.z * columns, ja = j0 + la, jb = j0 + lb;
    const bool own0 = ja < dv, own1 = jb < dv;
    const int seat = seats[req];
    float* mine = (seat >= 0 && seat < n_seats) ? state + (size_t)seat * state_stride + (size_t)head * d * dv : nullptr;
    float2 S0[2 * NX], S1[2 * NX];                       // pairs of key channels of this lane's first and second column
    auto state_at = [&](int x, int e) { return x * 64 + group * 4 + e; };
#pragma unroll
    for (int x = 0; x < NX; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = state_at(x, e);
            const float p = (own0 && i < d && mine) ? mine[(size_t)i * dv + ja] : 0.f;
            const float q = (own1 && i < d && mine) ? mine[(size_t)i * dv + jb] : 0.f;
            if (e & 1) S0[2 * x + (e >> 1)].y = p, S1[2 * x + (e >> 1)].y = q;
            else S0[2 * x + (e >> 1)].x = p, S1[2 * x + (e >> 1)].x = q;
        }
    for (int e = threadIdx.x; e < 2 * stage_floats; e += blockDim.x) smem[e] = 0.f;
    const int first = cu_q[req], n = cu_q[req + 1] - first;
    const int C = 2 * kv_heads * d + heads * dv;
    const float* qrows = qkv + (size_t)first * C + (size_t)(head / (heads / kv_heads)) * d;
    const float* krows = qrows + (size_t)kv_heads * d;
    const float* vrows = qkv + (size_t)first * C + 2 * (size_t)kv_heads * d + (size_t)head * dv + j0;
    const float* crows = coefs + (coef_row(cu_q, req) * heads + head) * COEFS;
    const int vcols = min(columns, dv - j0);
    __syncthreads();
    // rows of a tile beyond the portion's end are cleared: they meet beta = 0 and must be finite
    auto fetch = [&](int t0, float* stage) {
        const int count = min(SCAN_TILE, n - t0);
        float *qs = stage, *ks = qs + SCAN_TILE * ROW, *vs = ks + SCAN_TILE * ROW, *cs = vs + SCAN_TILE * columns;
        const int per = d / STEP;
        for (int e = threadIdx.x; e < SCAN_TILE * per; e += blockDim.x) {
            const int tt = e / per, i = (e - tt * per) * STEP;
            const int to = tt * ROW + i;
            if (tt < count) {
                copy_async<STEP * 4>(qs + to, qrows + (size_t)(t0 + tt) * C + i);
                copy_async<STEP * 4>(ks + to, krows + (size_t)(t0 + tt) * C + i);
            } else {
#pragma unroll
                for (int x = 0; x < STEP; ++x) qs[to + x] = ks[to + x] = 0.f;
            }
        }
        const int vper = (vcols + STEP - 1) / STEP;
        for (int e = threadIdx.x; e < SCAN_TILE * vper; e += blockDim.x) {
            const int tt = e / vper, c = (e - tt * vper) * STEP;
            if (tt < count) copy_async<STEP * 4>(vs + tt * columns + c, vrows + (size_t)(t0 + tt) * C + c);
            else {
#pragma unroll
                for (int x = 0; x < STEP; ++x) vs[tt * columns + c + x] = 0.f;
            }
        }
        const int pieces = (count + B - 1) / B * (COEFS / 4);
        for (int e = threadIdx.x; e < pieces; e += blockDim.x) {
            const int b = e / (COEFS / 4), x = (e - b * (COEFS / 4)) * 4;
            copy_async<16>(cs + b * COEFS + x, crows + (size_t)(t0 / B + b) * heads * COEFS + x);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (n > 0) fetch(0, smem);
    const int of_token = ((group >> 1) & 1) * 2 + ((group >> 2) & 1);            // whose sums this lane ends with, in its first column
    // eight sums (token by token, first column then second) over the sixteen groups of key channels: three rounds in which a lane
    // gives half of its sums away and adds the partner's to the other half, and one that adds the two halves of the groups
    auto over_groups = [&](const float (&r)[2 * B]) {
        float r4[4], r2[2];
#pragma unroll
        for (int i = 0; i < 4; ++i) r4[i] = r[2 * i] + __shfl_xor_sync(0xffffffffu, r[2 * i + 1], 1);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const float keep = group & 2 ? r4[2 + i] : r4[i], give = group & 2 ? r4[i] : r4[2 + i];
            r2[i] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
        }
        const float keep = group & 4 ? r2[1] : r2[0], give = group & 4 ? r2[0] : r2[1];
        const float sum = keep + __shfl_xor_sync(0xffffffffu, give, 4);
        return sum + __shfl_xor_sync(0xffffffffu, sum, 8);
    };
    float* orow = out + (size_t)first * heads * dv + (size_t)head * dv + ja;
    float4 kn[B][NX], qn[B][NX];                          // the next block's keys and queries
    auto ahead_k = [&](const float* ks) {
#pragma unroll
        for (int i = 0; i < B; ++i)
#pragma unroll
            for (int x = 0; x < NX; ++x) kn[i][x] = *reinterpret_cast<const float4*>(ks + i * ROW + x * 64 + group * 4);
    };
    auto ahead_q = [&](const float* qs) {
#pragma unroll
        for (int i = 0; i < B; ++i)
#pragma unroll
            for (int x = 0; x < NX; ++x) qn[i][x] = *reinterpret_cast<const float4*>(qs + i * ROW + x * 64 + group * 4);
    };
    // a block's first rows, its numbers and first token; ``more``: another block of this tile follows
    auto walk = [&](const float* qs, const float* ks, const float* vs, const float* cf, int t, bool more) {
        float4 k4[B][NX];
        float r[2 * B];
#pragma unroll
        for (int i = 0; i < B; ++i)
#pragma unroll
            for (int x = 0; x < NX; ++x) k4[i][x] = kn[i][x];
        if (more) ahead_k(ks + B * ROW);
#pragma unroll
        for (int i = 0; i < B; ++i) {
            float2 k0, k1;
#pragma unroll
            for (int x = 0; x < NX; ++x) {
                const float2 ka = make_float2(k4[i][x].x, k4[i][x].y), kb = make_float2(k4[i][x].z, k4[i][x].w);
                k0 = x == 0 ? __fmul2_rn(ka, S0[0]) : fma2(ka, S0[2 * x], k0);
                k1 = x == 0 ? __fmul2_rn(ka, S1[0]) : fma2(ka, S1[2 * x], k1);
                k0 = fma2(kb, S0[2 * x + 1], k0);
                k1 = fma2(kb, S1[2 * x + 1], k1);
            }
            r[2 * i] = k0.x + k0.y, r[2 * i + 1] = k1.x + k1.y;
        }
        const float ksum = over_groups(r);
#pragma unroll
        for (int i = 0; i < B; ++i) {
            float2 q0, q1;
#pragma unroll
            for (int x = 0; x < NX; ++x) {
                const float2 qa = make_float2(qn[i][x].x, qn[i][x].y), qb = make_float2(qn[i][x].z, qn[i][x].w);
                q0 = x == 0 ? __fmul2_rn(qa, S0[0]) : fma2(qa, S0[2 * x], q0);
                q1 = x == 0 ? __fmul2_rn(qa, S1[0]) : fma2(qa, S1[2 * x], q1);
                q0 = fma2(qb, S0[2 * x + 1], q0);
                q1 = fma2(qb, S1[2 * x + 1], q1);
            }
            r[2 * i] = q0.x + q0.y, r[2 * i + 1] = q1.x + q1.y;
        }
        if (more) ahead_q(qs + B * ROW);
        const float4 beta = *reinterpret_cast<const float4*>(cf + C_BETA), bp = *reinterpret_cast<const float4*>(cf + C_BP);
        const float4 m4 = *reinterpret_cast<const float4*>(cf + C_M);
        const float2 m2 = *reinterpret_cast<const float2*>(cf + C_M + 4);
        const float bb[B] = {beta.x, beta.y, beta.z, beta.w}, pp[B] = {bp.x, bp.y, bp.z, bp.w};
        const float mm[6] = {m4.x, m4.y, m4.z, m4.w, m2.x, m2.y};
        float ua[B], ub[B];                              // of the first and the second column
#pragma unroll
        for (int i = 0; i < B; ++i) {
            const int from = (lane & 16) + (i >> 1) * 2 + (i & 1) * 4;                // the lane with token i's sums, even group
            ua[i] = fmaf(-pp[i], __shfl_sync(0xffffffffu, ksum, from + odd), bb[i] * vs[i * columns + la]);
            ub[i] = fmaf(-pp[i], __shfl_sync(0xffffffffu, ksum, from + 1 - odd), bb[i] * vs[i * columns + lb]);
        }
#pragma unroll
        for (int i = 1; i < B; ++i)
#pragma unroll
            for (int m = 0; m < i; ++m) {
                ua[i] = fmaf(-mm[i * (i - 1) / 2 + m], ua[m], ua[i]);
                ub[i] = fmaf(-mm[i * (i - 1) / 2 + m], ub[m], ub[i]);
            }
        const float qsum = over_groups(r);
        const float* N = cf + C_N + of_token * (of_token + 1) / 2;
        float o = cf[C_P + of_token] * qsum;
#pragma unroll
        for (int m = 0; m < B; ++m) o = fmaf(m <= of_token ? N[m] : 0.f, ua[m], o);
        if (group < 8 && own0 && t + of_token < n) orow[(size_t)(t + of_token) * heads * dv] = o;
        const float2 P2 = both(cf[C_P + B - 1]);
        const float4 e4 = *reinterpret_cast<const float4*>(cf + C_E);
        const float ee[B] = {e4.x, e4.y, e4.z, e4.w};
        float2 wa[B], wb[B];
#pragma unroll
        for (int i = 0; i < B; ++i) wa[i] = both(ua[i] * ee[i]), wb[i] = both(ub[i] * ee[i]);
#pragma unroll
        for (int x = 0; x < NX; ++x)
#pragma unroll
            for (int y = 0; y < 2; ++y) {
                float2 s0 = __fmul2_rn(P2, S0[2 * x + y]), s1 = __fmul2_rn(P2, S1[2 * x + y]);
#pragma unroll
                for (int i = 0; i < B; ++i) {
                    const float2 kp = y == 0 ? make_float2(k4[i][x].x, k4[i][x].y) : make_float2(k4[i][x].z, k4[i][x].w);
                    s0 = fma2(kp, wa[i], s0);
                    s1 = fma2(kp, wb[i], s1);
                }
                S0[2 * x + y] = s0;
                S1[2 * x + y] = s1;
            }
    };
    for (int t0 = 0, at = 0; t0 < n; t0 += SCAN_TILE, at ^= 1) {
        if (t0 + SCAN_TILE < n) {
            fetch(t0 + SCAN_TILE, smem + (at ^ 1) * stage_floats);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* stage = smem + at * stage_floats;
        const float *qs = stage, *ks = qs + SCAN_TILE * ROW, *vs = ks + SCAN_TILE * ROW, *cs = vs + SCAN_TILE * columns;
        ahead_k(ks);
        ahead_q(qs);
        if (t0 + SCAN_TILE <= n) {                       // a full tile, unrolled: a block's loads and outputs fill its neighbours' waits
#pragma unroll
            for (int b = 0; b < SCAN_BLOCKS; ++b)
                walk(qs + b * B * ROW, ks + b * B * ROW, vs + b * B * columns, cs + b * COEFS, t0 + b * B, b + 1 < SCAN_BLOCKS);
        } else {
#pragma unroll 1
            for (int b = 0; t0 + b * B < n; ++b)
                walk(qs + b * B * ROW, ks + b * B * ROW, vs + b * B * columns, cs + b * COEFS, t0 + b * B, b + 1 < SCAN_BLOCKS);
        }
        __syncthreads();                                 // everyone is done with this half before it is filled again
    }
    if (mine) {
#pragma unroll
        for (int x = 0; x < NX; ++x)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = state_at(x, e);
                if (i >= d) continue;
                if (own0) mine[(size_t)i * dv + ja] = e & 1 ? S0[2 * x + (e >> 1)].y : S0[2 * x + (e >> 1)].x;
                if (own1) mine[(size_t)i * dv + jb] = e & 1 ? S1[2 * x + (e >> 1)].y : S1[2 * x + (e >> 1)].x;
            }
    }
}

template <int NX, bool VEC>
int launch_scan(const float* qkv, const float* coefs, float* state, long long state_stride, const int* seats, const int* cu_q, float* out,
                int requests, int heads, int kv_heads, int d, int dv, int n_seats, cudaStream_t stream) {
    // Blocks of four warps, sixteen value channels: two of them fit a multiprocessor, so that up to two warps a scheduler hide one
    // another's waits; fewer warps a block would copy the queries and keys of all key channels more often than that is worth.
    const int head_warps = (dv + 3) / 4, warps = head_warps < 4 ? head_warps : 4, slices = (head_warps + warps - 1) / warps;
    const size_t smem = 2 * ((size_t)SCAN_TILE * (2 * 64 * NX + warps * 4) + SCAN_BLOCKS * COEFS) * sizeof(float);
    if (smem > 48 * 1024) {
        const cudaError_t err = cudaFuncSetAttribute(delta_scan_kernel<NX, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        FE_REQUIRE(err == cudaSuccess, "delta_scan: %s", cudaGetErrorString(err));
    }
    fe::launch(delta_scan_kernel<NX, VEC>, dim3(requests, heads, slices), warps * 32, smem, stream, qkv, coefs, state, state_stride, seats,
               cu_q, out, heads, kv_heads, d, dv, n_seats);
    return fe_check_launch("delta_scan");
}

// ---------------------------------------------------------------------------------------------
// A step of ONE token a request.  The value heads that read one query/key head are shared out over the blocks of a thread-block
// cluster (``each`` heads a block); every block makes the query and key for itself, and the first one renews the convolutions'
// history of their channels after a cluster barrier behind which every block has read it.  A block's threads are ``groups`` runs
// of PER key channels x ``columns`` value channels; a state is read once into registers, asked for before anything else, and
// written once.
constexpr int PER = 16;

template <typename T>
__global__ void __launch_bounds__(1024)
delta_decode_kernel(const float* __restrict__ proj, long long ld, const float* __restrict__ conv, int taps, float* state,
                    long long state_stride, long long history_at, const int* __restrict__ seats, const float* __restrict__ a_log,
                    const float* __restrict__ dt_bias, const float* __restrict__ norm_weight, float eps, float unit_eps, float query_scale,
                    T* __restrict__ out, int heads, int kv_heads, int d, int dv, int n_seats, int groups, int each) {
    griddep_wait();
    griddep_launch_dependents();
    extern __shared__ __align__(16) float smem[];
    const int total = each * dv, columns = blockDim.x / groups;
    float* qs = smem;                               // [d]
    float* ks = qs + d;                             // [d]
    float* vs = ks + d;                             // [total]: values, later the outputs
    float* gate = vs + total;                       // [2 each]: decays, step sizes
    float* part = gate + 2 * each;                  // [2][groups][columns]
    float* red = part + 2 * groups * columns;       // [4]: the factors of q and k, k . q
    const int slice = blockIdx.x, kvh = blockIdx.y, r = blockIdx.z;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
    const int head0 = kvh * (heads / kv_heads) + slice * each;
    const int C = 2 * kv_heads * d + heads * dv;
    const float* row = proj + (size_t)r * ld;
    const int seat = seats[r];
    float* base = (seat >= 0 && seat < n_seats) ? state + (size_t)seat * state_stride : nullptr;
    float* hist = (taps > 1 && base) ? base + history_at : nullptr;
    const int g = tid / columns, jj = tid - g * columns, i0 = g * PER;
    float S[PER];
    auto column_of = [&](int col) -> float* {
        const int hh = col / dv;
        return base ? base + (size_t)(head0 + hh) * d * dv + (col - hh * dv) : nullptr;
    };
    auto ask = [&](int c0) {
        const int col = c0 + jj;
        const float* from = (g < groups && col < total) ? column_of(col) : nullptr;
#pragma unroll
        for (int x = 0; x < PER; ++x) S[x] = (from && i0 + x < d) ? from[(size_t)(i0 + x) * dv] : 0.f;
    };
    ask(0);
    const int v0 = 2 * kv_heads * d + head0 * dv;
    for (int c = tid; c < 2 * d + total; c += blockDim.x) {
        const int ch = c < d ? kvh * d + c : (c < 2 * d ? (kv_heads + kvh) * d + c - d : v0 + c - 2 * d);
        float acc;
        convolved<0, 1>(row, ld, conv, taps, C, hist, ch, 0, 1, &acc);
        smem[c] = silu(acc);
        if (hist && c >= 2 * d) keep_history(row, ld, taps, C, hist, ch, 1);     // a value channel is this thread's alone
    }
    for (int hh = tid; hh < each; hh += blockDim.x) {
        const float* b = row + C + (size_t)heads * dv;
        gate[each + hh] = sigmoid(b[head0 + hh]);
        gate[hh] = decay_of(b[heads + head0 + hh], dt_bias[head0 + hh], a_log[head0 + hh]);
    }
    __syncthreads();
    asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");       // this block has read the history of q and k
    if (warp == 0) {
        float sq = 0.f, sk = 0.f, dot = 0.f;
        for (int i = lane; i < d; i += 32) {
            sq = fmaf(qs[i], qs[i], sq);
            sk = fmaf(ks[i], ks[i], sk);
            dot = fmaf(qs[i], ks[i], dot);
        }
        const float fq = query_scale * rsqrtf(warp_sum(sq) + unit_eps), fk = rsqrtf(warp_sum(sk) + unit_eps);
        dot = warp_sum(dot);
        if (lane == 0) red[0] = fq, red[1] = fk, red[2] = dot * fq * fk;
    }
    for (int c0 = 0; c0 < total; c0 += columns) {
        const int col = c0 + jj;
        const bool own = g < groups && col < total;
        const int hh = own ? col / dv : 0;
        float ak = 0.f, aq = 0.f;
#pragma unroll
        for (int x = 0; x < PER; ++x) {
            if (i0 + x < d) {
                ak = fmaf(ks[i0 + x], S[x], ak);
                aq = fmaf(qs[i0 + x], S[x], aq);
            }
        }
        if (g < groups) {
            part[g * columns + jj] = ak;
            part[(groups + g) * columns + jj] = aq;
        }
        __syncthreads();
        const float fq = red[0], fk = red[1], dot = red[2];
        float o = 0.f;
        if (own) {
            float sk = 0.f;
            for (int x = 0; x < groups; ++x) sk += part[x * columns + jj];
            const float decay = gate[hh];
            const float u = gate[each + hh] * (vs[col] - decay * (sk * fk)), w = u * fk;
            float* mine = column_of(col);
            if (mine) {
#pragma unroll
                for (int x = 0; x < PER; ++x)
                    if (i0 + x < d) mine[(size_t)(i0 + x) * dv] = fmaf(decay, S[x], ks[i0 + x] * w);
            }
            if (g == 0) {
                float sq = 0.f;
                for (int x = 0; x < groups; ++x) sq += part[(groups + x) * columns + jj];
                o = fmaf(decay, sq * fq, dot * u);
            }
        }
        if (c0 + columns < total) ask(c0 + columns);
        __syncthreads();                                  // every run of this column has read its value and the sums
        if (g == 0 && own) vs[col] = o;
    }
    __syncthreads();
    // every head divided by its root mean square, times the weight, times silu of its gate row
    const float* grow = row + C + (size_t)head0 * dv;
    T* to = out + (size_t)r * heads * dv + (size_t)head0 * dv;
    for (int hh = warp; hh < each; hh += warps) {
        float ss = 0.f;
        for (int j = lane; j < dv; j += 32) ss = fmaf(vs[hh * dv + j], vs[hh * dv + j], ss);
        const float inv = rsqrtf(warp_sum(ss) / (float)dv + eps);
        for (int j = lane; j < dv; j += 32) to[hh * dv + j] = from_float<T>(vs[hh * dv + j] * inv * norm_weight[j] * silu(grow[hh * dv + j]));
    }
    __syncthreads();
    asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
    if (hist && slice == 0)
        for (int c = tid; c < 2 * d; c += blockDim.x) keep_history(row, ld, taps, C, hist, c < d ? kvh * d + c : (kv_heads + kvh) * d + c - d, 1);
}

template <typename T>
int launch_decode(const float* proj, long long ld, const float* conv, int taps, float* state, long long state_stride, long long history_at,
                  const int* seats, const float* a_log, const float* dt_bias, const float* norm_weight, float eps, float unit_eps,
                  float query_scale, void* out, int requests, int heads, int kv_heads, int d, int dv, int n_seats, cudaStream_t stream) {
    const int ratio = heads / kv_heads, groups = (d + PER - 1) / PER;
    int slices = ratio < 8 ? ratio : 8;                   // a cluster of up to eight blocks (the portable size) for a query/key head
    while (ratio % slices) --slices;
    const int each = ratio / slices, total = each * dv;
    int columns = (total + 31) / 32 * 32;
    const int most = 1024 / groups / 32 * 32;
    columns = columns > most ? most : columns;
    const size_t smem = (2 * (size_t)d + total + 2 * each + 2 * (size_t)groups * columns + 4) * sizeof(float);
    FE_REQUIRE(smem <= 200 * 1024, "delta_decode: %d value channels a block need more shared memory than it has", total);
    if (smem > 48 * 1024) {
        const cudaError_t err = cudaFuncSetAttribute(delta_decode_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        FE_REQUIRE(err == cudaSuccess, "delta_decode: %s", cudaGetErrorString(err));
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(slices, kv_heads, requests);
    cfg.blockDim = dim3(groups * columns);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = slices;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    const cudaError_t err = cudaLaunchKernelEx(&cfg, delta_decode_kernel<T>, proj, ld, conv, taps, state, state_stride, history_at, seats, a_log,
                                               dt_bias, norm_weight, eps, unit_eps, query_scale, (T*)out, heads, kv_heads, d, dv, n_seats, groups,
                                               each);
    FE_REQUIRE(err == cudaSuccess, "delta_decode (cluster of %d): %s", slices, cudaGetErrorString(err));
    return fe_check_launch("delta_decode");
}

}  // namespace

extern "C" int fe_delta_block_tokens() { return B; }
extern "C" int fe_delta_block_numbers() { return COEFS; }

// proj float [T, >= C + heads dv + 2 heads] (rows ld entries long): q | k | v (C channels: kv_heads heads of d twice, heads of dv),
// g, then b and a (one number a head); conv float [taps, C]; state float [n_seats, state_stride] with the histories (taps - 1 rows of
// C) at history_at; out float [T, C]; coefs float [T / 4 + requests, heads, 32]; most_tokens: the longest portion or more.
extern "C" int fe_delta_prepare(const float* proj, long long ld, const float* conv, int taps, float* state, long long state_stride,
                                long long history_at, const int* seats, const int* cu_q, const float* a_log, const float* dt_bias,
                                float unit_eps, float query_scale, float* out, float* coefs, int requests, int most_tokens, int heads,
                                int kv_heads, int d, int dv, int n_seats, cudaStream_t stream) {
    const long long C = 2LL * kv_heads * d + (long long)heads * dv;
    FE_REQUIRE(requests >= 0 && requests <= 65535 && most_tokens >= 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && d > 0 && dv > 0 &&
                   taps >= 1 && n_seats >= 0 && ld >= C + (long long)heads * dv + 2 * heads &&
                   history_at >= (long long)heads * d * dv && history_at + (taps - 1) * C <= state_stride,
               "delta_prepare: bad sizes (heads %d over %d, key size %d, value size %d, %d taps)", heads, kv_heads, d, dv, taps);
    if (requests == 0 || most_tokens == 0) return 0;
    FE_REQUIRE(taps - 1 <= PREP_TILE, "delta_prepare: %d taps; only a portion's first %d tokens may read the history", taps, PREP_TILE);
    const int tiles = (most_tokens + PREP_TILE - 1) / PREP_TILE, units = (kv_heads + heads + PREP_WARPS - 1) / PREP_WARPS;
    const size_t smem = (size_t)PREP_WARPS * 2 * B * d * sizeof(float);
    FE_REQUIRE(smem <= 48 * 1024 && units <= 65535, "delta_prepare: key size %d (up to 384) or %d heads", d, heads);
#define FE_DELTA_PREPARE(TAPS)                                                                                                       \
    fe::launch(delta_prepare_kernel<TAPS>, dim3(tiles, requests, units), PREP_WARPS * 32, smem, stream, proj, ld, conv, taps, state, \
               state_stride, history_at, seats, cu_q, a_log, dt_bias, unit_eps, query_scale, out, coefs, heads, kv_heads, d, dv, n_seats)
    if (taps == 2) FE_DELTA_PREPARE(2);
    else if (taps == 3) FE_DELTA_PREPARE(3);
    else if (taps == 4) FE_DELTA_PREPARE(4);
    else FE_DELTA_PREPARE(0);
#undef FE_DELTA_PREPARE
    return fe_check_launch("delta_prepare");
}

// qkv and coefs as fe_delta_prepare leaves them; out float [T, heads dv].
extern "C" int fe_delta_scan(const float* qkv, const float* coefs, float* state, long long state_stride, const int* seats, const int* cu_q,
                             float* out, int requests, int heads, int kv_heads, int d, int dv, int n_seats, cudaStream_t stream) {
    FE_REQUIRE(requests >= 0 && heads > 0 && heads <= 65535 && kv_heads > 0 && heads % kv_heads == 0 && d > 0 && d <= 256 && dv > 0 && n_seats >= 0 &&
                   (long long)heads * d * dv <= state_stride,
               "delta_scan: bad sizes (heads %d over %d, key size %d up to 256, value size %d)", heads, kv_heads, d, dv);
    if (requests == 0) return 0;
    const long long C = 2LL * kv_heads * d + (long long)heads * dv;
    const bool vec = d % 4 == 0 && dv % 4 == 0 && C % 4 == 0 && (((size_t)qkv | (size_t)coefs) & 15) == 0;
#define FE_DELTA_SCAN(NX)                                                                                                            \
    return vec ? launch_scan<NX, true>(qkv, coefs, state, state_stride, seats, cu_q, out, requests, heads, kv_heads, d, dv, n_seats, stream) \
               : launch_scan<NX, false>(qkv, coefs, state, state_stride, seats, cu_q, out, requests, heads, kv_heads, d, dv, n_seats, stream)
    if (d <= 64) { FE_DELTA_SCAN(1); }
    if (d <= 128) { FE_DELTA_SCAN(2); }
    FE_DELTA_SCAN(4);
#undef FE_DELTA_SCAN
}

// A step of one token a request in one kernel: proj, conv, state as fe_delta_prepare takes them (row r is request r's token); out
// [requests, heads dv] in ``dtype``: every head's output divided by its root mean square, times norm_weight [dv], times silu(g).
extern "C" int fe_delta_decode(const float* proj, long long ld, const float* conv, int taps, float* state, long long state_stride,
                               long long history_at, const int* seats, const float* a_log, const float* dt_bias, const float* norm_weight,
                               float eps, float unit_eps, float query_scale, void* out, int requests, int heads, int kv_heads, int d, int dv,
                               int n_seats, int dtype, cudaStream_t stream) {
    const long long C = 2LL * kv_heads * d + (long long)heads * dv;
    FE_REQUIRE(requests >= 0 && requests <= 65535 && heads > 0 && kv_heads > 0 && kv_heads <= 65535 && heads % kv_heads == 0 && d > 0 && d <= 512 && dv > 0 && taps >= 1 &&
                   n_seats >= 0 && ld >= C + (long long)heads * dv + 2 * heads && history_at >= (long long)heads * d * dv &&
                   history_at + (taps - 1) * C <= state_stride,
               "delta_decode: bad sizes (heads %d over %d, key size %d up to 512, value size %d, %d taps)", heads, kv_heads, d, dv, taps);
    FE_REQUIRE(dtype == FE_F32 || dtype == FE_BF16, "delta_decode: unknown dtype %d", dtype);
    if (requests == 0) return 0;
    if (dtype == FE_F32)
        return launch_decode<float>(proj, ld, conv, taps, state, state_stride, history_at, seats, a_log, dt_bias, norm_weight, eps, unit_eps,
                                    query_scale, out, requests, heads, kv_heads, d, dv, n_seats, stream);
    return launch_decode<bf16>(proj, ld, conv, taps, state, state_stride, history_at, seats, a_log, dt_bias, norm_weight, eps, unit_eps,
                               query_scale, out, requests, heads, kv_heads, d, dv, n_seats, stream);
}
