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

// The convolution of channel ``ch`` at the portion's token i: rows before the portion come from the history (oldest first).
__device__ __forceinline__ float convolved(const float* __restrict__ first_row, long long ld, const float* __restrict__ conv, int taps, int C,
                                           const float* hist, int ch, int i) {
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {
        const int from = i - (taps - 1 - j);
        float u = 0.f;
        if (from >= 0) u = first_row[(size_t)from * ld + ch];
        else if (hist) u = hist[(size_t)(taps - 1 + from) * C + ch];
        acc = fmaf(conv[(size_t)j * C + ch], u, acc);
    }
    return acc;
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
        for (int i = i0; i < i1; ++i)
            for (int c = lane; c < dv; c += 32)
                out[(size_t)(first + i) * C + ch0 + c] = silu(convolved(rows, ld, conv, taps, C, hist, ch0 + c, i));
        if (hist && i0 == 0)
            for (int c = lane; c < dv; c += 32) keep_history(rows, ld, taps, C, hist, ch0 + c, n);
        return;
    }
    float* qs = smem + (size_t)warp * 2 * B * d;         // [B][d] of the block at hand
    float* ks = qs + B * d;
    const int q0 = unit * d, k0 = (kv_heads + unit) * d, ratio = heads / kv_heads;
    for (int b0 = i0; b0 < i1; b0 += B) {
        for (int i = b0; i < b0 + B; ++i) {
            float* q = qs + (i - b0) * d;
            float* k = ks + (i - b0) * d;
            if (i >= n) {
                for (int c = lane; c < d; c += 32) q[c] = k[c] = 0.f;
                continue;
            }
            float sq = 0.f, sk = 0.f;
            for (int c = lane; c < d; c += 32) {
                const float a = silu(convolved(rows, ld, conv, taps, C, hist, q0 + c, i)), b = silu(convolved(rows, ld, conv, taps, C, hist, k0 + c, i));
                q[c] = a;
                k[c] = b;
                sq = fmaf(a, a, sq);
                sk = fmaf(b, b, sk);
            }
            const float fq = query_scale * rsqrtf(warp_sum(sq) + unit_eps), fk = rsqrtf(warp_sum(sk) + unit_eps);
            float* to = out + (size_t)(first + i) * C;
            for (int c = lane; c < d; c += 32) {         // a lane reads back what it wrote
                to[q0 + c] = q[c] *= fq;
                to[k0 + c] = k[c] *= fk;
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
// The recurrence.  A block owns a slice of the value channels of one (request, head); the lanes of a warp are 8 groups of key
// channels x 4 value channels; a thread keeps IPT key channels of one value channel of the state in registers (d <= 8 IPT;
// channels beyond d are zeros).  Tiles of SCAN_BLOCKS blocks of four tokens are copied into the other half of shared memory
// (cp.async) while this one is walked.
constexpr int SCAN_BLOCKS = 2;
constexpr int SCAN_TILE = SCAN_BLOCKS * B;

template <int BYTES> __device__ __forceinline__ void copy_async(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    if (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

// Multiply-adds and products of two floats at once.
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) { return __ffma2_rn(a, b, c); }
__device__ __forceinline__ float2 both(float x) { return make_float2(x, x); }

template <int IPT, bool VEC>
__global__ void __launch_bounds__(256)
delta_scan_kernel(const float* __restrict__ qkv, const float* __restrict__ coefs, float* state, long long state_stride,
                  const int* __restrict__ seats, const int* __restrict__ cu_q, float* __restrict__ out, int heads, int kv_heads, int d,
                  int dv, int n_seats) {
    griddep_wait();
    griddep_launch_dependents();
    constexpr int GP = IPT + 4;                          // a group's stretch in shared memory, padded against bank conflicts
    constexpr int ROW = 8 * GP;
    constexpr int STEP = VEC ? 4 : 1;
    extern __shared__ __align__(16) float smem[];
    const int columns = (blockDim.x >> 5) * 4;
    const int stage_floats = SCAN_TILE * (2 * ROW + columns) + SCAN_BLOCKS * COEFS;
    const int req = blockIdx.x, head = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int group = lane >> 2, local = warp * 4 + (lane & 3);
    const int j0 = blockIdx.z * columns, j = j0 + local;
    const bool own = j < dv;
    const int seat = seats[req];
    float* mine = (seat >= 0 && seat < n_seats) ? state + (size_t)seat * state_stride + (size_t)head * d * dv : nullptr;
    float2 S[IPT / 2];
#pragma unroll
    for (int x = 0; x < IPT / 2; ++x) {
        const int i = group * IPT + 2 * x;
        S[x].x = (own && i < d && mine) ? mine[(size_t)i * dv + j] : 0.f;
        S[x].y = (own && i + 1 < d && mine) ? mine[(size_t)(i + 1) * dv + j] : 0.f;
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
    // rows of a tile beyond the portion's end keep what the tile before last left there: finite numbers that meet beta = 0,
    // E = the last token's and N = 0 only; so they are cleared instead of copied
    auto fetch = [&](int t0, float* stage) {
        const int count = min(SCAN_TILE, n - t0);
        float *qs = stage, *ks = qs + SCAN_TILE * ROW, *vs = ks + SCAN_TILE * ROW, *cs = vs + SCAN_TILE * columns;
        const int per = d / STEP;
        for (int e = threadIdx.x; e < SCAN_TILE * per; e += blockDim.x) {
            const int tt = e / per, i = (e - tt * per) * STEP;
            const int to = tt * ROW + (i / IPT) * GP + i % IPT;
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
        const int blocks = (count + B - 1) / B;
        for (int e = threadIdx.x; e < blocks * COEFS; e += blockDim.x) {
            const int b = e / COEFS, x = e - b * COEFS;
            copy_async<4>(cs + e, crows + (size_t)(t0 / B + b) * heads * COEFS + x);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (n > 0) fetch(0, smem);
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
#pragma unroll
        for (int b = 0; b < SCAN_BLOCKS; ++b) {
            if (t0 + b * B >= n) break;                  // the same for the whole block
            const float* cf = cs + b * COEFS;
            float2 ak[B], aq[B];
#pragma unroll
            for (int i = 0; i < B; ++i) ak[i] = aq[i] = make_float2(0.f, 0.f);
#pragma unroll
            for (int x = 0; x < IPT; x += 4) {
#pragma unroll
                for (int i = 0; i < B; ++i) {
                    const float4 k4 = *reinterpret_cast<const float4*>(ks + (b * B + i) * ROW + group * GP + x);
                    const float4 q4 = *reinterpret_cast<const float4*>(qs + (b * B + i) * ROW + group * GP + x);
                    ak[i] = fma2(make_float2(k4.x, k4.y), S[x / 2], ak[i]);
                    ak[i] = fma2(make_float2(k4.z, k4.w), S[x / 2 + 1], ak[i]);
                    aq[i] = fma2(make_float2(q4.x, q4.y), S[x / 2], aq[i]);
                    aq[i] = fma2(make_float2(q4.z, q4.w), S[x / 2 + 1], aq[i]);
                }
            }
            // eight sums over the eight groups of key channels: every round a lane gives half of its sums away and adds the
            // partner's to the other half, so that group g ends with sum g (k of token g, then q of token g - 4)
            float r8[8];
#pragma unroll
            for (int i = 0; i < B; ++i) r8[i] = ak[i].x + ak[i].y, r8[B + i] = aq[i].x + aq[i].y;
            const bool hi = group & 4, mid = group & 2, low = group & 1;
            float r4[4], r2[2];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float keep = hi ? r8[4 + x] : r8[x], give = hi ? r8[x] : r8[4 + x];
                r4[x] = keep + __shfl_xor_sync(0xffffffffu, give, 16);
            }
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const float keep = mid ? r4[2 + x] : r4[x], give = mid ? r4[x] : r4[2 + x];
                r2[x] = keep + __shfl_xor_sync(0xffffffffu, give, 8);
            }
            const float keep = low ? r2[1] : r2[0], give = low ? r2[0] : r2[1];
            const float sum = keep + __shfl_xor_sync(0xffffffffu, give, 4);
            float u[B];
#pragma unroll
            for (int i = 0; i < B; ++i) {
                const float a = __shfl_sync(0xffffffffu, sum, (lane & 3) + 4 * i);
                u[i] = fmaf(cf[C_BETA + i], vs[(b * B + i) * columns + local], -cf[C_BP + i] * a);
#pragma unroll
                for (int m = 0; m < i; ++m) u[i] = fmaf(-cf[C_M + i * (i - 1) / 2 + m], u[m], u[i]);
            }
            if (hi) {                                    // group 4 + i holds S^T q_i and writes o_i
                const int i = group & 3, t = t0 + b * B + i;
                float o = cf[C_P + i] * sum;
#pragma unroll
                for (int m = 0; m < B; ++m)
                    if (m <= i) o = fmaf(cf[C_N + i * (i + 1) / 2 + m], u[m], o);
                if (own && t < n) out[(size_t)(first + t) * heads * dv + (size_t)head * dv + j] = o;
            }
            const float2 P2 = both(cf[C_P + B - 1]);
#pragma unroll
            for (int i = 0; i < B; ++i) u[i] *= cf[C_E + i];
#pragma unroll
            for (int x = 0; x < IPT; x += 4) {
                float2 s0 = __fmul2_rn(P2, S[x / 2]), s1 = __fmul2_rn(P2, S[x / 2 + 1]);
#pragma unroll
                for (int i = 0; i < B; ++i) {
                    const float4 k4 = *reinterpret_cast<const float4*>(ks + (b * B + i) * ROW + group * GP + x);
                    s0 = fma2(make_float2(k4.x, k4.y), both(u[i]), s0);
                    s1 = fma2(make_float2(k4.z, k4.w), both(u[i]), s1);
                }
                S[x / 2] = s0;
                S[x / 2 + 1] = s1;
            }
        }
        __syncthreads();                                 // everyone is done with this half before it is filled again
    }
    if (mine && own) {
#pragma unroll
        for (int x = 0; x < IPT / 2; ++x) {
            const int i = group * IPT + 2 * x;
            if (i < d) mine[(size_t)i * dv + j] = S[x].x;
            if (i + 1 < d) mine[(size_t)(i + 1) * dv + j] = S[x].y;
        }
    }
}

template <int IPT, bool VEC>
int launch_scan(const float* qkv, const float* coefs, float* state, long long state_stride, const int* seats, const int* cu_q, float* out,
                int requests, int heads, int kv_heads, int d, int dv, int n_seats, cudaStream_t stream) {
    // a head's value channels are cut into slices until the blocks about fill the device; a block keeps four warps, since every
    // block copies the queries and keys of all key channels for itself
    const long long units = (long long)requests * heads;
    const int head_warps = (dv + 3) / 4;
    const int most = (head_warps + 3) / 4;
    int slices = (int)((fe_sm_count() + units - 1) / units);
    slices = slices < 1 ? 1 : (slices > most ? most : slices);
    int warps = (head_warps + slices - 1) / slices;
    if (warps > 8) warps = 8;
    slices = (head_warps + warps - 1) / warps;
    const size_t smem = 2 * ((size_t)SCAN_TILE * (2 * 8 * (IPT + 4) + warps * 4) + SCAN_BLOCKS * COEFS) * sizeof(float);
    if (smem > 48 * 1024) {
        const cudaError_t err = cudaFuncSetAttribute(delta_scan_kernel<IPT, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        FE_REQUIRE(err == cudaSuccess, "delta_scan: %s", cudaGetErrorString(err));
    }
    fe::launch(delta_scan_kernel<IPT, VEC>, dim3(requests, heads, slices), warps * 32, smem, stream, qkv, coefs, state, state_stride, seats,
               cu_q, out, heads, kv_heads, d, dv, n_seats);
    return fe_check_launch("delta_scan");
}

// ---------------------------------------------------------------------------------------------
// A step of ONE token a request.  Block per (request, query/key head): the value heads that read this query/key head are its
// columns, so that the convolutions' history of every channel belongs to one block.  Threads are ``groups`` runs of PER key
// channels x ``columns`` value channels; a state is read once into registers and written once.
constexpr int PER = 16;

template <typename T>
__global__ void __launch_bounds__(1024)
delta_decode_kernel(const float* __restrict__ proj, long long ld, const float* __restrict__ conv, int taps, float* state,
                    long long state_stride, long long history_at, const int* __restrict__ seats, const float* __restrict__ a_log,
                    const float* __restrict__ dt_bias, const float* __restrict__ norm_weight, float eps, float unit_eps, float query_scale,
                    T* __restrict__ out, int heads, int kv_heads, int d, int dv, int n_seats, int groups) {
    griddep_wait();
    griddep_launch_dependents();
    extern __shared__ __align__(16) float smem[];
    const int ratio = heads / kv_heads, total = ratio * dv, columns = blockDim.x / groups;
    float* qs = smem;                               // [d]
    float* ks = qs + d;                             // [d]
    float* vs = ks + d;                             // [total]: values, later the outputs
    float* gate = vs + total;                       // [2 ratio]: decays, step sizes
    float* part = gate + 2 * ratio;                 // [2][groups][columns]
    float* red = part + 2 * groups * columns;       // [4]: the factors of q and k, k . q
    const int r = blockIdx.x, kvh = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
    const int C = 2 * kv_heads * d + heads * dv;
    const float* row = proj + (size_t)r * ld;
    const int seat = seats[r];
    float* base = (seat >= 0 && seat < n_seats) ? state + (size_t)seat * state_stride : nullptr;
    float* hist = (taps > 1 && base) ? base + history_at : nullptr;
    const int v0 = 2 * kv_heads * d + kvh * total;
    for (int c = tid; c < 2 * d + total; c += blockDim.x) {       // a thread reads and renews the history of its own channels
        const int ch = c < d ? kvh * d + c : (c < 2 * d ? (kv_heads + kvh) * d + c - d : v0 + c - 2 * d);
        smem[c] = silu(convolved(row, ld, conv, taps, C, hist, ch, 0));
        if (hist) keep_history(row, ld, taps, C, hist, ch, 1);
    }
    for (int hh = tid; hh < ratio; hh += blockDim.x) {
        const int head = kvh * ratio + hh;
        const float* b = row + C + (size_t)heads * dv;
        gate[ratio + hh] = sigmoid(b[head]);
        gate[hh] = decay_of(b[heads + head], dt_bias[head], a_log[head]);
    }
    __syncthreads();
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
    __syncthreads();
    const float fq = red[0], fk = red[1], dot = red[2];
    const int g = tid / columns, jj = tid - g * columns;
    const int i0 = g * PER;
    for (int c0 = 0; c0 < total; c0 += columns) {
        const int col = c0 + jj;
        const bool own = g < groups && col < total;
        const int hh = own ? col / dv : 0, j = col - hh * dv;
        float* mine = (own && base) ? base + (size_t)(kvh * ratio + hh) * d * dv + j : nullptr;
        float S[PER], ak = 0.f, aq = 0.f;
#pragma unroll
        for (int x = 0; x < PER; ++x) S[x] = (mine && i0 + x < d) ? mine[(size_t)(i0 + x) * dv] : 0.f;
#pragma unroll
        for (int x = 0; x < PER; ++x) {
            if (i0 + x < d) {
                ak = fmaf(ks[i0 + x], S[x], ak);
                aq = fmaf(qs[i0 + x], S[x], aq);
            }
        }
        if (g < groups) {
            part[g * columns + jj] = ak * fk;
            part[(groups + g) * columns + jj] = aq * fq;
        }
        __syncthreads();
        float o = 0.f;
        if (own) {
            float sk = 0.f;
            for (int x = 0; x < groups; ++x) sk += part[x * columns + jj];
            const float decay = gate[hh];
            const float u = gate[ratio + hh] * (vs[col] - decay * sk), w = u * fk;
            if (mine) {
#pragma unroll
                for (int x = 0; x < PER; ++x)
                    if (i0 + x < d) mine[(size_t)(i0 + x) * dv] = fmaf(decay, S[x], ks[i0 + x] * w);
            }
            if (g == 0) {
                float sq = 0.f;
                for (int x = 0; x < groups; ++x) sq += part[(groups + x) * columns + jj];
                o = fmaf(decay, sq, dot * u);
            }
        }
        __syncthreads();                                  // every run of this column has read its value and the sums
        if (g == 0 && own) vs[col] = o;
    }
    __syncthreads();
    // every head divided by its root mean square, times the weight, times silu of its gate row
    const float* grow = row + C + (size_t)kvh * total;
    T* to = out + (size_t)r * heads * dv + (size_t)kvh * total;
    for (int hh = warp; hh < ratio; hh += warps) {
        float ss = 0.f;
        for (int j = lane; j < dv; j += 32) ss = fmaf(vs[hh * dv + j], vs[hh * dv + j], ss);
        const float inv = rsqrtf(warp_sum(ss) / (float)dv + eps);
        for (int j = lane; j < dv; j += 32) to[hh * dv + j] = from_float<T>(vs[hh * dv + j] * inv * norm_weight[j] * silu(grow[hh * dv + j]));
    }
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
    fe::launch(delta_prepare_kernel, dim3(tiles, requests, units), PREP_WARPS * 32, smem, stream, proj, ld, conv, taps, state, state_stride,
               history_at, seats, cu_q, a_log, dt_bias, unit_eps, query_scale, out, coefs, heads, kv_heads, d, dv, n_seats);
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
    const bool vec = d % 4 == 0 && dv % 4 == 0 && C % 4 == 0 && ((size_t)qkv & 15) == 0;
#define FE_DELTA_SCAN(IPT)                                                                                                            \
    return vec ? launch_scan<IPT, true>(qkv, coefs, state, state_stride, seats, cu_q, out, requests, heads, kv_heads, d, dv, n_seats, stream) \
               : launch_scan<IPT, false>(qkv, coefs, state, state_stride, seats, cu_q, out, requests, heads, kv_heads, d, dv, n_seats, stream)
    if (d <= 32) { FE_DELTA_SCAN(4); }
    if (d <= 64) { FE_DELTA_SCAN(8); }
    if (d <= 128) { FE_DELTA_SCAN(16); }
    FE_DELTA_SCAN(32);
#undef FE_DELTA_SCAN
}

// A step of one token a request in one kernel: proj, conv, state as fe_delta_prepare takes them (row r is request r's token); out
// [requests, heads dv] in ``dtype``: every head's output divided by its root mean square, times norm_weight [dv], times silu(g).
extern "C" int fe_delta_decode(const float* proj, long long ld, const float* conv, int taps, float* state, long long state_stride,
                               long long history_at, const int* seats, const float* a_log, const float* dt_bias, const float* norm_weight,
                               float eps, float unit_eps, float query_scale, void* out, int requests, int heads, int kv_heads, int d, int dv,
                               int n_seats, int dtype, cudaStream_t stream) {
    const long long C = 2LL * kv_heads * d + (long long)heads * dv;
    FE_REQUIRE(requests >= 0 && heads > 0 && kv_heads > 0 && kv_heads <= 65535 && heads % kv_heads == 0 && d > 0 && d <= 512 && dv > 0 && taps >= 1 &&
                   n_seats >= 0 && ld >= C + (long long)heads * dv + 2 * heads && history_at >= (long long)heads * d * dv &&
                   history_at + (taps - 1) * C <= state_stride,
               "delta_decode: bad sizes (heads %d over %d, key size %d up to 512, value size %d, %d taps)", heads, kv_heads, d, dv, taps);
    FE_REQUIRE(dtype == FE_F32 || dtype == FE_BF16, "delta_decode: unknown dtype %d", dtype);
    if (requests == 0) return 0;
    const int ratio = heads / kv_heads, total = ratio * dv, groups = (d + PER - 1) / PER;
    int columns = (total + 31) / 32 * 32;
    const int most = 1024 / groups / 32 * 32;
    columns = columns > most ? most : columns;
    const size_t smem = (2 * (size_t)d + total + 2 * ratio + 2 * (size_t)groups * columns + 4) * sizeof(float);
    FE_REQUIRE(smem <= 200 * 1024, "delta_decode: %d value channels a query/key head need more shared memory than a block has", total);
    if (dtype == FE_F32) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(delta_decode_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        fe::launch(delta_decode_kernel<float>, dim3(requests, kv_heads), groups * columns, smem, stream, proj, ld, conv, taps, state, state_stride,
                   history_at, seats, a_log, dt_bias, norm_weight, eps, unit_eps, query_scale, (float*)out, heads, kv_heads, d, dv, n_seats, groups);
    } else {
        if (smem > 48 * 1024) cudaFuncSetAttribute(delta_decode_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        fe::launch(delta_decode_kernel<bf16>, dim3(requests, kv_heads), groups * columns, smem, stream, proj, ld, conv, taps, state, state_stride,
                   history_at, seats, a_log, dt_bias, norm_weight, eps, unit_eps, query_scale, (bf16*)out, heads, kv_heads, d, dv, n_seats, groups);
    }
    return fe_check_launch("delta_decode");
}
