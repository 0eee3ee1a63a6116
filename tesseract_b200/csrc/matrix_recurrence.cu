// Recurrences over a matrix per head, written by outer products and read by a query:
//
//   S_t = a_t S_(t-1) + k_t u_t^T        o_t = S_t^T q_t        (S: [dim, vdim], 32-bit, kept per request in its state slot)
//
// with a scalar decay a_t per head and token.  What is written, and where the decay comes from, is the kind:
//
//   STATE_SPACE  u = dt x,  a = exp(rate dt),  dt = softplus(z + bias);  o += skip x        (k: input matrix row, q: output
//                matrix row, x: the value; rate = -exp(A) per head)
//   MEMORY       u = e^(i - m) v,  a = e^(f + m' - m),  m = max(f + m', i)  with m' the m of the token in front (0 at the start),
//                i = cap tanh((z_i + b_i) / cap),  f = log sigmoid(cap tanh((z_f + b_f) / cap));  the same recurrence with v = 1 is
//                the normaliser n: it is one more value column, and n . q and m go to `aux` for the kernel behind
//   DELTA        u = beta (v - a S_(t-1)^T k),  a = exp(rate softplus(z_a + bias)),  beta = sigmoid(z_b), with q and k made unit
//                vectors, x / sqrt(sum x^2 + 1e-6), inside
//
// q (and so o) is multiplied by q_scale.  Head h reads q and k of head h / (heads / qk_heads).
//
// The state stays in registers while a sequence's rows of this step are walked.  Rows go in groups of four: with S the state in
// front of a group, g_i = a_0 .. a_i and p_ij = a_(j+1) .. a_i (products of at most four decays, never a quotient),
//
//   o_i = g_i (S^T q_i) + sum_(j <= i) p_ij (q_i . k_j) u_j          S' = g_3 S + sum_j p_3j k_j u_j^T
//   DELTA:  u_i = beta_i (v_i - g_i (S^T k_i) - sum_(j < i) p_ij (k_i . k_j) u_j)
//
// so that all products of a group read the same S and four rows cost one pass over it.  A block takes one (sequence, head, run of
// value columns); a warp holds 32 / LPC groups of two columns, a column's numbers are shared by LPC lanes (lane r takes the packets
// of four r, r + LPC, ...).  Four more warps run a tile of rows ahead, a warp a group of rows: they widen q, k and v into shared
// memory and leave the group's coefficients (decays, gates, norms, the products q_i . k_j and k_i . k_j).  Where the groups begin
// follows from where the step's rows begin, so cutting a prompt differently moves a result by rounding only.
//
// A step of single rows has a kernel of its own: a warp a run of columns, every number of the state read once and written once,
// straight from and to the slot.  State layout: [slots][heads][columns][dim rounded up to four].
//
// tb_recurrence_norm (behind it): per row and group of `size` numbers, optionally first v / (max(|n . q|, e^-m) + 1e-6) and / or
// v silu(gate), then v / sqrt(mean(v^2) + eps) * weight, then optionally times sigmoid or SiLU of the gate; rounded once.
#include "common.cuh"

namespace {

enum Kind : int { STATE_SPACE = 0, MEMORY = 1, DELTA = 2 };
constexpr int kWorkers = 8;          // the most warps that hold state
constexpr int kFewBlocks = 120;      // fewer blocks than this leave multiprocessors idle
constexpr int kProducers = 4;        // warps that prepare the next tile of rows

typedef unsigned long long pair32;   // two neighbouring 32-bit floats
__device__ __forceinline__ pair32 pack2(float x, float y) {
    pair32 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
    return r;
}
__device__ __forceinline__ float sum2(pair32 p) {
    float x, y;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(p));
    return x + y;
}
__device__ __forceinline__ pair32 fma2(pair32 a, pair32 b, pair32 c) {
    pair32 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ pair32 mul2(pair32 a, pair32 b) {
    pair32 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

__device__ __forceinline__ float softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
// e^x of a decay: near 1 through expm1f, whose result rounds to the nearest number once more; the plain function's last bit leans
// to one side there, which a state that remembers thousands of tokens adds up
__device__ __forceinline__ float decay_of(float x) { return x > -0.5f ? 1.0f + expm1f(x) : expf(x); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }

// four numbers in a row, widened / rounded
template <typename T>
__device__ __forceinline__ float4 load4(const T* p);
template <>
__device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <>
__device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(t.x << 16), __uint_as_float(t.x & 0xffff0000u), __uint_as_float(t.y << 16),
                       __uint_as_float(t.y & 0xffff0000u));
}
template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v);
template <>
__device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <>
__device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

__device__ __forceinline__ float widen(float v) { return v; }
__device__ __forceinline__ float widen(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T narrow(float v);
template <>
__device__ __forceinline__ float narrow<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 narrow<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

struct Recurrence {
    int64_t stride;                  // elements between rows of q, k and v
    int q_off, k_off, v_off;
    const float* gates;              // 32-bit logits: [heads] (STATE_SPACE) or [2 * heads] a row
    int64_t gate_stride;
    const float *p0, *p1, *p2;       // per head: rate, bias, skip | input gate's bias, forget gate's bias | rate, bias
    float cap, q_scale;
    float* state;
    float* running;                  // MEMORY: m, a copy per value column ([slots][heads][columns])
    float* out;                      // [rows, heads * vdim]
    float* aux;                      // MEMORY: (n . q, m) per row and head
    const int *row_start, *state_slots;
    int heads, qk_heads, dim, vdim, columns, workers, tile;
};

// A row's gate logits of one head, and (decay, write weight) from them; for MEMORY (log f, log i) instead.
template <int KIND>
__device__ __forceinline__ float2 logits_of(const Recurrence& p, int row, int head) {
    const float* gate = p.gates + (int64_t)row * p.gate_stride;
    return make_float2(gate[head], KIND == STATE_SPACE ? 0.0f : gate[p.heads + head]);
}
template <int KIND>
__device__ __forceinline__ float2 gates_of(float2 logits, float cap, float rate, float bias0, float bias1) {
    if (KIND == STATE_SPACE) {
        const float dt = softplus(logits.x + bias0);
        return make_float2(decay_of(rate * dt), dt);
    }
    if (KIND == DELTA) return make_float2(decay_of(rate * softplus(logits.x + bias0)), 1.0f / (1.0f + expf(-logits.y)));
    return make_float2(log_sigmoid(cap * tanhf((logits.y + bias1) / cap)), cap * tanhf((logits.x + bias0) / cap));
}

// sum over the lanes of COUNT (a power of two up to 32) values: afterwards lane l holds the sum of value l % COUNT
template <int COUNT>
__device__ __forceinline__ float spread_sums(float* v, int lane) {
#pragma unroll
    for (int half = COUNT / 2; half > 0; half >>= 1) {
        const bool upper = lane & half;
#pragma unroll
        for (int i = 0; i < half; ++i) {
            const float keep = upper ? v[i + half] : v[i], give = upper ? v[i] : v[i + half];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, give, half);
        }
    }
    float sum = v[0];
#pragma unroll
    for (int o = COUNT; o < 32; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    return sum;
}

constexpr int kGroup = 4;            // rows that share a pass over the state
constexpr int kTile = 16;            // the most rows of a tile
// a group's coefficients in shared memory: g_i iq_i [4], w_i or beta_i [4], p_3j ik_j [4], g_3 (and three unused), the triangle
// iq_i p_ij ik_j (q_i . k_j) [4][4] and, for DELTA, beta_i ik_i g_i [4], the strict triangle beta_i ik_i p_ij ik_j (k_i . k_j) [8]
template <int KIND>
struct Coefficients { static constexpr int N = KIND == DELTA ? 44 : 32; };

template <typename T, int KIND, int LPC, int NJ>
__global__ void __launch_bounds__((kWorkers + kProducers) * 32)
matrix_recurrence_kernel(const T* __restrict__ rows, Recurrence p) {
    constexpr int DP = 4 * LPC * NJ;                 // numbers of q or k in shared memory (zeros behind dim)
    constexpr int CPL = 2, CW = 32 / LPC * CPL;
    constexpr int E = DP / 32;                       // numbers of q or k a producer's lane carries
    constexpr bool AHEAD = E <= 4;                   // a producer asks for its next rows before it waits
    constexpr int CF = Coefficients<KIND>::N;
    constexpr int DOTS = KIND == DELTA ? 32 : 16;    // 10 q_i . k_j; DELTA: also 6 k_i . k_j, 4 q_i . q_i, 4 k_i . k_i
    extern __shared__ __align__(16) float smem[];
    pdl_trigger();
    const int W = p.workers, TT = p.tile, VC = W * CW;
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * VC;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int dim4 = (p.dim + 3) & ~3;
    const int stage = TT * (2 * DP + VC) + TT / kGroup * CF;      // floats of a buffer
    pdl_wait();                                      // rows, state and the step's metadata come from kernels in front
    const int first = p.row_start[seq], n = p.row_start[seq + 1] - first;
    if (n <= 0) return;
    const int tiles = (n + TT - 1) / TT;
    const int64_t of_slot = (int64_t)p.state_slots[seq] * p.heads + head;

    if (warp >= W) {
        // ------------------------------------------------------------------ producers: a warp a group of a tile's rows
        const int qk_head = head / (p.heads / p.qk_heads), mine = warp - W;
        const float rate = KIND == MEMORY ? 0.0f : p.p0[head];
        const float bias0 = KIND == MEMORY ? p.p0[head] : p.p1[head], bias1 = KIND == MEMORY ? p.p1[head] : 0.0f;
        float m = KIND == MEMORY ? p.running[of_slot * p.columns + col0] : 0.0f;      // (the same in every producer)
        // the next rows as they are stored: widened when they are used, so that nothing waits for them before
        T rq[kGroup][AHEAD ? E : 1], rk[kGroup][AHEAD ? E : 1], rv[kGroup];
        const T zero = narrow<T>(0.0f), one = narrow<T>(1.0f);
        const int groups = TT / kGroup;
        auto row_at = [&](int tile, int group, int t) { return first + tile * TT + group * kGroup + t; };
        auto there = [&](int tile, int group, int t) { return tile * TT + group * kGroup + t < n; };
        auto fetch_v = [&](int tile, int group, int t) {
            const int col = col0 + lane;
            if (lane >= VC || !there(tile, group, t)) return zero;
            if (col < p.vdim) return rows[(int64_t)row_at(tile, group, t) * p.stride + p.v_off + (int64_t)head * p.vdim + col];
            return KIND == MEMORY && col == p.vdim ? one : zero;
        };
        auto fetch_qk = [&](int tile, int group, int t, int e, bool key) {
            if (e >= p.dim || !there(tile, group, t)) return zero;
            return rows[(int64_t)row_at(tile, group, t) * p.stride + (key ? p.k_off : p.q_off) + (int64_t)qk_head * p.dim + e];
        };
        auto fetch = [&](int tile, int group) {
#pragma unroll
            for (int t = 0; t < kGroup; ++t) {
                rv[t] = fetch_v(tile, group, t);
                if constexpr (AHEAD) {
#pragma unroll
                    for (int i = 0; i < E; ++i) {
                        rq[t][i] = fetch_qk(tile, group, t, i * 32 + lane, false);
                        rk[t][i] = fetch_qk(tile, group, t, i * 32 + lane, true);
                    }
                }
            }
        };
        auto fetch_gates = [&](int tile) {            // a lane a row of the tile
            const int at = tile * TT + lane;
            return lane < TT && at < n ? logits_of<KIND>(p, first + at, head) : make_float2(0.0f, 0.0f);
        };
        float2 logits = fetch_gates(0);
        if (mine < groups) fetch(0, mine);
        for (int tile = -1; tile < tiles; ++tile) {
            const int next = tile + 1;
            if (next < tiles) {
                float* buffer = smem + (next & 1) * stage;
                float *qs = buffer, *ks = qs + TT * DP, *vs = ks + TT * DP, *cf = vs + TT * VC;
                const int count = min(TT, n - next * TT);
                const float2 gate = gates_of<KIND>(logits, p.cap, rate, bias0, bias1);
                float a = lane < count ? gate.x : 1.0f, w = lane < count ? gate.y : 0.0f;    // (nothing happens behind the last row)
                if (KIND == MEMORY) {
                    float before = 0.0f, now = 0.0f;
                    // in token order; behind the last row log f = 0 and log i = -inf leave m as it is
                    const float log_f = lane < count ? gate.x : 0.0f, log_i = lane < count ? gate.y : -INFINITY;
#pragma unroll
                    for (int t = 0; t < kTile; ++t) {
                        const float f = __shfl_sync(0xffffffffu, log_f, t), i = __shfl_sync(0xffffffffu, log_i, t);
                        const float to = fmaxf(f + m, i);
                        if (lane == t) { before = m; now = to; }
                        m = to;
                    }
                    a = lane < count ? decay_of(gate.x + before - now) : 1.0f;
                    w = lane < count ? expf(gate.y - now) : 0.0f;
                    if (mine == 0 && lane < count && col0 <= p.vdim && p.vdim < col0 + VC)
                        p.aux[((int64_t)(first + next * TT + lane) * p.heads + head) * 2 + 1] = now;
                }
                for (int group = mine; group < groups; group += kProducers) {
                    if (next * TT + group * kGroup >= n) break;
                    if (group != mine) fetch(next, group);
                    const int t0 = group * kGroup;
                    float dots[DOTS];
#pragma unroll
                    for (int i = 0; i < DOTS; ++i) dots[i] = 0.0f;
                    auto take = [&](int i, const float* q, const float* k) {      // four rows' numbers i * 32 + lane
#pragma unroll
                        for (int t = 0; t < kGroup; ++t) {
                            qs[(t0 + t) * DP + i * 32 + lane] = q[t];
                            ks[(t0 + t) * DP + i * 32 + lane] = k[t];
#pragma unroll
                            for (int j = 0; j <= t; ++j) dots[t * (t + 1) / 2 + j] = fmaf(q[t], k[j], dots[t * (t + 1) / 2 + j]);
                            if constexpr (KIND == DELTA) {
#pragma unroll
                                for (int j = 0; j < t; ++j) dots[10 + t * (t - 1) / 2 + j] = fmaf(k[t], k[j], dots[10 + t * (t - 1) / 2 + j]);
                                dots[16 + t] = fmaf(q[t], q[t], dots[16 + t]);
                                dots[20 + t] = fmaf(k[t], k[t], dots[20 + t]);
                            }
                        }
                    };
                    if constexpr (AHEAD) {
#pragma unroll
                        for (int i = 0; i < E; ++i) {
                            const float q[kGroup] = {widen(rq[0][i]), widen(rq[1][i]), widen(rq[2][i]), widen(rq[3][i])};
                            const float k[kGroup] = {widen(rk[0][i]), widen(rk[1][i]), widen(rk[2][i]), widen(rk[3][i])};
                            take(i, q, k);
                        }
                    } else {
#pragma unroll 2
                        for (int i = 0; i < E; ++i) {
                            float q[kGroup], k[kGroup];
#pragma unroll
                            for (int t = 0; t < kGroup; ++t) {
                                q[t] = widen(fetch_qk(next, group, t, i * 32 + lane, false));
                                k[t] = widen(fetch_qk(next, group, t, i * 32 + lane, true));
                            }
                            take(i, q, k);
                        }
                    }
                    if (lane < VC)
#pragma unroll
                        for (int t = 0; t < kGroup; ++t) vs[(t0 + t) * VC + lane] = widen(rv[t]);
                    const float dot = spread_sums<DOTS>(dots, lane);
                    // lane l: dot product l; its pair (i, j), and the decays between
                    float ga[kGroup], gw[kGroup];
#pragma unroll
                    for (int t = 0; t < kGroup; ++t) {
                        ga[t] = __shfl_sync(0xffffffffu, a, t0 + t);
                        gw[t] = __shfl_sync(0xffffffffu, w, t0 + t);
                    }
                    float inv = 1.0f;                     // DELTA: lanes 16 .. 19 one over the norms of q, 20 .. 23 of k
                    if (KIND == DELTA) inv = 1.0f / sqrtf(dot + 1e-6f);
                    const bool strict = lane >= 10;       // (10 .. 15: k_i . k_j)
                    const int pair = strict ? lane - 10 : lane;
                    int i = 0, j = 0;
                    if (strict) {
                        i = pair < 1 ? 1 : pair < 3 ? 2 : 3;
                        j = pair - i * (i - 1) / 2;
                    } else {
                        i = pair < 1 ? 0 : pair < 3 ? 1 : pair < 6 ? 2 : 3;
                        j = pair - i * (i + 1) / 2;
                    }
                    float between = 1.0f;                 // p_ij
#pragma unroll
                    for (int t = 1; t < kGroup; ++t)
                        if (t > j && t <= i) between *= ga[t];
                    float iq = p.q_scale, ik_i = 1.0f, ik_j = 1.0f;
                    if (KIND == DELTA) {
                        iq *= __shfl_sync(0xffffffffu, inv, 16 + (i & 3));
                        ik_i = __shfl_sync(0xffffffffu, inv, 20 + (i & 3));
                        ik_j = __shfl_sync(0xffffffffu, inv, 20 + (j & 3));
                    }
                    float* c = cf + group * CF;
                    if (lane < 10) {
                        c[16 + i * 4 + j] = iq * between * ik_j * dot;
                        if (i == j) {                     // lanes 0, 2, 5, 9: the row's own coefficients
                            float g = 1.0f, rest = 1.0f;
#pragma unroll
                            for (int t = 0; t < kGroup; ++t) {
                                if (t <= i) g *= ga[t];
                                else rest *= ga[t];
                            }
                            const float weight = i == 0 ? gw[0] : i == 1 ? gw[1] : i == 2 ? gw[2] : gw[3];
                            c[i] = g * iq;
                            c[4 + i] = weight;
                            c[8 + i] = rest * ik_i;
                            if (i == 3) c[12] = g;
                            if (KIND == DELTA) c[32 + i] = weight * ik_i * g;
                        } else {
                            c[16 + j * 4 + i] = 0.0f;     // (the triangle's other half)
                        }
                    } else if (KIND == DELTA && lane < 16) {
                        const float weight = i == 1 ? gw[1] : i == 2 ? gw[2] : gw[3];
                        c[36 + pair] = weight * ik_i * between * ik_j * dot;
                    }
                }
                if (next + 1 < tiles) {                   // the next tile's rows, asked for while the consumers work
                    logits = fetch_gates(next + 1);
                    if (mine < groups) fetch(next + 1, mine);
                }
            }
            __syncthreads();
        }
        if (KIND == MEMORY && mine == 0)
            for (int c = lane; c < VC && col0 + c < p.columns; c += 32) p.running[of_slot * p.columns + col0 + c] = m;
        return;
    }

    // ---------------------------------------------------------------------- consumers: the state of this warp's columns
    // (neighbouring lanes share a packet of q and k and own different columns: a shared-memory read serves them together)
    constexpr int LANES = 32 / LPC;
    const int r = lane / LANES, wcol = warp * CW + lane % LANES * CPL;
    pair32 S[CPL][NJ][2];
#pragma unroll
    for (int j = 0; j < CPL; ++j) {
        const int col = col0 + wcol + j;
        const float* at = p.state + (of_slot * p.columns + col) * dim4;
#pragma unroll
        for (int i = 0; i < NJ; ++i) {
            const int e = 4 * (r + LPC * i);
            ulonglong2 v = make_ulonglong2(0ull, 0ull);
            if (col < p.columns && e < dim4) v = *reinterpret_cast<const ulonglong2*>(at + e);
            S[j][i][0] = v.x;
            S[j][i][1] = v.y;
        }
    }
    const float skip = KIND == STATE_SPACE ? p.p2[head] : 0.0f;
    const int my_t = (r & 7) >> 1, my_col = col0 + wcol + (r & 1);      // whose output this lane writes
    __syncthreads();                                 // the first tile is there
    for (int tile = 0; tile < tiles; ++tile) {
        const float* buffer = smem + (tile & 1) * stage;
        const float *qs = buffer, *ks = qs + TT * DP, *vs = ks + TT * DP, *cf = vs + TT * VC;
        const int count = min(TT, n - tile * TT), row0 = first + tile * TT;
        for (int t0 = 0; t0 < count; t0 += kGroup) {
            const ulonglong2* q2 = reinterpret_cast<const ulonglong2*>(qs + t0 * DP) + r;
            const ulonglong2* k2 = reinterpret_cast<const ulonglong2*>(ks + t0 * DP) + r;
            const float* c = cf + t0 / kGroup * CF;
            const float4 weight = *reinterpret_cast<const float4*>(c + 4), own = *reinterpret_cast<const float4*>(c + 8);
            const float g3 = c[12];
            const pair32 g2 = pack2(g3, g3);
            float2 v[kGroup];
#pragma unroll
            for (int t = 0; t < kGroup; ++t) v[t] = *reinterpret_cast<const float2*>(vs + (t0 + t) * VC + wcol);
            float u[kGroup][CPL];
            u[0][0] = weight.x * v[0].x; u[1][0] = weight.y * v[1].x; u[2][0] = weight.z * v[2].x; u[3][0] = weight.w * v[3].x;
            u[0][1] = weight.x * v[0].y; u[1][1] = weight.y * v[1].y; u[2][1] = weight.z * v[2].y; u[3][1] = weight.w * v[3].y;
            pair32 dq[kGroup][CPL];
#pragma unroll
            for (int t = 0; t < kGroup; ++t)
#pragma unroll
                for (int j = 0; j < CPL; ++j) dq[t][j] = 0ull;
            auto update = [&](int i, const pair32 (*eu)[CPL]) {
                ulonglong2 kv[kGroup];
#pragma unroll
                for (int t = 0; t < kGroup; ++t) kv[t] = k2[t * (DP / 4) + LPC * i];
#pragma unroll
                for (int j = 0; j < CPL; ++j) {
                    S[j][i][0] = mul2(S[j][i][0], g2);
                    S[j][i][1] = mul2(S[j][i][1], g2);
#pragma unroll
                    for (int t = 0; t < kGroup; ++t) {
                        S[j][i][0] = fma2(kv[t].x, eu[t][j], S[j][i][0]);
                        S[j][i][1] = fma2(kv[t].y, eu[t][j], S[j][i][1]);
                    }
                }
            };
            auto written = [&](pair32 (*eu)[CPL]) {
                const float e[kGroup] = {own.x, own.y, own.z, own.w};
#pragma unroll
                for (int t = 0; t < kGroup; ++t)
#pragma unroll
                    for (int j = 0; j < CPL; ++j) eu[t][j] = pack2(e[t] * u[t][j], e[t] * u[t][j]);
            };
            pair32 eu[kGroup][CPL];
            if constexpr (KIND == DELTA) {
                pair32 dk[kGroup][CPL];
#pragma unroll
                for (int t = 0; t < kGroup; ++t)
#pragma unroll
                    for (int j = 0; j < CPL; ++j) dk[t][j] = 0ull;
#pragma unroll
                for (int i = 0; i < NJ; ++i)
#pragma unroll
                    for (int t = 0; t < kGroup; ++t) {
                        const ulonglong2 kv = k2[t * (DP / 4) + LPC * i], qv = q2[t * (DP / 4) + LPC * i];
#pragma unroll
                        for (int j = 0; j < CPL; ++j) {
                            dk[t][j] = fma2(S[j][i][0], kv.x, dk[t][j]);
                            dk[t][j] = fma2(S[j][i][1], kv.y, dk[t][j]);
                            dq[t][j] = fma2(S[j][i][0], qv.x, dq[t][j]);
                            dq[t][j] = fma2(S[j][i][1], qv.y, dq[t][j]);
                        }
                    }
                float d[8];
#pragma unroll
                for (int t = 0; t < kGroup; ++t)
#pragma unroll
                    for (int j = 0; j < CPL; ++j) d[t * 2 + j] = sum2(dk[t][j]);
                // the lanes' shares of S^T k meet; lane r then holds (row (r & 7) / 2, column r & 1), and every lane reads all eight
#pragma unroll
                for (int half = 4; half > 0; half >>= 1)
#pragma unroll
                    for (int i = 0; i < half; ++i) {
                        const bool upper = r & half;
                        const float keep = upper ? d[i + half] : d[i], give = upper ? d[i] : d[i + half];
                        d[i] = keep + __shfl_xor_sync(0xffffffffu, give, half * LANES);
                    }
                float sum = d[0];
#pragma unroll
                for (int o = 8; o < LPC; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o * LANES);
                const float4 share = *reinterpret_cast<const float4*>(c + 32), n0 = *reinterpret_cast<const float4*>(c + 36);
                const float2 n1 = *reinterpret_cast<const float2*>(c + 40);
#pragma unroll
                for (int j = 0; j < CPL; ++j) {
                    float k[kGroup];
#pragma unroll
                    for (int t = 0; t < kGroup; ++t) k[t] = __shfl_sync(0xffffffffu, sum, lane % LANES + (t * 2 + j) * LANES);
                    u[0][j] = fmaf(-share.x, k[0], u[0][j]);
                    u[1][j] = fmaf(-n0.x, u[0][j], fmaf(-share.y, k[1], u[1][j]));
                    u[2][j] = fmaf(-n0.z, u[1][j], fmaf(-n0.y, u[0][j], fmaf(-share.z, k[2], u[2][j])));
                    u[3][j] = fmaf(-n1.y, u[2][j], fmaf(-n1.x, u[1][j], fmaf(-n0.w, u[0][j], fmaf(-share.w, k[3], u[3][j]))));
                }
                written(eu);
#pragma unroll
                for (int i = 0; i < NJ; ++i) update(i, eu);
            } else {
                written(eu);
#pragma unroll
                for (int i = 0; i < NJ; ++i) {
#pragma unroll
                    for (int t = 0; t < kGroup; ++t) {
                        const ulonglong2 qv = q2[t * (DP / 4) + LPC * i];
#pragma unroll
                        for (int j = 0; j < CPL; ++j) {
                            dq[t][j] = fma2(S[j][i][0], qv.x, dq[t][j]);
                            dq[t][j] = fma2(S[j][i][1], qv.y, dq[t][j]);
                        }
                    }
                    update(i, eu);
                }
            }
            // the lanes' shares of S^T q meet the same way; a lane finishes one row's number of one column
            float d[8];
#pragma unroll
            for (int t = 0; t < kGroup; ++t)
#pragma unroll
                for (int j = 0; j < CPL; ++j) d[t * 2 + j] = sum2(dq[t][j]);
#pragma unroll
            for (int half = 4; half > 0; half >>= 1)
#pragma unroll
                for (int i = 0; i < half; ++i) {
                    const bool upper = r & half;
                    const float keep = upper ? d[i + half] : d[i], give = upper ? d[i] : d[i + half];
                    d[i] = keep + __shfl_xor_sync(0xffffffffu, give, half * LANES);
                }
            float sum = d[0];
#pragma unroll
            for (int o = 8; o < LPC; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o * LANES);
            const bool second = r & 1;
            const float4 inside = *reinterpret_cast<const float4*>(c + 16 + my_t * 4);
            float o = c[my_t] * sum;
            o = fmaf(inside.x, second ? u[0][1] : u[0][0], o);
            o = fmaf(inside.y, second ? u[1][1] : u[1][0], o);
            o = fmaf(inside.z, second ? u[2][1] : u[2][0], o);
            o = fmaf(inside.w, second ? u[3][1] : u[3][0], o);
            if (KIND == STATE_SPACE) o = fmaf(skip, vs[(t0 + my_t) * VC + wcol + (r & 1)], o);
            if (r < 8 && t0 + my_t < count) {
                const int64_t at = (int64_t)(row0 + t0 + my_t) * p.heads + head;
                if (my_col < p.vdim) p.out[at * p.vdim + my_col] = o;
                else if (KIND == MEMORY && my_col == p.vdim) p.aux[at * 2] = o;
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < CPL; ++j) {
        const int col = col0 + wcol + j;
        float* at = p.state + (of_slot * p.columns + col) * dim4;
#pragma unroll
        for (int i = 0; i < NJ; ++i) {
            const int e = 4 * (r + LPC * i);
            if (col < p.columns && e < dim4) *reinterpret_cast<ulonglong2*>(at + e) = make_ulonglong2(S[j][i][0], S[j][i][1]);
        }
    }
}

// A step of single rows: a warp a (sequence, head, run of columns).  o = a (S^T q) + (k . q) u,  S' = a S + k u^T.
constexpr int kStepWarps = 4;

template <typename T, int KIND, int LPC, int NJ>
__global__ void __launch_bounds__(kStepWarps * 32)
matrix_recurrence_step_kernel(const T* __restrict__ rows, Recurrence p, int runs, int vec) {
    constexpr int CPL = 2, CW = 32 / LPC * CPL;
    pdl_trigger();
    const int lane = threadIdx.x & 31, at = blockIdx.y * kStepWarps + (threadIdx.x >> 5);
    const int head = at / runs, col0 = at % runs * CW;
    if (head >= p.heads) return;                     // (a warp of its own: no block-wide barrier here)
    const int seq = blockIdx.x, dim4 = (p.dim + 3) & ~3, qk_head = head / (p.heads / p.qk_heads);
    const int r = lane % LPC, col = col0 + lane / LPC * CPL;
    const float rate = KIND == MEMORY ? 0.0f : p.p0[head];
    const float bias0 = KIND == MEMORY ? p.p0[head] : p.p1[head], bias1 = KIND == MEMORY ? p.p1[head] : 0.0f;
    const float skip = KIND == STATE_SPACE ? p.p2[head] : 0.0f;
    pdl_wait();                                      // rows, state and the step's metadata come from kernels in front
    const int row = p.row_start[seq];
    if (row >= p.row_start[seq + 1]) return;
    const int64_t of_slot = (int64_t)p.state_slots[seq] * p.heads + head;
    float* state = p.state + (of_slot * p.columns + col) * dim4;
    ulonglong2 S[CPL][NJ];
#pragma unroll
    for (int j = 0; j < CPL; ++j)
#pragma unroll
        for (int i = 0; i < NJ; ++i) {
            const int e = 4 * (r + LPC * i);
            S[j][i] = col + j < p.columns && e < dim4 ? *reinterpret_cast<const ulonglong2*>(state + (int64_t)j * dim4 + e)
                                                      : make_ulonglong2(0ull, 0ull);
        }
    const T* x = rows + (int64_t)row * p.stride;
    float q[NJ][4], k[NJ][4];
#pragma unroll
    for (int i = 0; i < NJ; ++i) {
        const int e = 4 * (r + LPC * i);
        const T* qp = x + p.q_off + (int64_t)qk_head * p.dim + e;
        const T* kp = x + p.k_off + (int64_t)qk_head * p.dim + e;
        if (vec && e < p.dim) {
            const float4 a = load4<T>(qp), b = load4<T>(kp);
            q[i][0] = a.x; q[i][1] = a.y; q[i][2] = a.z; q[i][3] = a.w;
            k[i][0] = b.x; k[i][1] = b.y; k[i][2] = b.z; k[i][3] = b.w;
        } else {
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                q[i][t] = e + t < p.dim ? Elem<T>::load(qp + t) : 0.0f;
                k[i][t] = e + t < p.dim ? Elem<T>::load(kp + t) : 0.0f;
            }
        }
    }
    float v[CPL];
#pragma unroll
    for (int j = 0; j < CPL; ++j)
        v[j] = col + j < p.vdim ? Elem<T>::load(x + p.v_off + (int64_t)head * p.vdim + col + j)
                                : (KIND == MEMORY && col + j == p.vdim ? 1.0f : 0.0f);
    const float2 gate = gates_of<KIND>(logits_of<KIND>(p, row, head), p.cap, rate, bias0, bias1);
    float a = gate.x, w = gate.y;
    if (KIND == MEMORY) {
        const float before = p.running[of_slot * p.columns + min(col, p.columns - 1)];     // (every column holds the same)
        const float now = fmaxf(gate.x + before, gate.y);
        a = decay_of(gate.x + before - now);
        w = expf(gate.y - now);
        __syncwarp();
        if (r == 0) {
#pragma unroll
            for (int j = 0; j < CPL; ++j)
                if (col + j < p.columns) p.running[of_slot * p.columns + col + j] = now;
            if (col <= p.vdim && p.vdim < col + CPL) p.aux[((int64_t)row * p.heads + head) * 2 + 1] = now;
        }
    }
    float sums[3] = {0.0f, 0.0f, 0.0f};              // k . q, q . q, k . k
#pragma unroll
    for (int i = 0; i < NJ; ++i)
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            sums[0] = fmaf(k[i][t], q[i][t], sums[0]);
            if (KIND == DELTA) {
                sums[1] = fmaf(q[i][t], q[i][t], sums[1]);
                sums[2] = fmaf(k[i][t], k[i][t], sums[2]);
            }
        }
#pragma unroll
    for (int o = 1; o < LPC; o <<= 1)
#pragma unroll
        for (int i = 0; i < (KIND == DELTA ? 3 : 1); ++i) sums[i] += __shfl_xor_sync(0xffffffffu, sums[i], o);
    float iq = p.q_scale, ik = 1.0f;
    if (KIND == DELTA) {
        iq *= 1.0f / sqrtf(sums[1] + 1e-6f);
        ik = 1.0f / sqrtf(sums[2] + 1e-6f);
    }
    const pair32 a2 = pack2(a, a);
    float dq[CPL], u[CPL];
#pragma unroll
    for (int j = 0; j < CPL; ++j) {
        pair32 with_q = 0ull, with_k = 0ull;
#pragma unroll
        for (int i = 0; i < NJ; ++i) {
            with_q = fma2(S[j][i].x, pack2(q[i][0], q[i][1]), with_q);
            with_q = fma2(S[j][i].y, pack2(q[i][2], q[i][3]), with_q);
            if (KIND == DELTA) {
                with_k = fma2(S[j][i].x, pack2(k[i][0], k[i][1]), with_k);
                with_k = fma2(S[j][i].y, pack2(k[i][2], k[i][3]), with_k);
            }
        }
        dq[j] = sum2(with_q);
        u[j] = w * v[j];
        if (KIND == DELTA) {
            float d = sum2(with_k);
#pragma unroll
            for (int o = 1; o < LPC; o <<= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
            u[j] = w * (v[j] - a * ik * d);
        }
        const pair32 u2 = pack2(ik * u[j], ik * u[j]);
#pragma unroll
        for (int i = 0; i < NJ; ++i) {
            const int e = 4 * (r + LPC * i);
            if (col + j < p.columns && e < dim4)
                *reinterpret_cast<ulonglong2*>(state + (int64_t)j * dim4 + e) =
                    make_ulonglong2(fma2(pack2(k[i][0], k[i][1]), u2, mul2(S[j][i].x, a2)),
                                    fma2(pack2(k[i][2], k[i][3]), u2, mul2(S[j][i].y, a2)));
        }
#pragma unroll
        for (int o = 1; o < LPC; o <<= 1) dq[j] += __shfl_xor_sync(0xffffffffu, dq[j], o);
    }
    if (r == 0) {
        const int64_t to = (int64_t)row * p.heads + head;
#pragma unroll
        for (int j = 0; j < CPL; ++j) {
            float o = fmaf(u[j], iq * ik * sums[0], a * iq * dq[j]);
            if (KIND == STATE_SPACE) o = fmaf(skip, v[j], o);
            if (col + j < p.vdim) p.out[to * p.vdim + col + j] = o;
            else if (KIND == MEMORY && col + j == p.vdim) p.aux[to * 2] = o;
        }
    }
}

template <typename T, int KIND, int LPC, int NJ>
int launch_as(const void* rows, Recurrence p, int num_seqs, int single, cudaStream_t stream) {
    constexpr int CW = 32 / LPC * 2, DP = 4 * LPC * NJ;
    cudaError_t launched;
    if (single) {
        const int runs = (p.columns + CW - 1) / CW;
        const int64_t blocks = ((int64_t)p.heads * runs + kStepWarps - 1) / kStepWarps;
        if (blocks > 65535) return TB_ERR_BAD_SIZE;
        const int vec = p.dim % 4 == 0 && p.stride % 4 == 0 && p.q_off % 4 == 0 && p.k_off % 4 == 0 && (uintptr_t)rows % (4 * sizeof(T)) == 0;
        launched = tb_launch_pdl(matrix_recurrence_step_kernel<T, KIND, LPC, NJ>, dim3(num_seqs, (unsigned)blocks), dim3(kStepWarps * 32),
                                 (size_t)0, stream, (const T*)rows, p, runs, vec);
        return launched == cudaSuccess ? tb_launch_status() : (int)launched;
    }
    // few blocks: fewer columns a block, so that more multiprocessors take part
    p.workers = min(kWorkers, 32 / CW);
    while (p.workers > 1 && (int64_t)num_seqs * p.heads * ((p.columns + p.workers * CW - 1) / (p.workers * CW)) < kFewBlocks) p.workers /= 2;
    p.tile = DP > 512 ? kTile / 2 : kTile;
    const int VC = p.workers * CW;
    const size_t smem = sizeof(float) * 2 * (p.tile * (2 * DP + VC) + p.tile / kGroup * Coefficients<KIND>::N);
    auto kernel = matrix_recurrence_kernel<T, KIND, LPC, NJ>;
    if (smem > 40 * 1024) {
        cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (err != cudaSuccess) return (int)err;
    }
    const int runs = (p.columns + VC - 1) / VC;
    if (runs > 65535) return TB_ERR_BAD_SIZE;
    launched = tb_launch_pdl(kernel, dim3(num_seqs, p.heads, runs), dim3((p.workers + kProducers) * 32), smem, stream, (const T*)rows, p);
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}

template <typename T, int KIND>
int launch_kind(const void* rows, const Recurrence& p, int num_seqs, int single, cudaStream_t stream) {
    const int packets = (p.dim + 3) / 4;
    if (packets <= 8) return launch_as<T, KIND, 8, 1>(rows, p, num_seqs, single, stream);
    if (packets <= 16) return launch_as<T, KIND, 8, 2>(rows, p, num_seqs, single, stream);
    if (packets <= 24) return launch_as<T, KIND, 8, 3>(rows, p, num_seqs, single, stream);
    if (packets <= 32) {
        // (where whole blocks of 32 columns would leave multiprocessors idle, a column is shared by twice the lanes)
        if (single || (int64_t)num_seqs * p.heads * ((p.columns + 31) / 32) >= kFewBlocks) return launch_as<T, KIND, 8, 4>(rows, p, num_seqs, single, stream);
        return launch_as<T, KIND, 16, 2>(rows, p, num_seqs, single, stream);
    }
    if (packets <= 48) return launch_as<T, KIND, 16, 3>(rows, p, num_seqs, single, stream);
    if (packets <= 64) return launch_as<T, KIND, 16, 4>(rows, p, num_seqs, single, stream);
    if (packets <= 128) return launch_as<T, KIND, 32, 4>(rows, p, num_seqs, single, stream);
    return launch_as<T, KIND, 32, 8>(rows, p, num_seqs, single, stream);
}

template <typename T>
int launch_dtype(int kind, const void* rows, const Recurrence& p, int num_seqs, int single, cudaStream_t stream) {
    if (kind == STATE_SPACE) return launch_kind<T, STATE_SPACE>(rows, p, num_seqs, single, stream);
    if (kind == MEMORY) return launch_kind<T, MEMORY>(rows, p, num_seqs, single, stream);
    return launch_kind<T, DELTA>(rows, p, num_seqs, single, stream);
}

// ----------------------------------------------------------------------------- behind the recurrence

enum NormGate : int { GATE_SIGMOID = 0, GATE_SILU = 1, GATE_SILU_FIRST = 2 };
constexpr int kNormThreads = 128, kKeepNumbers = 8;

// (in a bfloat16 run the fast exponential and division, good to a few units of 2^-22, in front of a rounding to 2^-9)
template <typename T>
__device__ __forceinline__ float gate_factor(float g, int gate_kind) {
    const float s = sizeof(T) == 4 ? 1.0f / (1.0f + expf(-g)) : __fdividef(1.0f, 1.0f + __expf(-g));
    return gate_kind == GATE_SIGMOID ? s : g * s;
}

// A warp (WIDE: the block) a (row, group); a lane keeps its first numbers in registers between the statistic and the output.
template <typename T, bool WIDE>
__global__ void __launch_bounds__(kNormThreads)
recurrence_norm_kernel(const float* __restrict__ v, const float* __restrict__ aux, const T* __restrict__ gate,
                       int64_t gate_stride, const float* __restrict__ weight, int weight_len, T* __restrict__ out,
                       int64_t out_stride, int groups, int size, float eps, int gate_kind) {
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    constexpr int STEP = WIDE ? kNormThreads : 32;
    const int lane = WIDE ? threadIdx.x : threadIdx.x & 31;
    const int row = blockIdx.x;
    const int g = WIDE ? blockIdx.y : blockIdx.y * (kNormThreads / 32) + (threadIdx.x >> 5);
    if (g >= groups) return;                         // (a warp of its own: the block-wide sum runs in WIDE only)
    const float* src = v + ((int64_t)row * groups + g) * size;
    const T* grow = gate + (int64_t)row * gate_stride + (int64_t)g * size;
    T* dst = out + (int64_t)row * out_stride + (int64_t)g * size;
    const float* w = weight + (weight_len == size ? 0 : (int64_t)g * size);
    float before = 1.0f;
    if (aux != nullptr) {
        const float* a = aux + ((int64_t)row * groups + g) * 2;
        before = 1.0f / (fmaxf(fabsf(a[0]), expf(-a[1])) + 1e-6f);
    }
    auto value = [&](int i) {
        const float x = src[i] * before;
        return gate_kind == GATE_SILU_FIRST ? x * gate_factor<T>(Elem<T>::load(grow + i), gate_kind) : x;
    };
    float kept[kKeepNumbers], ss = 0.0f;
#pragma unroll
    for (int e = 0; e < kKeepNumbers; ++e) {
        const int i = e * STEP + lane;
        kept[e] = i < size ? value(i) : 0.0f;
        ss = fmaf(kept[e], kept[e], ss);
    }
    for (int i = kKeepNumbers * STEP + lane; i < size; i += STEP) {
        const float x = value(i);
        ss = fmaf(x, x, ss);
    }
    const float total = WIDE ? block_sum(ss, scratch) : warp_sum(ss);
    const float inv = 1.0f / sqrtf(total / (float)size + eps);
    auto finish = [&](int i, float x) {
        x *= inv * w[i];
        if (gate_kind != GATE_SILU_FIRST) x *= gate_factor<T>(Elem<T>::load(grow + i), gate_kind);
        Elem<T>::store(dst + i, x);
    };
#pragma unroll
    for (int e = 0; e < kKeepNumbers; ++e) {
        const int i = e * STEP + lane;
        if (i < size) finish(i, kept[e]);
    }
    for (int i = kKeepNumbers * STEP + lane; i < size; i += STEP) finish(i, value(i));
}

// The same in packets of four numbers, where sizes and rows allow them.
template <typename T, bool WIDE, int KEEP>
__global__ void __launch_bounds__(WIDE ? 256 : kNormThreads)
recurrence_norm_packets_kernel(const float* __restrict__ v, const float* __restrict__ aux, const T* __restrict__ gate,
                               int64_t gate_stride, const float* __restrict__ weight, int weight_len, T* __restrict__ out,
                               int64_t out_stride, int groups, int size, float eps, int gate_kind) {
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    constexpr int STEP = WIDE ? 256 : 32;            // rows of up to 4 * STEP * KEEP numbers
    const int lane = WIDE ? threadIdx.x : threadIdx.x & 31;
    const int row = blockIdx.x;
    const int g = WIDE ? blockIdx.y : blockIdx.y * (kNormThreads / 32) + (threadIdx.x >> 5);
    if (g >= groups) return;
    const float* src = v + ((int64_t)row * groups + g) * size;
    const T* grow = gate + (int64_t)row * gate_stride + (int64_t)g * size;
    T* dst = out + (int64_t)row * out_stride + (int64_t)g * size;
    const float* w = weight + (weight_len == size ? 0 : (int64_t)g * size);
    const int packets = size / 4;
    float4 x[KEEP], z[KEEP];
    float before = 1.0f;
#pragma unroll
    for (int e = 0; e < KEEP; ++e) {                 // everything the row needs is asked for at once
        const int i = 4 * (e * STEP + lane);
        const bool there = e * STEP + lane < packets;
        x[e] = there ? *reinterpret_cast<const float4*>(src + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        z[e] = there ? load4<T>(grow + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    if (aux != nullptr) {
        const float* a = aux + ((int64_t)row * groups + g) * 2;
        before = 1.0f / (fmaxf(fabsf(a[0]), expf(-a[1])) + 1e-6f);
    }
    float ss = 0.0f;
#pragma unroll
    for (int e = 0; e < KEEP; ++e) {
        z[e].x = gate_factor<T>(z[e].x, gate_kind); z[e].y = gate_factor<T>(z[e].y, gate_kind);
        z[e].z = gate_factor<T>(z[e].z, gate_kind); z[e].w = gate_factor<T>(z[e].w, gate_kind);
        x[e].x *= before; x[e].y *= before; x[e].z *= before; x[e].w *= before;
        if (gate_kind == GATE_SILU_FIRST) { x[e].x *= z[e].x; x[e].y *= z[e].y; x[e].z *= z[e].z; x[e].w *= z[e].w; }
        ss = fmaf(x[e].x, x[e].x, ss); ss = fmaf(x[e].y, x[e].y, ss);
        ss = fmaf(x[e].z, x[e].z, ss); ss = fmaf(x[e].w, x[e].w, ss);
    }
    const float total = WIDE ? block_sum(ss, scratch) : warp_sum(ss);
    const float inv = 1.0f / sqrtf(total / (float)size + eps);
#pragma unroll
    for (int e = 0; e < KEEP; ++e) {
        const int i = 4 * (e * STEP + lane);
        if (e * STEP + lane >= packets) continue;
        const float4 f = *reinterpret_cast<const float4*>(w + i);
        float4 y = make_float4(x[e].x * inv * f.x, x[e].y * inv * f.y, x[e].z * inv * f.z, x[e].w * inv * f.w);
        if (gate_kind != GATE_SILU_FIRST) { y.x *= z[e].x; y.y *= z[e].y; y.z *= z[e].z; y.w *= z[e].w; }
        store4<T>(dst + i, y);
    }
}

template <typename T>
int launch_norm(const float* v, const float* aux, const void* gate, int64_t gate_stride, const float* weight, int weight_len,
                void* out, int64_t out_stride, int rows, int groups, int size, float eps, int gate_kind, cudaStream_t stream) {
    const uintptr_t bits = (uintptr_t)v | (uintptr_t)weight;
    const uintptr_t row_bits = (uintptr_t)gate | (uintptr_t)out;
    const bool packets = size % 4 == 0 && bits % 16 == 0 && row_bits % (4 * sizeof(T)) == 0 && gate_stride % 4 == 0 && out_stride % 4 == 0;
    cudaError_t launched;
#define TB_NORM(KERNEL, GRID, THREADS)                                                                                      \
    launched = tb_launch_pdl(KERNEL, GRID, dim3(THREADS), (size_t)0, stream, v, aux, (const T*)gate, gate_stride, weight,   \
                             weight_len, (T*)out, out_stride, groups, size, eps, gate_kind)
    const dim3 narrow(rows, (groups + 3) / 4), wide(rows, groups);
    if (packets && size <= 128) TB_NORM((recurrence_norm_packets_kernel<T, false, 1>), narrow, kNormThreads);
    else if (packets && size <= 256) TB_NORM((recurrence_norm_packets_kernel<T, false, 2>), narrow, kNormThreads);
    else if (packets && size <= 1024) TB_NORM((recurrence_norm_packets_kernel<T, false, 8>), narrow, kNormThreads);
    else if (packets && size <= 4096) TB_NORM((recurrence_norm_packets_kernel<T, true, 4>), wide, 256);
    else if (packets && size <= 8192) TB_NORM((recurrence_norm_packets_kernel<T, true, 8>), wide, 256);
    else if (size <= 256) TB_NORM((recurrence_norm_kernel<T, false>), narrow, kNormThreads);
    else TB_NORM((recurrence_norm_kernel<T, true>), wide, kNormThreads);
#undef TB_NORM
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}

}  // namespace

// rows: [rows, ...] in `dtype`, row stride `stride` (elements); q at column q_off and k at k_off ([qk_heads, dim] each), v at v_off
// ([heads, vdim]).  gates: float32 logits, a row [heads] (kind 0) or [2 * heads] (kind 1: input, forget; kind 2: decay, write).
// p0, p1, p2: float32 [heads], see Recurrence.  state: float32 [slots, heads, columns, dim rounded up to 4] with columns = vdim, or
// vdim + 1 for kind 1, and then running: float32 [slots, heads, columns].  out: float32 [rows, heads * vdim]; aux (kind 1): float32
// [rows, heads, 2].  single: every sequence brings at most one row.
TB_EXPORT int tb_matrix_recurrence(int kind, const void* rows, int64_t stride, int q_off, int k_off, int v_off,
                                   const float* gates, int64_t gate_stride, const float* p0, const float* p1, const float* p2,
                                   float cap, float q_scale, float* state, float* running, float* out, float* aux,
                                   const int* row_start, const int* state_slots, int num_seqs, int heads, int qk_heads, int dim,
                                   int vdim, int single, int dtype, cudaStream_t stream) {
    if (num_seqs == 0) return 0;
    if (kind < STATE_SPACE || kind > DELTA || heads < 1 || heads > 65535 || qk_heads < 1 || heads % qk_heads != 0 || dim < 1 ||
        dim > 1024 || vdim < 1)
        return TB_ERR_BAD_SIZE;
    if (kind == MEMORY && (running == nullptr || aux == nullptr || !(cap > 0.0f))) return TB_ERR_BAD_SIZE;
    if (kind == STATE_SPACE && p2 == nullptr) return TB_ERR_BAD_SIZE;
    if ((uintptr_t)state % 16 != 0) return TB_ERR_BAD_ALIGN;
    Recurrence p;
    p.stride = stride; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
    p.gates = gates; p.gate_stride = gate_stride; p.p0 = p0; p.p1 = p1; p.p2 = p2; p.cap = cap; p.q_scale = q_scale;
    p.state = state; p.running = running; p.out = out; p.aux = aux; p.row_start = row_start; p.state_slots = state_slots;
    p.heads = heads; p.qk_heads = qk_heads; p.dim = dim; p.vdim = vdim; p.columns = kind == MEMORY ? vdim + 1 : vdim;
    p.workers = 1; p.tile = kTile;
    if (dtype == TB_F32) return launch_dtype<float>(kind, rows, p, num_seqs, single, stream);
    if (dtype == TB_BF16) return launch_dtype<__nv_bfloat16>(kind, rows, p, num_seqs, single, stream);
    return TB_ERR_BAD_DTYPE;
}

// v: float32 [rows, groups * size], contiguous; aux: null or float32 [rows, groups, 2] as tb_matrix_recurrence leaves it; gate and out:
// [rows, >= groups * size] in `dtype`; weight: float32 of `size` (shared by the groups) or groups * size numbers.  gate_kind: 0
// sigmoid behind the norm, 1 SiLU behind it, 2 SiLU in front of it.
TB_EXPORT int tb_recurrence_norm(const float* v, const float* aux, const void* gate, int64_t gate_stride, const float* weight,
                                 int weight_len, void* out, int64_t out_stride, int rows, int groups, int size, float eps,
                                 int gate_kind, int dtype, cudaStream_t stream) {
    if (rows == 0) return 0;
    if (groups < 1 || groups > 65535 || size < 1 || (weight_len != size && weight_len != groups * size) || gate_kind < GATE_SIGMOID ||
        gate_kind > GATE_SILU_FIRST)
        return TB_ERR_BAD_SIZE;
    if (dtype == TB_F32)
        return launch_norm<float>(v, aux, gate, gate_stride, weight, weight_len, out, out_stride, rows, groups, size, eps, gate_kind, stream);
    if (dtype == TB_BF16)
        return launch_norm<__nv_bfloat16>(v, aux, gate, gate_stride, weight, weight_len, out, out_stride, rows, groups, size, eps,
                                          gate_kind, stream);
    return TB_ERR_BAD_DTYPE;
}
