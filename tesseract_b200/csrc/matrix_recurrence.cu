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
// A block takes one (sequence, head, run of value columns) and walks the sequence's rows of this step one after the other,
// the state in registers: a warp holds 32 / LPC groups of CPL columns, a column's numbers are shared by LPC lanes (lane r takes
// the packets of four r, r + LPC, ...).  Both products read the state in front of the token,
//
//   o = a (S_(t-1)^T q) + u (k . q),
//
// so a token's update does not wait for its own output.  Four more warps run a tile of rows ahead: they widen q, k and v into
// shared memory and take gates, norms and k . q.  A token's numbers depend on the state and on its own row alone, so a prompt
// may be cut anywhere without changing a bit.  State layout: [slots][heads][columns][dim rounded up to four].
//
// tb_recurrence_norm (behind it): per row and group of `size` numbers, optionally first v / (max(|n . q|, e^-m) + 1e-6) and / or
// v silu(gate), then v / sqrt(mean(v^2) + eps) * weight, then optionally times sigmoid or SiLU of the gate; rounded once.
#include "common.cuh"

namespace {

enum Kind : int { STATE_SPACE = 0, MEMORY = 1, DELTA = 2 };
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
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }

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

template <typename T, int KIND, int LPC, int NJ, int CPL>
__global__ void __launch_bounds__((4 + kProducers) * 32)
matrix_recurrence_kernel(const T* __restrict__ rows, Recurrence p) {
    constexpr int DP = 4 * LPC * NJ;                 // numbers of q or k in shared memory (zeros behind dim)
    constexpr int GROUPS = 32 / LPC, CW = GROUPS * CPL;
    constexpr int E = DP / 32;                       // numbers of q or k a producer's lane carries
    extern __shared__ __align__(16) float smem[];
    pdl_trigger();
    const int W = p.workers, TT = p.tile, VC = W * CW;
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * VC;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int dim4 = (p.dim + 3) & ~3;
    const int stage = TT * (2 * DP + VC + 5);        // floats of a buffer: q, k, v, then five scalars a row
    pdl_wait();                                      // rows, state and the step's metadata come from kernels in front
    const int first = p.row_start[seq], n = p.row_start[seq + 1] - first;
    if (n <= 0) return;
    const int tiles = (n + TT - 1) / TT;
    const int64_t of_slot = (int64_t)p.state_slots[seq] * p.heads + head;
    const bool produces = warp >= W;
    const int qk_head = head / (p.heads / p.qk_heads);

    // consumers: the state of this warp's columns
    const int r = lane % LPC, group = lane / LPC;
    const int wcol = warp * CW + group * CPL;        // the group's first column within the block
    pair32 S[CPL][NJ][2];
    if (!produces) {
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
    }
    float m = 0.0f;                                  // MEMORY: the running maximum, in the first producer's lanes
    if (KIND == MEMORY && warp == W) m = p.running[of_slot * p.columns + col0];
    const float bias0 = KIND == MEMORY ? p.p0[head] : p.p1[head], bias1 = KIND == MEMORY ? p.p1[head] : 0.0f;
    const float rate = KIND == MEMORY ? 0.0f : p.p0[head];
    const float skip = KIND == STATE_SPACE ? p.p2[head] : 0.0f;

    auto produce = [&](int tile, float* buffer) {
        float *qs = buffer, *ks = qs + TT * DP, *vs = ks + TT * DP, *sc = vs + TT * VC;   // sc: a, w, iq, ik, k.q
        const int count = min(TT, n - tile * TT), row0 = first + tile * TT;
        if (warp == W) {                             // gates: a lane a row
            float a = 0.0f, w = 0.0f;
            float log_f = 0.0f, log_i = 0.0f;
            if (lane < count) {
                const float* gate = p.gates + (int64_t)(row0 + lane) * p.gate_stride;
                if (KIND == STATE_SPACE) {
                    w = softplus(gate[head] + bias0);
                    a = expf(rate * w);
                } else if (KIND == DELTA) {
                    a = expf(rate * softplus(gate[head] + bias0));
                    w = 1.0f / (1.0f + expf(-gate[p.heads + head]));
                } else {
                    log_i = p.cap * tanhf((gate[head] + bias0) / p.cap);
                    log_f = log_sigmoid(p.cap * tanhf((gate[p.heads + head] + bias1) / p.cap));
                }
            }
            if (KIND == MEMORY) {
                float before = 0.0f, now = 0.0f;
                for (int t = 0; t < count; ++t) {    // in token order, whatever the tile
                    const float f = __shfl_sync(0xffffffffu, log_f, t), i = __shfl_sync(0xffffffffu, log_i, t);
                    const float next = fmaxf(f + m, i);
                    if (lane == t) { before = m; now = next; }
                    m = next;
                }
                a = expf(log_f + before - now);
                w = expf(log_i - now);
                if (lane < count && col0 <= p.vdim && p.vdim < col0 + VC)
                    p.aux[((int64_t)(row0 + lane) * p.heads + head) * 2 + 1] = now;
            }
            if (lane < count) {
                sc[lane * 5] = a;
                sc[lane * 5 + 1] = w;
            }
        }
        for (int t = warp - W; t < count; t += kProducers) {
            const T* row = rows + (int64_t)(row0 + t) * p.stride;
            const T* q = row + p.q_off + (int64_t)qk_head * p.dim;
            const T* k = row + p.k_off + (int64_t)qk_head * p.dim;
            const T* v = row + p.v_off + (int64_t)head * p.vdim + col0;
            float qv[E], kv[E];
#pragma unroll
            for (int i = 0; i < E; ++i) {
                const int e = i * 32 + lane;
                qv[i] = e < p.dim ? Elem<T>::load(q + e) : 0.0f;
                kv[i] = e < p.dim ? Elem<T>::load(k + e) : 0.0f;
            }
            for (int c = lane; c < VC; c += 32) {
                const int col = col0 + c;
                vs[t * VC + c] = col < p.vdim ? Elem<T>::load(v + c) : (KIND == MEMORY && col == p.vdim ? 1.0f : 0.0f);
            }
            float qq = 0.0f, kk = 0.0f, kq = 0.0f;
#pragma unroll
            for (int i = 0; i < E; ++i) {
                qs[t * DP + i * 32 + lane] = qv[i];
                ks[t * DP + i * 32 + lane] = kv[i];
                kq = fmaf(kv[i], qv[i], kq);
                if (KIND == DELTA) {
                    qq = fmaf(qv[i], qv[i], qq);
                    kk = fmaf(kv[i], kv[i], kk);
                }
            }
            kq = warp_sum(kq);
            float iq = p.q_scale, ik = 1.0f;
            if (KIND == DELTA) {
                iq *= 1.0f / sqrtf(warp_sum(qq) + 1e-6f);
                ik = 1.0f / sqrtf(warp_sum(kk) + 1e-6f);
            }
            if (lane == 0) {
                sc[t * 5 + 2] = iq;
                sc[t * 5 + 3] = ik;
                sc[t * 5 + 4] = iq * ik * kq;
            }
        }
    };

    if (produces) produce(0, smem);
    __syncthreads();
    for (int tile = 0; tile < tiles; ++tile) {
        float* buffer = smem + (tile & 1) * stage;
        if (produces) {
            if (tile + 1 < tiles) produce(tile + 1, smem + ((tile + 1) & 1) * stage);
        } else {
            const float *qs = buffer, *ks = qs + TT * DP, *vs = ks + TT * DP, *sc = vs + TT * VC;
            const int count = min(TT, n - tile * TT), row0 = first + tile * TT;
            for (int t = 0; t < count; ++t) {
                const ulonglong2* q2 = reinterpret_cast<const ulonglong2*>(qs + t * DP) + r;
                const ulonglong2* k2 = reinterpret_cast<const ulonglong2*>(ks + t * DP) + r;
                const float a = sc[t * 5], w = sc[t * 5 + 1], iq = sc[t * 5 + 2], ik = sc[t * 5 + 3], kq = sc[t * 5 + 4];
                float v[CPL], u[CPL];
#pragma unroll
                for (int j = 0; j < CPL; ++j) v[j] = vs[t * VC + wcol + j];
                const pair32 a2 = pack2(a, a);
                pair32 dq[CPL][2];
#pragma unroll
                for (int j = 0; j < CPL; ++j) dq[j][0] = dq[j][1] = 0ull;
                if (KIND == DELTA) {
                    pair32 dk[CPL][2];
#pragma unroll
                    for (int j = 0; j < CPL; ++j) dk[j][0] = dk[j][1] = 0ull;
#pragma unroll
                    for (int i = 0; i < NJ; ++i) {
                        const ulonglong2 kv = k2[LPC * i], qv = q2[LPC * i];
#pragma unroll
                        for (int j = 0; j < CPL; ++j) {
                            dk[j][0] = fma2(S[j][i][0], kv.x, dk[j][0]);
                            dk[j][1] = fma2(S[j][i][1], kv.y, dk[j][1]);
                            dq[j][0] = fma2(S[j][i][0], qv.x, dq[j][0]);
                            dq[j][1] = fma2(S[j][i][1], qv.y, dq[j][1]);
                        }
                    }
#pragma unroll
                    for (int j = 0; j < CPL; ++j) {
                        float d = sum2(dk[j][0]) + sum2(dk[j][1]);
#pragma unroll
                        for (int o = 1; o < LPC; o <<= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
                        u[j] = w * (v[j] - a * ik * d);
                    }
#pragma unroll
                    for (int j = 0; j < CPL; ++j) {
                        const pair32 u2 = pack2(ik * u[j], ik * u[j]);
#pragma unroll
                        for (int i = 0; i < NJ; ++i) {
                            const ulonglong2 kv = k2[LPC * i];
                            S[j][i][0] = fma2(kv.x, u2, mul2(S[j][i][0], a2));
                            S[j][i][1] = fma2(kv.y, u2, mul2(S[j][i][1], a2));
                        }
                    }
                } else {
                    pair32 u2[CPL];
#pragma unroll
                    for (int j = 0; j < CPL; ++j) {
                        u[j] = w * v[j];
                        u2[j] = pack2(u[j], u[j]);
                    }
#pragma unroll
                    for (int i = 0; i < NJ; ++i) {
                        const ulonglong2 kv = k2[LPC * i], qv = q2[LPC * i];
#pragma unroll
                        for (int j = 0; j < CPL; ++j) {
                            dq[j][0] = fma2(S[j][i][0], qv.x, dq[j][0]);
                            dq[j][1] = fma2(S[j][i][1], qv.y, dq[j][1]);
                            S[j][i][0] = fma2(kv.x, u2[j], mul2(S[j][i][0], a2));
                            S[j][i][1] = fma2(kv.y, u2[j], mul2(S[j][i][1], a2));
                        }
                    }
                }
                // the lanes' shares of S^T q: two columns meet in one butterfly, the odd lanes keeping the second
                static_assert(CPL == 2, "the butterfly below is written for two columns a group");
                const bool odd = r & 1;
                const float d0 = sum2(dq[0][0]) + sum2(dq[0][1]), d1 = sum2(dq[1][0]) + sum2(dq[1][1]);
                float d = (odd ? d1 : d0) + __shfl_xor_sync(0xffffffffu, odd ? d0 : d1, 1);
#pragma unroll
                for (int o = 2; o < LPC; o <<= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
                const float uj = odd ? u[1] : u[0];
                float o = fmaf(uj, kq, a * iq * d);
                if (KIND == STATE_SPACE) o = fmaf(skip, odd ? v[1] : v[0], o);
                const int col = col0 + wcol + (odd ? 1 : 0);
                if (r < 2) {
                    const int64_t at = (int64_t)(row0 + t) * p.heads + head;
                    if (col < p.vdim) p.out[at * p.vdim + col] = o;
                    else if (KIND == MEMORY && col == p.vdim) p.aux[at * 2] = o;
                }
            }
        }
        __syncthreads();
    }
    if (!produces) {
#pragma unroll
        for (int j = 0; j < CPL; ++j) {
            const int col = col0 + wcol + j;
            float* at = p.state + (of_slot * p.columns + col) * dim4;
#pragma unroll
            for (int i = 0; i < NJ; ++i) {
                const int e = 4 * (r + LPC * i);
                if (col < p.columns && e < dim4)
                    *reinterpret_cast<ulonglong2*>(at + e) = make_ulonglong2(S[j][i][0], S[j][i][1]);
            }
        }
    } else if (KIND == MEMORY && warp == W) {
        for (int c = lane; c < VC && col0 + c < p.columns; c += 32) p.running[of_slot * p.columns + col0 + c] = m;
    }
}

template <typename T, int KIND, int LPC, int NJ>
int launch_as(const void* rows, Recurrence p, int num_seqs, cudaStream_t stream) {
    constexpr int CPL = 2, CW = 32 / LPC * CPL, DP = 4 * LPC * NJ;
    // few blocks: fewer columns a block, so that more multiprocessors take part
    p.workers = 4;
    while (p.workers > 1 && (int64_t)num_seqs * p.heads * ((p.columns + p.workers * CW - 1) / (p.workers * CW)) < 120) p.workers /= 2;
    p.tile = DP > 512 ? 8 : 16;
    const int VC = p.workers * CW;
    const size_t smem = sizeof(float) * 2 * p.tile * (2 * DP + VC + 5);
    auto kernel = matrix_recurrence_kernel<T, KIND, LPC, NJ, CPL>;
    if (smem > 40 * 1024) {
        cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (err != cudaSuccess) return (int)err;
    }
    const int runs = (p.columns + VC - 1) / VC;
    if (runs > 65535) return TB_ERR_BAD_SIZE;
    cudaError_t launched = tb_launch_pdl(kernel, dim3(num_seqs, p.heads, runs), dim3((p.workers + kProducers) * 32), smem,
                                         stream, (const T*)rows, p);
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}

template <typename T, int KIND>
int launch_kind(const void* rows, const Recurrence& p, int num_seqs, cudaStream_t stream) {
    const int packets = (p.dim + 3) / 4;
    if (packets <= 8) return launch_as<T, KIND, 8, 1>(rows, p, num_seqs, stream);
    if (packets <= 16) return launch_as<T, KIND, 8, 2>(rows, p, num_seqs, stream);
    if (packets <= 24) return launch_as<T, KIND, 8, 3>(rows, p, num_seqs, stream);
    if (packets <= 32) return launch_as<T, KIND, 8, 4>(rows, p, num_seqs, stream);
    if (packets <= 48) return launch_as<T, KIND, 8, 6>(rows, p, num_seqs, stream);
    if (packets <= 64) return launch_as<T, KIND, 8, 8>(rows, p, num_seqs, stream);
    if (packets <= 128) return launch_as<T, KIND, 32, 4>(rows, p, num_seqs, stream);
    return launch_as<T, KIND, 32, 8>(rows, p, num_seqs, stream);
}

template <typename T>
int launch_dtype(int kind, const void* rows, const Recurrence& p, int num_seqs, cudaStream_t stream) {
    if (kind == STATE_SPACE) return launch_kind<T, STATE_SPACE>(rows, p, num_seqs, stream);
    if (kind == MEMORY) return launch_kind<T, MEMORY>(rows, p, num_seqs, stream);
    return launch_kind<T, DELTA>(rows, p, num_seqs, stream);
}

// ----------------------------------------------------------------------------- behind the recurrence

enum NormGate : int { GATE_SIGMOID = 0, GATE_SILU = 1, GATE_SILU_FIRST = 2 };
constexpr int kNormThreads = 128, kKeepNumbers = 8;

__device__ __forceinline__ float gate_factor(float g, int gate_kind) {
    const float s = 1.0f / (1.0f + expf(-g));
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
        return gate_kind == GATE_SILU_FIRST ? x * gate_factor(Elem<T>::load(grow + i), gate_kind) : x;
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
        if (gate_kind != GATE_SILU_FIRST) x *= gate_factor(Elem<T>::load(grow + i), gate_kind);
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

template <typename T, bool WIDE>
__global__ void __launch_bounds__(WIDE ? 256 : kNormThreads)
recurrence_norm_packets_kernel(const float* __restrict__ v, const float* __restrict__ aux, const T* __restrict__ gate,
                               int64_t gate_stride, const float* __restrict__ weight, int weight_len, T* __restrict__ out,
                               int64_t out_stride, int groups, int size, float eps, int gate_kind) {
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    constexpr int STEP = WIDE ? 256 : 32, KEEP = WIDE ? 8 : 2;
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
        z[e].x = gate_factor(z[e].x, gate_kind); z[e].y = gate_factor(z[e].y, gate_kind);
        z[e].z = gate_factor(z[e].z, gate_kind); z[e].w = gate_factor(z[e].w, gate_kind);
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
    if (packets && size <= 256) TB_NORM((recurrence_norm_packets_kernel<T, false>), narrow, kNormThreads);
    else if (packets && size <= 8192) TB_NORM((recurrence_norm_packets_kernel<T, true>), wide, 256);
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
// [rows, heads, 2].
TB_EXPORT int tb_matrix_recurrence(int kind, const void* rows, int64_t stride, int q_off, int k_off, int v_off,
                                   const float* gates, int64_t gate_stride, const float* p0, const float* p1, const float* p2,
                                   float cap, float q_scale, float* state, float* running, float* out, float* aux,
                                   const int* row_start, const int* state_slots, int num_seqs, int heads, int qk_heads, int dim,
                                   int vdim, int dtype, cudaStream_t stream) {
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
    p.workers = 4; p.tile = 16;
    if (dtype == TB_F32) return launch_dtype<float>(kind, rows, p, num_seqs, stream);
    if (dtype == TB_BF16) return launch_dtype<__nv_bfloat16>(kind, rows, p, num_seqs, stream);
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
