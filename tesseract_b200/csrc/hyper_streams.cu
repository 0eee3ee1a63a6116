// A residual stream kept as several 32-bit copies side by side ([rows, S * width], copy s at column s * width):
//
//   tb_mixed_streams_norm   with an update:  x_t <- sum_s mix[s, t] x_s + share[t] * y     (all copies from the old ones),
//                           y = scale_a * update_a + scale_b * update_b (the second optional); then, optionally, what the
//                           next sublayer reads:  u = sum_s take[s] x_s,  out = u / sqrt(mean(u^2) + eps) * weight
//   tb_bigram_embedding     every copy = table[token] + pairs[row], where row = (token in front * mul_prev + token * mul_cur)
//                           mod buckets, or `buckets` for a sequence's first token; the token in front of a step's first token
//                           comes from the request's state and the step's last token goes there
//
// One block a row of the stream.  A thread owns the same columns of all copies, so the copies are read once and written once, in
// place, and u stays in registers between the statistic and the output where the row is short enough.  The order of a row's sum
// of squares depends on the width alone.  All arithmetic is 32-bit; an output is rounded once.
#include "common.cuh"

namespace {

constexpr int kThreads = 256;
constexpr int kKeep = 4;             // packets of four a thread keeps: rows of up to 4096 numbers stay in registers
constexpr int kMaxStreams = 32;

struct Streams {
    const float *update_a, *update_b;
    float scale_a, scale_b;
    const float *mix, *share, *take, *weight;
    int width, streams;
    float eps;
};

// S > 0: that many copies, their packets in registers; S == 0: any number up to kMaxStreams, one column a thread at a time.
template <typename T, int S>
__global__ void __launch_bounds__(kThreads)
mixed_streams_norm_kernel(float* __restrict__ residual, T* __restrict__ out, Streams p) {
    __shared__ float scratch[32];
    pdl_trigger();
    const int W = p.width;
    constexpr int C = S > 0 ? S : 1;
    float mix[C][C], share[C], take[C];
    if (S > 0) {                                      // (weights: not written by any kernel in front)
#pragma unroll
        for (int t = 0; t < C; ++t) {
            share[t] = p.share != nullptr ? p.share[t] : 0.0f;
            take[t] = p.take != nullptr ? p.take[t] : 0.0f;
#pragma unroll
            for (int s = 0; s < C; ++s) mix[s][t] = p.mix != nullptr ? p.mix[s * C + t] : 0.0f;
        }
    }
    pdl_wait();
    const int64_t row = blockIdx.x;
    float* res = residual + row * p.streams * W;
    const float* ua = p.update_a == nullptr ? nullptr : p.update_a + row * W;
    const float* ub = p.update_b == nullptr ? nullptr : p.update_b + row * W;
    T* to = out == nullptr ? nullptr : out + row * W;
    float ss = 0.0f;
    if constexpr (S > 0) {
        float4 kept[kKeep];
        const int packets = W / 4;
        auto column = [&](int i) {                    // the new copies of columns i .. i + 3 are stored; what the next sublayer reads comes back
            float4 x[S];
#pragma unroll
            for (int s = 0; s < S; ++s) x[s] = *reinterpret_cast<const float4*>(res + (int64_t)s * W + i);
            if (ua != nullptr) {
                float4 y = *reinterpret_cast<const float4*>(ua + i);
                y.x *= p.scale_a; y.y *= p.scale_a; y.z *= p.scale_a; y.w *= p.scale_a;
                if (ub != nullptr) {
                    const float4 z = *reinterpret_cast<const float4*>(ub + i);
                    y.x = fmaf(p.scale_b, z.x, y.x); y.y = fmaf(p.scale_b, z.y, y.y);
                    y.z = fmaf(p.scale_b, z.z, y.z); y.w = fmaf(p.scale_b, z.w, y.w);
                }
                float4 n[S];
#pragma unroll
                for (int t = 0; t < S; ++t) {
                    n[t] = make_float4(share[t] * y.x, share[t] * y.y, share[t] * y.z, share[t] * y.w);
#pragma unroll
                    for (int s = 0; s < S; ++s) {
                        n[t].x = fmaf(mix[s][t], x[s].x, n[t].x); n[t].y = fmaf(mix[s][t], x[s].y, n[t].y);
                        n[t].z = fmaf(mix[s][t], x[s].z, n[t].z); n[t].w = fmaf(mix[s][t], x[s].w, n[t].w);
                    }
                    *reinterpret_cast<float4*>(res + (int64_t)t * W + i) = n[t];
                }
#pragma unroll
                for (int s = 0; s < S; ++s) x[s] = n[s];
            }
            float4 u = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (int s = 0; s < S; ++s) {
                u.x = fmaf(take[s], x[s].x, u.x); u.y = fmaf(take[s], x[s].y, u.y);
                u.z = fmaf(take[s], x[s].z, u.z); u.w = fmaf(take[s], x[s].w, u.w);
            }
            return u;
        };
        auto again = [&](int i) {                     // (its own stores)
            float4 u = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (int s = 0; s < S; ++s) {
                const float4 x = *reinterpret_cast<const float4*>(res + (int64_t)s * W + i);
                u.x = fmaf(take[s], x.x, u.x); u.y = fmaf(take[s], x.y, u.y);
                u.z = fmaf(take[s], x.z, u.z); u.w = fmaf(take[s], x.w, u.w);
            }
            return u;
        };
        auto square = [&](const float4& u) {
            ss = fmaf(u.x, u.x, ss); ss = fmaf(u.y, u.y, ss); ss = fmaf(u.z, u.z, ss); ss = fmaf(u.w, u.w, ss);
        };
#pragma unroll
        for (int n = 0; n < kKeep; ++n) {
            const int q = n * kThreads + threadIdx.x;
            if (q < packets) {
                kept[n] = column(q * 4);
                square(kept[n]);
            }
        }
        for (int q = kKeep * kThreads + threadIdx.x; q < packets; q += kThreads) square(column(q * 4));
        if (to == nullptr) return;
        const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)W + p.eps);
        auto finish = [&](int i, const float4& u) {
            const float4 w = *reinterpret_cast<const float4*>(p.weight + i);
            const float v[4] = {u.x * inv * w.x, u.y * inv * w.y, u.z * inv * w.z, u.w * inv * w.w};
            if constexpr (sizeof(T) == 4) {
                *reinterpret_cast<float4*>(to + i) = make_float4(v[0], v[1], v[2], v[3]);
            } else {
                __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
                *reinterpret_cast<uint2*>(to + i) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
            }
        };
#pragma unroll
        for (int n = 0; n < kKeep; ++n) {
            const int q = n * kThreads + threadIdx.x;
            if (q < packets) finish(q * 4, kept[n]);
        }
        for (int q = kKeep * kThreads + threadIdx.x; q < packets; q += kThreads) finish(q * 4, again(q * 4));
    } else {
        const int N = p.streams;
        for (int i = threadIdx.x; i < W; i += kThreads) {
            float old[kMaxStreams], y = 0.0f, u = 0.0f;
            for (int s = 0; s < N; ++s) old[s] = res[(int64_t)s * W + i];
            if (ua != nullptr) {
                y = p.scale_a * ua[i];
                if (ub != nullptr) y = fmaf(p.scale_b, ub[i], y);
            }
            for (int t = 0; t < N; ++t) {
                float x = old[t];
                if (ua != nullptr) {
                    x = p.share[t] * y;
                    for (int s = 0; s < N; ++s) x = fmaf(p.mix[s * N + t], old[s], x);
                    res[(int64_t)t * W + i] = x;
                }
                if (to != nullptr) u = fmaf(p.take[t], x, u);
            }
            ss = fmaf(u, u, ss);
        }
        if (to == nullptr) return;
        const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)W + p.eps);
        for (int i = threadIdx.x; i < W; i += kThreads) {
            float u = 0.0f;
            for (int t = 0; t < N; ++t) u = fmaf(p.take[t], res[(int64_t)t * W + i], u);
            Elem<T>::store(to + i, u * inv * p.weight[i]);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(kThreads)
bigram_embedding_kernel(const int* __restrict__ tokens, const int* __restrict__ positions, const int* __restrict__ seq_of_row,
                        const int* __restrict__ row_start, const int* __restrict__ state_slots, const T* __restrict__ table,
                        const T* __restrict__ pairs, int* __restrict__ before, float* __restrict__ out, int width, int copies,
                        int vocab, int buckets, int64_t mul_prev, int64_t mul_cur) {
    __shared__ int pair_row;
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x;
    const int token = min(max(tokens[row], 0), vocab - 1);
    if (threadIdx.x == 0) {
        const int seq = seq_of_row[row], first = row_start[seq];
        int prev = 0;
        if (row == first) {
            // the step's first token of its sequence: the only reader of the request's state also renews it
            int* mine = before + state_slots[seq];
            prev = *mine;
            *mine = tokens[row_start[seq + 1] - 1];
        } else {
            prev = tokens[row - 1];
        }
        pair_row = positions[row] == 0 ? buckets : (int)(((int64_t)max(prev, 0) * mul_prev + (int64_t)token * mul_cur) % buckets);
    }
    __syncthreads();
    const T* a = table + (int64_t)token * width;
    const T* b = pairs + (int64_t)pair_row * width;
    float* to = out + (int64_t)row * copies * width;
    constexpr int N = Packet<T>::N;
    if (width % N == 0) {
        for (int i = threadIdx.x * N; i < width; i += kThreads * N) {
            float x[N], y[N];
            Packet<T>::load(a + i, x);
            Packet<T>::load(b + i, y);
#pragma unroll
            for (int e = 0; e < N; ++e) x[e] += y[e];
            for (int c = 0; c < copies; ++c)
#pragma unroll
                for (int e = 0; e < N; e += 4) Packet<float>::store(to + (int64_t)c * width + i + e, x + e);
        }
    } else {
        for (int i = threadIdx.x; i < width; i += kThreads) {
            const float x = Elem<T>::load(a + i) + Elem<T>::load(b + i);
            for (int c = 0; c < copies; ++c) to[(int64_t)c * width + i] = x;
        }
    }
}

template <typename T>
int launch(float* residual, void* out, const Streams& p, int rows, cudaStream_t stream) {
    const uintptr_t bits = (uintptr_t)residual | (uintptr_t)out | (uintptr_t)p.update_a | (uintptr_t)p.update_b | (uintptr_t)p.weight;
    const bool packets = p.width % 4 == 0 && bits % 16 == 0;
    auto kernel = mixed_streams_norm_kernel<T, 0>;
    if (packets) {
        switch (p.streams) {
            case 1: kernel = mixed_streams_norm_kernel<T, 1>; break;
            case 2: kernel = mixed_streams_norm_kernel<T, 2>; break;
            case 3: kernel = mixed_streams_norm_kernel<T, 3>; break;
            case 4: kernel = mixed_streams_norm_kernel<T, 4>; break;
            case 5: kernel = mixed_streams_norm_kernel<T, 5>; break;
            case 6: kernel = mixed_streams_norm_kernel<T, 6>; break;
            case 8: kernel = mixed_streams_norm_kernel<T, 8>; break;
            default: break;
        }
    }
    cudaError_t launched = tb_launch_pdl(kernel, dim3(rows), dim3(kThreads), (size_t)0, stream, residual, (T*)out, p);
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}

}  // namespace

// residual: float32 [rows, streams * width]; update_a (null: the copies stay), update_b (null: none): float32 [rows, width]; mix: float32
// [streams, streams] ([from, to]) and share: float32 [streams], with an update; out: [rows, width] in `dtype` or null, then with
// take: float32 [streams] and weight: float32 [width].
TB_EXPORT int tb_mixed_streams_norm(float* residual, const float* update_a, float scale_a, const float* update_b, float scale_b,
                                    const float* mix, const float* share, const float* take, const float* weight, void* out,
                                    int rows, int width, int streams, float eps, int dtype, cudaStream_t stream) {
    if (rows == 0) return 0;
    if (width < 1 || streams < 1 || streams > kMaxStreams) return TB_ERR_BAD_SIZE;
    if (update_a == nullptr ? update_b != nullptr : (mix == nullptr || share == nullptr)) return TB_ERR_BAD_SIZE;
    if (out != nullptr && (take == nullptr || weight == nullptr)) return TB_ERR_BAD_SIZE;
    if (out == nullptr && update_a == nullptr) return 0;
    Streams p;
    p.update_a = update_a; p.update_b = update_b; p.scale_a = scale_a; p.scale_b = scale_b; p.mix = mix; p.share = share;
    p.take = take; p.weight = weight; p.width = width; p.streams = streams; p.eps = eps;
    if (dtype == TB_F32) return launch<float>(residual, out, p, rows, stream);
    if (dtype == TB_BF16) return launch<__nv_bfloat16>(residual, out, p, rows, stream);
    return TB_ERR_BAD_DTYPE;
}

// tokens, positions, seq_of_row: int32 [rows]; row_start: int32 [sequences + 1]; state_slots: int32 [sequences]; table: [vocab, width] and
// pairs: [buckets + 1, width] in `dtype`; before: int32 [slots]; out: float32 [rows, copies * width].
TB_EXPORT int tb_bigram_embedding(const int* tokens, const int* positions, const int* seq_of_row, const int* row_start,
                                  const int* state_slots, const void* table, const void* pairs, int* before, float* out, int rows,
                                  int width, int copies, int vocab, int buckets, int64_t mul_prev, int64_t mul_cur, int dtype,
                                  cudaStream_t stream) {
    if (rows == 0) return 0;
    if (width < 1 || copies < 1 || vocab < 1 || buckets < 1 || mul_prev < 0 || mul_cur < 0) return TB_ERR_BAD_SIZE;
    if (((uintptr_t)table | (uintptr_t)pairs | (uintptr_t)out) % 16 != 0) return TB_ERR_BAD_ALIGN;
    cudaError_t launched;
    if (dtype == TB_F32)
        launched = tb_launch_pdl(bigram_embedding_kernel<float>, dim3(rows), dim3(kThreads), (size_t)0, stream, tokens, positions,
                                 seq_of_row, row_start, state_slots, (const float*)table, (const float*)pairs, before, out, width,
                                 copies, vocab, buckets, mul_prev, mul_cur);
    else if (dtype == TB_BF16)
        launched = tb_launch_pdl(bigram_embedding_kernel<__nv_bfloat16>, dim3(rows), dim3(kThreads), (size_t)0, stream, tokens,
                                 positions, seq_of_row, row_start, state_slots, (const __nv_bfloat16*)table,
                                 (const __nv_bfloat16*)pairs, before, out, width, copies, vocab, buckets, mul_prev, mul_cur);
    else
        return TB_ERR_BAD_DTYPE;
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}
