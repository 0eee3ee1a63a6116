// Rotation in the rotate-half layout, division of every query and key head by its root mean square, and the write
// of keys and values into the request's cache pages: what stands between an attention mixer's input projection
// and its attention kernel, in one pass over the projected rows.
//
// A projected row holds, side by side, H query heads of d numbers, G key heads of d numbers and G value heads of
// dv numbers; with `bias` (32-bit, as wide as that row) the projections' biases are added first, in 32-bit.  For queries and keys, of every head's first `rot_dims` numbers, number i and number i + rot_dims / 2
// turn together by the angle position * inv_freq[i] (32-bit angle, sincosf), cosine and sine both multiplied by
// `amplitude`; the rest of the head passes.  Then, with `unit_norm`, the head is divided by
// sqrt(mean(head^2) + eps), the mean over all d numbers of the rotated head.  Queries go to q_out, keys and values
// into the pages: a page is [G][page_size][d] keys followed by [G][page_size][dv] values.
//
// Values may also be mixed with those of an earlier layer: `value_mode` 1 leaves this layer's values (bias added, 32-bit,
// [rows, G * dv]) in `first_values` for later layers, 2 stores (1 - mix) * v + mix * first_values instead of v, `mix` one
// number on the device.
//
// One warp per (row, head of q, k or v); rows that neither turn nor are normed take a kernel of their own, a thread a
// 16-byte packet of the row.  All arithmetic is 32-bit; each stored value is rounded once; the order
// of a head's sum of squares depends on d alone.
//
// tb_row_norm_rope_cache, for a mixer that norms its queries and its keys over the whole projection (all heads at once, a weight
// per number) in front of the rotation, does the same job with a block a row: the sums of squares of the row's q and of its k, the
// normed numbers turned with the row's sines and cosines (taken once a row), stored; the values are the row's own value columns
// or, with `values_from_keys`, the keys as projected (dv = d, no value columns).
//
// tb_pool_blocks, for a mixer that also attends to averaged blocks of old tokens, runs behind it: every row that ends a
// block of `pool` positions leaves the block's averaged key and value in pages of their own.
#include "common.cuh"

namespace {

constexpr int kWarps = 4;

struct HeadGeometry {
    int heads, kv_heads, dim, vdim;      // H, G, d, dv
    int rot_dims;                        // even, <= dim; 0: no rotation
    int page_size;
    int unit_norm;
    float amplitude, eps;
};

enum ValueMode : int { VALUES_PLAIN = 0, VALUES_LEAVE = 1, VALUES_MIX = 2 };
struct ValueMix {
    int mode;
    float* first;                        // [rows, G * dv]
    const float* mix;                    // one number
};

template <typename T>
__global__ void __launch_bounds__(kWarps * 32)
rope_norm_cache_kernel(const T* __restrict__ proj, int64_t proj_stride, T* __restrict__ q_out, int64_t q_stride,
                       T* __restrict__ cache, const int* __restrict__ positions, const int* __restrict__ seq_of_row,
                       const int* __restrict__ block_table, int bt_stride, const float* __restrict__ inv_freq,
                       const float* __restrict__ bias, HeadGeometry g, int write_kv, ValueMix values) {
    extern __shared__ float head_cache[];             // kWarps * dim
    pdl_trigger();
    pdl_wait();                                       // the projected rows and the step's metadata come from kernels in front
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row = blockIdx.x;
    const int slot = blockIdx.y * kWarps + warp;      // which head of the row: queries, then keys, then values
    const int slots = g.heads + 2 * g.kv_heads;
    if (slot >= slots) return;                        // the whole warp leaves; no block-wide barrier below
    const int pos = positions[row];
    const T* prow = proj + (int64_t)row * proj_stride;

    T* dst;
    if (slot >= g.heads) {
        if (!write_kv) return;
        const int seq = seq_of_row[row];
        const int page = block_table[(int64_t)seq * bt_stride + pos / g.page_size];
        const int in_page = pos % g.page_size;
        const int64_t page_elems = (int64_t)g.kv_heads * g.page_size * (g.dim + g.vdim);
        dst = cache + (int64_t)page * page_elems;
        if (slot < g.heads + g.kv_heads) {
            dst += ((int64_t)(slot - g.heads) * g.page_size + in_page) * g.dim;
        } else {
            // a value head: copied as it is
            const int head = slot - g.heads - g.kv_heads;
            dst += (int64_t)g.kv_heads * g.page_size * g.dim + ((int64_t)head * g.page_size + in_page) * g.vdim;
            const int64_t at = (int64_t)(g.heads + g.kv_heads) * g.dim + (int64_t)head * g.vdim;
            const T* src = prow + at;
            if (values.mode != VALUES_PLAIN) {
                float* first = values.first + (int64_t)row * g.kv_heads * g.vdim + (int64_t)head * g.vdim;
                const float mix = values.mode == VALUES_MIX ? *values.mix : 0.0f;
                for (int i = lane; i < g.vdim; i += 32) {
                    float v = Elem<T>::load(src + i) + (bias != nullptr ? bias[at + i] : 0.0f);
                    if (values.mode == VALUES_LEAVE) first[i] = v;
                    else v = fmaf(mix, first[i], (1.0f - mix) * v);
                    Elem<T>::store(dst + i, v);
                }
            } else if (bias == nullptr) {
                for (int i = lane; i < g.vdim; i += 32) dst[i] = src[i];
            } else {
                for (int i = lane; i < g.vdim; i += 32) Elem<T>::store(dst + i, Elem<T>::load(src + i) + bias[at + i]);
            }
            return;
        }
    } else {
        dst = q_out + (int64_t)row * q_stride + (int64_t)slot * g.dim;
    }
    const T* src = prow + (int64_t)slot * g.dim;      // query heads and key heads lie side by side in the row
    const float* add = bias == nullptr ? nullptr : bias + (int64_t)slot * g.dim;
    float* mine = head_cache + warp * g.dim;
    const int half = g.rot_dims >> 1;
    float ss = 0.0f;
    for (int i = lane; i < half; i += 32) {
        float sn, cs;
        sincosf((float)pos * inv_freq[i], &sn, &cs);
        sn *= g.amplitude;
        cs *= g.amplitude;
        float u = Elem<T>::load(src + i), v = Elem<T>::load(src + i + half);
        if (add != nullptr) {
            u += add[i];
            v += add[i + half];
        }
        const float r0 = u * cs - v * sn;
        const float r1 = v * cs + u * sn;
        mine[i] = r0;
        mine[i + half] = r1;
        ss = fmaf(r0, r0, ss);
        ss = fmaf(r1, r1, ss);
    }
    for (int i = g.rot_dims + lane; i < g.dim; i += 32) {
        const float v = Elem<T>::load(src + i) + (add != nullptr ? add[i] : 0.0f);
        mine[i] = v;
        ss = fmaf(v, v, ss);
    }
    float inv = 1.0f;
    if (g.unit_norm) inv = 1.0f / sqrtf(warp_sum(ss) / (float)g.dim + g.eps);
    __syncwarp();
    for (int i = lane; i < g.dim; i += 32) Elem<T>::store(dst + i, mine[i] * inv);
}


// Rows that neither turn nor are normed: a thread a 16-byte packet of a row's q, k and v (head sizes that are multiples of a
// packet, aligned rows).
template <typename T>
__global__ void __launch_bounds__(128)
bias_cache_packets_kernel(const T* __restrict__ proj, int64_t proj_stride, T* __restrict__ q_out, int64_t q_stride,
                          T* __restrict__ cache, const int* __restrict__ positions, const int* __restrict__ seq_of_row,
                          const int* __restrict__ block_table, int bt_stride, const float* __restrict__ bias, HeadGeometry g,
                          int write_kv, ValueMix values) {
    constexpr int N = Packet<T>::N;
    const int row = blockIdx.x;
    const int c0 = (blockIdx.y * blockDim.x + threadIdx.x) * N;
    const int q_width = g.heads * g.dim, k_end = q_width + g.kv_heads * g.dim, end = k_end + g.kv_heads * g.vdim;
    pdl_trigger();
    pdl_wait();
    if (c0 >= end) return;
    float v[N];
    Packet<T>::load(proj + (int64_t)row * proj_stride + c0, v);
    if (bias != nullptr) {
#pragma unroll
        for (int e = 0; e < N; e += 4) {
            const float4 b = *reinterpret_cast<const float4*>(bias + c0 + e);
            v[e] += b.x; v[e + 1] += b.y; v[e + 2] += b.z; v[e + 3] += b.w;
        }
    }
    if (c0 < q_width) {
        Packet<T>::store(q_out + (int64_t)row * q_stride + c0, v);
        return;
    }
    const bool is_value = c0 >= k_end;
    if (is_value && values.mode != VALUES_PLAIN) {
        float* first = values.first + (int64_t)row * g.kv_heads * g.vdim + (c0 - k_end);
        if (values.mode == VALUES_LEAVE) {
#pragma unroll
            for (int e = 0; e < N; e += 4) *reinterpret_cast<float4*>(first + e) = make_float4(v[e], v[e + 1], v[e + 2], v[e + 3]);
        } else {
            const float mix = *values.mix;
#pragma unroll
            for (int e = 0; e < N; e += 4) {
                const float4 f = *reinterpret_cast<const float4*>(first + e);
                v[e] = fmaf(mix, f.x, (1.0f - mix) * v[e]);
                v[e + 1] = fmaf(mix, f.y, (1.0f - mix) * v[e + 1]);
                v[e + 2] = fmaf(mix, f.z, (1.0f - mix) * v[e + 2]);
                v[e + 3] = fmaf(mix, f.w, (1.0f - mix) * v[e + 3]);
            }
        }
    }
    if (!write_kv) return;
    const int pos = positions[row];
    const int page = block_table[(int64_t)seq_of_row[row] * bt_stride + pos / g.page_size], in_page = pos % g.page_size;
    T* dst = cache + (int64_t)page * g.kv_heads * g.page_size * (g.dim + g.vdim);
    if (is_value) {
        const int head = (c0 - k_end) / g.vdim, e0 = (c0 - k_end) % g.vdim;
        dst += (int64_t)g.kv_heads * g.page_size * g.dim + ((int64_t)head * g.page_size + in_page) * g.vdim + e0;
    } else {
        const int head = (c0 - q_width) / g.dim, e0 = (c0 - q_width) % g.dim;
        dst += ((int64_t)head * g.page_size + in_page) * g.dim + e0;
    }
    Packet<T>::store(dst, v);
}

template <typename T>
int launch_rope_norm(const void* proj, int64_t proj_stride, void* q_out, int64_t q_stride, void* cache, const int* positions,
                     const int* seq_of_row, const int* block_table, int bt_stride, const float* inv_freq, const float* bias,
                     int rows, const HeadGeometry& g, int write_kv, const ValueMix& values, cudaStream_t stream) {
    constexpr int N = Packet<T>::N;
    const uintptr_t bits = (uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)cache | (uintptr_t)bias | (uintptr_t)values.first;
    cudaError_t launched;
    if (g.rot_dims == 0 && !g.unit_norm && g.dim % N == 0 && g.vdim % N == 0 && proj_stride % N == 0 && q_stride % N == 0 &&
        bits % 16 == 0) {
        const int packets = (g.heads * g.dim + g.kv_heads * (g.dim + g.vdim)) / N;
        const dim3 grid(rows, (packets + 127) / 128);
        if (grid.y > 65535) return TB_ERR_BAD_SIZE;
        launched = tb_launch_pdl(bias_cache_packets_kernel<T>, grid, dim3(128), 0, stream, (const T*)proj, proj_stride,
                                 (T*)q_out, q_stride, (T*)cache, positions, seq_of_row, block_table, bt_stride, bias, g,
                                 write_kv, values);
    } else {
        const size_t smem = (size_t)kWarps * g.dim * sizeof(float);
        if (smem > 40 * 1024) return TB_ERR_BAD_SIZE;
        const int slots = g.heads + 2 * g.kv_heads;
        const dim3 grid(rows, (slots + kWarps - 1) / kWarps);
        if (grid.y > 65535) return TB_ERR_BAD_SIZE;
        launched = tb_launch_pdl(rope_norm_cache_kernel<T>, grid, dim3(kWarps * 32), smem, stream, (const T*)proj, proj_stride,
                                 (T*)q_out, q_stride, (T*)cache, positions, seq_of_row, block_table, bt_stride, inv_freq,
                                 bias, g, write_kv, values);
    }
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}

// q and k of a row over their own root mean squares (all heads at once) times a weight, then the rotation; a block a row, the
// row's q and k widened in shared memory.  VEC: stores of a 16-byte packet (head sizes and half rotations that are multiples of a
// packet, or no rotation).
constexpr int kRowThreads = 256;

template <typename T, bool VEC>
__global__ void __launch_bounds__(kRowThreads)
row_norm_rope_cache_kernel(const T* __restrict__ proj, int64_t proj_stride, T* __restrict__ q_out, int64_t q_stride,
                           T* __restrict__ cache, const int* __restrict__ positions, const int* __restrict__ seq_of_row,
                           const int* __restrict__ block_table, int bt_stride, const float* __restrict__ inv_freq,
                           const float* __restrict__ weight, HeadGeometry g, int values_from_keys) {
    extern __shared__ __align__(16) float row_smem[];  // [q_width + k_width] numbers, then [half] cosines, [half] sines
    __shared__ float scratch[32];
    constexpr int N = VEC ? Packet<T>::N : 1;
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x, pos = positions[row];
    const int q_width = g.heads * g.dim, both = q_width + g.kv_heads * g.dim, half = g.rot_dims >> 1;
    float *cosines = row_smem + both, *sines = cosines + half;
    const T* prow = proj + (int64_t)row * proj_stride;
    // everything that comes from memory is asked for before the sines and cosines are taken: the thread's first numbers and
    // their weights, and the row's page
    auto load = [&](int i, float* v, float* w) {
        if constexpr (VEC) {
            Packet<T>::load(prow + i, v);
#pragma unroll
            for (int e = 0; e < N; e += 4) {
                const float4 f = *reinterpret_cast<const float4*>(weight + i + e);
                w[e] = f.x; w[e + 1] = f.y; w[e + 2] = f.z; w[e + 3] = f.w;
            }
        } else {
            v[0] = Elem<T>::load(prow + i);
            w[0] = weight[i];
        }
    };
    float qq = 0.0f, kk = 0.0f;
    auto take = [&](int i, const float* v, const float* w) {
        float sum = 0.0f;
#pragma unroll
        for (int e = 0; e < N; ++e) {
            row_smem[i + e] = v[e] * w[e];             // (the root mean square divides later)
            sum = fmaf(v[e], v[e], sum);
        }
        if (i < q_width) qq += sum; else kk += sum;    // (a packet does not straddle: widths are multiples of a head)
    };
    const int i0 = threadIdx.x * N;
    float v0[N], w0[N];
    if (i0 < both) load(i0, v0, w0);
    const int page = block_table[(int64_t)seq_of_row[row] * bt_stride + pos / g.page_size], in_page = pos % g.page_size;
    for (int i = threadIdx.x; i < half; i += kRowThreads) {
        float sn, cs;
        sincosf((float)pos * inv_freq[i], &sn, &cs);
        cosines[i] = cs * g.amplitude;
        sines[i] = sn * g.amplitude;
    }
    if (i0 < both) take(i0, v0, w0);
    for (int i = i0 + kRowThreads * N; i < both; i += kRowThreads * N) {
        load(i, v0, w0);
        take(i, v0, w0);
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    if ((threadIdx.x & 31) == 0) {
        scratch[threadIdx.x >> 5] = qq;
        scratch[kRowThreads / 32 + (threadIdx.x >> 5)] = kk;
    }
    __syncthreads();                                   // (the row, its sines and cosines and the warps' sums are there)
    qq = kk = 0.0f;
#pragma unroll
    for (int w = 0; w < kRowThreads / 32; ++w) {
        qq += scratch[w];
        kk += scratch[kRowThreads / 32 + w];
    }
    const float inv_q = 1.0f / sqrtf(qq / (float)q_width + g.eps);
    const float inv_k = 1.0f / sqrtf(kk / (float)(both - q_width) + g.eps);
    T* keys = cache + (int64_t)page * g.kv_heads * g.page_size * (g.dim + g.vdim);
    T* values = keys + (int64_t)g.kv_heads * g.page_size * g.dim;
    for (int i = threadIdx.x * N; i < both; i += kRowThreads * N) {
        const bool is_key = i >= q_width;
        const int head = (is_key ? i - q_width : i) / g.dim, at = (is_key ? i - q_width : i) % g.dim;
        const float inv = is_key ? inv_k : inv_q;
        float v[N];
#pragma unroll
        for (int e = 0; e < N; ++e) v[e] = row_smem[i + e] * inv;
        if (at < g.rot_dims) {                         // (with VEC a packet lies wholly in one half)
            const bool second = at >= half;
            const int other = second ? i - half : i + half, angle = second ? at - half : at;
#pragma unroll
            for (int e = 0; e < N; ++e) {
                const float w = row_smem[other + e] * inv;
                v[e] = second ? v[e] * cosines[angle + e] + w * sines[angle + e] : v[e] * cosines[angle + e] - w * sines[angle + e];
            }
        }
        T* dst = is_key ? keys + ((int64_t)head * g.page_size + in_page) * g.dim + at : q_out + (int64_t)row * q_stride + i;
        if constexpr (VEC) Packet<T>::store(dst, v);
        else Elem<T>::store(dst, v[0]);
    }
    const int v_width = g.kv_heads * g.vdim;
    const T* src = values_from_keys ? prow + q_width : prow + both;
    for (int i = threadIdx.x * N; i < v_width; i += kRowThreads * N) {
        T* dst = values + ((int64_t)(i / g.vdim) * g.page_size + in_page) * g.vdim + i % g.vdim;
        if constexpr (VEC) *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src + i);
        else *dst = src[i];
    }
}

template <typename T>
int launch_row_norm(const void* proj, int64_t proj_stride, void* q_out, int64_t q_stride, void* cache, const int* positions,
                    const int* seq_of_row, const int* block_table, int bt_stride, const float* inv_freq, const float* weight,
                    int rows, const HeadGeometry& g, int values_from_keys, cudaStream_t stream) {
    constexpr int N = Packet<T>::N;
    const uintptr_t bits = (uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)cache | (uintptr_t)weight;
    const bool vec = g.dim % N == 0 && g.vdim % N == 0 && (g.rot_dims / 2) % N == 0 && proj_stride % N == 0 && q_stride % N == 0 &&
                     bits % 16 == 0;
    const size_t smem = sizeof(float) * ((size_t)(g.heads + g.kv_heads) * g.dim + g.rot_dims);
    if (smem > 200 * 1024) return TB_ERR_BAD_SIZE;
    auto kernel = vec ? row_norm_rope_cache_kernel<T, true> : row_norm_rope_cache_kernel<T, false>;
    if (smem > 40 * 1024) {
        cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (err != cudaSuccess) return (int)err;
    }
    cudaError_t launched = tb_launch_pdl(kernel, dim3(rows), dim3(kRowThreads), smem, stream, (const T*)proj, proj_stride,
                                         (T*)q_out, q_stride, (T*)cache, positions, seq_of_row, block_table, bt_stride, inv_freq,
                                         weight, g, values_from_keys);
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}

// For every row of the step that ends a block of `pool` positions ((position + 1) % pool == 0): the averages of the block's
// keys and of its values, as the pages hold them, into entry position / pool of the request's pooled pages (same page
// layout).  A block of threads per (row, kv head), a thread a column, the block's tokens added in order in 32-bit.
template <typename T>
__global__ void __launch_bounds__(128)
pool_blocks_kernel(const T* __restrict__ cache, T* __restrict__ pool_cache, const int* __restrict__ positions,
                   const int* __restrict__ seq_of_row, const int* __restrict__ block_table, int bt_stride,
                   const int* __restrict__ pool_table, int pool_bt_stride, int kv_heads, int dim, int vdim, int page_size,
                   int pool) {
    pdl_trigger();
    pdl_wait();                                       // the pages were written by the kernel in front
    const int row = blockIdx.x, g = blockIdx.y;
    const int pos = positions[row];
    if ((pos + 1) % pool != 0) return;
    const int seq = seq_of_row[row];
    const int entry = pos / pool, first = pos - pool + 1;
    const int64_t page_elems = (int64_t)kv_heads * page_size * (dim + vdim);
    const int* table = block_table + (int64_t)seq * bt_stride;
    const int64_t to_page = (int64_t)pool_table[(int64_t)seq * pool_bt_stride + entry / page_size] * page_elems;
    const int to_in_page = entry % page_size;
    for (int col = threadIdx.x; col < dim + vdim; col += blockDim.x) {
        const bool is_key = col < dim;
        const int width = is_key ? dim : vdim, c = is_key ? col : col - dim;
        const int64_t part = is_key ? 0 : (int64_t)kv_heads * page_size * dim;
        float sum = 0.0f;
        for (int j0 = 0; j0 < pool; j0 += 8) {         // eight loads in flight, then their sum in position order
            float v[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int key = first + min(j0 + u, pool - 1);
                const int64_t page = (int64_t)table[key / page_size] * page_elems;
                v[u] = Elem<T>::load(cache + page + part + ((int64_t)g * page_size + key % page_size) * width + c);
            }
#pragma unroll
            for (int u = 0; u < 8; ++u)
                if (j0 + u < pool) sum += v[u];
        }
        Elem<T>::store(pool_cache + to_page + part + ((int64_t)g * page_size + to_in_page) * width + c, sum / (float)pool);
    }
}

}  // namespace

// proj: [rows, >= (H + G) * d + G * dv] with row stride proj_stride (elements); q_out: [rows, H * d] with row
// stride q_stride; cache: this layer's pages; inv_freq: 32-bit [rot_dims / 2] (may be null when rot_dims is 0); bias:
// null or 32-bit [(H + G) * d + G * dv].  value_mode: 0 values as they are, 1 also left in first_values (32-bit [rows, G * dv]),
// 2 mixed with first_values by *value_mix.
TB_EXPORT int tb_rope_norm_cache(const void* proj, int64_t proj_stride, void* q_out, int64_t q_stride, void* cache,
                                 const int* positions, const int* seq_of_row, const int* block_table, int bt_stride,
                                 const float* inv_freq, const float* bias, float amplitude, int rows, int heads, int kv_heads, int dim,
                                 int vdim, int rot_dims, int unit_norm, float eps, int page_size, int write_kv,
                                 int value_mode, float* first_values, const float* value_mix, int dtype,
                                 cudaStream_t stream) {
    if (rows == 0) return 0;
    if (value_mode < VALUES_PLAIN || value_mode > VALUES_MIX || (value_mode != VALUES_PLAIN && first_values == nullptr) ||
        (value_mode == VALUES_MIX && value_mix == nullptr))
        return TB_ERR_BAD_SIZE;
    if (heads < 1 || kv_heads < 1 || dim < 1 || vdim < 1 || page_size < 1) return TB_ERR_BAD_SIZE;
    if (rot_dims < 0 || rot_dims > dim || rot_dims % 2 != 0) return TB_ERR_BAD_SIZE;
    if (rot_dims > 0 && inv_freq == nullptr) return TB_ERR_BAD_SIZE;
    HeadGeometry g;
    g.heads = heads; g.kv_heads = kv_heads; g.dim = dim; g.vdim = vdim; g.rot_dims = rot_dims; g.page_size = page_size;
    g.unit_norm = unit_norm; g.amplitude = amplitude; g.eps = eps;
    ValueMix values;
    values.mode = value_mode; values.first = first_values; values.mix = value_mix;
    if (dtype == TB_F32)
        return launch_rope_norm<float>(proj, proj_stride, q_out, q_stride, cache, positions, seq_of_row, block_table,
                                       bt_stride, inv_freq, bias, rows, g, write_kv, values, stream);
    if (dtype == TB_BF16)
        return launch_rope_norm<__nv_bfloat16>(proj, proj_stride, q_out, q_stride, cache, positions, seq_of_row, block_table,
                                               bt_stride, inv_freq, bias, rows, g, write_kv, values, stream);
    return TB_ERR_BAD_DTYPE;
}

// proj: [rows, >= (H + G) * d (+ G * dv)] with row stride proj_stride; weight: 32-bit [(H + G) * d], the norm's weights of q then of k;
// values_from_keys: dv = d and the values are the keys as projected.  The rest as for tb_rope_norm_cache.
TB_EXPORT int tb_row_norm_rope_cache(const void* proj, int64_t proj_stride, void* q_out, int64_t q_stride, void* cache,
                                     const int* positions, const int* seq_of_row, const int* block_table, int bt_stride,
                                     const float* inv_freq, const float* weight, float amplitude, int rows, int heads, int kv_heads,
                                     int dim, int vdim, int rot_dims, float eps, int page_size, int values_from_keys, int dtype,
                                     cudaStream_t stream) {
    if (rows == 0) return 0;
    if (heads < 1 || kv_heads < 1 || dim < 1 || vdim < 1 || page_size < 1 || weight == nullptr) return TB_ERR_BAD_SIZE;
    if (rot_dims < 0 || rot_dims > dim || rot_dims % 2 != 0 || (rot_dims > 0 && inv_freq == nullptr)) return TB_ERR_BAD_SIZE;
    if (values_from_keys && dim != vdim) return TB_ERR_BAD_SIZE;
    HeadGeometry g;
    g.heads = heads; g.kv_heads = kv_heads; g.dim = dim; g.vdim = vdim; g.rot_dims = rot_dims; g.page_size = page_size;
    g.unit_norm = 0; g.amplitude = amplitude; g.eps = eps;
    if (dtype == TB_F32)
        return launch_row_norm<float>(proj, proj_stride, q_out, q_stride, cache, positions, seq_of_row, block_table, bt_stride,
                                      inv_freq, weight, rows, g, values_from_keys, stream);
    if (dtype == TB_BF16)
        return launch_row_norm<__nv_bfloat16>(proj, proj_stride, q_out, q_stride, cache, positions, seq_of_row, block_table,
                                              bt_stride, inv_freq, weight, rows, g, values_from_keys, stream);
    return TB_ERR_BAD_DTYPE;
}

// cache: the layer's pages of keys and values ([G][page_size][d] keys then [G][page_size][dv] values a page), already
// holding the step's rows; pool_cache: its pages of averaged blocks, same layout, entry b of a request's pooled pages
// being block b; pool_table: the requests' tables of those pages.
TB_EXPORT int tb_pool_blocks(const void* cache, void* pool_cache, const int* positions, const int* seq_of_row,
                             const int* block_table, int bt_stride, const int* pool_table, int pool_bt_stride, int rows,
                             int kv_heads, int dim, int vdim, int page_size, int pool, int dtype, cudaStream_t stream) {
    if (rows == 0) return 0;
    if (kv_heads < 1 || kv_heads > 65535 || dim < 1 || vdim < 1 || page_size < 1 || pool < 1) return TB_ERR_BAD_SIZE;
    const dim3 grid(rows, kv_heads);
    cudaError_t launched;
    if (dtype == TB_F32)
        launched = tb_launch_pdl(pool_blocks_kernel<float>, grid, dim3(128), (size_t)0, stream, (const float*)cache,
                                 (float*)pool_cache, positions, seq_of_row, block_table, bt_stride, pool_table,
                                 pool_bt_stride, kv_heads, dim, vdim, page_size, pool);
    else if (dtype == TB_BF16)
        launched = tb_launch_pdl(pool_blocks_kernel<__nv_bfloat16>, grid, dim3(128), (size_t)0, stream,
                                 (const __nv_bfloat16*)cache, (__nv_bfloat16*)pool_cache, positions, seq_of_row,
                                 block_table, bt_stride, pool_table, pool_bt_stride, kv_heads, dim, vdim, page_size, pool);
    else
        return TB_ERR_BAD_DTYPE;
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}
