// A short causal convolution per channel over the rows of every sequence, as a step of its own (the convolutions that
// belong to an attention mixer's queries, keys and values live with their rotation in conv_rope_cache.cu):
//
//   tb_short_conv        v[t, c] = proj[t, c] + in_bias[c]                       (in_bias may be null)
//                        y[t, c] = out_bias[c] + sum_{j < J} taps[j, c] * v[t - (J - 1) + j, c]     (out_bias may be null)
//                        and y <- silu(y) with `act`;
//                        with v = 0 at positions in front of the sequence's start.  Values at positions in front of this
//                        step's first token come from the request's convolution state: the last J - 1 rows of v, 32-bit,
//                        [slot][J - 1][channels]; position p lies at index p - (begin - (J - 1)).
//   tb_short_conv_state  the state of every sequence of the step renewed to its last J - 1 rows of v (a launch behind the
//                        convolution that has read the old state).  In a step where every sequence brings one row
//                        (`single` != 0) tb_short_conv renews the state itself: there the only reader of a sequence's old
//                        state is the thread that owns the channel.
//
// All arithmetic is 32-bit, an output is rounded once, and a channel's sum runs over its taps in order, oldest first,
// whatever the batch or the cut.  Any number of taps; up to four in 16-byte packets of channels.
#include "common.cuh"

namespace {

// SiLU: accurate for 32-bit outputs; in front of a rounding to bfloat16 with the fast exponential and division
template <typename T>
__device__ __forceinline__ float activated(float y, int act) {
    if (!act) return y;
    return sizeof(T) == 4 ? y / (1.0f + expf(-y)) : __fdividef(y, 1.0f + __expf(-y));
}

// A thread a (row, channel): any width, any number of taps.
template <typename T, bool SINGLE>
__global__ void __launch_bounds__(128)
short_conv_kernel(const T* __restrict__ proj, int64_t proj_stride, const float* __restrict__ in_bias,
                  const float* __restrict__ taps, const float* __restrict__ out_bias, float* __restrict__ state,
                  T* __restrict__ out, int64_t out_stride, const int* __restrict__ positions,
                  const int* __restrict__ seq_of_row, const int* __restrict__ row_start, const int* __restrict__ seq_begin,
                  const int* __restrict__ state_slots, int channels, int J, int act) {
    pdl_trigger();
    pdl_wait();                                   // the projected rows and the step's metadata come from kernels in front
    const int row = blockIdx.x;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int seq = seq_of_row[row], pos = positions[row];
    const int begin = seq_begin[seq], first_row = row_start[seq];
    float* st = state + (int64_t)state_slots[seq] * (J - 1) * channels + c;
    const float add = in_bias == nullptr ? 0.0f : in_bias[c];
    float sum = 0.0f;
    for (int j = 0; j < J; ++j) {
        const int p = pos - (J - 1) + j;
        float v = 0.0f;
        if (p >= begin) v = Elem<T>::load(proj + (int64_t)(first_row + (p - begin)) * proj_stride + c) + add;
        else if (p >= 0) v = st[(int64_t)(p - (begin - (J - 1))) * channels];
        sum = fmaf(taps[(int64_t)j * channels + c], v, sum);
        if (SINGLE && j > 0) st[(int64_t)(j - 1) * channels] = v;      // (index j - 1 has been read: the walk ascends)
    }
    if (out_bias != nullptr) sum += out_bias[c];
    Elem<T>::store(out + (int64_t)row * out_stride + c, activated<T>(sum, act));
}

template <int N>
__device__ __forceinline__ void load_floats(const float* p, float* v) {
#pragma unroll
    for (int e = 0; e < N; e += 4) {
        const float4 t = *reinterpret_cast<const float4*>(p + e);
        v[e] = t.x; v[e + 1] = t.y; v[e + 2] = t.z; v[e + 3] = t.w;
    }
}
template <int N>
__device__ __forceinline__ void store_floats(float* p, const float* v) {
#pragma unroll
    for (int e = 0; e < N; e += 4) *reinterpret_cast<float4*>(p + e) = make_float4(v[e], v[e + 1], v[e + 2], v[e + 3]);
}

// A thread a packet of channels for kRowTile neighbouring rows in turn: rows of one sequence slide through the
// registers, so every projected packet is read once (and the J - 1 packets in front of a tile once more).
constexpr int kRowTile = 8;

template <typename T, bool SINGLE, int J>
__global__ void __launch_bounds__(128)
short_conv_packets_kernel(const T* __restrict__ proj, int64_t proj_stride, const float* __restrict__ in_bias,
                          const float* __restrict__ taps, const float* __restrict__ out_bias, float* __restrict__ state,
                          T* __restrict__ out, int64_t out_stride, const int* __restrict__ positions,
                          const int* __restrict__ seq_of_row, const int* __restrict__ row_start,
                          const int* __restrict__ seq_begin, const int* __restrict__ state_slots, int channels, int rows,
                          int act) {
    constexpr int N = Packet<T>::N;
    constexpr int ROWS = SINGLE ? 1 : kRowTile;
    const int packet = blockIdx.y * blockDim.x + threadIdx.x;
    pdl_trigger();
    if (packet >= channels / N) return;
    const int c0 = packet * N;
    float w[J][N], add[N], behind[N];
#pragma unroll
    for (int j = 0; j < J; ++j) load_floats<N>(taps + (int64_t)j * channels + c0, w[j]);
#pragma unroll
    for (int e = 0; e < N; ++e) add[e] = behind[e] = 0.0f;
    if (in_bias != nullptr) load_floats<N>(in_bias + c0, add);
    if (out_bias != nullptr) load_floats<N>(out_bias + c0, behind);
    pdl_wait();                                   // (weights above; the projected rows come from the kernel in front)
    // the tile's own rows and their sequences, asked for at once
    uint4 own[ROWS];
    int row_seq[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const int row = min(blockIdx.x * ROWS + r, rows - 1);
        own[r] = *reinterpret_cast<const uint4*>(proj + (int64_t)row * proj_stride + c0);
        row_seq[r] = seq_of_row[row];
    }
    float v[J][N];
    int seq_before = -1;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const int row = blockIdx.x * ROWS + r;
        if (row >= rows) return;
        const int seq = row_seq[r];
        const bool slides = r > 0 && seq == seq_before;       // the row in front is the position in front
        seq_before = seq;
        float* st = nullptr;
        if (slides) {
#pragma unroll
            for (int j = 0; j + 1 < J; ++j)
#pragma unroll
                for (int e = 0; e < N; ++e) v[j][e] = v[j + 1][e];
        } else {
            const int pos = positions[row], begin = seq_begin[seq], first_row = row_start[seq];
            st = state + (int64_t)state_slots[seq] * (J - 1) * channels + c0;
#pragma unroll
            for (int j = 0; j + 1 < J; ++j) {
                const int p = pos - (J - 1) + j;
                if (p >= begin) {
                    Packet<T>::load(proj + (int64_t)(first_row + (p - begin)) * proj_stride + c0, v[j]);
#pragma unroll
                    for (int e = 0; e < N; ++e) v[j][e] += add[e];
                } else if (p >= 0) {
                    load_floats<N>(st + (int64_t)(p - (begin - (J - 1))) * channels, v[j]);
                } else {
#pragma unroll
                    for (int e = 0; e < N; ++e) v[j][e] = 0.0f;
                }
            }
        }
        Packet<T>::unpack(own[r], v[J - 1]);
#pragma unroll
        for (int e = 0; e < N; ++e) v[J - 1][e] += add[e];
        float y[N];
#pragma unroll
        for (int e = 0; e < N; ++e) {
            float sum = 0.0f;
#pragma unroll
            for (int j = 0; j < J; ++j) sum = fmaf(w[j][e], v[j][e], sum);
            y[e] = activated<T>(sum + behind[e], act);
        }
        if (SINGLE) {
#pragma unroll
            for (int j = 1; j < J; ++j) store_floats<N>(st + (int64_t)(j - 1) * channels, v[j]);
        }
        Packet<T>::store(out + (int64_t)row * out_stride + c0, y);
    }
}

// New state: index i holds position begin + n - (J - 1) + i, a row of this step, an older row of the state (index n + i,
// which is above i: an ascending walk reads it before it is overwritten), or zero.
template <typename T>
__global__ void __launch_bounds__(128)
short_conv_state_kernel(const T* __restrict__ proj, int64_t proj_stride, const float* __restrict__ in_bias,
                        float* __restrict__ state, const int* __restrict__ row_start, const int* __restrict__ seq_begin,
                        const int* __restrict__ state_slots, int channels, int J) {
    pdl_trigger();
    pdl_wait();                                   // the convolution in front still reads the old state
    const int seq = blockIdx.x;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int first_row = row_start[seq], n = row_start[seq + 1] - first_row, begin = seq_begin[seq];
    if (n <= 0) return;
    const float add = in_bias == nullptr ? 0.0f : in_bias[c];
    float* st = state + (int64_t)state_slots[seq] * (J - 1) * channels + c;
    for (int i = 0; i < J - 1; ++i) {
        const int p = begin + n - (J - 1) + i;
        float v = 0.0f;
        if (p >= begin) v = Elem<T>::load(proj + (int64_t)(first_row + (p - begin)) * proj_stride + c) + add;
        else if (p >= 0) v = st[(int64_t)(n + i) * channels];
        st[(int64_t)i * channels] = v;
    }
}

template <typename T>
int launch(const void* proj, int64_t proj_stride, const float* in_bias, const float* taps, const float* out_bias,
           float* state, void* out, int64_t out_stride, const int* positions, const int* seq_of_row, const int* row_start,
           const int* seq_begin, const int* state_slots, int rows, int channels, int J, int single, int act, cudaStream_t stream) {
    constexpr int N = Packet<T>::N;
    const uintptr_t bits = (uintptr_t)proj | (uintptr_t)in_bias | (uintptr_t)taps | (uintptr_t)out_bias | (uintptr_t)state |
                           (uintptr_t)out;
    cudaError_t launched;
    if (channels % N == 0 && J <= 4 && proj_stride % N == 0 && out_stride % N == 0 && bits % 16 == 0) {
        const int tile = single ? 1 : kRowTile;
        const dim3 grid((rows + tile - 1) / tile, (channels / N + 127) / 128);
#define TB_CONV(S, TAPS)                                                                                              \
    launched = tb_launch_pdl(short_conv_packets_kernel<T, S, TAPS>, grid, dim3(128), 0, stream, (const T*)proj,       \
                             proj_stride, in_bias, taps, out_bias, state, (T*)out, out_stride, positions, seq_of_row, \
                             row_start, seq_begin, state_slots, channels, rows, act)
        if (single) {
            if (J == 1) TB_CONV(true, 1); else if (J == 2) TB_CONV(true, 2); else if (J == 3) TB_CONV(true, 3); else TB_CONV(true, 4);
        } else {
            if (J == 1) TB_CONV(false, 1); else if (J == 2) TB_CONV(false, 2); else if (J == 3) TB_CONV(false, 3); else TB_CONV(false, 4);
        }
#undef TB_CONV
    } else {
        const dim3 grid(rows, (channels + 127) / 128);
        auto kernel = single ? short_conv_kernel<T, true> : short_conv_kernel<T, false>;
        launched = tb_launch_pdl(kernel, grid, dim3(128), 0, stream, (const T*)proj, proj_stride, in_bias, taps, out_bias,
                                 state, (T*)out, out_stride, positions, seq_of_row, row_start, seq_begin, state_slots,
                                 channels, J, act);
    }
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}

}  // namespace

// proj: [rows, channels] with row stride proj_stride (elements); taps: 32-bit [J, channels] (tap J - 1 multiplies the row
// itself, tap 0 the oldest); in_bias, out_bias: null or 32-bit [channels]; state: 32-bit [slots, J - 1, channels] (null
// for one tap); out: [rows, channels] in the dtype of proj; act: 1 applies SiLU to the sums.
TB_EXPORT int tb_short_conv(const void* proj, int64_t proj_stride, const float* in_bias, const float* taps,
                            const float* out_bias, float* state, void* out, int64_t out_stride, const int* positions,
                            const int* seq_of_row, const int* row_start, const int* seq_begin, const int* state_slots,
                            int rows, int channels, int taps_count, int single, int act, int dtype, cudaStream_t stream) {
    if (rows == 0) return 0;
    if (channels < 1 || taps_count < 1 || (channels + 127) / 128 > 65535) return TB_ERR_BAD_SIZE;
    if (taps_count > 1 && state == nullptr) return TB_ERR_BAD_SIZE;
    if (dtype == TB_F32)
        return launch<float>(proj, proj_stride, in_bias, taps, out_bias, state, out, out_stride, positions, seq_of_row,
                             row_start, seq_begin, state_slots, rows, channels, taps_count, single, act, stream);
    if (dtype == TB_BF16)
        return launch<__nv_bfloat16>(proj, proj_stride, in_bias, taps, out_bias, state, out, out_stride, positions,
                                     seq_of_row, row_start, seq_begin, state_slots, rows, channels, taps_count, single,
                                     act, stream);
    return TB_ERR_BAD_DTYPE;
}

TB_EXPORT int tb_short_conv_state(const void* proj, int64_t proj_stride, const float* in_bias, float* state,
                                  const int* row_start, const int* seq_begin, const int* state_slots, int num_seqs,
                                  int channels, int taps_count, int dtype, cudaStream_t stream) {
    if (num_seqs == 0 || taps_count <= 1) return 0;
    if (channels < 1 || (channels + 127) / 128 > 65535) return TB_ERR_BAD_SIZE;
    const dim3 grid(num_seqs, (channels + 127) / 128);
    cudaError_t launched;
    if (dtype == TB_F32)
        launched = tb_launch_pdl(short_conv_state_kernel<float>, grid, dim3(128), 0, stream, (const float*)proj, proj_stride,
                                 in_bias, state, row_start, seq_begin, state_slots, channels, taps_count);
    else if (dtype == TB_BF16)
        launched = tb_launch_pdl(short_conv_state_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream,
                                 (const __nv_bfloat16*)proj, proj_stride, in_bias, state, row_start, seq_begin, state_slots,
                                 channels, taps_count);
    else
        return TB_ERR_BAD_DTYPE;
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}
