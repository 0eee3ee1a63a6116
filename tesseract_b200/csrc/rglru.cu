// A real-gated linear recurrent unit: per channel c of block b (the channels are cut into `blocks` equal runs)
//
//   r_t = sigmoid(Ra_b u_t,b + ba)      i_t = sigmoid(Ri_b u_t,b + bi)           (square matrices over the block's channels)
//   log a_t = rate_c * r_t              (rate = -8 softplus(lam), one number a channel, made when the model is built)
//   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) * i_t * u_t                              S lives in 32-bit in the request's state slot
//   out_t = S_t * gelu_tanh(y_t + by)                                            (the block's second branch)
//
//   tb_rglru_gates   the two matrices of every block as one product (their rows alternate: 2c the row of Ra, 2c + 1 the
//                    row of Ri, so that a thread's neighbouring accumulators are r and i of one channel) and everything up
//                    to the pair (a_t, x_t = sqrt(1 - a_t^2) i_t u_t) behind it.  The pairs go to memory for tb_rglru_scan,
//                    or, in a step where every sequence brings one row (`single` != 0), the recurrence's one step and the
//                    output are taken on the spot.
//   tb_rglru_scan    the recurrence over the pairs, the gate of the second branch, the new state.  A block owns 16
//                    neighbouring channels of one sequence and cuts its rows into runs: S is affine in its start, so a
//                    run is first reduced to (A, B) with S_end = A S_start + B, the runs are chained from the slot's state,
//                    and every run is walked again from its own start.
//
// 1 - a^2 is taken as -(e^(2 log a) - 1) by that function's series where a is close to 1, as it is where the unit remembers.
// a itself takes the accurate exponential: its error is multiplied once a token for as long as a channel remembers; the
// sigmoids' and the output's divisions are single hardware approximations (an ulp or two).  Everything behind the two products'
// 32-bit sums is 32-bit; products of bfloat16 operands are exact in those sums.
#include "common.cuh"

namespace {

__device__ __forceinline__ float sigmoid_f32(float x) { return __fdividef(1.0f, 1.0f + expf(-x)); }
// 0.5 z (1 + tanh(k (z + 0.044715 z^3))) = z sigmoid(2 k (z + 0.044715 z^3)), k = sqrt(2 / pi)
__device__ __forceinline__ float gelu_tanh_f32(float z) {
    return z * sigmoid_f32(1.5957691216057308f * (z + 0.044715f * z * z * z));
}
// sqrt(1 - a^2) from log a <= 0 and a = e^(log a)
__device__ __forceinline__ float entering(float log_a, float a) {
    const float z = 2.0f * log_a;
    // 1 - e^z = -z (1 + z/2 (1 + z/3 (1 + ...))): eight terms, good to 1e-8 for |z| <= 1/2
    float series = fmaf(z, 1.0f / 8.0f, 1.0f);
    series = fmaf(z * (1.0f / 7.0f), series, 1.0f);
    series = fmaf(z * (1.0f / 6.0f), series, 1.0f);
    series = fmaf(z * (1.0f / 5.0f), series, 1.0f);
    series = fmaf(z * (1.0f / 4.0f), series, 1.0f);
    series = fmaf(z * (1.0f / 3.0f), series, 1.0f);
    series = fmaf(z * 0.5f, series, 1.0f);
    return sqrtf(z > -0.5f ? -z * series : fmaf(-a, a, 1.0f));
}

// What stands behind the gates' product, per (row, channel).  A thread first asks for all it reads of a row's channels
// (load), then finishes one after the other: what it stores never hides what it has yet to read.
template <typename T>
struct Behind {
    const T* u;                   // [rows, width]
    int64_t u_stride;
    const float *bias_r, *bias_i, *rate;      // [width]
    float2* pairs;                // [rows, width], or null: take the recurrence's step here
    float* state;                 // [slots, width]
    const int* slots;             // [sequences] (sequence of row t is t)
    const T* y;                   // [rows, width] of the second branch
    int64_t y_stride;
    const float* y_bias;
    T* out;
    int64_t out_stride;
    int width;

    struct Taken {
        float u, br, bi, rate, state, y;
    };
    __device__ __forceinline__ int64_t state_row(int row) const { return pairs == nullptr ? (int64_t)slots[row] * width : 0; }
    __device__ __forceinline__ Taken load(int row, int64_t at_state, int c) const {
        Taken t;
        t.u = Elem<T>::load(u + (int64_t)row * u_stride + c);
        t.br = bias_r[c];
        t.bi = bias_i[c];
        t.rate = rate[c];
        t.state = t.y = 0.0f;
        if (pairs == nullptr) {
            t.state = state[at_state + c];
            t.y = Elem<T>::load(y + (int64_t)row * y_stride + c) + y_bias[c];
        }
        return t;
    }
    __device__ __forceinline__ void finish(int row, int64_t at_state, int c, float acc_r, float acc_i, const Taken& t) const {
        const float r = sigmoid_f32(acc_r + t.br), i = sigmoid_f32(acc_i + t.bi);
        const float log_a = t.rate * r;
        const float a = expf(log_a);
        const float x = entering(log_a, a) * i * t.u;
        if (pairs != nullptr) {
            pairs[(int64_t)row * width + c] = make_float2(a, x);
            return;
        }
        const float s = fmaf(a, t.state, x);
        state[at_state + c] = s;
        Elem<T>::store(out + (int64_t)row * out_stride + c, s * gelu_tanh_f32(t.y));
    }
};

// Plain multiply-adds, operands widened to 32-bit (the true 32-bit product, and block sizes the tensor-core kernel does not
// take): 64 rows by 64 output rows of one block; every sum is one chain k = 0, 1, ..., S - 1.
constexpr int BM = 64, BN = 64, BK = 16;

template <typename T>
__global__ void __launch_bounds__(256)
rglru_gates_kernel(const T* __restrict__ W, Behind<T> behind, int rows, int S) {
    __shared__ float As[BK][BM + 4];
    __shared__ float Ws[BK][BN + 4];
    pdl_trigger();
    pdl_wait();
    const int tid = threadIdx.x, N = 2 * S, b = blockIdx.z;
    const T* Wb = W + (int64_t)b * N * S;
    const int n0 = blockIdx.x * BN, r0 = blockIdx.y * BM;
    const int tx = tid % 16, ty = tid / 16, load_row = tid / 4, load_k = (tid % 4) * 4;
    const T* a_src = r0 + load_row < rows ? behind.u + (int64_t)(r0 + load_row) * behind.u_stride + (int64_t)b * S : nullptr;
    const int wn = n0 + load_row;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;
    for (int k0 = 0; k0 < S; k0 += BK) {
        float a[4] = {0.f, 0.f, 0.f, 0.f}, w[4] = {0.f, 0.f, 0.f, 0.f};
        const int kk = k0 + load_k;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            if (a_src != nullptr && kk + e < S) a[e] = Elem<T>::load(a_src + kk + e);
            if (wn < N && kk + e < S) w[e] = Elem<T>::load(Wb + (int64_t)wn * S + kk + e);
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            As[load_k + e][load_row] = a[e];
            Ws[load_k + e][load_row] = w[e];
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < BK; ++k) {
            float ar[4], wr[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) ar[i] = As[k][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) wr[j] = Ws[k][tx * 4 + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(ar[i], wr[j], acc[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int row = r0 + ty * 4 + i;
        if (row >= rows) continue;
        const int64_t at_state = behind.state_row(row);
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
            const int n = n0 + tx * 4 + j, c = b * S + n / 2;    // n even: r of channel n / 2, and i beside it
            if (n < N) behind.finish(row, at_state, c, acc[i][j], acc[i][j + 1], behind.load(row, at_state, c));
        }
    }
}

// bfloat16 on the tensor cores (mma.sync m16n8k16, 32-bit accumulators), S a multiple of 64: WM x WN warps of 16 MI rows by
// 16 NJ output rows each; K in steps of 64 through a ring of three stages that cp.async fills two steps ahead, 16-byte
// chunks of a row XOR-swizzled by the row.  Two shapes: 64 rows by 128 output rows (64 channels) of a block for prompt
// portions, 16 by 64 in steps of few rows.
constexpr int PK = 64, PSTAGES = 3;

__device__ __forceinline__ void mma_bf16_16816(float* c, const uint32_t* a, const uint32_t* b) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, int bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t* r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
// byte offset of 16-byte chunk `chunk` (0..7) of row `row` in a tile whose rows are 128 bytes
__device__ __forceinline__ uint32_t swizzled(int row, int chunk) { return (uint32_t)(row * 128 + ((chunk ^ (row & 7)) << 4)); }

template <int MI, int NJ, int WM, int WN>
struct Shape {
    static constexpr int PM = 16 * MI * WM, PN = 16 * NJ * WN, THREADS = 32 * WM * WN;
    static constexpr int STAGE = (PM + PN) * 128, SMEM = PSTAGES * STAGE;
    static constexpr int A_CHUNKS = PM * 8 / THREADS, W_CHUNKS = PN * 8 / THREADS;
    static_assert(PM * 8 % THREADS == 0 && PN * 8 % THREADS == 0, "every thread copies as many chunks");
};

template <int MI, int NJ, int WM, int WN>
__global__ void __launch_bounds__(32 * WM * WN)
rglru_gates_mma_kernel(const __nv_bfloat16* __restrict__ W, Behind<__nv_bfloat16> behind, int rows, int S) {
    using Sh = Shape<MI, NJ, WM, WN>;
    extern __shared__ __align__(128) unsigned char pipe_smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int N = 2 * S, b = blockIdx.z, n0 = blockIdx.x * Sh::PN, r0 = blockIdx.y * Sh::PM;
    const __nv_bfloat16* Wb = W + (int64_t)b * N * S;
    const uint32_t base = (uint32_t)__cvta_generic_to_shared(pipe_smem);
    // a thread's chunks: chunk `tid & 7` of rows tid / 8, tid / 8 + THREADS / 8, ... of A and of W
    const int copy_row = tid >> 3, chunk = tid & 7;
    constexpr int ROW_STEP = Sh::THREADS / 8;
    const int steps = S / PK;
    auto fill_w = [&](int step) {
        const uint32_t stage = base + (uint32_t)(step % PSTAGES) * Sh::STAGE + Sh::PM * 128;
#pragma unroll
        for (int p = 0; p < Sh::W_CHUNKS; ++p) {
            const int r = copy_row + p * ROW_STEP, n = n0 + r;
            cp_async16(stage + swizzled(r, chunk), Wb + (n < N ? (int64_t)n * S : 0) + chunk * 8 + step * PK, n < N ? 16 : 0);
        }
    };
    auto fill_a = [&](int step) {
        const uint32_t stage = base + (uint32_t)(step % PSTAGES) * Sh::STAGE;
#pragma unroll
        for (int p = 0; p < Sh::A_CHUNKS; ++p) {
            const int r = copy_row + p * ROW_STEP;
            const bool there = r0 + r < rows;
            cp_async16(stage + swizzled(r, chunk),
                       behind.u + (there ? (int64_t)(r0 + r) * behind.u_stride : 0) + (int64_t)b * S + chunk * 8 + step * PK,
                       there ? 16 : 0);
        }
    };
    pdl_trigger();
    for (int s = 0; s < PSTAGES - 1; ++s)              // weights do not depend on the kernel in front
        if (s < steps) fill_w(s);
    pdl_wait();
    for (int s = 0; s < PSTAGES - 1; ++s) {
        if (s < steps) fill_a(s);
        cp_async_commit();                             // (the first group also holds the weights of both stages)
    }
    const int wm = warp / WN, wn = warp % WN;          // the warp's part of the tile
    float acc[MI][2 * NJ][4];
#pragma unroll
    for (int i = 0; i < MI; ++i)
#pragma unroll
        for (int j = 0; j < 2 * NJ; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.0f;
    for (int step = 0; step < steps; ++step) {
        cp_async_wait<PSTAGES - 2>();
        __syncthreads();                               // the stage is complete, and the stage filled next is free
        if (step + PSTAGES - 1 < steps) {
            fill_w(step + PSTAGES - 1);
            fill_a(step + PSTAGES - 1);
        }
        cp_async_commit();
        const uint32_t stage = base + (uint32_t)(step % PSTAGES) * Sh::STAGE;
#pragma unroll
        for (int ks = 0; ks < PK / 16; ++ks) {
            uint32_t a[MI][4], bb[NJ][4];
#pragma unroll
            for (int i = 0; i < MI; ++i)
                ldmatrix_x4(a[i], stage + swizzled((wm * MI + i) * 16 + (lane & 15), ks * 2 + (lane >> 4)));
#pragma unroll
            for (int j = 0; j < NJ; ++j)               // two n-tiles of eight output rows a load
                ldmatrix_x4(bb[j], stage + Sh::PM * 128 +
                                       swizzled((wn * NJ + j) * 16 + (lane & 7) + ((lane >> 4) << 3), ks * 2 + ((lane >> 3) & 1)));
#pragma unroll
            for (int i = 0; i < MI; ++i)
#pragma unroll
                for (int j = 0; j < 2 * NJ; ++j) mma_bf16_16816(acc[i][j], a[i], &bb[j >> 1][(j & 1) * 2]);
        }
    }
    cp_async_wait<0>();
    const int g = lane >> 2, t = lane & 3;
#pragma unroll
    for (int i = 0; i < MI; ++i)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int row = r0 + (wm * MI + i) * 16 + g + half * 8;
            if (row >= rows) continue;
            const int64_t at_state = behind.state_row(row);
            typename Behind<__nv_bfloat16>::Taken taken[2 * NJ];
#pragma unroll
            for (int j = 0; j < 2 * NJ; ++j) {         // n even: r of channel n / 2, and i beside it
                const int n = n0 + (wn * 2 * NJ + j) * 8 + 2 * t;
                if (n < N) taken[j] = behind.load(row, at_state, b * S + n / 2);
            }
#pragma unroll
            for (int j = 0; j < 2 * NJ; ++j) {
                const int n = n0 + (wn * 2 * NJ + j) * 8 + 2 * t;
                if (n < N) behind.finish(row, at_state, b * S + n / 2, acc[i][j][half * 2], acc[i][j][half * 2 + 1], taken[j]);
            }
        }
}

template <int MI, int NJ, int WM, int WN>
int launch_gates_mma(const __nv_bfloat16* W, const Behind<__nv_bfloat16>& behind, int rows, int blocks, int S, cudaStream_t stream) {
    using Sh = Shape<MI, NJ, WM, WN>;
    auto kernel = rglru_gates_mma_kernel<MI, NJ, WM, WN>;
    const dim3 grid((2 * S + Sh::PN - 1) / Sh::PN, (rows + Sh::PM - 1) / Sh::PM, blocks);
    if (grid.y > 65535) return TB_ERR_BAD_SIZE;
    if (Sh::SMEM > 40 * 1024) {
        cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::SMEM);
        if (err != cudaSuccess) return (int)err;
    }
    cudaError_t launched = tb_launch_pdl(kernel, grid, dim3(Sh::THREADS), (size_t)Sh::SMEM, stream, W, behind, rows, S);
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}
constexpr int kFewRows = 256;       // up to here a step takes the small tiles (a choice by the row count alone)

constexpr int kChannels = 16;       // channels of a block that cuts its rows into runs
constexpr int kMaxRuns = 64;        // runs of rows of a block (threads = runs * channels)
constexpr int kWideChannels = 128;  // channels of a block in steps of few rows (one run: the plain walk)

template <typename T>
__global__ void __launch_bounds__(kMaxRuns * kChannels)
rglru_scan_kernel(const float2* __restrict__ pairs, const T* __restrict__ y, int64_t y_stride,
                  const float* __restrict__ y_bias, float* __restrict__ state, T* __restrict__ out, int64_t out_stride,
                  const int* __restrict__ row_start, const int* __restrict__ state_slots, int width, int chans) {
    __shared__ float run_a[kMaxRuns * kChannels], run_b[kMaxRuns * kChannels];
    pdl_trigger();
    pdl_wait();
    const int ch = threadIdx.x % chans, run = threadIdx.x / chans, runs = blockDim.x / chans;
    const int seq = blockIdx.x;
    const int c = blockIdx.y * chans + ch;
    const bool active = c < width;
    const int first_row = row_start[seq];
    const int n = row_start[seq + 1] - first_row;
    const int per_run = (n + runs - 1) / runs;
    const int lo = min(n, run * per_run), hi = min(n, lo + per_run);
    float* slot_state = state + (int64_t)state_slots[seq] * width;
    float s = active ? slot_state[c] : 0.0f;
    const float by = active ? y_bias[c] : 0.0f;
    const float2* base = pairs + (int64_t)first_row * width + c;
    if (runs > 1 && n > per_run) {          // (the same for every thread of the block)
        float a = 1.0f, b = 0.0f;
        if (active) {
#pragma unroll 8
            for (int t = lo; t < hi; ++t) {
                const float2 p = base[(int64_t)t * width];
                a *= p.x;
                b = fmaf(p.x, b, p.y);
            }
        }
        run_a[run * chans + ch] = a;
        run_b[run * chans + ch] = b;
        __syncthreads();
        for (int k = 0; k < run; ++k) s = fmaf(run_a[k * chans + ch], s, run_b[k * chans + ch]);
    }
    if (!active) return;
#pragma unroll 8
    for (int t = lo; t < hi; ++t) {
        const float2 p = base[(int64_t)t * width];
        s = fmaf(p.x, s, p.y);
        const int64_t row = first_row + t;
        Elem<T>::store(out + row * out_stride + c, s * gelu_tanh_f32(Elem<T>::load(y + row * y_stride + c) + by));
    }
    if (hi == n && lo < n) slot_state[c] = s;
}

template <typename T>
Behind<T> behind_of(const void* u, int64_t u_stride, const float* bias_r, const float* bias_i, const float* rate, float* pairs,
                    float* state, const int* slots, const void* y, int64_t y_stride, const float* y_bias, void* out,
                    int64_t out_stride, int width) {
    Behind<T> b;
    b.u = (const T*)u; b.u_stride = u_stride; b.bias_r = bias_r; b.bias_i = bias_i; b.rate = rate;
    b.pairs = (float2*)pairs; b.state = state; b.slots = slots; b.y = (const T*)y; b.y_stride = y_stride;
    b.y_bias = y_bias; b.out = (T*)out; b.out_stride = out_stride; b.width = width;
    return b;
}

}  // namespace

// u: [rows, blocks * S] in dtype (row stride u_stride); W: [blocks, 2 S, S] in dtype, rows alternating (Ra, Ri); bias_r, bias_i,
// rate: 32-bit [blocks * S].  pairs: 32-bit [rows, blocks * S, 2] receives (a, x); or null, and then sequence t is row t
// and state (32-bit [slots, blocks * S]), state_slots, y, y_bias and out take part as in tb_rglru_scan.
TB_EXPORT int tb_rglru_gates(const void* u, int64_t u_stride, const void* W, const float* bias_r, const float* bias_i,
                             const float* rate, float* pairs, float* state, const int* state_slots, const void* y,
                             int64_t y_stride, const float* y_bias, void* out, int64_t out_stride, int rows, int blocks,
                             int S, int dtype, cudaStream_t stream) {
    if (rows == 0) return 0;
    if (blocks < 1 || blocks > 65535 || S < 1 || (rows + BM - 1) / BM > 65535) return TB_ERR_BAD_SIZE;
    if (pairs == nullptr && (state == nullptr || state_slots == nullptr || y == nullptr || y_bias == nullptr || out == nullptr))
        return TB_ERR_BAD_SIZE;
    if ((uintptr_t)pairs % 8 != 0) return TB_ERR_BAD_ALIGN;
    const int width = blocks * S;
    cudaError_t launched;
    if (dtype == TB_BF16 && S % PK == 0 && u_stride % 8 == 0 && ((uintptr_t)u | (uintptr_t)W) % 16 == 0) {
        const auto behind = behind_of<__nv_bfloat16>(u, u_stride, bias_r, bias_i, rate, pairs, state, state_slots, y, y_stride,
                                                     y_bias, out, out_stride, width);
        return rows <= kFewRows ? launch_gates_mma<1, 1, 1, 4>((const __nv_bfloat16*)W, behind, rows, blocks, S, stream)
                                : launch_gates_mma<2, 2, 2, 4>((const __nv_bfloat16*)W, behind, rows, blocks, S, stream);
    }
    const dim3 grid((2 * S + BN - 1) / BN, (rows + BM - 1) / BM, blocks);
    if (dtype == TB_F32)
        launched = tb_launch_pdl(rglru_gates_kernel<float>, grid, dim3(256), 0, stream, (const float*)W,
                                 behind_of<float>(u, u_stride, bias_r, bias_i, rate, pairs, state, state_slots, y, y_stride,
                                                  y_bias, out, out_stride, width), rows, S);
    else if (dtype == TB_BF16)
        launched = tb_launch_pdl(rglru_gates_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (const __nv_bfloat16*)W,
                                 behind_of<__nv_bfloat16>(u, u_stride, bias_r, bias_i, rate, pairs, state, state_slots, y,
                                                          y_stride, y_bias, out, out_stride, width), rows, S);
    else
        return TB_ERR_BAD_DTYPE;
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}

// pairs: 32-bit [rows, width, 2]; y: [rows, width] in dtype (row stride y_stride), y_bias: 32-bit [width]; state: 32-bit
// [slots, width]; out: [rows, width] in dtype; max_new: the most rows any sequence brings (it chooses the number of runs).
TB_EXPORT int tb_rglru_scan(const float* pairs, const void* y, int64_t y_stride, const float* y_bias, float* state, void* out,
                            int64_t out_stride, const int* row_start, const int* state_slots, int num_seqs, int width,
                            int max_new, int dtype, cudaStream_t stream) {
    if (num_seqs == 0) return 0;
    if (width < 1 || (width + kChannels - 1) / kChannels > 65535) return TB_ERR_BAD_SIZE;      // (grid.y)
    if ((uintptr_t)pairs % 8 != 0) return TB_ERR_BAD_ALIGN;
    int runs = 1;
    while (runs < kMaxRuns && runs * 16 < max_new) runs <<= 1;          // runs of at least 16 rows
    const int chans = runs == 1 ? kWideChannels : kChannels;
    const dim3 grid(num_seqs, (width + chans - 1) / chans);
    cudaError_t launched;
    if (dtype == TB_F32)
        launched = tb_launch_pdl(rglru_scan_kernel<float>, grid, dim3(runs * chans), 0, stream, (const float2*)pairs,
                                 (const float*)y, y_stride, y_bias, state, (float*)out, out_stride, row_start, state_slots,
                                 width, chans);
    else if (dtype == TB_BF16)
        launched = tb_launch_pdl(rglru_scan_kernel<__nv_bfloat16>, grid, dim3(runs * chans), 0, stream, (const float2*)pairs,
                                 (const __nv_bfloat16*)y, y_stride, y_bias, state, (__nv_bfloat16*)out, out_stride, row_start,
                                 state_slots, width, chans);
    else
        return TB_ERR_BAD_DTYPE;
    return launched == cudaSuccess ? tb_launch_status() : (int)launched;
}
