// Per-token vectors that are a product of two small matrices with the layer's input, z = W2 (W1 h): the decays of a
// recurrence with one decay per head and key channel, and the gate of its result.  W1 h of both rides in the layer's
// one projection product (float32 columns); here is the second half.
//
//   decays   w[t, i] = exp(-exp(A_log[i / d]) * softplus(z[t, i] + bias[i]))      (always float32)
//   plain    z[t, i]
//
// low_rank_rows: both products of a step in one launch, each with inner width r of any size, on CUDA cores with
// float32 sums: a warp per output entry, LR_ROWS tokens at a time (its row of W2 is then read once for them).  It is
// the form for decoding, for the float32 path and for small r.  For many tokens and large r the products run on the
// tensor cores (gemm_tc.cu) and channel_decay turns their result into decays in place.
#include "common.cuh"

#define LR_ROWS 8
#define LR_WARPS 8

struct LowRankJob {
    const float* low;      // [T, ld] columns of the projection: W1 h
    int rank;
    const void* w2;        // [n, rank]
    int n;
    float* out;            // [T, n]
};

__device__ __forceinline__ float lr_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float lr_decay(float z, float a_log) { return expf(-expf(a_log) * lr_softplus(z)); }

// grid (ceil((jobs' n) / LR_WARPS), ceil(T / LR_ROWS)); outputs 0 .. a.n-1 are the decays, then the plain ones
template <typename TW>
__global__ void __launch_bounds__(LR_WARPS * 32)
low_rank_rows_kernel(LowRankJob a, LowRankJob p, int ld, const float* __restrict__ bias, const float* __restrict__ A_log,
                     int d, int T) {
    const int lane = threadIdx.x & 31;
    int i = blockIdx.x * LR_WARPS + (threadIdx.x >> 5);
    const bool decays = i < a.n;
    if (!decays) i -= a.n;
    const LowRankJob& job = decays ? a : p;
    if (i >= job.n) return;
    const int t0 = blockIdx.y * LR_ROWS, rows = min(LR_ROWS, T - t0);
    const TW* w = reinterpret_cast<const TW*>(job.w2) + (size_t)i * job.rank;
    pdl_wait();
    pdl_launch();
    float acc[LR_ROWS];
#pragma unroll
    for (int r = 0; r < LR_ROWS; ++r) acc[r] = 0.f;
    for (int k = lane; k < job.rank; k += 32) {
        const float wv = to_f32<TW>(w[k]);
#pragma unroll
        for (int r = 0; r < LR_ROWS; ++r)
            if (r < rows) acc[r] = fmaf(wv, job.low[(size_t)(t0 + r) * ld + k], acc[r]);
    }
    float mine = 0.f;                                   // lane r keeps row r's sum
#pragma unroll
    for (int r = 0; r < LR_ROWS; ++r) {
        const float s = warp_sum(acc[r]);
        if (lane == r) mine = s;
    }
    if (lane >= rows) return;
    if (decays) mine = lr_decay(mine + bias[i], A_log[i / d]);
    job.out[(size_t)(t0 + lane) * job.n + i] = mine;
}

// low_a / low_p: columns of float32 rows with stride ld; w2_a [na, ra], w2_p [np, rp] of one dtype; bias [na],
// A_log [na / d]; decay [T, na], plain [T, np] float32.  np may be 0.
TQ_API int tq_low_rank_rows(const float* low_a, int ra, const void* w2_a, int na, const float* bias, const float* A_log,
                            int d, float* decay, const float* low_p, int rp, const void* w2_p, int np, float* plain,
                            int ld, int w_dtype, int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (!low_a || !w2_a || !bias || !A_log || !decay || ra <= 0 || na <= 0 || d <= 0 || na % d || np < 0 ||
        (np > 0 && (!low_p || !w2_p || !plain || rp <= 0)))
        return (int)cudaErrorInvalidValue;
    const LowRankJob a{low_a, ra, w2_a, na, decay}, p{low_p, rp, w2_p, np, plain};
    const dim3 grid((na + np + LR_WARPS - 1) / LR_WARPS, (n_tokens + LR_ROWS - 1) / LR_ROWS);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
    if (w_dtype == TQ_F32)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, low_rank_rows_kernel<float>, grid, dim3(LR_WARPS * 32), 0, stream, a, p, ld,
                             bias, A_log, d, n_tokens);
    if (w_dtype == TQ_BF16)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, low_rank_rows_kernel<bf16>, grid, dim3(LR_WARPS * 32), 0, stream, a, p, ld,
                             bias, A_log, d, n_tokens);
    return (int)cudaErrorInvalidValue;
}

// z [T, n] float32 (the product, without bias) -> decays, in place
__global__ void __launch_bounds__(256)
channel_decay_kernel(float* __restrict__ z, const float* __restrict__ bias, const float* __restrict__ A_log, int d, int n,
                     size_t total) {
    pdl_wait();
    pdl_launch();
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
        const int i = (int)(idx % n);
        z[idx] = lr_decay(z[idx] + bias[i], A_log[i / d]);
    }
}

TQ_API int tq_channel_decay(float* z, const float* bias, const float* A_log, int d, int n, int n_tokens,
                            cudaStream_t stream) {
    const size_t total = (size_t)n_tokens * n;
    if (total == 0) return 0;
    if (!z || !bias || !A_log || d <= 0 || n % d) return (int)cudaErrorInvalidValue;
    size_t blocks = (total + 255) / 256;
    if (blocks > 148 * 8) blocks = 148 * 8;
    return tq_launch_pdl(TQ_PDL_ELEMENTWISE, channel_decay_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, z, bias,
                         A_log, d, n, total);
}

// columns of float32 rows, rounded: out[t, i] = bfloat16(x[t * ld + i]), i < n
__global__ void __launch_bounds__(256)
round_columns_kernel(const float* __restrict__ x, int ld, bf16* __restrict__ out, int n, size_t total) {
    pdl_wait();
    pdl_launch();
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
        const size_t t = idx / n;
        out[idx] = __float2bfloat16_rn(x[t * ld + (idx - t * n)]);
    }
}

TQ_API int tq_round_columns(const float* x, int ld, void* out, int n, int n_tokens, cudaStream_t stream) {
    const size_t total = (size_t)n_tokens * n;
    if (total == 0) return 0;
    if (!x || !out || ld < n) return (int)cudaErrorInvalidValue;
    size_t blocks = (total + 255) / 256;
    if (blocks > 148 * 8) blocks = 148 * 8;
    return tq_launch_pdl(TQ_PDL_ELEMENTWISE, round_columns_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, x, ld,
                         (bf16*)out, n, total);
}
