// A gated recurrence per channel whose gates read the current token only (minGRU):
//
//   z = sigmoid(z~),  c = u + 1/2 for u >= 0, sigmoid(u) below      (z~, u: projections with their biases)
//   S_t = (1 - z_t) S_{t-1} + z_t c_t                                per channel, S zero at first
//   out_t = scale * S_t * silu(g_t)
//
// Since S_t is an affine function of S_{t-1}, a run of tokens is one too: S -> A S + B.  A block owns GRU_COLS
// neighbouring channels of one sequence and takes GRU_SEGS * GRU_LEN tokens at a time: each of its GRU_SEGS warps
// forms the (A, B) of its own GRU_LEN tokens (a lane per channel, the gates stay in registers), the runs' (A, B)
// meet in shared memory, every warp finds the state before its own tokens by walking the runs before it, and then
// walks its tokens once more for the results.  The state is read from the sequence's slot before the first token and
// written back after the last, so a prompt and a portion of one are the same kernel.  A decode step (one token per
// sequence) is a thread per channel.  Everything is float32; only the result is rounded to the activations' type.
#include "common.cuh"

#define GRU_COLS 32
#define GRU_SEGS 16
#define GRU_LEN 8

struct GruArgs {
    const float* z; const float* u; const float* g;     // columns of one projection buffer
    int ld;
    float* state; size_t state_stride;                   // [slots, W]
    const int* cu_seqlens; const int* slots;
    int W;
    float scale;
};

__device__ __forceinline__ float gru_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float gru_candidate(float u) { return u >= 0.f ? u + 0.5f : gru_sigmoid(u); }

template <typename TO>
__global__ void __launch_bounds__(GRU_COLS * GRU_SEGS) gru_scan_kernel(GruArgs a, TO* __restrict__ out) {
    __shared__ float2 runs[GRU_SEGS][GRU_COLS];
    const int lane = threadIdx.x & 31, seg = threadIdx.x >> 5;
    const int b = blockIdx.x, c = blockIdx.y * GRU_COLS + lane;
    const bool on = c < a.W;
    pdl_wait();
    pdl_launch();
    const int t0 = a.cu_seqlens[b], t1 = a.cu_seqlens[b + 1];
    if (t0 >= t1) return;
    float* sp = a.state + (size_t)a.slots[b] * a.state_stride + c;
    float S = on ? *sp : 0.f;                            // the state before this turn's tokens (the same in every warp)
    for (int base = t0; base < t1; base += GRU_SEGS * GRU_LEN) {
        const int first = base + seg * GRU_LEN;
        float keep[GRU_LEN], add[GRU_LEN], gv[GRU_LEN];
#pragma unroll
        for (int i = 0; i < GRU_LEN; ++i) {
            const bool ok = on && first + i < t1;
            const size_t at = (size_t)(first + i) * a.ld + c;
            keep[i] = ok ? a.z[at] : 0.f;
            add[i] = ok ? a.u[at] : 0.f;
            gv[i] = ok ? a.g[at] : 0.f;
        }
        float A = 1.f, B = 0.f;
#pragma unroll
        for (int i = 0; i < GRU_LEN; ++i) {
            const bool ok = on && first + i < t1;        // a token past the end leaves the state as it is
            const float z = gru_sigmoid(keep[i]);
            add[i] = ok ? z * gru_candidate(add[i]) : 0.f;
            keep[i] = ok ? 1.f - z : 1.f;
            A *= keep[i];
            B = fmaf(keep[i], B, add[i]);
        }
        runs[seg][lane] = make_float2(A, B);
        __syncthreads();
        float mine = S;
#pragma unroll
        for (int s = 0; s < GRU_SEGS; ++s) {
            const float2 r = runs[s][lane];
            S = fmaf(r.x, S, r.y);
            if (s + 1 == seg) mine = S;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < GRU_LEN; ++i) {
            mine = fmaf(keep[i], mine, add[i]);
            if (on && first + i < t1)
                out[(size_t)(first + i) * a.W + c] = from_f32<TO>(a.scale * mine * (gv[i] * gru_sigmoid(gv[i])));
        }
    }
    if (on && seg == 0) *sp = S;
}

// one token per sequence
template <typename TO>
__global__ void __launch_bounds__(128) gru_step_kernel(GruArgs a, TO* __restrict__ out, int n_seqs) {
    const int b = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
    pdl_wait();
    pdl_launch();
    if (c >= a.W) return;
    const int t = a.cu_seqlens[b];
    float* sp = a.state + (size_t)a.slots[b] * a.state_stride + c;
    const size_t at = (size_t)t * a.ld + c;
    const float z = gru_sigmoid(a.z[at]), g = a.g[at];
    const float S = fmaf(1.f - z, *sp, z * gru_candidate(a.u[at]));
    *sp = S;
    out[(size_t)t * a.W + c] = from_f32<TO>(a.scale * S * (g * gru_sigmoid(g)));
}

// z, u, g: float32 columns (row stride ld) of W entries per token; state points at the W entries of slot 0, slots are
// state_stride floats apart; out [T, W] float32 or bfloat16.  `single`: every sequence brings exactly one token.
TQ_API int tq_gru_scan(const float* z, const float* u, const float* g, int ld, float* state, long long state_stride,
                       const int* cu_seqlens, const int* slots, int n_seqs, int n_tokens, int single, int W, float scale,
                       void* out, int out_dtype, cudaStream_t stream) {
    if (n_seqs <= 0 || n_tokens <= 0) return 0;
    if (!z || !u || !g || !state || !cu_seqlens || !slots || !out || W <= 0 || state_stride < W || n_seqs > 65535)
        return (int)cudaErrorInvalidValue;
    if (single && n_tokens != n_seqs) return (int)cudaErrorInvalidValue;
    const GruArgs a{z, u, g, ld, state, (size_t)state_stride, cu_seqlens, slots, W, scale};
    const dim3 grid_s((W + 127) / 128, n_seqs), grid(n_seqs, (W + GRU_COLS - 1) / GRU_COLS);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
#define TQ_GRU(TO)                                                                                                   \
    return single ? tq_launch_pdl(TQ_PDL_ELEMENTWISE, gru_step_kernel<TO>, grid_s, dim3(128), 0, stream, a, (TO*)out, n_seqs) \
                  : tq_launch_pdl(TQ_PDL_ELEMENTWISE, gru_scan_kernel<TO>, grid, dim3(GRU_COLS * GRU_SEGS), 0, stream, a, (TO*)out)
    if (out_dtype == TQ_F32) TQ_GRU(float);
    if (out_dtype == TQ_BF16) TQ_GRU(bf16);
#undef TQ_GRU
    return (int)cudaErrorInvalidValue;
}
