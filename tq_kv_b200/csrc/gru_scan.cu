// A recurrence per channel with an update gate that does not look at the state (minGRU):
//
//   z = sigmoid(z~),  c = u + 1/2 for u >= 0, sigmoid(u) below      (z~, u: projections with their biases)
//   S_t = (1 - z_t) S_{t-1} + z_t c_t                                per channel, S zero at first
//   out_t = scale * S_t * silu(g_t)
//
// Since S_t is an affine function of S_{t-1}, a run of tokens is one too: S -> A S + B.  A thread-block cluster owns
// GRU_COLS neighbouring channels of one sequence; its blocks lie side by side in time and take GRU_SEGS * GRU_LEN
// tokens each per turn: every warp forms the (A, B) of its own GRU_LEN tokens (a lane per channel, the gates stay in
// registers), the warps' (A, B) meet in shared memory, the blocks' in one another's (read by rank order); every warp
// then finds the state before its own tokens by walking the runs before it, and walks its tokens once more for the
// results.  The next turn's inputs are asked for before this turn's are used.  The state is read from the sequence's
// slot before the first token and written back after the last, so a prompt and a portion of one are the same kernel.
// A decode step (one token per sequence) is a thread per channel.  Everything is float32; only the result is rounded
// to the activations' type.
#include <cooperative_groups.h>

#include "common.cuh"
namespace cg = cooperative_groups;

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

__device__ __forceinline__ float gru_sigmoid(float x) { return __fdividef(1.f, 1.f + expf(-x)); }     // (2 ulp; exp < 2^126 here or 0)
__device__ __forceinline__ float gru_candidate(float u) { return u >= 0.f ? u + 0.5f : gru_sigmoid(u); }

template <typename TO>
__global__ void __launch_bounds__(GRU_COLS * GRU_SEGS, 2) gru_scan_kernel(GruArgs a, TO* __restrict__ out) {
    __shared__ float2 runs[GRU_SEGS][GRU_COLS];
    __shared__ float2 whole[2][GRU_COLS];                // this block's run of a turn (read by the cluster's blocks)
    cg::cluster_group cluster = cg::this_cluster();
    const int n_ranks = (int)cluster.num_blocks(), rank = (int)cluster.block_rank();
    const int lane = threadIdx.x & 31, seg = threadIdx.x >> 5;
    const int b = blockIdx.y, c = (blockIdx.x / n_ranks) * GRU_COLS + lane;
    const bool on = c < a.W;
    pdl_wait();
    pdl_launch();
    const int t0 = a.cu_seqlens[b], t1 = a.cu_seqlens[b + 1];
    if (t0 >= t1) return;                                // (all blocks of a cluster alike)
    float* sp = a.state + (size_t)a.slots[b] * a.state_stride + c;
    float S = on ? *sp : 0.f;                            // the state before this turn's tokens (the same everywhere)
    const int turn = n_ranks * GRU_SEGS * GRU_LEN, mine0 = (rank * GRU_SEGS + seg) * GRU_LEN;
    float zn[GRU_LEN], un[GRU_LEN], gn[GRU_LEN];
    auto load = [&](int first) {
#pragma unroll
        for (int i = 0; i < GRU_LEN; ++i) {
            const bool ok = on && first + i < t1;
            const size_t at = (size_t)(first + i) * a.ld + c;
            zn[i] = ok ? a.z[at] : 0.f;
            un[i] = ok ? a.u[at] : 0.f;
            gn[i] = ok ? a.g[at] : 0.f;
        }
    };
    load(t0 + mine0);
    int parity = 0;
    for (int base = t0; base < t1; base += turn, parity ^= 1) {
        const int first = base + mine0;
        float keep[GRU_LEN], add[GRU_LEN], gv[GRU_LEN];
        float A = 1.f, B = 0.f;
#pragma unroll
        for (int i = 0; i < GRU_LEN; ++i) {
            const bool ok = on && first + i < t1;        // a token past the end leaves the state as it is
            const float z = gru_sigmoid(zn[i]);
            add[i] = ok ? z * gru_candidate(un[i]) : 0.f;
            keep[i] = ok ? 1.f - z : 1.f;
            gv[i] = gn[i];
            A *= keep[i];
            B = fmaf(keep[i], B, add[i]);
        }
        if (base + turn < t1) load(first + turn);
        runs[seg][lane] = make_float2(A, B);
        __syncthreads();
        A = 1.f, B = 0.f;                                // the run of this block's warps before this one, then of all
        float Am = 1.f, Bm = 0.f;
#pragma unroll
        for (int s = 0; s < GRU_SEGS; ++s) {
            if (s == seg) { Am = A; Bm = B; }
            const float2 r = runs[s][lane];
            A *= r.x;
            B = fmaf(r.x, B, r.y);
        }
        float mine = S;
        if (n_ranks > 1) {
            if (seg == 0) whole[parity][lane] = make_float2(A, B);
            cluster.sync();                              // (whole[] of the turn after next is written after the next sync)
            for (int p = 0; p < n_ranks; ++p) {
                const float2 r = cluster.map_shared_rank(&whole[parity][0], p)[lane];
                S = fmaf(r.x, S, r.y);
                if (p + 1 == rank) mine = S;
            }
        } else {
            S = fmaf(A, S, B);
            __syncthreads();                             // runs[] is read; the next turn may write it
        }
        mine = fmaf(Am, mine, Bm);
#pragma unroll
        for (int i = 0; i < GRU_LEN; ++i) {
            mine = fmaf(keep[i], mine, add[i]);
            if (on && first + i < t1)
                out[(size_t)(first + i) * a.W + c] = from_f32<TO>(a.scale * mine * (gv[i] * gru_sigmoid(gv[i])));
        }
    }
    if (on && seg == 0 && rank == 0) *sp = S;
    if (n_ranks > 1) cluster.sync();                     // a block keeps its shared memory until it was read
}

template <typename TO>
static int launch_gru_scan(const GruArgs& a, TO* out, int n_seqs, int n_tokens, cudaStream_t stream) {
    // blocks side by side in time: as many as the sequences' mean length keeps busy, while SMs are free for them
    const int tiles = (a.W + GRU_COLS - 1) / GRU_COLS;
    int ranks = 1;
    while (ranks < 8 && ranks * GRU_SEGS * GRU_LEN < n_tokens / n_seqs && (long long)tiles * n_seqs * ranks < 4ll * tq_sm_count())
        ranks *= 2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(tiles * ranks, n_seqs, 1);
    cfg.blockDim = dim3(GRU_COLS * GRU_SEGS, 1, 1);
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = ranks;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = tq_pdl_enabled(TQ_PDL_ELEMENTWISE) ? 1 : 0;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    cudaError_t e = cudaLaunchKernelEx(&cfg, gru_scan_kernel<TO>, a, out);
    if (e != cudaSuccess) return (int)e;
    return tq_launch_status();
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
    const dim3 grid_s((W + 127) / 128, n_seqs);
#define TQ_GRU(TO)                                                                                                   \
    return single ? tq_launch_pdl(TQ_PDL_ELEMENTWISE, gru_step_kernel<TO>, grid_s, dim3(128), 0, stream, a, (TO*)out, n_seqs) \
                  : launch_gru_scan<TO>(a, (TO*)out, n_seqs, n_tokens, stream)
    if (out_dtype == TQ_F32) TQ_GRU(float);
    if (out_dtype == TQ_BF16) TQ_GRU(bf16);
#undef TQ_GRU
    return (int)cudaErrorInvalidValue;
}
