// Attention through a latent: every token is cached as ONE row, the normed latent c (n values) followed by a
// rotated key part k_r (r values) that all heads share.  Head h's key would be [U_k[h] c, k_r] and its value
// U_v[h] c; instead of expanding the cache, the query is carried into the latent's space,
//
//   q~[h] = [U_k[h]^T q_flat[h], rot(q_rot[h])]       (n + r values),    score = q~[h] . [c, k_r] * scale,
//
// the attention kernels run with one shared key/value head whose rows are the cache rows (the value of a row being
// the row itself), and the result, a weighted mean of latents, is expanded afterwards:  o[h] = U_v[h] mean(c).
// The three kernels here are what stands around those attention kernels:
//
//   latent_rows    per token, from the float32 results of the down projections: the RMS-normed query latent (for the
//                  up projection that follows); the cache row [norm(c) * w, rot(k_r), 0 ...] written to the step's
//                  packed rows and / or the sequence's page; rows are padded with zeros to the width `rp` the
//                  attention kernels take
//   latent_query   per (token, head): q~ as above
//   latent_expand  per (token, head): o[h] = U_v[h] mean(c), times sigmoid(gate) entry by entry or (head_gate) with one
//                  gate per head
//
// In bfloat16 latent_query and latent_expand run on the tensor cores (latent_product_kernel), 16 tokens at a time.
//
//   latent_heads   for prompts that bring all their keys along: per (token, head) the query [q_flat, rot(q_rot), 0 ...],
//                  the expanded key [U_k[h] c, k_r, 0 ...] and the value [U_v[h] c, 0 ...], all `hw` wide, for the
//                  ordinary attention kernels (whose heads then are this mixer's heads); latent_expand without a
//                  matrix then only gates and narrows the result
//
// Rotation: of the r rotated entries the first `rot_dims` are turned by the angle pos * rate_i (tables of cosines and
// sines per position come ready-made), in neighbouring pairs (2i, 2i+1) if `paired`, else entry i with i + rot_dims/2.
// Norms, rotation and the per-head sums are float32.
#include "common.cuh"

__device__ __forceinline__ float rot_entry(const float* x, int i, int rot_dims, int paired, const float* cs,
                                           const float* sn) {
    if (i >= rot_dims) return x[i];
    const int half = rot_dims >> 1;
    if (paired) {
        const int p = i >> 1;
        return (i & 1) ? x[i] * cs[p] + x[i - 1] * sn[p] : x[i] * cs[p] - x[i + 1] * sn[p];
    }
    return i < half ? x[i] * cs[i] - x[i + half] * sn[i] : x[i] * cs[i - half] + x[i - half] * sn[i - half];
}

template <typename T>
__global__ void latent_rows_kernel(const float* __restrict__ proj, int ld, int off_q, int off_kv, int q_rank, int n, int r,
                                   int rp, const float* __restrict__ wq, const float* __restrict__ wkv, float eps,
                                   const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot_dims,
                                   int paired, const int* __restrict__ tok_pos, const int* __restrict__ tok_seq,
                                   const int* __restrict__ new_lens, T* __restrict__ cq_out, T* __restrict__ row_out,
                                   T* __restrict__ pages, const int* __restrict__ block_table, int table_width,
                                   int page_tokens, int ring_pages) {
    extern __shared__ float sh[];          // [r] the raw rotated part
    __shared__ float red[32];
    const int t = blockIdx.x;
    pdl_wait();
    pdl_launch();
    const float* row = proj + (size_t)t * ld;
    const int pos = tok_pos[t], b = tok_seq[t];
    // the query latent (q_rank == 0: the queries are projected directly and there is none)
    float ss = 0.f, inv = 0.f;
    if (q_rank > 0) {
        for (int i = threadIdx.x; i < q_rank; i += blockDim.x) ss = fmaf(row[off_q + i], row[off_q + i], ss);
        ss = block_sum(ss, red);
        inv = 1.f / sqrtf(ss / (float)q_rank + eps);
        for (int i = threadIdx.x; i < q_rank; i += blockDim.x)
            cq_out[(size_t)t * q_rank + i] = from_f32<T>(row[off_q + i] * inv * wq[i]);
    }
    // the cache row
    ss = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) ss = fmaf(row[off_kv + i], row[off_kv + i], ss);
    ss = block_sum(ss, red);
    inv = 1.f / sqrtf(ss / (float)n + eps);
    for (int i = threadIdx.x; i < r; i += blockDim.x) sh[i] = row[off_kv + n + i];
    __syncthreads();
    T* dst_page = nullptr;
    // in a ring (a window's cache) only the last ring_pages * page_tokens positions of a sequence are written
    if (pages && pos < new_lens[b] && (ring_pages <= 0 || pos >= new_lens[b] - ring_pages * page_tokens)) {
        const int lp = ring_pages > 0 ? (pos / page_tokens) % ring_pages : pos / page_tokens;
        const int page = block_table[(size_t)b * table_width + lp];
        dst_page = pages + ((size_t)page * page_tokens + (pos % page_tokens)) * rp;
    }
    T* dst_row = row_out ? row_out + (size_t)t * rp : nullptr;
    const float* cs = cos_t + (size_t)pos * (rot_dims >> 1);
    const float* sn = sin_t + (size_t)pos * (rot_dims >> 1);
    for (int i = threadIdx.x; i < rp; i += blockDim.x) {
        float v = 0.f;
        if (i < n) v = row[off_kv + i] * inv * wkv[i];
        else if (i < n + r) v = rot_entry(sh, i - n, rot_dims, paired, cs, sn);
        const T o = from_f32<T>(v);
        if (dst_page) dst_page[i] = o;
        if (dst_row) dst_row[i] = o;
    }
}

template <typename T>
__global__ void latent_query_kernel(const float* __restrict__ q, int ldq, int H, int d, int r, int n, int rp,
                                    const T* __restrict__ uk, const float* __restrict__ cos_t,
                                    const float* __restrict__ sin_t, int rot_dims, int paired,
                                    const int* __restrict__ tok_pos, T* __restrict__ out) {
    extern __shared__ float sh[];          // [d + r] this head's query
    const int t = blockIdx.x, h = blockIdx.y;
    pdl_wait();
    pdl_launch();
    const float* qr = q + (size_t)t * ldq + (size_t)h * (d + r);
    for (int i = threadIdx.x; i < d + r; i += blockDim.x) sh[i] = qr[i];
    __syncthreads();
    const int pos = tok_pos[t];
    const float* cs = cos_t + (size_t)pos * (rot_dims >> 1);
    const float* sn = sin_t + (size_t)pos * (rot_dims >> 1);
    T* o = out + ((size_t)t * H + h) * rp;
    const T* w = uk + (size_t)h * d * n;            // [d, n]: row k holds what flat key entry k takes of the latent
    for (int i = threadIdx.x; i < rp; i += blockDim.x) {
        float v = 0.f;
        if (i < n) {
            for (int k = 0; k < d; ++k) v = fmaf(sh[k], to_f32<T>(w[(size_t)k * n + i]), v);
        } else if (i < n + r) {
            v = rot_entry(sh + d, i - n, rot_dims, paired, cs, sn);
        }
        o[i] = from_f32<T>(v);
    }
}

// q float32 [T, H * (d + r)]; kfv float32 [T, ldk]: head h's flat key at column h * d, its value at off_v + h * e;
// rows [T, rp]: the cache rows, whose entries n .. n + r - 1 are the rotated key part.
template <typename T>
__global__ void latent_heads_kernel(const float* __restrict__ q, int ldq, const float* __restrict__ kfv, int ldk, int off_v,
                                    const T* __restrict__ rows, int rp, int n, int H, int d, int r, int e, int hw,
                                    const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot_dims,
                                    int paired, const int* __restrict__ tok_pos, T* __restrict__ q_out,
                                    T* __restrict__ k_out, T* __restrict__ v_out) {
    extern __shared__ float sh[];          // [r] this head's rotated query part, raw
    const int t = blockIdx.x, h = blockIdx.y;
    pdl_wait();
    pdl_launch();
    const float* qr = q + (size_t)t * ldq + (size_t)h * (d + r);
    for (int i = threadIdx.x; i < r; i += blockDim.x) sh[i] = qr[d + i];
    __syncthreads();
    const int pos = tok_pos[t];
    const float* cs = cos_t + (size_t)pos * (rot_dims >> 1);
    const float* sn = sin_t + (size_t)pos * (rot_dims >> 1);
    const size_t o = ((size_t)t * H + h) * hw;
    const float* kr = kfv + (size_t)t * ldk + (size_t)h * d;
    const float* vr = kfv + (size_t)t * ldk + off_v + (size_t)h * e;
    const T* rr = rows + (size_t)t * rp + n;
    for (int i = threadIdx.x; i < hw; i += blockDim.x) {
        T qv = from_f32<T>(0.f), kv = qv;
        if (i < d) { qv = from_f32<T>(qr[i]); kv = from_f32<T>(kr[i]); }
        else if (i < d + r) { qv = from_f32<T>(rot_entry(sh, i - d, rot_dims, paired, cs, sn)); kv = rr[i - d]; }
        q_out[o + i] = qv;
        k_out[o + i] = kv;
        v_out[o + i] = i < e ? from_f32<T>(vr[i]) : from_f32<T>(0.f);
    }
}

// The same for bfloat16 with d, r, e and hw in multiples of four and aligned rows: a block per token, a thread per four
// neighbouring entries of a head's q, k and v.
__device__ __forceinline__ void lh_store4(bf16* dst, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}
__global__ void __launch_bounds__(256)
latent_heads4_kernel(const float* __restrict__ q, int ldq, const float* __restrict__ kfv, int ldk, int off_v,
                     const bf16* __restrict__ rows, int rp, int n, int H, int d, int r, int e, int hw,
                     const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot_dims, int paired,
                     const int* __restrict__ tok_pos, bf16* __restrict__ q_out, bf16* __restrict__ k_out,
                     bf16* __restrict__ v_out) {
    const int t = blockIdx.x, hw4 = hw >> 2;
    pdl_wait();
    pdl_launch();
    const size_t at = (size_t)tok_pos[t] * (rot_dims >> 1);
    const float *cs = cos_t + at, *sn = sin_t + at;
    const float* qt = q + (size_t)t * ldq;
    const float* kt = kfv + (size_t)t * ldk;
    const bf16* rr = rows + (size_t)t * rp + n;
    const uint2 none = make_uint2(0u, 0u);
    for (int p = threadIdx.x; p < H * hw4; p += blockDim.x) {
        const int h = p / hw4, i = (p - h * hw4) * 4;
        const size_t o = ((size_t)t * H + h) * hw + i;
        const float* qr = qt + h * (d + r);
        if (i < d) {
            lh_store4(q_out + o, *reinterpret_cast<const float4*>(qr + i));
            lh_store4(k_out + o, *reinterpret_cast<const float4*>(kt + h * d + i));
        } else if (i < d + r) {
            float4 v;
            v.x = rot_entry(qr + d, i - d, rot_dims, paired, cs, sn);
            v.y = rot_entry(qr + d, i - d + 1, rot_dims, paired, cs, sn);
            v.z = rot_entry(qr + d, i - d + 2, rot_dims, paired, cs, sn);
            v.w = rot_entry(qr + d, i - d + 3, rot_dims, paired, cs, sn);
            lh_store4(q_out + o, v);
            *reinterpret_cast<uint2*>(k_out + o) = *reinterpret_cast<const uint2*>(rr + i - d);
        } else {
            *reinterpret_cast<uint2*>(q_out + o) = none;
            *reinterpret_cast<uint2*>(k_out + o) = none;
        }
        if (i < e) lh_store4(v_out + o, *reinterpret_cast<const float4*>(kt + off_v + h * e + i));
        else *reinterpret_cast<uint2*>(v_out + o) = none;
    }
}

template <typename T>
__global__ void latent_expand_kernel(const T* __restrict__ lat, int H, int n, int rp, int e, const T* __restrict__ uv,
                                     const float* __restrict__ gate, int ldg, int head_gate, T* __restrict__ out) {
    extern __shared__ float sh[];          // [n] the head's mean latent
    const int t = blockIdx.x, h = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    pdl_wait();
    pdl_launch();
    const T* lr = lat + ((size_t)t * H + h) * rp;
    for (int i = threadIdx.x; i < n; i += blockDim.x) sh[i] = to_f32<T>(lr[i]);
    __syncthreads();
    if (!uv) {                             // nothing to expand: the head's first e entries, gated
        for (int j = threadIdx.x; j < e; j += blockDim.x) {
            const size_t c = (size_t)h * e + j;
            float acc = sh[j];
            if (gate) acc *= 1.f / (1.f + expf(-gate[(size_t)t * ldg + (head_gate ? h : c)]));
            out[(size_t)t * H * e + c] = from_f32<T>(acc);
        }
        return;
    }
    for (int j = warp; j < e; j += n_warps) {
        const T* w = uv + ((size_t)h * e + j) * n;
        float acc = 0.f;
        for (int i = lane; i < n; i += 32) acc = fmaf(to_f32<T>(w[i]), sh[i], acc);
        acc = warp_sum(acc);
        if (lane == 0) {
            const size_t c = (size_t)h * e + j;
            if (gate) acc *= 1.f / (1.f + expf(-gate[(size_t)t * ldg + (head_gate ? h : c)]));
            out[(size_t)t * H * e + c] = from_f32<T>(acc);
        }
    }
}

// ---- the per-head products on the tensor cores (bfloat16) ------------------------------------------------------------
// C[t, h, :N] = A[t, h, :K] . B_h for 16 tokens and 64 columns of one head per block: the head's matrix is read once
// per 16 tokens instead of once per token.  KN: B_h lies [K, N] (latent_query: U_k[h], k rows of n entries), else
// [N, K] (latent_expand: U_v[h], e rows of n entries); both with rows of whole 16-byte pieces.  A (float32 queries or
// bfloat16 means) is rounded to bfloat16 in shared memory, sums are float32; K is walked in pieces of LP_KC.
// The epilogue rounds once: for queries the first column tile also writes the rotated part and the row's padding; for
// results the gate is applied.
#define LP_TOK 16
#define LP_COLS 64
#define LP_KC 128

__device__ __forceinline__ void lp_ldmatrix_x4(uint32_t* r, const void* smem) {
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void lp_ldmatrix_x4_trans(uint32_t* r, const void* smem) {
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void lp_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct LpQuery {          // what the query's epilogue needs beyond the product
    int d, r, rp, rot_dims, paired;
    const float *cos_t, *sin_t;
    const int* tok_pos;
};

template <typename TA, bool KN>
__global__ void __launch_bounds__(128)
latent_product_kernel(const TA* __restrict__ a, int lda, int a_head, const bf16* __restrict__ w, int H, int K, int N,
                      bf16* __restrict__ out, int out_head, int n_tokens, LpQuery qq, const float* __restrict__ gate,
                      int ldg, int head_gate, int a_vec) {
    constexpr int AW = LP_KC + 8;                              // padded rows: ldmatrix without bank conflicts
    constexpr int BW = KN ? LP_COLS + 8 : LP_KC + 8;
    constexpr int BROWS = KN ? LP_KC : LP_COLS;
    __shared__ __align__(16) bf16 a_s[LP_TOK * AW];
    __shared__ __align__(16) bf16 b_s[BROWS * BW];
    const int h = blockIdx.x, c0 = blockIdx.y * LP_COLS, t0 = blockIdx.z * LP_TOK;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const bf16 zero = __float2bfloat16_rn(0.f);
    const bf16* wh = w + (size_t)h * K * N;
    // the first piece of the head's matrix does not depend on the kernel before
    auto load_b = [&](int k0) {
        constexpr int PER = (KN ? LP_COLS : LP_KC) / 8, COPIES = BROWS * PER / 128;
        uint4 v[COPIES];                                       // all loads in flight before the first store
#pragma unroll
        for (int i = 0; i < COPIES; ++i) {
            const int p = threadIdx.x + 128 * i, row = p / PER, c = (p - row * PER) * 8;
            const int k = KN ? k0 + row : k0 + c, n = KN ? c0 + c : c0 + row;
            v[i] = make_uint4(0u, 0u, 0u, 0u);
            if (k < K && n < N) v[i] = *reinterpret_cast<const uint4*>(wh + (KN ? (size_t)k * N + n : (size_t)n * K + k));
        }
#pragma unroll
        for (int i = 0; i < COPIES; ++i) {
            const int p = threadIdx.x + 128 * i, row = p / PER, c = (p - row * PER) * 8;
            *reinterpret_cast<uint4*>(b_s + row * BW + c) = v[i];
        }
    };
    load_b(0);
    pdl_wait();
    pdl_launch();
    float acc[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) { acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f; }
    for (int k0 = 0; k0 < K; k0 += LP_KC) {
        const int kc = min(LP_KC, (K - k0 + 15) & ~15);
        if (k0 > 0) { __syncthreads(); load_b(k0); }
        if (a_vec) {                                           // rows of whole 16-byte pieces: four entries at a time
            constexpr int COPIES = LP_TOK * LP_KC / 4 / 128;
            float v[COPIES][4];
#pragma unroll
            for (int i = 0; i < COPIES; ++i) {
                const int p = threadIdx.x + 128 * i, row = p / (LP_KC / 4), k = k0 + (p - row * (LP_KC / 4)) * 4;
                v[i][0] = v[i][1] = v[i][2] = v[i][3] = 0.f;
                if (t0 + row < n_tokens && k < K) {
                    const TA* ar = a + (size_t)(t0 + row) * lda + (size_t)h * a_head + k;
                    if constexpr (sizeof(TA) == 4) load16_f32<TA>(ar, v[i]);
                    else {
                        const float2 x = load2_f32<TA>(ar), y = load2_f32<TA>(ar + 2);
                        v[i][0] = x.x; v[i][1] = x.y; v[i][2] = y.x; v[i][3] = y.y;
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < COPIES; ++i) {
                const int p = threadIdx.x + 128 * i, row = p / (LP_KC / 4), c = (p - row * (LP_KC / 4)) * 4;
                store2_f32<bf16>(a_s + row * AW + c, v[i][0], v[i][1]);
                store2_f32<bf16>(a_s + row * AW + c + 2, v[i][2], v[i][3]);
            }
        } else {
            for (int p = threadIdx.x; p < LP_TOK * LP_KC / 2; p += 128) {
                const int row = p / (LP_KC / 2), c = (p - row * (LP_KC / 2)) * 2, t = t0 + row, k = k0 + c;
                bf16 v0 = zero, v1 = zero;
                if (t < n_tokens) {
                    const TA* ar = a + (size_t)t * lda + (size_t)h * a_head;
                    if (k < K) v0 = from_f32<bf16>(to_f32<TA>(ar[k]));
                    if (k + 1 < K) v1 = from_f32<bf16>(to_f32<TA>(ar[k + 1]));
                }
                a_s[row * AW + c] = v0;
                a_s[row * AW + c + 1] = v1;
            }
        }
        __syncthreads();
        const int mat = lane >> 3, r8 = lane & 7;
        for (int ks = 0; ks < kc; ks += 16) {
            uint32_t af[4], bfr[4];
            lp_ldmatrix_x4(af, a_s + ((mat & 1) * 8 + r8) * AW + ks + (mat >> 1) * 8);
            if (KN) lp_ldmatrix_x4_trans(bfr, b_s + (ks + (mat & 1) * 8 + r8) * BW + warp * 16 + (mat >> 1) * 8);
            else lp_ldmatrix_x4(bfr, b_s + (warp * 16 + (mat >> 1) * 8 + r8) * BW + ks + (mat & 1) * 8);
            lp_mma(acc[0], af, bfr[0], bfr[1]);
            lp_mma(acc[1], af, bfr[2], bfr[3]);
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int t = t0 + (lane >> 2) + 8 * (e >> 1), n = c0 + warp * 16 + i * 8 + 2 * (lane & 3) + (e & 1);
            if (t < n_tokens && n < N) {
                float v = acc[i][e];
                if (gate) v *= 1.f / (1.f + expf(-gate[(size_t)t * ldg + (head_gate ? h : h * N + n)]));
                out[((size_t)t * H + h) * out_head + n] = from_f32<bf16>(v);
            }
        }
    if (KN && blockIdx.y == 0) {                               // the rotated part and the padding behind it
        const int rest = qq.rp - N;
        for (int p = threadIdx.x; p < LP_TOK * rest; p += 128) {
            const int row = p / rest, i = p - row * rest, t = t0 + row;
            if (t >= n_tokens) continue;
            float v = 0.f;
            if (i < qq.r) {
                const size_t at = (size_t)qq.tok_pos[t] * (qq.rot_dims >> 1);
                const TA* ar = a + (size_t)t * lda + (size_t)h * a_head + qq.d;
                if constexpr (sizeof(TA) == 4) v = rot_entry(ar, i, qq.rot_dims, qq.paired, qq.cos_t + at, qq.sin_t + at);
            }
            out[((size_t)t * H + h) * out_head + N + i] = from_f32<bf16>(v);
        }
    }
}

static bool lp_aligned(const void* p, int row) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && row % 8 == 0; }

TQ_API int tq_latent_rows(const float* proj, int ld, int off_q, int off_kv, int q_rank, int n, int r, int rp,
                          const float* wq, const float* wkv, float eps, const float* cos_t, const float* sin_t,
                          int rot_dims, int paired, const int* tok_pos, const int* tok_seq, const int* new_lens,
                          void* cq_out, void* row_out, void* pages, const int* block_table, int table_width,
                          int page_tokens, int ring_pages, int dtype, int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (!proj || !wkv || !cos_t || !sin_t || !tok_pos || !tok_seq || !new_lens || q_rank < 0 ||
        (q_rank > 0 && (!wq || !cq_out)) || n <= 0 ||
        r < 0 || rp < n + r || rot_dims < 0 || rot_dims > r || (rot_dims & 1) || (pages && (!block_table || page_tokens <= 0)))
        return (int)cudaErrorInvalidValue;
    const int threads = (n >= 512 || q_rank >= 512) ? 256 : 128;
    const size_t smem = (size_t)(r > 0 ? r : 1) * sizeof(float);
    if (dtype == TQ_F32)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_rows_kernel<float>, dim3(n_tokens), dim3(threads), smem, stream,
                             proj, ld, off_q, off_kv, q_rank, n, r, rp, wq, wkv, eps, cos_t, sin_t, rot_dims, paired,
                             tok_pos, tok_seq, new_lens, (float*)cq_out, (float*)row_out, (float*)pages, block_table,
                             table_width, page_tokens, ring_pages);
    if (dtype == TQ_BF16)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_rows_kernel<bf16>, dim3(n_tokens), dim3(threads), smem, stream,
                             proj, ld, off_q, off_kv, q_rank, n, r, rp, wq, wkv, eps, cos_t, sin_t, rot_dims, paired,
                             tok_pos, tok_seq, new_lens, (bf16*)cq_out, (bf16*)row_out, (bf16*)pages, block_table,
                             table_width, page_tokens, ring_pages);
    return (int)cudaErrorInvalidValue;
}

TQ_API int tq_latent_query(const float* q, int ldq, int H, int d, int r, int n, int rp, const void* uk, const float* cos_t,
                           const float* sin_t, int rot_dims, int paired, const int* tok_pos, void* out, int dtype,
                           int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (!q || !uk || !cos_t || !sin_t || !tok_pos || !out || H <= 0 || H > 65535 || d <= 0 || r < 0 || n <= 0 ||
        rp < n + r || rot_dims < 0 || rot_dims > r || (rot_dims & 1))
        return (int)cudaErrorInvalidValue;
    if (dtype == TQ_BF16 && lp_aligned(uk, n) && (n_tokens + LP_TOK - 1) / LP_TOK <= 65535 && (n + LP_COLS - 1) / LP_COLS <= 65535)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_product_kernel<float, true>,
                             dim3(H, (n + LP_COLS - 1) / LP_COLS, (n_tokens + LP_TOK - 1) / LP_TOK), dim3(128), 0, stream, q,
                             ldq, d + r, (const bf16*)uk, H, d, n, (bf16*)out, rp, n_tokens,
                             LpQuery{d, r, rp, rot_dims, paired, cos_t, sin_t, tok_pos}, (const float*)nullptr, 0, 0,
                             (int)(!((ldq | d | r) & 3) && (reinterpret_cast<uintptr_t>(q) & 15) == 0));
    const int threads = rp > 128 ? 256 : 128;
    const size_t smem = (size_t)(d + r) * sizeof(float);
    const dim3 grid(n_tokens, H);
    if (dtype == TQ_F32)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_query_kernel<float>, grid, dim3(threads), smem, stream, q, ldq, H, d, r,
                             n, rp, (const float*)uk, cos_t, sin_t, rot_dims, paired, tok_pos, (float*)out);
    if (dtype == TQ_BF16)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_query_kernel<bf16>, grid, dim3(threads), smem, stream, q, ldq, H, d, r,
                             n, rp, (const bf16*)uk, cos_t, sin_t, rot_dims, paired, tok_pos, (bf16*)out);
    return (int)cudaErrorInvalidValue;
}

TQ_API int tq_latent_expand(const void* lat, int H, int n, int rp, int e, const void* uv, const float* gate, int ldg,
                            int head_gate, void* out, int dtype, int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (!lat || !out || H <= 0 || H > 65535 || n <= 0 || rp < n || e <= 0 || (!uv && e > n)) return (int)cudaErrorInvalidValue;
    if (dtype == TQ_BF16 && uv && lp_aligned(uv, n) && (n_tokens + LP_TOK - 1) / LP_TOK <= 65535 &&
        (e + LP_COLS - 1) / LP_COLS <= 65535)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_product_kernel<bf16, false>,
                             dim3(H, (e + LP_COLS - 1) / LP_COLS, (n_tokens + LP_TOK - 1) / LP_TOK), dim3(128), 0, stream,
                             (const bf16*)lat, H * rp, rp, (const bf16*)uv, H, n, e, (bf16*)out, e, n_tokens,
                             LpQuery{0, 0, 0, 0, 0, nullptr, nullptr, nullptr}, gate, ldg, head_gate,
                             (int)(!((rp | n) & 3) && (reinterpret_cast<uintptr_t>(lat) & 7) == 0));
    const size_t smem = (size_t)n * sizeof(float);
    const dim3 grid(n_tokens, H);
    if (dtype == TQ_F32)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_expand_kernel<float>, grid, dim3(128), smem, stream,
                             (const float*)lat, H, n, rp, e, (const float*)uv, gate, ldg, head_gate, (float*)out);
    if (dtype == TQ_BF16)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_expand_kernel<bf16>, grid, dim3(128), smem, stream,
                             (const bf16*)lat, H, n, rp, e, (const bf16*)uv, gate, ldg, head_gate, (bf16*)out);
    return (int)cudaErrorInvalidValue;
}

TQ_API int tq_latent_heads(const float* q, int ldq, const float* kfv, int ldk, int off_v, const void* rows, int rp, int n, int H,
                           int d, int r, int e, int hw, const float* cos_t, const float* sin_t, int rot_dims, int paired,
                           const int* tok_pos, void* q_out, void* k_out, void* v_out, int dtype, int n_tokens,
                           cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (!q || !kfv || !rows || !cos_t || !sin_t || !tok_pos || !q_out || !k_out || !v_out || H <= 0 || H > 65535 ||
        d <= 0 || r < 0 || e <= 0 || hw < d + r || hw < e || rp < n + r || rot_dims < 0 || rot_dims > r || (rot_dims & 1))
        return (int)cudaErrorInvalidValue;
    auto al = [](const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; };
    if (dtype == TQ_BF16 && !((d | r | e | hw | n | ldq | ldk | off_v) & 3) && !(rp & 3) && al(q, 16) && al(kfv, 16) &&
        al(rows, 8) && al(q_out, 8) && al(k_out, 8) && al(v_out, 8))
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_heads4_kernel, dim3(n_tokens), dim3(256), 0, stream, q, ldq, kfv, ldk,
                             off_v, (const bf16*)rows, rp, n, H, d, r, e, hw, cos_t, sin_t, rot_dims, paired, tok_pos,
                             (bf16*)q_out, (bf16*)k_out, (bf16*)v_out);
    const dim3 grid(n_tokens, H);
    const size_t smem = (size_t)(r > 0 ? r : 1) * sizeof(float);
    if (dtype == TQ_F32)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_heads_kernel<float>, grid, dim3(128), smem, stream, q, ldq, kfv, ldk,
                             off_v, (const float*)rows, rp, n, H, d, r, e, hw, cos_t, sin_t, rot_dims, paired, tok_pos,
                             (float*)q_out, (float*)k_out, (float*)v_out);
    if (dtype == TQ_BF16)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, latent_heads_kernel<bf16>, grid, dim3(128), smem, stream, q, ldq, kfv, ldk,
                             off_v, (const bf16*)rows, rp, n, H, d, r, e, hw, cos_t, sin_t, rot_dims, paired, tok_pos,
                             (bf16*)q_out, (bf16*)k_out, (bf16*)v_out);
    return (int)cudaErrorInvalidValue;
}
