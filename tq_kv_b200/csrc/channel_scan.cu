// The delta rule with a decay per head and key channel over many tokens (one token per sequence: linear_scan.cu):
//
//   S' = diag(w_t) S_{t-1};   u_t = beta_t (v_t - S'^T k_t);   S_t = S' + k_t u_t^T;   o_t = S_t^T q_t
//
// per head a d x e state S.  Token by token this is a chain of two dependent passes over the state each; here the
// tokens go four at a time (CS_TOKENS).  With S_0 the state before the four, w_{a..b} the product of the decays of
// tokens a .. b (entry by entry; 1 if empty) and tokens numbered 0 .. 3:
//
//   u_i = beta_i (v_i - S_0^T k'_i - sum_{j<i} a_ij u_j),      k'_i = w_{0..i} * k_i,   a_ij = k_j . (w_{j+1..i} * k_i)
//   o_i = S_0^T q'_i + sum_{j<=i} b_ij u_j,                    q'_i = w_{0..i} * q_i,   b_ij = k_j . (w_{j+1..i} * q_i)
//   S_4 = diag(w_{0..3}) S_0 + sum_j k~_j u_j^T,               k~_j = w_{j+1..3} * k_j
//
// so that all eight products with the state are independent of one another, and what is left of the chain is a
// triangular solve over four numbers per column.  Every decay enters as a product of decays, never as a quotient:
// nothing overflows however fast a channel fades.  Everything is float32.
//
// channel_prepare   a warp per (four tokens, head) makes the primed vectors and the a_ij, b_ij once for all columns, as
//                   one record of 13 vectors and 40 numbers; it can make the decays themselves from their logits.
//                   Fours start at each sequence's first token of the step; the last one of a sequence is filled up
//                   with tokens that change nothing (w = 1, k = q = 0, beta = 0).
// channel_scan      a block owns some columns of one head of one sequence and walks the records in order, every thread
//                   4 (or 8) keys x 2 (or 4) columns of the state in registers, the records through shared memory two
//                   stages deep.
//                   The products of a thread's columns are summed over the lanes that share the columns by trading
//                   halves of the values: each lane ends with the sums it needs to hand on.  grid (sequence, head,
//                   column tile).
#include "common.cuh"

#define CS_TOKENS 4
#define CS_SCALARS 40                     // a [4][4], b [4][4], beta [4], padding

__host__ __device__ constexpr int cs_record(int dp) { return 13 * dp + CS_SCALARS; }
// the first record of sequence b, whose first token is t0: leaves room for every sequence's part-filled last four
__device__ __forceinline__ int cs_first_record(int t0, int b) { return (t0 + (CS_TOKENS - 1) * b) / CS_TOKENS; }

struct ChannelArgs {
    const float* q; const float* k; const float* v; int ldp;       // as in linear_scan.cu
    const float* w; int ldw;              // decays, or (with bias) their logits [T, H * d]
    const float* bias; const float* A_log;                         // decay = exp(-exp(A_log[h]) softplus(w + bias))
    const float* scal;                    // [T, H, 4], entry 1: beta
    int qk_div;
    float* rec;                           // records [n_rec][H][cs_record(dp)]
    int n_rec, dp;
    float* state; size_t state_stride;
    const int* cu_seqlens; const int* slots; int n_seqs;
    float* out; int ldo;
    int H, d, e, fours;                   // fours: records of a stage
    int vec;                              // v's rows can be copied in 16-byte pieces
};

__device__ __forceinline__ void cs_cp16(void* dst, const void* src) {
    const uint32_t p = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(p), "l"(src) : "memory");
}

// Sums V values over N lanes (powers of two; `l`: the lane's place among them) by trading halves: afterwards a lane
// holds the full sums of values l * (V / N) .. in v[0 ..] (N > V: of value l / (N / V)).
template <int N, int V>
__device__ __forceinline__ void cs_trade_sums(float (&v)[V], int l) {
    int count = V;
#pragma unroll
    for (int off = N / 2; off > 0; off >>= 1) {
        if (count > 1) {
            count >>= 1;
            const bool high = l & off;
#pragma unroll
            for (int i = 0; i < V / 2; ++i)
                if (i < count) {
                    const float give = high ? v[i] : v[i + count], keep = high ? v[i + count] : v[i];
                    v[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
                }
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], off);
        }
    }
}

__global__ void __launch_bounds__(128) channel_prepare_kernel(ChannelArgs a) {
    const int lane = threadIdx.x & 31;
    const long long job = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int r = (int)(job / a.H), h = (int)(job - (long long)r * a.H);
    if (r >= a.n_rec) return;
    pdl_wait();
    pdl_launch();
    int b = -1;                                          // whose record is it?
    for (int b0 = 0; b0 < a.n_seqs && b < 0; b0 += 32) {
        const int s = b0 + lane;
        bool hit = false;
        if (s < a.n_seqs) {
            const int t0 = a.cu_seqlens[s], first = cs_first_record(t0, s);
            hit = r >= first && r < first + (a.cu_seqlens[s + 1] - t0 + CS_TOKENS - 1) / CS_TOKENS;
        }
        const unsigned m = __ballot_sync(0xffffffffu, hit);
        if (m) b = b0 + __ffs(m) - 1;
    }
    if (b < 0) return;
    const int t0 = a.cu_seqlens[b], t1 = a.cu_seqlens[b + 1];
    const int t = t0 + (r - cs_first_record(t0, b)) * CS_TOKENS, n = min(CS_TOKENS, t1 - t);
    float* rec = a.rec + ((size_t)r * a.H + h) * cs_record(a.dp);
    const int hq = h / a.qk_div;
    const float fade = a.bias ? -expf(a.A_log[h]) : 0.f;
    float sums[16];                                      // a10 a20 a21 a30 a31 a32 | b00 b10 b11 b20 b21 b22 b30 .. b33
#pragma unroll
    for (int i = 0; i < 16; ++i) sums[i] = 0.f;
    for (int i0 = lane; i0 < a.dp; i0 += 32) {
        float w[CS_TOKENS], k[CS_TOKENS], q[CS_TOKENS];
#pragma unroll
        for (int i = 0; i < CS_TOKENS; ++i) {
            const bool on = i < n && i0 < a.d;
            w[i] = on ? a.w[(size_t)(t + i) * a.ldw + h * a.d + i0] : 1.f;
            k[i] = on ? a.k[(size_t)(t + i) * a.ldp + hq * a.d + i0] : 0.f;
            q[i] = on ? a.q[(size_t)(t + i) * a.ldp + hq * a.d + i0] : 0.f;
        }
        if (a.bias && i0 < a.d) {
            const float bias = a.bias[h * a.d + i0];
#pragma unroll
            for (int i = 0; i < CS_TOKENS; ++i)
                if (i < n) {
                    const float z = w[i] + bias;
                    w[i] = expf(fade * (z > 20.f ? z : log1pf(expf(z))));
                }
        }
        float run = 1.f, kt[CS_TOKENS];                  // kt[j]: k_j times the decays after it, so far
        int na = 0, nb = 6;
#pragma unroll
        for (int i = 0; i < CS_TOKENS; ++i) {
            run *= w[i];
            rec[i * a.dp + i0] = run * q[i];
            rec[(CS_TOKENS + i) * a.dp + i0] = run * k[i];
#pragma unroll
            for (int j = 0; j < i; ++j) {
                kt[j] *= w[i];
                sums[na] = fmaf(kt[j], k[i], sums[na]); ++na;
                sums[nb] = fmaf(kt[j], q[i], sums[nb]); ++nb;
            }
            kt[i] = k[i];
            sums[nb] = fmaf(k[i], q[i], sums[nb]); ++nb;
        }
#pragma unroll
        for (int j = 0; j < CS_TOKENS; ++j) rec[(2 * CS_TOKENS + j) * a.dp + i0] = kt[j];
        rec[3 * CS_TOKENS * a.dp + i0] = run;
    }
    cs_trade_sums<32, 16>(sums, lane);                       // lanes 2 s and 2 s + 1 hold sum s
    float* sc = rec + 13 * a.dp;
    if (lane < 20) {                                     // what the sums leave out: zeros above the diagonals, beta
        const int i = lane & 15, row = i >> 2, col = i & 3;
        if (lane < 16) {
            if (col >= row) sc[i] = 0.f;
            if (col > row) sc[16 + i] = 0.f;
        } else {
            const int tok = lane - 16;
            sc[32 + tok] = tok < n ? a.scal[((size_t)(t + tok) * a.H + h) * 4 + 1] : 0.f;
        }
    }
    if (!(lane & 1)) {
        const int s = lane >> 1;
        if (s < 6) {                                     // rows 1, 2, 3 with 1, 2, 3 entries
            const int row = s < 1 ? 1 : (s < 3 ? 2 : 3), col = s - row * (row - 1) / 2;
            sc[row * 4 + col] = sums[0];
        } else {                                         // rows 0 .. 3 with 1 .. 4 entries
            const int p = s - 6, row = p < 1 ? 0 : (p < 3 ? 1 : (p < 6 ? 2 : 3)), col = p - row * (row + 1) / 2;
            sc[16 + row * 4 + col] = sums[0];
        }
    }
}

// KG lanes share RC columns; each holds RK of their KG * RK (padded) keys.
template <int KG, int RK, int RC, int THREADS>
__global__ void __launch_bounds__(THREADS) channel_scan_kernel(ChannelArgs a) {
    constexpr int DP = KG * RK, REC = cs_record(DP), R4 = RK / 4, R2 = RK / 2;
    constexpr int CT = THREADS / KG * RC;
    constexpr int V = 2 * CS_TOKENS * RC;                // sums per four tokens and thread
    constexpr int PER = KG >= V ? 1 : V / KG;            // of which a lane holds this many after trading
    constexpr int SAME = KG >= V ? KG / V : 1;           // and this many lanes hold the same
    extern __shared__ __align__(16) float sm[];
    const int b = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * CT;
    const int tid = threadIdx.x, kg = tid % KG, cg = tid / KG;
    const int colb = col0 + cg * RC;
    const int d = a.d, e = a.e, F = a.fours;
    const int stage_floats = F * (REC + CS_TOKENS * CT);
    for (int i = tid; i < 2 * stage_floats; i += THREADS) sm[i] = 0.f;       // (columns past e stay zero)
    pdl_wait();
    pdl_launch();
    const int t0 = a.cu_seqlens[b], t1 = a.cu_seqlens[b + 1];
    const int n4 = (t1 - t0 + CS_TOKENS - 1) / CS_TOKENS;
    const float* rec0 = a.rec + ((size_t)cs_first_record(t0, b) * a.H + head) * REC;
    float* st = a.state + (size_t)a.slots[b] * a.state_stride + (size_t)head * d * e;
    float2 S[R2][RC];                                    // S[r][c]: keys 2r and 2r + 1 of this thread, column c
#pragma unroll
    for (int r = 0; r < RK; ++r) {
        const int key = ((r >> 2) * KG + kg) * 4 + (r & 3);
#pragma unroll
        for (int c = 0; c < RC; ++c) {
            const float x = (key < d && colb + c < e) ? st[(size_t)key * e + colb + c] : 0.f;
            if (r & 1) S[r >> 1][c].y = x; else S[r >> 1][c].x = x;
        }
    }
    __syncthreads();

    const int cols = min(CT, e - col0);
    auto stage_in = [&](int first, int s) {              // records first .. first + F - 1 and their tokens' values
        const int n = min(F, n4 - first);
        float* dst = sm + s * stage_floats;
        float* dv = dst + F * REC;
        for (int idx = tid; idx < n * (REC / 4); idx += THREADS) {
            const int f = idx / (REC / 4), i = (idx - f * (REC / 4)) * 4;
            cs_cp16(dst + f * REC + i, rec0 + (size_t)(first + f) * a.H * REC + i);
        }
        const int base = t0 + first * CS_TOKENS, nt = min(n * CS_TOKENS, t1 - base);
        if (a.vec && CT % 4 == 0) {
            const int c4 = cols >> 2;
            for (int idx = tid; idx < nt * c4; idx += THREADS) {
                const int tt = idx / c4, c = (idx - tt * c4) * 4;
                cs_cp16(dv + tt * CT + c, a.v + (size_t)(base + tt) * a.ldp + head * e + col0 + c);
            }
        } else {
            for (int idx = tid; idx < nt * cols; idx += THREADS) {
                const int tt = idx / cols, c = idx - tt * cols;
                dv[tt * CT + c] = a.v[(size_t)(base + tt) * a.ldp + head * e + col0 + c];
            }
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    // (where two lanes end with the same sum one of them hands it on)
    const bool o_lane = kg % SAME == 0;

    if (n4 > 0) stage_in(0, 0);
    int s = 0;
    for (int first = 0; first < n4; first += F, s ^= 1) {
        const int n = min(F, n4 - first);
        if (first + F < n4) {
            stage_in(first + F, s ^ 1);
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        const float* src = sm + s * stage_floats;
        const float* sv = src + F * REC + cg * RC;
        const int base = t0 + first * CS_TOKENS, left = t1 - base;       // tokens from this stage on
#pragma unroll 2
        for (int f = 0; f < n; ++f) {
            const float4* vecs = reinterpret_cast<const float4*>(src + f * REC) + kg;
            const float* sc = src + f * REC + 13 * DP;
            // the products with the state: value (type * 4 + token) * RC + column, type 0 keys, 1 queries
            float r[V];
#pragma unroll
            for (int type = 0; type < 2; ++type)
#pragma unroll
                for (int i = 0; i < CS_TOKENS; ++i) {
                    float2 acc[RC];
#pragma unroll
                    for (int g = 0; g < R4; ++g) {
                        const float4 p = vecs[(type == 0 ? CS_TOKENS + i : i) * (DP / 4) + g * KG];
#pragma unroll
                        for (int c = 0; c < RC; ++c) {
                            acc[c] = g == 0 ? __fmul2_rn(make_float2(p.x, p.y), S[0][c])
                                            : __ffma2_rn(make_float2(p.x, p.y), S[2 * g][c], acc[c]);
                            acc[c] = __ffma2_rn(make_float2(p.z, p.w), S[2 * g + 1][c], acc[c]);
                        }
                    }
#pragma unroll
                    for (int c = 0; c < RC; ++c) r[(type * CS_TOKENS + i) * RC + c] = acc[c].x + acc[c].y;
                }
            cs_trade_sums<KG, V>(r, kg);
            // every lane takes the keys' products back and solves for the four u of its columns
            const float4 a1 = *reinterpret_cast<const float4*>(sc + 4), a2 = *reinterpret_cast<const float4*>(sc + 8);
            const float4 a3 = *reinterpret_cast<const float4*>(sc + 12), be = *reinterpret_cast<const float4*>(sc + 32);
            float u[CS_TOKENS][RC], x[CS_TOKENS][RC];
#pragma unroll
            for (int i = 0; i < CS_TOKENS; ++i) {
                float v[RC];
#pragma unroll
                for (int c = 0; c < RC; c += 2) {
                    const float2 two = *reinterpret_cast<const float2*>(sv + (f * CS_TOKENS + i) * CT + c);
                    v[c] = two.x;
                    v[c + 1] = two.y;
                }
#pragma unroll
                for (int c = 0; c < RC; ++c) {
                    const int id = i * RC + c;
                    const int src_lane = (tid & 31 & ~(KG - 1)) + id / PER * SAME;
                    const float dot = __shfl_sync(0xffffffffu, r[id % PER], src_lane);
                    x[i][c] = (f * CS_TOKENS + i < left ? v[c] : 0.f) - dot;
                }
            }
#pragma unroll
            for (int c = 0; c < RC; ++c) {
                u[0][c] = be.x * x[0][c];
                u[1][c] = be.y * fmaf(-a1.x, u[0][c], x[1][c]);
                u[2][c] = be.z * fmaf(-a2.y, u[1][c], fmaf(-a2.x, u[0][c], x[2][c]));
                u[3][c] = be.w * fmaf(-a3.z, u[2][c], fmaf(-a3.y, u[1][c], fmaf(-a3.x, u[0][c], x[3][c])));
            }
            // the state after the four tokens
#pragma unroll
            for (int g = 0; g < R4; ++g) {
                const float4 p = vecs[3 * CS_TOKENS * (DP / 4) + g * KG];
#pragma unroll
                for (int c = 0; c < RC; ++c) {
                    S[2 * g][c] = __fmul2_rn(make_float2(p.x, p.y), S[2 * g][c]);
                    S[2 * g + 1][c] = __fmul2_rn(make_float2(p.z, p.w), S[2 * g + 1][c]);
                }
            }
#pragma unroll
            for (int j = 0; j < CS_TOKENS; ++j)
#pragma unroll
                for (int g = 0; g < R4; ++g) {
                    const float4 p = vecs[(2 * CS_TOKENS + j) * (DP / 4) + g * KG];
#pragma unroll
                    for (int c = 0; c < RC; ++c) {
                        const float2 uu = make_float2(u[j][c], u[j][c]);
                        S[2 * g][c] = __ffma2_rn(make_float2(p.x, p.y), uu, S[2 * g][c]);
                        S[2 * g + 1][c] = __ffma2_rn(make_float2(p.z, p.w), uu, S[2 * g + 1][c]);
                    }
                }
            // the lanes that hold the queries' products finish the results
#pragma unroll
            for (int p = 0; p < PER; ++p) {
                const int id = kg / SAME * PER + p;
                const int i = (id / RC) & 3, c = id % RC, tok = f * CS_TOKENS + i;
                const float4 bi = *reinterpret_cast<const float4*>(sc + 16 + 4 * i);
                float uc[CS_TOKENS];                     // the u of column c (whose low part p fixes)
#pragma unroll
                for (int j = 0; j < CS_TOKENS; ++j) {
                    uc[j] = u[j][p % RC];
#pragma unroll
                    for (int m = PER; m < RC; m += PER)
                        if (c == m + p) uc[j] = u[j][(m + p) % RC];
                }
                float o = fmaf(bi.x, uc[0], r[p]);
                o = fmaf(bi.y, uc[1], o);
                o = fmaf(bi.z, uc[2], o);
                o = fmaf(bi.w, uc[3], o);
                if (id >= CS_TOKENS * RC && o_lane && tok < left && colb + c < e)
                    a.out[(size_t)(base + tok) * a.ldo + head * e + colb + c] = o;
            }
        }
        __syncthreads();                                 // the stage may be refilled
    }
#pragma unroll
    for (int r = 0; r < RK; ++r) {
        const int key = ((r >> 2) * KG + kg) * 4 + (r & 3);
#pragma unroll
        for (int c = 0; c < RC; ++c)
            if (key < d && colb + c < e) st[(size_t)key * e + colb + c] = (r & 1) ? S[r >> 1][c].y : S[r >> 1][c].x;
    }
}

#define CS_SMEM_ALONE (116 * 1024)        // the most a block asks for
#define CS_SMEM_SM (230 * 1024)           // a little more than an SM has for all its blocks

template <int KG, int RK, int RC, int THREADS>
static int launch_channel_scan(const ChannelArgs& a, cudaStream_t stream) {
    constexpr int CT = THREADS / KG * RC, REC = cs_record(KG * RK);
    const dim3 grid(a.n_seqs, a.H, (a.e + CT - 1) / CT);
    // Blocks that start while the kernel before drains gather on the SMs that fall free first; so a block of a small
    // grid asks for as much shared memory as lets no SM take more than its share of them.
    const long long per_sm = ((long long)grid.x * grid.y * grid.z + tq_sm_count() - 1) / tq_sm_count();
    ChannelArgs args = a;
    args.fours = per_sm <= 2 && REC < 2000 ? 4 : 2;
    size_t smem = (size_t)2 * args.fours * (REC + CS_TOKENS * CT) * sizeof(float);
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(channel_scan_kernel<KG, RK, RC, THREADS>,
                                             cudaFuncAttributeMaxDynamicSharedMemorySize, CS_SMEM_ALONE);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    if (smem > CS_SMEM_ALONE) return (int)cudaErrorInvalidValue;
    if (per_sm <= 4) {
        const size_t share = (size_t)CS_SMEM_SM / (per_sm + 1);
        if (smem < share) smem = share;
    }
    return tq_launch_pdl(TQ_PDL_ELEMENTWISE, channel_scan_kernel<KG, RK, RC, THREADS>, grid, dim3(THREADS), smem, stream, args);
}

// Few sequences and heads: short chains count (four keys a thread, two columns), in blocks of eight warps while they
// still give most SMs one, in smaller ones where columns are few.  Many: reads of shared memory count (eight keys, four
// columns: a vector read serves twice the columns, its sums half the lanes).
template <int KG, int RK>
static int pick_channel_scan(const ChannelArgs& a, cudaStream_t stream) {
    auto blocks = [&](int kg, int rc, int threads) {
        const int ct = threads / kg * rc;
        return (long long)a.n_seqs * a.H * ((a.e + ct - 1) / ct);
    };
    if constexpr (RK == 4 && KG >= 16) {
        constexpr int HALF = KG / 2;
        if (blocks(HALF, 4, 128) > 2ll * tq_sm_count() && a.e >= 128 / HALF * 4)
            return launch_channel_scan<HALF, 8, 4, 128>(a, stream);
    }
    if (blocks(KG, 2, 256) >= tq_sm_count() / 2 && a.e >= 256 / KG * 2) return launch_channel_scan<KG, RK, 2, 256>(a, stream);
    if (blocks(KG, 2, 128) >= tq_sm_count() / 2 || KG == 8) return launch_channel_scan<KG, RK, 2, 128>(a, stream);
    return launch_channel_scan<KG, RK, 2, 64>(a, stream);
}

// Floats of the records for a step of n_tokens tokens in n_seqs sequences, heads H of d keys.
TQ_API long long tq_channel_scan_floats(int n_tokens, int n_seqs, int H, int d) {
    const int dp = d <= 32 ? 32 : (d <= 64 ? 64 : (d <= 128 ? 128 : 256));
    return (long long)((n_tokens + (CS_TOKENS - 1) * n_seqs) / CS_TOKENS + 1) * H * cs_record(dp);
}

// q, k [T, ldp] with H / qk_div heads of d (ready: activations, unit lengths and scales applied), v [T, ldp] with H heads
// of e, all columns of one float32 buffer; w [T, ldw] the decays of the H heads' d channels or, with bias [H * d] and
// A_log [H], their logits; scal [T, H, 4] with beta in entry 1; rec: tq_channel_scan_floats() floats of scratch (16-byte
// aligned); state: slot 0's [H, d, e] block, state_stride floats between slots.  Key widths up to 256.
TQ_API int tq_channel_scan(const float* q, const float* k, const float* v, int ldp, const float* w, int ldw,
                           const float* bias, const float* A_log, const float* scal, int qk_div, float* rec, float* state,
                           long long state_stride, const int* cu_seqlens, const int* slots, int n_seqs, int n_tokens,
                           float* out, int ldo, int H, int d, int e, cudaStream_t stream) {
    if (n_seqs <= 0 || n_tokens <= 0) return 0;
    if (!q || !k || !v || !w || !scal || !rec || !state || !cu_seqlens || !slots || !out || H <= 0 || H > 65535 || d <= 0 ||
        d > 256 || e <= 0 || qk_div <= 0 || H % qk_div || state_stride < (long long)H * d * e || ldw < H * d ||
        (bias && !A_log) || (reinterpret_cast<uintptr_t>(rec) & 15))
        return (int)cudaErrorInvalidValue;
    ChannelArgs a{};
    a.q = q; a.k = k; a.v = v; a.ldp = ldp; a.w = w; a.ldw = ldw; a.bias = bias; a.A_log = A_log; a.scal = scal;
    a.qk_div = qk_div; a.rec = rec; a.dp = d <= 32 ? 32 : (d <= 64 ? 64 : (d <= 128 ? 128 : 256));
    a.n_rec = (n_tokens + (CS_TOKENS - 1) * n_seqs) / CS_TOKENS + 1;
    a.state = state; a.state_stride = (size_t)state_stride; a.cu_seqlens = cu_seqlens; a.slots = slots; a.n_seqs = n_seqs;
    a.out = out; a.ldo = ldo; a.H = H; a.d = d; a.e = e;
    a.vec = e % 4 == 0 && ldp % 4 == 0 && (reinterpret_cast<uintptr_t>(v) & 15) == 0;
    const long long warps = (long long)a.n_rec * H, blocks = (warps + 3) / 4;
    if (blocks > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
    int st = tq_launch_pdl(TQ_PDL_ELEMENTWISE, channel_prepare_kernel, dim3((unsigned)blocks), dim3(128), 0, stream, a);
    if (st) return st;
    if (d <= 32) return pick_channel_scan<8, 4>(a, stream);
    if (d <= 64) return pick_channel_scan<16, 4>(a, stream);
    if (d <= 128) return pick_channel_scan<32, 4>(a, stream);
    return pick_channel_scan<32, 8>(a, stream);
}
