// From a token's projected row to the heads an attention kernel reads, and
// into the cache: one kernel for mixers whose projections come as one float32
// row per token, [q heads | k heads | (v heads) | (anything else)], at any
// column offsets.
//
//   q and k heads (hd entries each) are either rotated by position (rotate-half
//   layout: entry i < rot/2 is paired with entry i + rot/2; cosine and sine
//   come from tables [positions, rot/2], which may carry a common factor;
//   entries from `rot` on pass; with `paired` the neighbours 2i and 2i + 1 are
//   a pair instead) or, with norm_eps > 0, divided by their root
//   mean square, x / sqrt(mean(x^2) + norm_eps), or left as they are; with
//   `row_inv` (float32 [T, 2]: one factor per token for its whole q row and
//   one for its whole k row, made by row_inv_rms below) and weights over those
//   whole rows, q and k are first multiplied by factor * weight: an RMS norm
//   over the whole projection, before the heads are split and turned; with
//   norm_eps and weights of one head's size (shared by the heads) each head is
//   normed, weighted and then turned;
//   with `maps` > 1 every q and k head is `maps` vectors of hd entries, each
//   normed and turned for itself; a key row holds its head's maps side by side,
//   and every map's query becomes a head of its own (head h's map m is head
//   h * maps + m) whose row is zero but for its map's place: the product with a
//   key row is then the map's own score, and the ordinary grouped attention
//   kernels serve all maps of a key/value head in one pass over its rows;
//   rows may be wider than what they hold (kr, vr entries), zeros behind;
//   v heads (vd entries each) are copied, times v_scale: from their own columns, or — v_col < 0
//   — from the k columns as projected, before the rotation (vd == hd then).
//
// q goes to q_out [T, nh*hd]; k and v go to the packed outputs (if given) and
// into the paged cache (if given) under the rules of the rotary kernel of
// elementwise.cu: position p of step row b lands in logical page
// p / page_tokens (modulo ring_pages if > 0) at row p % page_tokens; in a ring
// only the last ring_pages*page_tokens positions of a sequence are written;
// a row at or past new_lens of its sequence is padding and is not cached.
//
// Also here: the sigmoid gate on the attention's result and the tanh cap.
#include "common.cuh"

#define HE_MAX_PER_LANE 16    // head widths up to 512

template <typename TC>
__global__ void __launch_bounds__(128)
head_encode_kernel(const float* __restrict__ proj, int ld, int q_col, int k_col, int v_col,
                   const float* __restrict__ cos_tab, const float* __restrict__ sin_tab, int rot, float norm_eps,
                   const int* __restrict__ tok_pos, const int* __restrict__ tok_seq,
                   const int* __restrict__ new_lens, const int* __restrict__ block_table, int table_width,
                   int ring_pages, int page_tokens, TC* __restrict__ q_out, TC* __restrict__ k_out,
                   TC* __restrict__ v_out, TC* __restrict__ k_pages, TC* __restrict__ v_pages, int nh, int nkv,
                   int hd, int vd, const float* __restrict__ row_inv, const float* __restrict__ q_w,
                   const float* __restrict__ k_w, int paired, float v_scale, int maps, int kr, int vr) {
    // grid (token, groups of four vectors), a warp per vector: nh * maps of q, then nkv * maps of k, then nkv of v
    const int t = blockIdx.x, lane = threadIdx.x & 31;
    const int head = blockIdx.y * 4 + (threadIdx.x >> 5);
    const int nq = nh * maps, nk = nkv * maps;
    if (head >= nq + nk + nkv) return;
    const int pos = tok_pos[t];
    const int b = tok_seq[t];
    const bool is_q = head < nq, is_k = !is_q && head < nq + nk;
    const int g = is_q ? head : (is_k ? head - nq : head - nq - nk);
    const int map = g % maps, map_off = map * hd;            // (of a q or k vector: its place in the row)
    const int width = (is_q || is_k) ? hd : vd;
    const float* x = proj + (size_t)t * ld +
                     (is_q ? q_col + g * hd : (is_k ? k_col + g * hd : (v_col >= 0 ? v_col + g * vd : k_col + g * hd)));

    TC* cache = nullptr;
    if (!is_q && k_pages != nullptr) {
        int lp = pos / page_tokens;
        bool keep = pos < new_lens[b];
        if (ring_pages > 0) {
            keep = keep && pos >= new_lens[b] - ring_pages * page_tokens;
            lp %= ring_pages;
        }
        if (keep) {
            const int page = block_table[(size_t)b * table_width + lp];
            const size_t row = ((size_t)page * nkv + (is_k ? g / maps : g)) * page_tokens + (pos % page_tokens);
            cache = is_k ? k_pages + row * kr + map_off : v_pages + row * vr;
        }
    }
    TC* dst = is_q ? q_out + ((size_t)t * nq + g) * kr + map_off
                   : (is_k ? (k_out ? k_out + ((size_t)t * nkv + g / maps) * kr + map_off : nullptr)
                           : (v_out ? v_out + ((size_t)t * nkv + g) * vr : nullptr));
    pdl_wait();
    pdl_launch();
    // zeros around a map's query, behind a key row's last map, behind a value row
    const TC zero = from_f32<TC>(0.f);
    if (is_q) {
        TC* row = dst - map_off;
        for (int d = lane; d < kr; d += 32)
            if (d < map_off || d >= map_off + hd) row[d] = zero;
    } else {
        const int from = is_k ? hd : vd;
        const int end = is_k ? (map == maps - 1 ? kr - map_off : hd) : vr;
        for (int d = from + lane; d < end; d += 32) {
            if (dst) dst[d] = zero;
            if (cache) cache[d] = zero;
        }
    }
    if (!is_q && !is_k) {                                    // values: a copy
        for (int d = lane; d < width; d += 32) {
            const TC r = from_f32<TC>(x[d] * v_scale);
            if (dst) dst[d] = r;
            if (cache) cache[d] = r;
        }
        return;
    }
    float inv = 1.f;
    if (norm_eps > 0.f) {
        float ss = 0.f;
        for (int d = lane; d < width; d += 32) ss = fmaf(x[d], x[d], ss);
        ss = warp_sum(ss);
        inv = 1.f / sqrtf(ss / (float)width + norm_eps);
    }
    const float* w = is_q ? q_w : k_w;                       // the norm's weights: of every head, or (whole-row norm) of this one
    if (row_inv) {
        inv = row_inv[2 * t + (is_q ? 0 : 1)];
        w += (size_t)g * hd;
    }
    const int half = rot >> 1;
    if (half > 0) {
        const float* cs = cos_tab + (size_t)pos * half;
        const float* sn = sin_tab + (size_t)pos * half;
        for (int j = lane; j < half; j += 32) {
            const int i0 = paired ? 2 * j : j, i1 = paired ? 2 * j + 1 : j + half;
            float x0 = x[i0] * inv, x1 = x[i1] * inv;
            if (w) { x0 *= w[i0]; x1 *= w[i1]; }
            const float c = cs[j], s = sn[j];
            const TC r0 = from_f32<TC>(x0 * c - x1 * s);
            const TC r1 = from_f32<TC>(x1 * c + x0 * s);
            if (dst) { dst[i0] = r0; dst[i1] = r1; }
            if (cache) { cache[i0] = r0; cache[i1] = r1; }
        }
    }
    for (int d = rot + lane; d < width; d += 32) {
        const TC r = from_f32<TC>(w ? x[d] * inv * w[d] : x[d] * inv);
        if (dst) dst[d] = r;
        if (cache) cache[d] = r;
    }
}

// The same for heads of up to 128 entries in pieces of four (hd, rot / 2, vd, kr, vr, the columns and the row stride
// multiples of four, halves layout, values of their own, no whole-row norm, one or two maps): LPV lanes per head, four
// neighbouring entries per lane, a head's maps one after the other with the same weights and table entries, the
// partner entries of a rotation by shuffles, 8-byte (16-byte) stores.
template <typename TC> __device__ __forceinline__ void he_store4(TC* p, const float* v);
template <> __device__ __forceinline__ void he_store4<float>(float* p, const float* v) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void he_store4<bf16>(bf16* p, const float* v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

template <typename TC, int LPV, int MAPS>
__global__ void __launch_bounds__(128)
head_encode4_kernel(const float* __restrict__ proj, int ld, int q_col, int k_col, int v_col,
                    const float* __restrict__ cos_tab, const float* __restrict__ sin_tab, int rot, float norm_eps,
                    const int* __restrict__ tok_pos, const int* __restrict__ tok_seq, const int* __restrict__ new_lens,
                    const int* __restrict__ block_table, int table_width, int ring_pages, int page_tokens,
                    TC* __restrict__ q_out, TC* __restrict__ k_out, TC* __restrict__ v_out, TC* __restrict__ k_pages,
                    TC* __restrict__ v_pages, int nh, int nkv, int hd, int vd, const float* __restrict__ q_w,
                    const float* __restrict__ k_w, float v_scale, int kr, int vr) {
    constexpr int PER_WARP = 32 / LPV;
    const int t = blockIdx.x, lane = threadIdx.x & 31, part = lane & (LPV - 1), d0 = part * 4;
    const int head = (blockIdx.y * 4 + (threadIdx.x >> 5)) * PER_WARP + lane / LPV;
    const bool live = head < nh + 2 * nkv;                     // (dead lanes stay for the shuffles)
    const bool is_q = head < nh, is_k = !is_q && head < nh + nkv;
    const int g = is_q ? head : (is_k ? head - nh : head - nh - nkv);
    const int pos = tok_pos[t];
    TC *dst = nullptr, *cache = nullptr;                       // this head's row(s), and its row in the cache
    if (live) {
        if (is_q) dst = q_out + ((size_t)t * nh + g) * MAPS * kr;
        else if (is_k) dst = k_out ? k_out + ((size_t)t * nkv + g) * kr : nullptr;
        else dst = v_out ? v_out + ((size_t)t * nkv + g) * vr : nullptr;
        if (!is_q && k_pages != nullptr) {
            const int b = tok_seq[t], n = new_lens[b];
            int lp = pos / page_tokens;
            const int in_page = pos - lp * page_tokens;
            bool keep = pos < n;
            if (ring_pages > 0) {
                keep = keep && pos >= n - ring_pages * page_tokens;
                lp %= ring_pages;
            }
            if (keep) {
                const size_t row = ((size_t)block_table[(size_t)b * table_width + lp] * nkv + g) * page_tokens + in_page;
                cache = is_k ? k_pages + row * kr : v_pages + row * vr;
            }
        }
    }
    const int half = rot >> 1;
    const bool mine = live && (is_q || is_k) && d0 < hd, turns = mine && d0 < rot, low = d0 < half;
    float w[4] = {1.f, 1.f, 1.f, 1.f}, cs[4] = {1.f, 1.f, 1.f, 1.f}, sn[4] = {0.f, 0.f, 0.f, 0.f};
    if (mine) {                                                // weights and tables do not depend on the kernel before
        const float* ww = is_q ? q_w : k_w;
        if (ww) load16_f32<float>(ww + d0, w);
        if (turns) {
            const int j = low ? d0 : d0 - half;
            load16_f32<float>(cos_tab + (size_t)pos * half + j, cs);
            load16_f32<float>(sin_tab + (size_t)pos * half + j, sn);
#pragma unroll
            for (int e = 0; e < 4; ++e) sn[e] = low ? -sn[e] : sn[e];
        }
    }
    pdl_wait();
    pdl_launch();
    const float* src = proj + (size_t)t * ld;
    const float none[4] = {0.f, 0.f, 0.f, 0.f};
    if (live && !is_q && !is_k) {                              // values: copied, zeros behind
        for (int d = d0; d < vr; d += 4 * LPV) {
            float x[4] = {0.f, 0.f, 0.f, 0.f};
            if (d < vd) load16_f32<float>(src + v_col + g * vd + d, x);
#pragma unroll
            for (int e = 0; e < 4; ++e) x[e] *= v_scale;
            if (dst) he_store4<TC>(dst + d, x);
            if (cache) he_store4<TC>(cache + d, x);
        }
    }
    float x[MAPS][4];
#pragma unroll
    for (int m = 0; m < MAPS; ++m) {
        x[m][0] = x[m][1] = x[m][2] = x[m][3] = 0.f;
        if (mine) load16_f32<float>(src + (is_q ? q_col : k_col) + (g * MAPS + m) * hd + d0, x[m]);
    }
    // entry i < half pairs with entry i + half, half / 4 lanes on
    const int from = (lane & ~(LPV - 1)) + ((low ? part + (half >> 2) : part - (half >> 2)) & (LPV - 1));
#pragma unroll
    for (int m = 0; m < MAPS; ++m) {
        float inv = 1.f;
        if (norm_eps > 0.f) {
            float ss = fmaf(x[m][0], x[m][0], fmaf(x[m][1], x[m][1], fmaf(x[m][2], x[m][2], x[m][3] * x[m][3])));
#pragma unroll
            for (int o = LPV / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            inv = 1.f / sqrtf(ss / (float)hd + norm_eps);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) x[m][e] = x[m][e] * inv * w[e];
        if (half > 0) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float y = __shfl_sync(0xffffffffu, x[m][e], from);
                if (turns) x[m][e] = x[m][e] * cs[e] + y * sn[e];
            }
        }
        if (mine) {
            if (dst) he_store4<TC>(dst + (is_q ? m * kr : 0) + m * hd + d0, x[m]);
            if (cache) he_store4<TC>(cache + m * hd + d0, x[m]);
        }
    }
    if (!live || !(is_q || is_k)) return;
    // zeros: around each map's query, behind a key row's last map
    if (is_q) {
#pragma unroll
        for (int m = 0; m < MAPS; ++m)
            for (int d = d0; d < kr; d += 4 * LPV)
                if (d < m * hd || d >= m * hd + hd) he_store4<TC>(dst + m * kr + d, none);
    } else {
        for (int d = MAPS * hd + d0; d < kr; d += 4 * LPV) {
            if (dst) he_store4<TC>(dst + d, none);
            if (cache) he_store4<TC>(cache + d, none);
        }
    }
}

TQ_API int tq_head_encode(const float* proj, int ld, int q_col, int k_col, int v_col, const float* cos_tab,
                          const float* sin_tab, int rot, float norm_eps, const int* tok_pos, const int* tok_seq,
                          const int* new_lens, const int* block_table, int table_width, int ring_pages,
                          int page_tokens, void* q_out, void* k_out, void* v_out, void* k_pages, void* v_pages,
                          int cache_dtype, int n_tokens, int nh, int nkv, int hd, int vd, const float* row_inv,
                          const float* q_w, const float* k_w, int paired, float v_scale, int maps, int kr, int vr,
                          cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (maps < 1 || kr < maps * hd || vr < vd) return (int)cudaErrorInvalidValue;
    if ((maps > 1 || kr != hd || vr != vd) && (row_inv || v_col < 0)) return (int)cudaErrorInvalidValue;
    if (row_inv && (!q_w || (nkv > 0 && !k_w) || norm_eps > 0.f)) return (int)cudaErrorInvalidValue;
    if ((q_w || k_w) && !row_inv && !(norm_eps > 0.f)) return (int)cudaErrorInvalidValue;
    if (rot < 0 || rot > hd || (rot & 1) || page_tokens <= 0 || hd <= 0 || vd <= 0) return (int)cudaErrorInvalidValue;
    if (rot > 0 && (!cos_tab || !sin_tab)) return (int)cudaErrorInvalidValue;
    if ((k_pages == nullptr) != (v_pages == nullptr)) return (int)cudaErrorInvalidValue;
    if (k_pages && !block_table) return (int)cudaErrorInvalidValue;
    if (nkv > 0 && v_col < 0 && vd != hd) return (int)cudaErrorInvalidValue;
    const int vectors = nh * maps + nkv * maps + nkv;
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    if (!row_inv && !paired && v_col >= 0 && maps <= 2 && hd <= 128 &&
        !((hd | (rot >> 1) | vd | kr | vr | ld | q_col | k_col | v_col) & 3) && aligned(proj) && aligned(q_out) &&
        aligned(k_out) && aligned(v_out) && aligned(k_pages) && aligned(v_pages) && aligned(cos_tab) && aligned(sin_tab) &&
        aligned(q_w) && aligned(k_w)) {
        const int lpv = hd <= 32 ? 8 : (hd <= 64 ? 16 : 32), per_block = 4 * (32 / lpv);
        const int blocks = (nh + 2 * nkv + per_block - 1) / per_block;
        if (blocks > 65535) return (int)cudaErrorInvalidValue;
#define TQ_LAUNCH4(TC, L, M)                                                                                            \
    return tq_launch_pdl(TQ_PDL_ELEMENTWISE, head_encode4_kernel<TC, L, M>, dim3(n_tokens, blocks), dim3(128), 0, stream, \
                         proj, ld, q_col, k_col, v_col, cos_tab, sin_tab, rot, norm_eps, tok_pos, tok_seq, new_lens,     \
                         block_table, table_width, ring_pages, page_tokens, (TC*)q_out, (TC*)k_out, (TC*)v_out,          \
                         (TC*)k_pages, (TC*)v_pages, nh, nkv, hd, vd, q_w, k_w, v_scale, kr, vr)
#define TQ_LAUNCH4_SIZES(TC, M)                                                                                         \
    do {                                                                                                                \
        if (lpv == 8) TQ_LAUNCH4(TC, 8, M);                                                                             \
        if (lpv == 16) TQ_LAUNCH4(TC, 16, M);                                                                           \
        TQ_LAUNCH4(TC, 32, M);                                                                                          \
    } while (0)
        if (cache_dtype == TQ_F32 && maps == 1) TQ_LAUNCH4_SIZES(float, 1);
        if (cache_dtype == TQ_F32) TQ_LAUNCH4_SIZES(float, 2);
        if (cache_dtype == TQ_BF16 && maps == 1) TQ_LAUNCH4_SIZES(bf16, 1);
        if (cache_dtype == TQ_BF16) TQ_LAUNCH4_SIZES(bf16, 2);
#undef TQ_LAUNCH4_SIZES
#undef TQ_LAUNCH4
        return (int)cudaErrorInvalidValue;
    }
    const int groups = (vectors + 3) / 4;
    if (groups > 65535) return (int)cudaErrorInvalidValue;
    const dim3 grid(n_tokens, groups);
#define TQ_LAUNCH(TC)                                                                                              \
    return tq_launch_pdl(TQ_PDL_ELEMENTWISE, head_encode_kernel<TC>, grid, dim3(128), 0, stream, proj, ld, q_col,  \
                         k_col, v_col, cos_tab, sin_tab, rot, norm_eps, tok_pos, tok_seq, new_lens, block_table,   \
                         table_width, ring_pages, page_tokens, (TC*)q_out, (TC*)k_out, (TC*)v_out, (TC*)k_pages,   \
                         (TC*)v_pages, nh, nkv, hd, vd, row_inv, q_w, k_w, paired, v_scale, maps, kr, vr)
    if (cache_dtype == TQ_F32) TQ_LAUNCH(float);
    if (cache_dtype == TQ_BF16) TQ_LAUNCH(bf16);
#undef TQ_LAUNCH
    return (int)cudaErrorInvalidValue;
}

// ---------------------------------------------------------------------------
// out[t, 0] = 1 / sqrt(sum(q row^2) / q_count + eps), out[t, 1] likewise for the k row (k_n == 0: no k row): the
// factors of an RMS norm over a token's whole q and k projections.  The counts are the rows' true lengths where
// the rows are padded with zeros.
// ---------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
row_inv_rms_kernel(const float* __restrict__ proj, int ld, int q_col, int q_n, int q_count, int k_col, int k_n,
                   int k_count, float eps, float* __restrict__ out) {
    __shared__ float red[32];
    const int t = blockIdx.x;
    pdl_wait();
    pdl_launch();
    const float* row = proj + (size_t)t * ld;
    float ss = 0.f;
    for (int i = threadIdx.x; i < q_n; i += blockDim.x) ss = fmaf(row[q_col + i], row[q_col + i], ss);
    ss = block_sum(ss, red);
    if (threadIdx.x == 0) out[2 * t] = 1.f / sqrtf(ss / (float)q_count + eps);
    if (k_n <= 0) return;
    ss = 0.f;
    for (int i = threadIdx.x; i < k_n; i += blockDim.x) ss = fmaf(row[k_col + i], row[k_col + i], ss);
    ss = block_sum(ss, red);
    if (threadIdx.x == 0) out[2 * t + 1] = 1.f / sqrtf(ss / (float)k_count + eps);
}

TQ_API int tq_row_inv_rms(const float* proj, int ld, int q_col, int q_n, int q_count, int k_col, int k_n, int k_count,
                          float eps, float* out, int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (!proj || !out || q_n <= 0 || q_count <= 0 || k_n < 0 || (k_n > 0 && k_count <= 0)) return (int)cudaErrorInvalidValue;
    return tq_launch_pdl(TQ_PDL_ELEMENTWISE, row_inv_rms_kernel, dim3(n_tokens), dim3(q_n >= 1024 ? 256 : 128), 0, stream,
                         proj, ld, q_col, q_n, q_count, k_col, k_n, k_count, eps, out);
}

// ---------------------------------------------------------------------------
// The difference of two attention maps per head: with a1, a2 the maps' results (rows of `row` float32 entries, map m
// of head h at row h * 2 + m of a token), o = a1 - factor * a2, then o / sqrt(mean(o^2) + eps) over the head's e
// entries, times out_scale, times sigmoid(gate[t, h]) if there is one; rounded once.  With `ml` the rows are the
// unnormalised sums over n_splits shares of the keys with their maxima and sums of weights (natural-log units), which
// are merged here in index order, as attention_merge_kernel does.  A warp per (token, head).
// ---------------------------------------------------------------------------
// V: entries a lane takes at a time (4: rows and heads of whole 16-byte pieces; 1: any), PER: how often.
template <typename TO, int V, int PER>
__global__ void __launch_bounds__(128)
difference_of_maps_kernel(const float* __restrict__ a, const float* __restrict__ ml, int n_splits, int row, int e, int H,
                          float factor, float eps, float out_scale, const float* __restrict__ gate, int ldg,
                          TO* __restrict__ out, int n_pairs) {
    const int pair = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (pair >= n_pairs) return;
    const int t = pair / H, h = pair - t * H;
    pdl_wait();
    pdl_launch();
    float o[PER][V];
#pragma unroll
    for (int i = 0; i < PER; ++i)
#pragma unroll
        for (int c = 0; c < V; ++c) o[i][c] = 0.f;
    auto add = [&](const float* src, float f) {                        // o += f * src
        float v[PER][V];
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int d = V * (lane + 32 * i);
#pragma unroll
            for (int c = 0; c < V; ++c) v[i][c] = 0.f;
            if (d < e) {
                if constexpr (V == 4) load16_f32<float>(src + d, v[i]);
                else v[i][0] = src[d];
            }
        }
#pragma unroll
        for (int i = 0; i < PER; ++i)
#pragma unroll
            for (int c = 0; c < V; ++c) o[i][c] = fmaf(f, v[i][c], o[i][c]);
    };
    const float* r0 = a + (size_t)pair * 2 * n_splits * row;           // [2 maps][n_splits][row]
    if (!ml) {
        add(r0, 1.f);
        add(r0 + row, -factor);
    } else {
        for (int m = 0; m < 2; ++m) {
            const float* mls = ml + ((size_t)pair * 2 + m) * n_splits * 2;
            const float* acc = r0 + (size_t)m * n_splits * row;
            float mx = -INFINITY;
            for (int s = lane; s < n_splits; s += 32) mx = fmaxf(mx, mls[2 * s]);
            mx = warp_max(mx);
            float l = 0.f;
            for (int s = lane; s < n_splits; s += 32)
                if (mls[2 * s] > -INFINITY) l += mls[2 * s + 1] * expf(mls[2 * s] - mx);
            l = warp_sum(l);
            const float sign = (m ? -factor : 1.f) / l;
            for (int s = 0; s < n_splits; ++s) {
                const float ms = mls[2 * s];
                if (ms > -INFINITY) add(acc + (size_t)s * row, expf(ms - mx) * sign);    // (an empty share holds nothing)
            }
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i)
#pragma unroll
        for (int c = 0; c < V; ++c) ss = fmaf(o[i][c], o[i][c], ss);
    ss = warp_sum(ss);
    float f = out_scale / sqrtf(ss / (float)e + eps);
    if (gate) f *= 1.f / (1.f + expf(-gate[(size_t)t * ldg + h]));
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int d = V * (lane + 32 * i);
        if (d < e) {
#pragma unroll
            for (int c = 0; c < V; ++c) o[i][c] *= f;
            if constexpr (V == 4) he_store4<TO>(out + (size_t)pair * e + d, o[i]);
            else out[(size_t)pair * e + d] = from_f32<TO>(o[i][0]);
        }
    }
}

TQ_API int tq_difference_of_maps(const float* a, const float* ml, int n_splits, int row, int e, int heads, float factor,
                                 float eps, float out_scale, const float* gate, int ldg, void* out, int dtype,
                                 int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (!a || !out || n_splits < 1 || (!ml && n_splits != 1) || e <= 0 || e > 512 || row < e || heads <= 0)
        return (int)cudaErrorInvalidValue;
    if ((long long)n_tokens * heads > 0x7fffffffll - 4) return (int)cudaErrorInvalidValue;
    const int n_pairs = n_tokens * heads;
    const dim3 grid((n_pairs + 3) / 4);
    const bool vec = !((e | row) & 3) && ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
#define TQ_DM(TO, V, PER)                                                                                               \
    return tq_launch_pdl(TQ_PDL_ELEMENTWISE, difference_of_maps_kernel<TO, V, PER>, grid, dim3(128), 0, stream, a, ml,    \
                         n_splits, row, e, heads, factor, eps, out_scale, gate, ldg, (TO*)out, n_pairs)
#define TQ_DM_SIZES(TO)                                                                                                 \
    do {                                                                                                                \
        if (vec && e <= 128) TQ_DM(TO, 4, 1);                                                                           \
        if (vec) TQ_DM(TO, 4, 4);                                                                                       \
        TQ_DM(TO, 1, 16);                                                                                               \
    } while (0)
    if (dtype == TQ_F32) TQ_DM_SIZES(float);
    if (dtype == TQ_BF16) TQ_DM_SIZES(bf16);
#undef TQ_DM_SIZES
#undef TQ_DM
    return (int)cudaErrorInvalidValue;
}

// ---------------------------------------------------------------------------
// x[t, i] *= sigmoid(gate[t * ldg + i / per]): a gate per entry (per = 1) on the heads side by side, or one per head of
// `per` entries.
// ---------------------------------------------------------------------------
template <typename TC>
__global__ void sigmoid_gate_kernel(TC* __restrict__ x, const float* __restrict__ gate, int ldg, int n, int per, size_t total) {
    pdl_wait();
    pdl_launch();
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (size_t)gridDim.x * blockDim.x) {
        const size_t t = idx / n;
        const int i = (int)(idx - t * n);
        const float g = gate[t * ldg + i / per];
        x[idx] = from_f32<TC>(to_f32<TC>(x[idx]) / (1.f + expf(-g)));
    }
}

TQ_API int tq_sigmoid_gate(void* x, int dtype, const float* gate, int ldg, int n_rows, int n, int per, cudaStream_t stream) {
    if (per < 1) return (int)cudaErrorInvalidValue;
    const size_t total = (size_t)n_rows * n;
    if (total == 0) return 0;
    const int threads = 256;
    size_t blocks = (total + threads - 1) / threads;
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == TQ_F32)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, sigmoid_gate_kernel<float>, dim3((unsigned)blocks), dim3(threads), 0,
                             stream, (float*)x, gate, ldg, n, per, total);
    if (dtype == TQ_BF16)
        return tq_launch_pdl(TQ_PDL_ELEMENTWISE, sigmoid_gate_kernel<bf16>, dim3((unsigned)blocks), dim3(threads), 0,
                             stream, (bf16*)x, gate, ldg, n, per, total);
    return (int)cudaErrorInvalidValue;
}

// ---------------------------------------------------------------------------
// x <- cap * tanh(x / cap), in place (float32).
// ---------------------------------------------------------------------------
__global__ void tanh_cap_kernel(float* __restrict__ x, size_t total, float cap) {
    pdl_wait();
    pdl_launch();
    const float inv = 1.f / cap;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (size_t)gridDim.x * blockDim.x)
        x[idx] = cap * tanhf(x[idx] * inv);
}

TQ_API int tq_tanh_cap(float* x, size_t total, float cap, cudaStream_t stream) {
    if (total == 0) return 0;
    if (!(cap > 0.f)) return (int)cudaErrorInvalidValue;
    size_t blocks = (total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    return tq_launch_pdl(TQ_PDL_ELEMENTWISE, tanh_cap_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, x, total, cap);
}
