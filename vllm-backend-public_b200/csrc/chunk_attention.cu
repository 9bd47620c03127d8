// chunk_attention.cu -- attention over a paged cache of keys and values per kv head, with parameters that designs set
// independently of each other:
//   * per-head RMS norm of queries and keys (a plain weight of size dk shared by the heads),
//   * a block-local causal mask: position i sees j <= i with floor(j / chunk) == floor(i / chunk), blocks counted from
//     position 0 of the sequence (chunk = 0: plain causal),
//   * a sink: `sink` is added to the softmax denominator as exp(sink_logit - max), a key with no value (sink = 0: none;
//     sink = 1 with logit 0 gives p_j = exp(s_j) / (1 + sum exp(s))); the logit may also be one learned number per
//     query head (sink_logits [H], not scaled),
//   * a sliding window that keeps the first tokens: position i sees j <= i with i - j < window or j < keep_first
//     (window = 0: no window).  A query then reads the kept keys and its window's keys and nothing between them,
//   * a sigmoid gate per (token, head) on the head's output,
//   * the weight of a visible key: its share of the softmax, or (B2_WEIGHT_SIGMOID) sigmoid(score + head_bias[h]), a number
//     of its own that no other key changes -- no maximum, no denominator, and a sink has no meaning,
//   * a cap on the scores: s <- cap * tanh(s / cap) before the mask and the softmax (cap = 0: none),
//   * two maps per head (differential attention): a head holds two queries and two keys of size dk, each pair of them is a
//     softmax attention of its own over the head's values, and the head's output is a1 - lambda * a2, divided by its own root
//     mean square over dv (eps inside the root) and multiplied by a constant.  The two maps of a head are neighbours in q
//     [T, H, maps, dk] and in the K pool; they are walked together, so a value row is read once for both.
// Key size dk and value size dv are independent; K and V live in separate paged pools
//   k_cache [num_blocks, G * maps, bs, dk],  v_cache [num_blocks, G, bs, dv]      (activation type).
//
//   b2_qknorm_cache      per token: q heads normalised into q_out; k heads normalised and written to the K pool, v copied
//                        to the V pool, through the token's slot (slot < 0 skips the write).
//   b2_qk_prep_cache     the same pass with the norm optional and a query temperature: the query of the token at position p
//                        is multiplied by 1 + coef * ln(floor((p + 1) / every) + 1) (fp32), so queries sharpen as the
//                        context grows in steps of `every` positions (coef = 0: none).
//   b2_qk_rope_cache     rows [q | k] or [q | k | v]: the first rot_dims entries of every q and k head are rotated by the
//                        token's position (pairs (i, i + rot_dims/2) or (2i, 2i + 1); fp32 table [max_pos, rot_dims] =
//                        cos | sin halves), q to q_out, rotated k to the K pool; the V pool receives v, or, for designs
//                        whose values ARE the keys, the k heads as projected (before the rotation).  The value heads may be
//                        fewer than the key heads (two key maps over one set of values).
//   b2_qk_norm_rope_cache  rows [q | k | v]: all of q (H * dk numbers) and all of k (G * dk) are RMS-normed as one row each,
//                        before the split into heads (fp32 weights of those sizes), then rotated and written as above; the
//                        numbers stay in fp32 between the norm and the rotation.
//   b2_chunk_attention   four kernels: prompt rows of bf16 models on mma.sync tiles of 64 rows; decode rows and short portions
//                        of bf16 models on mma.sync with a kv head's query heads as operand rows, or (head sizes the tensor
//                        cores do not take) one CTA per (row, kv head) on fp32 FMAs; fp32 and odd sizes one warp per
//                        (token, head).  Scores, softmax state and accumulators are fp32 in all of them.  With a mask a query
//                        touches only the keys it sees, wherever it stands; a decode row is a sequence with one query.
// Sequences are described like everywhere in this library: rows cu_q[i] .. cu_q[i+1]-1, ctx_start[i] cached tokens
// before them (< 0: padding, output rows are zeroed), block_tables[i, :].
#include "b2_act.cuh"

namespace {

constexpr int kMaxDvPerLane = 16;                    // dv <= 512

// The keys a query at position `pos` may see, as one compact index range [0, n): first the kept keys lo .. lo+nfirst-1
// (the sequence's first tokens that lie before the window), then wlo .. pos.  Without a window nfirst = 0 and wlo = lo.
struct KeySpan {
    int lo, nfirst, wlo, n;
    __device__ __forceinline__ int key(int c) const { return c < nfirst ? lo + c : wlo + (c - nfirst); }
};
__device__ __forceinline__ KeySpan key_span(int pos, int last, int chunk, int window, int keep_first) {
    KeySpan s;
    s.lo = chunk > 0 ? (pos / chunk) * chunk : 0;
    s.wlo = window > 0 ? max(s.lo, pos - window + 1) : s.lo;
    s.nfirst = (window > 0 && keep_first > s.lo) ? max(0, min(keep_first, s.wlo) - s.lo) : 0;
    s.n = s.nfirst + (last - s.wlo + 1);
    return s;
}
// what the masks leave of key j for the query at position i
__device__ __forceinline__ bool key_visible(int i, int j, int lo_i, int window, int keep_first) {
    return j <= i && j >= lo_i && (window <= 0 || i - j < window || j < keep_first);
}

// 1 / rms of all H * dk numbers of q and of all G * dk of k, which lie one after the other at `src` (block-wide)
template <typename T, int W>
__device__ __forceinline__ void qk_row_scales(const T* src, int nq, int nk, float eps, float* red, float& inv_q, float& inv_k) {
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x * W; i < nq + nk; i += blockDim.x * W) {
        float v[4] = {0.f, 0.f, 0.f, 0.f}, ss = 0.f;
        if (W == 4) b2::ld4(src + i, v); else v[0] = b2::ld(src + i);
#pragma unroll
        for (int c = 0; c < W; ++c) ss = fmaf(v[c], v[c], ss);
        if (i < nq) sq += ss; else sk += ss;
    }
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    sq = b2::warp_sum(sq);
    sk = b2::warp_sum(sk);
    if (lane == 0) {
        red[2 * wid] = sq;
        red[2 * wid + 1] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
    for (int x = 0; x < nw; ++x) {                   // at most eight warps: every thread adds them up itself
        sq += red[2 * x];
        sk += red[2 * x + 1];
    }
    inv_q = rsqrtf(sq / (float)nq + eps);
    inv_k = rsqrtf(sk / (float)nk + eps);
}

// Rows [q | k] (+ [v]): partial rotation of the q and k heads, K (rotated) and V pool writes; see the file comment.  NORM:
// q and k are first normed over their whole rows.
template <typename T, bool NORM>
__global__ void qk_rope_cache_kernel(const T* __restrict__ qkv, int64_t qkv_stride, int H, int G, int Gv, int dk, int dv, bool v_from_k,
                                     int rot_dims, bool interleaved, const int32_t* __restrict__ positions,
                                     const float* __restrict__ cos_sin, int max_pos, const int64_t* __restrict__ slots, int bs,
                                     const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                                     T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache) {
    __shared__ float red[16];
    const int row = blockIdx.x;
    const T* src = qkv + (size_t)row * qkv_stride;
    float inv_q = 1.f, inv_k = 1.f;
    if (NORM) qk_row_scales<T, 1>(src, H * dk, G * dk, eps, red, inv_q, inv_k);
    int pos = positions[row];
    pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
    const float* cs = cos_sin + (size_t)pos * rot_dims;
    const int half = rot_dims / 2;
    const int64_t slot = slots[row];
    const int64_t blk = slot >= 0 ? slot / bs : 0;
    const int off = slot >= 0 ? (int)(slot % bs) : 0;
    // q and k heads: element i of a head
    for (int idx = threadIdx.x; idx < (H + G) * dk; idx += blockDim.x) {
        const int hd = idx / dk, i = idx % dk;
        if (hd >= H && slot < 0) continue;
        const T* v = src + (size_t)hd * dk;
        const float* w = NORM ? (hd < H ? q_w + (size_t)hd * dk : k_w + (size_t)(hd - H) * dk) : nullptr;
        const float inv = hd < H ? inv_q : inv_k;
        float x = b2::ld(v + i);
        if (NORM) x *= inv * w[i];
        if (i < rot_dims) {
            int pr, partner;
            bool second;
            if (interleaved) { pr = i >> 1; partner = i ^ 1; second = i & 1; }
            else { second = i >= half; pr = second ? i - half : i; partner = second ? i - half : i + half; }
            const float c = cs[pr], sn = cs[half + pr], other = b2::ld(v + partner) * (NORM ? inv * w[partner] : 1.f);
            x = second ? fmaf(x, c, other * sn) : fmaf(x, c, -other * sn);
        }
        T* dst = hd < H ? q_out + ((size_t)row * H + hd) * dk : k_cache + (((size_t)blk * G + (hd - H)) * bs + off) * dk;
        b2::st(dst + i, x);
    }
    if (slot < 0) return;
    const T* vsrc = v_from_k ? src + (size_t)H * dk : src + (size_t)(H + G) * dk;
    for (int idx = threadIdx.x; idx < Gv * dv; idx += blockDim.x) {
        const int g = idx / dv, i = idx % dv;
        v_cache[(((size_t)blk * Gv + g) * bs + off) * dv + i] = vsrc[idx];
    }
}

// The same with four entries per access (8 or 16 bytes): every size a multiple of four, the rotated entries a multiple of
// eight in the (i, i + rot_dims/2) layout so that a group of four and its partners never straddle the halves.
template <typename T, bool NORM>
__global__ void __launch_bounds__(256)
qk_rope_cache_vec_kernel(const T* __restrict__ qkv, int64_t qkv_stride, int H, int G, int Gv, int dk, int dv, bool v_from_k, int rot_dims,
                         bool interleaved, const int32_t* __restrict__ positions, const float* __restrict__ cos_sin, int max_pos,
                         const int64_t* __restrict__ slots, int bs, const float* __restrict__ q_w, const float* __restrict__ k_w,
                         float eps, T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache) {
    __shared__ float red[16];
    const int row = blockIdx.x;
    const T* src = qkv + (size_t)row * qkv_stride;
    float inv_q = 1.f, inv_k = 1.f;
    if (NORM) qk_row_scales<T, 4>(src, H * dk, G * dk, eps, red, inv_q, inv_k);
    int pos = positions[row];
    pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
    const float* cs = cos_sin + (size_t)pos * rot_dims;
    const int half = rot_dims / 2;
    const int64_t slot = slots[row];
    const int64_t blk = slot >= 0 ? slot / bs : 0;
    const int off = slot >= 0 ? (int)(slot % bs) : 0;
    const int per = dk / 4, nqk = (slot >= 0 ? H + G : H) * per;
    for (int idx = threadIdx.x; idx < nqk; idx += blockDim.x) {
        const int hd = idx / per, i = (idx % per) * 4;
        const T* v = src + (size_t)hd * dk;
        const float* w = NORM ? (hd < H ? q_w + (size_t)hd * dk : k_w + (size_t)(hd - H) * dk) : nullptr;
        const float inv = hd < H ? inv_q : inv_k;
        float x[4];
        b2::ld4(v + i, x);
        if (NORM) {
#pragma unroll
            for (int c = 0; c < 4; ++c) x[c] *= inv * w[i + c];
        }
        if (i < rot_dims) {
            if (interleaved) {
#pragma unroll
                for (int c = 0; c < 4; c += 2) {
                    const float co = cs[(i + c) >> 1], si = cs[half + ((i + c) >> 1)], a = x[c], b = x[c + 1];
                    x[c] = fmaf(a, co, -b * si);
                    x[c + 1] = fmaf(b, co, a * si);
                }
            } else {
                const bool second = i >= half;
                const int pr = second ? i - half : i;
                const int pi = second ? i - half : i + half;
                float y[4];
                b2::ld4(v + pi, y);
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    if (NORM) y[c] *= inv * w[pi + c];
                    const float co = cs[pr + c], si = cs[half + pr + c];
                    x[c] = second ? fmaf(x[c], co, y[c] * si) : fmaf(x[c], co, -y[c] * si);
                }
            }
        }
        T* dst = hd < H ? q_out + ((size_t)row * H + hd) * dk : k_cache + (((size_t)blk * G + (hd - H)) * bs + off) * dk;
        b2::st4(dst + i, x);
    }
    if (slot < 0) return;
    const T* vsrc = v_from_k ? src + (size_t)H * dk : src + (size_t)(H + G) * dk;
    const int pv = dv / 4;
    for (int idx = threadIdx.x; idx < Gv * pv; idx += blockDim.x) {
        const int g = idx / pv, i = (idx % pv) * 4;
        float x[4];
        b2::ld4(vsrc + (size_t)g * dv + i, x);
        b2::st4(v_cache + (((size_t)blk * Gv + g) * bs + off) * dv + i, x);
    }
}

template <typename T>
__global__ void qknorm_cache_kernel(const T* __restrict__ qkv, int64_t qkv_stride, int H, int G, int dk, int dv,
                                    const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                                    const int64_t* __restrict__ slots, int bs, T* __restrict__ q_out,
                                    T* __restrict__ k_cache, T* __restrict__ v_cache, bool norm,
                                    const int32_t* __restrict__ positions, float temp_coef, int temp_every) {
    const int row = blockIdx.x;
    float q_factor = 1.f;
    if (positions && temp_coef != 0.f) q_factor = 1.f + temp_coef * logf((float)((positions[row] + 1) / temp_every + 1));
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const T* src = qkv + (size_t)row * qkv_stride;
    const int64_t slot = slots[row];
    const int64_t blk = slot >= 0 ? slot / bs : 0;
    const int off = slot >= 0 ? (int)(slot % bs) : 0;
    for (int hd = wid; hd < H + 2 * G; hd += nw) {
        if (hd < H + G) {                            // q or k head: x / sqrt(mean(x^2) + eps) * w
            const T* v = src + (size_t)hd * dk;
            float inv = hd < H ? q_factor : 1.f;
            if (norm) {
                float ss = 0.f;
                for (int i = lane; i < dk; i += 32) {
                    const float x = b2::ld(v + i);
                    ss = fmaf(x, x, ss);
                }
                inv = rsqrtf(b2::warp_sum(ss) / (float)dk + eps) * (hd < H ? q_factor : 1.f);
            }
            T* dst;
            const float* w;
            if (hd < H) {
                dst = q_out + ((size_t)row * H + hd) * dk;
                w = q_w;
            } else {
                if (slot < 0) continue;
                dst = k_cache + (((size_t)blk * G + (hd - H)) * bs + off) * dk;
                w = k_w;
            }
            for (int i = lane; i < dk; i += 32) b2::st(dst + i, b2::ld(v + i) * inv * (w ? w[i] : 1.f));
        } else {
            if (slot < 0) continue;
            const int g = hd - H - G;
            const T* v = src + (size_t)(H + G) * dk + (size_t)g * dv;
            T* dst = v_cache + (((size_t)blk * G + g) * bs + off) * dv;
            for (int i = lane; i < dv; i += 32) dst[i] = v[i];
        }
    }
}

// sigmoid of a score that is already in the exponent of 2
__device__ __forceinline__ float sigmoid2_f(float x2) { return __fdividef(1.f, 1.f + b2::fast_exp2(-x2)); }

// What happens to a score before its weight is taken, and to a head's output after the values are summed.
struct HeadShape {
    float cap;               // > 0: scores become cap * tanh(score / cap)
    float lambda;            // two maps: output = a1 - lambda * a2 ...
    float eps, out_scale;    // ... / sqrt(mean(output^2) + eps) * out_scale
};
// cap * tanh(s / cap); tanh x = 1 - 2 / (1 + e^2x), whose absolute error (times cap) is that of one fp32 rounding
__device__ __forceinline__ float cap_score(float s, float cap, float e_scale) {
    return fmaf(-cap, __fdividef(2.f, 1.f + b2::fast_exp2(s * e_scale)), cap);
}
__device__ __forceinline__ float cap_score_exact(float s, float cap) { return cap * tanhf(s / cap); }

template <typename T, bool SIG, int MAPS>
__global__ void chunk_attention_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                                       const int32_t* __restrict__ block_tables, int max_nb,
                                       const int32_t* __restrict__ cu_q, const int32_t* __restrict__ ctx_start, int n_seq,
                                       int rows, int H, int G, int dk, int dv, int bs, float scale, int chunk, int window,
                                       int keep_first, float sink, float sink_logit, const float* __restrict__ sink_logits,
                                       const float* __restrict__ head_bias, const T* __restrict__ gate, int64_t gate_stride,
                                       HeadShape hs, int skip_rows_from, T* __restrict__ out, int64_t out_stride) {
    extern __shared__ float q_sm[];                  // [warps, dk]
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
    const int item = blockIdx.x * (blockDim.x >> 5) + wid;       // (row, head)
    if (item >= rows * H) return;
    const int row = item / H, hh = item % H;
    const int seq = b2::seq_of_row(cu_q, n_seq, row);
    const int ctx = ctx_start[seq];
    T* dst = out + (size_t)row * out_stride + (size_t)hh * dv;
    if (skip_rows_from > 0 && ctx >= 0 && cu_q[seq + 1] - cu_q[seq] >= skip_rows_from) return;    // the tile kernel's
    if (ctx < 0) {
        for (int i = lane; i < dv; i += 32) b2::st(dst + i, 0.f);
        return;
    }
    const int pos = ctx + row - cu_q[seq];
    const KeySpan span = key_span(pos, pos, chunk, window, keep_first);
    const int g = hh / (H / G);
    float* qs = q_sm + (size_t)wid * dk;
    const int32_t* bt = block_tables + (size_t)seq * max_nb;
    const float bias = SIG && head_bias ? head_bias[hh] : 0.f;
    float first[MAPS > 1 ? kMaxDvPerLane : 1];       // the first map's output
    float acc[kMaxDvPerLane];
    float inv = 1.f;
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
        const T* qv = q + ((size_t)item * MAPS + mp) * dk;
        __syncwarp();
        for (int i = lane; i < dk; i += 32) qs[i] = b2::ld(qv + i) * scale;
        __syncwarp();
        float m = sink > 0.f ? (sink_logits ? sink_logits[hh] : sink_logit) : -INFINITY, l = sink;      // the sink seeds the running maximum and denominator
#pragma unroll
        for (int c = 0; c < kMaxDvPerLane; ++c) acc[c] = 0.f;
        for (int c0 = 0; c0 < span.n; c0 += 32) {
            const bool in = c0 + lane < span.n;
            const int j = span.key(c0 + lane);
            float s = -INFINITY;
            size_t vbase = 0;
            if (in) {
                const size_t page = bt[j / bs];
                const T* kr = k_cache + ((page * (G * MAPS) + g * MAPS + mp) * bs + (j % bs)) * dk;
                vbase = ((page * G + g) * bs + (j % bs)) * dv;
                float d = 0.f;
                for (int i = 0; i < dk; ++i) d = fmaf(qs[i], b2::ld(kr + i), d);
                s = hs.cap > 0.f ? cap_score_exact(d, hs.cap) : d;
            }
            float p;
            if (SIG) {
                p = in ? b2::sigmoid_f(s + bias) : 0.f;
            } else {
                const float m_new = fmaxf(m, b2::warp_max(s));
                const float corr = m == -INFINITY ? 0.f : __expf(m - m_new);
                p = in ? __expf(s - m_new) : 0.f;
                l = l * corr + b2::warp_sum(p);
                m = m_new;
#pragma unroll
                for (int c = 0; c < kMaxDvPerLane; ++c) acc[c] *= corr;
            }
            const int nk = min(32, span.n - c0);
            for (int kk = 0; kk < nk; ++kk) {
                const float pk = __shfl_sync(0xffffffffu, p, kk);
                const size_t vb = __shfl_sync(0xffffffffu, (unsigned long long)vbase, kk);
                const T* vr = v_cache + vb;
#pragma unroll
                for (int c = 0; c < kMaxDvPerLane; ++c) {
                    const int i = lane + 32 * c;
                    if (i < dv) acc[c] = fmaf(pk, b2::ld(vr + i), acc[c]);
                }
            }
        }
        inv = SIG ? 1.f : (l > 0.f ? 1.f / l : 0.f);
        if (MAPS > 1 && mp == 0) {
#pragma unroll
            for (int c = 0; c < kMaxDvPerLane; ++c) first[MAPS > 1 ? c : 0] = acc[c] * inv;
        }
    }
    if (MAPS > 1) {
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < kMaxDvPerLane; ++c) {
            acc[c] = first[MAPS > 1 ? c : 0] - hs.lambda * (acc[c] * inv);
            ss = fmaf(acc[c], acc[c], ss);           // columns past dv hold zeros
        }
        inv = rsqrtf(b2::warp_sum(ss) / (float)dv + hs.eps) * hs.out_scale;
    }
    if (gate) inv *= b2::sigmoid_f(b2::ld(gate + (size_t)row * gate_stride + hh));
#pragma unroll
    for (int c = 0; c < kMaxDvPerLane; ++c) {
        const int i = lane + 32 * c;
        if (i < dv) b2::st(dst + i, acc[c] * inv);
    }
}

// ------------------------------------------------------------------------------------------------- grouped decode kernel
// bf16 rows that neither tensor-core kernel takes (decode rows and short portions of other head sizes): one CTA per (row, kv head) serves ALL the
// query heads of that kv head, so K and V are read once per group instead of once per head.  Four warps share the visible
// keys 32 at a time (a lane per key, 16-byte loads of its K row, one dot product per query head), keep an online softmax
// per head, accumulate P.V with a lane per pair of value columns, and merge through shared memory; the sink enters
// through warp 0's initial state.  Up to kGroupMaxHeads query heads per pass (more: further passes over the keys).  With two
// maps the pass holds the heads' maps one after the other (an even number) and a key's two halves lie side by side in the tile.
constexpr int kGroupMaxHeads = 8, kGroupMaxPairs = 4;      // dv <= 256

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(b2::smem_u32(dst)), "l"(src) : "memory");
}

template <bool SIG, int MAPS>
__global__ void __launch_bounds__(128)
chunk_attention_group_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k_cache,
                             const __nv_bfloat16* __restrict__ v_cache, const int32_t* __restrict__ block_tables, int max_nb,
                             const int32_t* __restrict__ cu_q, const int32_t* __restrict__ ctx_start, int n_seq, int H, int G,
                             int dk, int dv, int bs, float scale, int chunk, int window, int keep_first, float sink,
                             float sink_logit, const float* __restrict__ sink_logits, const float* __restrict__ head_bias,
                             const __nv_bfloat16* __restrict__ gate, int64_t gate_stride, HeadShape hs, int skip_rows_from,
                             __nv_bfloat16* __restrict__ out, int64_t out_stride) {
    // q [QH][dk] | per warp: m [QH], l [QH], acc [QH][dv] | per warp: K tile [32][MAPS * dk + 8], V tile [32][dv] (bf16)
    extern __shared__ __align__(16) float grp_sm[];
    const int row = blockIdx.x, g = blockIdx.y;
    const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
    const int seq = b2::seq_of_row(cu_q, n_seq, row);
    const int ctx = ctx_start[seq];
    const int QHall = H / G;                               // query heads of this key head
    const int VHall = QHall * MAPS;                        // ... each with its maps
    if (skip_rows_from > 0 && ctx >= 0 && cu_q[seq + 1] - cu_q[seq] >= skip_rows_from) return;    // the tile kernel's
    if (ctx < 0) {
        for (int i = tid; i < QHall * dv; i += 128)
            out[(size_t)row * out_stride + (size_t)g * QHall * dv + i] = __float2bfloat16_rn(0.f);
        return;
    }
    const int pos = ctx + row - cu_q[seq];
    const KeySpan span = key_span(pos, pos, chunk, window, keep_first);
    const int32_t* bt = block_tables + (size_t)seq * max_nb;
    const int npairs = dv / 2;
    for (int h0 = 0; h0 < VHall; h0 += kGroupMaxHeads) {
        const int QH = min(kGroupMaxHeads, VHall - h0);
        float* qs = grp_sm;
        float* part = grp_sm + kGroupMaxHeads * dk;
        const int ldk = MAPS * dk + 8;                     // 16 bytes of padding: the lanes' rows spread over the banks
        __nv_bfloat16* kt = reinterpret_cast<__nv_bfloat16*>(part + 4 * kGroupMaxHeads * (2 + dv)) + (size_t)w * 32 * (ldk + dv);
        __nv_bfloat16* vt = kt + 32 * ldk;
        __syncthreads();                                   // a previous pass is done with the shared memory
        for (int i = tid; i < QH * dk; i += 128)
            qs[i] = __bfloat162float(q[((size_t)row * H * MAPS + (size_t)g * VHall + h0) * dk + i]) * scale;
        __syncthreads();
        float m[kGroupMaxHeads], l[kGroupMaxHeads], acc[kGroupMaxHeads][kGroupMaxPairs][2];
#pragma unroll
        for (int h = 0; h < kGroupMaxHeads; ++h) {
            m[h] = (w == 0 && sink > 0.f) ? (sink_logits ? sink_logits[g * QHall + (h0 + min(h, QH - 1)) / MAPS] : sink_logit) : -INFINITY;
            l[h] = w == 0 ? sink : 0.f;
            if (SIG) m[h] = head_bias ? head_bias[g * QHall + (h0 + min(h, QH - 1)) / MAPS] : 0.f;      // holds the head's bias instead
#pragma unroll
            for (int c = 0; c < kGroupMaxPairs; ++c) acc[h][c][0] = acc[h][c][1] = 0.f;
        }
        for (int c0 = w * 32; c0 < span.n; c0 += 128) {
            const bool valid = c0 + lane < span.n;
            float sc[kGroupMaxHeads];
#pragma unroll
            for (int h = 0; h < kGroupMaxHeads; ++h) sc[h] = 0.f;
            // the warp's 32 keys: K and V rows gathered from the pages with every 16-byte copy in flight at once
            const int nk = min(32, span.n - c0);
            __syncwarp();                                  // the previous tile has been read
            for (int idx = lane; idx < nk * MAPS * (dk / 8); idx += 32) {
                const int part_ = idx / (dk / 8), c = (idx % (dk / 8)) * 8, key = part_ / MAPS, mp = part_ % MAPS, jk = span.key(c0 + key);
                cp_async16(kt + key * ldk + mp * dk + c,
                           k_cache + (((size_t)bt[jk / bs] * (G * MAPS) + g * MAPS + mp) * bs + jk % bs) * dk + c);
            }
            for (int idx = lane; idx < nk * (dv / 8); idx += 32) {
                const int key = idx / (dv / 8), c = (idx % (dv / 8)) * 8, jk = span.key(c0 + key);
                cp_async16(vt + key * dv + c, v_cache + (((size_t)bt[jk / bs] * G + g) * bs + jk % bs) * dv + c);
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncwarp();
            if (valid) {
#pragma unroll
                for (int mp = 0; mp < MAPS; ++mp) {
                    const __nv_bfloat16* kr = kt + lane * ldk + mp * dk;
                    for (int c = 0; c < dk; c += 8) {
                        const uint4 raw = *reinterpret_cast<const uint4*>(kr + c);
                        const uint32_t wds[4] = {raw.x, raw.y, raw.z, raw.w};
                        float kf[8];
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            kf[2 * e] = __uint_as_float(wds[e] << 16);
                            kf[2 * e + 1] = __uint_as_float(wds[e] & 0xffff0000u);
                        }
#pragma unroll
                        for (int h = mp; h < kGroupMaxHeads; h += MAPS) {
                            if (h < QH) {
                                const float4 qa = *reinterpret_cast<const float4*>(qs + h * dk + c);
                                const float4 qb = *reinterpret_cast<const float4*>(qs + h * dk + c + 4);
                                sc[h] = fmaf(qa.x, kf[0], sc[h]); sc[h] = fmaf(qa.y, kf[1], sc[h]);
                                sc[h] = fmaf(qa.z, kf[2], sc[h]); sc[h] = fmaf(qa.w, kf[3], sc[h]);
                                sc[h] = fmaf(qb.x, kf[4], sc[h]); sc[h] = fmaf(qb.y, kf[5], sc[h]);
                                sc[h] = fmaf(qb.z, kf[6], sc[h]); sc[h] = fmaf(qb.w, kf[7], sc[h]);
                            }
                        }
                    }
                }
                if (hs.cap > 0.f) {
                    const float e_scale = 2.8853900817779268f / hs.cap;         // 2 log2(e) / cap
#pragma unroll
                    for (int h = 0; h < kGroupMaxHeads; ++h) sc[h] = cap_score(sc[h], hs.cap, e_scale);
                }
            }
            float pr[kGroupMaxHeads];
#pragma unroll
            for (int h = 0; h < kGroupMaxHeads; ++h) {
                pr[h] = 0.f;
                if (SIG) {
                    if (h < QH && valid) pr[h] = b2::sigmoid_f(sc[h] + m[h]);
                } else if (h < QH) {
                    const float x = valid ? sc[h] : -INFINITY;
                    const float mn = fmaxf(m[h], b2::warp_max(x));          // finite: the tile has at least one key
                    const float corr = m[h] == -INFINITY ? 0.f : __expf(m[h] - mn);
                    pr[h] = valid ? __expf(x - mn) : 0.f;
                    l[h] = l[h] * corr + b2::warp_sum(pr[h]);
                    m[h] = mn;
#pragma unroll
                    for (int c = 0; c < kGroupMaxPairs; ++c) {
                        acc[h][c][0] *= corr;
                        acc[h][c][1] *= corr;
                    }
                }
            }
            for (int kk = 0; kk < nk; ++kk) {
                float vx[kGroupMaxPairs], vy[kGroupMaxPairs];
#pragma unroll
                for (int c = 0; c < kGroupMaxPairs; ++c) {
                    const int pi = lane + 32 * c;
                    vx[c] = vy[c] = 0.f;
                    if (pi < npairs) {
                        const uint32_t wd = *reinterpret_cast<const uint32_t*>(vt + kk * dv + 2 * pi);
                        vx[c] = __uint_as_float(wd << 16);
                        vy[c] = __uint_as_float(wd & 0xffff0000u);
                    }
                }
#pragma unroll
                for (int h = 0; h < kGroupMaxHeads; ++h) {
                    if (h < QH) {
                        const float ph = __shfl_sync(0xffffffffu, pr[h], kk);
#pragma unroll
                        for (int c = 0; c < kGroupMaxPairs; ++c) {
                            acc[h][c][0] = fmaf(ph, vx[c], acc[h][c][0]);
                            acc[h][c][1] = fmaf(ph, vy[c], acc[h][c][1]);
                        }
                    }
                }
            }
        }
        // merge the four warps
        float* mine = part + (size_t)w * kGroupMaxHeads * (2 + dv);
#pragma unroll
        for (int h = 0; h < kGroupMaxHeads; ++h) {
            if (h < QH) {
                if (lane == 0) {
                    mine[h * (2 + dv)] = m[h];
                    mine[h * (2 + dv) + 1] = l[h];
                }
#pragma unroll
                for (int c = 0; c < kGroupMaxPairs; ++c) {
                    const int pi = lane + 32 * c;
                    if (pi < npairs) {
                        mine[h * (2 + dv) + 2 + 2 * pi] = acc[h][c][0];
                        mine[h * (2 + dv) + 3 + 2 * pi] = acc[h][c][1];
                    }
                }
            }
        }
        __syncthreads();
        // output of (virtual) head h at column col
        auto merged = [&](int h, int col) {
            float M = -INFINITY, L = 0.f, O = 0.f;
            if (SIG) {
                L = 1.f;
                for (int x = 0; x < 4; ++x) O += part[((size_t)x * kGroupMaxHeads + h) * (2 + dv) + 2 + col];
            } else {
                for (int x = 0; x < 4; ++x) M = fmaxf(M, part[((size_t)x * kGroupMaxHeads + h) * (2 + dv)]);
            }
            if (!SIG && M > -INFINITY) {
                for (int x = 0; x < 4; ++x) {
                    const float* px = part + ((size_t)x * kGroupMaxHeads + h) * (2 + dv);
                    const float f = px[0] == -INFINITY ? 0.f : __expf(px[0] - M);
                    L = fmaf(px[1], f, L);
                    O = fmaf(px[2 + col], f, O);
                }
            }
            return L > 0.f ? O / L : 0.f;
        };
        if (MAPS == 1) {
            for (int i = tid; i < QH * dv; i += 128) {
                const int h = i / dv, col = i % dv;
                float res = merged(h, col);
                if (gate) res *= b2::sigmoid_f(__bfloat162float(gate[(size_t)row * gate_stride + (size_t)g * QHall + h0 + h]));
                out[(size_t)row * out_stride + ((size_t)g * QHall + h0 + h) * dv + col] = __float2bfloat16_rn(res);
            }
        } else {
            for (int h = w; h < QH / MAPS; h += 4) {           // a warp per head: the norm runs over its dv columns
                const size_t head = (size_t)g * QHall + h0 / MAPS + h;
                float v[2 * kGroupMaxPairs], ss = 0.f;
#pragma unroll
                for (int c = 0; c < 2 * kGroupMaxPairs; ++c) {
                    const int col = lane + 32 * c;
                    v[c] = col < dv ? merged(h * MAPS, col) - hs.lambda * merged(h * MAPS + MAPS - 1, col) : 0.f;
                    ss = fmaf(v[c], v[c], ss);
                }
                float inv = rsqrtf(b2::warp_sum(ss) / (float)dv + hs.eps) * hs.out_scale;
                if (gate) inv *= b2::sigmoid_f(__bfloat162float(gate[(size_t)row * gate_stride + head]));
#pragma unroll
                for (int c = 0; c < 2 * kGroupMaxPairs; ++c) {
                    const int col = lane + 32 * c;
                    if (col < dv) out[(size_t)row * out_stride + head * dv + col] = __float2bfloat16_rn(v[c] * inv);
                }
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------- head-tile decode kernel
// The same rows for head sizes the tensor cores take (dk a multiple of 32, dv one of the prompt kernel's sizes): one CTA per
// (row, kv head), the query heads of that kv head as the rows of a 16-row operand (two maps: rows 0 - 7 hold the first maps of
// eight heads, rows 8 - 15 their second), so a K or V row is read once and multiplied for all of them at once.  Four warps take
// 32 visible keys at a time each, gather their K and V rows from the pages with cp.async (four lanes a row, one page lookup per
// key), run S = Q K^T and O += P V on mma.sync with the softmax in the accumulator registers, and merge through shared
// memory, which by then no longer holds tiles.  The keys a single row sees are one exact range: nothing to mask but its end.
constexpr int kHeadRows = 16, kHeadKeys = 32;

template <int DVT, bool SIG, int MAPS>
__global__ void __launch_bounds__(128)
chunk_attention_heads_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k_cache,
                             const __nv_bfloat16* __restrict__ v_cache, const int32_t* __restrict__ block_tables, int max_nb,
                             const int32_t* __restrict__ cu_q, const int32_t* __restrict__ ctx_start, int n_seq, int H, int G,
                             int dk, int bs, float scale_log2, int chunk, int window, int keep_first, float sink,
                             float sink_logit, const float* __restrict__ sink_logits, const float* __restrict__ head_bias,
                             const __nv_bfloat16* __restrict__ gate, int64_t gate_stride, HeadShape hs, int skip_rows_from,
                             __nv_bfloat16* __restrict__ out, int64_t out_stride) {
    constexpr int DV = 16 * DVT, LDV = DV + 8, PASS = kHeadRows / MAPS, PW = 2 + DV;
    constexpr float kLog2e = 1.4426950408889634f;
    // q [16][dk + 8], then per warp: K tile [32][MAPS * dk + 8], V tile [32][DV + 8]; the merge reuses the tiles' place
    extern __shared__ __align__(16) unsigned char head_sm[];
    const int row = blockIdx.x, g = blockIdx.y;
    const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
    const int seq = b2::seq_of_row(cu_q, n_seq, row);
    const int ctx = ctx_start[seq];
    const int QHall = H / G;
    if (skip_rows_from > 0 && ctx >= 0 && cu_q[seq + 1] - cu_q[seq] >= skip_rows_from) return;    // the tile kernel's
    if (ctx < 0) {
        for (int i = tid; i < QHall * DV; i += 128)
            out[(size_t)row * out_stride + (size_t)g * QHall * DV + i] = __float2bfloat16_rn(0.f);
        return;
    }
    const int pos = ctx + row - cu_q[seq];
    const KeySpan span = key_span(pos, pos, chunk, window, keep_first);
    const int32_t* bt = block_tables + (size_t)seq * max_nb;
    const int ldq = dk + 8, ldk = MAPS * dk + 8;
    __nv_bfloat16* q_sm = reinterpret_cast<__nv_bfloat16*>(head_sm);
    __nv_bfloat16* tiles = q_sm + kHeadRows * ldq;
    __nv_bfloat16* kt = tiles + (size_t)w * kHeadKeys * (ldk + LDV);
    __nv_bfloat16* vt = kt + kHeadKeys * ldk;
    float* part = reinterpret_cast<float*>(tiles);       // [4][16][m, l, O (DV)]
    const uint32_t q_base = b2::smem_u32(q_sm), k_base = b2::smem_u32(kt), v_base = b2::smem_u32(vt);
    const int gq = lane >> 2, tq = lane & 3;
    const float cap_log2 = hs.cap * kLog2e, cap_e = hs.cap > 0.f ? 2.f / hs.cap : 0.f;

    for (int h0 = 0; h0 < QHall; h0 += PASS) {
        const int QH = min(PASS, QHall - h0);
        __syncthreads();                                 // a previous pass is done with the shared memory
        for (int idx = tid; idx < kHeadRows * (dk / 8); idx += 128) {
            const int r = idx / (dk / 8), c = (idx % (dk / 8)) * 8, h = r % PASS, mp = r / PASS;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (h < QH) v = *reinterpret_cast<const uint4*>(q + (((size_t)row * H + (size_t)g * QHall + h0 + h) * MAPS + mp) * dk + c);
            *reinterpret_cast<uint4*>(q_sm + r * ldq + c) = v;
        }
        __syncthreads();
        // this thread's two rows and the heads they belong to
        const int ha = g * QHall + h0 + min(gq, QH - 1), hb = MAPS > 1 ? ha : g * QHall + h0 + min(gq + 8, QH - 1);
        float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f, ba = 0.f, bb = 0.f;
        if (w == 0 && sink > 0.f) {                      // the sink enters once, through the first warp
            m0 = (sink_logits ? sink_logits[ha] : sink_logit) * kLog2e;
            m1 = (sink_logits ? sink_logits[hb] : sink_logit) * kLog2e;
            l0 = l1 = tq == 0 ? sink : 0.f;
        }
        if (SIG && head_bias) {
            ba = head_bias[ha] * kLog2e;
            bb = head_bias[hb] * kLog2e;
        }
        float o[2 * DVT][4];
#pragma unroll
        for (int n = 0; n < 2 * DVT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;

        for (int c0 = w * kHeadKeys; c0 < span.n; c0 += 4 * kHeadKeys) {
            // keys past the end repeat the last one: finite numbers that the mask drops
            const int j = span.key(min(c0 + lane, span.n - 1));
            const int page = bt[j / bs], off = j % bs;
            __syncwarp();                                // the previous tile has been read
#pragma unroll
            for (int kq = 0; kq < kHeadKeys / 8; ++kq) {
                const int key = kq * 8 + (lane >> 2), c = (lane & 3) * 8;
                const size_t pg = __shfl_sync(0xffffffffu, page, key);
                const int of = __shfl_sync(0xffffffffu, off, key);
#pragma unroll
                for (int mp = 0; mp < MAPS; ++mp) {
                    const __nv_bfloat16* ks = k_cache + ((pg * (G * MAPS) + g * MAPS + mp) * bs + of) * dk + c;
                    __nv_bfloat16* kd = kt + key * ldk + mp * dk + c;
                    for (int t = 0; t < dk; t += 32) cp_async16(kd + t, ks + t);
                }
                const __nv_bfloat16* vs = v_cache + ((pg * G + g) * bs + of) * DV + c;
                __nv_bfloat16* vd = vt + key * LDV + c;
#pragma unroll
                for (int t = 0; t < DV; t += 32) cp_async16(vd + t, vs + t);
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncwarp();
            float sc[4][4], sd[MAPS > 1 ? 4 : 1][4];
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
                if (MAPS > 1) sd[MAPS > 1 ? n : 0][0] = sd[MAPS > 1 ? n : 0][1] = sd[MAPS > 1 ? n : 0][2] = sd[MAPS > 1 ? n : 0][3] = 0.f;
            }
            for (int kk = 0; kk < dk; kk += 16) {
                uint32_t a0, a1, a2, a3;
                b2::ldmatrix_x4(q_base + 2u * ((lane & 15) * ldq + kk + (lane >> 4) * 8), a0, a1, a2, a3);
#pragma unroll
                for (int n2 = 0; n2 < 2; ++n2) {
                    uint32_t b0, b1, b2_, b3;
                    const int key = n2 * 16 + (lane >> 4) * 8 + (lane & 7), dim = kk + ((lane >> 3) & 1) * 8;
                    b2::ldmatrix_x4(k_base + 2u * (key * ldk + dim), b0, b1, b2_, b3);
                    b2::mma_bf16_16816(sc[2 * n2], a0, a1, a2, a3, b0, b1);
                    b2::mma_bf16_16816(sc[2 * n2 + 1], a0, a1, a2, a3, b2_, b3);
                    if (MAPS > 1) {                      // rows 8 - 15 belong to the second maps and take their keys
                        b2::ldmatrix_x4(k_base + 2u * (key * ldk + dk + dim), b0, b1, b2_, b3);
                        b2::mma_bf16_16816(sd[MAPS > 1 ? 2 * n2 : 0], a0, a1, a2, a3, b0, b1);
                        b2::mma_bf16_16816(sd[MAPS > 1 ? 2 * n2 + 1 : 0], a0, a1, a2, a3, b2_, b3);
                    }
                }
            }
            if (MAPS > 1) {
#pragma unroll
                for (int n = 0; n < 4; ++n) {
                    sc[n][2] = sd[MAPS > 1 ? n : 0][2];
                    sc[n][3] = sd[MAPS > 1 ? n : 0][3];
                }
            }
            const bool whole = c0 + kHeadKeys <= span.n;
            float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
            for (int n = 0; n < 4; ++n) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    float x = sc[n][e] * scale_log2;
                    const bool in = whole || c0 + n * 8 + 2 * tq + (e & 1) < span.n;
                    if (SIG) {
                        x = in ? sigmoid2_f(x + (e < 2 ? ba : bb)) : 0.f;
                    } else {
                        if (hs.cap > 0.f) x = cap_score(x, cap_log2, cap_e);
                        if (!in) x = -INFINITY;
                        if (e < 2) mx0 = fmaxf(mx0, x); else mx1 = fmaxf(mx1, x);
                    }
                    sc[n][e] = x;
                }
            }
            if (!SIG) {
#pragma unroll
                for (int x = 1; x < 4; x <<= 1) {
                    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, x));
                    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, x));
                }
                const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);         // finite: the tile has at least one key
                const float f0 = b2::fast_exp2(m0 - mn0), f1 = b2::fast_exp2(m1 - mn1);
                m0 = mn0;
                m1 = mn1;
                l0 *= f0;
                l1 *= f1;
#pragma unroll
                for (int n = 0; n < 4; ++n) {
                    sc[n][0] = b2::fast_exp2(sc[n][0] - mn0);
                    sc[n][1] = b2::fast_exp2(sc[n][1] - mn0);
                    sc[n][2] = b2::fast_exp2(sc[n][2] - mn1);
                    sc[n][3] = b2::fast_exp2(sc[n][3] - mn1);
                    l0 += sc[n][0] + sc[n][1];
                    l1 += sc[n][2] + sc[n][3];
                }
#pragma unroll
                for (int n = 0; n < 2 * DVT; ++n) {
                    o[n][0] *= f0;
                    o[n][1] *= f0;
                    o[n][2] *= f1;
                    o[n][3] *= f1;
                }
            }
#pragma unroll
            for (int ks = 0; ks < 2; ++ks) {
                const uint32_t a0 = b2::pack_bf16x2(sc[2 * ks][0], sc[2 * ks][1]), a1 = b2::pack_bf16x2(sc[2 * ks][2], sc[2 * ks][3]);
                const uint32_t a2 = b2::pack_bf16x2(sc[2 * ks + 1][0], sc[2 * ks + 1][1]),
                               a3 = b2::pack_bf16x2(sc[2 * ks + 1][2], sc[2 * ks + 1][3]);
#pragma unroll
                for (int n2 = 0; n2 < DVT; ++n2) {
                    uint32_t b0, b1, b2_, b3;
                    const int key = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), col = n2 * 16 + (lane >> 4) * 8;
                    b2::ldmatrix_x4_trans(v_base + 2u * (key * LDV + col), b0, b1, b2_, b3);
                    b2::mma_bf16_16816(o[2 * n2], a0, a1, a2, a3, b0, b1);
                    b2::mma_bf16_16816(o[2 * n2 + 1], a0, a1, a2, a3, b2_, b3);
                }
            }
        }
#pragma unroll
        for (int x = 1; x < 4; x <<= 1) {
            l0 += __shfl_xor_sync(0xffffffffu, l0, x);
            l1 += __shfl_xor_sync(0xffffffffu, l1, x);
        }
        __syncthreads();                                 // every warp is done with its tiles: the partial results take their place
        float* pa = part + (size_t)(w * kHeadRows + gq) * PW;
        float* pb = pa + 8 * PW;
        if (tq == 0) {
            pa[0] = m0; pa[1] = l0;
            pb[0] = m1; pb[1] = l1;
        }
#pragma unroll
        for (int n = 0; n < 2 * DVT; ++n) {
            const int col = 2 + n * 8 + 2 * tq;
            *reinterpret_cast<float2*>(pa + col) = make_float2(o[n][0], o[n][1]);
            *reinterpret_cast<float2*>(pb + col) = make_float2(o[n][2], o[n][3]);
        }
        __syncthreads();
        // a warp per head: merged output of operand row r at column col
        for (int h = w; h < QH; h += 4) {
            const size_t head = (size_t)g * QHall + h0 + h;
            float f[MAPS][4];
#pragma unroll
            for (int mp = 0; mp < MAPS; ++mp) {
                const float* px = part + (size_t)(h + mp * PASS) * PW;
                float M = -INFINITY, L = 0.f;
#pragma unroll
                for (int x = 0; x < 4; ++x) M = fmaxf(M, px[(size_t)x * kHeadRows * PW]);
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    const float mx = px[(size_t)x * kHeadRows * PW];
                    f[mp][x] = SIG ? 1.f : (mx == -INFINITY ? 0.f : b2::fast_exp2(mx - M));
                    L = fmaf(px[(size_t)x * kHeadRows * PW + 1], f[mp][x], L);
                }
                const float inv = (SIG ? 1.f : (L > 0.f ? 1.f / L : 0.f)) * (mp == 0 ? 1.f : -hs.lambda);
#pragma unroll
                for (int x = 0; x < 4; ++x) f[mp][x] *= inv;
            }
            float v[DV / 32], ss = 0.f;
#pragma unroll
            for (int c = 0; c < DV / 32; ++c) {
                v[c] = 0.f;
#pragma unroll
                for (int mp = 0; mp < MAPS; ++mp) {
                    const float* px = part + (size_t)(h + mp * PASS) * PW + 2 + lane + 32 * c;
#pragma unroll
                    for (int x = 0; x < 4; ++x) v[c] = fmaf(px[(size_t)x * kHeadRows * PW], f[mp][x], v[c]);
                }
                ss = fmaf(v[c], v[c], ss);
            }
            float inv = MAPS > 1 ? rsqrtf(b2::warp_sum(ss) / (float)DV + hs.eps) * hs.out_scale : 1.f;
            if (gate) inv *= b2::sigmoid_f(__bfloat162float(gate[(size_t)row * gate_stride + head]));
#pragma unroll
            for (int c = 0; c < DV / 32; ++c)
                out[(size_t)row * out_stride + head * DV + lane + 32 * c] = __float2bfloat16_rn(v[c] * inv);
        }
    }
}

template <int DVT, bool SIG, int MAPS>
int launch_heads(const void* q, const void* k_cache, const void* v_cache, const int32_t* block_tables, int max_nb,
                 const int32_t* cu_q, const int32_t* ctx_start, int n_seq, int T, int H, int G, int dk, int bs, float scale, int chunk,
                 int window, int keep_first, float sink, float sink_logit, const float* sink_logits, const float* head_bias,
                 const void* gate, int64_t gate_stride, const HeadShape& hs, int skip_from, void* out, int64_t out_stride,
                 cudaStream_t st) {
    constexpr int DV = 16 * DVT;
    const size_t tiles = (size_t)4 * kHeadKeys * (MAPS * dk + 8 + DV + 8) * sizeof(__nv_bfloat16);
    const size_t merge = (size_t)4 * kHeadRows * (2 + DV) * sizeof(float);
    const size_t smem = (size_t)kHeadRows * (dk + 8) * sizeof(__nv_bfloat16) + (tiles > merge ? tiles : merge);
    auto kern = chunk_attention_heads_kernel<DVT, SIG, MAPS>;
    if (smem > 48 * 1024) B2_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kern<<<dim3(T, G), 128, smem, st>>>(static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k_cache),
                                       static_cast<const __nv_bfloat16*>(v_cache), block_tables, max_nb, cu_q, ctx_start, n_seq, H,
                                       G, dk, bs, scale * 1.4426950408889634f, chunk, window, keep_first, sink, sink_logit, sink_logits,
                                       head_bias, static_cast<const __nv_bfloat16*>(gate), gate_stride, hs, skip_from,
                                       static_cast<__nv_bfloat16*>(out), out_stride);
    B2_CUDA_OK(cudaGetLastError());
    return B2_OK;
}

// ------------------------------------------------------------------------------------------------- tiled prompt kernel
// bf16, dk and dv multiples of 16: one CTA = 64 consecutive query rows of one sequence x one head, four warps of 16 rows.
// Keys are walked 64 at a time from the first row's block start to the last row's position (at most chunk + 63 keys
// with a mask, the whole prefix without): K and V tiles are gathered from the pages into shared memory (cp.async, two
// threads per key row with one page lookup each, the next tile in flight while this one is multiplied), S = Q K^T and
// O += P V run on mma.sync m16n8k16 with ldmatrix operands, the online softmax lives in the accumulator registers
// (exp2 with the scale folded in, the sink seeding the running maximum and denominator).  A warp tests the mask per score
// only in tiles that its rows see in part.  Sequences with fewer than kTileMinRows rows (decode rows) are left to the warp
// kernel above.
constexpr int kTQ = 64, kTK = 64, kTileMinRows = 16;

template <int DKT, int DVT, bool SIG, int MAPS>
__global__ void __launch_bounds__(128)
chunk_attention_tile_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k_cache,
                            const __nv_bfloat16* __restrict__ v_cache, const int32_t* __restrict__ block_tables, int max_nb,
                            const int32_t* __restrict__ cu_q, const int32_t* __restrict__ ctx_start, int n_seq, int H, int G,
                            int bs, float scale_log2, int chunk, int window, int keep_first, float sink,
                            float sink_logit_log2, const float* __restrict__ sink_logits, const float* __restrict__ head_bias,
                            const __nv_bfloat16* __restrict__ gate, int64_t gate_stride, HeadShape hs, __nv_bfloat16* __restrict__ out,
                            int64_t out_stride) {
    constexpr int DK = 16 * DKT, DV = 16 * DVT, LDK = MAPS * DK + 8, LDV = DV + 8;
    extern __shared__ __align__(16) unsigned char tile_smem[];
    __nv_bfloat16* q_sm = reinterpret_cast<__nv_bfloat16*>(tile_smem);      // [64][LDK]
    __nv_bfloat16* k_sm = q_sm + kTQ * LDK;                                 // [2][64][LDK]
    __nv_bfloat16* v_sm = k_sm + 2 * kTK * LDK;                             // [2][64][LDV]
    __shared__ int s_info[2];
    const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
    if (tid == 0) {
        int want = blockIdx.x, found = -1, t0 = 0;
        for (int s = 0; s < n_seq; ++s) {
            const int len = cu_q[s + 1] - cu_q[s];
            if (len < kTileMinRows || ctx_start[s] < 0) continue;
            const int nt = (len + kTQ - 1) / kTQ;
            if (want < nt) { found = s; t0 = want * kTQ; break; }
            want -= nt;
        }
        s_info[0] = found;
        s_info[1] = t0;
    }
    __syncthreads();
    const int seq = s_info[0], t0 = s_info[1];
    if (seq < 0) return;
    const int hh = blockIdx.y, g = hh / (H / G);
    const int r0 = cu_q[seq] + t0;
    const int rows = min(kTQ, cu_q[seq + 1] - r0);
    const int p0 = ctx_start[seq] + t0, p_last = p0 + rows - 1;
    // the union of what the tile's rows see, as one compact range: kept first keys, then the first row's window .. p_last
    const KeySpan span = key_span(p0, p_last, chunk, window, keep_first);
    const int32_t* bt = block_tables + (size_t)seq * max_nb;

    for (int idx = tid; idx < kTQ * (MAPS * DK / 8); idx += 128) {
        const int r = idx / (MAPS * DK / 8), c = (idx % (MAPS * DK / 8)) * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < rows) v = *reinterpret_cast<const uint4*>(q + ((size_t)(r0 + r) * H + hh) * (MAPS * DK) + c);
        *reinterpret_cast<uint4*>(q_sm + r * LDK + c) = v;
    }
    const int gq = lane >> 2, tq = lane & 3;
    const int i0 = p0 + w * 16 + gq, i1 = i0 + 8;                           // positions of this thread's two rows
    const int lo0 = chunk > 0 ? (i0 / chunk) * chunk : 0, lo1 = chunk > 0 ? (i1 / chunk) * chunk : 0;
    const int w_first = p0 + w * 16, w_last = w_first + 15;
    const int w_clo = chunk > 0 ? (w_first / chunk) * chunk : 0;
    const int w_lo = window > 0 ? max(w_clo, w_first - window + 1) : w_clo;   // the lowest key of the warp's rows' windows
    if (sink_logits) sink_logit_log2 = sink_logits[hh] * 1.4426950408889634f;
    float m0[MAPS], m1[MAPS], l0[MAPS], l1[MAPS];                           // partial sums per lane; the sink counted once
    float o[MAPS][2 * DVT][4];
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
        m0[mp] = m1[mp] = sink > 0.f ? sink_logit_log2 : -INFINITY;
        l0[mp] = l1[mp] = tq == 0 ? sink : 0.f;
#pragma unroll
        for (int n = 0; n < 2 * DVT; ++n) o[mp][n][0] = o[mp][n][1] = o[mp][n][2] = o[mp][n][3] = 0.f;
    }
    const float bias_log2 = SIG && head_bias ? head_bias[hh] * 1.4426950408889634f : 0.f;
    const float cap_log2 = hs.cap * 1.4426950408889634f, cap_e = hs.cap > 0.f ? 2.f / hs.cap : 0.f;
    const uint32_t q_base = b2::smem_u32(q_sm), k_base0 = b2::smem_u32(k_sm), v_base0 = b2::smem_u32(v_sm);

    const int ld_key = tid >> 1, ld_half = tid & 1;
    auto issue = [&](int kv0, int buf) {                                    // kv0: compact key index of the tile's first key
        const int j = span.key(kv0 + ld_key);
        __nv_bfloat16* kd = k_sm + (buf * kTK + ld_key) * LDK;
        __nv_bfloat16* vd = v_sm + (buf * kTK + ld_key) * LDV;
        if (j <= p_last) {
            const int page = j / bs;
            const size_t blk = bt[page], off = j - page * bs;
            const __nv_bfloat16* vs = v_cache + ((blk * G + g) * bs + off) * DV;
#pragma unroll
            for (int mp = 0; mp < MAPS; ++mp) {
                const __nv_bfloat16* ks = k_cache + ((blk * (G * MAPS) + g * MAPS + mp) * bs + off) * DK;
#pragma unroll
                for (int c = 0; c < DKT; ++c) cp_async16(kd + mp * DK + (2 * c + ld_half) * 8, ks + (2 * c + ld_half) * 8);
            }
#pragma unroll
            for (int c = 0; c < DVT; ++c) cp_async16(vd + (2 * c + ld_half) * 8, vs + (2 * c + ld_half) * 8);
        } else {
#pragma unroll
            for (int c = 0; c < MAPS * DKT; ++c) *reinterpret_cast<uint4*>(kd + (2 * c + ld_half) * 8) = make_uint4(0, 0, 0, 0);
#pragma unroll
            for (int c = 0; c < DVT; ++c) *reinterpret_cast<uint4*>(vd + (2 * c + ld_half) * 8) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    issue(0, 0);
    for (int kv0 = 0, buf = 0; kv0 < span.n; kv0 += kTK, buf ^= 1) {
        if (kv0 + kTK < span.n) {
            issue(kv0 + kTK, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();                                                    // the tile (and, first time, Q) is in shared memory
        const uint32_t k_base = k_base0 + (uint32_t)(buf * kTK * LDK) * 2u, v_base = v_base0 + (uint32_t)(buf * kTK * LDV) * 2u;
        const int j_min = span.key(kv0), j_max = span.key(min(kv0 + kTK, span.n) - 1);
        // nothing in this tile is visible to the warp's rows: all keys after them, or all before their windows and not kept
        const bool none = j_min > w_last || (j_max < w_lo && (window <= 0 || j_min >= keep_first));
        // all of it is visible to all of them
        const bool full = kv0 + kTK <= span.n && j_max <= w_first && (chunk <= 0 || j_min >= (w_last / chunk) * chunk) &&
                          (window <= 0 || w_last - j_min < window || j_max < keep_first);
        if (!none) {
#pragma unroll
            for (int mp = 0; mp < MAPS; ++mp) {
                float sc[8][4];
#pragma unroll
                for (int n = 0; n < 8; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll
                for (int kk = 0; kk < DKT; ++kk) {
                    uint32_t a0, a1, a2, a3;
                    b2::ldmatrix_x4(q_base + 2u * ((w * 16 + (lane & 15)) * LDK + mp * DK + kk * 16 + (lane >> 4) * 8), a0, a1, a2, a3);
#pragma unroll
                    for (int n2 = 0; n2 < 4; ++n2) {
                        uint32_t b0, b1, b2_, b3;
                        const int key = n2 * 16 + (lane >> 4) * 8 + (lane & 7), dim = mp * DK + kk * 16 + ((lane >> 3) & 1) * 8;
                        b2::ldmatrix_x4(k_base + 2u * (key * LDK + dim), b0, b1, b2_, b3);
                        b2::mma_bf16_16816(sc[2 * n2], a0, a1, a2, a3, b0, b1);
                        b2::mma_bf16_16816(sc[2 * n2 + 1], a0, a1, a2, a3, b2_, b3);
                    }
                }
                if (SIG) {                                                          // every weight by itself: nothing to rescale
#pragma unroll
                    for (int n = 0; n < 8; ++n) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) sc[n][e] = sigmoid2_f(fmaf(sc[n][e], scale_log2, bias_log2));
                    }
                    if (!full) {
#pragma unroll
                        for (int n = 0; n < 8; ++n) {
#pragma unroll
                            for (int e = 0; e < 4; ++e) {
                                const int j = span.key(kv0 + n * 8 + 2 * tq + (e & 1));
                                const bool ok = e < 2 ? key_visible(i0, j, lo0, window, keep_first) : key_visible(i1, j, lo1, window, keep_first);
                                if (!ok) sc[n][e] = 0.f;
                            }
                        }
                    }
                } else {
                    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
                    for (int n = 0; n < 8; ++n) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) sc[n][e] *= scale_log2;
                    }
                    if (hs.cap > 0.f) {
#pragma unroll
                        for (int n = 0; n < 8; ++n) {
#pragma unroll
                            for (int e = 0; e < 4; ++e) sc[n][e] = cap_score(sc[n][e], cap_log2, cap_e);
                        }
                    }
                    if (!full) {
#pragma unroll
                        for (int n = 0; n < 8; ++n) {
#pragma unroll
                            for (int e = 0; e < 4; ++e) {
                                const int j = span.key(kv0 + n * 8 + 2 * tq + (e & 1));
                                const bool ok = e < 2 ? key_visible(i0, j, lo0, window, keep_first) : key_visible(i1, j, lo1, window, keep_first);
                                if (!ok) sc[n][e] = -INFINITY;
                            }
                        }
                    }
#pragma unroll
                    for (int n = 0; n < 8; ++n) {
                        mx0 = fmaxf(mx0, fmaxf(sc[n][0], sc[n][1]));
                        mx1 = fmaxf(mx1, fmaxf(sc[n][2], sc[n][3]));
                    }
                    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
                    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
                    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
                    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
                    const float mn0 = fmaxf(m0[mp], mx0), mn1 = fmaxf(m1[mp], mx1);
                    const float mu0 = mn0 == -INFINITY ? 0.f : mn0, mu1 = mn1 == -INFINITY ? 0.f : mn1;
                    const float c0 = b2::fast_exp2(m0[mp] - mu0), c1 = b2::fast_exp2(m1[mp] - mu1);             // exp2(-inf) = 0: nothing accumulated yet
                    m0[mp] = mn0;
                    m1[mp] = mn1;
                    float s0 = 0.f, s1 = 0.f;
#pragma unroll
                    for (int n = 0; n < 8; ++n) {
                        sc[n][0] = b2::fast_exp2(sc[n][0] - mu0);
                        sc[n][1] = b2::fast_exp2(sc[n][1] - mu0);
                        sc[n][2] = b2::fast_exp2(sc[n][2] - mu1);
                        sc[n][3] = b2::fast_exp2(sc[n][3] - mu1);
                        s0 += sc[n][0] + sc[n][1];
                        s1 += sc[n][2] + sc[n][3];
                    }
                    l0[mp] = l0[mp] * c0 + s0;
                    l1[mp] = l1[mp] * c1 + s1;
#pragma unroll
                    for (int n = 0; n < 2 * DVT; ++n) {
                        o[mp][n][0] *= c0;
                        o[mp][n][1] *= c0;
                        o[mp][n][2] *= c1;
                        o[mp][n][3] *= c1;
                    }
                }
#pragma unroll
                for (int ks = 0; ks < 4; ++ks) {
                    const uint32_t a0 = b2::pack_bf16x2(sc[2 * ks][0], sc[2 * ks][1]), a1 = b2::pack_bf16x2(sc[2 * ks][2], sc[2 * ks][3]);
                    const uint32_t a2 = b2::pack_bf16x2(sc[2 * ks + 1][0], sc[2 * ks + 1][1]),
                                   a3 = b2::pack_bf16x2(sc[2 * ks + 1][2], sc[2 * ks + 1][3]);
#pragma unroll
                    for (int n2 = 0; n2 < DVT; ++n2) {
                        uint32_t b0, b1, b2_, b3;
                        const int key = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), col = n2 * 16 + (lane >> 4) * 8;
                        b2::ldmatrix_x4_trans(v_base + 2u * (key * LDV + col), b0, b1, b2_, b3);
                        b2::mma_bf16_16816(o[mp][2 * n2], a0, a1, a2, a3, b0, b1);
                        b2::mma_bf16_16816(o[mp][2 * n2 + 1], a0, a1, a2, a3, b2_, b3);
                    }
                }
            }
        }
        __syncthreads();                                                    // the tile is consumed: its buffer may be refilled
    }
    float inv0 = 1.f, inv1 = 1.f;
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
#pragma unroll
        for (int x = 1; x < 4; x <<= 1) {
            l0[mp] += __shfl_xor_sync(0xffffffffu, l0[mp], x);
            l1[mp] += __shfl_xor_sync(0xffffffffu, l1[mp], x);
        }
        inv0 = SIG ? 1.f : (l0[mp] > 0.f ? 1.f / l0[mp] : 0.f);
        inv1 = SIG ? 1.f : (l1[mp] > 0.f ? 1.f / l1[mp] : 0.f);
        if (MAPS > 1) {
            const float f0 = mp == 0 ? inv0 : -hs.lambda * inv0, f1 = mp == 0 ? inv1 : -hs.lambda * inv1;
#pragma unroll
            for (int n = 0; n < 2 * DVT; ++n) {
                o[mp][n][0] *= f0;
                o[mp][n][1] *= f0;
                o[mp][n][2] *= f1;
                o[mp][n][3] *= f1;
            }
        }
    }
    const int ra = w * 16 + gq, rb = ra + 8;
    if (MAPS > 1) {                                                         // the difference and its norm over the head's columns
        float s0 = 0.f, s1 = 0.f;
#pragma unroll
        for (int n = 0; n < 2 * DVT; ++n) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                o[0][n][e] += o[MAPS - 1][n][e];
                if (e < 2) s0 = fmaf(o[0][n][e], o[0][n][e], s0);
                else s1 = fmaf(o[0][n][e], o[0][n][e], s1);
            }
        }
#pragma unroll
        for (int x = 1; x < 4; x <<= 1) {
            s0 += __shfl_xor_sync(0xffffffffu, s0, x);
            s1 += __shfl_xor_sync(0xffffffffu, s1, x);
        }
        inv0 = rsqrtf(s0 / (float)DV + hs.eps) * hs.out_scale;
        inv1 = rsqrtf(s1 / (float)DV + hs.eps) * hs.out_scale;
    }
    if (gate) {
        if (ra < rows) inv0 *= b2::sigmoid_f(__bfloat162float(gate[(size_t)(r0 + ra) * gate_stride + hh]));
        if (rb < rows) inv1 *= b2::sigmoid_f(__bfloat162float(gate[(size_t)(r0 + rb) * gate_stride + hh]));
    }
#pragma unroll
    for (int n = 0; n < 2 * DVT; ++n) {
        const int col = n * 8 + 2 * tq;
        if (ra < rows)
            *reinterpret_cast<uint32_t*>(out + (size_t)(r0 + ra) * out_stride + hh * DV + col) = b2::pack_bf16x2(o[0][n][0] * inv0, o[0][n][1] * inv0);
        if (rb < rows)
            *reinterpret_cast<uint32_t*>(out + (size_t)(r0 + rb) * out_stride + hh * DV + col) = b2::pack_bf16x2(o[0][n][2] * inv1, o[0][n][3] * inv1);
    }
}

template <int DKT, int DVT, bool SIG, int MAPS>
int launch_tile(const void* q, const void* k_cache, const void* v_cache, const int32_t* block_tables, int max_nb,
                const int32_t* cu_q, const int32_t* ctx_start, int n_seq, int T, int H, int G, int bs, float scale, int chunk,
                int window, int keep_first, float sink, float sink_logit, const float* sink_logits, const float* head_bias,
                const void* gate, int64_t gate_stride, const HeadShape& hs, void* out, int64_t out_stride, cudaStream_t st) {
    constexpr int DK = 16 * DKT, DV = 16 * DVT;
    const size_t smem = (size_t)(kTQ * (MAPS * DK + 8) + 2 * kTK * (MAPS * DK + 8) + 2 * kTK * (DV + 8)) * sizeof(__nv_bfloat16);
    auto kern = chunk_attention_tile_kernel<DKT, DVT, SIG, MAPS>;
    if (smem > 48 * 1024) B2_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const int tiles = (T + kTQ - 1) / kTQ + n_seq;          // upper bound on sum(ceil(len / 64)); spare CTAs leave at once
    kern<<<dim3(tiles, H), 128, smem, st>>>(static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k_cache),
                                           static_cast<const __nv_bfloat16*>(v_cache), block_tables, max_nb, cu_q, ctx_start,
                                           n_seq, H, G, bs, scale * 1.4426950408889634f, chunk, window, keep_first, sink,
                                           sink_logit * 1.4426950408889634f, sink_logits, head_bias,
                                           static_cast<const __nv_bfloat16*>(gate), gate_stride, hs, static_cast<__nv_bfloat16*>(out),
                                           out_stride);
    B2_CUDA_OK(cudaGetLastError());
    return B2_OK;
}

}  // namespace

extern "C" int b2_qknorm_cache(const void* qkv, int64_t qkv_stride, int act_dtype, int T, int H, int G, int dk, int dv,
                               const float* q_w, const float* k_w, float eps, const int64_t* slots, int bs, void* q_out,
                               void* k_cache, void* v_cache, void* stream) {
    B2_REQUIRE(T >= 0 && H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0 && bs > 0, B2_EINVAL, "qknorm_cache: bad sizes");
    if (T == 0) return B2_OK;
    B2_REQUIRE(qkv && slots && q_out && k_cache && v_cache, B2_EINVAL, "qknorm_cache: null pointer");
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const int warps = H + 2 * G < 8 ? H + 2 * G : 8;
    B2_DISPATCH_ACT(act_dtype, A, (qknorm_cache_kernel<A><<<T, warps * 32, 0, st>>>(
        static_cast<const A*>(qkv), qkv_stride, H, G, dk, dv, q_w, k_w, eps, slots, bs, static_cast<A*>(q_out),
        static_cast<A*>(k_cache), static_cast<A*>(v_cache), true, nullptr, 0.f, 1)));
    B2_CUDA_OK(cudaGetLastError());
    return B2_OK;
}

extern "C" int b2_qk_prep_cache(const void* qkv, int64_t qkv_stride, int act_dtype, int T, int H, int G, int dk, int dv,
                                int norm, const float* q_w, const float* k_w, float eps, const int32_t* positions,
                                float temp_coef, int temp_every, const int64_t* slots, int bs, void* q_out, void* k_cache,
                                void* v_cache, void* stream) {
    B2_REQUIRE(T >= 0 && H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0 && bs > 0, B2_EINVAL, "qk_prep_cache: bad sizes");
    B2_REQUIRE(temp_coef == 0.f || (positions && temp_every >= 1), B2_EINVAL,
               "qk_prep_cache: a query temperature needs positions and a period of at least 1");
    if (T == 0) return B2_OK;
    B2_REQUIRE(qkv && slots && q_out && k_cache && v_cache, B2_EINVAL, "qk_prep_cache: null pointer");
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const int warps = H + 2 * G < 8 ? H + 2 * G : 8;
    B2_DISPATCH_ACT(act_dtype, A, (qknorm_cache_kernel<A><<<T, warps * 32, 0, st>>>(
        static_cast<const A*>(qkv), qkv_stride, H, G, dk, dv, q_w, k_w, eps, slots, bs, static_cast<A*>(q_out),
        static_cast<A*>(k_cache), static_cast<A*>(v_cache), norm != 0, positions, temp_coef, temp_every > 0 ? temp_every : 1)));
    B2_CUDA_OK(cudaGetLastError());
    return B2_OK;
}

extern "C" int b2_qk_rope_cache(const void* qkv, int64_t qkv_stride, int act_dtype, int T, int H, int G, int dk, int dv,
                                int v_from_k, int rot_dims, int interleaved, const int32_t* positions, const float* cos_sin,
                                int max_pos, const int64_t* slots, int bs, void* q_out, void* k_cache, void* v_cache,
                                void* stream) {
    return b2_qk_norm_rope_cache(qkv, qkv_stride, act_dtype, T, H, G, G, dk, dv, v_from_k, nullptr, nullptr, 0.f, rot_dims, interleaved,
                                 positions, cos_sin, max_pos, slots, bs, q_out, k_cache, v_cache, stream);
}

extern "C" int b2_qk_norm_rope_cache(const void* qkv, int64_t qkv_stride, int act_dtype, int T, int H, int G, int Gv, int dk, int dv,
                                     int v_from_k, const float* q_w, const float* k_w, float eps, int rot_dims, int interleaved,
                                     const int32_t* positions, const float* cos_sin, int max_pos, const int64_t* slots, int bs,
                                     void* q_out, void* k_cache, void* v_cache, void* stream) {
    B2_REQUIRE(T >= 0 && H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0 && bs > 0, B2_EINVAL, "qk_rope_cache: bad sizes");
    B2_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dk, B2_EINVAL,
               "qk_rope_cache: %d rotated entries in heads of %d", rot_dims, dk);
    B2_REQUIRE(Gv > 0 && Gv <= G, B2_EINVAL, "qk_rope_cache: %d value heads beside %d key heads", Gv, G);
    B2_REQUIRE(!v_from_k || (dv == dk && Gv == G), B2_EINVAL, "qk_rope_cache: values taken from the keys need dv == dk and a value head per key head");
    B2_REQUIRE(rot_dims == 0 || max_pos > 0, B2_EINVAL, "qk_rope_cache: empty rotation table");
    B2_REQUIRE(!q_w == !k_w, B2_EINVAL, "qk_rope_cache: the norm needs the weights of both q and k");
    if (T == 0) return B2_OK;
    B2_REQUIRE(qkv && slots && q_out && k_cache && v_cache && positions && (cos_sin || rot_dims == 0), B2_EINVAL,
               "qk_rope_cache: null pointer");
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const size_t esz = act_dtype == B2_ACT_BF16 ? 2 : 4;
    auto al = [&](const void* p) { return reinterpret_cast<uintptr_t>(p) % (4 * esz) == 0; };
    const bool vec = dk % 4 == 0 && dv % 4 == 0 && qkv_stride % 4 == 0 && rot_dims % (interleaved ? 4 : 8) == 0 && al(qkv) && al(q_out) &&
                     al(k_cache) && al(v_cache);
    const int work = (H + G) * dk / (vec ? 4 : 1);
    const int threads = work >= 256 ? 256 : (work >= 128 ? 128 : 64);
#define B2_ROPE(KERN, NORM)                                                                                                     \
    KERN<A, NORM><<<T, threads, 0, st>>>(static_cast<const A*>(qkv), qkv_stride, H, G, Gv, dk, dv, v_from_k != 0, rot_dims,         \
                                         interleaved != 0, positions, cos_sin, max_pos > 0 ? max_pos : 1, slots, bs, q_w, k_w, eps, \
                                         static_cast<A*>(q_out), static_cast<A*>(k_cache), static_cast<A*>(v_cache))
    B2_DISPATCH_ACT(act_dtype, A, {
        if (vec && q_w) B2_ROPE(qk_rope_cache_vec_kernel, true);
        else if (vec) B2_ROPE(qk_rope_cache_vec_kernel, false);
        else if (q_w) B2_ROPE(qk_rope_cache_kernel, true);
        else B2_ROPE(qk_rope_cache_kernel, false);
    });
#undef B2_ROPE
    B2_CUDA_OK(cudaGetLastError());
    return B2_OK;
}

extern "C" int b2_chunk_attention(void* out, const void* q, const void* k_cache, const void* v_cache, int act_dtype,
                                  const int32_t* block_tables, int max_nb, const int32_t* cu_q, const int32_t* ctx_start,
                                  int n_seq, int T, int H, int G, int dk, int dv, int bs, float scale, int chunk, float sink,
                                  float sink_logit, void* stream) {
    return b2_masked_attention(out, q, k_cache, v_cache, act_dtype, block_tables, max_nb, cu_q, ctx_start, n_seq, T, H, G, dk, dv,
                               bs, scale, chunk, 0, 0, sink, sink_logit, nullptr, B2_WEIGHT_SOFTMAX, nullptr, nullptr, 0, 0.f, 1, 0.f,
                               0.f, 1.f, (int64_t)H * dv, stream);
}

extern "C" int b2_masked_attention(void* out, const void* q, const void* k_cache, const void* v_cache, int act_dtype,
                                   const int32_t* block_tables, int max_nb, const int32_t* cu_q, const int32_t* ctx_start,
                                   int n_seq, int T, int H, int G, int dk, int dv, int bs, float scale, int chunk, int window,
                                   int keep_first, float sink, float sink_logit, const float* sink_logits, int weight_kind,
                                   const float* head_bias, const void* gate, int64_t gate_stride, float softcap, int maps,
                                   float map_lambda, float map_eps, float map_scale, int64_t out_stride, void* stream) {
    B2_REQUIRE(T >= 0 && H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0 && bs > 0 && chunk >= 0 && sink >= 0.f && window >= 0 &&
               keep_first >= 0, B2_EINVAL, "masked_attention: bad sizes");
    B2_REQUIRE(!gate || gate_stride >= H, B2_EINVAL, "masked_attention: gate rows shorter than the heads");
    B2_REQUIRE(weight_kind == B2_WEIGHT_SOFTMAX || weight_kind == B2_WEIGHT_SIGMOID, B2_EINVAL,
               "masked_attention: unknown weight kind %d", weight_kind);
    const bool sig = weight_kind == B2_WEIGHT_SIGMOID;
    B2_REQUIRE(sig ? sink == 0.f : !head_bias, B2_EINVAL,
               "masked_attention: sigmoid weights have no sink, and only they take a bias per head");
    B2_REQUIRE(maps == 1 || maps == 2, B2_EINVAL, "masked_attention: %d maps per head", maps);
    B2_REQUIRE(!sig || (maps == 1 && softcap == 0.f), B2_EINVAL, "masked_attention: sigmoid weights have one map and no cap");
    B2_REQUIRE(softcap >= 0.f, B2_EINVAL, "masked_attention: negative cap");
    B2_REQUIRE(out_stride >= (int64_t)H * dv, B2_EINVAL, "masked_attention: output rows shorter than the heads");
    B2_REQUIRE(dv <= 32 * kMaxDvPerLane, B2_EUNSUPPORTED, "chunk_attention: value size %d above %d", dv, 32 * kMaxDvPerLane);
    if (T == 0 || n_seq == 0) return B2_OK;
    B2_REQUIRE(out && q && k_cache && v_cache && block_tables && cu_q && ctx_start, B2_EINVAL, "chunk_attention: null pointer");
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const HeadShape hs{softcap, map_lambda, map_eps, map_scale};
    const int warps = 4;
    const size_t smem = (size_t)warps * dk * sizeof(float);
    B2_REQUIRE(smem <= 48 * 1024, B2_EUNSUPPORTED, "chunk_attention: key size %d too large", dk);
    const int items = T * H, blocks = (items + warps - 1) / warps;
    // prompt chunks of bf16 models with tensor-core friendly head sizes go to the tiled kernel (a sequence needs at least
    // kTileMinRows rows, so a batch of T rows over n_seq sequences can only hold one when T - n_seq >= kTileMinRows - 1)
    int skip_from = 0;
    const bool wide = dv == 192 || dv == 256;                // one softmax map only: the accumulators of two would not fit
    if (act_dtype == B2_ACT_BF16 && T - n_seq >= kTileMinRows - 1 && dk % 32 == 0 && dv % 32 == 0 && dk <= 128 &&
        (dv <= 128 || (wide && maps == 1 && !sig)) &&
        b2_aligned16(q) && b2_aligned16(k_cache) && b2_aligned16(v_cache) && b2_aligned16(out) && out_stride % 8 == 0) {
        skip_from = kTileMinRows;
        int rc = B2_OK;
#define B2_TILE_RUN(a, b, SIG, MAPS)                                                                                      \
    launch_tile<a, b, SIG, MAPS>(q, k_cache, v_cache, block_tables, max_nb, cu_q, ctx_start, n_seq, T, H, G, bs, scale, chunk, \
                                 window, keep_first, sink, sink_logit, sink_logits, head_bias, gate, gate_stride, hs, out, \
                                 out_stride, st)
#define B2_TILE(a, b)                                                                                                     \
    if (dk == 16 * a && dv == 16 * b)                                                                                     \
        rc = sig ? B2_TILE_RUN(a, b, true, 1) : (maps == 2 ? B2_TILE_RUN(a, b, false, 2) : B2_TILE_RUN(a, b, false, 1));
#define B2_TILE_WIDE(a, b) if (dk == 16 * a && dv == 16 * b) rc = B2_TILE_RUN(a, b, false, 1);
        B2_TILE(2, 2) B2_TILE(2, 4) B2_TILE(2, 6) B2_TILE(2, 8) B2_TILE(4, 2) B2_TILE(4, 4) B2_TILE(4, 6) B2_TILE(4, 8)
        B2_TILE(6, 2) B2_TILE(6, 4) B2_TILE(6, 6) B2_TILE(6, 8) B2_TILE(8, 2) B2_TILE(8, 4) B2_TILE(8, 6) B2_TILE(8, 8)
        B2_TILE_WIDE(2, 12) B2_TILE_WIDE(4, 12) B2_TILE_WIDE(6, 12) B2_TILE_WIDE(8, 12)
        B2_TILE_WIDE(2, 16) B2_TILE_WIDE(4, 16) B2_TILE_WIDE(6, 16) B2_TILE_WIDE(8, 16)
#undef B2_TILE
#undef B2_TILE_WIDE
#undef B2_TILE_RUN
        if (rc != B2_OK) return rc;
    }
    if (act_dtype == B2_ACT_BF16 && dk % 32 == 0 && dk <= 256 && b2_aligned16(q) && b2_aligned16(k_cache) && b2_aligned16(v_cache)) {
        int rc = B2_EUNSUPPORTED;
#define B2_HEADS_RUN(b, SIG, MAPS)                                                                                        \
    launch_heads<b, SIG, MAPS>(q, k_cache, v_cache, block_tables, max_nb, cu_q, ctx_start, n_seq, T, H, G, dk, bs, scale, chunk, \
                               window, keep_first, sink, sink_logit, sink_logits, head_bias, gate, gate_stride, hs, skip_from, out, \
                               out_stride, st)
#define B2_HEADS(b) if (dv == 16 * b) rc = sig ? B2_HEADS_RUN(b, true, 1) : (maps == 2 ? B2_HEADS_RUN(b, false, 2) : B2_HEADS_RUN(b, false, 1));
        B2_HEADS(2) B2_HEADS(4) B2_HEADS(6) B2_HEADS(8) B2_HEADS(12) B2_HEADS(16)
#undef B2_HEADS
#undef B2_HEADS_RUN
        if (rc != B2_EUNSUPPORTED) return rc;
    }
    if (act_dtype == B2_ACT_BF16 && dk % 8 == 0 && dv % 8 == 0 && dv <= 64 * kGroupMaxPairs && b2_aligned16(q) &&
        b2_aligned16(k_cache) && b2_aligned16(v_cache) && b2_aligned16(out)) {
        const size_t gsm = (size_t)(kGroupMaxHeads * dk + 4 * kGroupMaxHeads * (2 + dv)) * sizeof(float) +
                           (size_t)4 * 32 * (maps * dk + 8 + dv) * sizeof(__nv_bfloat16);
        if (gsm <= 200 * 1024) {
            auto kern = sig ? chunk_attention_group_kernel<true, 1>
                            : (maps == 2 ? chunk_attention_group_kernel<false, 2> : chunk_attention_group_kernel<false, 1>);
            if (gsm > 48 * 1024) B2_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)gsm));
            kern<<<dim3(T, G), 128, gsm, st>>>(static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k_cache),
                                               static_cast<const __nv_bfloat16*>(v_cache), block_tables, max_nb, cu_q, ctx_start,
                                               n_seq, H, G, dk, dv, bs, scale, chunk, window, keep_first, sink, sink_logit,
                                               sink_logits, head_bias, static_cast<const __nv_bfloat16*>(gate), gate_stride, hs,
                                               skip_from, static_cast<__nv_bfloat16*>(out), out_stride);
            B2_CUDA_OK(cudaGetLastError());
            return B2_OK;
        }
    }
#define B2_WARP_ATTENTION(SIG, MAPS)                                                                                          \
    chunk_attention_kernel<A, SIG, MAPS><<<blocks, warps * 32, smem, st>>>(                                                   \
        static_cast<const A*>(q), static_cast<const A*>(k_cache), static_cast<const A*>(v_cache), block_tables, max_nb, cu_q, \
        ctx_start, n_seq, T, H, G, dk, dv, bs, scale, chunk, window, keep_first, sink, sink_logit, sink_logits, head_bias,    \
        static_cast<const A*>(gate), gate_stride, hs, skip_from, static_cast<A*>(out), out_stride)
    B2_DISPATCH_ACT(act_dtype, A, {
        if (sig) B2_WARP_ATTENTION(true, 1);
        else if (maps == 2) B2_WARP_ATTENTION(false, 2);
        else B2_WARP_ATTENTION(false, 1);
    });
#undef B2_WARP_ATTENTION
    B2_CUDA_OK(cudaGetLastError());
    return B2_OK;
}
