// Rotated attention over a paged K/V cache with a sliding window that may keep the first keys of the sequence, a sink in the
// softmax's denominator and a gate per head or per entry of the output.
//
//     key j is visible to position i  iff  j <= i and (window == 0 or i - j < window or j < keep_first)
//     s_ij = (q_i . k_j) * scale;   s <- cap tanh(s / cap) if given
//     p = softmax over the visible keys, the denominator also holding exp(sink_h) if given
//     o_i = sum_j p_ij v_j,  times sigmoid(gate) (one number per head, or one per entry)
//
// Keys have `dk` entries per head, values `dv` (they may differ).  Kept keys keep their true positions: they were rotated and
// stored like every other key, so nothing but the mask knows about them.
//
// Kernels:
//   rotary_table_scaled   cos and sin of position * frequency, the product and the functions in float64, both multiplied by a
//                         magnitude (frequency tables that were rescaled for long contexts bring one); float32 [N, half, 2]
//   rotate_unit_store     per token and head: rotation of the first `rot` entries of q and k (entry i with entry i + rot / 2),
//                         THEN optionally each head of q and k divided by its root mean square (no weight); q to the
//                         attention's rows, k and v (as projected) to their cache cells
//   head_norm_store       per token and head: q and k divided by their root mean square, times a weight per entry (optional); v,
//                         optionally mixed with another row of values, keep * v + share * first; q to the attention's rows, k and
//                         v to their cache cells.  A head is a group of lanes of a warp, 16 bytes a lane
//   window_attention      general form (any element type and sizes up to 512): one warp per (token, head), keys in tiles of 32
//                         that start at multiples of 32 of the ABSOLUTE key position, so the order of every sum depends on the
//                         token's own position only
#include "common.cuh"

namespace iian {

constexpr int kWaMaxDim = 512;
constexpr int kWaWarps = 4;

__global__ void rotary_table_scaled_kernel(const double * __restrict__ inv_freq, const int * __restrict__ positions,
                                           float2 * __restrict__ table, int half, long long total, double magnitude) {
    pdl_wait();
    pdl_launch_dependents();
    const long long idx = (long long) blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const int t = (int) (idx / half), p = (int) (idx % half);
    double sn, cs;
    sincos((double) positions[t] * inv_freq[p], &sn, &cs);
    table[idx] = make_float2((float) (cs * magnitude), (float) (sn * magnitude));
}

// proj rows: q (nh * dk) at q_off, k (nkv * dk) at k_off, v (nkv * dv) at v_off, row stride ld.  q_out: [N, nh, dk].
// caches: K [pages, nkv, page_size, dk], V [pages, nkv, page_size, dv]; k_cache == null: q only.
// table: float2 [N, rot / 2] (cos, sin) or null (no rotation).
template <typename A>
__global__ void rotate_unit_store_kernel(const A * __restrict__ proj, long long ld, int q_off, int k_off, int v_off,
                                         A * __restrict__ q_out, A * __restrict__ k_cache, A * __restrict__ v_cache,
                                         const float2 * __restrict__ table, const int * __restrict__ slots, int N, int nh, int nkv,
                                         int dk, int dv, int rot, int page_size, long long n_cells, float eps, int unit_norm) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float xs[kWaWarps][kWaMaxDim];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int per_token = nh + (k_cache != nullptr ? nkv : 0);
    const long long item = (long long) blockIdx.x * kWaWarps + warp;
    if (item >= (long long) N * per_token) return;
    const int t = (int) (item / per_token), hh = (int) (item % per_token);
    const bool is_q = hh < nh;
    const int g = is_q ? hh : hh - nh;
    const A * row = proj + (size_t) t * ld;
    A * dst;
    if (is_q) {
        dst = q_out + ((size_t) t * nh + g) * dk;
    } else {
        const long long cell = slots[t];
        if (cell < 0 || cell >= n_cells) return;            // padding token: nothing is stored
        const long long page = cell / page_size, off = cell % page_size;
        dst = k_cache + ((page * nkv + g) * page_size + off) * dk;
        const A * vs = row + v_off + (size_t) g * dv;
        A * vd = v_cache + ((page * nkv + g) * page_size + off) * dv;
        for (int d = lane; d < dv; d += 32) vd[d] = vs[d];
    }
    const A * src = row + (is_q ? q_off : k_off) + (size_t) g * dk;
    for (int d = lane; d < dk; d += 32) xs[warp][d] = to_f32(src[d]);
    __syncwarp();
    const int half = rot / 2;
    const float2 * tab = table != nullptr ? table + (size_t) t * half : nullptr;
    float ss = 0.0f;
    float vals[kWaMaxDim / 32];
#pragma unroll
    for (int i = 0; i < kWaMaxDim / 32; i++) {
        const int d = lane + 32 * i;
        float v = 0.0f;
        if (d < dk) {
            v = xs[warp][d];
            if (tab != nullptr && d < 2 * half) {
                if (d < half) {
                    const float2 cs = tab[d];
                    v = rot_lo(v, xs[warp][d + half], cs.x, cs.y);
                } else {
                    const float2 cs = tab[d - half];
                    v = rot_hi(xs[warp][d - half], v, cs.x, cs.y);
                }
            }
        }
        vals[i] = v;
        ss = fmaf(v, v, ss);
    }
    float inv = 1.0f;
    if (unit_norm) {
        ss = warp_sum(ss);
        inv = 1.0f / sqrtf(ss / (float) dk + eps);
    }
#pragma unroll
    for (int i = 0; i < kWaMaxDim / 32; i++) {
        const int d = lane + 32 * i;
        if (d < dk) dst[d] = from_f32<A>(vals[i] * inv);
    }
}

template <int U, typename A> __device__ __forceinline__ void wa_load(const A * p, float * f) {
    if constexpr (U == 8) {
        unpack8(*reinterpret_cast<const uint4 *>(p), f);
    } else if constexpr (U == 4) {
        const float4 v = *reinterpret_cast<const float4 *>(p);
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
    } else {
        f[0] = to_f32(*p);
    }
}
template <int U, typename A> __device__ __forceinline__ void wa_store(A * p, const float * f) {
    if constexpr (U == 8) {
        __nv_bfloat162 r[4];
#pragma unroll
        for (int i = 0; i < 4; i++) r[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
        *reinterpret_cast<uint4 *>(p) = *reinterpret_cast<uint4 *>(r);
    } else if constexpr (U == 4) {
        *reinterpret_cast<float4 *>(p) = make_float4(f[0], f[1], f[2], f[3]);
    } else {
        *p = from_f32<A>(f[0]);
    }
}

// proj rows as above.  q_weight, k_weight: float32 [dk], both or neither (no norm).  first: rows of nkv * dv values with row stride
// ld_first (null: v as projected).  U entries per access, up to R accesses a lane, L lanes per head (a power of two up to 32).
template <int U, int R, typename A>
__global__ void head_norm_store_kernel(const A * __restrict__ proj, long long ld, int q_off, int k_off, int v_off, A * __restrict__ q_out,
                                       A * __restrict__ k_cache, A * __restrict__ v_cache, const float * __restrict__ q_weight,
                                       const float * __restrict__ k_weight, const A * __restrict__ first, long long ld_first, float keep,
                                       float share, const int * __restrict__ slots, unsigned items, int nh, int nkv, int dk, int dv,
                                       int log_l, int page_size, int n_cells, float eps) {
    pdl_wait();
    pdl_launch_dependents();
    const int L = 1 << log_l;
    const unsigned item = blockIdx.x * (blockDim.x >> log_l) + (threadIdx.x >> log_l);
    const int lane = threadIdx.x & (L - 1);
    const unsigned per_token = nh + 2 * nkv;
    const bool live = item < items;                          // (every lane of a warp takes part in the sums)
    const unsigned tok = live ? item / per_token : 0;
    const int hh = live ? (int) (item - tok * per_token) : 0;
    const long long t = tok;
    const int kind = hh < nh ? 0 : hh < nh + nkv ? 1 : 2;    // query, key, value
    const int g = kind == 0 ? hh : kind == 1 ? hh - nh : hh - nh - nkv;
    const int n = kind == 2 ? dv : dk;
    const A * src = proj + t * ld + (kind == 0 ? q_off : kind == 1 ? k_off : v_off) + (long long) g * n;
    float f[R][U];
    float ss = 0.0f;
#pragma unroll
    for (int r = 0; r < R; r++) {
        const int c = (lane + r * L) * U;
#pragma unroll
        for (int i = 0; i < U; i++) f[r][i] = 0.0f;
        if (live && c < n) wa_load<U>(src + c, f[r]);
#pragma unroll
        for (int i = 0; i < U; i++) ss = fmaf(f[r][i], f[r][i], ss);
    }
    for (int o = L >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!live) return;
    A * dst;
    if (kind == 0) {
        dst = q_out + (t * nh + g) * (long long) dk;
    } else {
        const int cell = slots[t];
        if (cell < 0 || cell >= n_cells) return;             // padding token: nothing is stored
        const int page = cell / page_size;
        const long long row = ((long long) page * nkv + g) * page_size + (cell - page * page_size);
        dst = kind == 1 ? k_cache + row * dk : v_cache + row * dv;
    }
    const float * w = kind == 0 ? q_weight : kind == 1 ? k_weight : nullptr;
    const float inv = w != nullptr ? 1.0f / sqrtf(ss / (float) dk + eps) : 1.0f;
    const A * other = kind == 2 && first != nullptr ? first + t * ld_first + (long long) g * dv : nullptr;
#pragma unroll
    for (int r = 0; r < R; r++) {
        const int c = (lane + r * L) * U;
        if (c >= n) continue;
        if (w != nullptr) {
            if constexpr (U > 1) {                           // (the weights are 16-byte aligned and c a multiple of 4)
#pragma unroll
                for (int i = 0; i < U; i += 4) {
                    const float4 w4 = *reinterpret_cast<const float4 *>(w + c + i);
                    f[r][i] *= inv * w4.x; f[r][i + 1] *= inv * w4.y; f[r][i + 2] *= inv * w4.z; f[r][i + 3] *= inv * w4.w;
                }
            } else {
                f[r][0] *= inv * w[c];
            }
        } else if (other != nullptr) {
            float o[U];
            wa_load<U>(other + c, o);
#pragma unroll
            for (int i = 0; i < U; i++) f[r][i] = mixed_value(f[r][i], o[i], keep, share);
        }
        wa_store<U>(dst + c, f[r]);
    }
}

template <typename A>
__global__ void window_attention_kernel(
    const A * __restrict__ q, long long ld_q, const A * __restrict__ k_cache, const A * __restrict__ v_cache,
    A * __restrict__ out, const int * __restrict__ positions, const int * __restrict__ seq_of_token,
    const int * __restrict__ block_table, int max_blocks, const int * __restrict__ ctx_len,
    int N, int nh, int nkv, int dk, int dv, int page_size, int num_pages, float scale, float cap, int window, int keep_first,
    const float * __restrict__ sink, const A * __restrict__ gate, long long ld_gate, int gate_per_head) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float qs[kWaWarps][kWaMaxDim];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long) blockIdx.x * kWaWarps + warp;
    if (item >= (long long) N * nh) return;
    const int t = (int) (item / nh), h = (int) (item % nh);
    const int kvh = h / (nh / nkv);
    A * o = out + ((size_t) t * nh + h) * dv;
    const int s = seq_of_token[t];
    if (s < 0) {   // padding token
        for (int d = lane; d < dv; d += 32) o[d] = from_f32<A>(0.0f);
        return;
    }
    const int p = positions[t];
    int hi = p;
    if (ctx_len != nullptr) hi = min(hi, ctx_len[s] - 1);
    const int lo = window > 0 ? max(0, p - window + 1) : 0;
    const int kept = min(keep_first, lo);                    // keys [0, kept) are seen although the window has passed them
    const int lo_tile = (lo / 32) * 32;
    const int kept_end = ((kept + 31) / 32) * 32;            // first tile start at or behind the kept keys

    const A * qp = q + (size_t) t * ld_q + (size_t) h * dk;
    for (int d = lane; d < dk; d += 32) qs[warp][d] = to_f32(qp[d]);
    __syncwarp();

    constexpr int kAcc = kWaMaxDim / 32;
    float acc[kAcc];
#pragma unroll
    for (int i = 0; i < kAcc; i++) acc[i] = 0.0f;
    float m = -INFINITY, l = 0.0f;
    if (sink != nullptr) {       // the running softmax starts at the sink: maximum sink, sum 1, no value
        m = sink[h];
        l = 1.0f;
    }
    const int * bt = block_table + (size_t) s * max_blocks;

    for (int kb = 0; kb <= hi; kb += 32) {
        if (kb >= kept_end && kb < lo_tile) {
            kb = lo_tile - 32;                               // jump over the tiles between the kept keys and the window
            continue;
        }
        const int j = kb + lane;
        bool valid = j <= hi && (j >= lo || j < kept);
        const A * kp = nullptr;
        const A * vp = nullptr;
        if (valid) {
            const int page = bt[j / page_size];
            if (page < 0 || page >= num_pages) {
                valid = false;
            } else {
                const size_t cell = ((size_t) page * nkv + kvh) * page_size + (j % page_size);
                kp = k_cache + cell * dk;
                vp = v_cache + cell * dv;
            }
        }
        float sc = -INFINITY;
        if (valid) {
            float dot = 0.0f;
            for (int d = 0; d < dk; d++) dot = fmaf(qs[warp][d], to_f32(kp[d]), dot);
            sc = dot * scale;
            if (cap > 0.0f) sc = cap * tanhf(sc / cap);
        }
        const float tile_max = warp_max(sc);
        if (tile_max == -INFINITY) continue;
        const float m_new = fmaxf(m, tile_max);
        const float pj = valid ? expf(sc - m_new) : 0.0f;
        const float corr = (m == -INFINITY) ? 0.0f : expf(m - m_new);
        l = l * corr + warp_sum(pj);
#pragma unroll
        for (int i = 0; i < kAcc; i++) acc[i] *= corr;
        m = m_new;
        for (int jj = 0; jj < 32; jj++) {
            const float pjj = __shfl_sync(0xffffffffu, pj, jj);
            const unsigned long long vaddr = __shfl_sync(0xffffffffu, (unsigned long long) vp, jj);
            if (pjj == 0.0f) continue;
            const A * vrow = (const A *) vaddr;
#pragma unroll
            for (int i = 0; i < kAcc; i++) {
                const int d = lane + 32 * i;
                if (d < dv) acc[i] = fmaf(pjj, to_f32(vrow[d]), acc[i]);
            }
        }
    }
    float inv = l > 0.0f ? 1.0f / l : 0.0f;
    if (gate != nullptr && gate_per_head) inv *= 1.0f / (1.0f + expf(-to_f32(gate[(size_t) t * ld_gate + h])));
#pragma unroll
    for (int i = 0; i < kAcc; i++) {
        const int d = lane + 32 * i;
        if (d < dv) {
            float v = acc[i] * inv;
            if (gate != nullptr && !gate_per_head) v *= 1.0f / (1.0f + expf(-to_f32(gate[(size_t) t * ld_gate + h * dv + d])));
            o[d] = from_f32<A>(v);
        }
    }
}

}  // namespace iian

using namespace iian;

IIAN_API int iian_rotary_table_scaled(const double * inv_freq, const int * positions, void * table, int N, int half,
                                      double magnitude, cudaStream_t stream) {
    const long long total = (long long) N * half;
    if (total <= 0) return IIAN_OK;
    const int threads = 128;
    return iian_launch(rotary_table_scaled_kernel, dim3((unsigned) ((total + threads - 1) / threads)), dim3(threads), 0, stream,
                       inv_freq, positions, (float2 *) table, half, total, magnitude);
}

IIAN_API int iian_rotate_unit_store(const void * proj, long long ld, int q_off, int k_off, int v_off, void * q_out, void * k_cache,
                                    void * v_cache, const void * table, const int * slots, int act_dtype, int N, int nh, int nkv,
                                    int dk, int dv, int rot, int page_size, long long n_cells, float eps, int unit_norm,
                                    cudaStream_t stream) {
    if (N <= 0) return IIAN_OK;
    if (nh <= 0 || nkv < 0 || dk <= 0 || dk > kWaMaxDim || dv <= 0 || rot < 0 || rot > dk || (rot & 1) || page_size <= 0)
        return IIAN_ERR_SHAPE;
    if (k_cache != nullptr && (v_cache == nullptr || slots == nullptr || nkv <= 0)) return IIAN_ERR_SHAPE;
    if (rot > 0 && table == nullptr) return IIAN_ERR_SHAPE;
    const long long items = (long long) N * (nh + (k_cache != nullptr ? nkv : 0));
    const unsigned blocks = (unsigned) ((items + kWaWarps - 1) / kWaWarps);
    const float2 * tab = rot > 0 ? (const float2 *) table : nullptr;
    if (act_dtype == IIAN_F32)
        return iian_launch(rotate_unit_store_kernel<float>, dim3(blocks), dim3(kWaWarps * 32), 0, stream, (const float *) proj, ld,
                           q_off, k_off, v_off, (float *) q_out, (float *) k_cache, (float *) v_cache, tab, slots, N, nh, nkv, dk, dv,
                           rot, page_size, n_cells, eps, unit_norm);
    if (act_dtype == IIAN_BF16)
        return iian_launch(rotate_unit_store_kernel<__nv_bfloat16>, dim3(blocks), dim3(kWaWarps * 32), 0, stream,
                           (const __nv_bfloat16 *) proj, ld, q_off, k_off, v_off, (__nv_bfloat16 *) q_out, (__nv_bfloat16 *) k_cache,
                           (__nv_bfloat16 *) v_cache, tab, slots, N, nh, nkv, dk, dv, rot, page_size, n_cells, eps, unit_norm);
    return IIAN_ERR_DTYPE;
}

// proj rows: q (nh * dk) at q_off, k (nkv * dk) at k_off, v (nkv * dv) at v_off, row stride ld.  q_out [N, nh, dk]; caches
// K [pages, nkv, page_size, dk], V [pages, nkv, page_size, dv].  q_weight, k_weight f32 [dk] or both null; first: rows of nkv * dv with
// row stride ld_first, or null: v <- keep * v + share * first.
IIAN_API int iian_head_norm_store(const void * proj, long long ld, int q_off, int k_off, int v_off, void * q_out, void * k_cache,
                                  void * v_cache, const float * q_weight, const float * k_weight, const void * first, long long ld_first,
                                  float keep, float share, const int * slots, int act_dtype, int N, int nh, int nkv, int dk, int dv,
                                  int page_size, long long n_cells, float eps, cudaStream_t stream) {
    if (N <= 0) return IIAN_OK;
    if (nh <= 0 || nkv <= 0 || dk <= 0 || dk > kWaMaxDim || dv <= 0 || dv > kWaMaxDim || page_size <= 0) return IIAN_ERR_SHAPE;
    if (k_cache == nullptr || v_cache == nullptr || slots == nullptr || (q_weight == nullptr) != (k_weight == nullptr)) return IIAN_ERR_SHAPE;
    if (act_dtype != IIAN_F32 && act_dtype != IIAN_BF16) return IIAN_ERR_DTYPE;
    const int full = act_dtype == IIAN_F32 ? 4 : 8;
    const bool vec = dk % full == 0 && dv % full == 0 && ld % full == 0 && q_off % full == 0 && k_off % full == 0 && v_off % full == 0 &&
                     ld_first % full == 0 &&
                     (((uintptr_t) proj | (uintptr_t) q_out | (uintptr_t) k_cache | (uintptr_t) v_cache | (uintptr_t) first |
                       (uintptr_t) q_weight | (uintptr_t) k_weight) & 15) == 0;
    const int U = vec ? full : 1;
    const int units = ((dk > dv ? dk : dv) + U - 1) / U;
    int log_l = 0;
    while ((1 << log_l) < units && log_l < 5) log_l++;
    const int L = 1 << log_l, R = (units + L - 1) / L;
    const long long items = (long long) N * (nh + 2 * nkv);
    if (items > (1LL << 30) || n_cells > 2147483647LL) return IIAN_ERR_LIMIT;
    const unsigned blocks = (unsigned) ((items * L + 255) / 256);
#define IIAN_HNS(U, R, A) return iian_launch(head_norm_store_kernel<U, R, A>, dim3(blocks), dim3(256), 0, stream, (const A *) proj, ld, q_off, \
        k_off, v_off, (A *) q_out, (A *) k_cache, (A *) v_cache, q_weight, k_weight, (const A *) first, ld_first, keep, share, slots, (unsigned) items, \
        nh, nkv, dk, dv, log_l, page_size, (int) n_cells, eps)
    if (act_dtype == IIAN_F32) {
        if (vec && R == 1) IIAN_HNS(4, 1, float);
        if (vec) IIAN_HNS(4, 4, float);
        IIAN_HNS(1, 16, float);
    }
    if (vec && R == 1) IIAN_HNS(8, 1, __nv_bfloat16);
    if (vec) IIAN_HNS(8, 2, __nv_bfloat16);
    IIAN_HNS(1, 16, __nv_bfloat16);
#undef IIAN_HNS
}

// q: rows of nh * dk with row stride ld_q; out: [N, nh * dv]; sink: float32 [nh] or null; gate: rows with row stride ld_gate
// holding nh numbers (gate_per_head) or nh * dv, or null.  cap: 0 = scores as they are.  window: 0 = every earlier key; keep_first
// only with a window.
IIAN_API int iian_window_attention(const void * q, long long ld_q, const void * k_cache, const void * v_cache, void * out,
                                   const int * positions, const int * seq_of_token, const int * block_table, int max_blocks,
                                   const int * ctx_len, int act_dtype, int N, int nh, int nkv, int dk, int dv, int page_size,
                                   int num_pages, float scale, float cap, int window, int keep_first, const float * sink,
                                   const void * gate, long long ld_gate, int gate_per_head, cudaStream_t stream) {
    if (N <= 0) return IIAN_OK;
    if (dk <= 0 || dk > kWaMaxDim || dv <= 0 || dv > kWaMaxDim || nkv <= 0 || nh % nkv != 0 || page_size <= 0 || window < 0 ||
        keep_first < 0 || cap < 0.0f) return IIAN_ERR_SHAPE;
    const long long items = (long long) N * nh;
    const unsigned blocks = (unsigned) ((items + kWaWarps - 1) / kWaWarps);
    if (act_dtype == IIAN_F32)
        return iian_launch(window_attention_kernel<float>, dim3(blocks), dim3(kWaWarps * 32), 0, stream, (const float *) q, ld_q,
                           (const float *) k_cache, (const float *) v_cache, (float *) out, positions, seq_of_token, block_table,
                           max_blocks, ctx_len, N, nh, nkv, dk, dv, page_size, num_pages, scale, cap, window, keep_first, sink,
                           (const float *) gate, ld_gate, gate_per_head);
    if (act_dtype == IIAN_BF16)
        return iian_launch(window_attention_kernel<__nv_bfloat16>, dim3(blocks), dim3(kWaWarps * 32), 0, stream,
                           (const __nv_bfloat16 *) q, ld_q, (const __nv_bfloat16 *) k_cache, (const __nv_bfloat16 *) v_cache,
                           (__nv_bfloat16 *) out, positions, seq_of_token, block_table, max_blocks, ctx_len, N, nh, nkv, dk, dv,
                           page_size, num_pages, scale, cap, window, keep_first, sink, (const __nv_bfloat16 *) gate, ld_gate,
                           gate_per_head);
    return IIAN_ERR_DTYPE;
}
