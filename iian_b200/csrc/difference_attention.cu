// Attention whose heads are the difference of two softmax maps over the same values, over a paged K/V cache.
//
// A query head has two maps, each with queries and keys of `d` entries of its own; both weigh the SAME values (`dv` entries):
//     s^m_ij = (q^m_i . k^m_j) * scale,  then  s <- cap * tanh(s / cap)  (cap 0: as it is);   key j visible iff j <= i
//     a^m_i = sum_j softmax(s^m)_ij v_j;     o = a^1 - lambda a^2;     o <- o / sqrt(mean(o^2) + eps) * factor
// Query head h reads key/value head h / (H / G).  A key cell of the cache holds both maps side by side: K [pages, G, page, 2 d],
// V [pages, G, page, dv]; query rows are [H][2][d].
//
// Kernels:
//   rotate_pairs_store     per token: rotation of the first `rot` entries of every map of q and k, entries 2i and 2i + 1 by angle
//                          i; q to the attention's rows, k and the values as projected to their cache cells.  A pair is a
//                          neighbour, so a thread works on 16 bytes by itself.
//   difference_attention   general form (any element type and sizes up to 512): one warp per (token, head) walks both maps over
//                          the same keys, in tiles of 32 that start at multiples of 32 of the ABSOLUTE key position, so the
//                          order of every sum depends on the token's own position only
#include "common.cuh"

namespace iian {

constexpr int kDaMaxDim = 512;
constexpr int kDaWarps = 4;

template <int U, typename A> __device__ __forceinline__ void da_load(const A * p, float * f) {
    if constexpr (U == 8) {
        unpack8(*reinterpret_cast<const uint4 *>(p), f);
    } else if constexpr (U == 4) {
        const float4 v = *reinterpret_cast<const float4 *>(p);
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
    } else {
        f[0] = to_f32(*p);
    }
}
template <int U, typename A> __device__ __forceinline__ void da_store(A * p, const float * f) {
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

// proj rows: q (nq sub-heads of d) at q_off, k (G * maps sub-heads of d) at k_off, v (G * dv) at v_off, row stride ld.
// q_out [N, nq * d]; K cache [pages, G, page_size, maps * d], V cache [pages, G, page_size, dv] (both null: q only).
// table: float2 [N, rot / 2] (cos, sin) or null.  Grid (N, blocks over a token's units of U entries).
template <int U, typename A>
__global__ void rotate_pairs_store_kernel(const A * __restrict__ proj, long long ld, int q_off, int k_off, int v_off,
                                          A * __restrict__ q_out, A * __restrict__ k_cache, A * __restrict__ v_cache,
                                          const float2 * __restrict__ table, const int * __restrict__ slots, int nq, int G, int maps,
                                          int d, int dv, int rot, int page_size, long long n_cells) {
    pdl_wait();
    pdl_launch_dependents();
    const size_t t = blockIdx.x;
    const int q_units = nq * d / U, k_units = k_cache != nullptr ? G * maps * d / U : 0, v_units = k_cache != nullptr ? G * dv / U : 0;
    int u = blockIdx.y * blockDim.x + threadIdx.x;
    if (u >= q_units + k_units + v_units) return;
    const A * row = proj + t * ld;
    const float2 * tab = table != nullptr ? table + t * (size_t) (rot / 2) : nullptr;
    long long cell = -1;
    if (u >= q_units) {
        cell = slots[t];
        if (cell < 0 || cell >= n_cells) return;             // padding token: nothing is stored
    }
    const long long page = cell >= 0 ? cell / page_size : 0, off = cell >= 0 ? cell % page_size : 0;
    float f[U];
    if (u >= q_units + k_units) {                            // values, as projected
        const int e = (u - q_units - k_units) * U;
        const int g = e / dv, c = e - g * dv;
        da_load<U>(row + v_off + e, f);
        da_store<U>(v_cache + ((page * G + g) * page_size + off) * dv + c, f);
        return;
    }
    const bool is_q = u < q_units;
    const int e = (is_q ? u : u - q_units) * U;
    const int c = e % d;                                     // place in the map
    const A * src = row + (is_q ? q_off : k_off) + e;
    da_load<U>(src, f);
    if (tab != nullptr && c < rot) {
        if constexpr (U == 1) {
            const float2 cs = tab[c >> 1];
            const float other = to_f32(src[(c & 1) ? -1 : 1]);
            f[0] = (c & 1) ? rot_hi(other, f[0], cs.x, cs.y) : rot_lo(f[0], other, cs.x, cs.y);
        } else {
#pragma unroll
            for (int i = 0; i < U; i += 2) {
                if (c + i < rot) {
                    const float2 cs = tab[(c + i) >> 1];
                    const float a = rot_lo(f[i], f[i + 1], cs.x, cs.y), b = rot_hi(f[i], f[i + 1], cs.x, cs.y);
                    f[i] = a;
                    f[i + 1] = b;
                }
            }
        }
    }
    if (is_q) {
        da_store<U>(q_out + t * (size_t) (nq * d) + e, f);
    } else {
        const int md = maps * d;
        const int g = e / md, cc = e - g * md;
        da_store<U>(k_cache + ((page * G + g) * page_size + off) * md + cc, f);
    }
}

// NV: registers of 32 columns of a value a lane holds; U: entries of a key read at once (16 bytes, or 1)
template <int NV, int U, typename A>
__global__ void __launch_bounds__(kDaWarps * 32)
difference_attention_kernel(const A * __restrict__ q, const A * __restrict__ k_cache, const A * __restrict__ v_cache, A * __restrict__ out,
                            const int * __restrict__ positions, const int * __restrict__ seq_of_token,
                            const int * __restrict__ block_table, int max_blocks, const int * __restrict__ ctx_len, int N, int H, int G,
                            int d, int dv, int page_size, int num_pages, float scale, float cap, float lambda, float factor, float eps) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ __align__(16) float qs[kDaWarps][2 * kDaMaxDim];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long) blockIdx.x * kDaWarps + warp;
    if (item >= (long long) N * H) return;
    const int t = (int) (item / H), h = (int) (item % H);
    const int g = h / (H / G);
    A * o = out + ((size_t) t * H + h) * dv;
    const int s = seq_of_token[t];
    if (s < 0) {                                             // padding token
        for (int c = lane; c < dv; c += 32) o[c] = from_f32<A>(0.0f);
        return;
    }
    int hi = positions[t];
    if (ctx_len != nullptr) hi = min(hi, ctx_len[s] - 1);
    const A * qp = q + ((size_t) t * H + h) * 2 * d;
    for (int c = lane; c < 2 * d; c += 32) qs[warp][c] = to_f32(qp[c]);
    __syncwarp();
    float acc[2][NV];
#pragma unroll
    for (int i = 0; i < NV; i++) acc[0][i] = acc[1][i] = 0.0f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
    const int * bt = block_table + (size_t) s * max_blocks;
    for (int kb = 0; kb <= hi; kb += 32) {
        const int j = kb + lane;
        bool valid = j <= hi;
        const A * kp = k_cache;
        const A * vp = nullptr;
        if (valid) {
            const int page = bt[j / page_size];
            if (page < 0 || page >= num_pages) {
                valid = false;
            } else {
                const size_t cell = ((size_t) page * G + g) * page_size + (j % page_size);
                kp = k_cache + cell * 2 * d;
                vp = v_cache + cell * dv;
            }
        }
        float p[2];
        bool any = false;
#pragma unroll
        for (int map = 0; map < 2; map++) {
            float sc = -INFINITY;
            if (valid) {
                float dot = 0.0f;
                for (int c = 0; c < d; c += U) {
                    float f[U];
                    da_load<U>(kp + map * d + c, f);
#pragma unroll
                    for (int i = 0; i < U; i++) dot = fmaf(qs[warp][map * d + c + i], f[i], dot);
                }
                sc = dot * scale;
                if (cap > 0.0f) sc = cap * tanhf(sc / cap);
            }
            const float tile_max = warp_max(sc);
            p[map] = 0.0f;
            if (tile_max == -INFINITY) continue;
            any = true;
            const float m_new = fmaxf(m[map], tile_max);
            p[map] = valid ? expf(sc - m_new) : 0.0f;
            const float corr = m[map] == -INFINITY ? 0.0f : expf(m[map] - m_new);
            l[map] = l[map] * corr + warp_sum(p[map]);
#pragma unroll
            for (int i = 0; i < NV; i++) acc[map][i] *= corr;
            m[map] = m_new;
        }
        if (!any) continue;
        for (int jj = 0; jj < 32; jj++) {
            const float p0 = __shfl_sync(0xffffffffu, p[0], jj), p1 = __shfl_sync(0xffffffffu, p[1], jj);
            const A * vrow = (const A *) __shfl_sync(0xffffffffu, (unsigned long long) vp, jj);
            if (vrow == nullptr) continue;
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int c = lane + 32 * i;
                if (c < dv) {
                    const float v = to_f32(vrow[c]);
                    acc[0][i] = fmaf(p0, v, acc[0][i]);
                    acc[1][i] = fmaf(p1, v, acc[1][i]);
                }
            }
        }
    }
    const float i0 = l[0] > 0.0f ? 1.0f / l[0] : 0.0f, i1 = l[1] > 0.0f ? lambda / l[1] : 0.0f;
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; i++) {
        acc[0][i] = acc[0][i] * i0 - acc[1][i] * i1;          // (columns beyond dv stay zero)
        ss = fmaf(acc[0][i], acc[0][i], ss);
    }
    ss = warp_sum(ss);
    const float r = factor / sqrtf(ss / (float) dv + eps);
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = lane + 32 * i;
        if (c < dv) o[c] = from_f32<A>(acc[0][i] * r);
    }
}

}  // namespace iian

using namespace iian;

IIAN_API int iian_rotate_pairs_store(const void * proj, long long ld, int q_off, int k_off, int v_off, void * q_out, void * k_cache,
                                     void * v_cache, const void * table, const int * slots, int act_dtype, int N, int nq, int G, int maps,
                                     int d, int dv, int rot, int page_size, long long n_cells, cudaStream_t stream) {
    if (N <= 0) return IIAN_OK;
    if (nq <= 0 || G < 0 || maps <= 0 || d <= 0 || dv <= 0 || rot < 0 || rot > d || (rot & 1) || page_size <= 0) return IIAN_ERR_SHAPE;
    if ((k_cache == nullptr) != (v_cache == nullptr) || (k_cache != nullptr && (slots == nullptr || G <= 0))) return IIAN_ERR_SHAPE;
    if (rot > 0 && table == nullptr) return IIAN_ERR_SHAPE;
    if (act_dtype != IIAN_F32 && act_dtype != IIAN_BF16) return IIAN_ERR_DTYPE;
    const int U = act_dtype == IIAN_F32 ? 4 : 8;
    const bool vec = d % U == 0 && dv % U == 0 && ld % U == 0 && q_off % U == 0 && k_off % U == 0 && v_off % U == 0 &&
                     (((uintptr_t) proj | (uintptr_t) q_out | (uintptr_t) k_cache | (uintptr_t) v_cache) & 15) == 0;
    const float2 * tab = rot > 0 ? (const float2 *) table : nullptr;
    const long long entries = (long long) nq * d + (k_cache != nullptr ? (long long) G * (maps * d + dv) : 0);
    const long long units = vec ? entries / U : entries;
    const int threads = units >= 256 ? 256 : (int) ((units + 31) / 32 * 32);
    const long long by = (units + threads - 1) / threads;
    if (by > 65535) return IIAN_ERR_LIMIT;
    const dim3 grid(N, (unsigned) by);
#define IIAN_ROT(U, A) iian_launch(rotate_pairs_store_kernel<U, A>, grid, dim3(threads), 0, stream, (const A *) proj, ld, q_off, k_off, v_off, \
                                   (A *) q_out, (A *) k_cache, (A *) v_cache, tab, slots, nq, G, maps, d, dv, rot, page_size, n_cells)
    if (act_dtype == IIAN_F32) return vec ? IIAN_ROT(4, float) : IIAN_ROT(1, float);
    return vec ? IIAN_ROT(8, __nv_bfloat16) : IIAN_ROT(1, __nv_bfloat16);
#undef IIAN_ROT
}

// q: [N, H, 2, d]; out: [N, H * dv]; cap 0: scores as they are.
IIAN_API int iian_difference_attention(const void * q, const void * k_cache, const void * v_cache, void * out, const int * positions,
                                       const int * seq_of_token, const int * block_table, int max_blocks, const int * ctx_len,
                                       int act_dtype, int N, int H, int G, int d, int dv, int page_size, int num_pages, float scale,
                                       float cap, float lambda, float factor, float eps, cudaStream_t stream) {
    if (N <= 0) return IIAN_OK;
    if (d <= 0 || d > kDaMaxDim || dv <= 0 || dv > kDaMaxDim || G <= 0 || H % G != 0 || page_size <= 0 || cap < 0.0f) return IIAN_ERR_SHAPE;
    if (act_dtype != IIAN_F32 && act_dtype != IIAN_BF16) return IIAN_ERR_DTYPE;
    const long long items = (long long) N * H;
    const unsigned blocks = (unsigned) ((items + kDaWarps - 1) / kDaWarps);
    const int U = act_dtype == IIAN_F32 ? 4 : 8;
    const bool vec = d % U == 0 && ((uintptr_t) k_cache & 15) == 0;
    const int nv = dv <= 64 ? 2 : dv <= 128 ? 4 : 16;
#define IIAN_DA(NV, U, A) return iian_launch(difference_attention_kernel<NV, U, A>, dim3(blocks), dim3(kDaWarps * 32), 0, stream, \
        (const A *) q, (const A *) k_cache, (const A *) v_cache, (A *) out, positions, seq_of_token, block_table, max_blocks, ctx_len, \
        N, H, G, d, dv, page_size, num_pages, scale, cap, lambda, factor, eps)
#define IIAN_DA_NV(U, A) do { if (nv == 2) IIAN_DA(2, U, A); if (nv == 4) IIAN_DA(4, U, A); IIAN_DA(16, U, A); } while (0)
    if (act_dtype == IIAN_F32) { if (vec) IIAN_DA_NV(4, float); IIAN_DA_NV(1, float); }
    if (vec) IIAN_DA_NV(8, __nv_bfloat16);
    IIAN_DA_NV(1, __nv_bfloat16);
#undef IIAN_DA_NV
#undef IIAN_DA
}
