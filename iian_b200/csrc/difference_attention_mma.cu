// Tensor-core form of attention whose heads are the difference of two softmax maps over the same values, for decoded tokens and
// short portions (bf16; maps of 64 entries, values of 128; see difference_attention.cu for the formula).
//
// A key cell holds both maps (128 entries), a value cell 128: a tile of 64 keys is two tiles of 64 x 128, the layout of plain heads
// of 128, and is fetched once for both maps.  A CTA owns up to 16 rows ((token, head) pairs that share a KV head) of one sequence
// and walks the keys in tiles of 64; its four warps are two per map, each with 32 keys of the tile, and keep a running (max, sum,
// output) of their own.  At the end the two warps of a map are merged through shared memory, the maps are subtracted, the row is
// divided by its root mean square and written.  With n_split > 1 the CTAs of a row tile are one thread-block cluster and each
// takes a part of the keys; a warp per row then merges the parts of both maps through distributed shared memory.
//
// Scores are kept in units of log2 behind scale and cap: t = cap * log2(e) * tanh(s * scale / cap), the hyperbolic tangent as
// 1 - 2 / (1 + e^2x) from the hardware's exponential and reciprocal (absolute error of a few 1e-7).
#include <cuda.h>

#include "paged_mma.cuh"
#include <cooperative_groups.h>

namespace iian {

namespace cg = cooperative_groups;

constexpr int DM_HD = 128;                      // entries of a key cell (two maps) and of a value cell
constexpr int DM_MAP = 64;

struct DiffParams {
    const __nv_bfloat16 * q;        // [N, nh, 2, 64]
    const __nv_bfloat16 * k_cache;  // [pages, nkv, page_size, 128]
    const __nv_bfloat16 * v_cache;  // [pages, nkv, page_size, 128]
    __nv_bfloat16 * out;            // [N, nh * 128]
    const int * cu_q;               // [S + 1]
    const int * ctx_len;            // [S]
    const int * block_table;        // [S, max_blocks]
    int max_blocks, nh, nkv, page_size, num_pages, n_split;
    float scale_log2;               // scale * log2(e), used without a cap
    float cap_in, cap_log2;         // scale / cap and cap * log2(e); cap_in 0: no cap
    float lambda, factor, eps;
    int * status;                   // {code, where}, zero before the launch; null: cp.async instead of TMA
};

template <bool CLUSTER, int STAGES, bool TMA>
__global__ void __launch_bounds__(128, STAGES == 2 ? 3 : 2) difference_decode_kernel(const DiffParams p, const __grid_constant__ KvMaps maps) {
    constexpr int NW = 4, BM = 16, HD = DM_HD;
    constexpr int CH = HD / 8, KS = DM_MAP / 16, DT = HD / 8;
    constexpr int TILE_BYTES = BN * HD * 2;
    extern __shared__ __align__(128) unsigned char smem_raw[];
    // (the swizzle of a TMA tile is a function of the address: tiles start on 1024-byte boundaries)
    unsigned char * smem = TMA ? (unsigned char *) (((uintptr_t) smem_raw + 1023) & ~(uintptr_t) 1023) : smem_raw;
    unsigned char * sQ = smem;                               // [16][128]
    unsigned char * sK = sQ + BM * HD * 2;                   // [STAGES][64][128]
    unsigned char * sV = sK + STAGES * TILE_BYTES;           // [STAGES][64][128]
    __shared__ long long s_cell[TMA ? 1 : STAGES][BN];
    __shared__ __align__(8) unsigned long long full_bar[STAGES];

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int g_ = lane >> 2, t_ = lane & 3;
    const int map = warp >> 1, kbase = (warp & 1) * 32;      // this warp's map and its first key of a tile
    const int kvh = blockIdx.y;
    const int s = blockIdx.z / p.n_split, split = blockIdx.z % p.n_split;
    const int G = p.nh / p.nkv;
    const int q0 = p.cu_q[s];
    const int q_len = p.cu_q[s + 1] - q0;
    const int ctx = p.ctx_len[s];
    const int pos0 = ctx - q_len;
    const int rows_total = q_len * G;
    const int row0 = blockIdx.x * BM;
    if (row0 >= rows_total) return;                          // (the same for every CTA of a cluster: they share the row tile)

    const int tok_min = row0 / G;
    const int tok_max = min(rows_total - 1, row0 + BM - 1) / G;
    const int k_hi = pos0 + tok_max;
    const int n_tiles = k_hi / BN + 1;
    const int per = (n_tiles + p.n_split - 1) / p.n_split;
    const int tile_begin = split * per;
    const int tile_end = min(n_tiles, tile_begin + per);
    const int n_my = max(0, tile_end - tile_begin);
    const int * bt = p.block_table + (size_t) s * p.max_blocks;

    // cp.async form: row bases are looked up into shared memory a tile ahead of the copies that use them
    const int page_shift = (p.page_size & (p.page_size - 1)) == 0 ? __ffs(p.page_size) - 1 : -1;
    auto lookup_rows = [&](int tile, int slot) {
        if (tid < BN) {
            const int j = tile * BN + tid;
            long long cell = -1;
            if (tile < tile_end && j <= k_hi) {
                const int blk = page_shift >= 0 ? j >> page_shift : j / p.page_size;
                const int page = bt[blk];
                if (page >= 0 && page < p.num_pages)
                    cell = (((long long) page * p.nkv + kvh) * p.page_size + (j - blk * p.page_size)) * HD;
            }
            s_cell[slot][tid] = cell;
        }
    };
    constexpr int ROWS_PER_PASS = NW * 32 / CH;
    const int ld_row = tid / CH, ld_ch = tid % CH;
    const unsigned ld_dst = swz<HD>(ld_row, ld_ch);
    auto load_kv = [&](int stage) {
        const unsigned dK = smem_u32(sK + stage * TILE_BYTES) + ld_dst;
        const unsigned dV = smem_u32(sV + stage * TILE_BYTES) + ld_dst;
#pragma unroll
        for (int i = 0; i < BN / ROWS_PER_PASS; i++) {
            const long long cell = s_cell[stage][ld_row + i * ROWS_PER_PASS];
            const bool valid = cell >= 0;
            const size_t off = valid ? (size_t) cell + ld_ch * 8 : 0;
            cp_async16(dK + i * ROWS_PER_PASS * HD * 2, p.k_cache + off, valid);
            cp_async16(dV + i * ROWS_PER_PASS * HD * 2, p.v_cache + off, valid);
        }
    };
    // TMA form: lane l of warp 0 fetches one box of a tile: half l & 1 of the cell, K or V by bit 1, page l >> 2 of the tile
    const int ld_half = lane & 1, ld_which = (lane >> 1) & 1, ld_pg = lane >> 2;
    const bool ld_lane = TMA && warp == 0 && ld_pg * p.page_size < BN;
    auto tma_page = [&](int tile) -> int {
        int page = p.num_pages;                              // out of range: the box is filled with zeros
        if (ld_lane && tile < tile_end) {
            const int j0 = tile * BN + ld_pg * p.page_size;
            if (j0 <= k_hi) {
                const int pg = bt[page_shift >= 0 ? j0 >> page_shift : j0 / p.page_size];
                if (pg >= 0 && pg < p.num_pages) page = pg;
            }
        }
        return page;
    };
    auto tma_issue = [&](int stage, int page) {              // warp 0, all lanes
        const unsigned bar = smem_u32(&full_bar[stage]);
        if (lane == 0) dk_expect_tx(bar, 2 * TILE_BYTES);
        __syncwarp();
        if (ld_lane) {
            unsigned char * base = (ld_which == 0 ? sK : sV) + stage * TILE_BYTES + ld_half * (BN * 128) + ld_pg * p.page_size * 128;
            dk_tma_4d(smem_u32(base), ld_which == 0 ? &maps.k : &maps.v, ld_half * 64, 0, kvh, page, bar);
        }
    };
    int pg_q[STAGES];
    if (TMA) {
        if (tid == 0) {
#pragma unroll
            for (int st = 0; st < STAGES; st++) dk_mbar_init(smem_u32(&full_bar[st]), 1);
            asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        }
#pragma unroll
        for (int st = 0; st < STAGES; st++) pg_q[st] = tma_page(tile_begin + st);
    } else if (n_my > 0) {
#pragma unroll
        for (int st = 0; st < STAGES; st++) lookup_rows(tile_begin + st, st);
    }

    float o[DT][4];
#pragma unroll
    for (int i = 0; i < DT; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
    int row_tok[2], row_ok[2];
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int R = row0 + g_ + 8 * h;
        row_ok[h] = R < rows_total;
        row_tok[h] = pos0 + (row_ok[h] ? R / G : 0);
    }
    const int pos_min = pos0 + tok_min;
    const bool rows_full = row0 + BM <= rows_total;

    pdl_wait();
    if (n_my > 0) {
        __syncthreads();
        for (int c = tid; c < BM * CH; c += NW * 32) {       // Q rows: both maps of a head are 128 neighbouring entries
            const int r = c / CH, ch = c % CH;
            const int R = row0 + r;
            const bool valid = R < rows_total;
            const int tok = valid ? R / G : 0, head = kvh * G + (valid ? R % G : 0);
            cp_async16(smem_u32(sQ + swz<HD>(r, ch)), p.q + ((size_t) (q0 + tok) * p.nh + head) * HD + ch * 8, valid);
        }
#pragma unroll
        for (int st = 0; st < STAGES - 1; st++) {            // the first STAGES - 1 tiles
            if (TMA) {
                if (st < n_my && warp == 0) tma_issue(st, pg_q[st]);
            } else {
                if (st < n_my) load_kv(st);
                cp_async_commit();
            }
        }
        unsigned qf[KS][4];
        int pg_next = TMA ? pg_q[STAGES - 1] : 0;
        bool failed = false;
        for (int i = 0; i < n_my; i++) {
            if (TMA) {
                if (i + STAGES - 1 < n_my && warp == 0) tma_issue((i + STAGES - 1) % STAGES, pg_next);
                pg_next = tma_page(tile_begin + i + STAGES);
                if (!dk_wait(smem_u32(&full_bar[i % STAGES]), (unsigned) (i / STAGES) & 1u)) failed = true;
                if (i == 0) {                                // the Q rows came by cp.async
                    cp_async_commit();
                    cp_async_wait<0>();
                    __syncthreads();
                }
            } else {
                if (i + STAGES - 1 < n_my) load_kv((i + STAGES - 1) % STAGES);
                cp_async_commit();
                cp_async_wait<STAGES - 1>();
                __syncthreads();
                lookup_rows(tile_begin + i + STAGES, i % STAGES);
            }
            if (i == 0) {
#pragma unroll
                for (int ks = 0; ks < KS; ks++)
                    ldmatrix_x4(qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3],
                                smem_u32(sQ + swz<HD>(lane & 15, map * (DM_MAP / 8) + ks * 2 + (lane >> 4))));
            }
            const unsigned char * tK = sK + (i % STAGES) * TILE_BYTES;
            const unsigned char * tV = sV + (i % STAGES) * TILE_BYTES;
            float sc[4][4];
#pragma unroll
            for (int n = 0; n < 4; n++) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.0f;
#pragma unroll
            for (int ks = 0; ks < KS; ks++) {
#pragma unroll
                for (int np = 0; np < 2; np++) {
                    unsigned b0, b1, b2, b3;
                    const int r = kbase + np * 16 + (lane & 7) + ((lane >> 4) << 3);
                    ldmatrix_x4(b0, b1, b2, b3, smem_u32(tK + kv_off<HD, TMA>(r, map * (DM_MAP / 8) + ks * 2 + ((lane >> 3) & 1))));
                    mma16816(sc[2 * np], qf[ks], b0, b1);
                    mma16816(sc[2 * np + 1], qf[ks], b2, b3);
                }
            }
            // ---- scale and cap, mask, online softmax (all in units of log2) -----------------------------------------
            const int key0 = (tile_begin + i) * BN + kbase;
#pragma unroll
            for (int nt = 0; nt < 4; nt++)
#pragma unroll
                for (int e = 0; e < 4; e++)
                    sc[nt][e] = p.cap_in > 0.0f ? p.cap_log2 * score_tanh(sc[nt][e] * p.cap_in) : sc[nt][e] * p.scale_log2;
            if (key0 + 31 > pos_min || !rows_full) {
#pragma unroll
                for (int nt = 0; nt < 4; nt++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int h = e >> 1;
                        const int j = key0 + nt * 8 + 2 * t_ + (e & 1);
                        if (!row_ok[h] || j > row_tok[h]) sc[nt][e] = -INFINITY;
                    }
            }
            float corr[2], neg[2], sum[2] = {0.0f, 0.0f};
#pragma unroll
            for (int h = 0; h < 2; h++) {
                float m = m_run[h];
#pragma unroll
                for (int nt = 0; nt < 4; nt++) m = fmaxf(m, fmaxf(sc[nt][2 * h], sc[nt][2 * h + 1]));
                m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 1));
                m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 2));
                corr[h] = m == -INFINITY ? 1.0f : exp2f(m_run[h] - m);          // m_run = -inf gives 0
                neg[h] = m == -INFINITY ? 0.0f : m;
                m_run[h] = m;
            }
#pragma unroll
            for (int nt = 0; nt < 4; nt++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int h = e >> 1;
                    const float pv = fast_exp2(sc[nt][e] - neg[h]);              // 2^-inf = 0 for masked keys
                    sc[nt][e] = pv;
                    sum[h] += pv;
                }
#pragma unroll
            for (int h = 0; h < 2; h++) l_run[h] = l_run[h] * corr[h] + sum[h];
            if (corr[0] != 1.0f || corr[1] != 1.0f) {
#pragma unroll
                for (int dt = 0; dt < DT; dt++) {
                    o[dt][0] *= corr[0]; o[dt][1] *= corr[0];
                    o[dt][2] *= corr[1]; o[dt][3] *= corr[1];
                }
            }
#pragma unroll
            for (int kk = 0; kk < 2; kk++) {
                unsigned a[4];
                a[0] = pack_bf16(sc[2 * kk][0], sc[2 * kk][1]);
                a[1] = pack_bf16(sc[2 * kk][2], sc[2 * kk][3]);
                a[2] = pack_bf16(sc[2 * kk + 1][0], sc[2 * kk + 1][1]);
                a[3] = pack_bf16(sc[2 * kk + 1][2], sc[2 * kk + 1][3]);
#pragma unroll
                for (int dp = 0; dp < DT / 2; dp++) {
                    unsigned b0, b1, b2, b3;
                    const int r = kbase + kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
                    ldmatrix_x4_trans(b0, b1, b2, b3, smem_u32(tV + kv_off<HD, TMA>(r, dp * 2 + (lane >> 4))));
                    mma16816(o[2 * dp], a, b0, b1);
                    mma16816(o[2 * dp + 1], a, b2, b3);
                }
            }
            if (TMA) {
                // a wait that gave up ends the walk for the whole CTA: the result is not valid, the status words say so
                if (__syncthreads_or(failed ? 1 : 0)) {
                    if (tid == 0 && p.status != nullptr) { p.status[0] = 12; p.status[1] = i; }
                    break;
                }
            } else {
                __syncthreads();
            }
        }
    }
    cp_async_wait<0>();
    pdl_launch_dependents();

    // ---- merge the two warps of each map, then subtract --------------------------------------------------------------
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
    }
    float * mo = reinterpret_cast<float *>(sK);              // [NW][16][128]   (stage memory is free now)
    float * ml = mo + NW * BM * HD;                          // [NW][16][2]
    float * cO = ml + NW * BM * 2;                           // [2 maps][16][128] unnormalised output of this CTA (cluster form)
    float * cML = cO + 2 * BM * HD;                          // [2 maps][16][2]   its max and sum
    static_assert((NW * BM * HD + NW * BM * 2 + 2 * BM * HD + 2 * BM * 2) * 4 <= 2 * 2 * TILE_BYTES, "the merge fits two stages");
    __syncthreads();
#pragma unroll
    for (int dt = 0; dt < DT; dt++) {
        const int d = dt * 8 + 2 * t_;
        *reinterpret_cast<float2 *>(mo + ((size_t) warp * BM + g_) * HD + d) = make_float2(o[dt][0], o[dt][1]);
        *reinterpret_cast<float2 *>(mo + ((size_t) warp * BM + g_ + 8) * HD + d) = make_float2(o[dt][2], o[dt][3]);
    }
    if (t_ == 0) {
        ml[(warp * BM + g_) * 2] = m_run[0];         ml[(warp * BM + g_) * 2 + 1] = l_run[0];
        ml[(warp * BM + g_ + 8) * 2] = m_run[1];     ml[(warp * BM + g_ + 8) * 2 + 1] = l_run[1];
    }
    __syncthreads();
    const int mr = tid >> 3, mpart = tid & 7;                // 8 threads per row, 16 columns each
    const int mR = row0 + mr;
    float w_a[2][2], m_map[2], l_map[2];
#pragma unroll
    for (int m = 0; m < 2; m++) {
        const float m0 = ml[((2 * m) * BM + mr) * 2], m1 = ml[((2 * m + 1) * BM + mr) * 2];
        m_map[m] = fmaxf(m0, m1);
        w_a[m][0] = m0 == -INFINITY ? 0.0f : exp2f(m0 - m_map[m]);
        w_a[m][1] = m1 == -INFINITY ? 0.0f : exp2f(m1 - m_map[m]);
        l_map[m] = w_a[m][0] * ml[((2 * m) * BM + mr) * 2 + 1] + w_a[m][1] * ml[((2 * m + 1) * BM + mr) * 2 + 1];
    }
    if constexpr (!CLUSTER) {
        const float i0 = l_map[0] > 0.0f ? 1.0f / l_map[0] : 0.0f, i1 = l_map[1] > 0.0f ? p.lambda / l_map[1] : 0.0f;
        float v[16], ss = 0.0f;
#pragma unroll
        for (int c = 0; c < 16; c += 4) {
            const size_t d = (size_t) mr * HD + mpart * 16 + c;
            float4 x[NW];
#pragma unroll
            for (int w = 0; w < NW; w++) x[w] = *reinterpret_cast<const float4 *>(mo + (size_t) w * BM * HD + d);
            v[c] = (w_a[0][0] * x[0].x + w_a[0][1] * x[1].x) * i0 - (w_a[1][0] * x[2].x + w_a[1][1] * x[3].x) * i1;
            v[c + 1] = (w_a[0][0] * x[0].y + w_a[0][1] * x[1].y) * i0 - (w_a[1][0] * x[2].y + w_a[1][1] * x[3].y) * i1;
            v[c + 2] = (w_a[0][0] * x[0].z + w_a[0][1] * x[1].z) * i0 - (w_a[1][0] * x[2].z + w_a[1][1] * x[3].z) * i1;
            v[c + 3] = (w_a[0][0] * x[0].w + w_a[0][1] * x[1].w) * i0 - (w_a[1][0] * x[2].w + w_a[1][1] * x[3].w) * i1;
#pragma unroll
            for (int k = 0; k < 4; k++) ss = fmaf(v[c + k], v[c + k], ss);
        }
#pragma unroll
        for (int x = 4; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);        // the row's eight threads
        if (mR < rows_total) {
            const float r = p.factor / sqrtf(ss / (float) HD + p.eps);
            unsigned w[8];
#pragma unroll
            for (int c = 0; c < 8; c++) w[c] = pack_bf16(v[2 * c] * r, v[2 * c + 1] * r);
            uint4 * dst = reinterpret_cast<uint4 *>(p.out + ((size_t) (q0 + mR / G) * p.nh + kvh * G + mR % G) * HD + mpart * 16);
            dst[0] = make_uint4(w[0], w[1], w[2], w[3]);
            dst[1] = make_uint4(w[4], w[5], w[6], w[7]);
        }
    } else {
#pragma unroll
    for (int m = 0; m < 2; m++) {
#pragma unroll
        for (int c = 0; c < 16; c += 4) {
            const size_t d = (size_t) mr * HD + mpart * 16 + c;
            const float4 a = *reinterpret_cast<const float4 *>(mo + (size_t) (2 * m) * BM * HD + d);
            const float4 b = *reinterpret_cast<const float4 *>(mo + (size_t) (2 * m + 1) * BM * HD + d);
            *reinterpret_cast<float4 *>(cO + (size_t) m * BM * HD + d) =
                make_float4(w_a[m][0] * a.x + w_a[m][1] * b.x, w_a[m][0] * a.y + w_a[m][1] * b.y, w_a[m][0] * a.z + w_a[m][1] * b.z,
                            w_a[m][0] * a.w + w_a[m][1] * b.w);
        }
        if (mpart == 0) { cML[(m * BM + mr) * 2] = m_map[m]; cML[(m * BM + mr) * 2 + 1] = l_map[m]; }
    }
    // Every CTA of the cluster gets here, so the barriers are complete.  A warp per row merges the parts of both maps.
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    const int ns = p.n_split, rank = (int) cluster.block_rank();
    const int n_rows = min(BM, rows_total - row0);
    for (int r = rank * NW + warp; r < n_rows; r += ns * NW) {
        float4 v[2];
#pragma unroll
        for (int m = 0; m < 2; m++) {
            // lane c holds part c's maximum and sum; the row's maximum over the parts by shuffles
            float mc = -INFINITY, lc = 0.0f;
            if (lane < ns) {
                const float * src = cluster.map_shared_rank(cML, lane) + (m * BM + r) * 2;
                mc = src[0];
                lc = src[1];
            }
            const float mx = warp_max(mc);
            const float fc = mc == -INFINITY ? 0.0f : exp2f(mc - mx);
            const float l = warp_sum(fc * lc);
            v[m] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            for (int c = 0; c < ns; c++) {                   // in the order of the parts, whatever their timing
                const float f = __shfl_sync(0xffffffffu, fc, c);
                const float4 x = *reinterpret_cast<const float4 *>(cluster.map_shared_rank(cO, c) + ((size_t) m * BM + r) * HD + 4 * lane);
                if (f == 0.0f) continue;
                v[m].x = fmaf(f, x.x, v[m].x); v[m].y = fmaf(f, x.y, v[m].y); v[m].z = fmaf(f, x.z, v[m].z); v[m].w = fmaf(f, x.w, v[m].w);
            }
            const float inv = l > 0.0f ? (m == 0 ? 1.0f : p.lambda) / l : 0.0f;
            v[m].x *= inv; v[m].y *= inv; v[m].z *= inv; v[m].w *= inv;
        }
        const float4 d = make_float4(v[0].x - v[1].x, v[0].y - v[1].y, v[0].z - v[1].z, v[0].w - v[1].w);
        const float ss = warp_sum(d.x * d.x + d.y * d.y + d.z * d.z + d.w * d.w);
        const float f = p.factor / sqrtf(ss / (float) HD + p.eps);
        const int R = row0 + r;
        const size_t ri = (size_t) (q0 + R / G) * p.nh + kvh * G + R % G;
        *reinterpret_cast<uint2 *>(p.out + ri * HD + 4 * lane) = make_uint2(pack_bf16(d.x * f, d.y * f), pack_bf16(d.z * f, d.w * f));
    }
    cluster.sync();                                          // nobody leaves while its shared memory is being read
    }
}

template <bool CLUSTER, int STAGES, bool TMA>
static int launch_diff(const DiffParams & p, const KvMaps & maps, int S, int max_rows, cudaStream_t stream) {
    const size_t smem = (size_t) 16 * DM_HD * 2 + 2 * STAGES * BN * DM_HD * 2 + (TMA ? 1024 : 0);
    auto kernel = difference_decode_kernel<CLUSTER, STAGES, TMA>;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int) smem);
        if (e == cudaSuccess && CLUSTER) e = cudaFuncSetAttribute(kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
        if (e != cudaSuccess) return 1000 + (int) e;
        configured = true;
    }
    const dim3 grid((max_rows + 15) / 16, p.nkv, S * p.n_split);
    if (!CLUSTER) return iian_launch(kernel, grid, dim3(128), smem, stream, p, maps);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(128);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = (unsigned) p.n_split;         // the parts of one row tile are consecutive in z
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, p, maps);
    return e == cudaSuccess ? IIAN_OK : 1000 + (int) e;
}

}  // namespace iian

using namespace iian;

// q [N, nh, 2, 64], caches [pages, nkv, page_size, 128], out [N, nh * 128], all bf16 and 16-byte aligned.  n_split 1 to 16: parts
// of the keys, merged inside a thread-block cluster.  cap 0: no cap (needs scale > 0); with a cap scale / cap must be positive.
// status: two ints on the device, zero before the launch, or null (then K and V come by cp.async instead of TMA).
IIAN_API int iian_difference_attention_mma(const void * q, const void * k_cache, const void * v_cache, void * out, const int * cu_q,
                                           const int * ctx_len, const int * block_table, int max_blocks, int S, int max_q_len, int nh,
                                           int nkv, int page_size, int num_pages, float scale, float cap, float lambda, float factor,
                                           float eps, int n_split, int * status, cudaStream_t stream) {
    if (S <= 0 || max_q_len <= 0) return IIAN_OK;
    if (nkv <= 0 || nh % nkv != 0 || page_size <= 0 || n_split < 1 || n_split > 16 || !(scale > 0.0f) || cap < 0.0f) return IIAN_ERR_SHAPE;
    if (((uintptr_t) q | (uintptr_t) k_cache | (uintptr_t) v_cache | (uintptr_t) out) & 15) return IIAN_ERR_ALIGN;
    if ((long long) S * n_split > 65535 || nkv > 65535) return IIAN_ERR_LIMIT;
    DiffParams p;
    p.q = (const __nv_bfloat16 *) q; p.k_cache = (const __nv_bfloat16 *) k_cache; p.v_cache = (const __nv_bfloat16 *) v_cache;
    p.out = (__nv_bfloat16 *) out; p.cu_q = cu_q; p.ctx_len = ctx_len; p.block_table = block_table; p.max_blocks = max_blocks;
    p.nh = nh; p.nkv = nkv; p.page_size = page_size; p.num_pages = num_pages; p.n_split = n_split;
    p.scale_log2 = scale * 1.4426950408889634f;
    p.cap_in = cap > 0.0f ? scale / cap : 0.0f;
    p.cap_log2 = cap * 1.4426950408889634f;
    p.lambda = lambda; p.factor = factor; p.eps = eps; p.status = status;
    const int max_rows = max_q_len * (nh / nkv);
    const bool tma = status != nullptr && (page_size == 8 || page_size == 16 || page_size == 32 || page_size == 64) && S * nkv >= 32;
    KvMaps maps = {};
    if (tma) {
        int rc = kv_map_for(k_cache, num_pages, nkv, page_size, &maps.k);
        if (rc == IIAN_OK) rc = kv_map_for(v_cache, num_pages, nkv, page_size, &maps.v);
        if (rc != IIAN_OK) return rc;
    }
    // unsplit keys: three stages (two CTAs per SM) unless that needs a wave of CTAs more than two stages (three per SM)
    bool deep = false;
    if (n_split == 1) {
        const int sms = decode_sm_count();
        const long long ctas = (long long) ((max_rows + 15) / 16) * nkv * S;
        const long long waves3 = (ctas + 2 * sms - 1) / (2 * sms), waves2 = (ctas + 3 * sms - 1) / (3 * sms);
        deep = waves3 * 100 <= waves2 * 115;
    }
    if (n_split > 1) return tma ? launch_diff<true, 2, true>(p, maps, S, max_rows, stream) : launch_diff<true, 2, false>(p, maps, S, max_rows, stream);
    if (deep) return tma ? launch_diff<false, 3, true>(p, maps, S, max_rows, stream) : launch_diff<false, 3, false>(p, maps, S, max_rows, stream);
    return tma ? launch_diff<false, 2, true>(p, maps, S, max_rows, stream) : launch_diff<false, 2, false>(p, maps, S, max_rows, stream);
}
