// The flash attention kernel and its launcher template (instantiated by prefill.cu and flash_ragged.cu).
#pragma once

#include "prefill.cuh"

namespace cb {

// -------------------------------------------------------------------------------------
// Flash attention forward (prefill + ViT): 64 query rows x one head per CTA, 64-key tiles,
// bf16 mma.sync m16n8k16 with f32 accumulation and an online (base-2) softmax.
// Keys/values come either from KV pages (one tile == one page) or from a strided buffer.
// -------------------------------------------------------------------------------------
__device__ __forceinline__ void ldmatrix_x4(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16_16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, int src_bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(src_bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// SPLIT: q, k, v (and the probabilities) are hi + lo bf16 pairs; every product keeps its three leading terms
//   S = qh.kh + qh.kl + ql.kh          O += ph.vh + ph.vl + pl.vh
// so the result carries ~16 mantissa bits instead of 8 (the f32-oracle parity mode; 3x the tensor work of 4 % of the flops).
// RAGGED: D and DV are the tile's widths, the operands' own come at run time (k_w, v_w, dv; columns past them are filled with zeros).
template <int D, int DV, bool CAUSAL, bool PAGED, bool SPLIT, bool RAGGED = false>
__global__ void __launch_bounds__(256, D == 64 && DV == 64 ? 2 : 1)
flash_prefill_kernel(FlashArgs a) {
    pdl_wait();
    pdl_launch_dependents();
    constexpr int BM = 64;
    constexpr int DM = D > DV ? D : DV;
    constexpr int BN = DM > 256 ? 16 : (SPLIT || DM > 128) ? 32 : 64;     // smaller key tiles wherever a 64-key tile x 2 groups x 2 stages would not fit
    constexpr int STG = (SPLIT && DM > 128) ? 1 : 2;      // stages per group (D = 256 with hi + lo planes: one)
    constexpr int LDS = D + 8;                 // padded row (elements): conflict-free ldmatrix
    constexpr int LDV = DV + 8;
    constexpr int TILE = BN * LDS, TILEV = BN * LDV;      // elements per K / V tile plane
    constexpr int CPR = D / 8, CPV = DV / 8;   // 16-byte chunks per K / V row
    constexpr int P = SPLIT ? 2 : 1;           // planes per operand
    constexpr int STAGE = P * (TILE + TILEV);  // K hi | K lo | V hi | V lo
    extern __shared__ __align__(16) unsigned char fsm[];
    bf16* q_s = reinterpret_cast<bf16*>(fsm);  // [P][BM x LDS]
    bf16* kv_s = q_s + P * BM * LDS;           // [2 groups][STG][K hi | K lo | V hi | V lo]

    // Two groups of four warps work on the SAME 64 query rows: group 0 takes the even key tiles, group 1 the odd ones, each through
    // its own double-buffered tile ring, and the two online-softmax states are merged at the end.
    // A causal CTA's critical path -- q tile i needs i + 1 key tiles, the last one 8 at 454 rows -- is halved that way.
    const int tid = threadIdx.x, lane = tid & 31, grp = tid >> 7, gtid = tid & 127, warp = (tid >> 5) & 3;
    const int g = lane >> 2, tq = lane & 3;
    const int head = blockIdx.y, z = blockIdx.z;
    const int row0 = a.seq_start ? a.seq_start[z] : 0;
    const int S = a.seq_len ? a.seq_len[z] : a.S;
    const int q0 = blockIdx.x * BM;
    if (q0 >= S) return;
    const int kv_off = CAUSAL ? (a.seq_kv_offset ? a.seq_kv_offset[z] : a.kv_offset) : 0;
    const int T = CAUSAL ? (kv_off + S) : S;   // keys available
    const int* btab = (PAGED && a.seq_slot) ? a.block_table + (size_t)a.seq_slot[z] * a.bt_stride : a.block_table;
    const int kvh = head / (a.nh / a.nkv);
    const int kw = RAGGED ? a.k_w : D, vw = RAGGED ? a.v_w : DV;          // row widths of keys (and of a query head) and of values
    const int nkh = RAGGED && a.k_heads ? a.k_heads : a.nkv, kkh = RAGGED ? head / (a.nh / nkh) : kvh;
    const int n_tiles = CAUSAL ? min((T + BN - 1) / BN, (kv_off + q0 + BM - 1) / BN + 1) : (T + BN - 1) / BN;
    // sliding window: the first query row of the tile is the one that reaches furthest back
    const int t_first = (CAUSAL && a.window > 0) ? max(0, kv_off + q0 - a.window + 1) / BN : 0;

    // ---- Q tile -> smem (zero-fill rows past S) ----
    for (int c = tid; c < BM * CPR; c += 256) {
        const int r = c / CPR, ch = c % CPR;
        const int qr = q0 + r;
        const bool in = qr < S && (!RAGGED || ch * 8 < kw);
        const bf16* src = a.q + (size_t)(row0 + min(qr, S - 1)) * a.q_stride + head * kw + (!RAGGED || in ? ch * 8 : 0);
        cp_async16(smem_u32(q_s + r * LDS + ch * 8), src, in ? 16 : 0);
        if (SPLIT) cp_async16(smem_u32(q_s + BM * LDS + r * LDS + ch * 8), src + a.q_lo_off, in ? 16 : 0);
    }
    auto load_kv = [&](int tile, int stage) {
        bf16* ks = kv_s + (grp * STG + stage) * STAGE;
        bf16* vs = ks + P * TILE;
        const int kv0 = tile * BN;
        if constexpr (RAGGED || D != DV) {                // (paged launches only)
            const size_t page = (size_t)btab[kv0 / KV_PAGE], base = (page * nkh + kkh) * KV_PAGE + (kv0 % KV_PAGE), vbase = (page * a.nkv + kvh) * KV_PAGE + (kv0 % KV_PAGE);
            for (int c = gtid; c < BN * CPR; c += 128) {
                const int r = c / CPR, ch = c % CPR, sz = kv0 + r < T && (!RAGGED || ch * 8 < kw) ? 16 : 0;
                const bf16* src = a.k_pool + (base + r) * kw + (!RAGGED || sz ? ch * 8 : 0);
                cp_async16(smem_u32(ks + r * LDS + ch * 8), src, sz);
                if (SPLIT) cp_async16(smem_u32(ks + TILE + r * LDS + ch * 8), src + a.kv_lo_off, sz);
            }
            for (int c = gtid; c < BN * CPV; c += 128) {
                const int r = c / CPV, ch = c % CPV, sz = kv0 + r < T && (!RAGGED || ch * 8 < vw) ? 16 : 0;
                const bf16* src = a.v_pool + (vbase + r) * vw + (!RAGGED || sz ? ch * 8 : 0);
                cp_async16(smem_u32(vs + r * LDV + ch * 8), src, sz);
                if (SPLIT) cp_async16(smem_u32(vs + TILEV + r * LDV + ch * 8), src + a.kv_lo_off, sz);
            }
            return;
        }
        for (int c = gtid; c < BN * CPR; c += 128) {
            const int r = c / CPR, ch = c % CPR;
            const int t = kv0 + r;
            const bool ok = t < T;
            const bf16 *ksrc, *vsrc;
            if (PAGED) {
                const int page = btab[kv0 / KV_PAGE];     // a tile is a whole page or an aligned half of one
                const size_t off = (((size_t)page * a.nkv + kvh) * KV_PAGE + (kv0 % KV_PAGE) + r) * D + ch * 8;
                ksrc = a.k_pool + off; vsrc = a.v_pool + off;
            } else {
                const size_t off = (size_t)(row0 + (ok ? t : 0)) * a.kv_stride + kvh * D + ch * 8;
                ksrc = a.k + off; vsrc = a.v + off;
            }
            cp_async16(smem_u32(ks + r * LDS + ch * 8), ksrc, ok ? 16 : 0);
            cp_async16(smem_u32(vs + r * LDS + ch * 8), vsrc, ok ? 16 : 0);
            if (SPLIT) {
                cp_async16(smem_u32(ks + TILE + r * LDS + ch * 8), ksrc + a.kv_lo_off, ok ? 16 : 0);
                cp_async16(smem_u32(vs + TILE + r * LDS + ch * 8), vsrc + a.kv_lo_off, ok ? 16 : 0);
            }
        }
    };
    cp_async_commit();
    cp_async_wait<0>();
    __syncthreads();                           // the Q tile is complete for both groups
    auto group_sync = [&]() { asm volatile("bar.sync %0, 128;" ::"r"(1 + grp) : "memory"); };

    float o_acc[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) { o_acc[i][0] = o_acc[i][1] = o_acc[i][2] = o_acc[i][3] = 0.f; }
    float m_row[2] = {-INFINITY, -INFINITY}, l_row[2] = {0.f, 0.f};
    const float sl2 = a.scale * 1.4426950408889634f;
    const bool mods = CAUSAL && (a.softcap > 0.f || a.dist_r1 || a.dist_table);
    const float inv_cap = a.softcap > 0.f ? 1.f / a.softcap : 0.f;
    const float dr1 = (CAUSAL && a.dist_r1) ? a.dist_r1[head] : 0.f, dr2 = (CAUSAL && a.dist_r1) ? a.dist_r2[head] : 0.f;
    const float* dtab = (CAUSAL && a.dist_table) ? a.dist_table + (size_t)head * a.dist_rows : nullptr;
    uint32_t qf[SPLIT ? 1 : D / 16][4];        // plain mode keeps the Q fragments in registers; SPLIT re-reads them from smem

    bool first = true;
    // the tiles of the kept first keys that the window does not reach come first, then the window's own
    const int keep = (CAUSAL && a.window > 0) ? a.keep_first : 0, n_keep = min((keep + BN - 1) / BN, t_first), n_walk = n_keep + n_tiles - t_first;
    auto tile_at = [&](int i) { return i < n_keep ? i : t_first + i - n_keep; };
    if (grp < n_walk) load_kv(tile_at(grp), 0);
    cp_async_commit();
    int it = 0;
    for (int ti = grp; ti < n_walk; ti += 2, ++it) {
        const int tile = tile_at(ti), stage = STG == 2 ? (it & 1) : 0;
        if (STG == 2) {
            if (ti + 2 < n_walk) load_kv(tile_at(ti + 2), stage ^ 1);
            cp_async_commit();
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        group_sync();
        if (!SPLIT && first) {
#pragma unroll
            for (int kk = 0; kk < D / 16; ++kk) {
                const int r = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
                const int c = kk * 16 + (lane >> 4) * 8;
                ldmatrix_x4(qf[SPLIT ? 0 : kk][0], qf[SPLIT ? 0 : kk][1], qf[SPLIT ? 0 : kk][2], qf[SPLIT ? 0 : kk][3], smem_u32(q_s + r * LDS + c));
            }
        }
        const bf16* ks = kv_s + (grp * STG + stage) * STAGE;
        const bf16* vs = ks + P * TILE;
        // ---- S = Q K^T ----
        float s_acc[BN / 8][4];
#pragma unroll
        for (int j = 0; j < BN / 8; ++j) { s_acc[j][0] = s_acc[j][1] = s_acc[j][2] = s_acc[j][3] = 0.f; }
        if constexpr (!SPLIT) {
#pragma unroll
            for (int j = 0; j < BN / 8; ++j) {
#pragma unroll
                for (int kk = 0; kk < D / 16; kk += 2) {
                    uint32_t b0, b1, b2, b3;
                    const int r = j * 8 + (lane & 7);
                    const int c = kk * 16 + (lane >> 3) * 8;
                    ldmatrix_x4(b0, b1, b2, b3, smem_u32(ks + r * LDS + c));
                    mma_bf16_16816(s_acc[j], qf[SPLIT ? 0 : kk], b0, b1);
                    mma_bf16_16816(s_acc[j], qf[SPLIT ? 0 : kk + 1], b2, b3);
                }
            }
        } else {
#pragma unroll 1
            for (int kk = 0; kk < D / 16; kk += 2) {
                uint32_t qh0[4], qh1[4], ql0[4], ql1[4];
                {
                    const int r = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
                    const int c = kk * 16 + (lane >> 4) * 8;
                    ldmatrix_x4(qh0[0], qh0[1], qh0[2], qh0[3], smem_u32(q_s + r * LDS + c));
                    ldmatrix_x4(qh1[0], qh1[1], qh1[2], qh1[3], smem_u32(q_s + r * LDS + c + 16));
                    ldmatrix_x4(ql0[0], ql0[1], ql0[2], ql0[3], smem_u32(q_s + BM * LDS + r * LDS + c));
                    ldmatrix_x4(ql1[0], ql1[1], ql1[2], ql1[3], smem_u32(q_s + BM * LDS + r * LDS + c + 16));
                }
#pragma unroll
                for (int j = 0; j < BN / 8; ++j) {
                    uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
                    const int r = j * 8 + (lane & 7);
                    const int c = kk * 16 + (lane >> 3) * 8;
                    ldmatrix_x4(h0, h1, h2, h3, smem_u32(ks + r * LDS + c));
                    ldmatrix_x4(l0, l1, l2, l3, smem_u32(ks + TILE + r * LDS + c));
                    mma_bf16_16816(s_acc[j], ql0, h0, h1);      // small terms first
                    mma_bf16_16816(s_acc[j], ql1, h2, h3);
                    mma_bf16_16816(s_acc[j], qh0, l0, l1);
                    mma_bf16_16816(s_acc[j], qh1, l2, l3);
                    mma_bf16_16816(s_acc[j], qh0, h0, h1);
                    mma_bf16_16816(s_acc[j], qh1, h2, h3);
                }
            }
        }
        // ---- mask + online softmax (rows g and g+8 of this warp's 16) ----
        const int kv0 = tile * BN;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < BN / 8; ++j) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int col = kv0 + j * 8 + tq * 2 + (e & 1);
                const int qrow = q0 + warp * 16 + g + (e >> 1) * 8;
                const bool vis = (col < T) && (!CAUSAL || (col <= kv_off + qrow && (a.window <= 0 || kv_off + qrow - col < a.window || col < keep)));
                float v = vis ? s_acc[j][e] * sl2 : -INFINITY;
                if (CAUSAL && mods && vis) {          // cap, then the distance terms, in f32 on the scaled score
                    float sc = s_acc[j][e] * a.scale;
                    const int dist = kv_off + qrow - col;
                    if (a.softcap > 0.f) {            // tanh(x) = 1 - 2 / (e^{2x} + 1), with the hardware exponential and reciprocal (1e-7 of the cap)
                        const float t = __expf(fminf(2.f * sc * inv_cap, 40.f));      // (tanh(20) is 1 to the last bit; no overflow into the reciprocal)
                        sc = a.softcap * (1.f - __fdividef(2.f, t + 1.f));
                    }
                    if (a.dist_r1) sc -= dr1 * log1pf(dr2 * (float)dist);
                    if (dtab) sc += dtab[min(dist, a.dist_rows - 1)];
                    v = sc * 1.4426950408889634f;
                }
                s_acc[j][e] = v;
                mx[e >> 1] = fmaxf(mx[e >> 1], v);
            }
        }
        float corr[2], muse[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            const float mn = fmaxf(m_row[r], mx[r]);
            muse[r] = (mn == -INFINITY) ? 0.f : mn;
            corr[r] = exp2f(m_row[r] - muse[r]);      // m_row = -inf -> 0
            m_row[r] = mn;
            l_row[r] *= corr[r];
        }
        float ps[2] = {0.f, 0.f};
#pragma unroll
        for (int j = 0; j < BN / 8; ++j) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float p = exp2f(s_acc[j][e] - muse[e >> 1]);
                s_acc[j][e] = p;
                ps[e >> 1] += p;
            }
        }
        l_row[0] += ps[0];
        l_row[1] += ps[1];
#pragma unroll
        for (int i = 0; i < DV / 8; ++i) {
            o_acc[i][0] *= corr[0]; o_acc[i][1] *= corr[0];
            o_acc[i][2] *= corr[1]; o_acc[i][3] *= corr[1];
        }
        // ---- O += P V ----
#pragma unroll
        for (int kt = 0; kt < BN / 16; ++kt) {
            uint32_t pa[4], pl[4];
            split_bf16x2(s_acc[2 * kt][0], s_acc[2 * kt][1], pa[0], pl[0]);
            split_bf16x2(s_acc[2 * kt][2], s_acc[2 * kt][3], pa[1], pl[1]);
            split_bf16x2(s_acc[2 * kt + 1][0], s_acc[2 * kt + 1][1], pa[2], pl[2]);
            split_bf16x2(s_acc[2 * kt + 1][2], s_acc[2 * kt + 1][3], pa[3], pl[3]);
#pragma unroll
            for (int dj = 0; dj < DV / 8; dj += 2) {
                uint32_t b0, b1, b2, b3;
                const int r = kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
                const int c = dj * 8 + (lane >> 4) * 8;
                ldmatrix_x4_trans(b0, b1, b2, b3, smem_u32(vs + r * LDV + c));
                if constexpr (SPLIT) {
                    uint32_t c0, c1, c2, c3;
                    ldmatrix_x4_trans(c0, c1, c2, c3, smem_u32(vs + TILEV + r * LDV + c));
                    mma_bf16_16816(o_acc[dj], pl, b0, b1);
                    mma_bf16_16816(o_acc[dj + 1], pl, b2, b3);
                    mma_bf16_16816(o_acc[dj], pa, c0, c1);
                    mma_bf16_16816(o_acc[dj + 1], pa, c2, c3);
                }
                mma_bf16_16816(o_acc[dj], pa, b0, b1);
                mma_bf16_16816(o_acc[dj + 1], pa, b2, b3);
            }
        }
        first = false;
        group_sync();      // the group is done with this stage before it is refilled
        if (STG == 1 && ti + 2 < n_walk) { load_kv(tile_at(ti + 2), 0); cp_async_commit(); }
    }
    cp_async_wait<0>();
    // ---- merge the two groups' states (group 1 -> group 0 through its own, now idle, tile buffer) ----
    {
        float* mg = reinterpret_cast<float*>(RAGGED ? kv_s : kv_s + STG * STAGE);        // group 1's ring (RAGGED: both): [128 threads][DV / 2 + 4] floats
        constexpr int MW = DV / 2 + 4;
        __syncthreads();
        if (grp == 1) {
            float* d = mg + (size_t)gtid * MW;
#pragma unroll
            for (int i = 0; i < DV / 8; ++i) { d[4 * i] = o_acc[i][0]; d[4 * i + 1] = o_acc[i][1]; d[4 * i + 2] = o_acc[i][2]; d[4 * i + 3] = o_acc[i][3]; }
            d[DV / 2] = m_row[0]; d[DV / 2 + 1] = m_row[1]; d[DV / 2 + 2] = l_row[0]; d[DV / 2 + 3] = l_row[1];
        }
        __syncthreads();
        if (grp == 1) return;
        const float* d = mg + (size_t)gtid * MW;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const float mo = d[DV / 2 + r], lo = d[DV / 2 + 2 + r];
            const float mn = fmaxf(m_row[r], mo);
            const float c0 = (m_row[r] == -INFINITY) ? 0.f : exp2f(m_row[r] - mn), c1 = (mo == -INFINITY) ? 0.f : exp2f(mo - mn);
            m_row[r] = mn;
            l_row[r] = l_row[r] * c0 + lo * c1;
#pragma unroll
            for (int i = 0; i < DV / 8; ++i) {
                o_acc[i][2 * r] = o_acc[i][2 * r] * c0 + d[4 * i + 2 * r] * c1;
                o_acc[i][2 * r + 1] = o_acc[i][2 * r + 1] * c0 + d[4 * i + 2 * r + 1] * c1;
            }
        }
    }
    // ---- normalise and store ----
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l_row[r] += __shfl_xor_sync(0xffffffffu, l_row[r], 1);
        l_row[r] += __shfl_xor_sync(0xffffffffu, l_row[r], 2);
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int qrow = q0 + warp * 16 + g + r * 8;
        if (qrow < S) {
            float inv = 1.f / l_row[r];
            if (a.sink) {        // the sink joins the denominator only: rescale to the larger of the row maximum and the sink
                const float s2 = a.sink[head] * 1.4426950408889634f, mn = fmaxf(m_row[r], s2);
                const float c = exp2f(m_row[r] - mn);
                inv = c / (l_row[r] * c + exp2f(s2 - mn));
            }
            inv *= a.out_mult;
            if (a.gate && a.gate_heads) inv *= 1.f / (1.f + __expf(-a.gate[(size_t)(row0 + qrow) * a.g_stride + head]));
            bf16* o = a.out + (size_t)(row0 + qrow) * a.o_stride + head * (RAGGED ? a.dv : DV);
            const float* gt = (a.gate && !a.gate_heads) ? a.gate + (size_t)(row0 + qrow) * a.g_stride + head * DV : nullptr;
#pragma unroll
            for (int i = 0; i < DV / 8; ++i) {
                uint32_t hi, lo;
                if (RAGGED && i * 8 + tq * 2 >= a.dv) break;
                float o0 = o_acc[i][2 * r] * inv, o1 = o_acc[i][2 * r + 1] * inv;
                if (gt) {        // sigmoid output gate, in f32
                    const float2 gv = *reinterpret_cast<const float2*>(gt + i * 8 + tq * 2);
                    o0 *= 1.f / (1.f + __expf(-gv.x)); o1 *= 1.f / (1.f + __expf(-gv.y));
                }
                split_bf16x2(o0, o1, hi, lo);
                *reinterpret_cast<uint32_t*>(o + i * 8 + tq * 2) = hi;
                if (SPLIT) *reinterpret_cast<uint32_t*>(o + a.out_lo_off + i * 8 + tq * 2) = lo;
            }
        }
    }
}

template <int D, int DV, bool CAUSAL, bool PAGED, bool SPLIT, bool RAGGED = false>
static int flash_launch_t(cudaStream_t st, const FlashArgs& a) {
    constexpr int P = SPLIT ? 2 : 1, GROUPS = 2, DM = D > DV ? D : DV, BN = DM > 256 ? 16 : (SPLIT || DM > 128) ? 32 : 64, STG = (SPLIT && DM > 128) ? 1 : 2;
    constexpr int SMEM = (P * 64 * (D + 8) + GROUPS * STG * P * BN * (D + DV + 16)) * 2;
    static_assert((RAGGED ? GROUPS : 1) * STG * P * BN * (D + DV + 16) * 2 >= 128 * (DV / 2 + 4) * 4, "the merge buffer lives in group 1's ring");
    static_assert(SMEM <= 227 * 1024, "flash tile does not fit");
    static SmemOptIn seen;
    if (const int e = ensure_dyn_smem(flash_prefill_kernel<D, DV, CAUSAL, PAGED, SPLIT, RAGGED>, (size_t)SMEM, seen)) return e;
    const int max_len = a.seq_len ? a.max_len : a.S;
    dim3 grid((max_len + 63) / 64, a.nh, a.seq_len ? a.nseq : 1);
    return launch_k(flash_prefill_kernel<D, DV, CAUSAL, PAGED, SPLIT, RAGGED>, grid, dim3(256), SMEM, st, prefill_pdl(), a);
}

}  // namespace cb
