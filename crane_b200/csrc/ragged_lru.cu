// Gated linear recurrence with a real decay per channel (see ragged.cuh): S <- a S + sqrt(1 - a^2) i u, a = exp(-rate r), where u is a
// carried causal convolution of the input branch and r, i are sigmoids of block-diagonal linears of u.  Two launches for portions:
//   coefficients : tiles of LRU_TOK tokens of one entry x LRU_COLS channels of one block.  The convolution's outputs of the whole block
//                  (the linears' inputs) are built in shared memory slab by slab and multiplied on the tensor cores as bf16 pairs hi + lo
//                  (the weights are bf16: the products carry ~17 bits; the exact mode multiplies in f32), a and the gated input leave as
//                  f32, and so does what the tile does to a state: the product of its decays and the state it reaches from zero;
//   scan         : the same tiles; a block folds the tiles ahead of its own into its start state (the recurrence is linear in S), walks
//                  its tokens and writes S gelu_tanh(y); the last tile leaves the sequence's state and its last inputs.
// Steps of one token per sequence take one launch.  Inputs of a sequence's last `taps` tokens live in a ring indexed by the position
// (nothing moves, and no two tokens of a step share a place), so blocks that read old inputs and the block that stores the new one
// do not meet.  Everything that enters the recurrence is f32; a row's result depends on its own sequence only.
#include "ragged.cuh"
#include "ragged_dev.cuh"

#include <algorithm>

namespace cb {

namespace {

inline int last_err() { return (int)cudaGetLastError(); }

constexpr int LRU_TOK = 64, LRU_COLS = LRU_TILE_COLS, LRU_SLAB = 128, LRU_THREADS = 256;
constexpr int LRU_LDU = LRU_SLAB + 8, LRU_LDW = 2 * LRU_COLS + 8, LRU_KS = 32;      // padded rows (bf16 elements): conflict-free ldmatrix

__device__ __forceinline__ float lru_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// the convolution's input `back` tokens before the row at `in_entry` / `pos`, with its bias; zeros ahead of the sequence
__device__ __forceinline__ float lru_input(const LruArgs& a, int slot, int r, int in_entry, int pos, int back, int c) {
    if (pos < back) return 0.f;
    if (in_entry >= back) return a.proj[(size_t)(r - back) * a.ld + a.x_col + c] + a.x_b[c];
    return a.ring[((size_t)slot * a.taps + (pos - back) % a.taps) * a.width + c];
}
__device__ __forceinline__ float lru_conv(const LruArgs& a, int slot, int r, int in_entry, int pos, int c) {
    float acc = a.conv_b[c];
    for (int k = 0; k < a.taps; ++k) acc = fmaf(a.conv_w[(size_t)c * a.taps + k], lru_input(a, slot, r, in_entry, pos, a.taps - 1 - k, c), acc);
    return acc;
}
// decay and gated input of one channel and token
__device__ __forceinline__ void lru_coef(float zr, float zi, float rate, float u, float& dec, float& in) {
    const float la = -rate * lru_sigmoid(zr);
    dec = expf(la);
    in = sqrtf(-expm1f(2.f * la)) * lru_sigmoid(zi) * u;
}
// which entry and which of its LRU_TOK-token tiles tile number t is; false past the last
__device__ __forceinline__ bool lru_tile(const RaggedBatch& rb, int t, int& e, int& k) {
    for (e = 0; e < rb.E; ++e) {
        const int n = (rb.ent_len[e] + LRU_TOK - 1) / LRU_TOK;
        if (t < n) { k = t; return true; }
        t -= n;
    }
    return false;
}

__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Grid (tiles of tokens, column tiles of a block, blocks).  Weights: [blocks][column tiles][pad32(n)][LRU_COLS r | LRU_COLS i], zeros behind n.
template <bool EXACT>
__global__ void __launch_bounds__(LRU_THREADS) lru_coef_kernel(RaggedBatch rb, LruArgs a) {
    extern __shared__ __align__(16) unsigned char lsm[];
    __shared__ float so[LRU_TOK][LRU_COLS + 1];               // the convolution's outputs of the tile's own channels
    int e, k;
    if (!lru_tile(rb, blockIdx.x, e, k)) return;
    const int n = a.width / a.blocks, np = (n + 31) / 32 * 32, ct = blockIdx.y, blk = blockIdx.z, cb0 = blk * n, col0 = ct * LRU_COLS;
    const int slot = rb.ent_slot[e], i0 = k * LRU_TOK, nt = min(LRU_TOK, rb.ent_len[e] - i0), r0 = rb.ent_row0[e] + i0, p0 = rb.ent_pos0[e] + i0;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const bf16* wt = a.w_gates + ((size_t)blk * gridDim.y + ct) * np * 2 * LRU_COLS;
    auto emit = [&](int t, int c, float zr, float zi, float* sa, float* sb) {      // -> the tile's decays and gated inputs, in shared memory
        float dec = 1.f, in = 0.f;
        if (t < nt && col0 + c < n) {
            const int ch = cb0 + col0 + c;
            lru_coef(zr + a.r_b[ch], zi + a.i_b[ch], a.rate[ch], so[t][c], dec, in);
        }
        sa[t * (LRU_COLS + 1) + c] = dec; sb[t * (LRU_COLS + 1) + c] = in;
    };
    float* sa = reinterpret_cast<float*>(lsm);                // after the products: [LRU_TOK][LRU_COLS + 1] decays, then gated inputs
    float* sb = sa + LRU_TOK * (LRU_COLS + 1);
    if constexpr (EXACT) {
        float* su = reinterpret_cast<float*>(lsm);            // [LRU_TOK][LRU_SLAB + 1]
        constexpr int NR = LRU_TOK * LRU_COLS / LRU_THREADS;  // 16 tokens of one channel per thread
        const int c = tid % LRU_COLS, tg = tid / LRU_COLS;
        float zr[NR], zi[NR];
#pragma unroll
        for (int q = 0; q < NR; ++q) zr[q] = zi[q] = 0.f;
        for (int s0 = 0; s0 < n; s0 += LRU_SLAB) {
            const int sn = min(LRU_SLAB, n - s0);
            __syncthreads();
            for (int i = tid; i < LRU_TOK * sn; i += LRU_THREADS) {
                const int t = i / sn, j = i % sn;
                const float u = t < nt ? lru_conv(a, slot, r0 + t, i0 + t, p0 + t, cb0 + s0 + j) : 0.f;
                su[t * (LRU_SLAB + 1) + j] = u;
                if (s0 + j >= col0 && s0 + j < col0 + LRU_COLS) so[t][s0 + j - col0] = u;
            }
            __syncthreads();
            for (int j = 0; j < sn; ++j) {
                const float wr = __bfloat162float(wt[(size_t)(s0 + j) * 2 * LRU_COLS + c]), wi = __bfloat162float(wt[(size_t)(s0 + j) * 2 * LRU_COLS + LRU_COLS + c]);
#pragma unroll
                for (int q = 0; q < NR; ++q) {
                    const float u = su[(tg + q * (LRU_THREADS / LRU_COLS)) * (LRU_SLAB + 1) + j];
                    zr[q] = fmaf(wr, u, zr[q]); zi[q] = fmaf(wi, u, zi[q]);
                }
            }
        }
        __syncthreads();
#pragma unroll
        for (int q = 0; q < NR; ++q) emit(tg + q * (LRU_THREADS / LRU_COLS), c, zr[q], zi[q], sa, sb);
    } else {
        bf16* uh = reinterpret_cast<bf16*>(lsm);              // [LRU_TOK][LRU_LDU] hi, then lo
        bf16* ul = uh + LRU_TOK * LRU_LDU;
        bf16* ws = ul + LRU_TOK * LRU_LDU;                    // [2][LRU_KS][LRU_LDW]
        const int wr0 = (warp & 3) * 16, wc0 = (warp >> 2) * 32;      // a warp owns 16 tokens x 32 channels (both gates)
        float acc[2][4][4] = {};                              // [gate][8-channel group][fragment]
        const int g = lane >> 2, tq = lane & 3;
        for (int s0 = 0; s0 < np; s0 += LRU_SLAB) {
            const int sn = min(LRU_SLAB, np - s0), nks = sn / LRU_KS;
            auto fetch = [&](int ks, int st) {                // LRU_KS rows of the weights' slab
                const bf16* src = wt + (size_t)(s0 + ks * LRU_KS) * 2 * LRU_COLS;
                for (int i = tid; i < LRU_KS * 2 * LRU_COLS / 8; i += LRU_THREADS) {
                    const int row = i / (2 * LRU_COLS / 8), ch = i % (2 * LRU_COLS / 8);
                    cp_async16s(ws + ((size_t)st * LRU_KS + row) * LRU_LDW + ch * 8, src + (size_t)row * 2 * LRU_COLS + ch * 8);
                }
                asm volatile("cp.async.commit_group;" ::: "memory");
            };
            __syncthreads();                                  // the last slab's readers are done
            fetch(0, 0);
            // the slab of convolution outputs; a thread walks one channel down the tokens with its taps in registers where they are few
            if (const int j = tid % LRU_SLAB, tg = tid / LRU_SLAB; j < sn) {
                constexpr int TS = LRU_TOK / (LRU_THREADS / LRU_SLAB);        // tokens per thread
                const int t0 = tg * TS, c = cb0 + s0 + j, oc = s0 + j - col0;
                const bool live = s0 + j < n, own = oc >= 0 && oc < LRU_COLS;
                float w[4], h[4], bias = 0.f, xb = 0.f;
                const bool small = a.taps <= 4;
                if (live) { bias = a.conv_b[c]; xb = a.x_b[c]; }
#pragma unroll
                for (int q = 0; q < 4; ++q) {                 // w[3] weighs the current token, w[2] the one before, ...
                    w[q] = (live && small && q >= 4 - a.taps) ? a.conv_w[(size_t)c * a.taps + q - (4 - a.taps)] : 0.f;
                    h[q] = (live && small && q < 3 && q >= 4 - a.taps && t0 < nt) ? lru_input(a, slot, r0 + t0, i0 + t0, p0 + t0, 3 - q, c) : 0.f;
                }
                const float* px = a.proj + (size_t)(r0 + t0) * a.ld + a.x_col + c;
                for (int tb = 0; tb < TS; tb += 8) {
                    float xv[8];
#pragma unroll
                    for (int q = 0; q < 8; ++q) xv[q] = (live && t0 + tb + q < nt) ? px[(size_t)(tb + q) * a.ld] + xb : 0.f;
#pragma unroll
                    for (int q = 0; q < 8; ++q) {
                        const int t = t0 + tb + q;
                        float u = 0.f;
                        if (live && t < nt) {
                            if (small) {
                                u = fmaf(w[3], xv[q], fmaf(w[2], h[2], fmaf(w[1], h[1], fmaf(w[0], h[0], bias))));
                                h[0] = h[1]; h[1] = h[2]; h[2] = xv[q];
                            } else u = lru_conv(a, slot, r0 + t, i0 + t, p0 + t, c);
                        }
                        if (own) so[t][oc] = u;
                        const bf16 hi = __float2bfloat16_rn(u);
                        uh[t * LRU_LDU + j] = hi; ul[t * LRU_LDU + j] = __float2bfloat16_rn(u - __bfloat162float(hi));
                    }
                }
            }
            for (int ks = 0; ks < nks; ++ks) {
                if (ks + 1 < nks) { fetch(ks + 1, (ks + 1) & 1); asm volatile("cp.async.wait_group 1;" ::: "memory"); }
                else asm volatile("cp.async.wait_group 0;" ::: "memory");
                __syncthreads();
                const bf16* wk = ws + (size_t)(ks & 1) * LRU_KS * LRU_LDW;
#pragma unroll
                for (int kk = 0; kk < LRU_KS; kk += 16) {
                    uint32_t ah[4], al[4];
                    const int arow = wr0 + (lane & 7) + ((lane >> 3) & 1) * 8, acol = ks * LRU_KS + kk + (lane >> 4) * 8;
                    ldsm4(ah, smem_u32(uh + arow * LRU_LDU + acol));
                    ldsm4(al, smem_u32(ul + arow * LRU_LDU + acol));
#pragma unroll
                    for (int gate = 0; gate < 2; ++gate)
#pragma unroll
                        for (int j = 0; j < 4; j += 2) {
                            uint32_t b[4];
                            ldsm4t(b, smem_u32(wk + (kk + (lane & 7) + ((lane >> 3) & 1) * 8) * LRU_LDW + gate * LRU_COLS + wc0 + j * 8 + (lane >> 4) * 8));
                            mma16816(acc[gate][j], al, b[0], b[1]);
                            mma16816(acc[gate][j + 1], al, b[2], b[3]);
                            mma16816(acc[gate][j], ah, b[0], b[1]);
                            mma16816(acc[gate][j + 1], ah, b[2], b[3]);
                        }
                }
                __syncthreads();
            }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int q = 0; q < 4; ++q) emit(wr0 + g + (q >> 1) * 8, wc0 + j * 8 + tq * 2 + (q & 1), acc[0][j][q], acc[1][j][q], sa, sb);
    }
    __syncthreads();
    for (int i = tid; i < nt * LRU_COLS; i += LRU_THREADS) {
        const int t = i / LRU_COLS, c = i % LRU_COLS;
        if (col0 + c >= n) continue;
        const size_t at = (size_t)(r0 + t) * a.width + cb0 + col0 + c;
        a.dec[at] = sa[t * (LRU_COLS + 1) + c]; a.gin[at] = sb[t * (LRU_COLS + 1) + c];
    }
    // what the tile does to a state: four threads of a channel take a quarter of the tokens each, joined in order
    const int c = tid / 4, qd = tid & 3;
    float A = 1.f, S = 0.f;
    for (int t = qd * (LRU_TOK / 4); t < (qd + 1) * (LRU_TOK / 4); ++t) {      // (past the last token: decay 1, input 0)
        const float d = sa[t * (LRU_COLS + 1) + c];
        A *= d; S = fmaf(d, S, sb[t * (LRU_COLS + 1) + c]);
    }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
        const float A2 = __shfl_down_sync(0xffffffffu, A, o), S2 = __shfl_down_sync(0xffffffffu, S, o);
        if ((qd & (2 * o - 1)) == 0) { S = fmaf(A2, S, S2); A *= A2; }
    }
    if (qd == 0 && col0 + c < n) {
        float* ag = a.agg + (size_t)blockIdx.x * 2 * a.width + cb0 + col0 + c;
        ag[0] = A; ag[a.width] = S;
    }
}

// Grid (tiles of tokens, 128-channel columns): thread = channel.
__global__ void __launch_bounds__(128) lru_scan_kernel(RaggedBatch rb, LruArgs a) {
    int e, k;
    if (!lru_tile(rb, blockIdx.x, e, k)) return;
    const int c = blockIdx.y * 128 + threadIdx.x;
    if (c >= a.width) return;
    const int slot = rb.ent_slot[e], len = rb.ent_len[e], i0 = k * LRU_TOK, nt = min(LRU_TOK, len - i0), r0 = rb.ent_row0[e] + i0;
    const bool last = i0 + nt == len;
    float S = a.state[(size_t)slot * a.width + c];            // (stays as it is until the closing kernel: every tile folds from it)
    {
        const float* ag = a.agg + (size_t)(blockIdx.x - k) * 2 * a.width + c;
        int q = 0;
        for (; q + 8 <= k; q += 8) {
            float A[8], L[8];
#pragma unroll
            for (int v = 0; v < 8; ++v) { A[v] = ag[(size_t)(q + v) * 2 * a.width]; L[v] = ag[(size_t)(q + v) * 2 * a.width + a.width]; }
#pragma unroll
            for (int v = 0; v < 8; ++v) S = fmaf(A[v], S, L[v]);
        }
        for (; q < k; ++q) S = fmaf(ag[(size_t)q * 2 * a.width], S, ag[(size_t)q * 2 * a.width + a.width]);
    }
    const float yb = a.y_b[c];
    for (int tb = 0; tb < nt; tb += 8) {
        float d[8], in[8], y[8];
#pragma unroll
        for (int v = 0; v < 8; ++v) {
            const bool ok = tb + v < nt;
            const size_t r = (size_t)(r0 + tb + v);
            d[v] = ok ? a.dec[r * a.width + c] : 1.f; in[v] = ok ? a.gin[r * a.width + c] : 0.f; y[v] = ok ? a.proj[r * a.ld + a.y_col + c] + yb : 0.f;
        }
#pragma unroll
        for (int v = 0; v < 8; ++v) {
            if (tb + v >= nt) break;
            S = fmaf(d[v], S, in[v]);
            store_act(a.out, r0 + tb + v, a.out_col + c, S * gelu_tanh_f(y[v]) * a.out_mult);
        }
    }
    if (last) a.next[(size_t)e * a.width + c] = S;
}
// After the scan: every entry's new state, and its last inputs into the ring.
__global__ void __launch_bounds__(128) lru_close_kernel(RaggedBatch rb, LruArgs a) {
    const int e = blockIdx.y, c = blockIdx.x * 128 + threadIdx.x;
    if (c >= a.width) return;
    const int slot = rb.ent_slot[e], len = rb.ent_len[e], r0 = rb.ent_row0[e], p0 = rb.ent_pos0[e];
    a.state[(size_t)slot * a.width + c] = a.next[(size_t)e * a.width + c];
    for (int i = max(0, len - a.taps); i < len; ++i)
        a.ring[((size_t)slot * a.taps + (p0 + i) % a.taps) * a.width + c] = a.proj[(size_t)(r0 + i) * a.ld + a.x_col + c] + a.x_b[c];
}

// Every entry one token.  Grid (column tiles of a block, blocks, entries), LRS_WARPS warps: the block's convolution outputs into shared memory,
// the warps split the linears' input rows between them (a lane owns four of the tile's 2 x 64 columns; partial sums meet in warp order),
// then LRU_COLS threads run the recurrence.
constexpr int LRS_WARPS = 16;
__global__ void __launch_bounds__(LRS_WARPS * 32) lru_step_kernel(RaggedBatch rb, LruArgs a) {
    extern __shared__ __align__(16) float ssm[];
    const int n = a.width / a.blocks, np = (n + 31) / 32 * 32, ct = blockIdx.x, blk = blockIdx.y, e = blockIdx.z, cb0 = blk * n, col0 = ct * LRU_COLS;
    const int r = rb.ent_row0[e], slot = rb.ent_slot[e], pos = rb.ent_pos0[e], tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float* su = ssm;                                          // [np]
    float* part = ssm + np;                                   // [LRS_WARPS][2 LRU_COLS]
    const bf16* wt = a.w_gates + ((size_t)blk * gridDim.x + ct) * np * 2 * LRU_COLS + 4 * lane;
    const int per = (np + LRS_WARPS - 1) / LRS_WARPS, j0 = warp * per, j1 = min(np, j0 + per);
    uint2 wv[8];                                              // the first weights do not depend on the step's inputs
#pragma unroll
    for (int q = 0; q < 8; ++q) wv[q] = j0 + q < j1 ? *reinterpret_cast<const uint2*>(wt + (size_t)(j0 + q) * 2 * LRU_COLS) : make_uint2(0u, 0u);
    for (int j = tid; j < np; j += LRS_WARPS * 32) su[j] = j < n ? lru_conv(a, slot, r, 0, pos, cb0 + j) : 0.f;
    __syncthreads();
    float acc[4] = {};
    for (int jb = j0; jb < j1; jb += 8) {
        if (jb > j0) {
#pragma unroll
            for (int q = 0; q < 8; ++q) wv[q] = jb + q < j1 ? *reinterpret_cast<const uint2*>(wt + (size_t)(jb + q) * 2 * LRU_COLS) : make_uint2(0u, 0u);
        }
#pragma unroll
        for (int q = 0; q < 8; ++q) {
            const float u = jb + q < j1 ? su[jb + q] : 0.f;
            acc[0] = fmaf(u, bf16lo(wv[q].x), acc[0]); acc[1] = fmaf(u, bf16hi(wv[q].x), acc[1]);
            acc[2] = fmaf(u, bf16lo(wv[q].y), acc[2]); acc[3] = fmaf(u, bf16hi(wv[q].y), acc[3]);
        }
    }
    *reinterpret_cast<float4*>(part + warp * 2 * LRU_COLS + 4 * lane) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    __syncthreads();
    if (tid >= LRU_COLS || col0 + tid >= n) return;
    const int c = cb0 + col0 + tid;
    float zr = a.r_b[c], zi = a.i_b[c], dec, in;
    for (int w = 0; w < LRS_WARPS; ++w) { zr += part[w * 2 * LRU_COLS + tid]; zi += part[w * 2 * LRU_COLS + LRU_COLS + tid]; }
    lru_coef(zr, zi, a.rate[c], su[col0 + tid], dec, in);
    const float S = fmaf(dec, a.state[(size_t)slot * a.width + c], in);
    a.state[(size_t)slot * a.width + c] = S;
    a.ring[((size_t)slot * a.taps + pos % a.taps) * a.width + c] = a.proj[(size_t)r * a.ld + a.x_col + c] + a.x_b[c];
    store_act(a.out, r, a.out_col + c, S * gelu_tanh_f(a.proj[(size_t)r * a.ld + a.y_col + c] + a.y_b[c]) * a.out_mult);
}

}  // namespace

size_t lru_gate_weights(int width, int blocks) {
    const int n = width / blocks;
    return (size_t)blocks * ((n + LRU_COLS - 1) / LRU_COLS) * ((n + 31) / 32 * 32) * 2 * LRU_COLS;
}
size_t lru_agg_floats(int rows, int entries, int width) { return ((size_t)rows / LRU_TOK + entries) * 2 * width; }
int lru_launch_count(const LruArgs& a) { return a.single_rows ? 1 : 3; }
int lru_mixer_launch(cudaStream_t st, const RaggedBatch& rb, const LruArgs& a) {
    if (a.width < 1 || a.blocks < 1 || a.width % a.blocks || a.taps < 1) return -1000;
    const int n = a.width / a.blocks, np = (n + 31) / 32 * 32, nct = (n + LRU_COLS - 1) / LRU_COLS;
    if (a.single_rows) {
        const size_t smem = ((size_t)np + LRS_WARPS * 2 * LRU_COLS) * sizeof(float);
        static SmemOptIn seen;
        if (const int er = ensure_dyn_smem(lru_step_kernel, smem, seen)) return er;
        lru_step_kernel<<<dim3(nct, a.blocks, rb.E), LRS_WARPS * 32, smem, st>>>(rb, a);
        return last_err();
    }
    const int tiles = rb.T / LRU_TOK + rb.E;                  // an upper bound: blocks past the last tile leave at once
    const size_t agg = (size_t)2 * LRU_TOK * (LRU_COLS + 1) * sizeof(float);
    const size_t smem = std::max(agg, a.exact ? (size_t)LRU_TOK * (LRU_SLAB + 1) * sizeof(float) : (size_t)(2 * LRU_TOK * LRU_LDU + 2 * LRU_KS * LRU_LDW) * sizeof(bf16));
    const dim3 grid(tiles, nct, a.blocks);
    static SmemOptIn seen_e, seen_t;
    if (a.exact) {
        if (const int er = ensure_dyn_smem(lru_coef_kernel<true>, smem, seen_e)) return er;
        lru_coef_kernel<true><<<grid, LRU_THREADS, smem, st>>>(rb, a);
    } else {
        if (const int er = ensure_dyn_smem(lru_coef_kernel<false>, smem, seen_t)) return er;
        lru_coef_kernel<false><<<grid, LRU_THREADS, smem, st>>>(rb, a);
    }
    if (const int er = last_err()) return er;
    lru_scan_kernel<<<dim3(tiles, (a.width + 127) / 128), 128, 0, st>>>(rb, a);
    if (const int er = last_err()) return er;
    lru_close_kernel<<<dim3((a.width + 127) / 128, rb.E), 128, 0, st>>>(rb, a);
    return last_err();
}

}  // namespace cb
