// The gated delta rule over long portions, 16 tokens at a time (see DeltaArgs in ragged.cuh).  Within a chunk that starts from the state S0,
// with G_i = prod_{m <= i} decay_m and E_ij = prod_{j < m <= i} decay_m (per key channel, plain products: no logarithms, no quotients),
//   u_i = beta_i (v_i - S0^T (G_i k_i) - sum_{j < i} A_ij u_j),   A_ij = k_i . (E_ij k_j)
// so U = U' - W S0 with   w_i = beta_i (G_i k_i - sum_{j < i} A_ij w_j),   u'_i = beta_i (v_i - sum_{j < i} A_ij u'_j),
//   o_i = S0^T (G_i q_i) + sum_{j <= i} P_ij u_j,   P_ij = q_i . (E_ij k_j),      S_16 = diag(G_16) S0 + sum_j (E_16,j k_j) u_j^T.
// The first kernel prepares A, P, W, U' and the scaled q and k of every chunk, all chunks side by side, in f32; the second walks the
// chunks in order, four products per chunk on the tensor cores.  Its operands are f32 numbers taken as two tf32 parts each, three
// products per pair (what is dropped lies below 2^-20 of a product), summed in f32; the state stays in f32 accumulators throughout.
#include "ragged.cuh"
#include "ragged_dev.cuh"

#include <algorithm>

namespace cb {

namespace {

inline int last_err() { return (int)cudaGetLastError(); }

constexpr int DC = 16;           // tokens per chunk
constexpr int DC_COLS = 16;      // value columns per block of the second kernel
constexpr int DC_STAGES = 3;

// One chunk of one head as the second kernel copies it into shared memory: W [16][DP + 8] | Q [16][DP + 8] | K [16][DP + 4] | G [DP] |
// P [16][16], DP = the key width rounded up to 32, 64, 128 or 256 (zeros behind it).  The row paddings spread the fragment loads of a warp
// over all banks.  The values U'^T [dv rounded up to 16][16] follow in an array of their own.
__host__ __device__ inline int dc_pad(int d) { return d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : 256; }
__host__ __device__ constexpr int dc_floats(int DP) { return 2 * DC * (DP + 8) + DC * (DP + 4) + DP + DC * DC; }
__host__ __device__ inline int dc_vpad(int dv) { return (dv + 15) & ~15; }
// chunk slots of an entry: consecutive from here (rounding each entry's rows up separately never makes two entries meet)
__device__ __forceinline__ size_t dc_slot0(const RaggedBatch& rb, int e) { return (size_t)(rb.ent_row0[e] / DC + e); }

// ---------------------------------------------------------------------------------------------------------------- chunks side by side
template <int DP>
__global__ void __launch_bounds__(256) delta_chunk_prep_kernel(RaggedBatch rb, DeltaArgs a, float* __restrict__ ws, float* __restrict__ ut) {
    extern __shared__ __align__(16) float sm[];
    float *sk = sm, *sq = sk + DC * DP, *sg = sq + DC * DP, *sA = sg + DC * DP, *sP = sA + DC * DC, *sb = sP + DC * DC;
    const int ch = blockIdx.x, h = blockIdx.y, e = blockIdx.z, len = rb.ent_len[e], t0 = ch * DC;
    if (t0 >= len) return;
    const int nt = min(DC, len - t0), r0 = rb.ent_row0[e] + t0, d = a.d, dv = a.dv, H = a.H, Hk = a.Hk, hk = h / (H / Hk);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const size_t slot = (dc_slot0(rb, e) + ch) * H + h;
    for (int i = threadIdx.x; i < DC * DP; i += 256) {        // tokens past the end: nothing decays, nothing is written
        const int t = i / DP, c = i % DP;
        const bool ok = t < nt && c < d;
        const size_t r = (size_t)(r0 + t);
        sk[i] = ok ? a.kn[(r * Hk + hk) * d + c] : 0.f;
        sq[i] = ok ? a.qn[(r * Hk + hk) * d + c] : 0.f;
        sg[i] = ok ? a.dec[r * a.lddec + (a.per_channel ? h * d + c : h)] : 1.f;
    }
    if (threadIdx.x < DC) sb[threadIdx.x] = (int)threadIdx.x < nt ? a.beta[(size_t)(r0 + threadIdx.x) * H + h] : 0.f;
    sA[threadIdx.x] = 0.f; sP[threadIdx.x] = 0.f;
    __syncthreads();
    // column j of A and P: a warp carries E_ij k_j of all channels down the rows i = j .. 15; warp w has the columns w and 15 - w
    constexpr int NV = DP / 32;
    for (int half = 0; half < 2; ++half) {
        const int j = half ? DC - 1 - warp : warp;
        float ek[NV];
#pragma unroll
        for (int v = 0; v < NV; ++v) ek[v] = sk[j * DP + lane + 32 * v];
        for (int i = j; i < DC; ++i) {
            float ss = 0.f, sp = 0.f;
#pragma unroll
            for (int v = 0; v < NV; ++v) {
                const int o = i * DP + lane + 32 * v;
                if (i > j) ek[v] *= sg[o];
                ss = fmaf(sk[o], ek[v], ss); sp = fmaf(sq[o], ek[v], sp);
            }
            // both sums at once: the lower half-warp ends with the first, the upper with the second
            float x = lane < 16 ? ss : sp, y = lane < 16 ? sp : ss;
            x += __shfl_xor_sync(0xffffffffu, y, 16);
#pragma unroll
            for (int m = 8; m > 0; m >>= 1) x += __shfl_xor_sync(0xffffffffu, x, m);
            if (lane == 0 && i > j) sA[i * DC + j] = x;
            if (lane == 16) sP[i * DC + j] = x;
        }
    }
    __syncthreads();
    float* W = ws + slot * dc_floats(DP);
    float *Q = W + DC * (DP + 8), *K = Q + DC * (DP + 8), *G = K + DC * (DP + 4), *P = G + DP;
    P[threadIdx.x] = sP[threadIdx.x];
    const int VP = dc_vpad(dv);
    for (int it = threadIdx.x; it < DP + VP; it += 256) {     // one key channel or one value column per thread: forward substitution
        float w[DC];
        if (it < DP) {
            float gam = 1.f;
#pragma unroll
            for (int i = 0; i < DC; ++i) {
                gam *= sg[i * DP + it];
                float acc = gam * sk[i * DP + it];
                Q[i * (DP + 8) + it] = gam * sq[i * DP + it];
#pragma unroll
                for (int j = 0; j < i; ++j) acc = fmaf(-sA[i * DC + j], w[j], acc);
                w[i] = sb[i] * acc;
                W[i * (DP + 8) + it] = w[i];
            }
            G[it] = gam;
            float ek = 1.f;
#pragma unroll
            for (int i = DC - 1; i >= 0; --i) {
                K[i * (DP + 4) + it] = ek * sk[i * DP + it];
                ek *= sg[i * DP + it];
            }
        } else {
            const int p = it - DP;
#pragma unroll
            for (int i = 0; i < DC; ++i) w[i] = (i < nt && p < dv) ? a.v[((size_t)(r0 + i) * H + h) * dv + p] : 0.f;
#pragma unroll
            for (int i = 0; i < DC; ++i) {
                float acc = w[i];
#pragma unroll
                for (int j = 0; j < i; ++j) acc = fmaf(-sA[i * DC + j], w[j], acc);
                w[i] = sb[i] * acc;
            }
            float4* o = reinterpret_cast<float4*>(ut + (slot * VP + p) * DC);
#pragma unroll
            for (int i = 0; i < DC / 4; ++i) o[i] = make_float4(w[4 * i], w[4 * i + 1], w[4 * i + 2], w[4 * i + 3]);
        }
    }
}

// ---------------------------------------------------------------------------------------------------------------- chunks in order
struct Tf2 { uint32_t hi, lo; };
// x = hi + lo + what lies below 2^-21 of it: the leading 11 bits of the significand, then the leading 11 bits of the rest
__device__ __forceinline__ Tf2 tf32_split(float x) {
    Tf2 t;
    t.hi = __float_as_uint(x) & 0xffffe000u;
    t.lo = __float_as_uint(x - __uint_as_float(t.hi)) & 0xffffe000u;
    return t;
}
__device__ __forceinline__ void mma_tf32(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// The A operand of a product is always a 16 x 8 tile that an earlier product left in accumulator layout: its columns 2 (lane % 4) and
// 2 (lane % 4) + 1 become the operand's k = lane % 4 and k = lane % 4 + 4.  The sum runs over k, so B only has to be loaded in that order.
struct FragA {
    Tf2 v[4];
    __device__ __forceinline__ void from(const float* c) { v[0] = tf32_split(c[0]); v[1] = tf32_split(c[2]); v[2] = tf32_split(c[1]); v[3] = tf32_split(c[3]); }
};
struct FragB {
    Tf2 x, y;
    __device__ __forceinline__ void from(float b0, float b1) { x = tf32_split(b0); y = tf32_split(b1); }
};
// the three products of a pair, small terms first; callers interleave the terms of independent accumulators
template <int TERM>
__device__ __forceinline__ void mma_term(float* c, const FragA& a, const FragB& b) {
    if constexpr (TERM == 0) mma_tf32(c, a.v[0].lo, a.v[1].lo, a.v[2].lo, a.v[3].lo, b.x.hi, b.y.hi);
    else if constexpr (TERM == 1) mma_tf32(c, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, b.x.lo, b.y.lo);
    else mma_tf32(c, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, b.x.hi, b.y.hi);
}

// Block = (entry, head, 16 value columns).  Warp w keeps S^T[columns, DS * w ..] as DS / 8 accumulator tiles.  Per chunk: its share of
// S0^T W^T and S0^T Q^T (columns x tokens); the warps' shares meet in shared memory, in warp order, one pair of neighbouring tokens per
// thread; every warp then reads U^T and adds U^T K to its part of the decayed state, and two warps finish eight tokens of the output each.
template <int DS, int NW>
__global__ void __launch_bounds__(NW * 32) delta_chunk_state_kernel(RaggedBatch rb, DeltaArgs a, const float* __restrict__ ws, const float* __restrict__ ut) {
    extern __shared__ __align__(16) float sm[];
    constexpr int DP = NW * DS, NF = dc_floats(DP), STG = NF + DC_COLS * DC, NTL = DS / 8, NT = NW * 32;
    const int e = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * DC_COLS, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, q2 = 2 * (lane & 3);
    const int len = rb.ent_len[e], slot = rb.ent_slot[e], r0 = rb.ent_row0[e], d = a.d, dv = a.dv, H = a.H, ds0 = warp * DS, VP = dc_vpad(dv);
    const size_t slot0 = dc_slot0(rb, e);
    float* red = sm + DC_STAGES * STG;                        // [NW][4 tiles][32 lanes][4]: the shares
    float* sum = red + NW * 512;                              // [2][4 tiles][32 lanes][4]: U^T (two tiles), S0^T Q^T (two tiles)
    float* S = a.state + ((size_t)slot * H + h) * d * dv;
    float s[NTL][4];
#pragma unroll
    for (int k = 0; k < NTL; ++k)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int dd = ds0 + 8 * k + q2 + (x & 1), p = p0 + g + (x >> 1) * 8;
            s[k][x] = (dd < d && p < dv) ? S[(size_t)dd * dv + p] : 0.f;
        }
    const int nch = (len + DC - 1) / DC;
    const float* src = ws + (slot0 * H + h) * (size_t)NF;
    const float* usrc = ut + ((slot0 * H + h) * (size_t)VP + p0) * DC;
    auto fetch = [&](int ch) {                                // one flat copy: the chunk lies in global memory as it is read here
        if (ch < nch) {
            float* dst = sm + (ch % DC_STAGES) * STG;
            const float* w = src + (size_t)ch * H * NF;
#pragma unroll
            for (int i = 0; i < (NF / 4 + NT - 1) / NT; ++i) {
                const int o = 4 * (threadIdx.x + i * NT);
                if ((i + 1) * NT <= NF / 4 || o < NF) cp_async16s(dst + o, w + o);
            }
            if (threadIdx.x < DC_COLS * DC / 4) cp_async16s(dst + NF + 4 * threadIdx.x, usrc + (size_t)ch * H * VP * DC + 4 * threadIdx.x);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int c = 0; c < DC_STAGES - 1; ++c) fetch(c);
    for (int ch = 0; ch < nch; ++ch) {
        asm volatile("cp.async.wait_group %0;" ::"n"(DC_STAGES - 2) : "memory");
        __syncthreads();                                      // chunk ch has landed for everyone; the stage of chunk ch - 1 and the shares are free
        fetch(ch + DC_STAGES - 1);
        const float* W = sm + (ch % DC_STAGES) * STG;
        const float *Q = W + DC * (DP + 8), *K = Q + DC * (DP + 8), *G = K + DC * (DP + 4), *P = G + DP, *U = W + NF;
        float acc[4][4] = {};                                 // S0^T W^T: tokens 0..7, 8..15;  S0^T Q^T: tokens 0..7, 8..15
#pragma unroll
        for (int k = 0; k < NTL; ++k) {
            FragA A;
            FragB B[4];
            A.from(s[k]);
            const int c = ds0 + 8 * k + q2;
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                const float2 b = *reinterpret_cast<const float2*>((n < 2 ? W : Q) + (8 * (n & 1) + g) * (DP + 8) + c);
                B[n].from(b.x, b.y);
            }
#pragma unroll
            for (int n = 0; n < 4; ++n) mma_term<0>(acc[n], A, B[n]);
#pragma unroll
            for (int n = 0; n < 4; ++n) mma_term<1>(acc[n], A, B[n]);
#pragma unroll
            for (int n = 0; n < 4; ++n) mma_term<2>(acc[n], A, B[n]);
        }
        float4* rd = reinterpret_cast<float4*>(red);
#pragma unroll
        for (int n = 0; n < 4; ++n) rd[(warp * 4 + n) * 32 + lane] = make_float4(acc[n][0], acc[n][1], acc[n][2], acc[n][3]);
        // meanwhile: the next state's decayed part and its operands
        FragB B[NTL][2];
#pragma unroll
        for (int k = 0; k < NTL; ++k) {
            const float2 gg = *reinterpret_cast<const float2*>(G + ds0 + 8 * k + q2);
            s[k][0] *= gg.x; s[k][1] *= gg.y; s[k][2] *= gg.x; s[k][3] *= gg.y;
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const float* kp = K + (8 * n + q2) * (DP + 4) + ds0 + 8 * k + g;
                B[k][n].from(kp[0], kp[DP + 4]);
            }
        }
        __syncthreads();
        float* sm_sum = sum + (ch & 1) * 512;
#pragma unroll
        for (int i = 0; i < 256 / NT; ++i) {                  // pair i of sums: U^T = U'^T - S0^T W^T (the first 128 pairs), S0^T Q^T
            const int f = 2 * (threadIdx.x + i * NT), n = f >> 7, l = (f >> 2) & 31, x = f & 3;
            float2 t = make_float2(0.f, 0.f);
#pragma unroll
            for (int w = 0; w < NW; ++w) { const float2 v = *reinterpret_cast<const float2*>(red + w * 512 + f); t.x += v.x; t.y += v.y; }
            if (n < 2) {
                const float2 u = *reinterpret_cast<const float2*>(U + ((l >> 2) + 4 * x) * DC + 8 * n + 2 * (l & 3));
                t.x = u.x - t.x; t.y = u.y - t.y;
            }
            *reinterpret_cast<float2*>(sm_sum + f) = t;
        }
        __syncthreads();
        FragA D[2];
#pragma unroll
        for (int n = 0; n < 2; ++n) { const float4 v = reinterpret_cast<const float4*>(sm_sum)[n * 32 + lane]; const float t[4] = {v.x, v.y, v.z, v.w}; D[n].from(t); }
#pragma unroll
        for (int n = 0; n < 2; ++n) {                         // S^T <- S^T diag(G) + U^T K
#pragma unroll
            for (int k = 0; k < NTL; ++k) mma_term<0>(s[k], D[n], B[k][n]);
#pragma unroll
            for (int k = 0; k < NTL; ++k) mma_term<1>(s[k], D[n], B[k][n]);
#pragma unroll
            for (int k = 0; k < NTL; ++k) mma_term<2>(s[k], D[n], B[k][n]);
        }
        if (warp < 2) {                                       // O^T = S0^T Q^T + U^T P^T, tokens 8 warp .. 8 warp + 7
            const float4 v = reinterpret_cast<const float4*>(sm_sum)[(2 + warp) * 32 + lane];
            float o[2][4] = {{v.x, v.y, v.z, v.w}, {0.f, 0.f, 0.f, 0.f}};
            FragB b[2];
#pragma unroll
            for (int n = 0; n < 2; ++n) { const float2 t = *reinterpret_cast<const float2*>(P + (8 * warp + g) * DC + 8 * n + q2); b[n].from(t.x, t.y); }
#pragma unroll
            for (int n = 0; n < 2; ++n) mma_term<0>(o[n], D[n], b[n]);
#pragma unroll
            for (int n = 0; n < 2; ++n) mma_term<1>(o[n], D[n], b[n]);
#pragma unroll
            for (int n = 0; n < 2; ++n) mma_term<2>(o[n], D[n], b[n]);
            float* y = a.y + ((size_t)(r0 + ch * DC + 8 * warp + q2) * H + h) * dv + p0 + g;
            const int left = len - ch * DC - 8 * warp - q2;
#pragma unroll
            for (int x = 0; x < 4; ++x)
                if ((x & 1) < left && p0 + g + (x >> 1) * 8 < dv) y[(x & 1) * H * dv + (x >> 1) * 8] = o[0][x] + o[1][x];
        }
    }
#pragma unroll
    for (int k = 0; k < NTL; ++k)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int dd = ds0 + 8 * k + q2 + (x & 1), p = p0 + g + (x >> 1) * 8;
            if (dd < d && p < dv) S[(size_t)dd * dv + p] = s[k][x];
        }
}

}  // namespace

// ---------------------------------------------------------------------------------------------------------------- launchers
size_t delta_chunk_ws_floats(int rows, int entries, int H, int d, int dv) {
    return ((size_t)rows / DC + entries + 1) * H * ((size_t)dc_floats(dc_pad(d)) + (size_t)dc_vpad(dv) * DC);
}
int delta_chunk_launch(cudaStream_t st, const RaggedBatch& rb, const DeltaArgs& a) {
    if (!a.chunk_ws || a.d < 1 || a.d > 256 || a.max_len < 1) return -1000;
    const int DP = dc_pad(a.d), nw = DP <= 64 ? 4 : 8, nch = (a.max_len + DC - 1) / DC;
    float* ws = a.chunk_ws;
    float* ut = ws + ((size_t)rb.T / DC + rb.E + 1) * a.H * (size_t)dc_floats(DP);
    const size_t psm = (size_t)(3 * DC * DP + 2 * DC * DC + DC) * sizeof(float);
    const size_t ssm = (size_t)(DC_STAGES * (dc_floats(DP) + DC_COLS * DC) + (nw + 2) * 512) * sizeof(float);      // <= 181 KB at a key width of 256
    static SmemOptIn seen_p[4], seen_s[4];
    auto run = [&](auto prep, auto state, int i) -> int {
        if (const int e = ensure_dyn_smem(prep, psm, seen_p[i])) return e;
        if (const int e = ensure_dyn_smem(state, ssm, seen_s[i])) return e;
        prep<<<dim3(nch, a.H, rb.E), 256, psm, st>>>(rb, a, ws, ut);
        if (const int e = last_err()) return e;
        state<<<dim3(rb.E, a.H, (a.dv + DC_COLS - 1) / DC_COLS), nw * 32, ssm, st>>>(rb, a, ws, ut);
        return last_err();
    };
    switch (DP) {
        case 32: return run(delta_chunk_prep_kernel<32>, delta_chunk_state_kernel<8, 4>, 0);
        case 64: return run(delta_chunk_prep_kernel<64>, delta_chunk_state_kernel<16, 4>, 1);
        case 128: return run(delta_chunk_prep_kernel<128>, delta_chunk_state_kernel<16, 8>, 2);
        default: return run(delta_chunk_prep_kernel<256>, delta_chunk_state_kernel<32, 8>, 3);
    }
}

}  // namespace cb
