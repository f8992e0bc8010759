// The gated delta rule on ragged batches (see ragged.cuh), and the embedding of the token that joins behind a layer.
//   prep : per (q / k head | value head | gates): convolution over time with the carried window, SiLU, unit norms, q . k, the decays
//          and step sizes -- f32 throughout, one warp per head and tile of rows, the tap window in registers;
//   scan : the recurrence token by token, a thread keeps its share of the state in registers for the whole portion, the inputs of DR_CH
//          tokens at a time staged in shared memory (cp.async, double-buffered); long portions go 16 tokens at a time instead
//          (ragged_delta_chunk.cu);
//   out  : norm over the value width, gate;
//   step : all of it in one launch, for steps whose entries are one row each.
// A row's result depends on its own sequence only: the split of the state over lanes and the order of the lane sums are launch
// constants.
#include "ragged.cuh"
#include "ragged_dev.cuh"

#include <algorithm>

namespace cb {

namespace {

inline int last_err() { return (int)cudaGetLastError(); }

__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

// ---------------------------------------------------------------------------------------------------------------- prep
constexpr int DP_ROWS = 16;      // rows a warp walks
template <int NC, int TAPS>
__global__ void __launch_bounds__(128) delta_prep_kernel(RaggedBatch rb, DeltaArgs a, int tile) {
    const int lane = threadIdx.x & 31, unit = blockIdx.y * 4 + (threadIdx.x >> 5), r0 = blockIdx.x * tile, r1 = min(rb.T, r0 + tile);
    const int Hk = a.Hk, H = a.H, d = a.d, dv = a.dv, n_dec = a.per_channel ? H : 0;
    if (unit >= Hk + H + n_dec + 1) return;
    const ConvSrc cs{a.proj + a.col0, a.ld, a.conv_w, a.conv_state, 2 * Hk * d + H * dv, a.taps};
    if (unit < Hk) {                                          // a q / k head: convolution, SiLU, unit vectors, their product
        ConvWalk<NC, TAPS> q, k;
        q.init(cs, unit * d, d, lane);
        k.init(cs, (Hk + unit) * d, d, lane);
        for (int rb0 = r0; rb0 < r1; rb0 += 4) {              // four rows requested before the first is used
            float xq[4][NC], xk[4][NC];
#pragma unroll
            for (int u = 0; u < 4; ++u)
#pragma unroll
                for (int i = 0; i < NC; ++i) {
                    const bool ok = rb0 + u < r1 && lane + 32 * i < d;
                    const float* p = a.proj + (size_t)(rb0 + u) * a.ld + a.col0 + unit * d + lane + 32 * i;
                    xq[u][i] = ok ? p[0] : 0.f; xk[u][i] = ok ? p[Hk * d] : 0.f;
                }
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int r = rb0 + u;
                if (r >= r1) break;
                const int e = rb.row_entry[r], in_entry = r - rb.ent_row0[e], slot = rb.ent_slot[e];
                if (r == r0 || in_entry == 0) { q.refill(cs, slot, in_entry, r); k.refill(cs, slot, in_entry, r); }
                float yq[NC], yk[NC], sq = 0.f, sk = 0.f, sqk = 0.f;
                q.step(cs, slot, in_entry, r, xq[u], yq, a.single_rows != 0 && a.taps > 1);
                k.step(cs, slot, in_entry, r, xk[u], yk, a.single_rows != 0 && a.taps > 1);
#pragma unroll
                for (int i = 0; i < NC; ++i) {
                    yq[i] = silu_f(yq[i]); yk[i] = silu_f(yk[i]);
                    sq = fmaf(yq[i], yq[i], sq); sk = fmaf(yk[i], yk[i], sk); sqk = fmaf(yq[i], yk[i], sqk);
                }
                sq = warp_sum(sq); sk = warp_sum(sk); sqk = warp_sum(sqk);
                const float iq = a.q_scale / sqrtf(sq + 1e-6f), ik = 1.f / sqrtf(sk + 1e-6f);
#pragma unroll
                for (int i = 0; i < NC; ++i)
                    if (lane + 32 * i < d) {
                        const size_t o = ((size_t)r * Hk + unit) * d + lane + 32 * i;
                        a.qn[o] = yq[i] * iq; a.kn[o] = yk[i] * ik;
                    }
                if (lane == 0) a.qk[(size_t)r * Hk + unit] = sqk * iq * ik;
            }
        }
    } else if (unit < Hk + H) {                               // a value head
        const int h = unit - Hk;
        for (int cb = 0; cb < dv; cb += 32 * NC) {
            ConvWalk<NC, TAPS> v;
            v.init(cs, 2 * Hk * d + h * dv + cb, min(32 * NC, dv - cb), lane);
            for (int rb0 = r0; rb0 < r1; rb0 += 4) {
                float x[4][NC];
#pragma unroll
                for (int u = 0; u < 4; ++u)
#pragma unroll
                    for (int i = 0; i < NC; ++i)
                        x[u][i] = (rb0 + u < r1 && lane + 32 * i < v.width) ? a.proj[(size_t)(rb0 + u) * a.ld + a.col0 + v.c0 + lane + 32 * i] : 0.f;
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    const int r = rb0 + u;
                    if (r >= r1) break;
                    const int e = rb.row_entry[r], in_entry = r - rb.ent_row0[e], slot = rb.ent_slot[e];
                    if (r == r0 || in_entry == 0) v.refill(cs, slot, in_entry, r);
                    float y[NC];
                    v.step(cs, slot, in_entry, r, x[u], y, a.single_rows != 0 && a.taps > 1);
#pragma unroll
                    for (int i = 0; i < NC; ++i) if (lane + 32 * i < v.width) a.v[((size_t)r * H + h) * dv + cb + lane + 32 * i] = silu_f(y[i]);
                }
            }
        }
    } else if (unit < Hk + H + n_dec) {                       // the decays of a head's key channels
        const int h = unit - Hk - H;
        const float rate = a.rate[h];
        for (int c = lane; c < d; c += 32) {
            const float b = a.dt_bias[h * d + c];
            for (int rb0 = r0; rb0 < r1; rb0 += 8) {          // (dec may be z itself: the rows are requested ahead of the first store)
                float z[8];
#pragma unroll
                for (int u = 0; u < 8; ++u) z[u] = rb0 + u < r1 ? a.z[(size_t)(rb0 + u) * a.ldz + h * d + c] : 0.f;
#pragma unroll
                for (int u = 0; u < 8; ++u) if (rb0 + u < r1) a.dec[(size_t)(rb0 + u) * a.lddec + h * d + c] = expf(-rate * softplus_f(z[u] + b));
            }
        }
    } else {                                                  // step sizes (and the decays of whole heads)
        for (int i = lane; i < (r1 - r0) * H; i += 32) {
            const int r = r0 + i / H, h = i % H;
            a.beta[(size_t)r * H + h] = sigmoid_f(a.proj[(size_t)r * a.ld + a.b_col + h]);
            if (!a.per_channel) a.dec[(size_t)r * a.lddec + h] = expf(-a.rate[h] * softplus_f(a.z[(size_t)r * a.ldz + h] + a.dt_bias[h]));
        }
    }
}

// ---------------------------------------------------------------------------------------------------------------- scan
// Block = (entry, head, DR_COLS value columns); thread (pl, ns) owns rows ns * R .. ns * R + R - 1 of column p0 + pl of S in registers.
// A token's two products with the decayed state -- S^T k for the correction, S^T q for the output -- are reduced over the eight lanes of
// a column together; the output then is S^T q + (q . k) u, which is the read-out after the write.  Tokens go in groups of four whose
// operands are read ahead of the first reduction; a group's tokens past the end have decay 1 and step size 0.
constexpr int DR_NS = 8, DR_COLS = 16, DR_CH = 16;
// a staged vector is cut into eight runs of R, from R = 4 on each followed by 4 pad floats: spreads the runs of a warp over all banks
__host__ __device__ inline int dr_idx(int n, int R) { return R >= 4 ? n + 4 * (n / R) : n; }
__host__ __device__ inline int dr_pad(int R) { return R >= 4 ? DR_NS * (R + 4) : DR_NS * R; }
template <int R>
__device__ __forceinline__ void load_run(const float* p, float* o) {
    if constexpr ((R & 3) == 0) {
#pragma unroll
        for (int i = 0; i < R / 4; ++i) { const float4 t = reinterpret_cast<const float4*>(p)[i]; o[4 * i] = t.x; o[4 * i + 1] = t.y; o[4 * i + 2] = t.z; o[4 * i + 3] = t.w; }
    } else {
#pragma unroll
        for (int i = 0; i < R; ++i) o[i] = p[i];
    }
}
template <int R, bool PC>
__global__ void __launch_bounds__(DR_COLS * DR_NS) delta_scan_kernel(RaggedBatch rb, DeltaArgs a) {
    extern __shared__ __align__(16) float sm[];
    constexpr int NV = PC ? 3 : 2;                            // staged vectors per token: q | k (| decay)
    const int e = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * DR_COLS, ns = threadIdx.x & (DR_NS - 1), pl = threadIdx.x / DR_NS, p = p0 + pl;
    const int d = a.d, dv = a.dv, H = a.H, Hk = a.Hk, hk = h / (H / Hk), DPD = dr_pad(R), PT = NV * DPD + DR_COLS + 4;
    const bool live = p < dv;
    const int len = rb.ent_len[e], slot = rb.ent_slot[e], r0 = rb.ent_row0[e], ncol = min(DR_COLS, dv - p0), n0 = ns * R;
    float* stage[2] = {sm, sm + DR_CH * PT};
    float* sy = sm + 2 * DR_CH * PT;                          // [CH][COLS]
    for (int i = threadIdx.x; i < 2 * DR_CH * PT; i += blockDim.x) sm[i] = 0.f;       // rows past d, columns past dv stay zero
    float* S = a.state + ((size_t)slot * H + h) * d * dv + (live ? p : 0);
    float s[R];
#pragma unroll
    for (int i = 0; i < R; ++i) s[i] = (live && n0 + i < d) ? S[(size_t)(n0 + i) * dv] : 0.f;
    __syncthreads();
    const bool wide = ((d | dv | (PC ? a.lddec : 0)) & 3) == 0 && R >= 4;          // then every piece starts on a 16-byte boundary
    auto fetch = [&](int ch, float* dst) {
        const int t0 = ch * DR_CH, nt = min(DR_CH, len - t0);
        if (wide) {
            const int nq = d >> 2, per = NV * nq + (ncol >> 2);
            for (int i = threadIdx.x; i < nt * per; i += blockDim.x) {
                const int t = i / per, k = i - t * per, r = r0 + t0 + t;
                float* d0 = dst + t * PT;
                if (k < nq) cp_async16s(d0 + dr_idx(4 * k, R), a.qn + ((size_t)r * Hk + hk) * d + 4 * k);
                else if (k < 2 * nq) cp_async16s(d0 + DPD + dr_idx(4 * (k - nq), R), a.kn + ((size_t)r * Hk + hk) * d + 4 * (k - nq));
                else if (PC && k < 3 * nq) cp_async16s(d0 + 2 * DPD + dr_idx(4 * (k - 2 * nq), R), a.dec + (size_t)r * a.lddec + h * d + 4 * (k - 2 * nq));
                else cp_async16s(d0 + NV * DPD + 4 * (k - NV * nq), a.v + ((size_t)r * H + h) * dv + p0 + 4 * (k - NV * nq));
            }
        } else {
            const int per = NV * d + ncol;
            for (int i = threadIdx.x; i < nt * per; i += blockDim.x) {
                const int t = i / per, k = i - t * per, r = r0 + t0 + t;
                float* d0 = dst + t * PT;
                if (k < d) cp_async4(d0 + dr_idx(k, R), a.qn + ((size_t)r * Hk + hk) * d + k);
                else if (k < 2 * d) cp_async4(d0 + DPD + dr_idx(k - d, R), a.kn + ((size_t)r * Hk + hk) * d + k - d);
                else if (PC && k < 3 * d) cp_async4(d0 + 2 * DPD + dr_idx(k - 2 * d, R), a.dec + (size_t)r * a.lddec + h * d + k - 2 * d);
                else cp_async4(d0 + NV * DPD + k - NV * d, a.v + ((size_t)r * H + h) * dv + p0 + k - NV * d);
            }
        }
        if (threadIdx.x < 3 * nt) {
            const int t = threadIdx.x / 3, w = threadIdx.x % 3, r = r0 + t0 + t;
            const float* src = w == 0 ? a.beta + (size_t)r * H + h : w == 1 ? a.qk + (size_t)r * Hk + hk : a.dec + (size_t)r * a.lddec + (PC ? h * d : h);
            cp_async4(dst + t * PT + NV * DPD + DR_COLS + w, src);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        for (int t = nt; t < ((nt + 3) & ~3); ++t) {          // the last group's tokens past the end leave the state as it is
            float* d0 = dst + t * PT;
            if (PC) for (int i = threadIdx.x; i < DPD; i += blockDim.x) d0[2 * DPD + i] = 1.f;
            if (threadIdx.x == 0) { d0[NV * DPD + DR_COLS] = 0.f; d0[NV * DPD + DR_COLS + 2] = 1.f; }
        }
    };
    const int nch = (len + DR_CH - 1) / DR_CH;
    fetch(0, stage[0]);
    for (int ch = 0; ch < nch; ++ch) {
        if (ch + 1 < nch) { fetch(ch + 1, stage[(ch + 1) & 1]); asm volatile("cp.async.wait_group 1;" ::: "memory"); }
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const float* st = stage[ch & 1];
        const int nt = min(DR_CH, len - ch * DR_CH);
        for (int tg = 0; tg < nt; tg += 4) {
            float o[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float* tk = st + (tg + u) * PT;
                float kk[R], qq[R];
                load_run<R>(tk + dr_idx(n0, R), qq);
                load_run<R>(tk + DPD + dr_idx(n0, R), kk);
                const float4 sc = *reinterpret_cast<const float4*>(tk + NV * DPD + DR_COLS);      // step size, q . k, decay of the head
                const float vv = tk[NV * DPD + pl];
                float k0 = 0.f, k1 = 0.f, q0 = 0.f, q1 = 0.f;
                if constexpr (PC) {
                    float g[R];
                    load_run<R>(tk + 2 * DPD + dr_idx(n0, R), g);
#pragma unroll
                    for (int i = 0; i < R; ++i) s[i] *= g[i];
                }
#pragma unroll
                for (int i = 0; i < R; i += 2) {
                    k0 = fmaf(s[i], kk[i], k0); q0 = fmaf(s[i], qq[i], q0);
                    if (i + 1 < R) { k1 = fmaf(s[i + 1], kk[i + 1], k1); q1 = fmaf(s[i + 1], qq[i + 1], q1); }
                }
                float ks = k0 + k1, qs = q0 + q1;
#pragma unroll
                for (int m = DR_NS / 2; m > 0; m >>= 1) { ks += __shfl_xor_sync(0xffffffffu, ks, m); qs += __shfl_xor_sync(0xffffffffu, qs, m); }
                const float dec = PC ? 1.f : sc.z, uu = sc.x * (vv - dec * ks);
                if constexpr (PC) {
#pragma unroll
                    for (int i = 0; i < R; ++i) s[i] = fmaf(kk[i], uu, s[i]);
                } else {
#pragma unroll
                    for (int i = 0; i < R; ++i) s[i] = fmaf(dec, s[i], kk[i] * uu);
                }
                o[u] = fmaf(sc.y, uu, dec * qs);
            }
            if (ns == 0) {
#pragma unroll
                for (int u = 0; u < 4; ++u) sy[(tg + u) * DR_COLS + pl] = o[u];
            }
        }
        __syncthreads();
        for (int i = threadIdx.x; i < nt * DR_COLS; i += blockDim.x) {
            const int t = i / DR_COLS, c = i % DR_COLS;
            if (c < ncol) a.y[((size_t)(r0 + ch * DR_CH + t) * H + h) * dv + p0 + c] = sy[i];
        }
        __syncthreads();                                      // the stage is free for chunk ch + 2
    }
#pragma unroll
    for (int i = 0; i < R; ++i) if (live && n0 + i < d) S[(size_t)(n0 + i) * dv] = s[i];
}

// one warp per (row, head)
__global__ void __launch_bounds__(128) delta_out_kernel(DeltaArgs a, int T) {
    const int lane = threadIdx.x & 31, wid = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (wid >= T * a.H) return;
    const int r = wid / a.H, h = wid % a.H, dv = a.dv;
    const float* y = a.y + ((size_t)r * a.H + h) * dv;
    const float* g = a.g + (size_t)r * a.ldg + h * dv;
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) ss = fmaf(y[c], y[c], ss);
    const float inv = a.out_mult / sqrtf(warp_sum(ss) / (float)dv + a.eps);
    for (int c = lane; c < dv; c += 32) store_act(a.out, r, a.out_col + h * dv + c, y[c] * inv * a.norm_w[c] * (a.gate_silu ? silu_f(g[c]) : sigmoid_f(g[c])));
}

// ---------------------------------------------------------------------------------------------------------------- a decode step
// Every entry one row: the whole mixer between the merged projection and the output projection in one launch.  Block = (head, 32 value
// columns, entry); the blocks of the heads that share a q / k head form a cluster.  Convolution and unit norms (every block for itself), the
// low-rank products (w_a2 != nullptr: z and the gate's pre-activations are taken here from the first factors in proj; a head's blocks
// share the decays' rows and hand the results round), decays and step size; then the state, read once and written once, a thread owning
// R rows of one column; norm over the head's blocks, gate.  The windows move on after every block of the cluster has read them.
constexpr int DS_NS = 8, DS_TAPS = 8, DS_NT = DS_NS * 32, DS_CONV = 3;      // row slices, most taps, threads, channels per thread at most
__device__ __forceinline__ void cluster_store(float* p, int rank, float v) {     // to the same place in another block of the cluster
    uint32_t a;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(smem_u32(p)), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(a), "f"(v) : "memory");
}
__device__ __forceinline__ void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
template <int R>
__global__ void __launch_bounds__(DS_NT, 1) delta_step_kernel(RaggedBatch rb, DeltaArgs a) {
    extern __shared__ __align__(16) float xs[];           // the first factors' outputs (low-rank form)
    constexpr int DR = DS_NS * R;
    __shared__ __align__(16) float sq[DR], sk[DR], sdec[DR], sv[32], sg[32], part[2][DS_NS][32], sz[DR + 32];
    __shared__ float scal[3], ssum[8];                    // 1 / |q| (with q_scale), 1 / |k|, their product before the norms; the blocks' sums of squares
    const int d = a.d, dv = a.dv, H = a.H, Hk = a.Hk, rep = H / Hk, nz = (dv + 31) / 32, h = blockIdx.x / nz, z = blockIdx.x % nz, e = blockIdx.y;
    const int hk = h / rep, C = 2 * Hk * d + H * dv, taps = a.taps, rank0 = (h % rep) * nz, p0 = 32 * z, nc = min(32, dv - p0), n_ch = 2 * d + nc;
    const int tid = threadIdx.x, lane = tid & 31, ns = tid >> 5, n0 = ns * R, p = p0 + lane;
    const int r = rb.ent_row0[e], slot = rb.ent_slot[e];
    const bool clustered = rep * nz > 1, low = a.w_a2 != nullptr, live = lane < nc;
    const int ra4 = (a.a_rank + 3) & ~3, rg4 = (a.g_rank + 3) & ~3;
    const float* row = a.proj + (size_t)r * a.ld;
    float* S = a.state + ((size_t)slot * H + h) * d * dv + p;
    if (clustered) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");      // (waited for ahead of the first store into another block)
    float s[R];                                           // the state is requested before anything else
#pragma unroll
    for (int i = 0; i < R; ++i) s[i] = (live && n0 + i < d) ? S[(size_t)(n0 + i) * dv] : 0.f;
    const int dper = (d + nz - 1) / nz, d_lo = min(d, z * dper), nd = min(d, d_lo + dper) - d_lo;      // this block's rows of the decays' product
    if (low) {                                            // the second factors' rows are on their way to L2 while the convolution runs
        const int la = (a.a_rank + 63) / 64, lg = (a.g_rank + 63) / 64;
        for (int i = tid; i < nd * la; i += DS_NT) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.w_a2 + (size_t)(h * d + d_lo + i / la) * a.ld_a2 + 64 * (i % la)));
        for (int i = tid; i < nc * lg; i += DS_NT) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.w_g2 + (size_t)(h * dv + p0 + i / lg) * a.ld_g2 + 64 * (i % lg)));
        for (int i = tid; i < ra4; i += DS_NT) xs[i] = i < a.a_rank ? row[a.a_col + i] : 0.f;
        for (int i = tid; i < rg4; i += DS_NT) xs[ra4 + i] = i < a.g_rank ? row[a.g_col + i] : 0.f;
    }
    const float rate = a.rate[h], step_z = row[a.b_col + h], nw = live ? a.norm_w[p] : 0.f;
    const float dt_b = tid < d ? a.dt_bias[a.per_channel ? h * d + (low ? min(d_lo + tid, d - 1) : tid) : h] : 0.f;
    float w[DS_CONV][DS_TAPS];                            // convolution: q | k | v channels of this block
#pragma unroll
    for (int u = 0; u < DS_CONV; ++u) {
        const int t = tid + u * DS_NT;
        if (t >= n_ch) break;
        const int ch = t < d ? hk * d + t : t < 2 * d ? Hk * d + hk * d + t - d : 2 * Hk * d + h * dv + p0 + t - 2 * d;
        const float* win = a.conv_state + (size_t)slot * (taps - 1) * C + ch;
        const float own = row[a.col0 + ch];
        float acc = 0.f;
#pragma unroll
        for (int k = 0; k < DS_TAPS; ++k)
            if (k < taps) {
                w[u][k] = k < taps - 1 ? win[(size_t)k * C] : own;
                acc = fmaf(a.conv_w[(size_t)ch * taps + k], w[u][k], acc);
            }
        acc = silu_f(acc);
        if (t < d) sq[t] = acc; else if (t < 2 * d) sk[t - d] = acc; else sv[t - 2 * d] = acc;
    }
    for (int i = d + tid; i < DR; i += DS_NT) { sq[i] = 0.f; sk[i] = 0.f; sdec[i] = 0.f; }
    __syncthreads();
    if (low) {
        constexpr int NR = 4;                             // rows of the second factors in flight per warp
        for (int i0 = ns * NR; i0 < nd + nc; i0 += DS_NS * NR) {
            float acc[NR];
#pragma unroll
            for (int u = 0; u < NR; ++u) {
                const int i = min(i0 + u, nd + nc - 1);
                const bool dec = i < nd;
                const bf16* wr = dec ? a.w_a2 + (size_t)(h * d + d_lo + i) * a.ld_a2 : a.w_g2 + (size_t)(h * dv + p0 + i - nd) * a.ld_g2;
                const float* x = dec ? xs : xs + ra4;
                const int n = dec ? ra4 : rg4;
                acc[u] = 0.f;
                for (int k = 4 * lane; k < n; k += 128) {
                    const uint2 t = *reinterpret_cast<const uint2*>(wr + k);
                    const float4 xv = *reinterpret_cast<const float4*>(x + k);
                    acc[u] = fmaf(bf16lo(t.x), xv.x, acc[u]); acc[u] = fmaf(bf16hi(t.x), xv.y, acc[u]);
                    acc[u] = fmaf(bf16lo(t.y), xv.z, acc[u]); acc[u] = fmaf(bf16hi(t.y), xv.w, acc[u]);
                }
            }
#pragma unroll
            for (int u = 0; u < NR; ++u) acc[u] = warp_sum(acc[u]);
            if (lane == 0) {
#pragma unroll
                for (int u = 0; u < NR; ++u) if (i0 + u < nd + nc) sz[i0 + u] = acc[u];
            }
        }
    }
    if (ns == DS_NS - 1) {                                // |q|^2, |k|^2, q . k
        float qq = 0.f, kk = 0.f, qk = 0.f;
        for (int i = lane; i < d; i += 32) { qq = fmaf(sq[i], sq[i], qq); kk = fmaf(sk[i], sk[i], kk); qk = fmaf(sq[i], sk[i], qk); }
        qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
        if (lane == 0) { scal[0] = a.q_scale / sqrtf(qq + 1e-6f); scal[1] = 1.f / sqrtf(kk + 1e-6f); scal[2] = qk; }
    }
    __syncthreads();
    if (clustered) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    if (low) {
        if (tid < nd) {
            const float g = expf(-rate * softplus_f(sz[tid] + dt_b));
            if (nz > 1) { for (int b = 0; b < nz; ++b) cluster_store(sdec + d_lo + tid, rank0 + b, g); } else sdec[tid] = g;
        }
        if (tid < nc) { const float g = sz[nd + tid]; sg[tid] = a.gate_silu ? silu_f(g) : sigmoid_f(g); }
    } else {
        if (tid < d) sdec[tid] = expf(-rate * softplus_f(a.z[(size_t)r * a.ldz + (a.per_channel ? h * d + tid : h)] + dt_b));
        if (tid < nc) { const float g = a.g[(size_t)r * a.ldg + h * dv + p0 + tid]; sg[tid] = a.gate_silu ? silu_f(g) : sigmoid_f(g); }
    }
    if (clustered) cluster_sync(); else __syncthreads();  // every block has its decays, and has read the windows
    const float iq = scal[0], ik = scal[1], qk = scal[2] * iq * ik, beta = sigmoid_f(step_z);
    float ks = 0.f, qs = 0.f;
#pragma unroll
    for (int i = 0; i < R; ++i) { s[i] *= sdec[n0 + i]; ks = fmaf(s[i], sk[n0 + i], ks); qs = fmaf(s[i], sq[n0 + i], qs); }
    part[0][ns][lane] = ks; part[1][ns][lane] = qs;
    __syncthreads();
    float kt = 0.f, qt = 0.f;
#pragma unroll
    for (int n = 0; n < DS_NS; ++n) { kt += part[0][n][lane]; qt += part[1][n][lane]; }
    const float u = live ? beta * (sv[lane] - ik * kt) : 0.f, uk = u * ik, o = live ? fmaf(qk, u, iq * qt) : 0.f;
    if (ns == 0) {
        const float ss = warp_sum(o * o);
        if (lane < nz) { if (nz > 1) cluster_store(ssum + z, rank0 + lane, ss); else ssum[0] = ss; }
    }
#pragma unroll
    for (int i = 0; i < R; ++i) if (live && n0 + i < d) S[(size_t)(n0 + i) * dv] = fmaf(sk[n0 + i], uk, s[i]);
#pragma unroll
    for (int v = 0; v < DS_CONV; ++v) {                   // the windows move on; a q / k head's by the first block that shares it
        const int t = tid + v * DS_NT;
        if (t >= n_ch) break;
        if (t < 2 * d && (z || h % rep)) continue;
        const int ch = t < d ? hk * d + t : t < 2 * d ? Hk * d + hk * d + t - d : 2 * Hk * d + h * dv + p0 + t - 2 * d;
        float* win = a.conv_state + (size_t)slot * (taps - 1) * C + ch;
#pragma unroll
        for (int k = 0; k < DS_TAPS - 1; ++k) if (k < taps - 1) win[(size_t)k * C] = w[v][k + 1];
    }
    if (nz > 1) cluster_sync(); else __syncthreads();
    if (ns == 0 && live) {
        float tot = 0.f;
        for (int b = 0; b < nz; ++b) tot += ssum[b];
        store_act(a.out, r, a.out_col + h * dv + p, o * (a.out_mult / sqrtf(tot / (float)dv + a.eps)) * nw * sg[lane]);
    }
}

// ---------------------------------------------------------------------------------------------------------------- the token's own embedding
__global__ void token_gate_kernel(const float* __restrict__ z, int ldz, int n, const int* __restrict__ ids, const bf16* __restrict__ table, int ldt, int col0, ActOut out) {
    const int r = blockIdx.y, j = blockIdx.x * blockDim.x + threadIdx.x;
    if (j >= n) return;
    store_act(out, r, j, gelu_tanh_f(z[(size_t)r * ldz + j]) * __bfloat162float(table[(size_t)ids[r] * ldt + col0 + j]));
}
// Block = (output j, row): 128 threads share the dot of length K, 16-byte loads of the bf16 weights.
__global__ void __launch_bounds__(128) token_gate_step_kernel(const float* __restrict__ x, int ldx, const bf16* __restrict__ w, int ldw, int K, const int* __restrict__ ids,
                                                              const bf16* __restrict__ table, int ldt, int col0, ActOut out) {
    __shared__ float red[4];
    const int j = blockIdx.x, r = blockIdx.y;
    const uint4* w8 = reinterpret_cast<const uint4*>(w + (size_t)j * ldw);
    const float4* x4 = reinterpret_cast<const float4*>(x + (size_t)r * ldx);
    float acc = 0.f;
    for (int k = threadIdx.x; k < K / 8; k += 128) {
        const uint4 ww = w8[k];
        const float4 a = x4[2 * k], b = x4[2 * k + 1];
        acc = fmaf(bf16lo(ww.x), a.x, acc); acc = fmaf(bf16hi(ww.x), a.y, acc); acc = fmaf(bf16lo(ww.y), a.z, acc); acc = fmaf(bf16hi(ww.y), a.w, acc);
        acc = fmaf(bf16lo(ww.z), b.x, acc); acc = fmaf(bf16hi(ww.z), b.y, acc); acc = fmaf(bf16lo(ww.w), b.z, acc); acc = fmaf(bf16hi(ww.w), b.w, acc);
    }
    acc = warp_sum(acc);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = acc;
    __syncthreads();
    if (threadIdx.x == 0) store_act(out, r, j, gelu_tanh_f((red[0] + red[1]) + (red[2] + red[3])) * __bfloat162float(table[(size_t)ids[r] * ldt + col0 + j]));
}

}  // namespace

// ---------------------------------------------------------------------------------------------------------------- launchers
static bool by_chunks(const DeltaArgs& a) { return a.chunk_ws && a.max_len >= DELTA_CHUNK_MIN; }
int delta_launch_count(const DeltaArgs& a) { return 3 + (!a.single_rows && a.taps > 1 ? 1 : 0) + (by_chunks(a) ? 1 : 0); }
bool delta_step_fits(int H, int Hk, int d, int dv, int taps) {
    return Hk >= 1 && H % Hk == 0 && d >= 1 && d <= 256 && dv >= 1 && (H / Hk) * ((dv + 31) / 32) <= 8 && taps >= 1 && taps <= DS_TAPS;
}
int delta_step_launch(cudaStream_t st, const RaggedBatch& rb, const DeltaArgs& a) {
    if (!delta_step_fits(a.H, a.Hk, a.d, a.dv, a.taps) || rb.T != rb.E || a.a_rank > 4096 || a.g_rank > 4096 || (a.w_a2 && (!a.w_g2 || ((a.ld_a2 | a.ld_g2) & 3)))) return -1000;
    static_assert(DS_CONV * DS_NT >= 2 * 256 + 32, "a block's channels");
    const int nz = (a.dv + 31) / 32;
    const size_t smem = (size_t)(a.a_rank + a.g_rank + 8) * sizeof(float);
    static SmemOptIn seen[4];
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.H * nz, rb.E); cfg.blockDim = dim3(DS_NT); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = (a.H / a.Hk) * nz; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr; cfg.numAttrs = 1;
    auto run = [&](auto k, SmemOptIn& s) -> int {
        if (const int e = ensure_dyn_smem(k, smem, s)) return e;
        return (int)cudaLaunchKernelEx(&cfg, k, rb, a);
    };
    return a.d <= 32 ? run(delta_step_kernel<4>, seen[0]) : a.d <= 64 ? run(delta_step_kernel<8>, seen[1]) : a.d <= 128 ? run(delta_step_kernel<16>, seen[2]) : run(delta_step_kernel<32>, seen[3]);
}
int delta_mixer_launch(cudaStream_t st, const RaggedBatch& rb, const DeltaArgs& a) {
    if (a.d < 1 || a.d > 256 || a.dv < 1 || a.Hk < 1 || a.H % a.Hk || a.taps < 1 || !a.conv_w || (a.taps > 1 && !a.conv_state)) return -1000;
    const int units = a.Hk + a.H + (a.per_channel ? a.H : 0) + 1, tile = a.single_rows ? 1 : rb.T >= 1024 ? DP_ROWS : 4, w = std::max(a.d, std::min(a.dv, 128));
    const dim3 pgrid((rb.T + tile - 1) / tile, (units + 3) / 4);
    auto prep = [&](auto k0, auto k1, auto k2, auto k3, auto k4) {
        auto k = a.taps == 1 ? k1 : a.taps == 2 ? k2 : a.taps == 3 ? k3 : a.taps == 4 ? k4 : k0;
        k<<<pgrid, 128, 0, st>>>(rb, a, tile);
    };
    if (w <= 64) prep(delta_prep_kernel<2, 0>, delta_prep_kernel<2, 1>, delta_prep_kernel<2, 2>, delta_prep_kernel<2, 3>, delta_prep_kernel<2, 4>);
    else if (w <= 128) prep(delta_prep_kernel<4, 0>, delta_prep_kernel<4, 1>, delta_prep_kernel<4, 2>, delta_prep_kernel<4, 3>, delta_prep_kernel<4, 4>);
    else prep(delta_prep_kernel<8, 0>, delta_prep_kernel<8, 1>, delta_prep_kernel<8, 2>, delta_prep_kernel<8, 3>, delta_prep_kernel<8, 4>);
    int e = last_err();
    if (e) return e;
    if (!a.single_rows && a.taps > 1) {
        CausalConvArgs ca = {};
        ca.in = a.proj + a.col0; ca.ld = a.ld; ca.C = 2 * a.Hk * a.d + a.H * a.dv; ca.taps = a.taps; ca.state = a.conv_state;
        if ((e = causal_conv_window_launch(st, rb, ca))) return e;
    }
    const int nr = (a.d + DR_NS - 1) / DR_NS, R = nr <= 2 ? 2 : nr <= 4 ? 4 : nr <= 8 ? 8 : nr <= 16 ? 16 : 32;
    const size_t smem = (size_t)(2 * DR_CH * ((a.per_channel ? 3 : 2) * dr_pad(R) + DR_COLS + 4) + DR_CH * DR_COLS) * sizeof(float);      // <= 113 KB at d = 256
    static SmemOptIn seen[2][5];
    auto run = [&](auto kern, SmemOptIn& s) -> int {
        if (const int er = ensure_dyn_smem(kern, smem, s)) return er;
        kern<<<dim3(rb.E, a.H, (a.dv + DR_COLS - 1) / DR_COLS), DR_COLS * DR_NS, smem, st>>>(rb, a);
        return last_err();
    };
    if (by_chunks(a)) e = delta_chunk_launch(st, rb, a);
    else if (a.per_channel) e = R == 2 ? run(delta_scan_kernel<2, true>, seen[1][0]) : R == 4 ? run(delta_scan_kernel<4, true>, seen[1][1]) : R == 8 ? run(delta_scan_kernel<8, true>, seen[1][2])
                         : R == 16 ? run(delta_scan_kernel<16, true>, seen[1][3]) : run(delta_scan_kernel<32, true>, seen[1][4]);
    else e = R == 2 ? run(delta_scan_kernel<2, false>, seen[0][0]) : R == 4 ? run(delta_scan_kernel<4, false>, seen[0][1]) : R == 8 ? run(delta_scan_kernel<8, false>, seen[0][2])
           : R == 16 ? run(delta_scan_kernel<16, false>, seen[0][3]) : run(delta_scan_kernel<32, false>, seen[0][4]);
    if (e) return e;
    delta_out_kernel<<<(rb.T * a.H + 3) / 4, 128, 0, st>>>(a, rb.T);
    return last_err();
}
int token_gate_launch(cudaStream_t st, const float* z, int ldz, int T, int n, const int* ids, const bf16* table, int ldt, int col0, const ActOut& out) {
    if (n < 1) return -1000;
    token_gate_kernel<<<dim3((n + 127) / 128, T), 128, 0, st>>>(z, ldz, n, ids, table, ldt, col0, out);
    return last_err();
}
int token_gate_step_launch(cudaStream_t st, const float* x, int ldx, const bf16* w, int ldw, int K, int T, int n, const int* ids, const bf16* table, int ldt,
                           int col0, const ActOut& out) {
    if (n < 1 || (K & 7) || (ldw & 7) || (ldx & 3)) return -1000;
    token_gate_step_kernel<<<dim3(n, T), 128, 0, st>>>(x, ldx, w, ldw, K, ids, table, ldt, col0, out);
    return last_err();
}

}  // namespace cb
