// Attention of a few rows whose heads all read ONE key row per token (latent attention; scores mixed over the heads as products with all key
// heads side by side).  A row's heads then form the M side of a matrix product with the keys: block = (row, sixteen heads, split of the keys),
// every cached byte comes to an SM once for all of them, scores and weighted sums run on the tensor cores (bf16 pairs hi + lo keep the three
// leading terms of every product), the softmax between them in f32.  Splits leave (maximum, sum, unnormalised output) in the scratch
// that sink_attention_merge_kernel -- or the head-wise linear that follows -- joins in split order.
#include "ragged.cuh"
#include "ragged_dev.cuh"
#include "decode.cuh"

#include <algorithm>

namespace cb {

namespace {

inline int last_err() { return (int)cudaGetLastError(); }

constexpr int SK_WARPS = 8, SK_KEYS = 32, SK_HEADS = 16, SK_LDP = SK_KEYS + 8;

__device__ __forceinline__ void sk_ldsm4(uint32_t* r, const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void sk_ldsm2(uint32_t* r, const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void sk_ldsm4t(uint32_t* r, const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void sk_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16z(void* dst, const void* src, bool in) {      // zeros where the source is past the end
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(in ? 16 : 0) : "memory");
}

struct SkGeom { int ldk, ldv, stage, smem; };      // row strides (elements) of staged keys and values; elements per stage; bytes in all
inline __host__ __device__ SkGeom sk_geom(int d, int vcols, bool shared, int planes, int stages) {
    SkGeom g;
    g.ldk = (d + 15) / 16 * 16 + 8;
    g.ldv = shared ? g.ldk : vcols + 8;
    g.stage = planes * SK_KEYS * (g.ldk + (shared ? 0 : g.ldv));
    g.smem = (planes * SK_HEADS * g.ldk + stages * g.stage + 2 * SK_HEADS * SK_LDP) * 2 + (2 * SK_HEADS * (SK_KEYS + 1) + 3 * SK_HEADS) * 4;
    return g;
}

// NT: 8-column tiles of the output per warp
template <bool SPLIT, int NT>
__global__ void __launch_bounds__(SK_WARPS * 32) shared_key_kernel(RaggedBatch rb, SinkAttnArgs a, int stages) {
    extern __shared__ __align__(16) unsigned char sksm[];
    constexpr int P = SPLIT ? 2 : 1;
    const int r = blockIdx.x, h0 = blockIdx.y * SK_HEADS, sp = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int nh = min(SK_HEADS, a.H - h0), d = a.d, v_row = a.v_row ? a.v_row : a.dv, vt = (a.dv + 7) / 8, vcols = a.G * vt * 8;
    const bool shared = a.kv_shared != 0;
    const SkGeom ge = sk_geom(d, vcols, shared, P, stages);
    const int ldk = ge.ldk, ldv = ge.ldv, dk16 = (d + 15) / 16;
    bf16* sq = reinterpret_cast<bf16*>(sksm);                 // [P][16][ldk]
    bf16* ring = sq + P * SK_HEADS * ldk;                     // [stages][K hi | K lo | V hi | V lo]
    bf16* pp = ring + (size_t)stages * ge.stage;              // [2][16][SK_LDP] probabilities hi, lo
    float* ss = reinterpret_cast<float*>(pp + 2 * SK_HEADS * SK_LDP);      // [2][16][33] scores, one half of the columns each
    float* sm_m = ss + 2 * SK_HEADS * (SK_KEYS + 1);
    float* sm_l = sm_m + SK_HEADS;
    float* sm_c = sm_l + SK_HEADS;
    const int e = rb.row_entry[r], pos = rb.row_pos[r], slot = rb.ent_slot[e];
    const int* bt = a.block_table + (size_t)slot * a.max_pages;
    const int nkeys = pos + 1, key0 = (a.window > 0 && nkeys > a.window) ? nkeys - a.window : 0;
    const int t0 = key0 / SK_KEYS, n_all = (nkeys + SK_KEYS - 1) / SK_KEYS - t0, per = (n_all + a.nsplit - 1) / a.nsplit;
    const int lo = min(n_all, sp * per), n = min(n_all, lo + per) - lo;
    auto load = [&](int i, int st) {
        const int k0 = (t0 + lo + i) * SK_KEYS, cnt = min(SK_KEYS, nkeys - k0);
        const size_t page = (size_t)bt[k0 / KV_PAGE];         // (a 32-key tile never straddles a 64-token page)
        const bf16* kp = (const bf16*)a.k_pool + (page * KV_PAGE + k0 % KV_PAGE) * d;
        bf16* ks = ring + (size_t)st * ge.stage;
        const int kc = dk16 * 2;                              // 16-byte pieces per key row, zeros behind the row's own
        for (int q = tid; q < P * SK_KEYS * kc; q += SK_WARPS * 32) {
            const int pl = q / (SK_KEYS * kc), row = q / kc % SK_KEYS, ch = q % kc;
            const bool in = row < cnt && ch * 8 < d;
            cp_async16z(ks + ((size_t)pl * SK_KEYS + row) * ldk + ch * 8, kp + (in ? (size_t)row * d + ch * 8 + (pl ? a.kv_lo_off : 0) : 0), in);
        }
        if (!shared) {
            bf16* vs = ks + (size_t)P * SK_KEYS * ldk;
            const int per_row = a.G * vt;
            for (int q = tid; q < P * SK_KEYS * per_row; q += SK_WARPS * 32) {
                const int pl = q / (SK_KEYS * per_row), row = q / per_row % SK_KEYS, g = q % per_row / vt, ch = q % vt;
                const bool in = row < cnt;
                const bf16* vp = (const bf16*)a.v_pool + ((page * a.G + g) * KV_PAGE + k0 % KV_PAGE + (in ? row : 0)) * v_row + ch * 8;
                cp_async16z(vs + ((size_t)pl * SK_KEYS + row) * ldv + (g * vt + ch) * 8, vp + (pl ? a.kv_lo_off : 0), in);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (n > 0) load(0, 0);
    // queries times the scale, as bf16 planes; rows past the last head and columns past the width are zeros
    for (int i = tid; i < SK_HEADS * dk16 * 16; i += SK_WARPS * 32) {
        const int h = i / (dk16 * 16), c = i % (dk16 * 16);
        const float v = (h < nh && c < d) ? a.q[(size_t)r * a.ldq + (size_t)(h0 + h) * d + c] * a.scale : 0.f;
        const bf16 hi = __float2bfloat16_rn(v);
        sq[h * ldk + c] = hi;
        if (SPLIT) sq[SK_HEADS * ldk + h * ldk + c] = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
    if (tid < SK_HEADS) { sm_m[tid] = -INFINITY; sm_l[tid] = 0.f; }
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) { acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f; }
    const int g4 = lane >> 2, tq = lane & 3, total = a.G * vt;
    for (int i = 0; i < n; ++i) {
        const int st = stages == 2 ? (i & 1) : 0, k0 = (t0 + lo + i) * SK_KEYS;
        if (stages == 2 && i + 1 < n) { load(i + 1, st ^ 1); asm volatile("cp.async.wait_group 1;" ::: "memory"); }
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const bf16* ks = ring + (size_t)st * ge.stage;
        {   // scores: a warp takes eight keys and one half of the width
            const int kt = warp & 3, half = warp >> 2, mid = (dk16 + 1) / 2, c0 = half ? mid : 0, c1 = half ? dk16 : mid;
            float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
            for (int kk = c0; kk < c1; ++kk) {
                uint32_t qh[4], kh[2];
                const int qo = ((lane & 7) + ((lane >> 3) & 1) * 8) * ldk + kk * 16 + (lane >> 4) * 8;
                const int ko = (kt * 8 + (lane & 7)) * ldk + kk * 16 + ((lane >> 3) & 1) * 8;
                sk_ldsm4(qh, sq + qo);
                sk_ldsm2(kh, ks + ko);
                if (SPLIT) {
                    uint32_t ql[4], kl[2];
                    sk_ldsm4(ql, sq + SK_HEADS * ldk + qo);
                    sk_ldsm2(kl, ks + SK_KEYS * ldk + ko);
                    sk_mma(s2, ql, kh[0], kh[1]);
                    sk_mma(s2, qh, kl[0], kl[1]);
                }
                sk_mma(s, qh, kh[0], kh[1]);
            }
            float* d0 = ss + (half * SK_HEADS + g4) * (SK_KEYS + 1) + kt * 8 + tq * 2;
            d0[0] = s[0] + s2[0]; d0[1] = s[1] + s2[1];
            d0[8 * (SK_KEYS + 1)] = s[2] + s2[2]; d0[8 * (SK_KEYS + 1) + 1] = s[3] + s2[3];
        }
        __syncthreads();
        for (int h = warp; h < SK_HEADS; h += SK_WARPS) {     // lane = key
            const int j = k0 + lane;
            const bool seen = j < nkeys && j >= key0;
            const float sv = seen ? ss[h * (SK_KEYS + 1) + lane] + ss[(SK_HEADS + h) * (SK_KEYS + 1) + lane] : -INFINITY;
            const float mo = sm_m[h], mn = fmaxf(mo, warp_max(sv));
            const float p = seen ? __expf(sv - mn) : 0.f, corr = mo == -INFINITY ? 0.f : __expf(mo - mn), sum = warp_sum(p);
            const bf16 hi = __float2bfloat16_rn(p);
            pp[h * SK_LDP + lane] = hi;
            pp[(SK_HEADS + h) * SK_LDP + lane] = __float2bfloat16_rn(p - __bfloat162float(hi));
            __syncwarp();
            if (lane == 0) { sm_m[h] = mn; sm_l[h] = sm_l[h] * corr + sum; sm_c[h] = corr; }
        }
        __syncthreads();
        {   // weighted sums: a warp takes every eighth 8-column tile (of all value heads; a head keeps its own value head's columns)
            const float cl = sm_c[g4], ch = sm_c[g4 + 8];
            const bf16* vs = shared ? ks : ks + (size_t)P * SK_KEYS * ldk;
            uint32_t ph[2][4], pl[2][4];
#pragma unroll
            for (int kt = 0; kt < 2; ++kt) {
                const int po = ((lane & 7) + ((lane >> 3) & 1) * 8) * SK_LDP + kt * 16 + (lane >> 4) * 8;
                sk_ldsm4(ph[kt], pp + po);
                sk_ldsm4(pl[kt], pp + SK_HEADS * SK_LDP + po);
            }
#pragma unroll
            for (int q = 0; q < NT; ++q) {
                const int tile = warp + q * SK_WARPS;
                acc[q][0] *= cl; acc[q][1] *= cl; acc[q][2] *= ch; acc[q][3] *= ch;
                if (tile >= total) continue;
                uint32_t v[4];                                // keys 0..7, 8..15, 16..23, 24..31 of the tile's eight columns
                sk_ldsm4t(v, vs + lane * ldv + tile * 8);
                sk_mma(acc[q], pl[0], v[0], v[1]); sk_mma(acc[q], pl[1], v[2], v[3]);
                if (SPLIT) {
                    uint32_t w[4];
                    sk_ldsm4t(w, vs + (size_t)SK_KEYS * ldv + lane * ldv + tile * 8);
                    sk_mma(acc[q], ph[0], w[0], w[1]); sk_mma(acc[q], ph[1], w[2], w[3]);
                }
                sk_mma(acc[q], ph[0], v[0], v[1]); sk_mma(acc[q], ph[1], v[2], v[3]);
            }
        }
        __syncthreads();                                      // the stage and the probabilities are free
        if (stages == 1 && i + 1 < n) load(i + 1, 0);
    }
    if (n == 0) __syncthreads();
    const int rep = a.H / a.G;
#pragma unroll
    for (int q = 0; q < NT; ++q) {
        const int tile = warp + q * SK_WARPS;
        if (tile >= total) continue;
        const int g = tile / vt, c = (tile % vt) * 8 + tq * 2;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const int h = g4 + (w >> 1) * 8, col = c + (w & 1);
            if (h < nh && (h0 + h) / rep == g && col < a.dv) a.part[(((size_t)r * a.H + h0 + h) * a.nsplit + sp) * (a.dv + 2) + 2 + col] = acc[q][w];
        }
    }
    if (tid < nh) {
        float* o = a.part + (((size_t)r * a.H + h0 + tid) * a.nsplit + sp) * (a.dv + 2);
        o[0] = sm_m[tid]; o[1] = sm_l[tid];
    }
}

}  // namespace

int shared_key_heads() { return SK_HEADS; }
int shared_key_tile() { return SK_KEYS; }
bool shared_key_fits(int d, int G, int dv, bool kv_shared, bool split) {
    const int vcols = G * ((dv + 7) / 8) * 8;
    return (d & 7) == 0 && vcols <= 1024 && sk_geom(d, vcols, kv_shared, split ? 2 : 1, 1).smem <= 220 * 1024;
}
int shared_key_attention_launch(cudaStream_t st, const RaggedBatch& rb, const SinkAttnArgs& a) {
    const bool split = a.kv_lo_off != 0;
    const int v_row = a.v_row ? a.v_row : a.dv, vt = (a.dv + 7) / 8, planes = split ? 2 : 1;
    if (a.kv_f32 || (a.Gk ? a.Gk : a.G) != 1 || a.H % a.G || a.gate || a.softcap > 0.f || a.dist_r1 || a.dist_table || a.keep_first || !a.part || a.nsplit < 1 || a.nsplit > 64) return -1000;
    if (!shared_key_fits(a.d, a.G, a.dv, a.kv_shared != 0, split) || (v_row & 7) || v_row < vt * 8) return -1000;
    if (a.kv_shared && (a.k_pool != a.v_pool || v_row != a.d)) return -1000;
    const int stages = sk_geom(a.d, a.G * vt * 8, a.kv_shared != 0, planes, 2).smem <= 220 * 1024 ? 2 : 1;
    const size_t smem = sk_geom(a.d, a.G * vt * 8, a.kv_shared != 0, planes, stages).smem;
    const dim3 grid(rb.T, (a.H + SK_HEADS - 1) / SK_HEADS, a.nsplit);
    const int nt = (a.G * vt + SK_WARPS - 1) / SK_WARPS;
    auto go = [&](auto kern, SmemOptIn& seen) -> int {
        if (const int e = ensure_dyn_smem(kern, smem, seen)) return e;
        kern<<<grid, SK_WARPS * 32, smem, st>>>(rb, a, stages);
        return last_err();
    };
    static SmemOptIn seen[6];
    if (split) return nt <= 4 ? go(shared_key_kernel<true, 4>, seen[0]) : nt <= 8 ? go(shared_key_kernel<true, 8>, seen[1]) : go(shared_key_kernel<true, 16>, seen[2]);
    return nt <= 4 ? go(shared_key_kernel<false, 4>, seen[3]) : nt <= 8 ? go(shared_key_kernel<false, 8>, seen[4]) : go(shared_key_kernel<false, 16>, seen[5]);
}

}  // namespace cb
