// The residual as several parallel copies of the stream (see ragged.cuh): what lies between two sublayers is one pass over a row --
// the last sublayer's output joins the copies through their mixing table, the next sublayer's input is their weighted sum, and its RMS
// norm leaves as the linears' operand.  f32 throughout; a row's result depends on that row only.
#include "ragged.cuh"
#include "ragged_dev.cuh"

#include <algorithm>

namespace cb {

namespace {

inline int last_err() { return (int)cudaGetLastError(); }

// Block per row, NC columns per thread, everything the row needs requested up front: one trip to memory.  The sum of squares is a
// thread's columns in order, the warp's tree, the warps in order.
template <int S, int NC>
__global__ void __launch_bounds__(1024) stream_rows_kernel(StreamArgs a) {
    __shared__ float red[32];
    const int r = blockIdx.x, src = a.rows ? a.rows[r] : r, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
    float* xr = a.xs + (size_t)src * S * a.ldx;
    float x[NC][S], yv[NC], wn[NC];
    const bf16* e = a.ids ? a.embed + (size_t)a.ids[src] * a.W : nullptr;
#pragma unroll
    for (int k = 0; k < NC; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        const bool in = c < a.W;
        if (e) {
            const float v = in ? __bfloat162float(e[c]) : 0.f;
#pragma unroll
            for (int s = 0; s < S; ++s) x[k][s] = v;
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s) x[k][s] = in ? xr[(size_t)s * a.ldx + c] : 0.f;
        }
        yv[k] = (in && a.y) ? a.y[(size_t)src * a.ldy + c] : 0.f;
        wn[k] = in ? a.norm_w[c] : 0.f;
    }
    float cin[S];
#pragma unroll
    for (int s = 0; s < S; ++s) cin[s] = a.in ? a.in[s] : 1.f;
    if (a.y) {
        float m[S][S], o[S];
#pragma unroll
        for (int s = 0; s < S; ++s) {
            o[s] = a.out[s];
#pragma unroll
            for (int t = 0; t < S; ++t) m[s][t] = a.mix[s * S + t];
        }
#pragma unroll
        for (int k = 0; k < NC; ++k) {
            float nx[S];
#pragma unroll
            for (int t = 0; t < S; ++t) {
                nx[t] = o[t] * yv[k];
#pragma unroll
                for (int s = 0; s < S; ++s) nx[t] = fmaf(m[s][t], x[k][s], nx[t]);
            }
#pragma unroll
            for (int t = 0; t < S; ++t) x[k][t] = nx[t];
        }
    }
    float u[NC], ss = 0.f;
#pragma unroll
    for (int k = 0; k < NC; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        u[k] = 0.f;
#pragma unroll
        for (int s = 0; s < S; ++s) u[k] = fmaf(cin[s], x[k][s], u[k]);
        ss = fmaf(u[k], u[k], ss);
        if (a.store && c < a.W) {
#pragma unroll
            for (int s = 0; s < S; ++s) xr[(size_t)s * a.ldx + c] = x[k][s];
        }
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < nwarp; ++w) tot += red[w];
    const float inv = 1.f / sqrtf(tot / (float)a.W + a.eps);
#pragma unroll
    for (int k = 0; k < NC; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        if (c < a.W) store_act(a.h, r, c, u[k] * inv * wn[k]);
    }
}

template <int S>
int stream_rows_s(cudaStream_t st, const StreamArgs& a, int R) {
    // many rows: small blocks, more columns per thread; a few rows: one column per thread as far as that goes
    const int want = R > 16 ? 256 : 1024, threads = std::min(want, (a.W + 31) / 32 * 32), nc = (a.W + threads - 1) / threads;
    auto go = [&](auto kern, int n) { kern<<<R, std::min(1024, ((a.W + n - 1) / n + 31) / 32 * 32), 0, st>>>(a); return last_err(); };
    if (nc <= 1) return go(stream_rows_kernel<S, 1>, 1);
    if (nc <= 2) return go(stream_rows_kernel<S, 2>, 2);
    if (nc <= 4) return go(stream_rows_kernel<S, 4>, 4);
    return go(stream_rows_kernel<S, 8>, 8);
}

}  // namespace

int stream_rows_launch(cudaStream_t st, const StreamArgs& a, int R) {
    if (a.W < 1 || a.W > STREAM_MAX_W || (!a.ids && !a.xs) || (a.store && !a.xs) || (a.y && (!a.mix || !a.out))) return -1000;
    switch (a.S) {
        case 1: return stream_rows_s<1>(st, a, R);
        case 2: return stream_rows_s<2>(st, a, R);
        case 3: return stream_rows_s<3>(st, a, R);
        case 4: return stream_rows_s<4>(st, a, R);
        case 5: return stream_rows_s<5>(st, a, R);
        case 6: return stream_rows_s<6>(st, a, R);
        case 7: return stream_rows_s<7>(st, a, R);
        case 8: return stream_rows_s<8>(st, a, R);
        default: return -1000;
    }
}

}  // namespace cb
