// seq_ssm.cuh -- the state-space mixer of the layered sequence engine (scalar decay per head, shared input / output maps per group):
//
//     [z | x | B | C | dt] = W_in h                 x, B, C: causal depth-wise convolution with bias and silu (short_conv_* of seq_headmix.cuh)
//     dt <- softplus(dt + dt_bias)
//     S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T     S: [N state rows][dv value columns] per head, fp32, one per live sequence
//     y_t = S_t^T C_t + D x_t                                   (head h reads the B, C of group h / (heads / groups))
//     y <- rms_parts(y * silu(z)) * norm                        (each of `parts` equal pieces by its own root mean square)
//
// ssm_scan_kernel runs the recurrence token by token; the other kernels finish a row.  Everything is fp32 in both compute modes.
#pragma once
#include "seq_headmix.cuh"
#include "seq_kernels.cuh"

namespace tib {
namespace seq {

__device__ __forceinline__ float softplus_f32(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

// Few rows, attention and a state-space mixer side by side: the attention's preparation of row blockIdx.x (blockIdx.y 0) and the
// convolution in front of the state-space recurrence (the other blockIdx.y) in one launch -- both only read the front product.
__global__ void __launch_bounds__(kPrepareFewThreads) attn_prepare_conv_kernel(float* qkvg, StepMeta m, AttnShape s, const float* inv_freq, float* k_pool, float* v_pool,
                                                                              const float* x, ConvForm f, int channels, int taps, const float* w, float* state, float* y) {
    pdl_launch_dependents();
    pdl_wait_prior_grid();
    if (blockIdx.y == 0) attn_prepare_row(blockIdx.x, qkvg, m, s, inv_freq, k_pool, v_pool);
    else short_conv_row<1>(blockIdx.x, (blockIdx.y - 1) * blockDim.x + threadIdx.x, (gridDim.y - 1) * blockDim.x, x, f, m, channels, taps, w, state, y);
}

struct SsmArgs {
    const float* xbc;             // [T][ld]: x [heads * dv], B [groups * N], C [groups * N] behind the convolution
    int ld;
    const float* dt;              // row t, head h at [t * ld_dt + h], as projected
    int ld_dt;
    const float *dt_bias, *A_log; // [heads]
    float* state;                 // [slots][heads][N][dv]
    float* out;                   // S^T C: row t, head h at [t * ldo + h * dv]
    int ldo;
    int heads, N, dv, groups;
};

// One block per (entry, head, 32 value columns): 8 warps split the state rows, a lane keeps RP entries of its column in registers
// (N <= 8 RP; rows behind N carry zeros).  Tokens are taken 8 at a time: warp c stages token c's B, C, decay and dt x while the
// operands of the next eight are already requested; every warp runs the eight tokens over its rows and leaves a partial output per
// token; the partials are summed in warp order.
constexpr int kSsmChunk = 8;
template <int RP>
__global__ void __launch_bounds__(256) ssm_scan_kernel(SsmArgs a, StepMeta m) {
    pdl_launch_dependents();
    pdl_wait_prior_grid();
    constexpr int CH = kSsmChunk, NP = 8 * RP, PER = (NP + 31) / 32;
    __shared__ __align__(16) float Bs[CH][NP], Cs[CH][NP];
    __shared__ float xs[CH][32], dec[CH];
    __shared__ float part[8][CH][32];
    const int e = blockIdx.x, hd = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int N = a.N, dv = a.dv, j = blockIdx.z * 32 + lane, g = hd / (a.heads / a.groups);
    const bool own = j < dv;
    const int offB = a.heads * dv + g * N, offC = offB + a.groups * N;
    float* Sg = a.state + ((size_t)m.ent_slot[e] * a.heads + hd) * (size_t)N * dv;
    const bool fresh = (m.ent_pos0[e] == 0);
    const float rate = -expf(a.A_log[hd]), bias = a.dt_bias[hd];
    float S[RP];
#pragma unroll
    for (int i = 0; i < RP; ++i) S[i] = (own && !fresh && warp * RP + i < N) ? Sg[(size_t)(warp * RP + i) * dv + j] : 0.f;
    const int t0 = m.ent_row0[e], t1 = m.ent_row0[e + 1];
    float nB[PER], nC[PER], nx, ndt;
    auto fetch = [&](int tc) {   // warp c: token tc + c
        const size_t t = (size_t)min(tc + warp, t1 - 1);
        const float* row = a.xbc + t * a.ld;
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int n = lane + 32 * p;
            nB[p] = n < N ? row[offB + n] : 0.f;
            nC[p] = n < N ? row[offC + n] : 0.f;
        }
        nx = own ? row[hd * dv + j] : 0.f;
        ndt = a.dt[t * a.ld_dt + hd];
    };
    auto emit = [&](int tc) {
        const int t = tc + warp;
        if (t < t1 && own) {
            float s = part[0][warp][lane];
#pragma unroll
            for (int w = 1; w < 8; ++w) s += part[w][warp][lane];
            a.out[(size_t)t * a.ldo + (size_t)hd * dv + j] = s;
        }
    };
    fetch(t0);
    for (int tc = t0; tc < t1; tc += CH) {
        if (tc > t0) emit(tc - CH);
        const float dt = softplus_f32(ndt + bias);
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int n = lane + 32 * p;
            if (n < NP) {
                Bs[warp][n] = nB[p];
                Cs[warp][n] = nC[p];
            }
        }
        xs[warp][lane] = dt * nx;
        if (lane == 0) dec[warp] = expf(rate * dt);
        __syncthreads();
        if (tc + CH < t1) fetch(tc + CH);
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            if (tc + c < t1) {
                const float v = xs[c][lane], d = dec[c];
                float acc0 = 0.f, acc1 = 0.f, acc2 = 0.f, acc3 = 0.f;
#pragma unroll
                for (int i = 0; i < RP; i += 4) {
                    const float4 b4 = *reinterpret_cast<const float4*>(&Bs[c][warp * RP + i]);
                    const float4 c4 = *reinterpret_cast<const float4*>(&Cs[c][warp * RP + i]);
                    S[i] = fmaf(d, S[i], b4.x * v);
                    acc0 = fmaf(c4.x, S[i], acc0);
                    S[i + 1] = fmaf(d, S[i + 1], b4.y * v);
                    acc1 = fmaf(c4.y, S[i + 1], acc1);
                    S[i + 2] = fmaf(d, S[i + 2], b4.z * v);
                    acc2 = fmaf(c4.z, S[i + 2], acc2);
                    S[i + 3] = fmaf(d, S[i + 3], b4.w * v);
                    acc3 = fmaf(c4.w, S[i + 3], acc3);
                }
                part[warp][c][lane] = (acc0 + acc1) + (acc2 + acc3);
            }
        }
        __syncthreads();
    }
    emit(t0 + (t1 - t0 - 1) / CH * CH);
    if (own) {
#pragma unroll
        for (int i = 0; i < RP; ++i)
            if (warp * RP + i < N) Sg[(size_t)(warp * RP + i) * dv + j] = S[i];
    }
}
constexpr int kSsmMaxState = 8 * 64;   // the largest instantiation

// y = (y + D x) silu(z) -> y / rms(y) over the part * w * scale, in place (row stride ldy): one block per (row, part)
struct SsmFinishArgs {
    float* y;
    int ldy;
    const float *x, *z;   // row strides ldx, ldz
    int ldx, ldz;
    const float *D, *w;   // [heads], [inner]
    int inner, dv, parts;
    float eps, scale;
};
__global__ void ssm_finish_kernel(SsmFinishArgs a) {
    pdl_launch_dependents();
    pdl_wait_prior_grid();
    __shared__ float red[32];
    const size_t t = blockIdx.x;
    const int size = a.inner / a.parts, c0 = blockIdx.y * size;
    float* y = a.y + t * a.ldy + c0;
    const float *x = a.x + t * a.ldx + c0, *z = a.z + t * a.ldz + c0;
    float ss = 0.f;
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
        const float zv = z[i], v = fmaf(a.D[(c0 + i) / a.dv], x[i], y[i]) * (zv / (1.f + expf(-zv)));
        y[i] = v;   // (the thread that wrote it scales it below)
        ss += v * v;
    }
    ss = block_sum(ss, red);
    const float sc = a.scale / sqrtf(ss / (float)size + a.eps);
    for (int i = threadIdx.x; i < size; i += blockDim.x) y[i] *= sc * a.w[c0 + i];
}

}  // namespace seq
}  // namespace tib
