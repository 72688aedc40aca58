// seq_delta.cuh -- the gated delta rule of the layered sequence engine (a linear recurrence whose write removes what the state already
// answers for the key), beside the gated linear recurrences of seq_recurrent.cuh:
//
//     q, k, v behind causal depth-wise convolutions and silu (short_conv_* of seq_headmix.cuh), side by side in one row
//     k <- k / sqrt(sum k^2 + 1e-6), q <- q / sqrt(sum q^2 + 1e-6) * qscale           per head
//     g = exp(-exp(A_log) softplus(a + dt_bias)), beta = sigmoid(b)                   one number a head
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q                    S: [dk][dv] per head, fp32, one per live sequence
//
// Value head h reads the q and k of head h / (heads / kv_heads).  The columns of S are independent of one another, so column j lives in
// the registers of eight lanes of a warp (each holds an eighth of the key channels), and a token costs one round of three shuffles:
// both S^T k and S^T q are taken from the state before the write, o = g (S^T q) + (k . q) u.  Everything is fp32 in both compute modes.
#pragma once
#include "seq_kernels.cuh"
#include "seq_ssm.cuh"

namespace tib {
namespace seq {

struct DeltaArgs {
    const float* qkv;             // [T][ld]: q [kv_heads * dk] | k [kv_heads * dk] | v [heads * dv] behind convolution and silu
    int ld;
    const float *a, *b;           // row t, head h at [t * ld_ab + h], as projected
    int ld_ab;
    const float *dt_bias, *A_log; // [heads]
    float* state;                 // [slots][heads][dv][dk] (a column of S is contiguous)
    float* out;                   // row t, head h at [t * ldo + h * dv]
    int ldo;
    int heads, kv_heads, dk, dv;
    float qscale;
};

constexpr float kUnitEps = 1e-6f;
constexpr int kDeltaCols = 16;    // value columns of a block: 4 warps x 4 columns
// RP key channels a lane: dk <= 8 RP.  Lane p = lane % 8 of a column holds channels 4 (p + 8 i) .. + 3, i < RP / 4.
template <int RP, int CH>
__global__ void __launch_bounds__(128) delta_scan_kernel(DeltaArgs a, StepMeta m) {
    pdl_launch_dependents();
    pdl_wait_prior_grid();
    constexpr int NP = 8 * RP, PER = NP / 32, TPW = CH / 4;   // PER: values of a token's q (k) a lane stages; TPW: tokens of a chunk a warp stages
    static_assert(RP % 4 == 0 && CH % 4 == 0 && CH <= 8, "layout");
    __shared__ __align__(16) float ks[CH][NP], qs[CH][NP];
    __shared__ float vs[CH][kDeltaCols], gs[CH], bs[CH], kqs[CH];
    const int e = blockIdx.x, hd = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int dk = a.dk, dv = a.dv, p = lane & 7, cl = warp * 4 + (lane >> 3), col0 = blockIdx.z * kDeltaCols, j = col0 + cl;
    const int G = a.kv_heads, kh = hd / (a.heads / G);
    const int offq = kh * dk, offk = (G + kh) * dk, offv = 2 * G * dk + hd * dv + col0;
    const bool own = j < dv, vec = dk % 4 == 0;
    float* Sg = a.state + (((size_t)m.ent_slot[e] * a.heads + hd) * (size_t)dv + min(j, dv - 1)) * dk;
    const bool fresh = (m.ent_pos0[e] == 0);
    const float rate = -expf(a.A_log[hd]), bias = a.dt_bias[hd];
    float S[RP];
#pragma unroll
    for (int i = 0; i < RP / 4; ++i) {
        const int c = 4 * (p + 8 * i);
        if (fresh || !own) {
            S[4 * i] = S[4 * i + 1] = S[4 * i + 2] = S[4 * i + 3] = 0.f;
        } else if (vec) {
            const float4 v = c < dk ? *reinterpret_cast<const float4*>(Sg + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            S[4 * i] = v.x; S[4 * i + 1] = v.y; S[4 * i + 2] = v.z; S[4 * i + 3] = v.w;
        } else {
#pragma unroll
            for (int x = 0; x < 4; ++x) S[4 * i + x] = c + x < dk ? Sg[c + x] : 0.f;
        }
    }
    const int t0 = m.ent_row0[e], t1 = m.ent_row0[e + 1];
    float nq[TPW][PER], nk[TPW][PER], nv[TPW], na[TPW], nb[TPW];
    auto fetch = [&](int tc) {   // warp w: tokens tc + w, tc + w + 4
#pragma unroll
        for (int x = 0; x < TPW; ++x) {
            const size_t t = (size_t)min(tc + warp + 4 * x, t1 - 1);
            const float* row = a.qkv + t * a.ld;
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int c = lane + 32 * i;
                nq[x][i] = c < dk ? row[offq + c] : 0.f;
                nk[x][i] = c < dk ? row[offk + c] : 0.f;
            }
            nv[x] = lane < kDeltaCols && col0 + lane < dv ? row[offv + lane] : 0.f;
            na[x] = a.a[t * a.ld_ab + hd];
            nb[x] = a.b[t * a.ld_ab + hd];
        }
    };
    fetch(t0);
    for (int tc = t0; tc < t1; tc += CH) {
#pragma unroll
        for (int x = 0; x < TPW; ++x) {   // unit key, unit scaled query, their product, decay and step size
            const int c = warp + 4 * x;
            float sq = 0.f, sk = 0.f, kq = 0.f;
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                sq = fmaf(nq[x][i], nq[x][i], sq);
                sk = fmaf(nk[x][i], nk[x][i], sk);
                kq = fmaf(nk[x][i], nq[x][i], kq);
            }
            sq = a.qscale / sqrtf(warp_sum(sq) + kUnitEps);
            sk = 1.f / sqrtf(warp_sum(sk) + kUnitEps);
            kq = warp_sum(kq) * sq * sk;
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                qs[c][lane + 32 * i] = nq[x][i] * sq;
                ks[c][lane + 32 * i] = nk[x][i] * sk;
            }
            if (lane < kDeltaCols) vs[c][lane] = nv[x];
            if (lane == 0) {
                gs[c] = expf(rate * softplus_f32(na[x] + bias));
                bs[c] = sigmoid_f32(nb[x]);
                kqs[c] = kq;
            }
        }
        __syncthreads();
        if (tc + CH < t1) fetch(tc + CH);
        float keep = 0.f;   // lane p keeps token p's output of its column
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            if (tc + c < t1) {
                float dk0 = 0.f, dk1 = 0.f, dq0 = 0.f, dq1 = 0.f;
#pragma unroll
                for (int i = 0; i < RP / 4; ++i) {
                    const float4 k4 = *reinterpret_cast<const float4*>(&ks[c][4 * (p + 8 * i)]);
                    const float4 q4 = *reinterpret_cast<const float4*>(&qs[c][4 * (p + 8 * i)]);
                    dk0 = fmaf(k4.x, S[4 * i], dk0);
                    dk1 = fmaf(k4.y, S[4 * i + 1], dk1);
                    dq0 = fmaf(q4.x, S[4 * i], dq0);
                    dq1 = fmaf(q4.y, S[4 * i + 1], dq1);
                    dk0 = fmaf(k4.z, S[4 * i + 2], dk0);
                    dk1 = fmaf(k4.w, S[4 * i + 3], dk1);
                    dq0 = fmaf(q4.z, S[4 * i + 2], dq0);
                    dq1 = fmaf(q4.w, S[4 * i + 3], dq1);
                }
                float sk = dk0 + dk1, sq = dq0 + dq1;
#pragma unroll
                for (int o = 1; o < 8; o <<= 1) {
                    sk += __shfl_xor_sync(0xFFFFFFFFu, sk, o);
                    sq += __shfl_xor_sync(0xFFFFFFFFu, sq, o);
                }
                const float g = gs[c], u = bs[c] * fmaf(-g, sk, vs[c][cl]);
                const float o = fmaf(u, kqs[c], g * sq);
                if (p == c) keep = o;
#pragma unroll
                for (int i = 0; i < RP / 4; ++i) {
                    const float4 k4 = *reinterpret_cast<const float4*>(&ks[c][4 * (p + 8 * i)]);
                    S[4 * i] = fmaf(k4.x, u, g * S[4 * i]);
                    S[4 * i + 1] = fmaf(k4.y, u, g * S[4 * i + 1]);
                    S[4 * i + 2] = fmaf(k4.z, u, g * S[4 * i + 2]);
                    S[4 * i + 3] = fmaf(k4.w, u, g * S[4 * i + 3]);
                }
            }
        }
        if (own && p < CH && tc + p < t1) a.out[(size_t)(tc + p) * a.ldo + (size_t)hd * dv + j] = keep;
        __syncthreads();
    }
    if (own) {
#pragma unroll
        for (int i = 0; i < RP / 4; ++i) {
            const int c = 4 * (p + 8 * i);
            if (vec) {
                if (c < dk) *reinterpret_cast<float4*>(Sg + c) = make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
            } else {
#pragma unroll
                for (int x = 0; x < 4; ++x)
                    if (c + x < dk) Sg[c + x] = S[4 * i + x];
            }
        }
    }
}
constexpr int kDeltaMaxKey = 8 * 64;   // the largest instantiation

}  // namespace seq
}  // namespace tib
