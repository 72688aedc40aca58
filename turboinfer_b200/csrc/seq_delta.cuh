// seq_delta.cuh -- the gated delta rule of the layered sequence engine (a linear recurrence whose write removes what the state already
// answers for the key), beside the gated linear recurrences of seq_recurrent.cuh:
//
//     q, k, v behind causal depth-wise convolutions and silu (short_conv_* of seq_headmix.cuh), side by side in one row
//     k <- k / sqrt(sum k^2 + 1e-6), q <- q / sqrt(sum q^2 + 1e-6) * qscale           per head
//     g = exp(-exp(A_log) softplus(a + dt_bias)), beta = sigmoid(b)                   one number a head
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q                    S: [dk][dv] per head, fp32, one per live sequence
//
// Value head h reads the q and k of head h / (heads / kv_heads).  Everything is fp32 (FMA) in both compute modes.  Two forms:
//
//   token by token (delta_scan_kernel; decoded tokens, short portions, key sizes the other form does not take).  The columns of S are
//   independent of one another, so column j lives in the registers of eight lanes of a warp (each holds an eighth of the key channels),
//   and a token costs one round of three shuffles: both S^T k and S^T q are taken from the state before the write, o = g (S^T q) + (k . q) u.
//
//   in chunks of 64 tokens (prompt portions).  With L_i the sum of log g up to token i of the chunk, D_ij = exp(L_i - L_j), S_0 the state in
//   front of the chunk and rows of K, Q, V, U as tokens, the writes of a chunk solve a triangular system and the rest are products:
//       (I + M) U = diag(beta) (V - diag(e^L) K S_0),   M_ij = beta_i D_ij (k_i . k_j) below the diagonal
//       O = diag(e^L) Q S_0 + A U,                      A_ij = D_ij (q_i . k_j) on and below the diagonal
//       S = e^(L_last) S_0 + sum_i e^(L_last - L_i) k_i u_i^T
//   delta_chunk_prepare_kernel works out A, Wk = (I + M)^-1 diag(beta e^L) K and Wv = (I + M)^-1 diag(beta) V for all chunks at once (they
//   do not depend on the state); delta_chunk_scan_kernel then walks the chunks with U = Wv - Wk S_0.  The inverse is bounded: its entries
//   are beta_i k_i^T (product of contractions) k_j.  L is summed in double precision, so that D is exact to fp32 however strong the decays are.
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
    int max_rows;                 // delta_scan_kernel: entries with more rows are left to the chunked form (0: none are)
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
    if (a.max_rows > 0 && m.ent_row0[e + 1] - m.ent_row0[e] > a.max_rows) return;
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

// ---- the chunked form ---------------------------------------------------------------------------------------------------------------
constexpr int kDeltaChunk = 64;
constexpr int kDeltaChunkMaxKey = 128;   // key sizes in fours up to this
struct DeltaChunkArgs {
    DeltaArgs d;
    const int* tiles;           // prepare: tiles[2 i] = first row, tiles[2 i + 1] = rows (<= 64) of chunk i
    float *wk, *wv, *am;        // [heads][T][dk], [heads][T][dv], [heads][T][64]
    float *sq, *sk, *eg;        // [heads][T] each: e^L / |q| * qscale, e^(L_last - L) / |k|, e^L
    int min_rows;               // scan: entries with fewer rows are left to delta_scan_kernel
};
// out[row][c] = sum_(j <= row) Tm[row][j] X[j][c] over COLS columns, by 256 threads; Tm lower triangular with row stride 68, X with row stride LDX
template <int COLS, int LDX>
__device__ __forceinline__ void delta_apply(const float* Tm, const float* X, float* out, size_t ldo, int n, int cols, bool vec) {
    constexpr int TXN = COLS / 4, TYN = 256 / TXN, RI = kDeltaChunk / TYN;
    const int tx = threadIdx.x % TXN, ty = threadIdx.x / TXN;
    float acc[RI][4];
#pragma unroll
    for (int i = 0; i < RI; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll 1
    for (int j = 0; j < kDeltaChunk; j += 4) {
        float4 x[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) x[q] = *reinterpret_cast<const float4*>(X + (j + q) * LDX + 4 * tx);
#pragma unroll
        for (int i = 0; i < RI; ++i) {
            if (TYN * i + TYN - 1 < j) continue;   // (above the diagonal)
            const float4 t = *reinterpret_cast<const float4*>(Tm + (ty + TYN * i) * 68 + j);
            acc[i][0] = fmaf(t.x, x[0].x, fmaf(t.y, x[1].x, fmaf(t.z, x[2].x, fmaf(t.w, x[3].x, acc[i][0]))));
            acc[i][1] = fmaf(t.x, x[0].y, fmaf(t.y, x[1].y, fmaf(t.z, x[2].y, fmaf(t.w, x[3].y, acc[i][1]))));
            acc[i][2] = fmaf(t.x, x[0].z, fmaf(t.y, x[1].z, fmaf(t.z, x[2].z, fmaf(t.w, x[3].z, acc[i][2]))));
            acc[i][3] = fmaf(t.x, x[0].w, fmaf(t.y, x[1].w, fmaf(t.z, x[2].w, fmaf(t.w, x[3].w, acc[i][3]))));
        }
    }
#pragma unroll
    for (int i = 0; i < RI; ++i) {
        const int r = ty + TYN * i, c = 4 * tx;
        if (r >= n) continue;
        float* o = out + (size_t)r * ldo + c;
        if (vec) {
            if (c < cols) *reinterpret_cast<float4*>(o) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        } else {
#pragma unroll
            for (int q = 0; q < 4; ++q)
                if (c + q < cols) o[q] = acc[i][q];
        }
    }
}
template <int DKP> constexpr size_t delta_prepare_smem_bytes() { return sizeof(float) * ((size_t)kDeltaChunk * (DKP + 4) + (size_t)kDeltaChunk * 132 + 2 * (size_t)kDeltaChunk * 68); }
// grid (chunks, heads).  DKP: key channels padded with zeros (64 or 128).
template <int DKP>
__global__ void __launch_bounds__(256) delta_chunk_prepare_kernel(DeltaChunkArgs c, StepMeta m) {
    pdl_launch_dependents();
    pdl_wait_prior_grid();
    constexpr int C = kDeltaChunk, LDK = DKP + 4, LDV = 132;
    extern __shared__ __align__(16) float dsm[];
    float* Ks = dsm;                 // [C][LDK] keys
    float* Qs = Ks + C * LDK;        // [C][LDK] queries, later [C][LDV] values
    float* Ms = Qs + C * LDV;        // [C][68]
    float* Ts = Ms + C * 68;         // [C][68]
    __shared__ double Ld[C];
    __shared__ float beta[C], el[C], rk[C], rq[C];
    const DeltaArgs& a = c.d;
    const int row0 = c.tiles[2 * blockIdx.x], n = c.tiles[2 * blockIdx.x + 1], hd = blockIdx.y;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int dk = a.dk, dv = a.dv, G = a.kv_heads, kh = hd / (a.heads / G);
    const float* src = a.qkv + (size_t)row0 * a.ld;
    const size_t base = (size_t)hd * m.T + row0;
    for (int i = tid; i < C * (DKP / 4); i += 256) {
        const int r = i / (DKP / 4), k = (i % (DKP / 4)) * 4;
        float4 kv = make_float4(0.f, 0.f, 0.f, 0.f), qv = kv;
        if (r < n && k < dk) {
            kv = *reinterpret_cast<const float4*>(src + (size_t)r * a.ld + (G + kh) * dk + k);
            qv = *reinterpret_cast<const float4*>(src + (size_t)r * a.ld + kh * dk + k);
        }
        *reinterpret_cast<float4*>(Ks + r * LDK + k) = kv;
        *reinterpret_cast<float4*>(Qs + r * LDK + k) = qv;
    }
    if (tid < C) {   // rows behind the last one: no decay, no write
        float lg = 0.f, b = 0.f;
        if (tid < n) {
            const size_t t = (size_t)(row0 + tid);
            lg = -expf(a.A_log[hd]) * softplus_f32(a.a[t * a.ld_ab + hd] + a.dt_bias[hd]);
            b = sigmoid_f32(a.b[t * a.ld_ab + hd]);
        }
        Ld[tid] = (double)lg;
        beta[tid] = b;
    }
    __syncthreads();
    if (warp == 0) {   // inclusive sums of log g, two a lane
        const double x0 = Ld[2 * lane], x1 = Ld[2 * lane + 1];
        double s = x0 + x1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double u = __shfl_up_sync(0xFFFFFFFFu, s, o);
            if (lane >= o) s += u;
        }
        double before = __shfl_up_sync(0xFFFFFFFFu, s, 1);
        if (lane == 0) before = 0.0;
        Ld[2 * lane] = before + x0;
        Ld[2 * lane + 1] = before + (x0 + x1);
        el[2 * lane] = expf((float)(before + x0));
        el[2 * lane + 1] = expf((float)(before + (x0 + x1)));
    }
    for (int r = warp; r < C; r += 8) {
        float sk = 0.f, sq = 0.f;
#pragma unroll
        for (int k = 0; k < DKP; k += 32) {
            const float x = Ks[r * LDK + k + lane], y = Qs[r * LDK + k + lane];
            sk = fmaf(x, x, sk);
            sq = fmaf(y, y, sq);
        }
        sk = warp_sum(sk);
        sq = warp_sum(sq);
        if (lane == 0) {
            rk[r] = 1.f / sqrtf(sk + kUnitEps);
            rq[r] = a.qscale / sqrtf(sq + kUnitEps);
        }
    }
    __syncthreads();
    if (tid < n) {
        c.sq[base + tid] = el[tid] * rq[tid];
        c.sk[base + tid] = expf((float)(Ld[n - 1] - Ld[tid])) * rk[tid];
        c.eg[base + tid] = el[tid];
    }
    {   // K K^T and Q K^T: rows ty, ty + 32 of both, columns tx + 8 j
        const int ty = tid >> 3, tx = tid & 7;
        float acc[4][8];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[i][j] = 0.f;
#pragma unroll 2
        for (int k = 0; k < DKP; k += 4) {
            float4 w[4];
            w[0] = *reinterpret_cast<const float4*>(Ks + ty * LDK + k);
            w[1] = *reinterpret_cast<const float4*>(Ks + (ty + 32) * LDK + k);
            w[2] = *reinterpret_cast<const float4*>(Qs + ty * LDK + k);
            w[3] = *reinterpret_cast<const float4*>(Qs + (ty + 32) * LDK + k);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float4 x = *reinterpret_cast<const float4*>(Ks + (tx + 8 * j) * LDK + k);
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    if (j < 4 || (i & 1)) acc[i][j] = fmaf(w[i].x, x.x, fmaf(w[i].y, x.y, fmaf(w[i].z, x.z, fmaf(w[i].w, x.w, acc[i][j]))));
            }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int r = ty + 32 * i;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const int col = tx + 8 * j;
                const float dec = col <= r ? expf((float)(Ld[r] - Ld[col])) * rk[col] : 0.f;
                Ms[r * 68 + col] = col < r ? acc[i][j] * dec * rk[r] * beta[r] : 0.f;
                Ts[r * 68 + col] = 0.f;
                if (r < n) c.am[(base + r) * C + col] = acc[2 + i][j] * dec * rq[r];
            }
        }
    }
    __syncthreads();
    const bool vecv = dv % 4 == 0;
    auto load_values = [&](int c0) {   // V columns c0 .. c0 + 127, rows scaled by beta
        for (int i = tid; i < C * 32; i += 256) {
            const int r = i >> 5, k = (i & 31) * 4;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (r < n && c0 + k < dv) {
                const float* p = src + (size_t)r * a.ld + 2 * G * dk + hd * dv + c0 + k;
                if (vecv) v = *reinterpret_cast<const float4*>(p);
                else v = make_float4(p[0], c0 + k + 1 < dv ? p[1] : 0.f, c0 + k + 2 < dv ? p[2] : 0.f, c0 + k + 3 < dv ? p[3] : 0.f);
                const float b = beta[r];
                v.x *= b; v.y *= b; v.z *= b; v.w *= b;
            }
            *reinterpret_cast<float4*>(Qs + r * LDV + k) = v;
        }
    };
    for (int i = tid; i < C * (DKP / 4); i += 256) {   // keys scaled for the first product
        const int r = i / (DKP / 4), k = (i % (DKP / 4)) * 4;
        float4* p = reinterpret_cast<float4*>(Ks + r * LDK + k);
        const float f = beta[r] * el[r] * rk[r];
        *p = make_float4(p->x * f, p->y * f, p->z * f, p->w * f);
    }
    load_values(0);
    // (I + M)^-1: the four diagonal blocks of 16 column by column, then pairs of blocks, then the pair of pairs
    if (tid < 64) {
        const int b = (tid >> 4) * 16, j = tid & 15;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float s = i == j ? 1.f : 0.f;
#pragma unroll
            for (int k = 0; k < i; ++k) s = fmaf(-Ms[(b + i) * 68 + b + k], x[k], s);
            x[i] = s;
            Ts[(b + i) * 68 + b + j] = s;
        }
    }
    __syncthreads();
#pragma unroll
    for (int half = 16; half <= 32; half *= 2) {
        // below the diagonal of every 2 half x 2 half block: -T22 (M21 T11); the inner product waits in the block's upper right corner
        const int per = half * half, tot = (C / (2 * half)) * per;
        for (int i = tid; i < tot; i += 256) {
            const int b = i / per * 2 * half, r = (i % per) / half, col = i % half;
            float s = 0.f;
            for (int k = col; k < half; ++k) s = fmaf(Ms[(b + half + r) * 68 + b + k], Ts[(b + k) * 68 + b + col], s);
            Ts[(b + r) * 68 + b + half + col] = s;
        }
        __syncthreads();
        for (int i = tid; i < tot; i += 256) {
            const int b = i / per * 2 * half, r = (i % per) / half, col = i % half;
            float s = 0.f;
            for (int k = 0; k <= r; ++k) s = fmaf(-Ts[(b + half + r) * 68 + b + half + k], Ts[(b + k) * 68 + b + half + col], s);
            Ts[(b + half + r) * 68 + b + col] = s;
        }
        __syncthreads();
        for (int i = tid; i < tot; i += 256) Ts[(i / per * 2 * half + (i % per) / half) * 68 + i / per * 2 * half + half + i % half] = 0.f;
        __syncthreads();
    }
    delta_apply<DKP, LDK>(Ts, Ks, c.wk + base * dk, dk, n, dk, true);
    for (int c0 = 0; c0 < dv; c0 += 128) {
        if (c0) {
            __syncthreads();
            load_values(c0);
            __syncthreads();
        }
        if (dv - c0 <= 64) delta_apply<64, LDV>(Ts, Qs, c.wv + base * dv + c0, dv, n, dv - c0, vecv);
        else delta_apply<128, LDV>(Ts, Qs, c.wv + base * dv + c0, dv, n, min(128, dv - c0), vecv);
    }
}

template <int DKP> constexpr size_t delta_chunk_smem_bytes() {
    return sizeof(float) * (2 * (size_t)kDeltaChunk * (DKP + 8) + (size_t)kDeltaChunk * (DKP + 16) + (size_t)kDeltaChunk * 72 + (size_t)kDeltaChunk * 36 + (size_t)DKP * 20);
}
// One block per (entry, head, 16 value columns).  The 64 (DKP) x 16 products are register tiles: a thread owns four columns; lanes that
// differ in their lowest bit(s) share an output tile and split the inner dimension in interleaved fours.
template <int DKP>
__global__ void __launch_bounds__(256, 1) delta_chunk_scan_kernel(DeltaChunkArgs c, StepMeta m) {
    pdl_launch_dependents();
    pdl_wait_prior_grid();
    constexpr int C = kDeltaChunk, LDW = DKP + 8, LDK = DKP + 16, LDA = 72, LDU = 20, IH = 256 / DKP, IB = IH == 2 ? 1 : 2;   // IH lanes share a state tile
    static_assert(IH == 2 || IH == 4, "key sizes 64 and 128");
    const DeltaArgs& a = c.d;
    const int e = blockIdx.x, hd = blockIdx.y, t0 = m.ent_row0[e], t1 = m.ent_row0[e + 1];
    if (t1 - t0 < c.min_rows) return;
    extern __shared__ __align__(16) float dsm[];
    float* Ws = dsm;                 // [C][LDW]
    float* Qs = Ws + C * LDW;        // [C][LDW]
    float* Kc = Qs + C * LDW;        // [C][LDK]
    float* As = Kc + C * LDK;        // [C][LDA]
    float* Us = As + C * LDA;        // [C][LDU]
    float* Up = Us + C * LDU;        // [C][16]: rows of U times e^(L_last - L) / |k|
    float* Ss = Up + C * 16;         // [DKP][LDU]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int dk = a.dk, dv = a.dv, G = a.kv_heads, kh = hd / (a.heads / G), col0 = blockIdx.z * kDeltaCols;
    // products with the state and A: inner half hb, columns 4 tx, rows ty and ty + 32; state update: inner part ih, columns 4 sx, channels 4 kg
    const int hb = lane & 1, tx = (lane >> 1) & 3, ty = warp * 4 + (lane >> 3);
    const int ih = lane & (IH - 1), sx = (lane >> IB) & 3, kg = warp * (8 / IH) + (lane >> (IB + 2));
    const size_t hbase = (size_t)hd * m.T;
    const int my = ty + 32 * hb;   // the row of U and O this lane finishes
    auto fetch_wq = [&](int t) {
        for (int i = tid; i < C * (DKP / 4); i += 256) {
            const int r = i / (DKP / 4), k = (i % (DKP / 4)) * 4;
            const bool ok = t + r < t1 && k < dk;
            const size_t tr = (size_t)(ok ? t + r : t);
            const int kk = ok ? k : 0;
            cp_async16(Ws + r * LDW + k, c.wk + (hbase + tr) * dk + kk, ok);
            cp_async16(Qs + r * LDW + k, a.qkv + tr * a.ld + kh * dk + kk, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto fetch_ak = [&](int t) {
        for (int i = tid; i < C * (DKP / 4); i += 256) {
            const int r = i / (DKP / 4), k = (i % (DKP / 4)) * 4;
            const bool ok = t + r < t1 && k < dk;
            cp_async16(Kc + r * LDK + k, a.qkv + (size_t)(ok ? t + r : t) * a.ld + (G + kh) * dk + (ok ? k : 0), ok);
        }
        for (int i = tid; i < C * (C / 4); i += 256) {
            const int r = i >> 4, k = (i & 15) * 4;
            const bool ok = t + r < t1;
            cp_async16(As + r * LDA + k, c.am + (hbase + (ok ? t + r : t)) * C + k, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch_wq(t0);
    fetch_ak(t0);
    // the state: rows 4 kg .. + 3, columns 4 sx .. + 3 in registers (the same in all IH lanes), a copy in shared memory for the products
    float S[4][4];
    float* Sg = a.state + ((size_t)m.ent_slot[e] * a.heads + hd) * (size_t)dv * dk;
    const bool fresh = (m.ent_pos0[e] == 0);
#pragma unroll
    for (int q = 0; q < 4; ++q) {
        const int col = col0 + 4 * sx + q;
        const float4 v = (!fresh && col < dv && 4 * kg < dk) ? *reinterpret_cast<const float4*>(Sg + (size_t)col * dk + 4 * kg) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[0][q] = v.x; S[1][q] = v.y; S[2][q] = v.z; S[3][q] = v.w;
    }
    auto put_state = [&]() {
#pragma unroll
        for (int x = 0; x < 4; ++x)
            if (x / (4 / IH) == ih) *reinterpret_cast<float4*>(Ss + (4 * kg + x) * LDU + 4 * sx) = make_float4(S[x][0], S[x][1], S[x][2], S[x][3]);
    };
    put_state();
    const bool vec_v = dv % 4 == 0;
    const bool vec_o = vec_v && a.ldo % 4 == 0 && (reinterpret_cast<uintptr_t>(a.out) & 15) == 0;
    const int cx = col0 + 4 * tx;
    for (int t = t0; t < t1; t += C) {
        const int n = min(C, t1 - t);
        float wv[4] = {0.f, 0.f, 0.f, 0.f}, sq = 0.f, sk = 0.f;
        if (my < n) {
            const float* p = c.wv + (hbase + t + my) * dv + cx;
            if (vec_v) {
                if (cx < dv) {
                    const float4 v = *reinterpret_cast<const float4*>(p);
                    wv[0] = v.x; wv[1] = v.y; wv[2] = v.z; wv[3] = v.w;
                }
            } else {
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (cx + q < dv) wv[q] = p[q];
            }
            sq = c.sq[hbase + t + my];
            sk = c.sk[hbase + t + my];
        }
        const float eg = c.eg[hbase + t + n - 1];
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        float acc[4][4];   // Wk S and Q S, rows ty and ty + 32
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll 4
        for (int k8 = 0; k8 < DKP; k8 += 8) {
            const int k = k8 + 4 * hb;
            float4 s[4], w[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) s[q] = *reinterpret_cast<const float4*>(Ss + (k + q) * LDU + 4 * tx);
            w[0] = *reinterpret_cast<const float4*>(Ws + ty * LDW + k);
            w[1] = *reinterpret_cast<const float4*>(Ws + (ty + 32) * LDW + k);
            w[2] = *reinterpret_cast<const float4*>(Qs + ty * LDW + k);
            w[3] = *reinterpret_cast<const float4*>(Qs + (ty + 32) * LDW + k);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                acc[i][0] = fmaf(w[i].x, s[0].x, fmaf(w[i].y, s[1].x, fmaf(w[i].z, s[2].x, fmaf(w[i].w, s[3].x, acc[i][0]))));
                acc[i][1] = fmaf(w[i].x, s[0].y, fmaf(w[i].y, s[1].y, fmaf(w[i].z, s[2].y, fmaf(w[i].w, s[3].y, acc[i][1]))));
                acc[i][2] = fmaf(w[i].x, s[0].z, fmaf(w[i].y, s[1].z, fmaf(w[i].z, s[2].z, fmaf(w[i].w, s[3].z, acc[i][2]))));
                acc[i][3] = fmaf(w[i].x, s[0].w, fmaf(w[i].y, s[1].w, fmaf(w[i].z, s[2].w, fmaf(w[i].w, s[3].w, acc[i][3]))));
            }
        }
        float o[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            float p[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) p[i] = acc[i][q] + __shfl_xor_sync(0xFFFFFFFFu, acc[i][q], 1);
            wv[q] -= hb ? p[1] : p[0];
            o[q] = sq * (hb ? p[3] : p[2]);
        }
        *reinterpret_cast<float4*>(Us + my * LDU + 4 * tx) = make_float4(wv[0], wv[1], wv[2], wv[3]);
        *reinterpret_cast<float4*>(Up + my * 16 + 4 * tx) = make_float4(sk * wv[0], sk * wv[1], sk * wv[2], sk * wv[3]);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (t + C < t1) fetch_wq(t + C);
        float ao[2][4];   // A U, rows ty (keys below 32 only) and ty + 32
#pragma unroll
        for (int q = 0; q < 4; ++q) ao[0][q] = ao[1][q] = 0.f;
#pragma unroll
        for (int j8 = 0; j8 < C; j8 += 8) {
            const int j = j8 + 4 * hb;
            float4 u[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) u[q] = *reinterpret_cast<const float4*>(Us + (j + q) * LDU + 4 * tx);
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                if (i == 0 && j8 >= 32) continue;
                const float4 w = *reinterpret_cast<const float4*>(As + (ty + 32 * i) * LDA + j);
                ao[i][0] = fmaf(w.x, u[0].x, fmaf(w.y, u[1].x, fmaf(w.z, u[2].x, fmaf(w.w, u[3].x, ao[i][0]))));
                ao[i][1] = fmaf(w.x, u[0].y, fmaf(w.y, u[1].y, fmaf(w.z, u[2].y, fmaf(w.w, u[3].y, ao[i][1]))));
                ao[i][2] = fmaf(w.x, u[0].z, fmaf(w.y, u[1].z, fmaf(w.z, u[2].z, fmaf(w.w, u[3].z, ao[i][2]))));
                ao[i][3] = fmaf(w.x, u[0].w, fmaf(w.y, u[1].w, fmaf(w.z, u[2].w, fmaf(w.w, u[3].w, ao[i][3]))));
            }
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const float x = ao[0][q] + __shfl_xor_sync(0xFFFFFFFFu, ao[0][q], 1), y = ao[1][q] + __shfl_xor_sync(0xFFFFFFFFu, ao[1][q], 1);
            o[q] += hb ? y : x;
        }
        if (my < n) {
            float* p = a.out + (size_t)(t + my) * a.ldo + (size_t)hd * dv + cx;
            if (vec_o) {
                if (cx < dv) *reinterpret_cast<float4*>(p) = make_float4(o[0], o[1], o[2], o[3]);
            } else {
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (cx + q < dv) p[q] = o[q];
            }
        }
        float up[4][4];   // sum_i k_i u'_i^T
#pragma unroll
        for (int x = 0; x < 4; ++x) up[x][0] = up[x][1] = up[x][2] = up[x][3] = 0.f;
#pragma unroll 8
        for (int i = ih; i < C; i += IH) {
            const float4 k4 = *reinterpret_cast<const float4*>(Kc + i * LDK + 4 * kg), u4 = *reinterpret_cast<const float4*>(Up + i * 16 + 4 * sx);
            const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, uu[4] = {u4.x, u4.y, u4.z, u4.w};
#pragma unroll
            for (int x = 0; x < 4; ++x)
#pragma unroll
                for (int q = 0; q < 4; ++q) up[x][q] = fmaf(kk[x], uu[q], up[x][q]);
        }
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                float v = up[x][q];
#pragma unroll
                for (int s = 1; s < IH; s <<= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, s);
                S[x][q] = fmaf(eg, S[x][q], v);
            }
        put_state();   // (the products of this chunk with the old state lie behind the last barrier)
        __syncthreads();
        if (t + C < t1) fetch_ak(t + C);
    }
    if (ih == 0 && 4 * kg < dk) {
#pragma unroll
        for (int q = 0; q < 4; ++q)
            if (col0 + 4 * sx + q < dv) *reinterpret_cast<float4*>(Sg + (size_t)(col0 + 4 * sx + q) * dk + 4 * kg) = make_float4(S[0][q], S[1][q], S[2][q], S[3][q]);
    }
}

}  // namespace seq
}  // namespace tib
