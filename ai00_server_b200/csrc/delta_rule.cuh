// Gated delta rule, and the short causal convolutions in front of it.
//
// Per value head, with the [dk, dv] f32 state S, unit-length key k and query q (q also times dk^-1/2), a decay g in (0, 1) (one
// number per head, or one per key channel acting on the rows of S) and a write strength beta in (0, 1):
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q                (the read-out sees this token's write)
//     g = exp(-exp(A_h) * softplus(z)),  z = projection + bias,  beta = sigmoid(b)
// The read-out is divided by its root mean square over dv, times a weight vector shared by the heads, times a gate (sigmoid or
// silu of a projection).  Several value heads may share one key / query head (value head h uses head h / (H / G)).
//
//   short_conv_kernel     y[t, c] = silu(sum_j w[c, j] x[t - (taps - 1) + j, c]): per-channel causal convolution over time, the
//                         last column is the current token's; inputs before the step come from the sequence's tail rows
//                         (the last taps - 1 inputs, zeros at the start of a sequence)
//   conv_commit_kernel    the step's last taps - 1 inputs become the sequence's new tail rows (own launch: every token of the
//                         step has read the old tail by then)
//   short_conv_step_kernel   both at once for steps of one token per sequence
//   delta_scan_kernel     the recurrence over the step's tokens of one sequence (state_scan.cuh)
// Decays, logarithms, softplus, gates, unit norms, state and read-out are f32.
#pragma once
#include <cuda_runtime.h>
#include "common.cuh"
#include "state_scan.cuh"

namespace b200 {

struct ShortConvParams {
    const float* x; int ldx;                      // [T, >= C] inputs (projection output rows)
    float* y; int ldy;                            // [T, C] silu(conv), or conv
    const float* w;                               // [C][taps]
    float* tail;                                  // [S][taps - 1][C] of this layer; row taps - 2 is the most recent input
    int C, taps;
    MetaView meta;
    int silu = 1;                                 // 0: the plain convolution
};

__global__ void __launch_bounds__(256) short_conv_kernel(const ShortConvParams p) {
    const int t = blockIdx.x;
    if (t >= p.meta.T()) return;
    const int slot = p.meta.tok_slot()[t];
    // index of the token inside its sequence's run of this step: walk the prev links (runs are contiguous: t - first)
    int first = t;
    {
        const int* prev = p.meta.tok_prev();
        // tok_prev[t] = t - 1 inside a run, -1 at its first token; only taps - 1 steps back matter
        for (int d = 0; d < p.taps - 1 && prev[first] >= 0; ++d) first = prev[first];
    }
    const int back = t - first;                   // rows of this step available behind t (capped at taps - 1)
    const float* tl = p.tail + (size_t)slot * (p.taps - 1) * p.C;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < p.C; c += gridDim.y * blockDim.x) {
        float acc = 0.f;
        for (int j = 0; j < p.taps; ++j) {
            const int d = p.taps - 1 - j;         // steps back
            const float xv = d <= back ? p.x[(size_t)(t - d) * p.ldx + c] : tl[(size_t)(p.taps - 1 + back - d) * p.C + c];
            acc = fmaf(p.w[(size_t)c * p.taps + j], xv, acc);
        }
        p.y[(size_t)t * p.ldy + c] = p.silu ? acc / (1.f + expf(-acc)) : acc;
    }
}

__global__ void __launch_bounds__(256) conv_commit_kernel(const ShortConvParams p) {
    const int i = blockIdx.x;
    if (i >= p.meta.nslots()) return;
    const int slot = p.meta.slot_id()[i], t0 = p.meta.slot_start()[i], nt = p.meta.slot_count()[i];
    const int keep = p.taps - 1;
    float* tl = p.tail + (size_t)slot * keep * p.C;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < p.C; c += gridDim.y * blockDim.x) {
        // new row r holds the input nt - keep + r of this step, or, for a short step, the old row r + nt (read before any
        // later row is written: r ascends and r + nt > r)
        for (int r = 0; r < keep; ++r) {
            const int idx = nt - keep + r;
            tl[(size_t)r * p.C + c] = idx >= 0 ? p.x[(size_t)(t0 + idx) * p.ldx + c] : tl[(size_t)(r + nt) * p.C + c];
        }
    }
}

// steps of one token per sequence: convolution and new tail in one pass (the thread that reads a channel's tail also moves it on)
__global__ void __launch_bounds__(256) short_conv_step_kernel(const ShortConvParams p) {
    const int t = blockIdx.x;
    if (t >= p.meta.T()) return;
    const int keep = p.taps - 1;
    float* tl = p.tail + (size_t)p.meta.tok_slot()[t] * keep * p.C;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < p.C; c += gridDim.y * blockDim.x) {
        const float xv = p.x[(size_t)t * p.ldx + c];
        float acc = 0.f;
        for (int j = 0; j < keep; ++j) {
            const float u = tl[(size_t)j * p.C + c];
            acc = fmaf(p.w[(size_t)c * p.taps + j], u, acc);
            if (j > 0) tl[(size_t)(j - 1) * p.C + c] = u;
        }
        if (keep > 0) tl[(size_t)(keep - 1) * p.C + c] = xv;
        acc = fmaf(p.w[(size_t)c * p.taps + keep], xv, acc);
        p.y[(size_t)t * p.ldy + c] = p.silu ? acc / (1.f + expf(-acc)) : acc;
    }
}

struct DeltaScanParams {
    const float* q; const float* k; const float* v; int ld;      // conv outputs: q, k [T, G * dk], v [T, H * dv], row stride ld
    const float* z; int ldz;                      // decay pre-activation, bias added: [T, H * dk], or [T, H] with one decay per head
    const float* b; int ldb;                      // write-strength logits [T, H]
    const float* a_log;                           // [H]
    float* state;                                 // [S][H] state records of this layer
    int H, G, dk, dv;
    float q_scale, unit_eps;
    ScanShape s;                                  // rows = 3 (k, q, decays) with a decay per channel, else 2
    HeadNormParams norm;                          // norm.x: raw read-outs, normed and gated in place
};

template <bool CHANNEL, bool STEP>
__global__ void __launch_bounds__(SCAN_THREADS, STEP ? 2 : 1) delta_scan_kernel(const DeltaScanParams p) {
    const ScanShape& sh = p.s;
    const int h = blockIdx.x / sh.ncta, cb = blockIdx.x % sh.ncta, si = blockIdx.y;
    const MetaView& meta = p.norm.meta;
    if (si >= meta.nslots()) return;
    const int slot = meta.slot_id()[si], t0 = meta.slot_start()[si], nt = meta.slot_count()[si];
    const int dk = p.dk, dv = p.dv, hk = h / (p.H / p.G), ks = sh.ks;
    const int x = threadIdx.x, warp = x >> 5, lane = x & 31, nw = blockDim.x >> 5;
    const int part = x & (ks - 1), col = x >> sh.lks, j = cb * sh.cols + col, ncol = min(sh.cols, dv - cb * sh.cols);
    extern __shared__ __align__(16) float scan_smem[];
    const int krow = ks * SCAN_ROW, tokf = sh.tok_floats();
    float* sbuf = scan_smem;                      // [nbuf][tc][k | q | (decays) | value entries]
    float4* sscal = reinterpret_cast<float4*>(sbuf + (size_t)sh.nbuf * sh.tc * tokf);      // [tc] (decay, beta, 1 / |k|, q_scale / |q|)
    float* sraw = reinterpret_cast<float*>(sscal + sh.tc);        // [nbuf][tc][2] decay and write-strength logits
    float* rec = p.state + ((size_t)slot * p.H + h) * ((size_t)ks * sh.rt * dv);
    __shared__ float red[SCAN_THREADS / 32];
    const bool mine = part == 0 && col < ncol;    // this thread writes the column's read-outs
    float s[SCAN_R];
    scan_load_state(sh, rec, dv, j, part, s);
    const float a_log = p.a_log[h];
    float g_j = 0.f, w_j = 0.f, o_last = 0.f;     // STEP: gate and weight of the column, asked for early
    if (STEP && mine && sh.ncta == 1) {
        g_j = p.norm.gate[(size_t)t0 * p.norm.ldg + (size_t)h * dv + j];
        w_j = p.norm.w[(size_t)h * p.norm.w_hstride + j];
    }
    for (int e = x; e < sh.nbuf * sh.tc * tokf; e += blockDim.x) sbuf[e] = 0.f;
    __syncthreads();
    auto stage = [&](int c) {
        float* buf = sbuf + (size_t)(c % sh.nbuf) * sh.tc * tokf;
        float* raw = sraw + (size_t)(c % sh.nbuf) * sh.tc * 2;
        const int ta = t0 + c * sh.tc, n = min(sh.tc, nt - c * sh.tc);
        scan_stage_keys(sh, buf, tokf, p.k + (size_t)ta * p.ld + (size_t)hk * dk, p.ld, n, dk);
        scan_stage_keys(sh, buf + krow, tokf, p.q + (size_t)ta * p.ld + (size_t)hk * dk, p.ld, n, dk);
        if (CHANNEL) scan_stage_keys(sh, buf + 2 * krow, tokf, p.z + (size_t)ta * p.ldz + (size_t)h * dk, p.ldz, n, dk);
        scan_stage_cols(buf + sh.rows * krow, tokf, p.v + (size_t)ta * p.ld + (size_t)h * dv + cb * sh.cols, p.ld, n, ncol);
        if (x < n) {
            if (!CHANNEL) cp_async4(raw + 2 * x, p.z + (size_t)(ta + x) * p.ldz + h);
            cp_async4(raw + 2 * x + 1, p.b + (size_t)(ta + x) * p.ldb + h);
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    const int nc = STEP ? 1 : (nt + sh.tc - 1) / sh.tc;
    stage(0);
    const float rate = expf(a_log);
    for (int c = 0; c < nc; ++c) {
        const int n = STEP ? 1 : min(sh.tc, nt - c * sh.tc);
        float* buf = sbuf + (size_t)(c % sh.nbuf) * sh.tc * tokf;
        const float* raw = sraw + (size_t)(c % sh.nbuf) * sh.tc * 2;
        if (!STEP && c + 1 < nc) {
            stage(c + 1);                          // into the buffer that group c - 1 used: everyone left it at the barrier below
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        for (int t = warp; t < n; t += nw) {       // per token: lengths of k and q, decay, write strength
            float* kr = buf + (size_t)t * tokf;
            float kk = 0.f, qq = 0.f;
            for (int i = lane; i < krow; i += 32) {
                const float kv = kr[i], qv = kr[krow + i];
                kk = fmaf(kv, kv, kk); qq = fmaf(qv, qv, qq);
                if (CHANNEL) {
                    const float z = kr[2 * krow + i];
                    kr[2 * krow + i] = expf(-rate * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))));
                }
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) { kk += __shfl_xor_sync(0xffffffffu, kk, o); qq += __shfl_xor_sync(0xffffffffu, qq, o); }
            if (lane == 0) {
                float g = 1.f;
                if (!CHANNEL) {
                    const float z = raw[2 * t];
                    g = expf(-rate * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))));
                }
                sscal[t] = make_float4(g, 1.f / (1.f + expf(-raw[2 * t + 1])), 1.f / sqrtf(kk + p.unit_eps), p.q_scale / sqrtf(qq + p.unit_eps));
            }
        }
        __syncthreads();
        float* orow = p.norm.x + (size_t)(t0 + c * sh.tc) * p.norm.ldx + (size_t)h * dv + j;
        for (int t = 0; t < n; ++t) {
            const float* kr = buf + (size_t)t * tokf + part * SCAN_ROW;
            const float4 sc = sscal[t];
            const float vj = buf[(size_t)t * tokf + sh.rows * krow + col];
            float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
#pragma unroll
            for (int r = 0; r < SCAN_R; r += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(kr + r);
                if (CHANNEL) {
                    const float4 g4 = *reinterpret_cast<const float4*>(kr + 2 * krow + r);
                    s[r] *= g4.x; s[r + 1] *= g4.y; s[r + 2] *= g4.z; s[r + 3] *= g4.w;
                } else {
                    s[r] *= sc.x; s[r + 1] *= sc.x; s[r + 2] *= sc.x; s[r + 3] *= sc.x;
                }
                d0 = fmaf(s[r], k4.x, d0); d1 = fmaf(s[r + 1], k4.y, d1); d2 = fmaf(s[r + 2], k4.z, d2); d3 = fmaf(s[r + 3], k4.w, d3);
            }
            const float d = scan_part_sum((d0 + d1) + (d2 + d3), ks);
            const float u = sc.y * (vj - d * sc.z) * sc.z;         // u / |k|: the write is (k / |k|) u^T
            if (STEP) asm volatile("" ::: "memory");     // read the key again below instead of keeping it: 64 registers, two CTAs per SM
            float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
            for (int r = 0; r < SCAN_R; r += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(kr + r), q4 = *reinterpret_cast<const float4*>(kr + krow + r);
                s[r] = fmaf(k4.x, u, s[r]); s[r + 1] = fmaf(k4.y, u, s[r + 1]); s[r + 2] = fmaf(k4.z, u, s[r + 2]); s[r + 3] = fmaf(k4.w, u, s[r + 3]);
                o0 = fmaf(s[r], q4.x, o0); o1 = fmaf(s[r + 1], q4.y, o1); o2 = fmaf(s[r + 2], q4.z, o2); o3 = fmaf(s[r + 3], q4.w, o3);
            }
            const float o = scan_part_sum((o0 + o1) + (o2 + o3), ks) * sc.w;
            if (STEP && sh.ncta == 1) o_last = o;
            else if (mine) orow[(size_t)t * p.norm.ldx] = o;
        }
        if (!STEP) __syncthreads();
    }
    scan_store_state(sh, rec, dv, j, part, s);
    if constexpr (STEP) {
        if (sh.ncta == 1) {                        // the CTA holds the head: norm and gate from registers
            float ss = mine ? o_last * o_last : 0.f;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            if (lane == 0) red[warp] = ss;
            __syncthreads();
            ss = 0.f;
            for (int w = 0; w < nw; ++w) ss += red[w];
            if (mine) p.norm.x[(size_t)t0 * p.norm.ldx + (size_t)h * dv + j] = head_norm_value(p.norm, o_last, 1.f, ss, w_j, g_j);
        }
    } else if (sh.ncta == 1) {
        for (int t = warp; t < nt; t += nw) head_norm_row(p.norm, t0 + t, h, lane);
    }
}

}  // namespace b200
