// Gated linear attention: per head a [dk, dv] f32 state with a per-key-channel decay,
//     S_t = diag(alpha_t) S_{t-1} + k_t v_t^T,    o_t = q_scale S_t^T q_t,    alpha = sigmoid(z)^(1/tau) = exp(logsigmoid(z) / tau)
// followed by an RMS norm of o over dv (weight shared by heads) and an output gate silu(g).
//
//   gla_scan_kernel   the recurrence over the step's tokens of one sequence: state columns in registers as in state_scan.cuh.  Keys,
//                     queries and decay logits of the next tokens arrive by cp.async while the current ones are worked on; a staged
//                     group's logits become decays before its token loop, which then has no dependence but the state itself.
// Decay, state, read-out and norm are f32.
#pragma once
#include <cuda_runtime.h>
#include "common.cuh"
#include "state_scan.cuh"

namespace b200 {

struct GlaParams {
    const float* q; const float* k; const float* v; int ld;      // projection rows: q, k [T, H dk], v [T, H dv], row stride ld
    const float* z; int ldz;                      // decay logits [T, H dk], bias added
    float* state;                                 // [S][H] state records of this layer
    int H, dk, dv;
    float inv_tau, q_scale;
    ScanShape s;                                  // rows = 3 (k, q, decays)
    HeadNormParams norm;                          // norm.x: raw read-outs, normed and gated in place
};

template <bool STEP>
__global__ void __launch_bounds__(SCAN_THREADS, STEP ? 2 : 1) gla_scan_kernel(const GlaParams p) {
    const ScanShape& sh = p.s;
    const int h = blockIdx.x / sh.ncta, cb = blockIdx.x % sh.ncta, si = blockIdx.y;
    const MetaView& meta = p.norm.meta;
    if (si >= meta.nslots()) return;
    const int slot = meta.slot_id()[si], t0 = meta.slot_start()[si], nt = meta.slot_count()[si];
    const int dk = p.dk, dv = p.dv, ks = sh.ks;
    const int x = threadIdx.x, warp = x >> 5, lane = x & 31, nw = blockDim.x >> 5;
    const int part = x & (ks - 1), col = x >> sh.lks, j = cb * sh.cols + col, ncol = min(sh.cols, dv - cb * sh.cols);
    extern __shared__ __align__(16) float scan_smem[];
    const int krow = ks * SCAN_ROW, tokf = sh.tok_floats();
    float* sbuf = scan_smem;                      // [nbuf][tc][k | q | decays | value entries]
    float* rec = p.state + ((size_t)slot * p.H + h) * ((size_t)ks * sh.rt * dv);
    __shared__ float red[SCAN_THREADS / 32];
    const bool mine = part == 0 && col < ncol;    // this thread writes the column's read-outs
    float s[SCAN_R];
    scan_load_state(sh, rec, dv, j, part, s);
    float g_j = 0.f, w_j = 0.f, o_last = 0.f;     // STEP: gate and weight of the column, asked for early
    if (STEP && mine && sh.ncta == 1) {
        g_j = p.norm.gate[(size_t)t0 * p.norm.ldg + (size_t)h * dv + j];
        w_j = p.norm.w[(size_t)h * p.norm.w_hstride + j];
    }
    for (int e = x; e < sh.nbuf * sh.tc * tokf; e += blockDim.x) sbuf[e] = 0.f;
    __syncthreads();
    auto stage = [&](int c) {
        float* buf = sbuf + (size_t)(c % sh.nbuf) * sh.tc * tokf;
        const int ta = t0 + c * sh.tc, n = min(sh.tc, nt - c * sh.tc);
        scan_stage_keys(sh, buf, tokf, p.k + (size_t)ta * p.ld + (size_t)h * dk, p.ld, n, dk);
        scan_stage_keys(sh, buf + krow, tokf, p.q + (size_t)ta * p.ld + (size_t)h * dk, p.ld, n, dk);
        scan_stage_keys(sh, buf + 2 * krow, tokf, p.z + (size_t)ta * p.ldz + (size_t)h * dk, p.ldz, n, dk);
        scan_stage_cols(buf + 3 * krow, tokf, p.v + (size_t)ta * p.ld + (size_t)h * dv + cb * sh.cols, p.ld, n, ncol);
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    const int nc = STEP ? 1 : (nt + sh.tc - 1) / sh.tc;
    stage(0);
    for (int c = 0; c < nc; ++c) {
        const int n = STEP ? 1 : min(sh.tc, nt - c * sh.tc);
        float* buf = sbuf + (size_t)(c % sh.nbuf) * sh.tc * tokf;
        if (!STEP && c + 1 < nc) {
            stage(c + 1);                          // into the buffer that group c - 1 used: everyone left it at the barrier below
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        for (int t = warp; t < n; t += nw) {       // decay logits -> decays (padding belongs to state entries that stay zero)
            float* zr = buf + (size_t)t * tokf + 2 * krow;
            for (int i = lane; i < krow; i += 32) {
                const float z = zr[i];
                zr[i] = expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * p.inv_tau);
            }
        }
        __syncthreads();
        float* orow = p.norm.x + (size_t)(t0 + c * sh.tc) * p.norm.ldx + (size_t)h * dv + j;
        for (int t = 0; t < n; ++t) {
            const float* kr = buf + (size_t)t * tokf + part * SCAN_ROW;
            const float vj = buf[(size_t)t * tokf + 3 * krow + col];
            float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
            for (int r = 0; r < SCAN_R; r += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(kr + r), q4 = *reinterpret_cast<const float4*>(kr + krow + r);
                const float4 a4 = *reinterpret_cast<const float4*>(kr + 2 * krow + r);
                s[r] = fmaf(k4.x, vj, s[r] * a4.x); s[r + 1] = fmaf(k4.y, vj, s[r + 1] * a4.y);
                s[r + 2] = fmaf(k4.z, vj, s[r + 2] * a4.z); s[r + 3] = fmaf(k4.w, vj, s[r + 3] * a4.w);
                o0 = fmaf(s[r], q4.x, o0); o1 = fmaf(s[r + 1], q4.y, o1); o2 = fmaf(s[r + 2], q4.z, o2); o3 = fmaf(s[r + 3], q4.w, o3);
            }
            const float o = scan_part_sum((o0 + o1) + (o2 + o3), ks) * p.q_scale;
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
