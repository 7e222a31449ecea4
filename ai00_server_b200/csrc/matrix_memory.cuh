// Matrix memory with exponential gates (the mLSTM of xLSTM).  Per head, with the [dk, dv] f32 state S, the [dk] normaliser n, a
// running maximum m (all zero at the start of a sequence), key k, query q (times dk^-1/2), value v and two scalar gates
//     i = cap tanh(zi / cap),   f = logsigmoid(cap tanh(zf / cap)):
//     m' = max(f + m, i);   S <- e^(f + m - m') S + e^(i - m') k v^T;   n <- e^(f + m - m') n + e^(i - m') k;   m <- m'
//     o = S^T q / (max(|n . q|, e^-m) + 1e-6)
// The running maximum keeps both exponentials at most one.  The read-out is divided by its root mean square over dv, times a weight
// per (head, entry), times sigmoid of a gate projection, times a constant (state_scan.cuh: head_norm_row).
//
//   matrix_memory_kernel  the recurrence over the step's tokens of one sequence: state columns in registers as in state_scan.cuh.
//                         The gates and maxima of a staged group of tokens are worked out by one warp before the group (they do
//                         not depend on the state), so the token loop has no dependence but the state itself.  The CTA with a
//                         head's first columns also carries n, spread over all its threads; the per-token factor
//                         dk^-1/2 / (max(...) + 1e-6) goes to `norm.fac`.  Every column keeps a copy of m: the CTAs of one head
//                         then read and write disjoint memory and need not wait for one another.
// Gates, maxima, exponentials, state, normaliser and read-out are f32.
#pragma once
#include <cuda_runtime.h>
#include "common.cuh"
#include "state_scan.cuh"

namespace b200 {

struct MatrixMemoryParams {
    const float* q; const float* k; const float* v; int ld;      // projection rows: q, k [T, H dk], v [T, H dv], row stride ld
    const float* zi; const float* zf;             // gate pre-activations, bias added: [T, H], row stride ld
    float* state;                                 // [S][H] state records of this layer
    float* n;                                     // [S][H][dk]
    float* m;                                     // [S][H][dv] (all entries of a head are equal)
    float* fac;                                   // [T, H] the same memory as norm.fac
    int H, dk, dv;
    float cap, q_scale, den_eps;
    ScanShape s;                                  // rows = 2 (k, q)
    HeadNormParams norm;                          // norm.x: raw read-outs, normed and gated in place
};

constexpr int MM_MAX_N = SCAN_MAX_DK / SCAN_THREADS_PROMPT;      // normaliser entries per thread

template <bool STEP>
__global__ void __launch_bounds__(SCAN_THREADS, STEP ? 2 : 1) matrix_memory_kernel(const MatrixMemoryParams p) {
    const ScanShape& sh = p.s;
    const int h = blockIdx.x / sh.ncta, cb = blockIdx.x % sh.ncta, si = blockIdx.y;
    const MetaView& meta = p.norm.meta;
    if (si >= meta.nslots()) return;
    const int slot = meta.slot_id()[si], t0 = meta.slot_start()[si], nt = meta.slot_count()[si];
    const int dk = p.dk, dv = p.dv, ks = sh.ks, nthr = blockDim.x;
    const int x = threadIdx.x, warp = x >> 5, lane = x & 31, nw = nthr >> 5;
    const int part = x & (ks - 1), col = x >> sh.lks, j = cb * sh.cols + col, ncol = min(sh.cols, dv - cb * sh.cols);
    extern __shared__ __align__(16) float scan_smem[];
    const int krow = ks * SCAN_ROW, tokf = sh.tok_floats();
    float* sbuf = scan_smem;                      // [nbuf][tc][k | q | value entries]
    float4* sscal = reinterpret_cast<float4*>(sbuf + (size_t)sh.nbuf * sh.tc * tokf);      // [tc] (keep, add, e^-m, -)
    float* sraw = reinterpret_cast<float*>(sscal + sh.tc);        // [nbuf][tc][2] gate pre-activations
    float* snq = sraw + (size_t)sh.nbuf * sh.tc * 2;              // [tc][warps] shares of n . q
    const size_t hs = (size_t)slot * p.H + h;
    float* rec = p.state + hs * ((size_t)ks * sh.rt * dv);
    float* gn = p.n + hs * dk;
    float* gm = p.m + hs * dv + cb * sh.cols;
    __shared__ float red[SCAN_THREADS / 32];
    const bool mine = part == 0 && col < ncol;     // this thread writes the column's read-outs
    float s[SCAN_R];
    scan_load_state(sh, rec, dv, j, part, s);
    float g_j = 0.f, w_j = 0.f, o_last = 0.f;      // STEP: gate and weight of the column, asked for early
    if (STEP && mine && sh.ncta == 1) {
        g_j = p.norm.gate[(size_t)t0 * p.norm.ldg + (size_t)h * dv + j];
        w_j = p.norm.w[(size_t)h * p.norm.w_hstride + j];
    }
    constexpr int NE = STEP ? 1 : MM_MAX_N;        // STEP: the first entry is asked for early, further ones are met in memory
    float n[NE];
    int noff[NE];                                  // staged place of this thread's entries of the key dimension
    auto place = [&](int i) { return i / sh.rt * SCAN_ROW + i % sh.rt; };
#pragma unroll
    for (int e = 0; e < NE; ++e) {
        const int i = e * nthr + x;
        n[e] = 0.f; noff[e] = SCAN_R;              // place 32 of part 0 is padding: always zero
        if (cb == 0 && i < dk) { n[e] = gn[i]; noff[e] = place(i); }
    }
    float m_run = gm[0];                           // meaningful in warp 0
    for (int e = x; e < sh.nbuf * sh.tc * tokf; e += nthr) sbuf[e] = 0.f;
    __syncthreads();
    auto stage = [&](int c) {
        float* buf = sbuf + (size_t)(c % sh.nbuf) * sh.tc * tokf;
        float* raw = sraw + (size_t)(c % sh.nbuf) * sh.tc * 2;
        const int ta = t0 + c * sh.tc, cnt = min(sh.tc, nt - c * sh.tc);
        scan_stage_keys(sh, buf, tokf, p.k + (size_t)ta * p.ld + (size_t)h * dk, p.ld, cnt, dk);
        scan_stage_keys(sh, buf + krow, tokf, p.q + (size_t)ta * p.ld + (size_t)h * dk, p.ld, cnt, dk);
        scan_stage_cols(buf + 2 * krow, tokf, p.v + (size_t)ta * p.ld + (size_t)h * dv + cb * sh.cols, p.ld, cnt, ncol);
        if (x < cnt) {
            cp_async4(raw + 2 * x, p.zi + (size_t)(ta + x) * p.ld + h);
            cp_async4(raw + 2 * x + 1, p.zf + (size_t)(ta + x) * p.ld + h);
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    const int nc = STEP ? 1 : (nt + sh.tc - 1) / sh.tc;
    stage(0);
    for (int c = 0; c < nc; ++c) {
        const int cnt = STEP ? 1 : min(sh.tc, nt - c * sh.tc);
        float* buf = sbuf + (size_t)(c % sh.nbuf) * sh.tc * tokf;
        const float* raw = sraw + (size_t)(c % sh.nbuf) * sh.tc * 2;
        if (!STEP && c + 1 < nc) {
            stage(c + 1);                          // into the buffer that group c - 1 used: everyone left it at the barrier below
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        if (warp == 0) {                           // lane t: gates of token t; the maxima one after the other
            float ig = 0.f, fg = 0.f, m_prev = 0.f, m_new = 0.f;
            if (lane < cnt) {
                ig = p.cap * tanhf(raw[2 * lane] / p.cap);
                const float z = p.cap * tanhf(raw[2 * lane + 1] / p.cap);
                fg = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
            }
            for (int u = 0; u < cnt; ++u) {
                const float m_next = fmaxf(__shfl_sync(0xffffffffu, fg, u) + m_run, __shfl_sync(0xffffffffu, ig, u));
                if (lane == u) { m_prev = m_run; m_new = m_next; }
                m_run = m_next;
            }
            if (lane < cnt) sscal[lane] = make_float4(expf(fg + m_prev - m_new), expf(ig - m_new), expf(-m_new), 0.f);
        }
        __syncthreads();
        float* orow = p.norm.x + (size_t)(t0 + c * sh.tc) * p.norm.ldx + (size_t)h * dv + j;
        for (int t = 0; t < cnt; ++t) {
            const float* row = buf + (size_t)t * tokf;
            const float* kr = row + part * SCAN_ROW;
            const float4 sc = sscal[t];
            const float vj = row[2 * krow + col] * sc.y;
            float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
            for (int r = 0; r < SCAN_R; r += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(kr + r), q4 = *reinterpret_cast<const float4*>(kr + krow + r);
                s[r] = fmaf(k4.x, vj, s[r] * sc.x); s[r + 1] = fmaf(k4.y, vj, s[r + 1] * sc.x);
                s[r + 2] = fmaf(k4.z, vj, s[r + 2] * sc.x); s[r + 3] = fmaf(k4.w, vj, s[r + 3] * sc.x);
                o0 = fmaf(s[r], q4.x, o0); o1 = fmaf(s[r + 1], q4.y, o1); o2 = fmaf(s[r + 2], q4.z, o2); o3 = fmaf(s[r + 3], q4.w, o3);
            }
            const float o = scan_part_sum((o0 + o1) + (o2 + o3), ks);
            if (STEP && sh.ncta == 1) o_last = o;
            else if (mine) orow[(size_t)t * p.norm.ldx] = o;
            if (cb == 0) {                         // the normaliser and its product with the query
                float nq = 0.f;
#pragma unroll
                for (int e = 0; e < NE; ++e) {
                    if (e * nthr >= dk) break;     // the same for all threads
                    n[e] = fmaf(sc.y, row[noff[e]], sc.x * n[e]);
                    nq = fmaf(n[e], row[krow + noff[e]], nq);
                }
                if (STEP)
                    for (int i = nthr + x; i < dk; i += nthr) {
                        const float v = fmaf(sc.y, row[place(i)], sc.x * gn[i]);
                        gn[i] = v;
                        nq = fmaf(v, row[krow + place(i)], nq);
                    }
#pragma unroll
                for (int o2_ = 16; o2_ > 0; o2_ >>= 1) nq += __shfl_xor_sync(0xffffffffu, nq, o2_);
                if (lane == 0) snq[t * nw + warp] = nq;
            }
        }
        if constexpr (STEP) {
            float ss = mine ? o_last * o_last : 0.f;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            if (lane == 0) red[warp] = ss;
        }
        __syncthreads();
        if (STEP ? cb == 0 : (cb == 0 && x < cnt)) {
            const int u = STEP ? 0 : x;
            float nq = 0.f;
            for (int w = 0; w < nw; ++w) nq += snq[u * nw + w];
            const float fac = p.q_scale / (fmaxf(fabsf(nq * p.q_scale), sscal[u].z) + p.den_eps);
            if (STEP && sh.ncta == 1) {            // the CTA holds the head: norm and gate from registers
                float ss = 0.f;
                for (int w = 0; w < nw; ++w) ss += red[w];
                if (mine) p.norm.x[(size_t)t0 * p.norm.ldx + (size_t)h * dv + j] = head_norm_value(p.norm, o_last, fac, ss, w_j, g_j);
            } else if (!STEP || x == 0) {
                p.fac[(size_t)(t0 + c * sh.tc + u) * p.H + h] = fac;
            }
        }
    }
    scan_store_state(sh, rec, dv, j, part, s);
    if (cb == 0)
#pragma unroll
        for (int e = 0; e < NE; ++e)
            if (e * nthr + x < dk) gn[e * nthr + x] = n[e];
    if (warp == 0)
        for (int i = lane; i < ncol; i += 32) gm[i] = m_run;
    if (!STEP && sh.ncta == 1) {
        __syncthreads();                           // the factors of all tokens are written
        for (int t = warp; t < nt; t += nw) head_norm_row(p.norm, t0 + t, h, lane);
    }
}

}  // namespace b200
