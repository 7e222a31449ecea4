// What the recurrent mixers with a matrix state [dk, dv] per head share (delta_rule.cuh, matrix_memory.cuh): how a head's state is
// spread over threads and stored between steps, how tokens are staged, and the norm and gate on the read-out.
//
// The columns of a state (one per value entry) are independent of one another.  A CTA owns `cols` of them; a column belongs to
// `ks` neighbouring lanes, each keeping `rt` of its dk entries in registers for all tokens of the step, so a product with the key
// or query is straight-line FMA on registers followed by log2(ks) exchanges, and no barrier separates the tokens.  Heads whose
// columns do not fit one CTA are split over `ncta` of them (prompt steps always prefer many small CTAs).  Keys, queries and the
// CTA's value entries of the next `tc` tokens arrive by cp.async while the current ones are worked on.
//
// A head's record in memory is float4 [rt / 4][dv * ks]: thread (column j, part s) finds its r-th four entries at
// [r][j ks + s], so that loads and stores are contiguous over a CTA whatever its width.  Entry i of the key dimension is entry
// i % rt of part i / rt; entries past dk are zero and stay zero.
//
// The raw read-outs go to the output rows; the root-mean-square norm over a head, its weight, a gate and a constant are applied in
// place afterwards: by the same CTA where it holds the whole head, by head_norm_kernel otherwise.  In steps of one token per sequence
// (kernel template STEP) a CTA that holds the whole head keeps the read-outs in registers and finishes them on the spot.
#pragma once
#include <cuda_runtime.h>
#include "common.cuh"
#include "linear.cuh"

namespace b200 {

constexpr int SCAN_R = 32;                         // most state entries of one column a thread keeps
constexpr int SCAN_ROW = SCAN_R + 4;               // staged floats per part: eight parts' 16-byte reads fall into different banks
constexpr int SCAN_MAX_DK = 32 * SCAN_R;
constexpr int SCAN_THREADS = 512;                  // most threads per CTA (a whole head at once: steps of one token per sequence)
constexpr int SCAN_THREADS_PROMPT = 128;
constexpr int SCAN_SMEM = 64 * 1024;               // most shared memory of a launch
constexpr int SCAN_SMEM_FIVE = 44 * 1024;          // ... with five CTAs on an SM

struct ScanShape {
    int ks, lks, rt;                               // lanes per column (a power of two and its logarithm), entries per lane (a multiple of 4)
    int threads, cols, ncta;                       // block size, columns per CTA, CTAs per head
    int tc, nbuf;                                  // tokens per staged group, staging buffers
    int rows;                                      // staged vectors of the key dimension per token (key, query, ...)
    __host__ __device__ int tok_floats() const { return rows * ks * SCAN_ROW + ((cols + 3) & ~3); }
    __host__ __device__ size_t smem_floats() const { return (size_t)nbuf * tc * (tok_floats() + 2) + (size_t)tc * (4 + threads / 32); }
};

__host__ inline void scan_parts(int dk, int& ks, int& lks, int& rt) {
    ks = 1; lks = 0;
    while (ks * SCAN_R < dk) { ks *= 2; ++lks; }
    rt = ((dk + ks - 1) / ks + 3) / 4 * 4;
}

// floats of one head's state record
__host__ inline size_t scan_state_floats(int dk, int dv) {
    int ks, lks, rt;
    scan_parts(dk, ks, lks, rt);
    return (size_t)ks * rt * dv;
}

__host__ inline ScanShape scan_shape(int dk, int dv, int rows, bool decode) {
    ScanShape s;
    scan_parts(dk, s.ks, s.lks, s.rt);
    s.rows = rows;
    const int need = (dv * s.ks + 31) / 32 * 32;   // threads that hold a whole head
    s.threads = SCAN_THREADS_PROMPT;
    if (decode && need <= SCAN_THREADS) s.threads = need > SCAN_THREADS_PROMPT ? need : SCAN_THREADS_PROMPT;
    s.cols = s.threads / s.ks;
    s.ncta = (dv + s.cols - 1) / s.cols;
    s.nbuf = decode ? 1 : 2;
    s.tc = decode ? 1 : 16;
    // five CTAs per SM (their registers allow no more): many heads and sequences then still fit one wave
    while (s.tc > 1 && s.smem_floats() * sizeof(float) > (s.tc > 4 ? SCAN_SMEM_FIVE : SCAN_SMEM)) s.tc /= 2;
    return s;
}

__device__ __forceinline__ void cp_async4(void* smem_dst, const void* gsrc) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(smem_dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(d), "l"(gsrc) : "memory");
}

// a head's vector of dk floats of `nt` consecutive tokens -> staged rows (padding is left alone)
__device__ __forceinline__ void scan_stage_keys(const ScanShape& s, float* dst, int tok_stride, const float* src, int ld, int nt, int dk) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    if (dk % 4 == 0 && ld % 4 == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0) {
        for (int i = lane * 4; i < dk; i += 128) {
            const int part = i / s.rt, at = part * SCAN_ROW + (i - part * s.rt);
            for (int t = warp; t < nt; t += nw) cp_async16(dst + (size_t)t * tok_stride + at, src + (size_t)t * ld + i);
        }
    } else {
        for (int i = lane; i < dk; i += 32) {
            const int part = i / s.rt, at = part * SCAN_ROW + (i - part * s.rt);
            for (int t = warp; t < nt; t += nw) cp_async4(dst + (size_t)t * tok_stride + at, src + (size_t)t * ld + i);
        }
    }
}

// `n` neighbouring floats of `nt` consecutive tokens
__device__ __forceinline__ void scan_stage_cols(float* dst, int tok_stride, const float* src, int ld, int nt, int n) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int i = lane; i < n; i += 32)
        for (int t = warp; t < nt; t += nw) cp_async4(dst + (size_t)t * tok_stride + i, src + (size_t)t * ld + i);
}

__device__ __forceinline__ float scan_part_sum(float v, int ks) {
    for (int o = 1; o < ks; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// this thread's share of a state record <-> registers
__device__ __forceinline__ void scan_load_state(const ScanShape& s, const float* rec, int dv, int j, int part, float st[SCAN_R]) {
    const float4* r4 = reinterpret_cast<const float4*>(rec) + (size_t)j * s.ks + part;
    const size_t plane = (size_t)dv * s.ks;
#pragma unroll
    for (int r = 0; r < SCAN_R / 4; ++r) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < dv && 4 * r < s.rt) v = r4[r * plane];
        st[4 * r] = v.x; st[4 * r + 1] = v.y; st[4 * r + 2] = v.z; st[4 * r + 3] = v.w;
    }
}
__device__ __forceinline__ void scan_store_state(const ScanShape& s, float* rec, int dv, int j, int part, const float st[SCAN_R]) {
    float4* r4 = reinterpret_cast<float4*>(rec) + (size_t)j * s.ks + part;
    const size_t plane = (size_t)dv * s.ks;
#pragma unroll
    for (int r = 0; r < SCAN_R / 4; ++r)
        if (j < dv && 4 * r < s.rt) r4[r * plane] = make_float4(st[4 * r], st[4 * r + 1], st[4 * r + 2], st[4 * r + 3]);
}

// x[t, h, :] <- f x / rms(f x) * w * act(gate) * mul   in place, f = fac[t, h] (1 without fac), act = sigmoid or silu
struct HeadNormParams {
    float* x; int ldx;                             // [T, H dv]
    const float* fac;                              // [T, H] (nullptr: 1)
    const float* gate; int ldg;                    // [T, H dv]
    const float* w; int w_hstride;                 // weight of head h at w + h w_hstride (0: shared by the heads)
    int H, dv;
    float eps, mul;
    int silu;                                      // gate activation: 0 sigmoid, 1 silu
    MetaView meta;
};

__device__ __forceinline__ void head_norm_row(const HeadNormParams& p, int t, int h, int lane) {
    float* x = p.x + (size_t)t * p.ldx + (size_t)h * p.dv;
    const float* g = p.gate + (size_t)t * p.ldg + (size_t)h * p.dv;
    const float* w = p.w + (size_t)h * p.w_hstride;
    const float f = p.fac ? p.fac[(size_t)t * p.H + h] : 1.f;
    float ss = 0.f;
    for (int j = lane; j < p.dv; j += 32) { const float v = x[j] * f; ss = fmaf(v, v, ss); }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float r = 1.f / sqrtf(ss / (float)p.dv + p.eps);
    for (int j = lane; j < p.dv; j += 32) {
        const float gl = g[j], a = lin_sigmoid(gl);
        x[j] = x[j] * f * r * w[j] * (p.silu ? gl * a : a) * p.mul;
    }
}

// the same for one entry o of a read-out whose sum of squares is known
__device__ __forceinline__ float head_norm_value(const HeadNormParams& p, float o, float f, float ss, float w, float gate) {
    const float a = lin_sigmoid(gate);
    return o * f / sqrtf(f * f * ss / (float)p.dv + p.eps) * w * (p.silu ? gate * a : a) * p.mul;
}

__global__ void __launch_bounds__(128) head_norm_kernel(const HeadNormParams p) {
    const int t = blockIdx.x;
    if (t >= p.meta.T()) return;
    for (int h = blockIdx.y * 4 + (threadIdx.x >> 5); h < p.H; h += gridDim.y * 4) head_norm_row(p, t, h, threadIdx.x & 31);
}

}  // namespace b200
