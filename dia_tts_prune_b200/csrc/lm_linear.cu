// lm_linear.cu - kernels around the linear-attention recurrences and of the per-layer token input (sm_100a).
//
// Same step layout and the same rule as lm_kernels.cu: every kernel computes a row's result from that row and the
// sequence state it points at, in an order of operations that does not depend on what else is in the batch.  Decays,
// step sizes, gates of the recurrence and norms are fp32.
//
//   decay_proj_kernel         gated linear attention: the second step of the decay projection (a handful of inner channels), its
//                             bias and sigmoid(z)^(1 / tau) in one launch, fp32 arithmetic
//   ssm_prep_kernel           state-space mixer: short causal convolution + bias + silu of x, B and C (previous inputs from the
//                             step or the sequence's tail), softplus step sizes and the decay per head
//   gate_norm_kernel          state-space mixer: y silu(z), then an RMS norm over equal parts of the row, x weight
//   side_act_kernel           token input: gelu(z) times the token's slice of the second embedding table
//   side_gate_rows_kernel     the same with the product in front, for a handful of rows
//
// The recurrences themselves run in lm_scan.cu, the convolution's tail is kept by conv_tail_kernel of lm_mixers.cu, and the
// token input's own norm and residual add are options of streams_step_kernel.
#include <algorithm>

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "lm_device.cuh"
#include "lm_internal.h"

namespace lm {

// ---------------------------------------------------------------------------------------------------------------------
// One thread per channel, RT rows per CTA: a channel's weights are read once for the RT rows, whose inner vectors wait in
// shared memory.
template <int RT>
__global__ void __launch_bounds__(128)
decay_proj_kernel(const float* __restrict__ a, int lda, const __nv_bfloat16* __restrict__ W, const float* __restrict__ bias, float tau,
                  float* __restrict__ out, int C, int rank, int M) {
    extern __shared__ float as[];                             // [RT][rank]
    pdl_release();
    pdl_wait();
    const int r0 = blockIdx.y * RT, c = blockIdx.x * blockDim.x + threadIdx.x;
    for (int i = threadIdx.x; i < RT * rank; i += blockDim.x) {
        const int r = i / rank, k = i - r * rank;
        as[i] = r0 + r < M ? a[(size_t)(r0 + r) * lda + k] : 0.f;
    }
    __syncthreads();
    if (c >= C) return;
    const __nv_bfloat16* w = W + (size_t)c * rank;
    float acc[RT];
#pragma unroll
    for (int r = 0; r < RT; ++r) acc[r] = 0.f;
    if (rank % 8 == 0 && (reinterpret_cast<uintptr_t>(W) & 15) == 0) {
        for (int k = 0; k < rank; k += 8) {
            const uint4 wv = *reinterpret_cast<const uint4*>(w + k);
            const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&wv);
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float w0 = __low2float(p[u]), w1 = __high2float(p[u]);
#pragma unroll
                for (int r = 0; r < RT; ++r) {
                    acc[r] = fmaf(w0, as[r * rank + k + 2 * u], acc[r]);
                    acc[r] = fmaf(w1, as[r * rank + k + 2 * u + 1], acc[r]);
                }
            }
        }
    } else {
        for (int k = 0; k < rank; ++k) {
            const float wk = bf(w[k]);
#pragma unroll
            for (int r = 0; r < RT; ++r) acc[r] = fmaf(wk, as[r * rank + k], acc[r]);
        }
    }
    const float b = bias ? bias[c] : 0.f;
#pragma unroll
    for (int r = 0; r < RT; ++r)
        if (r0 + r < M) out[(size_t)(r0 + r) * C + c] = expf(-softplusf_(-(acc[r] + b)) / tau);      // ln sigmoid(z) = -softplus(-z)
}

// ---------------------------------------------------------------------------------------------------------------------
// One thread per channel and up to kSsmRows rows.  Channels 0 .. C are those of the convolution, C .. C + H the step sizes.
constexpr int kSsmRows = 8;

__global__ void __launch_bounds__(128)
ssm_prep_kernel(const float* __restrict__ proj, int ld, int x_off, int C, int H, int taps, const float* __restrict__ cw,
                const float* __restrict__ cb, const float* __restrict__ tail, const float* __restrict__ a_log,
                const float* __restrict__ dt_bias, const int* __restrict__ row_slot, const int* __restrict__ row_pos,
                const int* __restrict__ row_start, float* __restrict__ rec, int ldr, int M) {
    pdl_release();
    pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x, r0 = blockIdx.y * kSsmRows, r1 = min(M, r0 + kSsmRows), T1 = taps - 1;
    if (c >= C + H) return;
    if (c >= C) {
        const int h = c - C;
        const float A = expf(a_log[h]), b = dt_bias[h];
        for (int r = r0; r < r1; ++r) {
            const float dt = softplusf_(proj[(size_t)r * ld + x_off + c] + b);
            rec[(size_t)r * ldr + C + h] = expf(-A * dt);
            rec[(size_t)r * ldr + C + H + h] = dt;
        }
        return;
    }
    const float* w = cw + (size_t)c * taps;
    const float b = cb ? cb[c] : 0.f;
    // a full tile inside one sequence whose earlier inputs all stand in this step: every input is loaded once, all of them in
    // flight together (the sums run in the same order as below; taps that are not there weigh 0)
    constexpr int KT = 4;
    if (taps <= KT && r1 - r0 == kSsmRows && row_slot[r1 - 1] == row_slot[r0] && row_pos[r1 - 1] - row_pos[r0] == kSsmRows - 1 &&
        row_pos[r0] - row_start[r0] >= KT - 1) {
        float u[kSsmRows + KT - 1], wt[KT];
#pragma unroll
        for (int i = 0; i < kSsmRows + KT - 1; ++i) u[i] = proj[(size_t)(r0 - (KT - 1) + i) * ld + x_off + c];
#pragma unroll
        for (int o = 0; o < KT; ++o) wt[o] = o < taps ? w[taps - 1 - o] : 0.f;
#pragma unroll
        for (int i = 0; i < kSsmRows; ++i) {
            float acc = b;
#pragma unroll
            for (int o = 0; o < KT; ++o) acc = fmaf(wt[o], u[i + KT - 1 - o], acc);
            rec[(size_t)(r0 + i) * ldr + c] = siluf_(acc);
        }
        return;
    }
    for (int r = r0; r < r1; ++r) {
        const int slot = row_slot[r], pos = row_pos[r], start = row_start[r];
        float acc = b;
        for (int o = 0; o < taps; ++o) {
            const int p = pos - o;
            if (p < 0) break;
            const float u = p >= start ? proj[(size_t)(r - o) * ld + x_off + c]
                                       : tail[((size_t)slot * T1 + (p - (start - T1))) * C + c];
            acc = fmaf(w[taps - 1 - o], u, acc);
        }
        rec[(size_t)r * ldr + c] = siluf_(acc);
    }
}

// ---------------------------------------------------------------------------------------------------------------------
// One CTA per (row, part)
__global__ void __launch_bounds__(256)
gate_norm_kernel(float* __restrict__ o, int ldo, __nv_bfloat16* __restrict__ o_b, const float* __restrict__ z, int ldz,
                 const float* __restrict__ w, int size, float eps, float out_scale) {
    __shared__ float red[32];
    pdl_release();
    pdl_wait();
    const int c0 = blockIdx.y * size;
    float* row = o + (size_t)blockIdx.x * ldo + c0;
    const float* zr = z + (size_t)blockIdx.x * ldz + c0;
    float ss = 0.f;
    for (int c = threadIdx.x; c < size; c += blockDim.x) {
        const float v = row[c] * siluf_(zr[c]);
        row[c] = v;                                           // (read back by this thread alone)
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)size + eps);
    for (int c = threadIdx.x; c < size; c += blockDim.x) {
        const float v = row[c] * inv * w[c0 + c] * out_scale;
        row[c] = v;
        if (o_b) o_b[(size_t)blockIdx.x * ldo + c0 + c] = __float2bfloat16_rn(v);
    }
}

// ---------------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ float side_value(const __nv_bfloat16* table, int ld, int off, int vocab, int id, int c) {
    return id >= 0 && id < vocab ? bf(table[(size_t)id * ld + off + c]) : 0.f;
}

__global__ void side_act_kernel(const float* __restrict__ z, const __nv_bfloat16* __restrict__ table, int ld, int off, int n,
                                const int* __restrict__ ids, int vocab, float* __restrict__ g, __nv_bfloat16* __restrict__ g_b) {
    pdl_release();
    pdl_wait();
    const size_t r = blockIdx.x;
    const int id = ids[r];
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
        const float v = gelu_tanhf_(z[r * n + c]) * side_value(table, ld, off, vocab, id, c);
        if (g) g[r * n + c] = v;
        if (g_b) g_b[r * n + c] = __float2bfloat16_rn(v);
    }
}

__global__ void __launch_bounds__(256)
side_gate_rows_kernel(const float* __restrict__ x, int D, const __nv_bfloat16* __restrict__ W, const __nv_bfloat16* __restrict__ table,
                      int ld, int off, int n, const int* __restrict__ ids, int vocab, float* __restrict__ g) {
    pdl_release();
    const int r = blockIdx.y, lane = threadIdx.x & 31, c = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (c >= n) return;
    const float z = warp_dot(x + (size_t)r * D, W + (size_t)c * D, D, D, 1.f, lane, true);
    if (lane == 0) g[(size_t)r * n + c] = gelu_tanhf_(z) * side_value(table, ld, off, vocab, ids[r], c);
}

// ---- launchers --------------------------------------------------------------------------------------------------------
cudaError_t launch_decay_proj(const float* a, int lda, const void* W, const float* bias, float tau, float* out, int C, int rank,
                              int M, cudaStream_t st) {
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(W);
    const int cols = (C + 127) / 128;
    if (M <= kRowsKernelMax)
        return launch_pdl(decay_proj_kernel<1>, dim3(cols, M), dim3(128), (size_t)rank * 4, st, a, lda, w, bias, tau, out, C, rank, M);
    constexpr int RT = 8;
    const size_t smem = (size_t)RT * rank * 4;
    if (smem > 48 * 1024) return cudaErrorNotSupported;
    return launch_pdl(decay_proj_kernel<RT>, dim3(cols, (M + RT - 1) / RT), dim3(128), smem, st, a, lda, w, bias, tau, out, C, rank, M);
}

cudaError_t launch_ssm_prep(const float* proj, int ld, int x_off, const SsmShape& d, const float* tail, const RowMeta& rm, float* rec,
                            int ldr, int M, cudaStream_t st) {
    if (d.taps < 1 || d.taps > kMaxTaps) return cudaErrorNotSupported;
    const int C = d.heads * d.vdim + 2 * d.groups * d.state;
    return launch_pdl(ssm_prep_kernel, dim3((C + d.heads + 127) / 128, (M + kSsmRows - 1) / kSsmRows), dim3(128), 0, st, proj, ld, x_off,
                      C, d.heads, d.taps, d.conv_w, d.conv_b, tail, d.a_log, d.dt_bias, rm.slot, rm.pos, rm.start, rec, ldr, M);
}

cudaError_t launch_gate_norm(float* o, int ldo, void* o_bf16, const float* z, int ldz, const float* w, int n, int parts, float eps,
                             float out_scale, int M, cudaStream_t st) {
    if (parts < 1 || parts > 65535 || n % parts) return cudaErrorInvalidValue;
    const int size = n / parts, threads = size <= 64 ? 32 : size <= 512 ? 128 : 256;
    return launch_pdl(gate_norm_kernel, dim3(M, parts), dim3(threads), 0, st, o, ldo, reinterpret_cast<__nv_bfloat16*>(o_bf16), z, ldz, w,
                      size, eps, out_scale);
}

cudaError_t launch_side_act(const float* z, const TokenSide& ts, float* g, void* g_bf16, int M, cudaStream_t st) {
    return launch_pdl(side_act_kernel, dim3(M), dim3(ts.n <= 64 ? 32 : 128), 0, st, z, reinterpret_cast<const __nv_bfloat16*>(ts.table),
                      ts.ld, ts.off, ts.n, ts.ids, ts.vocab, g, reinterpret_cast<__nv_bfloat16*>(g_bf16));
}

cudaError_t launch_side_gate_rows(const float* x, int D, const void* W, const TokenSide& ts, float* g, int M, cudaStream_t st) {
    return launch_pdl(side_gate_rows_kernel, dim3((ts.n + 7) / 8, M), dim3(256), 0, st, x, D, reinterpret_cast<const __nv_bfloat16*>(W),
                      reinterpret_cast<const __nv_bfloat16*>(ts.table), ts.ld, ts.off, ts.n, ts.ids, ts.vocab, g);
}

}  // namespace lm
