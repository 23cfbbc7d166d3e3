// lm_device.cuh - device helpers and the launch helper shared by the language-model kernels (lm_kernels.cu,
// lm_mixers.cu).  Everything here has internal linkage.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math_constants.h>
#include <stdint.h>

namespace lm {
namespace {

__device__ __forceinline__ float bf(const __nv_bfloat16 v) { return __bfloat162float(v); }

__device__ __forceinline__ float dyt(float x, float alpha, float w, float b) { return fmaf(tanhf(alpha * x), w, b); }

// Programmatic dependent launch: a kernel of a short step lets the next one start as soon as it runs itself
// (pdl_release) and reads what earlier kernels wrote - or writes anything - only after pdl_wait.  Before the wait a
// kernel may fetch weights, which no kernel writes.  Launched without the attribute both are no-ops.
__device__ __forceinline__ void pdl_release() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// fixed-tree block reductions (red: one float per warp); every thread gets the result
__device__ __forceinline__ float block_sum(float v, float* red) {
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) red[w] = v;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < nw; ++i) t += red[i];
    return t;
}

__device__ __forceinline__ float sigmoidf_(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float siluf_(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplusf_(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// activation of a gated unit on its gate g and up u products.  kGluSilu: silu(g) u.  kGluClamped: both are clamped first
// (g from above, u on both sides), the gate's sigmoid is 1.702 times steeper and the up branch is offset by one:
// g' sigmoid(1.702 g') (u' + 1).  kGluGelu: gelu(g) u with the tanh form of gelu
constexpr int kGluSilu = 0, kGluClamped = 1, kGluGelu = 2;
__device__ __forceinline__ float gelu_tanhf_(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z)));
}
// activation of a unit that is not gated (kAct* of lm_internal.h).  xIELU: z > 0: ap z^2 + z / 2;  z <= 0: an (e^z - 1 - z) + z / 2
__device__ __forceinline__ float unit_act(int act, float z, float ap, float an) {
    switch (act) {
        case 1: return z > 0.f ? fmaf(ap * z, z, 0.5f * z) : fmaf(an, expm1f(z) - z, 0.5f * z);
        case 2: return fmaxf(z, 0.f) * fmaxf(z, 0.f);
        case 3: return gelu_tanhf_(z);
        default: return z;
    }
}
// the first key a query at position i sees behind the kept first ones: its window's, and its chunk's where they are bounded
__device__ __forceinline__ int first_key(int i, int window, int chunk) {
    const int w = window > 0 ? max(0, i - window + 1) : 0;
    return chunk > 0 ? max(w, i - i % chunk) : w;
}
__device__ __forceinline__ float glu_act(int kind, float g, float u, float limit) {
    if (kind == kGluClamped) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g * sigmoidf_(1.702f * g) * (u + 1.0f);
    }
    return (kind == kGluGelu ? gelu_tanhf_(g) : siluf_(g)) * u;
}

// one warp's dot product of a bf16 weight row with an fp32 activation row (x sc), 16 bytes of weights per lane and load;
// every lane gets the sum
// wait_first: the first weight loads go out before pdl_wait, the activations are read after it
__device__ __forceinline__ float warp_dot(const float* __restrict__ arow, const __nv_bfloat16* __restrict__ wrow, int K, int lda,
                                          float sc, int lane, bool wait_first = false) {
    float acc = 0.f;
    const bool vec = (K % 8 == 0) && (lda % 4 == 0) && ((reinterpret_cast<uintptr_t>(wrow) & 15) == 0) &&
                     ((reinterpret_cast<uintptr_t>(arow) & 15) == 0);
    if (vec) {
        // eight 16-byte weight loads per lane in flight before their products (the sum keeps its order: k ascending)
        for (int k0 = lane * 8; k0 < K; k0 += 2048) {
            uint4 wv[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int k = k0 + 256 * u;
                wv[u] = k < K ? *reinterpret_cast<const uint4*>(wrow + k) : make_uint4(0u, 0u, 0u, 0u);
            }
            if (wait_first) { pdl_wait(); wait_first = false; }
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int k = k0 + 256 * u;
                if (k >= K) break;
                const float4 x0 = *reinterpret_cast<const float4*>(arow + k);
                const float4 x1 = *reinterpret_cast<const float4*>(arow + k + 4);
                const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&wv[u]);
                acc = fmaf(x0.x * sc, __low2float(p[0]), acc);
                acc = fmaf(x0.y * sc, __high2float(p[0]), acc);
                acc = fmaf(x0.z * sc, __low2float(p[1]), acc);
                acc = fmaf(x0.w * sc, __high2float(p[1]), acc);
                acc = fmaf(x1.x * sc, __low2float(p[2]), acc);
                acc = fmaf(x1.y * sc, __high2float(p[2]), acc);
                acc = fmaf(x1.z * sc, __low2float(p[3]), acc);
                acc = fmaf(x1.w * sc, __high2float(p[3]), acc);
            }
        }
    } else {
        if (wait_first) pdl_wait();
        for (int k = lane; k < K; k += 32) acc = fmaf(arow[k] * sc, bf(wrow[k]), acc);
    }
    if (wait_first) pdl_wait();                               // (K == 0: nothing was loaded)
    return warp_sum(acc);
}

// the kernels of a short step are launched with programmatic stream serialization (see pdl_release / pdl_wait)
// early == false: a plain launch, which starts when its predecessor has ended.  For a kernel of few, long-running CTAs
// behind a kernel of thousands of short ones (a recurrence scan behind its per-row preparation) that is the faster
// order: CTAs that arrive while the predecessor drains are placed wherever a slot frees first, several to an SM, and
// stay there for the whole scan.
template <typename... KArgs, typename... Args>
cudaError_t launch_pdl_if(bool early, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = early ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}
template <typename... KArgs, typename... Args>
cudaError_t launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, Args... args) {
    return launch_pdl_if(true, kernel, grid, block, smem, st, args...);
}

}  // namespace
}  // namespace lm
