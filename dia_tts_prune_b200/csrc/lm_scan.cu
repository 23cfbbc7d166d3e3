// lm_scan.cu - the recurrences of the language-model path (sm_100a): one kernel for every mixer that carries a matrix state.
//
// Per head a state S [dim][vdim], fp32; every value column c of S evolves on its own:
//   S[:, c] <- a_t S[:, c]      a_t: one decay per key channel, or one per head (a column of the row, or fixed for all tokens)
//   tied:   S[:, c] += (1 - a_t) v_t[c]
//   delta:  u = b_t (v_t[c] - S[:, c] . k_t),  S[:, c] += k_t u
//   write:  S[:, c] += k_t (b_t v_t[c])        b_t = 1 where a mixer has no write strength
//   o_t[c] = q_mul (S[:, c] . q_t) [+ skip_h v_t[c]]
// A normaliser is one more value column whose value is the constant 1.  q and k may be shared by groups of heads.
//
// A group of P = 8, 16 or 32 lanes carries two columns of one head of one scheduled sequence; lane `part` of it holds the rows
// 4 P j + 4 part + (0 .. 3) of both, at most 8 per column, so that even one sequence gives enough warps.  The vectors of a token are
// read from shared memory in 16-byte pieces that serve both columns, and the arithmetic is packed fp32x2.  Sixteen tokens are
// staged at a time (asynchronous copies, two buffers).  A dot product is summed in four interleaved partial sums per lane and
// then across the P lanes (distances P / 2 .. 1); the read-outs of four tokens and two columns share one such exchange.  The order of operations of a column depends on nothing but the column.
// The state is read when the sequence's first row is not position 0 and written back at the end: state[slot][h][c][dim].
#include <algorithm>

#include <cuda_runtime.h>
#include <stdint.h>

#include "lm_device.cuh"
#include "lm_internal.h"

namespace lm {

namespace {

constexpr int kTokens = 16;                                   // tokens per staged chunk
constexpr int kMaxWarps = 8;

// lanes that share a pair of columns
template <int DP> constexpr int kParts = DP > 64 ? DP / 8 : 8;

using f2 = unsigned long long;                                // two packed fp32
__device__ __forceinline__ f2 pack2(float lo, float hi) {
    f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void unpack2(f2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
    f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
    f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ float sum2(f2 a, f2 b) {
    float x, y, z, w;
    unpack2(a, x, y);
    unpack2(b, z, w);
    return (x + y) + (z + w);
}
// asynchronous copies into shared memory; `ok` false writes zeros
__device__ __forceinline__ void copy16(float* dst, const float* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 16 : 0)
                 : "memory");
}
__device__ __forceinline__ void copy4(float* dst, const float* src, bool ok) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 4 : 0)
                 : "memory");
}

struct ScanArgs {
    const float* in; int ld, q_off, k_off, v_off, b_off;      // b_off < 0: write strength 1
    const float* a_in; int lda;                               // decays: column h * dim + d, or column h (one per head)
    const float* fixed_decay;                                 // [H] instead of a_in; null: none
    const float* skip;                                        // [H]; null: none
    float q_mul;
    int H, G, dim, vdim, vcols;                               // vcols: vdim, + 1 with a normaliser
    float* state;
    const int *seq_slot, *seq_row0, *seq_count, *row_pos;
    float* o; int ldo;
    int vec_qk, vec_a;                                        // whether 16-byte pieces are aligned
};

// DP: dim padded to a multiple of 32 (a power of two); VA: one decay per key channel
template <int DP, int RULE, bool VA>
__global__ void __launch_bounds__(kMaxWarps * 32, 1)
state_scan_kernel(const ScanArgs p) {
    extern __shared__ __align__(16) float sh[];
    constexpr bool KEYS = RULE != kScanTied;
    constexpr int P = kParts<DP>, CW = 64 / P, J = DP / (4 * P), VECS = 1 + (KEYS ? 1 : 0) + (VA ? 1 : 0);
    const int VC = CW * (blockDim.x >> 5);                    // value columns of the CTA
    const int stage = kTokens * (VECS * DP + VC + 2);
    pdl_release();
    pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * VC, g = h / (p.H / p.G);
    const int tid = threadIdx.x, lane = tid & 31, part = lane & (P - 1), cb = (tid >> 5) * CW + lane / P * 2;   // first column in the CTA
    const int slot = p.seq_slot[s], row0 = p.seq_row0[s], n = p.seq_count[s], start = p.row_pos[row0];
    const float a_fix = p.fixed_decay ? p.fixed_decay[h] : 0.f, sd = p.skip ? p.skip[h] : 0.f;
    const bool vec_state = p.dim % 4 == 0;

    f2 S[2][2 * J];
    float* st[2];
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        const int col = col0 + cb + c;
        const bool live = start > 0 && col < p.vcols;
        st[c] = p.state + (((size_t)slot * p.H + h) * p.vcols + (col < p.vcols ? col : 0)) * p.dim;
#pragma unroll
        for (int j = 0; j < J; ++j) {
            const int d = 4 * P * j + 4 * part;
            float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
            if (live && d < p.dim) {
                if (vec_state) t = *reinterpret_cast<const float4*>(st[c] + d);
                else {
                    t.x = st[c][d];
                    if (d + 1 < p.dim) t.y = st[c][d + 1];
                    if (d + 2 < p.dim) t.z = st[c][d + 2];
                    if (d + 3 < p.dim) t.w = st[c][d + 3];
                }
            }
            S[c][2 * j] = pack2(t.x, t.y);
            S[c][2 * j + 1] = pack2(t.z, t.w);
        }
    }

    // one staged vector: kTokens rows of DP channels (zeros beyond dim)
    auto stage_vec = [&](float* dst, const float* src, int ld, int nt, bool vec) {
        if (vec) {
            for (int i = tid; i < nt * (DP / 4); i += blockDim.x) {
                const int t = i / (DP / 4), c = 4 * (i - t * (DP / 4));
                copy16(dst + t * DP + c, src + (size_t)t * ld + (c < p.dim ? c : 0), c < p.dim);
            }
        } else {
            for (int i = tid; i < nt * DP; i += blockDim.x) {
                const int t = i / DP, c = i - t * DP;
                copy4(dst + i, src + (size_t)t * ld + (c < p.dim ? c : 0), c < p.dim);
            }
        }
    };
    auto stage_chunk = [&](int t0, float* buf) {
        const int nt = min(kTokens, n - t0);
        const float* base = p.in + (size_t)(row0 + t0) * p.ld;
        float* dst = buf;
        stage_vec(dst, base + p.q_off + g * p.dim, p.ld, nt, p.vec_qk);
        dst += kTokens * DP;
        if (KEYS) {
            stage_vec(dst, base + p.k_off + g * p.dim, p.ld, nt, p.vec_qk);
            dst += kTokens * DP;
        }
        if (VA) {
            stage_vec(dst, p.a_in + (size_t)(row0 + t0) * p.lda + h * p.dim, p.lda, nt, p.vec_a);
            dst += kTokens * DP;
        }
        for (int i = tid; i < nt * VC; i += blockDim.x) {
            const int t = i / VC, c = col0 + i - t * VC;
            if (c == p.vdim && c < p.vcols) dst[i] = 1.f;     // the normaliser's value
            else copy4(dst + i, base + (size_t)t * p.ld + p.v_off + h * p.vdim + (c < p.vdim ? c : 0), c < p.vdim);
        }
        dst += kTokens * VC;
        if (tid < nt) {
            if (!VA) {
                if (p.fixed_decay) dst[tid] = a_fix;
                else copy4(dst + tid, p.a_in + (size_t)(row0 + t0 + tid) * p.lda + h, true);
            }
            if (p.b_off >= 0) copy4(dst + kTokens + tid, base + (size_t)tid * p.ld + p.b_off + h, true);
            else dst[kTokens + tid] = 1.f;
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    stage_chunk(0, sh);
    for (int t0 = 0, cur = 0; t0 < n; t0 += kTokens, cur ^= 1) {
        const int nt = min(kTokens, n - t0);
        if (t0 + kTokens < n) {                               // (the other buffer was released at the end of the last turn)
            stage_chunk(t0 + kTokens, sh + (cur ^ 1) * stage);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* sq = sh + cur * stage;
        const float* sk = sq + kTokens * DP;
        const float* sa = sk + (KEYS ? kTokens * DP : 0);
        const float* sv = sa + (VA ? kTokens * DP : 0);
        const float* ss = sv + kTokens * VC;                  // decay per token, then write strength per token

        auto token = [&](int t, float& d0, float& d1) {
            const ulonglong2* q = reinterpret_cast<const ulonglong2*>(sq + t * DP) + part;
            const ulonglong2* k = reinterpret_cast<const ulonglong2*>(sk + t * DP) + part;
            const ulonglong2* a = reinterpret_cast<const ulonglong2*>(sa + t * DP) + part;
            const float2 v = *reinterpret_cast<const float2*>(sv + t * VC + cb);
            const float bt = ss[kTokens + t];
            f2 as = 0;
            if (!VA) as = pack2(ss[t], ss[t]);
            f2 acc[2][2] = {{0, 0}, {0, 0}};
            if (RULE == kScanDelta) {
                f2 e[2][2] = {{0, 0}, {0, 0}};
                ulonglong2 kk[J];
#pragma unroll
                for (int j = 0; j < J; ++j) {
                    kk[j] = k[P * j];
                    ulonglong2 aa;
                    if (VA) aa = a[P * j];
                    else aa.x = aa.y = as;
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        S[c][2 * j] = mul2(aa.x, S[c][2 * j]);
                        S[c][2 * j + 1] = mul2(aa.y, S[c][2 * j + 1]);
                        e[c][0] = fma2(S[c][2 * j], kk[j].x, e[c][0]);
                        e[c][1] = fma2(S[c][2 * j + 1], kk[j].y, e[c][1]);
                    }
                }
                float e0 = sum2(e[0][0], e[0][1]), e1 = sum2(e[1][0], e[1][1]);
#pragma unroll
                for (int o = P / 2; o > 0; o >>= 1) {
                    e0 += __shfl_xor_sync(0xffffffffu, e0, o);
                    e1 += __shfl_xor_sync(0xffffffffu, e1, o);
                }
                const float u0 = bt * (v.x - e0), u1 = bt * (v.y - e1);
                const f2 u[2] = {pack2(u0, u0), pack2(u1, u1)};
#pragma unroll
                for (int j = 0; j < J; ++j) {
                    const ulonglong2 qq = q[P * j];
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        S[c][2 * j] = fma2(kk[j].x, u[c], S[c][2 * j]);
                        S[c][2 * j + 1] = fma2(kk[j].y, u[c], S[c][2 * j + 1]);
                        acc[c][0] = fma2(S[c][2 * j], qq.x, acc[c][0]);
                        acc[c][1] = fma2(S[c][2 * j + 1], qq.y, acc[c][1]);
                    }
                }
            } else {
                const float w0 = RULE == kScanWrite ? bt * v.x : v.x, w1 = RULE == kScanWrite ? bt * v.y : v.y;
                const f2 u[2] = {pack2(w0, w0), pack2(w1, w1)};
                const f2 one = pack2(1.f, 1.f), minus = pack2(-1.f, -1.f);
#pragma unroll
                for (int j = 0; j < J; ++j) {
                    const ulonglong2 qq = q[P * j];
                    ulonglong2 aa, kk;
                    if (VA) aa = a[P * j];
                    else aa.x = aa.y = as;
                    if (KEYS) kk = k[P * j];
                    else { kk.x = fma2(aa.x, minus, one); kk.y = fma2(aa.y, minus, one); }     // tied: 1 - a
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        S[c][2 * j] = fma2(aa.x, S[c][2 * j], mul2(kk.x, u[c]));
                        S[c][2 * j + 1] = fma2(aa.y, S[c][2 * j + 1], mul2(kk.y, u[c]));
                        acc[c][0] = fma2(S[c][2 * j], qq.x, acc[c][0]);
                        acc[c][1] = fma2(S[c][2 * j + 1], qq.y, acc[c][1]);
                    }
                }
            }
            d0 = sum2(acc[0][0], acc[0][1]);
            d1 = sum2(acc[1][0], acc[1][1]);
        };
        auto store = [&](int t, int c, float dot) {
            const int col = col0 + cb + c;
            if (col < p.vcols) p.o[(size_t)(row0 + t0 + t) * p.ldo + h * p.vcols + col] = fmaf(sd, sv[t * VC + cb + c], dot * p.q_mul);
        };
        int t = 0;
        for (; t + 4 <= nt; t += 4) {
            float d[8];
#pragma unroll
            for (int i = 0; i < 4; ++i) token(t + i, d[2 * i], d[2 * i + 1]);
            // eight values over P lanes: at the first three distances a lane keeps the half of the values that its bit names and
            // gives the other away, then the last value is summed over the lanes that hold it
#pragma unroll
            for (int m = 4, o = P / 2; m > 0; m >>= 1, o >>= 1) {
                const bool up = part & o;
#pragma unroll
                for (int i = 0; i < m; ++i) {
                    const float give = up ? d[i] : d[i + m], keep = up ? d[i + m] : d[i];
                    d[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
                }
            }
#pragma unroll
            for (int o = P / 16; o > 0; o >>= 1) d[0] += __shfl_xor_sync(0xffffffffu, d[0], o);
            const int at = part / (P / 8);                    // the value that this lane holds: token at >> 1, column at & 1
            if (part % (P / 8) == 0) store(t + (at >> 1), at & 1, d[0]);
        }
        for (; t < nt; ++t) {
            float d0, d1;
            token(t, d0, d1);
#pragma unroll
            for (int o = P / 2; o > 0; o >>= 1) {
                d0 += __shfl_xor_sync(0xffffffffu, d0, o);
                d1 += __shfl_xor_sync(0xffffffffu, d1, o);
            }
            if (part < 2) store(t, part, part ? d1 : d0);
        }
        __syncthreads();                                      // this buffer is consumed
    }
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        if (col0 + cb + c >= p.vcols) continue;
#pragma unroll
        for (int j = 0; j < J; ++j) {
            const int d = 4 * P * j + 4 * part;
            if (d >= p.dim) continue;
            float4 t;
            unpack2(S[c][2 * j], t.x, t.y);
            unpack2(S[c][2 * j + 1], t.z, t.w);
            if (vec_state) *reinterpret_cast<float4*>(st[c] + d) = t;
            else {
                st[c][d] = t.x;
                if (d + 1 < p.dim) st[c][d + 1] = t.y;
                if (d + 2 < p.dim) st[c][d + 2] = t.z;
                if (d + 3 < p.dim) st[c][d + 3] = t.w;
            }
        }
    }
}

template <int DP, int RULE, bool VA>
cudaError_t launch_inst(const ScanArgs& p, int n_seq, bool early, cudaStream_t st) {
    // warps of a CTA share the staged vectors: as many as leave a CTA for every SM
    constexpr int CW = 64 / kParts<DP>;
    const long long total = (long long)n_seq * p.H * ((p.vcols + CW - 1) / CW);
    int warps = 1;
    while (warps < kMaxWarps && total >= 120 * 2 * warps && CW * warps < p.vcols) warps *= 2;
    if (warps == kMaxWarps && total < 16 * 148) warps /= 2;
    constexpr int VECS = 1 + (RULE != kScanTied ? 1 : 0) + (VA ? 1 : 0);
    const int VC = 64 / kParts<DP> * warps;
    const size_t smem = (size_t)2 * kTokens * (VECS * DP + VC + 2) * 4;
    static size_t allowed[64] = {};
    if (smem > 48 * 1024) {
        int dev = 0;
        cudaError_t e = cudaGetDevice(&dev);
        if (e != cudaSuccess) return e;
        if (dev < 0 || dev >= 64 || allowed[dev] < smem) {
            e = cudaFuncSetAttribute(state_scan_kernel<DP, RULE, VA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return e;
            if (dev >= 0 && dev < 64) allowed[dev] = smem;
        }
    }
    return launch_pdl_if(early, state_scan_kernel<DP, RULE, VA>, dim3(n_seq, p.H, (p.vcols + VC - 1) / VC), dim3(32 * warps), smem, st, p);
}

template <int RULE, bool VA>
cudaError_t launch_scan(const ScanArgs& p, int n_seq, bool early, cudaStream_t st) {
    if (p.dim > 256 || p.H % p.G || p.H > 65535) return cudaErrorNotSupported;
    if (p.dim <= 32) return launch_inst<32, RULE, VA>(p, n_seq, early, st);
    if (p.dim <= 64) return launch_inst<64, RULE, VA>(p, n_seq, early, st);
    if (p.dim <= 128) return launch_inst<128, RULE, VA>(p, n_seq, early, st);
    return launch_inst<256, RULE, VA>(p, n_seq, early, st);
}

bool aligned16(const float* base, int ld, int off, int dim) {
    return dim % 4 == 0 && ld % 4 == 0 && off % 4 == 0 && (reinterpret_cast<uintptr_t>(base) & 15) == 0;
}

}  // namespace

cudaError_t launch_column_scan(const float* in, int ld, const ScanInputs& si, int rule, int H, int G, int dim, int vdim, float* state,
                               const SeqMeta& sm, const RowMeta& rm, int n_seq, float* o, int ldo, cudaStream_t st, bool head_decay,
                               bool early, const float* decay, int ldd, float q_mul) {
    if (G <= 0 || H <= 0) return cudaErrorInvalidValue;
    const float* a = decay ? decay : in + si.a_off;
    const int lda = decay ? ldd : ld;
    ScanArgs p{in, ld, si.q_off, si.k_off, si.v_off, rule == kScanDelta ? si.beta_off : -1, a, lda, nullptr, nullptr, q_mul, H, G, dim, vdim,
               vdim, state, sm.slot, sm.row0, sm.count, rm.pos, o, ldo, 0, 0};
    p.vec_qk = aligned16(in, ld, si.q_off, dim) && (rule == kScanTied || aligned16(in, ld, si.k_off, dim));
    p.vec_a = aligned16(a, lda, 0, dim);
    switch (rule) {
        case kScanTied: return head_decay ? cudaErrorNotSupported : launch_scan<kScanTied, true>(p, n_seq, early, st);
        case kScanDelta:
            return head_decay ? launch_scan<kScanDelta, false>(p, n_seq, early, st) : launch_scan<kScanDelta, true>(p, n_seq, early, st);
        case kScanWrite: return head_decay ? cudaErrorNotSupported : launch_scan<kScanWrite, true>(p, n_seq, early, st);
        default: return cudaErrorInvalidValue;
    }
}

cudaError_t launch_scalar_gate_scan(const float* in, int ld, const ScanInputs& si, int H, int dim, int vdim, float* state,
                                    const SeqMeta& sm, const RowMeta& rm, int n_seq, float* o, int ldo, cudaStream_t st,
                                    const float* fixed_decay, bool normaliser, bool early, int G, const float* skip) {
    if (G <= 0) G = H;
    ScanArgs p{in, ld, si.q_off, si.k_off, si.v_off, fixed_decay ? -1 : si.beta_off, in + si.a_off, ld, fixed_decay, skip, 1.f, H, G, dim, vdim,
               vdim + (normaliser ? 1 : 0), state, sm.slot, sm.row0, sm.count, rm.pos, o, ldo, 0, 0};
    p.vec_qk = aligned16(in, ld, si.q_off, dim) && aligned16(in, ld, si.k_off, dim);
    return launch_scan<kScanWrite, false>(p, n_seq, early, st);
}

}  // namespace lm
