// Rank-one memories: matrix states with one decay and one write strength per head and token -- the gated delta rule and
// state-space layers (see umbs_memory_t in include/umbrella_b200_seq.h).  fp32 arithmetic throughout; the state is fp32
// [slots, heads, vdim, dim], key index last, so that a value column is contiguous.
//
//   umbs_memory_prep : short causal convolution + silu, unit norms of q and k, decay and strength, the dot product k . q.
//   umbs_memory_run  : the recurrence, one block per (value columns, head, sequence).
//   umbs_gated_norm  : unit RMS of the parts of the output, weight, silu gate (in front of the norm or behind it).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "seq_internal.h"

namespace umbs {

__device__ __forceinline__ float warp_sum_mem(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float silu_mem(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_mem(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------------------------------------ preparation
constexpr int kPrepWarps = 4, kPrepVals = 4;       // warps per block; channels per lane of a value task

// A warp's task: one query / key head (both vectors, their norms and their dot product), 128 value channels, or the gates
// of all heads -- for TT consecutive tokens.  TAPS > 0: the number of taps is known, the tile's projected values and the
// rows in front of it are loaded into registers together and every convolution reads them there; TAPS == 0: any number, one
// value at a time.  A lane's sums run in a fixed order, so a token's result does not depend on what else is in the step.
template <int NC, int TAPS, int TT>
__global__ void __launch_bounds__(32 * kPrepWarps) memory_prep_kernel(const float* __restrict__ proj, int64_t ld, umbs_memory_t m, Batch b,
                                                                      int slots, float* __restrict__ qkv, int64_t ld_qkv,
                                                                      float* __restrict__ gates, float* __restrict__ kq) {
    const int lane = threadIdx.x & 31, task = blockIdx.y * kPrepWarps + (threadIdx.x >> 5);
    const int G = m.kv_heads, D = m.dim, cv = m.heads * m.vdim, C = 2 * G * D + cv, taps = TAPS > 0 ? TAPS : m.taps, keep = taps - 1;
    const int vtasks = (cv + 32 * kPrepVals - 1) / (32 * kPrepVals);
    const int t0 = blockIdx.x * TT, nt = min(TT, b.n_tokens - t0);
    if (task > G + vtasks) return;
    if (task == G + vtasks) {
        for (int i = lane; i < nt * m.heads; i += 32) {
            const int t = t0 + i / m.heads, h = i % m.heads;
            const float* row = proj + (int64_t)t * ld;
            const float dt = softplus_mem(row[m.off_decay + h] + m.dt_bias[h]);
            float* g = gates + ((int64_t)t * m.heads + h) * 2;
            g[0] = -m.decay_rate[h] * dt;
            g[1] = m.off_strength >= 0 ? 1.f / (1.f + expf(-row[m.off_strength + h])) : dt;
        }
        return;
    }
    int start[TT], pos0[TT];                       // per token: first row of its sequence in the step, position of that row
    int64_t st_in[TT];                             // where its sequence's carried rows begin
    bool last[TT];
#pragma unroll
    for (int j = 0; j < TT; ++j) {
        const int s = j < nt ? b.tok_seq[t0 + j] : b.tok_seq[t0];
        start[j] = b.seq_start[s];
        pos0[j] = b.seq_pos0[s];
        st_in[j] = ((int64_t)b.seq_parity[s] * slots + b.seq_slot[s]) * keep * C;
        last[j] = keep > 0 && j < nt && t0 + j == start[j] + b.seq_len[s] - 1;
    }
    // channel c of the row `back` rows in front of the first row of token j's sequence: a carried row, or zero in front of the sequence
    auto carried = [&](int j, int c, int back) -> float {
        return pos0[j] >= back ? m.conv_state[st_in[j] + (int64_t)(keep - back) * C + c] : 0.f;
    };
    // the other half of the buffer: the sequence's last token of the step leaves the rows the next step starts from
    auto carry_slot = [&](int j) -> float* {
        const int s = b.tok_seq[t0 + j];
        return m.conv_state + ((int64_t)(b.seq_parity[s] ^ 1) * slots + b.seq_slot[s]) * keep * C;
    };
    constexpr int KEEP = TAPS > 1 ? TAPS - 1 : 0, ROWS = TAPS > 0 ? TT + KEEP : 1;
    // One channel: raw[] are its projected values at rows t0 - KEEP .. t0 + TT - 1 of the step.
    auto fetch = [&](int c, float (&raw)[ROWS]) {
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int r = 0; r < ROWS; ++r) {
                const int t = t0 - KEEP + r;
                raw[r] = (t >= 0 && t < t0 + nt) ? proj[(int64_t)t * ld + m.off_conv + c] : 0.f;
            }
        }
    };
    auto conv = [&](int j, int c, const float (&raw)[ROWS], const float (&w)[TAPS > 0 ? TAPS : 1], float bias) -> float {
        float acc = bias;
        const int r0 = t0 + j - start[j];          // the token's row in its sequence's part of the step
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int x = 0; x < TAPS; ++x) {
                const int r = r0 - KEEP + x;
                acc = fmaf(w[x], r >= 0 ? raw[j + x] : carried(j, c, -r), acc);
            }
        } else {
            for (int x = 0; x < taps; ++x) {
                const int r = r0 - keep + x;
                acc = fmaf(m.conv_w[(int64_t)c * taps + x], r >= 0 ? proj[(int64_t)(start[j] + r) * ld + m.off_conv + c] : carried(j, c, -r), acc);
            }
        }
        return silu_mem(acc);
    };
    auto carry = [&](int j, int c, const float (&raw)[ROWS]) {
        float* out = carry_slot(j);
        const int r0 = t0 + j - start[j];
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int x = 0; x < KEEP; ++x) {
                const int r = r0 - KEEP + 1 + x;
                out[(int64_t)x * C + c] = r >= 0 ? raw[j + 1 + x] : carried(j, c, -r);
            }
        } else {
            for (int x = 0; x < keep; ++x) {
                const int r = r0 - keep + 1 + x;
                out[(int64_t)x * C + c] = r >= 0 ? proj[(int64_t)(start[j] + r) * ld + m.off_conv + c] : carried(j, c, -r);
            }
        }
    };
    auto weights = [&](int c, float (&w)[TAPS > 0 ? TAPS : 1]) -> float {
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int x = 0; x < TAPS; ++x) w[x] = m.conv_w[(int64_t)c * TAPS + x];
        }
        return m.conv_b != nullptr ? m.conv_b[c] : 0.f;
    };
    if (task < G) {
        // the head's query, then its key: convolved values of the whole tile in registers, then the norms and the dot product
        float y[2][TT][NC];
#pragma unroll
        for (int v = 0; v < 2; ++v) {
            const int c0 = (v == 0 ? m.off_q : m.off_k) + task * D;
#pragma unroll
            for (int i = 0; i < NC; ++i) {
                const int d = lane + 32 * i, c = c0 + d;
#pragma unroll
                for (int j = 0; j < TT; ++j) y[v][j][i] = 0.f;
                if (d >= D) continue;
                float raw[ROWS], w[TAPS > 0 ? TAPS : 1];
                fetch(c, raw);
                const float bias = weights(c, w);
#pragma unroll
                for (int j = 0; j < TT; ++j) {
                    if (j >= nt) break;
                    y[v][j][i] = conv(j, c, raw, w, bias);
                    if (last[j]) carry(j, c, raw);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < TT; ++j) {
            if (j >= nt) break;
            float fq = 1.f, fk = 1.f, dot = 0.f;
            if (m.unit) {
                float qq = 0.f, kk = 0.f;
#pragma unroll
                for (int i = 0; i < NC; ++i) { qq = fmaf(y[0][j][i], y[0][j][i], qq); kk = fmaf(y[1][j][i], y[1][j][i], kk); }
                fq = 1.f / sqrtf(warp_sum_mem(qq) + 1e-6f) * (1.f / sqrtf((float)D));
                fk = 1.f / sqrtf(warp_sum_mem(kk) + 1e-6f);
            }
            float* out = qkv + (int64_t)(t0 + j) * ld_qkv;
#pragma unroll
            for (int i = 0; i < NC; ++i) {
                const int d = lane + 32 * i;
                const float q = y[0][j][i] * fq, k = y[1][j][i] * fk;
                dot = fmaf(q, k, dot);
                if (d < D) { out[m.off_q + task * D + d] = q; out[m.off_k + task * D + d] = k; }
            }
            dot = warp_sum_mem(dot);
            if (lane == 0) kq[(int64_t)(t0 + j) * G + task] = dot;
        }
    } else {
        const int c0 = (task - G) * 32 * kPrepVals;
#pragma unroll
        for (int i = 0; i < kPrepVals; ++i) {
            const int e = c0 + lane + 32 * i, c = m.off_v + e;
            if (e >= cv) continue;
            float raw[ROWS], w[TAPS > 0 ? TAPS : 1];
            fetch(c, raw);
            const float bias = weights(c, w);
#pragma unroll
            for (int j = 0; j < TT; ++j) {
                if (j >= nt) break;
                qkv[(int64_t)(t0 + j) * ld_qkv + c] = conv(j, c, raw, w, bias);
                if (last[j]) carry(j, c, raw);
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------ recurrence
constexpr int kMemWarps = 4, kMemStages = 3;

__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src));
}

// Two fp32 numbers in one 64-bit register and the packed multiply-add on them (each half rounds as its scalar form does).
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float a, float b) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// RL lanes share a value column and hold RPL of its rows each (rows 4 (r + RL i) .. + 3 of lane r, so that the 16-byte loads
// of the lanes that share a column are consecutive); a lane holds CPL columns.  The whole state slice stays in registers for
// the step.  Tokens run in order; TB at a time are staged (q, k, the block's value columns, decay, strength, k . q) in a ring
// of shared-memory stages filled by asynchronous copies.  Both products with the state use the state in front of the
// token's write, S^T q after it being decay (S^T q) + (k . q) u, so one pass over the rows and one round of shuffles serve
// the write and the read-out.  The order of every addition is fixed by the layout: a token's result does not depend on how
// the sequence was cut into steps.
template <int RL, int RPL, int CPL, int TB, bool DELTA>
__global__ void __launch_bounds__(32 * kMemWarps) memory_kernel(const float* __restrict__ qkv, int64_t ld, const float* __restrict__ gates,
                                                                const float* __restrict__ kq, umbs_memory_t m, Batch b,
                                                                float* __restrict__ o, int vec) {
    constexpr int DP = RL * RPL, WC = 32 / RL * CPL, CT = kMemWarps * WC;         // padded rows; columns per warp and per block
    constexpr int STAGE = TB * (2 * DP + CT + 4);
    extern __shared__ __align__(16) float mem_sm[];
    float* so = mem_sm + kMemStages * STAGE;                                       // [TB][CT]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rl = lane % RL, cl = lane / RL;
    const int h = blockIdx.y, s = blockIdx.z, c0 = blockIdx.x * CT, D = m.dim, V = m.vdim;
    const int grp = h / (m.heads / m.kv_heads);
    const int start = b.seq_start[s], len = b.seq_len[s], pos0 = b.seq_pos0[s], slot = b.seq_slot[s];
    const int cq = m.off_q + grp * D, ck = m.off_k + grp * D, cv = m.off_v + h * V + c0;
    const int hv = m.heads * V, ncol = min(CT, V - c0);
    const float skip = m.skip != nullptr ? m.skip[h] : 0.f;
    float* st = m.state + ((int64_t)slot * m.heads + h) * V * D;                   // S[column][row]
    f32x2 S[CPL][RPL / 2];                                                         // neighbouring rows in pairs
    int col[CPL];
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
        col[c] = warp * WC + c * (32 / RL) + cl;
        const float* sc = st + (int64_t)(c0 + col[c]) * D;
        const bool have = pos0 > 0 && col[c] < ncol;
#pragma unroll
        for (int i = 0; i < RPL / 4; ++i) {
            const int r = 4 * (rl + RL * i);
            float f[4];
            if (have && D % 4 == 0) {
                *reinterpret_cast<float4*>(f) = r < D ? *reinterpret_cast<const float4*>(sc + r) : make_float4(0.f, 0.f, 0.f, 0.f);
            } else {
#pragma unroll
                for (int x = 0; x < 4; ++x) f[x] = (have && r + x < D) ? sc[r + x] : 0.f;
            }
            S[c][2 * i] = pack2(f[0], f[1]);
            S[c][2 * i + 1] = pack2(f[2], f[3]);
        }
    }
    // rows beyond dim and columns beyond vdim of every stage stay zero
    if (D < DP || ncol < CT) {
        for (int i = tid; i < kMemStages * STAGE; i += 32 * kMemWarps) mem_sm[i] = 0.f;
        __syncthreads();
    }
    constexpr int NT = 32 * kMemWarps, P4 = DP / 4, C4 = CT / 4;
    auto issue = [&](int g) {
        float* sq = mem_sm + (g % kMemStages) * STAGE;
        float* sk = sq + TB * DP;
        float* sv = sk + TB * DP;
        float* sg = sv + TB * CT;                                                  // [TB][4] decay, strength, k . q
        const int t0 = g * TB, nt = min(TB, len - t0);
        const float* base = qkv + (int64_t)(start + t0) * ld;
        if (vec) {
#pragma unroll
            for (int i = tid; i < TB * P4; i += NT) {
                const int tt = i / P4, d = (i % P4) * 4;
                if (tt < nt && d < D) {
                    cp_async16(sq + tt * DP + d, base + (int64_t)tt * ld + cq + d);
                    cp_async16(sk + tt * DP + d, base + (int64_t)tt * ld + ck + d);
                }
            }
            for (int i = tid; i < TB * C4; i += NT) {
                const int tt = i / C4, d = (i % C4) * 4;
                if (tt < nt && d < ncol) cp_async16(sv + tt * CT + d, base + (int64_t)tt * ld + cv + d);
            }
        } else {
            for (int i = tid; i < TB * DP; i += NT) {
                const int tt = i / DP, d = i % DP;
                if (tt < nt && d < D) {
                    cp_async4(sq + tt * DP + d, base + (int64_t)tt * ld + cq + d);
                    cp_async4(sk + tt * DP + d, base + (int64_t)tt * ld + ck + d);
                }
            }
            for (int i = tid; i < TB * CT; i += NT) {
                const int tt = i / CT, d = i % CT;
                if (tt < nt && d < ncol) cp_async4(sv + tt * CT + d, base + (int64_t)tt * ld + cv + d);
            }
        }
        if (tid < nt) {
            const int64_t t = start + t0 + tid;
            cp_async4(sg + 4 * tid, gates + (t * m.heads + h) * 2);
            cp_async4(sg + 4 * tid + 1, gates + (t * m.heads + h) * 2 + 1);
            cp_async4(sg + 4 * tid + 2, kq + t * m.kv_heads + grp);
        }
    };
    const int groups = (len + TB - 1) / TB;
    for (int g = 0; g < kMemStages - 1; ++g) {
        if (g < groups) issue(g);
        asm volatile("cp.async.commit_group;\n" ::);
    }
    for (int g = 0; g < groups; ++g) {
        // (the stage this writes was walked in the previous iteration, which ended with a barrier)
        if (g + kMemStages - 1 < groups) issue(g + kMemStages - 1);
        asm volatile("cp.async.commit_group;\n" ::);
        asm volatile("cp.async.wait_group %0;\n" ::"n"(kMemStages - 1));           // this thread's copies of group g have landed
        float* sq = mem_sm + (g % kMemStages) * STAGE;
        float* sk = sq + TB * DP;
        float* sv = sk + TB * DP;
        float* sg = sv + TB * CT;
        const int t0 = g * TB, nt = min(TB, len - t0);
        if (tid < nt) sg[4 * tid] = expf(sg[4 * tid]);                             // (the thread that copied it)
        __syncthreads();
        // the operands of a token are in registers before the token in front of it is worked on
        struct Operands { f32x2 k[RPL / 2], q[RPL / 2]; float v[CPL]; float4 g; } op[2];
        auto load = [&](Operands& x, int tt) {
            x.g = *reinterpret_cast<const float4*>(sg + 4 * tt);
#pragma unroll
            for (int i = 0; i < RPL / 4; ++i) {
                const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(sk + tt * DP + 4 * (rl + RL * i));
                const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(sq + tt * DP + 4 * (rl + RL * i));
                x.k[2 * i] = k4.x; x.k[2 * i + 1] = k4.y;
                x.q[2 * i] = q4.x; x.q[2 * i + 1] = q4.y;
            }
#pragma unroll
            for (int c = 0; c < CPL; ++c) x.v[c] = sv[tt * CT + col[c]];
        };
        auto walk = [&](const Operands& x, int tt) {
            const float dec = x.g.x, str = x.g.y, dot = x.g.z;
            const f32x2 dec2 = pack2(dec, dec);
            float dq[CPL], dk[CPL];
#pragma unroll
            for (int c = 0; c < CPL; ++c) {
                f32x2 aq[2] = {0ull, 0ull}, ak[2] = {0ull, 0ull};
#pragma unroll
                for (int i = 0; i < RPL / 2; ++i) {
                    if (DELTA) ak[i & 1] = fma2(S[c][i], x.k[i], ak[i & 1]);
                    aq[i & 1] = fma2(S[c][i], x.q[i], aq[i & 1]);
                }
                const float2 q0 = unpack2(aq[0]), q1 = unpack2(aq[1]), k0 = unpack2(ak[0]), k1 = unpack2(ak[1]);
                dq[c] = (q0.x + q0.y) + (q1.x + q1.y);
                dk[c] = (k0.x + k0.y) + (k1.x + k1.y);
            }
#pragma unroll
            for (int w = RL / 2; w > 0; w >>= 1)
#pragma unroll
                for (int c = 0; c < CPL; ++c) {
                    if (DELTA) dk[c] += __shfl_xor_sync(0xffffffffu, dk[c], w);
                    dq[c] += __shfl_xor_sync(0xffffffffu, dq[c], w);
                }
#pragma unroll
            for (int c = 0; c < CPL; ++c) {
                const float u = DELTA ? str * fmaf(-dec, dk[c], x.v[c]) : str * x.v[c];
                const f32x2 u2 = pack2(u, u);
#pragma unroll
                for (int i = 0; i < RPL / 2; ++i) S[c][i] = fma2(dec2, S[c][i], mul2(x.k[i], u2));
                if (rl == 0) so[tt * CT + col[c]] = fmaf(skip, x.v[c], fmaf(dot, u, dec * dq[c]));
            }
        };
        load(op[0], 0);
        for (int tt = 0; tt < nt; tt += 2) {
            load(op[1], tt + 1);                                                   // (TB is even: a place of the stage)
            walk(op[0], tt);
            if (tt + 1 >= nt) break;
            load(op[0], min(tt + 2, TB - 1));
            walk(op[1], tt + 1);
        }
        __syncthreads();
        for (int i = tid; i < nt * CT; i += NT) {
            const int tt = i / CT, c = i % CT;
            if (c < ncol) o[(int64_t)(start + t0 + tt) * hv + h * V + c0 + c] = so[i];
        }
    }
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
        if (col[c] >= ncol) continue;
        float* sc = st + (int64_t)(c0 + col[c]) * D;
#pragma unroll
        for (int i = 0; i < RPL / 4; ++i) {
            const int r = 4 * (rl + RL * i);
            const float2 lo = unpack2(S[c][2 * i]), hi = unpack2(S[c][2 * i + 1]);
            const float f[4] = {lo.x, lo.y, hi.x, hi.y};
            if (D % 4 == 0) {
                if (r < D) *reinterpret_cast<float4*>(sc + r) = make_float4(f[0], f[1], f[2], f[3]);
            } else {
#pragma unroll
                for (int x = 0; x < 4; ++x)
                    if (r + x < D) sc[r + x] = f[x];
            }
        }
    }
}

template <int RL, int RPL, int CPL, int TB, bool DELTA>
static int launch_memory(const float* qkv, int64_t ld, const float* gates, const float* kq, const umbs_memory_t& m, const Batch& b, float* o,
                         int vec, cudaStream_t st) {
    constexpr int CT = kMemWarps * (32 / RL * CPL);
    constexpr size_t smem = ((size_t)kMemStages * TB * (2 * RL * RPL + CT + 4) + (size_t)TB * CT) * sizeof(float);
    static bool set = false;
    if (smem > 48 * 1024 && !set) {
        cudaError_t e = cudaFuncSetAttribute(memory_kernel<RL, RPL, CPL, TB, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        set = true;
    }
    const dim3 grid((m.vdim + CT - 1) / CT, m.heads, b.n_seqs);
    memory_kernel<RL, RPL, CPL, TB, DELTA><<<grid, 32 * kMemWarps, smem, st>>>(qkv, ld, gates, kq, m, b, o, vec);
    return 0;
}

// ------------------------------------------------------------------------------------------------ gated norm
__device__ __forceinline__ float gate_mem(float z, int act) { return act == UMBS_GATE_SIGMOID ? 1.f / (1.f + expf(-z)) : silu_mem(z); }
// A warp (or, for long parts, a block) per part of a row.
template <typename T>
__global__ void gated_norm_kernel(const float* __restrict__ o, const float* __restrict__ gate, int64_t ldg, int n_parts, int width, int parts,
                                  const float* __restrict__ w, int w_len, int gate_first, int gate_act, float eps, int whole_block, T* __restrict__ out) {
    __shared__ float red[32];
    const int nw = blockDim.x >> 5, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int p = whole_block ? blockIdx.x : blockIdx.x * nw + warp;
    const int me = whole_block ? threadIdx.x : lane, step = whole_block ? blockDim.x : 32;
    if (p >= n_parts) return;                       // (never a part of a block that meets the barrier below)
    const int t = p / parts, size = width / parts, e0 = (p - t * parts) * size;
    const float* orow = o + (int64_t)t * width + e0;
    const float* grow = gate + (int64_t)t * ldg + e0;
    float ss = 0.f;
    for (int e = me; e < size; e += step) {
        const float y = gate_first ? orow[e] * gate_mem(grow[e], gate_act) : orow[e];
        ss = fmaf(y, y, ss);
    }
    ss = warp_sum_mem(ss);
    if (whole_block) {
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        ss = warp_sum_mem(lane < nw ? red[lane] : 0.f);
    }
    const float inv = 1.f / sqrtf(ss / (float)size + eps);
    for (int e = me; e < size; e += step)
        out[(int64_t)t * width + e0 + e] = from_f32<T>(orow[e] * gate_mem(grow[e], gate_act) * inv * w[(e0 + e) % w_len]);
}

// The same in 16-byte pieces, a part's values held in registers (KEEP4 pieces per lane of the warp, or per thread of the block, that a
// part has).
template <typename T, int KEEP4>
__global__ void gated_norm_vec_kernel(const float* __restrict__ o, const float* __restrict__ gate, int64_t ldg, int n_parts, int width, int parts,
                                      const float* __restrict__ w, int w_len, int gate_first, int gate_act, float eps, int whole_block, T* __restrict__ out) {
    __shared__ float red[32];
    const int nw = blockDim.x >> 5, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int p = whole_block ? blockIdx.x : blockIdx.x * nw + warp;
    const int me = whole_block ? threadIdx.x : lane, step = whole_block ? blockDim.x : 32;
    if (p >= n_parts) return;                       // (never a part of a block that meets the barrier below)
    const int t = p / parts, size = width / parts, e0 = (p - t * parts) * size, n4 = size / 4;
    const float4* orow = reinterpret_cast<const float4*>(o + (int64_t)t * width + e0);
    const float4* grow = reinterpret_cast<const float4*>(gate + (int64_t)t * ldg + e0);
    float4 y[KEEP4], g[KEEP4];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP4; ++i) {
        const int e = me + i * step;
        y[i] = g[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (e < n4) { y[i] = orow[e]; g[i] = grow[e]; }
    }
#pragma unroll
    for (int i = 0; i < KEEP4; ++i) {
        g[i] = make_float4(gate_mem(g[i].x, gate_act), gate_mem(g[i].y, gate_act), gate_mem(g[i].z, gate_act), gate_mem(g[i].w, gate_act));
        const float4 v = make_float4(y[i].x * g[i].x, y[i].y * g[i].y, y[i].z * g[i].z, y[i].w * g[i].w);
        const float4 q = gate_first ? v : y[i];
        ss = fmaf(q.x, q.x, fmaf(q.y, q.y, fmaf(q.z, q.z, fmaf(q.w, q.w, ss))));
        y[i] = v;
    }
    ss = warp_sum_mem(ss);
    if (whole_block) {
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        ss = warp_sum_mem(lane < nw ? red[lane] : 0.f);
    }
    const float inv = 1.f / sqrtf(ss / (float)size + eps);
#pragma unroll
    for (int i = 0; i < KEEP4; ++i) {
        const int e = me + i * step;
        if (e >= n4) continue;
        const float4 ww = *reinterpret_cast<const float4*>(w + (e0 + 4 * e) % w_len);
        T* dst = out + (int64_t)t * width + e0 + 4 * e;
        const float r[4] = {y[i].x * inv * ww.x, y[i].y * inv * ww.y, y[i].z * inv * ww.z, y[i].w * inv * ww.w};
        if constexpr (sizeof(T) == 4) {
            *reinterpret_cast<float4*>(dst) = make_float4(r[0], r[1], r[2], r[3]);
        } else {
            __nv_bfloat162 a = __floats2bfloat162_rn(r[0], r[1]), b = __floats2bfloat162_rn(r[2], r[3]);
            *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
        }
    }
}

template <typename T>
static void launch_gated_norm(const float* o, const float* gate, int64_t ldg, int n, int width, int parts, const float* w, int w_len,
                              int gate_first, int gate_act, float eps, T* out, cudaStream_t st) {
    const int size = width / parts, n_parts = n * parts;
    const uintptr_t ptrs = (uintptr_t)o | (uintptr_t)gate | (uintptr_t)w | (uintptr_t)out;
    if (size % 4 == 0 && ldg % 4 == 0 && w_len % 4 == 0 && ptrs % 16 == 0 && size <= 16384) {
        const int block = size > 512, threads = block ? ((size / 4 + 3) / 4 + 31) / 32 * 32 : 128;
        const unsigned grid = block ? n_parts : (n_parts + 3) / 4;
        if (size <= 128) gated_norm_vec_kernel<T, 1><<<grid, threads, 0, st>>>(o, gate, ldg, n_parts, width, parts, w, w_len, gate_first, gate_act, eps, block, out);
        else if (size <= 256) gated_norm_vec_kernel<T, 2><<<grid, threads, 0, st>>>(o, gate, ldg, n_parts, width, parts, w, w_len, gate_first, gate_act, eps, block, out);
        else gated_norm_vec_kernel<T, 4><<<grid, threads, 0, st>>>(o, gate, ldg, n_parts, width, parts, w, w_len, gate_first, gate_act, eps, block, out);
    } else {
        const int block = size > 256, threads = block ? (size >= 2048 ? 512 : 256) : 128;
        gated_norm_kernel<T><<<block ? n_parts : (n_parts + 3) / 4, threads, 0, st>>>(o, gate, ldg, n_parts, width, parts, w, w_len,
                                                                                     gate_first, gate_act, eps, block, out);
    }
}

}  // namespace umbs

using namespace umbs;

static int check_memory(const umbs_memory_t* m) {
    if (m == nullptr || m->heads < 1 || m->kv_heads < 1 || m->heads % m->kv_heads != 0 || m->dim < 1 || m->vdim < 1) return UMB_ERR_ARG;
    if (m->rule != UMBS_MEMORY_ADD && m->rule != UMBS_MEMORY_DELTA) return UMB_ERR_ARG;
    return m->dim > 512 ? UMB_ERR_UNSUPPORTED : 0;
}

extern "C" int umbs_memory_prep(const float* proj, int64_t ld, const umbs_memory_t* m, const umbs_batch_t* batch, int slots, float* qkv,
                                int64_t ld_qkv, float* gates, float* kq, umbs_stream_t stream) {
    if (batch->n_tokens <= 0) return 0;
    const int rc = check_memory(m);
    if (rc) return rc;
    if (proj == nullptr || qkv == nullptr || gates == nullptr || kq == nullptr || m->taps < 1 || m->conv_w == nullptr ||
        m->decay_rate == nullptr || m->dt_bias == nullptr || (m->taps > 1 && m->conv_state == nullptr))
        return UMB_ERR_ARG;
    cudaStream_t st = (cudaStream_t)stream;
    const int tasks = m->kv_heads + (m->heads * m->vdim + 32 * kPrepVals - 1) / (32 * kPrepVals) + 1;
    // a long step: tiles of consecutive tokens, as long as the registers of a head's size allow
    const bool wide = batch->n_tokens > 256 && m->taps == 4;
    const int nc = m->dim <= 64 ? 2 : (m->dim <= 128 ? 4 : (m->dim <= 256 ? 8 : 16)), tile = wide ? 16 / nc : 1;
    const dim3 grid((batch->n_tokens + tile - 1) / tile, (tasks + kPrepWarps - 1) / kPrepWarps);
#define UMBS_PREP(NC, TAPS, TT) memory_prep_kernel<NC, TAPS, TT><<<grid, 32 * kPrepWarps, 0, st>>>(proj, ld, *m, *batch, slots, qkv, ld_qkv, gates, kq)
#define UMBS_PREP_NC(NC)                              \
    do {                                              \
        if (wide) UMBS_PREP(NC, 4, 16 / NC);          \
        else if (m->taps == 4) UMBS_PREP(NC, 4, 1);   \
        else UMBS_PREP(NC, 0, 1);                     \
    } while (0)
    if (nc == 2) UMBS_PREP_NC(2);
    else if (nc == 4) UMBS_PREP_NC(4);
    else if (nc == 8) UMBS_PREP_NC(8);
    else UMBS_PREP_NC(16);
#undef UMBS_PREP_NC
#undef UMBS_PREP
    count_launches(1);
    return (int)cudaGetLastError();
}

extern "C" int umbs_memory_run(const float* qkv, int64_t ld_qkv, const float* gates, const float* kq, const umbs_memory_t* m,
                               const umbs_batch_t* batch, float* o, umbs_stream_t stream) {
    if (batch->n_tokens <= 0) return 0;
    const int rc0 = check_memory(m);
    if (rc0) return rc0;
    if (qkv == nullptr || gates == nullptr || kq == nullptr || o == nullptr || m->state == nullptr) return UMB_ERR_ARG;
    cudaStream_t st = (cudaStream_t)stream;
    // 16-byte copies: every row, head and column tile must start on a 16-byte boundary
    const int vec = m->dim % 4 == 0 && m->vdim % 4 == 0 && ld_qkv % 4 == 0 && m->off_q % 4 == 0 && m->off_k % 4 == 0 && m->off_v % 4 == 0 &&
                    (uintptr_t)qkv % 16 == 0;
#define UMBS_MEM(RL, RPL, CPL, TB)                                                                                                     \
    (m->rule == UMBS_MEMORY_DELTA ? launch_memory<RL, RPL, CPL, TB, true>(qkv, ld_qkv, gates, kq, *m, *batch, o, vec, st)            \
                                  : launch_memory<RL, RPL, CPL, TB, false>(qkv, ld_qkv, gates, kq, *m, *batch, o, vec, st))
    // few blocks (one long prompt): a column per lane, the shortest walk; many: two, so that a staged q and k serve both (the same
    // additions in the same order either way)
    const bool many = (int64_t)((m->vdim + 15) / 16) * m->heads * batch->n_seqs >= 4 * 148;
    // decoding: nothing to stage ahead, small blocks of shared memory
    const bool one = batch->max_seq_len == 1;
    int rc;
    if (one && m->dim <= 32) rc = UMBS_MEM(8, 4, 1, 2);
    else if (one && m->dim <= 64) rc = UMBS_MEM(8, 8, 1, 2);
    else if (one && m->dim <= 128) rc = UMBS_MEM(8, 16, 1, 2);
    else if (one && m->dim <= 256) rc = UMBS_MEM(8, 32, 1, 2);
    else if (m->dim <= 32) rc = many ? UMBS_MEM(8, 4, 2, 16) : UMBS_MEM(8, 4, 1, 16);
    else if (m->dim <= 64) rc = many ? UMBS_MEM(8, 8, 2, 16) : UMBS_MEM(8, 8, 1, 16);
    else if (m->dim <= 128) rc = many ? UMBS_MEM(8, 16, 2, 16) : UMBS_MEM(8, 16, 1, 16);
    else if (m->dim <= 256) rc = UMBS_MEM(8, 32, 1, 8);
    else rc = UMBS_MEM(16, 32, 1, 8);
#undef UMBS_MEM
    if (rc) return rc;
    count_launches(1);
    return (int)cudaGetLastError();
}

extern "C" int umbs_gated_norm(int dtype, const float* o, const float* gate, int64_t ldg, int n, int width, int parts, const float* w,
                               int w_len, int gate_first, float eps, void* out, umbs_stream_t stream) {
    return umbs_gated_norm_ex(dtype, o, gate, ldg, n, width, parts, w, w_len, gate_first, UMBS_GATE_SILU, eps, out, stream);
}

extern "C" int umbs_gated_norm_ex(int dtype, const float* o, const float* gate, int64_t ldg, int n, int width, int parts, const float* w,
                                  int w_len, int gate_first, int gate_act, float eps, void* out, umbs_stream_t stream) {
    if (n <= 0) return 0;
    if (gate_act != UMBS_GATE_SILU && gate_act != UMBS_GATE_SIGMOID) return UMB_ERR_ARG;
    if (o == nullptr || gate == nullptr || w == nullptr || out == nullptr || parts < 1 || width % parts != 0 || w_len < 1) return UMB_ERR_ARG;
    cudaStream_t st = (cudaStream_t)stream;
    if (dtype == UMBS_BF16) launch_gated_norm(o, gate, ldg, n, width, parts, w, w_len, gate_first, gate_act, eps, (__nv_bfloat16*)out, st);
    else if (dtype == UMBS_F32) launch_gated_norm(o, gate, ldg, n, width, parts, w, w_len, gate_first, gate_act, eps, (float*)out, st);
    else return UMB_ERR_ARG;
    count_launches(1);
    return (int)cudaGetLastError();
}
