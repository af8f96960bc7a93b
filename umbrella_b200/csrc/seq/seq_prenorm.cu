// Kernels of the pre-norm layer form (see include/umbrella_b200_seq.h): residual add fused with the RMS norm that
// follows it, the logit soft cap, and what stands between an attention layer's in-projection and its attention kernel:
// bias, short causal convolution with its carried rows, rotary positions, the step's key/value rows in the cache's
// layout, and the mean key/value of every block of tokens a step completes.  fp32 arithmetic throughout.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <algorithm>
#include <stdint.h>

#include "seq_internal.h"

namespace umbs {

__device__ __forceinline__ float warp_sum_pn(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// One block per row.  The row is read once into registers (up to 8 values per thread, more are re-read), its sum of
// squares reduced in a fixed tree (warp shuffles, then warp 0 over the per-warp partials): the result does not depend on
// what else is in the step.
template <typename T>
__global__ void add_rms_norm_kernel(float* __restrict__ x, const float* __restrict__ delta, const int32_t* __restrict__ rows,
                                    const float* __restrict__ w, float w_offset, int width, float eps, T* __restrict__ y,
                                    float* __restrict__ copy) {
    __shared__ float red[33];
    const int r = blockIdx.x;
    const int64_t src = rows ? rows[r] : r;
    float* xr = x + src * width;
    const float* dr = delta ? delta + src * width : nullptr;
    constexpr int KEEP = 8;
    float v[KEEP];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int e = threadIdx.x + i * blockDim.x;
        v[i] = 0.f;
        if (e < width) {
            v[i] = xr[e] + (dr ? dr[e] : 0.f);
            ss = fmaf(v[i], v[i], ss);
        }
    }
    for (int e = threadIdx.x + KEEP * blockDim.x; e < width; e += blockDim.x) {
        const float u = xr[e] + (dr ? dr[e] : 0.f);
        ss = fmaf(u, u, ss);
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    ss = warp_sum_pn(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    if (warp == 0) {
        float s = lane < nw ? red[lane] : 0.f;
        s = warp_sum_pn(s);
        if (lane == 0) red[32] = s;
    }
    __syncthreads();
    const float inv = 1.f / sqrtf(red[32] / (float)width + eps);
    const bool write_x = rows == nullptr && dr != nullptr;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int e = threadIdx.x + i * blockDim.x;
        if (e < width) {
            if (write_x) xr[e] = v[i];
            if (copy != nullptr) copy[(int64_t)r * width + e] = v[i];
            if (y != nullptr) y[(int64_t)r * width + e] = from_f32<T>(v[i] * inv * (w_offset + w[e]));
        }
    }
    for (int e = threadIdx.x + KEEP * blockDim.x; e < width; e += blockDim.x) {
        const float u = xr[e] + (dr ? dr[e] : 0.f);
        if (write_x) xr[e] = u;
        if (copy != nullptr) copy[(int64_t)r * width + e] = u;
        if (y != nullptr) y[(int64_t)r * width + e] = from_f32<T>(u * inv * (w_offset + w[e]));
    }
}

// Residual add + norm for any pending block output (dense, routed experts' pairs, gated shared expert; layer scale and
// residual multiplier) and either norm.  One block per row, the row in registers (8 values per thread); sums in a fixed
// tree, so a row's result does not depend on what else is in the step.  The layer norm takes its mean first and the mean
// of the squared deviations second.
__device__ __forceinline__ float block_sum_pn(float v, float* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    v = warp_sum_pn(v);
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float s = lane < nw ? red[lane] : 0.f;
        s = warp_sum_pn(s);
        if (lane == 0) red[32] = s;
    }
    __syncthreads();
    return red[32];
}

constexpr int kNormNone = -1;          // y gets the row as it is (umbs_add_rows)

template <typename T>
__global__ void add_norm_kernel(float* __restrict__ x, umbs_delta_t d, int has_d, const int32_t* __restrict__ rows, int kind,
                                const float* __restrict__ w, const float* __restrict__ bias, float w_offset, float alpha, int width,
                                float eps, T* __restrict__ y, int64_t ldy, float* __restrict__ copy) {
    __shared__ float red[33];
    constexpr int KEEP = 8, TOPS = 16;              // up to TOPS routed pairs per token are held in shared memory
    __shared__ float s_w[TOPS];
    __shared__ const float* s_p[TOPS];
    const int r = blockIdx.x;
    const int64_t src = rows ? rows[r] : r;
    float* xr = x + src * width;
    float v[KEEP];
    const float sg = (has_d && d.shared != nullptr && d.shared_gate != nullptr) ? d.shared_gate[src] : 1.f;
    const bool routed = has_d && d.pair_out != nullptr;
    const int top_s = routed ? min(d.top, TOPS) : 0;
    if (threadIdx.x < top_s) {                      // the token's weights and the rows of its experts' outputs, read once
        s_w[threadIdx.x] = d.sel_w[src * d.top + threadIdx.x];
        s_p[threadIdx.x] = d.pair_out + (int64_t)d.pair_pos[src * d.top + threadIdx.x] * width;
    }
    if (routed) __syncthreads();
    // the routed experts' rows first, expert by expert: the thread's eight loads of a row are in flight together
    float ff[KEEP];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) ff[i] = 0.f;
    for (int k = 0; routed && k < d.top; ++k) {
        const float wk = k < top_s ? s_w[k] : d.sel_w[src * d.top + k];
        const float* pk = k < top_s ? s_p[k] : d.pair_out + (int64_t)d.pair_pos[src * d.top + k] * width;
#pragma unroll
        for (int i = 0; i < KEEP; ++i) {
            const int e = threadIdx.x + i * blockDim.x;
            if (e < width) ff[i] = fmaf(wk, pk[e], ff[i]);
        }
    }
    float sum = 0.f, dsum = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int e = threadIdx.x + i * blockDim.x;
        float dl = 0.f;
        if (e < width && has_d) {
            if (d.delta != nullptr) dl = d.delta[src * width + e] * d.delta_mult;
            if (d.delta2 != nullptr) dl = fmaf(d.delta2[src * width + e], d.delta2_mult, dl);
            dl += ff[i];
            if (d.shared != nullptr) dl = fmaf(d.shared[src * width + e], sg, dl);
        }
        ff[i] = dl;                                       // the block's whole output
        dsum = fmaf(dl, dl, dsum);
    }
    const bool post = has_d && d.norm_w != nullptr;       // a norm behind the block: its output's own statistics first
    const float dinv = post ? 1.f / sqrtf(block_sum_pn(dsum, red) / (float)width + eps) : 1.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int e = threadIdx.x + i * blockDim.x;
        v[i] = 0.f;
        if (e < width) {
            float dl = ff[i];
            if (post) dl = dl * dinv * d.norm_w[e];
            if (has_d) {
                if (d.scale != nullptr) dl *= d.scale[e];
                dl *= d.mult;
            }
            v[i] = xr[e] + dl;
            sum += kind == UMBS_NORM_LAYER ? v[i] : v[i] * v[i];
        }
    }
    float mean = 0.f, inv = 0.f;
    if (y != nullptr && kind != UMBS_NORM_DYT && kind != kNormNone) {          // (the tanh norm takes no statistics)
        sum = block_sum_pn(sum, red);
        if (kind == UMBS_NORM_LAYER) {
            mean = sum / (float)width;
            float dev = 0.f;
#pragma unroll
            for (int i = 0; i < KEEP; ++i)
                if (threadIdx.x + i * blockDim.x < width) dev = fmaf(v[i] - mean, v[i] - mean, dev);
            sum = block_sum_pn(dev, red);
        }
        inv = 1.f / sqrtf(sum / (float)width + eps);
    }
    const bool write_x = rows == nullptr && has_d;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int e = threadIdx.x + i * blockDim.x;
        if (e < width) {
            if (write_x) xr[e] = v[i];
            if (copy != nullptr) copy[(int64_t)r * width + e] = v[i];
            if (y != nullptr) {
                float o = v[i];
                if (kind != kNormNone) {
                    o = kind == UMBS_NORM_DYT ? tanhf(alpha * v[i]) * (w_offset + w[e]) : (v[i] - mean) * inv * (w_offset + w[e]);
                    if (kind != UMBS_NORM_RMS && bias != nullptr) o += bias[e];
                }
                y[(int64_t)r * ldy + e] = from_f32<T>(o);
            }
        }
    }
}

// The common cases of add_norm_kernel in 16-byte pieces: one dense pending output or the routed experts' rows (TOP > 0: that
// many per token), with or without a norm of its own, times a number, and an RMS norm (or none) of the sum.  KEEP4 pieces per
// thread; the block's sums as fixed trees, one barrier each (every warp adds up the warps' partial sums itself).
__device__ __forceinline__ float block_sum_one_barrier(float v, float* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    v = warp_sum_pn(v);
    if (lane == 0) red[warp] = v;
    __syncthreads();
    return warp_sum_pn(lane < nw ? red[lane] : 0.f);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

template <typename T, int KEEP4, bool ROUTED>
__global__ void add_norm_vec_kernel(float* __restrict__ x, const float* __restrict__ delta, const float* __restrict__ sel_w,
                                    const int32_t* __restrict__ pair_pos, int top, const float* __restrict__ post_w, float mult,
                                    const int32_t* __restrict__ rows, const float* __restrict__ w, float w_offset, int width, float eps,
                                    T* __restrict__ y, int64_t ldy, float* __restrict__ copy) {
    __shared__ float red[2][32];
    const int r = blockIdx.x, n4 = width / 4;
    const int64_t src = rows ? rows[r] : r;
    float4* xr = reinterpret_cast<float4*>(x + src * width);
    float4 v[KEEP4], d[KEEP4];
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP4; ++i) {
        const int e = threadIdx.x + i * blockDim.x;
        v[i] = d[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (e < n4) {
            v[i] = xr[e];
            if (!ROUTED) d[i] = reinterpret_cast<const float4*>(delta + src * width)[e];
        }
    }
    if (ROUTED) {                       // delta: the experts' output rows; the token's rows one after the other, two in flight
#pragma unroll 2
        for (int k = 0; k < top; ++k) {
            const float wk = sel_w[src * top + k];
            const float4* pr = reinterpret_cast<const float4*>(delta + (int64_t)pair_pos[src * top + k] * width);
#pragma unroll
            for (int i = 0; i < KEEP4; ++i) {
                const int e = threadIdx.x + i * blockDim.x;
                if (e < n4) {
                    const float4 p = pr[e];
                    d[i] = make_float4(fmaf(wk, p.x, d[i].x), fmaf(wk, p.y, d[i].y), fmaf(wk, p.z, d[i].z), fmaf(wk, p.w, d[i].w));
                }
            }
        }
    }
    if (post_w != nullptr) {
#pragma unroll
        for (int i = 0; i < KEEP4; ++i)
            sum = fmaf(d[i].x, d[i].x, fmaf(d[i].y, d[i].y, fmaf(d[i].z, d[i].z, fmaf(d[i].w, d[i].w, sum))));
        const float inv = 1.f / sqrtf(block_sum_one_barrier(sum, red[0]) / (float)width + eps);
#pragma unroll
        for (int i = 0; i < KEEP4; ++i) {
            const int e = threadIdx.x + i * blockDim.x;
            if (e < n4) {
                const float4 p = reinterpret_cast<const float4*>(post_w)[e];
                d[i] = make_float4(d[i].x * inv * p.x, d[i].y * inv * p.y, d[i].z * inv * p.z, d[i].w * inv * p.w);
            }
        }
    }
    sum = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP4; ++i) {
        v[i] = make_float4(fmaf(mult, d[i].x, v[i].x), fmaf(mult, d[i].y, v[i].y), fmaf(mult, d[i].z, v[i].z), fmaf(mult, d[i].w, v[i].w));
        sum = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, sum))));
    }
    const float inv = w != nullptr ? 1.f / sqrtf(block_sum_one_barrier(sum, red[1]) / (float)width + eps) : 1.f;
#pragma unroll
    for (int i = 0; i < KEEP4; ++i) {
        const int e = threadIdx.x + i * blockDim.x;
        if (e >= n4) continue;
        if (rows == nullptr) xr[e] = v[i];
        if (copy != nullptr) reinterpret_cast<float4*>(copy + (int64_t)r * width)[e] = v[i];
        if (y != nullptr) {
            float4 o = v[i];
            if (w != nullptr) {
                const float4 g = reinterpret_cast<const float4*>(w)[e];
                o = make_float4(o.x * inv * (w_offset + g.x), o.y * inv * (w_offset + g.y), o.z * inv * (w_offset + g.z), o.w * inv * (w_offset + g.w));
            }
            store4(y + (int64_t)r * ldy + 4 * e, o);
        }
    }
}

template <typename T, bool ROUTED>
static void launch_add_norm_vec(float* x, const umbs_delta_t& d, const int32_t* rows, int n, const float* w, float w_offset, int width,
                                float eps, T* y, int64_t ldy, float* copy, cudaStream_t st) {
    // few rows: spread each over as many threads as there are pieces; many: four pieces per thread
    const int n4 = width / 4, keep = n <= 148 ? (n4 <= 1024 ? 1 : 2) : 4;
    const int threads = ((n4 + keep - 1) / keep + 31) / 32 * 32;
    const float* delta = ROUTED ? d.pair_out : d.delta;
#define UMBS_ANV(K) add_norm_vec_kernel<T, K, ROUTED><<<n, threads, 0, st>>>(x, delta, d.sel_w, d.pair_pos, d.top, d.norm_w, d.mult, rows, w, w_offset, width, eps, y, ldy, copy)
    if (keep == 1) UMBS_ANV(1);
    else if (keep == 2) UMBS_ANV(2);
    else UMBS_ANV(4);
#undef UMBS_ANV
}

// One block per token: the embedding row through an RMS norm, in fp32 and (for a product that reads it) as T.
template <typename T>
__global__ void embedding_norm_kernel(const int32_t* __restrict__ ids, const T* __restrict__ table, float scale, const float* __restrict__ w,
                                      float eps, float* __restrict__ y, T* __restrict__ y2, int64_t ld2, int width) {
    __shared__ float red[33];
    const int t = blockIdx.x;
    const T* row = table + (int64_t)ids[t] * width;
    float ss = 0.f;
    for (int e = threadIdx.x; e < width; e += blockDim.x) {
        const float v = to_f32(row[e]) * scale;
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.f / sqrtf(block_sum_pn(ss, red) / (float)width + eps);
    for (int e = threadIdx.x; e < width; e += blockDim.x) {
        const float v = to_f32(row[e]) * scale * inv * w[e];
        y[(int64_t)t * width + e] = v;
        if (y2 != nullptr) y2[(int64_t)t * ld2 + e] = from_f32<T>(v);
    }
}

// One block per token of a latent-attention layer: RMS norms of the query latent and of the key latent, the turn of the shared key
// part and of every head's rope part by the token's position; each where its source is given.
template <typename T>
__global__ void latent_prep_kernel(umbs_latent_prep_t p, Batch b) {
    extern __shared__ float cs[];                 // cos | sin [rot_dims]
    __shared__ float red[33];
    const int t = blockIdx.x, pos = b.tok_pos[t], half = p.rot_dims / 2, hd = p.dim + p.rope_dim;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float ang = (float)pos * p.inv_freq[i];
        cs[i] = cosf(ang) * p.rot_mag;
        cs[half + i] = sinf(ang) * p.rot_mag;
    }
    // the turn of component j of a rope part that starts at r
    auto turned = [&](const float* r, int j) -> float {
        if (j < half) return r[j] * cs[j] - r[j + half] * cs[half + j];
        if (j < p.rot_dims) return r[j] * cs[j - half] + r[j - half] * cs[j];     // cs[j] = sin of pair j - half
        return r[j];
    };
    __syncthreads();
    if (p.dq != nullptr) {
        const float* row = p.dq + (int64_t)t * p.ld_dq;
        float ss = 0.f;
        for (int e = threadIdx.x; e < p.q_rank; e += blockDim.x) ss = fmaf(row[e], row[e], ss);
        const float inv = 1.f / sqrtf(block_sum_pn(ss, red) / (float)p.q_rank + p.eps);
        T* out = (T*)p.cq + (int64_t)t * p.q_rank;
        for (int e = threadIdx.x; e < p.q_rank; e += blockDim.x) out[e] = from_f32<T>(row[e] * inv * p.q_norm[e]);
    }
    if (p.low != nullptr) {
        const float* low = p.low + (int64_t)t * p.ld_low;
        const int R = p.kv_rank;
        float ss = 0.f;
        for (int e = threadIdx.x; e < R; e += blockDim.x) ss = fmaf(low[e], low[e], ss);
        const float inv = 1.f / sqrtf(block_sum_pn(ss, red) / (float)R + p.eps);
        T* crow = (T*)p.c + (int64_t)t * (R + p.rope_dim);
        for (int e = threadIdx.x; e < R; e += blockDim.x) crow[e] = from_f32<T>(low[e] * inv * p.kv_norm[e]);
        for (int j = threadIdx.x; j < p.rope_dim; j += blockDim.x) crow[R + j] = from_f32<T>(turned(low + R, j));
    }
    if (p.qsrc != nullptr) {
        const float* row = p.qsrc + (int64_t)t * p.ld_q;
        T* qrow = (T*)p.q + (int64_t)t * p.heads * hd;
        for (int i = threadIdx.x; i < p.heads * hd; i += blockDim.x) {
            const int h = i / hd, e = i - h * hd;
            float o = row[i];
            if (e >= p.dim) {
                o = turned(row + (int64_t)h * hd + p.dim, e - p.dim);
                if (p.q_rot != nullptr) p.q_rot[((int64_t)t * p.heads + h) * p.ld_qrot + (e - p.dim)] = o;
            }
            qrow[i] = from_f32<T>(o);
        }
    }
}

__global__ void softcap_kernel(float* __restrict__ z, int64_t n, float cap) {
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) z[i] = cap * tanhf(z[i] / cap);
}

// One block per token.  Channels of q | k go through bias and convolution into shared memory, are turned there, and leave
// as q and as the key part of the token's kv row; values follow (own projection, or the keys before the turn).
template <typename T>
__global__ void attention_prep_kernel(const float* __restrict__ proj, int64_t ld, const float* __restrict__ bias, Batch b,
                                      int heads, int kv_heads, int dim, int vdim, int values_are_keys, int taps,
                                      const float* __restrict__ conv_w, float* __restrict__ conv_state, int slots, int rot_dims,
                                      const float* __restrict__ inv_freq, float rot_mag, int maps,
                                      const float* __restrict__ q_norm_w, const float* __restrict__ k_norm_w, float eps,
                                      umbs_prep_opts_t po, T* __restrict__ q_out, T* __restrict__ kv_out) {
    extern __shared__ float sm[];                 // [heads dim + kv_heads dim] convolved q | k, then cos | sin [rot_dims]
    const int Cq = heads * maps * dim, Ck = kv_heads * maps * dim, C = Cq + Ck, Cv = kv_heads * vdim;
    float* y = sm;
    float* cs = sm + C;
    const int t = blockIdx.x, s = b.tok_seq[t], pos = b.tok_pos[t];
    const int start = b.seq_start[s], len = b.seq_len[s], pos0 = b.seq_pos0[s], slot = b.seq_slot[s], par = b.seq_parity[s];
    const int keep = taps - 1;
    const float* st_in = conv_state ? conv_state + ((int64_t)par * slots + slot) * keep * C : nullptr;
    const float* row = proj + (int64_t)t * ld;
    const int half = rot_dims / 2;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float ang = (float)pos * inv_freq[i];
        cs[i] = cosf(ang) * rot_mag;
        cs[half + i] = sinf(ang) * rot_mag;
    }
    // u(c, p): the projected value (bias added) of channel c at position p -- this step's row, the carried rows, or zero
    auto u_at = [&](int c, int p) -> float {
        if (p >= pos0) return proj[(int64_t)(start + p - pos0) * ld + c] + (bias ? bias[c] : 0.f);
        if (p < 0 || st_in == nullptr) return 0.f;
        return st_in[(int64_t)(p - (pos0 - keep)) * C + c];       // carried row r holds position pos0 - keep + r
    };
    for (int c = threadIdx.x; c < C; c += blockDim.x) {
        float acc;
        if (taps <= 1) {
            acc = row[c] + (bias ? bias[c] : 0.f);
        } else {
            acc = 0.f;
            for (int j = 0; j < taps; ++j) acc = fmaf(conv_w[(int64_t)c * taps + j], u_at(c, pos - keep + j), acc);
        }
        y[c] = acc;
    }
    // the sequence's last token of the step leaves the rows the next step's convolution starts from (other buffer half)
    if (keep > 0 && conv_state != nullptr && t == start + len - 1) {
        float* st_out = conv_state + ((int64_t)(par ^ 1) * slots + slot) * keep * C;
        const int end = pos0 + len;                              // carried row r will hold position end - keep + r
        for (int i = threadIdx.x; i < keep * C; i += blockDim.x) {
            const int r = i / C, c = i - r * C;
            st_out[i] = u_at(c, end - keep + r);
        }
    }
    __syncthreads();
    if (q_norm_w != nullptr || k_norm_w != nullptr) {
        // RMS norm of every (head, map): a warp per group of dim channels, lanes striding over it
        const int lane = threadIdx.x & 31, nw = blockDim.x >> 5;
        for (int grp = threadIdx.x >> 5; grp < C / dim; grp += nw) {
            const float* nwt = grp * dim < Cq ? q_norm_w : k_norm_w;
            if (nwt == nullptr) continue;
            float* yg = y + grp * dim;
            float ss = 0.f;
            for (int d = lane; d < dim; d += 32) ss = fmaf(yg[d], yg[d], ss);
            ss = warp_sum_pn(ss);
            const float inv = 1.f / sqrtf(ss / (float)dim + eps);
            for (int d = lane; d < dim; d += 32) yg[d] = yg[d] * inv * nwt[d];
        }
        __syncthreads();
    }
    if (po.q_norm_all_w != nullptr || po.k_norm_all_w != nullptr) {
        // RMS norm over all of the token's query numbers, and over all of its key numbers
        __shared__ float red[2][33];
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
        float sq = 0.f, sk = 0.f;
        for (int c = threadIdx.x; c < C; c += blockDim.x) {
            const float u = y[c];
            if (c < Cq) sq = fmaf(u, u, sq);
            else sk = fmaf(u, u, sk);
        }
        sq = warp_sum_pn(sq);
        sk = warp_sum_pn(sk);
        if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
        __syncthreads();
        sq = warp_sum_pn(lane < nw ? red[0][lane] : 0.f);
        sk = warp_sum_pn(lane < nw ? red[1][lane] : 0.f);
        const float iq = 1.f / sqrtf(sq / (float)Cq + eps), ik = Ck > 0 ? 1.f / sqrtf(sk / (float)Ck + eps) : 0.f;
        for (int c = threadIdx.x; c < C; c += blockDim.x) {
            if (c < Cq) { if (po.q_norm_all_w != nullptr) y[c] = y[c] * iq * po.q_norm_all_w[c]; }
            else if (po.k_norm_all_w != nullptr) y[c] = y[c] * ik * po.k_norm_all_w[c - Cq];
        }
        __syncthreads();
    }
    const int row_kv = Ck + Cv;
    T* qo = q_out + (int64_t)t * Cq;
    T* ko = kv_out + (int64_t)t * row_kv;
    for (int c = threadIdx.x; c < C; c += blockDim.x) {
        const int d = c % dim;                                   // Cq is a multiple of dim: the same for q and k channels
        float v = y[c];
        if (d < rot_dims) {
            const int f = d < half ? d : d - half;
            const float other = y[d < half ? c + half : c - half];
            v = d < half ? v * cs[f] - other * cs[half + f] : v * cs[f] + other * cs[half + f];
        }
        if (c < Cq) qo[c] = from_f32<T>(v);
        else {
            ko[c - Cq] = from_f32<T>(v);
            if (values_are_keys) ko[Ck + (c - Cq)] = from_f32<T>(y[c]);
        }
    }
    if (!values_are_keys && kv_out != nullptr)
        for (int c = threadIdx.x; c < Cv; c += blockDim.x) {
            float v = row[C + c] + (bias ? bias[C + c] : 0.f);
            if (po.v_mix == UMBS_VMIX_SOURCE) po.v_source[(int64_t)t * Cv + c] = v;
            else if (po.v_mix == UMBS_VMIX_MIX) v = (1.f - po.v_lambda) * v + po.v_lambda * po.v_source[(int64_t)t * Cv + c];
            ko[Ck + c] = from_f32<T>(v);
        }
}

// One block per (block of tokens completed by the step, sequence, 256 columns): the fp32 mean, in position order, of the
// block's kv rows as the cache holds them.  Eight rows are loaded ahead of the additions, which stay in position order.
template <typename T>
__global__ void kv_pool_kernel(const T* __restrict__ kv, const T* __restrict__ kv_cache, int kv_len, T* __restrict__ pool_cache,
                               int pool_len, Batch b, int row, int pool) {
    const int s = blockIdx.y, pos0 = b.seq_pos0[s], len = b.seq_len[s], start = b.seq_start[s], slot = b.seq_slot[s];
    const int blk = pos0 / pool + blockIdx.x;                    // first block whose last token is in the step, onwards
    if ((int64_t)(blk + 1) * pool > (int64_t)pos0 + len || blk >= pool_len) return;
    const int c = blockIdx.z * blockDim.x + threadIdx.x;
    if (c >= row) return;
    auto at = [&](int j) -> float {
        const T* src = j >= pos0 ? kv + (int64_t)(start + j - pos0) * row : kv_cache + ((int64_t)slot * kv_len + j % kv_len) * row;
        return to_f32(src[c]);
    };
    float acc = 0.f;
    const int j0 = blk * pool;
    int j = 0;
    for (; j + 8 <= pool; j += 8) {
        float x[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) x[u] = at(j0 + j + u);
#pragma unroll
        for (int u = 0; u < 8; ++u) acc += x[u];
    }
    for (; j < pool; ++j) acc += at(j0 + j);
    pool_cache[((int64_t)slot * pool_len + blk) * row + c] = from_f32<T>(acc / (float)pool);
}

}  // namespace umbs

using namespace umbs;

#define UMBS_DISPATCH_T(dtype, ...)                              \
    do {                                                         \
        if ((dtype) == UMBS_BF16) { using T = __nv_bfloat16; __VA_ARGS__; } \
        else if ((dtype) == UMBS_F32) { using T = float; __VA_ARGS__; }     \
        else return UMB_ERR_ARG;                                 \
    } while (0)

extern "C" int umbs_add_rms_norm(int dtype, float* x, const float* delta, const int32_t* rows, int n, const float* w,
                                 float w_offset, int width, float eps, void* y, float* copy, umbs_stream_t stream) {
    if (n <= 0) return 0;
    if (x == nullptr || width <= 0 || (y != nullptr && w == nullptr)) return UMB_ERR_ARG;
    cudaStream_t st = (cudaStream_t)stream;
    const int threads = width >= 2048 ? 256 : (width >= 512 ? 128 : 64);
    UMBS_DISPATCH_T(dtype, add_rms_norm_kernel<T><<<n, threads, 0, st>>>(x, delta, rows, w, w_offset, width, eps, (T*)y, copy));
    count_launches(1);
    return (int)cudaGetLastError();
}

extern "C" int umbs_add_norm(int dtype, float* x, const umbs_delta_t* d, const int32_t* rows, int n, int kind, const float* w,
                             const float* b, float w_offset, int width, float eps, void* y, float* copy, umbs_stream_t stream) {
    return umbs_add_norm_ex(dtype, x, d, rows, n, kind, w, b, w_offset, 1.f, width, eps, y, copy, stream);
}

static int add_norm_run(int dtype, float* x, const umbs_delta_t* d, const int32_t* rows, int n, int kind, const float* w,
                        const float* b, float w_offset, float alpha, int width, float eps, void* y, int64_t ldy, float* copy,
                        umbs_stream_t stream) {
    if (width > 8192) return UMB_ERR_UNSUPPORTED;                 // a row lives in the block's registers
    if (d != nullptr && d->pair_out != nullptr && (d->sel_w == nullptr || d->pair_pos == nullptr || d->top < 1)) return UMB_ERR_ARG;
    cudaStream_t st = (cudaStream_t)stream;
    int threads = ((width + 7) / 8 + 31) / 32 * 32;
    if (threads < 64) threads = 64;
    umbs_delta_t dd{};
    if (d != nullptr) dd = *d;
    if (dd.delta_mult == 0.f && dd.delta2 == nullptr) dd.delta_mult = 1.f;
    const uintptr_t ptrs = (uintptr_t)x | (uintptr_t)dd.delta | (uintptr_t)dd.norm_w | (uintptr_t)w | (uintptr_t)copy | (uintptr_t)y;
    const bool vec = d != nullptr && dd.shared == nullptr && dd.delta2 == nullptr && dd.scale == nullptr && dd.delta_mult == 1.f &&
                     (kind == UMBS_NORM_RMS || kind == kNormNone) && width % 4 == 0 && ldy % 4 == 0 && ptrs % 16 == 0;
    const float* vw = kind == kNormNone ? nullptr : w;
    if (vec && dd.delta != nullptr && dd.pair_out == nullptr)
        UMBS_DISPATCH_T(dtype, (launch_add_norm_vec<T, false>(x, dd, rows, n, vw, w_offset, width, eps, (T*)y, ldy, copy, st)));
    else if (vec && dd.delta == nullptr && dd.pair_out != nullptr && (uintptr_t)dd.pair_out % 16 == 0)
        UMBS_DISPATCH_T(dtype, (launch_add_norm_vec<T, true>(x, dd, rows, n, vw, w_offset, width, eps, (T*)y, ldy, copy, st)));
    else
        UMBS_DISPATCH_T(dtype, add_norm_kernel<T><<<n, threads, 0, st>>>(x, dd, d != nullptr, rows, kind, w, b, w_offset, alpha, width,
                                                                         eps, (T*)y, ldy, copy));
    count_launches(1);
    return (int)cudaGetLastError();
}

extern "C" int umbs_add_norm_ex(int dtype, float* x, const umbs_delta_t* d, const int32_t* rows, int n, int kind, const float* w,
                                const float* b, float w_offset, float alpha, int width, float eps, void* y, float* copy,
                                umbs_stream_t stream) {
    if (n <= 0) return 0;
    if (x == nullptr || width <= 0 || (y != nullptr && w == nullptr)) return UMB_ERR_ARG;
    if (kind != UMBS_NORM_RMS && kind != UMBS_NORM_LAYER && kind != UMBS_NORM_DYT) return UMB_ERR_ARG;
    return add_norm_run(dtype, x, d, rows, n, kind, w, b, w_offset, alpha, width, eps, y, width, copy, stream);
}

extern "C" int umbs_add_rows(int dtype, float* x, const umbs_delta_t* d, int n, int width, float eps, void* y, int64_t ldy, float* copy,
                             umbs_stream_t stream) {
    if (n <= 0) return 0;
    if (x == nullptr || width <= 0 || y == nullptr || ldy < width) return UMB_ERR_ARG;
    return add_norm_run(dtype, x, d, nullptr, n, kNormNone, nullptr, nullptr, 0.f, 1.f, width, eps, y, ldy, copy, stream);
}

extern "C" int umbs_embedding_norm(int dtype, const int32_t* ids, const void* table, float scale, const float* w, float eps, float* y,
                                   void* y2, int64_t ld2, int n, int width, umbs_stream_t stream) {
    if (n <= 0) return 0;
    if (ids == nullptr || table == nullptr || w == nullptr || y == nullptr || width <= 0) return UMB_ERR_ARG;
    const int threads = width >= 1024 ? 256 : (width >= 256 ? 128 : 64);
    UMBS_DISPATCH_T(dtype, embedding_norm_kernel<T><<<n, threads, 0, (cudaStream_t)stream>>>(ids, (const T*)table, scale, w, eps, y, (T*)y2,
                                                                                           ld2, width));
    count_launches(1);
    return (int)cudaGetLastError();
}

extern "C" int umbs_latent_prep(int dtype, const float* proj, int64_t ld, const umbs_batch_t* batch, int heads, int dim,
                                int rope_dim, int kv_rank, const float* kv_norm, float eps, int rot_dims, const float* inv_freq,
                                float rot_mag, void* q, void* c, float* q_rot, int64_t ld_qrot, umbs_stream_t stream) {
    if (batch->n_tokens <= 0) return 0;
    if (heads < 1 || dim < 0 || rope_dim < 0 || kv_rank < 1 || rot_dims < 0 || rot_dims > rope_dim || (rot_dims & 1)) return UMB_ERR_ARG;
    if (rot_dims > 0 && inv_freq == nullptr) return UMB_ERR_ARG;
    if (proj == nullptr || kv_norm == nullptr || q == nullptr || c == nullptr) return UMB_ERR_ARG;
    umbs_latent_prep_t p{};
    p.low = proj + (int64_t)heads * (dim + rope_dim); p.ld_low = ld; p.kv_rank = kv_rank; p.kv_norm = kv_norm; p.c = c;
    p.qsrc = proj; p.ld_q = ld; p.heads = heads; p.dim = dim; p.q = q; p.q_rot = q_rot; p.ld_qrot = ld_qrot;
    p.rope_dim = rope_dim; p.rot_dims = rot_dims; p.inv_freq = inv_freq; p.rot_mag = rot_mag; p.eps = eps;
    return umbs_latent_prep_parts(dtype, &p, batch, stream);
}

extern "C" int umbs_latent_prep_parts(int dtype, const umbs_latent_prep_t* p, const umbs_batch_t* batch, umbs_stream_t stream) {
    if (batch->n_tokens <= 0) return 0;
    if (p->rope_dim < 0 || p->rot_dims < 0 || p->rot_dims > p->rope_dim || (p->rot_dims & 1) || (p->rot_dims > 0 && p->inv_freq == nullptr)) return UMB_ERR_ARG;
    if (p->dq == nullptr && p->low == nullptr && p->qsrc == nullptr) return UMB_ERR_ARG;
    if (p->dq != nullptr && (p->q_rank < 1 || p->q_norm == nullptr || p->cq == nullptr)) return UMB_ERR_ARG;
    if (p->low != nullptr && (p->kv_rank < 1 || p->kv_norm == nullptr || p->c == nullptr)) return UMB_ERR_ARG;
    if (p->qsrc != nullptr && (p->heads < 1 || p->dim < 0 || p->q == nullptr)) return UMB_ERR_ARG;
    cudaStream_t st = (cudaStream_t)stream;
    const int work = p->qsrc != nullptr ? p->heads * (p->dim + p->rope_dim) : (p->dq != nullptr ? p->q_rank : 0) + p->kv_rank + p->rope_dim;
    const int threads = work >= 4096 ? 512 : (work >= 1024 ? 256 : 128);
    UMBS_DISPATCH_T(dtype, latent_prep_kernel<T><<<batch->n_tokens, threads, (size_t)(p->rot_dims + 2) * sizeof(float), st>>>(*p, *batch));
    count_launches(1);
    return (int)cudaGetLastError();
}

extern "C" int umbs_softcap(float* z, int64_t n, float cap, umbs_stream_t stream) {
    if (n <= 0) return 0;
    if (!(cap > 0.f)) return UMB_ERR_ARG;
    softcap_kernel<<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(z, n, cap);
    count_launches(1);
    return (int)cudaGetLastError();
}

extern "C" int umbs_attention_prep(int dtype, const float* proj, int64_t ld, const float* bias, const umbs_batch_t* batch,
                                   int heads, int kv_heads, int dim, int vdim, int values_are_keys, int taps,
                                   const float* conv_w, float* conv_state, int slots, int rot_dims, const float* inv_freq,
                                   float rot_mag, void* q, void* kv, umbs_stream_t stream) {
    if (kv_heads < 1) return UMB_ERR_ARG;
    return umbs_attention_prep_ex(dtype, proj, ld, bias, batch, heads, kv_heads, dim, vdim, values_are_keys, taps, conv_w, conv_state,
                                  slots, rot_dims, inv_freq, rot_mag, 1, nullptr, nullptr, 0.f, q, kv, stream);
}

extern "C" int umbs_attention_prep_ex(int dtype, const float* proj, int64_t ld, const float* bias, const umbs_batch_t* batch,
                                      int heads, int kv_heads, int dim, int vdim, int values_are_keys, int taps,
                                      const float* conv_w, float* conv_state, int slots, int rot_dims, const float* inv_freq,
                                      float rot_mag, int maps, const float* q_norm_w, const float* k_norm_w, float eps, void* q,
                                      void* kv, umbs_stream_t stream) {
    return umbs_attention_prep_opts(dtype, proj, ld, bias, batch, heads, kv_heads, dim, vdim, values_are_keys, taps, conv_w, conv_state,
                                    slots, rot_dims, inv_freq, rot_mag, maps, q_norm_w, k_norm_w, eps, nullptr, q, kv, stream);
}

extern "C" int umbs_attention_prep_opts(int dtype, const float* proj, int64_t ld, const float* bias, const umbs_batch_t* batch, int heads,
                                        int kv_heads, int dim, int vdim, int values_are_keys, int taps, const float* conv_w,
                                        float* conv_state, int slots, int rot_dims, const float* inv_freq, float rot_mag, int maps,
                                        const float* q_norm_w, const float* k_norm_w, float eps, const umbs_prep_opts_t* opts, void* q,
                                        void* kv, umbs_stream_t stream) {
    umbs_prep_opts_t po{};
    if (opts != nullptr) po = *opts;
    if (po.v_mix < UMBS_VMIX_NONE || po.v_mix > UMBS_VMIX_MIX) return UMB_ERR_ARG;
    if (po.v_mix != UMBS_VMIX_NONE && (po.v_source == nullptr || values_are_keys || kv_heads < 1)) return UMB_ERR_ARG;
    if (batch->n_tokens <= 0) return 0;
    if (maps < 1) maps = 1;
    if (rot_dims < 0 || rot_dims > dim || (rot_dims & 1) || taps < 1 || kv_heads < 0 || heads < 1) return UMB_ERR_ARG;
    if (kv_heads > 0 ? (heads % kv_heads != 0 || kv == nullptr) : values_are_keys) return UMB_ERR_ARG;
    if (values_are_keys && vdim != dim) return UMB_ERR_ARG;
    if (taps > 1 && (conv_w == nullptr || conv_state == nullptr)) return UMB_ERR_ARG;
    cudaStream_t st = (cudaStream_t)stream;
    const int C = (heads + kv_heads) * maps * dim;
    const size_t smem = ((size_t)C + rot_dims + 2) * sizeof(float);
    if (smem > 48 * 1024) return UMB_ERR_UNSUPPORTED;
    // a small step (decoding) has few blocks: spread a token's channels over up to 1024 threads
    const int threads = batch->n_tokens <= 64 ? std::min(1024, (C + 31) / 32 * 32) : (C >= 1024 ? 256 : 128);
    UMBS_DISPATCH_T(dtype, attention_prep_kernel<T><<<batch->n_tokens, threads, smem, st>>>(
                               proj, ld, bias, *batch, heads, kv_heads, dim, vdim, values_are_keys, taps, conv_w, conv_state, slots,
                               rot_dims, inv_freq, rot_mag, maps, q_norm_w, k_norm_w, eps, po, (T*)q, (T*)kv));
    count_launches(1);
    return (int)cudaGetLastError();
}

extern "C" int umbs_kv_pool(int dtype, const void* kv, const void* kv_cache, int kv_len, void* pool_cache, int pool_len,
                            const umbs_batch_t* batch, int row, int pool, umbs_stream_t stream) {
    if (batch->n_tokens <= 0 || pool <= 0) return 0;
    if (kv_len < pool) return UMB_ERR_ARG;               // a block's older tokens must still sit in the cache
    cudaStream_t st = (cudaStream_t)stream;
    const dim3 grid(batch->max_seq_len / pool + 1, batch->n_seqs, (row + 255) / 256);
    UMBS_DISPATCH_T(dtype, kv_pool_kernel<T><<<grid, 256, 0, st>>>((const T*)kv, (const T*)kv_cache, kv_len, (T*)pool_cache,
                                                                   pool_len, *batch, row, pool));
    count_launches(1);
    return (int)cudaGetLastError();
}
