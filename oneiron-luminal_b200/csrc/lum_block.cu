// Row-wise kernels of decoder layers that are described one by one, and their attention: norms, residual streams, query / key
// preparation with the cache append, and attention over a window or a chunk with learned per-head temperature and distance bias, or
// as the difference of two maps.
//
//   norm_rows     RMS or layer norm of rows of the residual stream -> operand of the next product
//   stream_rows   several residual streams: a sublayer's output taken in, the next sublayer's input mixed and normalised
//   qkv_rows      queries and keys normalised over the whole projection, queries scaled (score factor x temperature), values mixed
//                 with the first mixing layer's; keys and values rounded to the cache type and appended
//   qkv_head_rows the same for heads prepared one by one: short convolution, norm per head, rotation
//   attn_band     attention of single rows over the cache: any head sizes, any number of query heads per K/V head, f32 or bf16
//                 cache.  PREP 1 / 2: one row, with all of qkv_rows / qkv_head_rows in the prologue (a decode step's attention is one
//                 kernel).
// Everything here is computed in f32.  The tensor-core form for prompts is in lum_attn_tc.cu.
#include <cuda_bf16.h>
#include <cstdlib>

#include "lum_gemv_dev.cuh"
#include "lum_dense.cuh"

namespace lum {

// ------------------------------------------------------------------------------------------------ norms
__global__ void __launch_bounds__(256) norm_rows(const NormRowsArgs a) {
    extern __shared__ __align__(16) float nr_row[];
    __shared__ float red[32];
    const int m = blockIdx.x, tid = threadIdx.x, W = a.norm.width;
    const float* x = a.x + (size_t)(a.row_index ? a.row_index[m] : m) * a.ldx;
    float s = 0.0f;
    const bool vec = (W & 3) == 0 && (a.ldx & 3) == 0;
    if (vec) {
#pragma unroll 4
        for (int i = tid; i < W / 4; i += 256) { const float4 v = ((const float4*)x)[i]; ((float4*)nr_row)[i] = v; s += (v.x + v.y) + (v.z + v.w); }
    } else {
        for (int i = tid; i < W; i += 256) { const float v = x[i]; nr_row[i] = v; s += v; }
    }
    float mean = 0.0f;
    if (a.norm.mode == NORM_LAYER) mean = block_sum(s, red, tid, 256, 1) / (float)W;
    s = 0.0f;
    if (vec) {
        for (int i = tid; i < W / 4; i += 256) {
            const float4 v = ((const float4*)nr_row)[i];
            const float d0 = v.x - mean, d1 = v.y - mean, d2 = v.z - mean, d3 = v.w - mean;
            s = fmaf(d0, d0, s); s = fmaf(d1, d1, s); s = fmaf(d2, d2, s); s = fmaf(d3, d3, s);
        }
    } else {
        for (int i = tid; i < W; i += 256) { const float d = nr_row[i] - mean; s = fmaf(d, d, s); }
    }
    const float inv = 1.0f / sqrtf(block_sum(s, red, tid, 256, 1) / (float)W + a.norm.eps);
    auto value = [&](int k) -> float {
        if (k >= W) return 0.0f;
        float v = (nr_row[k] - mean) * inv * (a.norm.gain0 + a.norm.gain[k]);
        return a.norm.bias ? v + a.norm.bias[k] : v;
    };
    if (a.kind == WK_BF16) {
        for (int g = tid; g < a.out.chunks * 8; g += 256) {
            float f[8];
            if (vec && g * 8 + 8 <= W) {
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    const float4 v = ((const float4*)nr_row)[g * 2 + h];
                    float4 gn = ((const float4*)a.norm.gain)[g * 2 + h];
                    const float z = a.norm.gain0;
                    gn = make_float4(gn.x + z, gn.y + z, gn.z + z, gn.w + z);
                    const float4 b = a.norm.bias ? ((const float4*)a.norm.bias)[g * 2 + h] : make_float4(0.f, 0.f, 0.f, 0.f);
                    f[4 * h] = (v.x - mean) * inv * gn.x + b.x; f[4 * h + 1] = (v.y - mean) * inv * gn.y + b.y;
                    f[4 * h + 2] = (v.z - mean) * inv * gn.z + b.z; f[4 * h + 3] = (v.w - mean) * inv * gn.w + b.w;
                }
            } else {
#pragma unroll
                for (int i = 0; i < 8; i++) f[i] = value(g * 8 + i);
            }
            uint32_t w[4];
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const __nv_bfloat162 b = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
                w[i] = *(const uint32_t*)&b;
            }
            *(uint4*)((unsigned char*)a.out.p + row_operand_off(WK_BF16, a.out.chunks, m, g * 8)) = make_uint4(w[0], w[1], w[2], w[3]);
        }
    } else {
        float* o = (float*)a.out.p + (size_t)m * a.out.chunks * 32;
        for (int k = tid; k < a.out.chunks * 32; k += 256) o[k] = value(k);
    }
}
cudaError_t launch_norm_rows(const NormRowsArgs& a, cudaStream_t st) {
    if (a.M <= 0 || a.norm.mode == NORM_NONE || a.norm.width > a.out.chunks * chunk_elems(a.kind)) return cudaErrorInvalidValue;
    const size_t smem = (size_t)a.norm.width * 4;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute((const void*)norm_rows, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) return e;
        if (smem > 200 * 1024) return cudaErrorInvalidValue;
    }
    norm_rows<<<a.M, 256, smem, st>>>(a);
    return cudaGetLastError();
}

// ------------------------------------------------------------------------------------------------ queries, keys, values
// 1 / root mean square of n elements (1 without a gain); called by all 256 threads
__device__ __forceinline__ float proj_inv_rms(const float* v, int n, const float* gain, float eps, float* red, int tid) {
    if (!gain) return 1.0f;
    float s = 0.0f;
#pragma unroll 16
    for (int i = tid; i < n; i += 256) { const float t = v[i]; s = fmaf(t, t, s); }
    return 1.0f / sqrtf(block_sum(s, red, tid, 256, 1) / (float)n + eps);
}
__device__ __forceinline__ float prep_query(const QkvArgs& p, const float* q, float inv, int head, int e) {
    if (e >= p.dk) return 0.0f;
    const int i = head * p.dk + e;
    const float v = p.q_gain ? q[i] * inv * p.q_gain[i] : q[i];
    return v * (p.temp ? p.scale * p.temp[head] : p.scale);
}
__device__ __forceinline__ float prep_key(const QkvArgs& p, const float* k, float inv, int kvh, int e) {
    if (e >= p.dk) return 0.0f;
    const int i = kvh * p.dk + e;
    return p.k_gain ? k[i] * inv * p.k_gain[i] : k[i];
}
__device__ __forceinline__ float prep_value(const QkvArgs& p, const float* v, const float* v_first, int kvh, int e) {
    if (e >= p.dv) return 0.0f;
    const int i = kvh * p.dv + e;
    if (p.mix != 2) return v[i];
    const float l = p.lambda[0];
    return (1.0f - l) * v[i] + l * v_first[i];
}
__device__ __forceinline__ void cache_store(void* cache, int bf16, size_t off, float v) {
    if (bf16) ((__nv_bfloat16*)cache)[off] = __float2bfloat16_rn(v);
    else ((float*)cache)[off] = v;
}

__global__ void __launch_bounds__(256) qkv_rows(const BandArgs a) {
    __shared__ float red[32];
    const QkvArgs& p = a.p;
    const int m = blockIdx.x, tid = threadIdx.x;
    const int pos = a.row_pos[m], seq = a.row_seq ? a.row_seq[m] : a.seq0;
    if (pos < 0 || pos >= a.max_seq || seq < 0 || seq >= a.max_batch) {
        if (tid == 0) atomicOr(a.status, LUM_ST_BAD_POS);
        return;
    }
    const float* row = p.qkv + (size_t)m * p.ld;
    const float *q = row + p.q_off, *k = row + p.k_off, *v = row + p.v_off;
    const float iq = proj_inv_rms(q, p.n_q * p.dk, p.q_gain, p.eps, red, tid), ik = proj_inv_rms(k, p.n_kv * p.dk, p.k_gain, p.eps, red, tid);
    if (p.q_gain && (p.dk & 3) == 0 && ((p.ld | p.q_off) & 3) == 0) {      // four at a time (dkp is a multiple of 16)
        const int n4 = p.dkp / 4;
#pragma unroll 4
        for (int i = tid; i < p.n_q * n4; i += 256) {
            const int h = i / n4, e = (i - h * n4) * 4, src = (h * p.dk + e) / 4;
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
            if (e < p.dk) {
                const float4 v = ((const float4*)q)[src], g = ((const float4*)p.q_gain)[src];
                const float f = p.temp ? p.scale * p.temp[h] : p.scale;
                o = make_float4(v.x * iq * g.x * f, v.y * iq * g.y * f, v.z * iq * g.z * f, v.w * iq * g.w * f);
            }
            ((float4*)(a.q_out + (size_t)m * p.n_q * p.dkp))[i] = o;
        }
    } else {
        for (int i = tid; i < p.n_q * p.dkp; i += 256) a.q_out[(size_t)m * p.n_q * p.dkp + i] = prep_query(p, q, iq, i / p.dkp, i % p.dkp);
    }
    const size_t prow = kv_phys_row(a.pg, seq, a.max_seq, pos);
    const size_t ko = prow * p.n_kv * p.dkp, vo = prow * p.n_kv * p.dvp;
    for (int i = tid; i < p.n_kv * p.dkp; i += 256) cache_store(a.k_cache, a.kv_bf16, ko + i, prep_key(p, k, ik, i / p.dkp, i % p.dkp));
    float* vf = p.mix ? p.v_first + (size_t)m * p.ld_vfirst : nullptr;
    for (int i = tid; i < p.n_kv * p.dvp; i += 256) cache_store(a.v_cache, a.kv_bf16, vo + i, prep_value(p, v, vf, i / p.dvp, i % p.dvp));
    if (p.mix == 1) for (int i = tid; i < p.n_kv * p.dv; i += 256) vf[i] = v[i];
}
cudaError_t launch_qkv_rows(const BandArgs& a, cudaStream_t st) {
    if (a.M <= 0) return cudaErrorInvalidValue;
    qkv_rows<<<a.M, 256, 0, st>>>(a);
    return cudaGetLastError();
}

// ------------------------------------------------------------------------------------------------ heads prepared one by one
// One head (and map) of n dimensions in shared memory, by one warp: RMS norm with a shared gain, then the rotation, in place.
__device__ __forceinline__ void head_norm_rotate(float* v, int n, const float* gain, float eps, const float2* rot, int rot_dims, int lane) {
    __syncwarp();
    if (gain) {
        float s = 0.0f;
        for (int e = lane; e < n; e += 32) s = fmaf(v[e], v[e], s);
        const float inv = 1.0f / sqrtf(warp_sum(s) / (float)n + eps);
        for (int e = lane; e < n; e += 32) v[e] = v[e] * inv * gain[e];
        __syncwarp();
    }
    const int half = rot_dims / 2;
    for (int e = lane; e < half; e += 32) {
        const float2 cs = rot[e];
        const float x = v[e], y = v[e + half];
        v[e] = x * cs.x - y * cs.y;
        v[e + half] = fmaf(y, cs.x, x * cs.y);
    }
    __syncwarp();
}
// Rows of a pass: a warp takes one head (of a map) of queries or keys, or 32 NJ columns of values, of RB rows.  A lane owns the columns
// lane + 32 j; the convolution's window slides over the rows in registers, the norms of the rows are summed side by side, and the
// rotation finds its other half in shared memory.
template <int NJ, int RB>
__global__ void __launch_bounds__(256) qkv_head_rows(const BandArgs a) {
    extern __shared__ __align__(16) float qh[];
    const QkvArgs& p = a.p;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int nq = p.n_q * p.maps, nk = p.n_kv * p.maps, vd = p.n_kv * p.dv, half = p.rot_dims / 2;
    const int job = blockIdx.x * 8 + warp, m0 = blockIdx.y * RB, nr = min(RB, a.M - m0);
    if (job >= nq + nk + (vd + 32 * NJ - 1) / (32 * NJ)) return;
    const bool is_q = job < nq, is_v = job >= nq + nk;
    const int v0 = (job - nq - nk) * 32 * NJ;                              // first column of a value piece
    const int n = is_v ? min(32 * NJ, vd - v0) : p.dk;
    const int c0 = is_q ? p.q_off + job * p.dk : is_v ? p.v_off + v0 : p.k_off + (job - nq) * p.dk;
    float* buf = qh + warp * RB * 32 * NJ;
    int pos[RB], seq[RB];
    bool bad = false;
#pragma unroll
    for (int r = 0; r < RB; r++) {
        pos[r] = r < nr ? a.row_pos[m0 + r] : 0;
        seq[r] = r < nr && a.row_seq ? a.row_seq[m0 + r] : a.seq0;
        bad = bad || pos[r] < 0 || pos[r] >= a.max_seq || seq[r] < 0 || seq[r] >= a.max_batch;
    }
    if (bad) {
        if (lane == 0) atomicOr(a.status, LUM_ST_BAD_POS);
        return;
    }
    float x[RB][NJ];
    if (p.conv.taps == 4 && !a.row_seq && m0 >= 3) {                       // the rows before are in this pass
        const float* src = p.qkv + (size_t)(m0 - 3) * p.ld + c0 + lane;
        float h[3][NJ];
        float4 w[NJ];
#pragma unroll
        for (int j = 0; j < NJ; j++) {
            const bool in = lane + 32 * j < n;
            w[j] = in ? *(const float4*)(p.conv.w + (size_t)(c0 + lane + 32 * j) * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int d = 0; d < 3; d++) h[d][j] = in ? src[(size_t)d * p.ld + 32 * j] : 0.0f;
#pragma unroll
            for (int r = 0; r < RB; r++) x[r][j] = in && r < nr ? src[(size_t)(r + 3) * p.ld + 32 * j] : 0.0f;
        }
#pragma unroll
        for (int j = 0; j < NJ; j++)
#pragma unroll
            for (int r = 0; r < RB; r++) {
                const float now = x[r][j];
                x[r][j] = fmaf(w[j].w, now, fmaf(w[j].z, h[2][j], fmaf(w[j].y, h[1][j], w[j].x * h[0][j])));
                h[0][j] = h[1][j]; h[1][j] = h[2][j]; h[2][j] = now;
            }
    } else {
#pragma unroll
        for (int r = 0; r < RB; r++) {
            float* ring = p.conv.ring + (size_t)seq[r] * p.conv.taps * p.conv.ch;
            const float* src = p.qkv + (size_t)(m0 + r) * p.ld;
#pragma unroll
            for (int j = 0; j < NJ; j++) {
                const int e = lane + 32 * j;
                x[r][j] = 0.0f;
                if (r < nr && e < n) {
                    x[r][j] = conv_at(p.conv, ring, src, p.ld, a.row_seq ? 0 : m0 + r, pos[r], c0 + e);
                    // one row of its sequence: its value takes the place in the ring that no row of this pass reads
                    if (p.conv.taps > 0 && (a.row_seq || a.M == 1)) ring[(size_t)(pos[r] % p.conv.taps) * p.conv.ch + c0 + e] = src[c0 + e];
                }
            }
        }
    }
    if (is_v) {
#pragma unroll
        for (int r = 0; r < RB; r++) {
            if (r >= nr) continue;
            const size_t vo = kv_phys_row(a.pg, seq[r], a.max_seq, pos[r]) * p.n_kv * p.dvp;
#pragma unroll
            for (int j = 0; j < NJ; j++) {
                const int c = v0 + lane + 32 * j, h = c / p.dv;
                if (lane + 32 * j < n) cache_store(a.v_cache, a.kv_bf16, vo + (size_t)h * p.dvp + (c - h * p.dv), x[r][j]);      // (padding stays zero)
            }
        }
        return;
    }
    const float* gain = is_q ? p.q_gain : p.k_gain;
    if (gain) {
        float s[RB];
#pragma unroll
        for (int r = 0; r < RB; r++) {
            s[r] = 0.0f;
#pragma unroll
            for (int j = 0; j < NJ; j++) s[r] = fmaf(x[r][j], x[r][j], s[r]);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int r = 0; r < RB; r++) s[r] += __shfl_xor_sync(0xffffffffu, s[r], o);
#pragma unroll
        for (int r = 0; r < RB; r++) s[r] = 1.0f / sqrtf(s[r] / (float)n + p.eps);
#pragma unroll
        for (int j = 0; j < NJ; j++) {
            const float g = lane + 32 * j < n ? gain[lane + 32 * j] : 0.0f;
#pragma unroll
            for (int r = 0; r < RB; r++) x[r][j] *= s[r] * g;
        }
    }
    if (half == 16 * NJ) {                                     // the whole head turns, and both halves of a pair lie in this lane
#pragma unroll
        for (int r = 0; r < RB; r++) {
            const float2* rot = p.rot + (size_t)pos[r] * half + lane;
#pragma unroll
            for (int j = 0; j < NJ / 2; j++) {
                const float2 cs = rot[32 * j];
                const float u = x[r][j], v = x[r][j + NJ / 2];
                x[r][j] = u * cs.x - v * cs.y;
                x[r][j + NJ / 2] = fmaf(v, cs.x, u * cs.y);
            }
        }
    } else if (half > 0) {
#pragma unroll
        for (int r = 0; r < RB; r++)
#pragma unroll
            for (int j = 0; j < NJ; j++) buf[(r * NJ + j) * 32 + lane] = x[r][j];
        __syncwarp();
#pragma unroll
        for (int r = 0; r < RB; r++)
#pragma unroll
            for (int j = 0; j < NJ; j++) {
                const int e = lane + 32 * j, i = e < half ? e : e - half;
                if (e < 2 * half && r < nr) {
                    const float2 cs = p.rot[(size_t)pos[r] * half + i];
                    const float o = buf[r * NJ * 32 + (e < half ? e + half : i)];
                    x[r][j] = e < half ? x[r][j] * cs.x - o * cs.y : fmaf(x[r][j], cs.x, o * cs.y);
                }
            }
    }
#pragma unroll
    for (int r = 0; r < RB; r++) {
        if (r >= nr) continue;
        if (is_q) {
            float* o = a.q_out + ((size_t)(m0 + r) * nq + job) * p.dkp + lane;
#pragma unroll
            for (int j = 0; j < NJ; j++) if (lane + 32 * j < p.dkp) o[32 * j] = x[r][j] * p.scale;
        } else {
            const size_t ko = kv_phys_row(a.pg, seq[r], a.max_seq, pos[r]) * nk * p.dkp + (size_t)(job - nq) * p.dkp;
#pragma unroll
            for (int j = 0; j < NJ; j++) if (lane + 32 * j < p.dkp) cache_store(a.k_cache, a.kv_bf16, ko + lane + 32 * j, x[r][j]);
        }
    }
}
cudaError_t launch_qkv_head_rows(const BandArgs& a, cudaStream_t st) {
    const QkvArgs& p = a.p;
    if (a.M <= 0 || !p.per_head || p.maps < 1 || p.dkp > 1024 || p.dk > p.dkp) return cudaErrorInvalidValue;
    const int NJ = p.dkp <= 64 ? 2 : p.dkp <= 128 ? 4 : p.dkp <= 256 ? 8 : 32, RB = NJ == 32 || a.row_seq || a.M < 32 ? 1 : NJ == 8 ? 4 : 8;
    const void* fn = NJ == 32 ? (const void*)qkv_head_rows<32, 1>
                     : RB == 1 ? (NJ == 2 ? (const void*)qkv_head_rows<2, 1> : NJ == 4 ? (const void*)qkv_head_rows<4, 1> : (const void*)qkv_head_rows<8, 1>)
                               : (NJ == 2 ? (const void*)qkv_head_rows<2, 8> : NJ == 4 ? (const void*)qkv_head_rows<4, 8> : (const void*)qkv_head_rows<8, 4>);
    const int jobs = (p.n_q + p.n_kv) * p.maps + (p.n_kv * p.dv + 32 * NJ - 1) / (32 * NJ);
    const size_t smem = (size_t)8 * RB * 32 * NJ * 4;                      // at most 32 KB
    BandArgs b = a;
    void* params[] = {&b};
    return cudaLaunchKernel(fn, dim3((jobs + 7) / 8, (a.M + RB - 1) / RB), dim3(256), params, smem, st);
}

// ------------------------------------------------------------------------------------------------ residual streams
// One CTA per row.  SM: streams the registers are laid out for.
template <int SM>
__global__ void __launch_bounds__(256) stream_rows(const StreamRowsArgs a) {
    extern __shared__ __align__(16) float sr_row[];
    __shared__ float red[32], mix[SM * SM], out[SM], nxt[SM];
    const StreamArgs& h = a.hc;
    const int m = blockIdx.x, tid = threadIdx.x, W = a.width, n = h.n;
    if (tid < n) {
        out[tid] = h.out ? h.out[tid] : 1.0f;
        nxt[tid] = h.next ? h.next[tid] : 1.0f;
    }
    for (int i = tid; i < n * n; i += 256) mix[i] = h.mix ? h.mix[i] : (i / n == i % n ? 1.0f : 0.0f);
    if (a.use_pdl) { pdl_launch_dependents(); pdl_grid_wait(); }
    int tok = 0;
    if (!a.y) {
        tok = a.state ? a.state->tok : a.row_tok[m];
        const int pos = a.state ? a.state->pos : a.row_pos[m];
        if (tok < 0 || tok >= a.vocab) { if (tid == 0) atomicOr(a.status, LUM_ST_BAD_TOKEN); tok = 0; }
        if (pos < 0 || pos >= a.max_seq) { if (tid == 0) atomicOr(a.status, LUM_ST_BAD_POS); }
    }
    __syncthreads();
    float* x = h.x + (size_t)m * n * h.ldx;
    float ss = 0.0f;
    const bool vec_table = (W & 3) == 0;
    for (int i = tid; i < h.ldx / 4; i += 256) {
        float4 y, u = make_float4(0.f, 0.f, 0.f, 0.f);
        if (a.y) {
            y = ((const float4*)(a.y + (size_t)m * a.ldy))[i];
            float4 old[SM];
#pragma unroll
            for (int s = 0; s < SM; s++) if (s < n) old[s] = ((const float4*)(x + (size_t)s * h.ldx))[i];
#pragma unroll
            for (int t = 0; t < SM; t++) {
                if (t < n) {
                    const float o = out[t];
                    float4 v = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
                    for (int s = 0; s < SM; s++)
                        if (s < n) {
                            const float w = mix[s * n + t];
                            v.x = fmaf(w, old[s].x, v.x); v.y = fmaf(w, old[s].y, v.y); v.z = fmaf(w, old[s].z, v.z); v.w = fmaf(w, old[s].w, v.w);
                        }
                    ((float4*)(x + (size_t)t * h.ldx))[i] = v;
                    const float g = nxt[t];
                    u.x = fmaf(g, v.x, u.x); u.y = fmaf(g, v.y, u.y); u.z = fmaf(g, v.z, u.z); u.w = fmaf(g, v.w, u.w);
                }
            }
        } else {
            float e[4] = {0.f, 0.f, 0.f, 0.f};
            const size_t o = (size_t)tok * W + 4 * i;
            if (vec_table && a.table_kind == WK_BF16) {
                const uint2 b = *(const uint2*)((const uint16_t*)a.table + o);
                e[0] = __uint_as_float(b.x << 16); e[1] = __uint_as_float(b.x & 0xffff0000u); e[2] = __uint_as_float(b.y << 16); e[3] = __uint_as_float(b.y & 0xffff0000u);
                if (4 * i >= W) e[0] = e[1] = e[2] = e[3] = 0.0f;
            } else {
#pragma unroll
                for (int k = 0; k < 4; k++)
                    if (4 * i + k < W) e[k] = a.table_kind == WK_BF16 ? bf16_bits_to_f32(((const uint16_t*)a.table)[o + k]) : ((const float*)a.table)[o + k];
            }
            y = make_float4(e[0] * a.scale, e[1] * a.scale, e[2] * a.scale, e[3] * a.scale);
            for (int t = 0; t < n; t++) {
                ((float4*)(x + (size_t)t * h.ldx))[i] = y;
                const float g = nxt[t];
                u.x = fmaf(g, y.x, u.x); u.y = fmaf(g, y.y, u.y); u.z = fmaf(g, y.z, u.z); u.w = fmaf(g, y.w, u.w);
            }
        }
        if (h.u) ((float4*)(h.u + (size_t)m * h.ldx))[i] = u;
        else {
            ((float4*)sr_row)[i] = u;
            ss = fmaf(u.x, u.x, ss); ss = fmaf(u.y, u.y, ss); ss = fmaf(u.z, u.z, ss); ss = fmaf(u.w, u.w, ss);      // (columns beyond W are zero)
        }
    }
    if (h.u) return;
    const float inv = 1.0f / sqrtf(block_sum(ss, red, tid, 256, 1) / (float)W + a.norm.eps);
    if (a.kind == WK_BF16) {
        for (int g = tid; g < a.out.chunks * 8; g += 256) {
            uint32_t w[4];
            float f[8];
#pragma unroll
            for (int i = 0; i < 8; i++) f[i] = g * 8 + i < W ? sr_row[g * 8 + i] * inv * (a.norm.gain0 + a.norm.gain[g * 8 + i]) : 0.0f;
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const __nv_bfloat162 b = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
                w[i] = *(const uint32_t*)&b;
            }
            *(uint4*)((unsigned char*)a.out.p + row_operand_off(WK_BF16, a.out.chunks, m, g * 8)) = make_uint4(w[0], w[1], w[2], w[3]);
        }
    } else {
        float* o = (float*)a.out.p + (size_t)m * a.out.chunks * 32;
        for (int k = tid; k < a.out.chunks * 32; k += 256) o[k] = k < W ? sr_row[k] * inv * (a.norm.gain0 + a.norm.gain[k]) : 0.0f;
    }
}
cudaError_t launch_stream_rows(const StreamRowsArgs& a_in, cudaStream_t st) {
    StreamRowsArgs a = a_in;
    if (a.M <= 0 || a.hc.n < 1 || a.hc.n > kMaxStreams || a.hc.ldx % 8 || a.hc.ldx < a.width || (!a.hc.u && (a.norm.mode != NORM_RMS || a.width > a.out.chunks * chunk_elems(a.kind))))
        return cudaErrorInvalidValue;
    const void* fn = a.hc.n <= 1 ? (const void*)stream_rows<1> : a.hc.n <= 2 ? (const void*)stream_rows<2> : a.hc.n <= 4 ? (const void*)stream_rows<4> : (const void*)stream_rows<8>;
    const size_t smem = a.hc.u ? 0 : (size_t)a.hc.ldx * 4;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) return e;
        if (smem > 200 * 1024) return cudaErrorInvalidValue;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.M); cfg.blockDim = dim3(256); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization; at[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at; cfg.numAttrs = a.use_pdl ? 1 : 0;
    void* params[] = {&a};
    return cudaLaunchKernelExC(&cfg, fn, params);
}

// ------------------------------------------------------------------------------------------------ attention, row by row
// One CTA = (split of the visible keys, K/V head and block of up to 8 of its query heads, row).  64 keys at a time:
//   scores   4 lanes per key, each a share of the head dimension for all 8 queries; two shuffles; distance bias; shared memory
//   softmax  one warp per query head: running maximum and sum
//   values   thread = two value dimensions and a share of the keys
// A tile's key and value loads are all issued before anything of the previous tile is waited for again: the next tile's keys are in
// flight during this tile's softmax, its values during its scores.
// The splits of a row are the CTAs of a thread-block cluster and fold their (maximum, sum, vector) through its shared memory.
// With two maps the cluster holds the splits of both (rank = map * splits + split): keys and queries are the map's, values are shared,
// and the fold subtracts the maps, head by head.
namespace {
constexpr int kBdTK = 64, kBdR = 8, kBdMaxSplits = 16;    // (splits of both maps together)
constexpr int kBdKv = 4, kBdVv = 16;     // 16-byte key groups / value pairs of a tile a thread keeps in registers (longer heads: the rest is loaded where used)
struct BdSmem {      // offsets in floats
    int q, sc, red, o, ml, wgt, knew, vnew, part, total;
};
__host__ __device__ inline BdSmem bd_layout(int dkp, int dvp) {
    BdSmem s;
    s.q = 0;
    s.sc = s.q + kBdR * dkp;
    s.red = s.sc + kBdR * kBdTK;                         // scores / weights [key][8]
    s.ml = s.red + 32;                                   // maximum [8], sum [8], correction [8]
    s.wgt = s.ml + 32;                                   // [splits][8]
    s.o = s.wgt + kBdMaxSplits * kBdR;
    s.knew = s.o + kBdR * dvp;                           // the new row in the cache's type (room for f32)
    s.vnew = s.knew + dkp;
    s.part = s.vnew + dvp;                               // [shares of the keys][8][dvp]
    const int npair = dvp / 2, nsub = npair >= 256 ? 1 : 256 / npair;
    s.total = s.part + nsub * kBdR * dvp;
    return s;
}
}  // namespace

template <bool BF16> struct BandPair { using type = uint32_t; };      // two values as they lie in the cache
template <> struct BandPair<false> { using type = float2; };
__device__ __forceinline__ float2 band_pair(uint32_t w) { return make_float2(__uint_as_float(w << 16), __uint_as_float(w & 0xffff0000u)); }
__device__ __forceinline__ float2 band_pair(float2 v) { return v; }

// RB: query heads the registers are laid out for (4 or 8)
// PREP: 0 rows prepared before, 1 prologue over the whole projection, 2 prologue head by head
template <bool BF16, int PREP, int RB>
__global__ void __launch_bounds__(256, 2) attn_band(const BandArgs a, int S, int HB) {
    extern __shared__ __align__(16) float bd[];
    const QkvArgs& p = a.p;
    const BdSmem L = bd_layout(p.dkp, p.dvp);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    constexpr bool FUSED = PREP != 0;
    const int maps = PREP == 1 ? 1 : p.maps, map = blockIdx.x / S, sp = blockIdx.x - map * S;
    const int kvh = blockIdx.y / HB, hb = blockIdx.y % HB, m = blockIdx.z;
    const int R = p.n_q / p.n_kv, r0 = hb * kBdR, nr = min(kBdR, R - r0), head0 = kvh * R + r0;
    float *q_s = bd + L.q, *sc = bd + L.sc, *red = bd + L.red, *o_s = bd + L.o, *m_s = bd + L.ml, *l_s = m_s + 8, *c_s = m_s + 16;
    __shared__ float lam_s;
    if (FUSED) pdl_launch_dependents();
    if (maps == 2 && warp == 7) {                              // the second map's weight (weights only: nothing to wait for)
        float d1 = 0.0f, d2 = 0.0f;
        for (int e = lane; e < p.dk; e += 32) { d1 = fmaf(a.lq1[e], a.lk1[e], d1); d2 = fmaf(a.lq2[e], a.lk2[e], d2); }
        d1 = warp_sum(d1); d2 = warp_sum(d2);
        if (lane == 0) lam_s = expf(d1) - expf(d2) + a.diff;
    }
    if (FUSED) pdl_grid_wait();
    const int pos = FUSED ? a.state->pos : a.row_pos[m];
    const int seq = FUSED ? (PREP == 2 ? a.seq0 : 0) : (a.row_seq ? a.row_seq[m] : a.seq0);
    if (pos < 0 || pos >= a.max_seq || seq < 0 || seq >= a.max_batch) {          // (the same for every CTA of the cluster)
        if (FUSED && tid == 0 && sp == 0) atomicOr(a.status, LUM_ST_BAD_POS);
        return;
    }
    const size_t k_row = (size_t)p.n_kv * maps * p.dkp, v_row = (size_t)p.n_kv * p.dvp;
    const int kh = kvh * maps + map;                           // this map's keys

    if (PREP == 2) {
        const size_t prow = kv_phys_row(a.pg, 0, 0, pos);
        float* ring = p.conv.ring ? p.conv.ring + (size_t)seq * p.conv.taps * p.conv.ch : nullptr;
        float* ring_now = ring + (size_t)(p.conv.taps ? pos % p.conv.taps : 0) * p.conv.ch;
        const float2* rot = p.rot + (size_t)pos * (p.rot_dims / 2);
        // a warp per head: this CTA's queries, its key, its value; the step's own values enter the ring once per head (the CTA of the
        // first split; the row of the ring they replace is read by nobody)
        for (int job = warp; job < kBdR + 2; job += 8) {
            const bool is_q = job < kBdR, is_k = job == kBdR;
            float* v = is_q ? q_s + job * p.dkp : bd + L.part + (is_k ? p.dvp : 0);      // (f32 forms of key and value: the shares' area is free yet)
            const int n = job == kBdR + 1 ? p.dv : p.dk, np = job == kBdR + 1 ? p.dvp : p.dkp;
            const int c0 = is_q ? p.q_off + ((head0 + job) * maps + map) * p.dk : is_k ? p.k_off + kh * p.dk : p.v_off + kvh * p.dv;
            const bool real = !is_q || job < nr, keep = sp == 0 && (is_q || (hb == 0 && (is_k || map == 0)));
            for (int e = lane; e < np; e += 32) {
                float t = 0.0f;
                if (real && e < n) {
                    t = conv_at(p.conv, ring, p.qkv, 0, 0, pos, c0 + e);
                    if (keep && p.conv.taps > 0) ring_now[c0 + e] = p.qkv[c0 + e];
                }
                v[e] = t;
            }
            if (is_q) {
                if (real) {
                    head_norm_rotate(v, p.dk, p.q_gain, p.eps, rot, p.rot_dims, lane);
                    for (int e = lane; e < p.dk; e += 32) v[e] *= p.scale;
                }
            } else if (is_k) {
                head_norm_rotate(v, p.dk, p.k_gain, p.eps, rot, p.rot_dims, lane);
                for (int e = lane; e < p.dkp; e += 32) {
                    cache_store(bd + L.knew, BF16, e, v[e]);
                    if (keep) cache_store(a.k_cache, BF16, prow * k_row + (size_t)kh * p.dkp + e, v[e]);
                }
            } else {
                for (int e = lane; e < p.dvp; e += 32) {
                    const float t = v[e];
                    cache_store(bd + L.vnew, BF16, e, t);
                    if (keep) cache_store(a.v_cache, BF16, prow * v_row + (size_t)kvh * p.dvp + e, t);
                }
            }
        }
    } else if (PREP == 1) {
        const float *q = p.qkv + p.q_off, *k = p.qkv + p.k_off, *v = p.qkv + p.v_off;
        const float iq = proj_inv_rms(q, p.n_q * p.dk, p.q_gain, p.eps, red, tid), ik = proj_inv_rms(k, p.n_kv * p.dk, p.k_gain, p.eps, red, tid);
        for (int i = tid; i < kBdR * p.dkp; i += 256) {
            const int r = i / p.dkp;
            q_s[i] = r < nr ? prep_query(p, q, iq, head0 + r, i - r * p.dkp) : 0.0f;
        }
        const size_t prow = kv_phys_row(a.pg, 0, 0, pos);
        const bool keep = sp == 0 && hb == 0;
        for (int i = tid; i < p.dkp; i += 256) {
            const float t = prep_key(p, k, ik, kvh, i);
            cache_store(bd + L.knew, BF16, i, t);
            if (keep) cache_store(a.k_cache, BF16, prow * k_row + (size_t)kvh * p.dkp + i, t);
        }
        for (int i = tid; i < p.dvp; i += 256) {
            const float t = prep_value(p, v, p.v_first, kvh, i);
            cache_store(bd + L.vnew, BF16, i, t);
            if (keep) {
                cache_store(a.v_cache, BF16, prow * v_row + (size_t)kvh * p.dvp + i, t);
                if (p.mix == 1 && i < p.dv) p.v_first[kvh * p.dv + i] = t;
            }
        }
    } else {
        for (int i = tid; i < kBdR * p.dkp; i += 256) {
            const int r = i / p.dkp;
            q_s[i] = r < nr ? a.q[(((size_t)m * p.n_q + head0 + r) * maps + map) * p.dkp + (i - r * p.dkp)] : 0.0f;
        }
    }
    if (tid < 8) { m_s[tid] = -INFINITY; l_s[tid] = 0.0f; }
    const int lo = a.chunk > 0 ? pos / a.chunk * a.chunk : (a.window > 0 && pos + 1 > a.window) ? pos + 1 - a.window : 0;
    const int per = (pos + 1 - lo + S - 1) / S, k0 = lo + sp * per, k1 = min(pos + 1, k0 + per);
    const int npair = p.dvp / 2, nsub = npair >= 256 ? 1 : 256 / npair, sub = tid / npair, dv2 = tid - sub * npair;
    float acc[RB][2];
#pragma unroll
    for (int r = 0; r < RB; r++) acc[r][0] = acc[r][1] = 0.0f;

    const int key = tid >> 2, part = tid & 3, kgr = p.dkp / (BF16 ? 8 : 4);
    const size_t esz = BF16 ? 2 : 4;
    // row `j` of this K/V head (the row of this very step: from shared memory, its store to the cache may still be on the way)
    auto key_row = [&](int j) -> const char* {
        if (FUSED && j == pos) return (const char*)(bd + L.knew);
        return (const char*)a.k_cache + (kv_phys_row(a.pg, FUSED ? 0 : seq, FUSED ? 0 : a.max_seq, j) * k_row + (size_t)kh * p.dkp) * esz;
    };
    using VRaw = typename BandPair<BF16>::type;
    auto value_pair = [&](int j) -> VRaw {
        const char* vr = (const char*)(bd + L.vnew);
        if (!(FUSED && j == pos)) vr = (const char*)a.v_cache + (kv_phys_row(a.pg, FUSED ? 0 : seq, FUSED ? 0 : a.max_seq, j) * v_row + (size_t)kvh * p.dvp) * esz;
        return *((const VRaw*)vr + dv2);
    };
    float d[RB];
    auto dot_group = [&](const uint4& raw, int c) {
        if (BF16) {
            const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
            float kf[8];
#pragma unroll
            for (int t = 0; t < 4; t++) { kf[2 * t] = __uint_as_float(w[t] << 16); kf[2 * t + 1] = __uint_as_float(w[t] & 0xffff0000u); }
#pragma unroll
            for (int r = 0; r < RB; r++) {
                const float4 q0 = *(const float4*)(q_s + r * p.dkp + c * 8), q1 = *(const float4*)(q_s + r * p.dkp + c * 8 + 4);
                d[r] = fmaf(q0.x, kf[0], d[r]); d[r] = fmaf(q0.y, kf[1], d[r]); d[r] = fmaf(q0.z, kf[2], d[r]); d[r] = fmaf(q0.w, kf[3], d[r]);
                d[r] = fmaf(q1.x, kf[4], d[r]); d[r] = fmaf(q1.y, kf[5], d[r]); d[r] = fmaf(q1.z, kf[6], d[r]); d[r] = fmaf(q1.w, kf[7], d[r]);
            }
        } else {
            const float kf[4] = {__uint_as_float(raw.x), __uint_as_float(raw.y), __uint_as_float(raw.z), __uint_as_float(raw.w)};
#pragma unroll
            for (int r = 0; r < RB; r++) {
                const float4 q0 = *(const float4*)(q_s + r * p.dkp + c * 4);
                d[r] = fmaf(q0.x, kf[0], d[r]); d[r] = fmaf(q0.y, kf[1], d[r]); d[r] = fmaf(q0.z, kf[2], d[r]); d[r] = fmaf(q0.w, kf[3], d[r]);
            }
        }
    };
    uint4 kreg[kBdKv];
    auto load_keys = [&](int j0, int nk) {
        if (key < nk) {
            const uint4* kr = (const uint4*)key_row(j0 + key);
#pragma unroll
            for (int i = 0; i < kBdKv; i++) if (part + 4 * i < kgr) kreg[i] = kr[part + 4 * i];
        }
    };
    __syncthreads();
    if (k0 < k1) load_keys(k0, min(kBdTK, k1 - k0));

    for (int j0 = k0; j0 < k1; j0 += kBdTK) {
        const int nk = min(kBdTK, k1 - j0);
        VRaw vreg[kBdVv];
        if (sub < nsub) {
#pragma unroll
            for (int i = 0; i < kBdVv; i++) if (sub + i * nsub < nk) vreg[i] = value_pair(j0 + sub + i * nsub);
        }
        {   // scores
            const int j = j0 + key;
#pragma unroll
            for (int r = 0; r < RB; r++) d[r] = 0.0f;
            if (key < nk) {
#pragma unroll
                for (int i = 0; i < kBdKv; i++) if (part + 4 * i < kgr) dot_group(kreg[i], part + 4 * i);
                if (kgr > 4 * kBdKv) {
                    const uint4* kr = (const uint4*)key_row(j);
                    for (int c = part + 4 * kBdKv; c < kgr; c += 4) dot_group(kr[c], c);
                }
            }
#pragma unroll
            for (int r = 0; r < RB; r++) {
                d[r] += __shfl_xor_sync(0xffffffffu, d[r], 1);
                d[r] += __shfl_xor_sync(0xffffffffu, d[r], 2);
            }
#pragma unroll
            for (int r = 0; r < RB; r++) {
                if ((r & 3) == part && r < nr) {
                    float s = d[r];
                    if (a.r1) s -= distance_bias(a.r1[head0 + r], a.r2[head0 + r], (float)(pos - j));
                    sc[key * kBdR + r] = key < nk ? s : -INFINITY;
                }
            }
        }
        if (j0 + kBdTK < k1) load_keys(j0 + kBdTK, min(kBdTK, k1 - j0 - kBdTK));
        __syncthreads();
        if (warp < nr) {   // softmax bookkeeping of query head `warp`
            float* s = sc + warp;
            const float s0 = s[lane * kBdR], s1 = s[(lane + 32) * kBdR];
            float mx = fmaxf(s0, s1);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mo = m_s[warp], mn = fmaxf(mo, mx);          // finite: a tile holds at least one key
            const float p0 = expf(s0 - mn), p1 = expf(s1 - mn);      // exp(-inf) = 0 beyond the last key
            const float ps = warp_sum(p0 + p1);
            __syncwarp();
            s[lane * kBdR] = p0; s[(lane + 32) * kBdR] = p1;
            if (lane == 0) { const float c = mo == -INFINITY ? 0.0f : expf(mo - mn); m_s[warp] = mn; l_s[warp] = l_s[warp] * c + ps; c_s[warp] = c; }
        }
        __syncthreads();
        if (sub < nsub) {
#pragma unroll
            for (int r = 0; r < RB; r++) if (r < nr) { const float c = c_s[r]; acc[r][0] *= c; acc[r][1] *= c; }
            auto take = [&](const VRaw& raw, int t) {
                const float2 v = band_pair(raw);
                float w[RB];                                       // (heads beyond nr: whatever is there, never read back)
#pragma unroll
                for (int r = 0; r < RB; r += 4) *(float4*)&w[r] = *(const float4*)(sc + t * kBdR + r);
#pragma unroll
                for (int r = 0; r < RB; r++) { acc[r][0] = fmaf(w[r], v.x, acc[r][0]); acc[r][1] = fmaf(w[r], v.y, acc[r][1]); }
            };
#pragma unroll
            for (int i = 0; i < kBdVv; i++) if (sub + i * nsub < nk) take(vreg[i], sub + i * nsub);
            for (int t = sub + kBdVv * nsub; t < nk; t += nsub) take(value_pair(j0 + t), t);
        }
        __syncthreads();
    }
    // ---- fold the key shares, then the splits
    if (sub < nsub)
#pragma unroll
        for (int r = 0; r < RB; r++)
            if (r < nr) *(float2*)(bd + L.part + (sub * kBdR + r) * p.dvp + 2 * dv2) = make_float2(acc[r][0], acc[r][1]);
    __syncthreads();
    for (int i = tid; i < nr * p.dvp; i += 256) {
        float t = 0.0f;
        for (int s = 0; s < nsub; s++) t += bd[L.part + s * kBdR * p.dvp + i];
        o_s[i] = t;
    }
    __syncthreads();
    float* wgt = bd + L.wgt;
    if (maps == 2) {
        const int C = 2 * S, rank = blockIdx.x;
        cluster_arrive_release();
        cluster_wait_acquire();
        const uint32_t ml = smem_u32(m_s), ob = smem_u32(o_s);
        if (tid < 2 * nr) {                                    // weights of the splits of (map, head)
            const int mp = tid / nr, r = tid - mp * nr;
            float M = -INFINITY, Ls = 0.0f;
            for (int s = 0; s < S; s++) M = fmaxf(M, cluster_ld_f32(cluster_map(ml + r * 4, (uint32_t)(mp * S + s))));
            for (int s = 0; s < S; s++) {
                const uint32_t from = (uint32_t)(mp * S + s);
                const float ms = cluster_ld_f32(cluster_map(ml + r * 4, from)), c = ms == -INFINITY ? 0.0f : expf(ms - M);
                Ls = fmaf(cluster_ld_f32(cluster_map(ml + 32 + r * 4, from)), c, Ls);
                wgt[from * kBdR + r] = c;
            }
            const float f = (mp ? -lam_s : 1.0f) / Ls;
            for (int s = 0; s < S; s++) wgt[(mp * S + s) * kBdR + r] *= f;
        }
        __syncthreads();
        float* dif = bd + L.part;
        for (int r = rank; r < nr; r += C) {                   // whole heads, dealt to the CTAs of the cluster
            float ss = 0.0f;
            for (int e = tid; e < p.dv; e += 256) {
                float v = 0.0f;
                for (int s = 0; s < C; s++) v = fmaf(cluster_ld_f32(cluster_map(ob + (r * p.dvp + e) * 4, (uint32_t)s)), wgt[s * kBdR + r], v);
                dif[e] = v;
                ss = fmaf(v, v, ss);
            }
            const float f = (1.0f - a.diff) / sqrtf(block_sum(ss, red, tid, 256, 1) / (float)p.dv + p.eps);
            for (int e = tid; e < p.dv; e += 256) {
                const float v = dif[e] * f;
                const int col = (head0 + r) * p.dv + e;
                if (FUSED) a.out_x[col] = v;
                else {
                    unsigned char* o = (unsigned char*)a.out.p + row_operand_off(a.out_kind, a.out.chunks, m, col);
                    if (a.out_kind == WK_BF16) *(__nv_bfloat16*)o = __float2bfloat16_rn(v);
                    else *(float*)o = v;
                }
            }
        }
        cluster_arrive_release();
        cluster_wait_acquire();
        return;
    }
    if (S > 1) {
        cluster_arrive_release();
        cluster_wait_acquire();
        const uint32_t ml = smem_u32(m_s);
        if (tid < nr) {
            float M = -INFINITY, Ls = 0.0f;
            for (int s = 0; s < S; s++) M = fmaxf(M, cluster_ld_f32(cluster_map(ml + tid * 4, (uint32_t)s)));
            for (int s = 0; s < S; s++) {
                const float ms = cluster_ld_f32(cluster_map(ml + tid * 4, (uint32_t)s)), c = ms == -INFINITY ? 0.0f : expf(ms - M);
                Ls = fmaf(cluster_ld_f32(cluster_map(ml + 32 + tid * 4, (uint32_t)s)), c, Ls);
                wgt[s * kBdR + tid] = c;
            }
            for (int s = 0; s < S; s++) wgt[s * kBdR + tid] *= 1.0f / Ls;
        }
    } else if (tid < nr) {
        wgt[tid] = 1.0f / l_s[tid];
    }
    __syncthreads();
    const uint32_t ob = smem_u32(o_s);
    for (int i = S > 1 ? tid * S + sp : tid; i < nr * p.dvp; i += S > 1 ? 256 * S : 256) {
        const int r = i / p.dvp, e = i - r * p.dvp;
        if (e >= p.dv) continue;
        float v = 0.0f;
        if (S > 1) for (int s = 0; s < S; s++) v = fmaf(cluster_ld_f32(cluster_map(ob + i * 4, (uint32_t)s)), wgt[s * kBdR + r], v);
        else v = o_s[i] * wgt[r];
        const int col = (head0 + r) * p.dv + e;
        if (FUSED) a.out_x[col] = v;
        else {
            unsigned char* o = (unsigned char*)a.out.p + row_operand_off(a.out_kind, a.out.chunks, m, col);
            if (a.out_kind == WK_BF16) *(__nv_bfloat16*)o = __float2bfloat16_rn(v);
            else *(float*)o = v;
        }
    }
    if (S > 1) { cluster_arrive_release(); cluster_wait_acquire(); }
}

bool band_supported(int n_q, int n_kv, int dkp, int dvp) {
    return n_kv > 0 && n_q % n_kv == 0 && dkp % 16 == 0 && dvp % 16 == 0 && dkp <= 1024 && dvp <= 512 && (size_t)bd_layout(dkp, dvp).total * 4 <= 200 * 1024;
}

static cudaError_t launch_band(const BandArgs& a_in, int rows, bool fused, int sm_count, cudaStream_t st) {
    BandArgs a = a_in;
    if (a.p.maps < 1) a.p.maps = 1;
    const QkvArgs& p = a.p;
    if (p.maps > 2 || (p.maps == 2 && fused && !p.per_head)) return cudaErrorInvalidValue;
    if (!band_supported(p.n_q, p.n_kv, p.dkp, p.dvp) || rows <= 0) return cudaErrorInvalidValue;
    const int R = p.n_q / p.n_kv;
    int HB = (R + kBdR - 1) / kBdR;
    const size_t smem = (size_t)bd_layout(p.dkp, p.dvp).total * 4;
#define LUM_BAND_FNS(BF) {{(const void*)attn_band<BF, 0, 4>, (const void*)attn_band<BF, 0, 8>}, {(const void*)attn_band<BF, 1, 4>, (const void*)attn_band<BF, 1, 8>}, \
                          {(const void*)attn_band<BF, 2, 4>, (const void*)attn_band<BF, 2, 8>}}
    static const void* const fns[2][3][2] = {LUM_BAND_FNS(false), LUM_BAND_FNS(true)};
#undef LUM_BAND_FNS
    const void* fn = fns[a.kv_bf16 ? 1 : 0][fused ? (p.per_head ? 2 : 1) : 0][R > 4 ? 1 : 0];
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) return e;
    }
    // splits: enough CTAs for the SMs, none shorter than half a tile of keys at full reach
    const int mask = a.chunk > 0 ? a.chunk : a.window, reach = mask > 0 && mask < a.max_seq ? mask : a.max_seq;
    static const int env_s = [] { const char* e = getenv("LUM_BAND_SPLITS"); return e ? atoi(e) : kBdMaxSplits; }();
    int S = 1;
    while (S < env_s && S * p.maps < kBdMaxSplits && (long long)p.n_kv * p.maps * HB * rows * S * 2 <= sm_count && reach >= S * 2 * kBdTK / 2) S *= 2;
    const int C = S * p.maps;
    if (C > 8) {      // beyond the portable cluster size
        const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
        if (e != cudaSuccess) return e;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(C, p.n_kv * HB, rows); cfg.blockDim = dim3(256); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute at[2];
    int na = 0;
    if (a.use_pdl && fused) { at[na].id = cudaLaunchAttributeProgrammaticStreamSerialization; at[na].val.programmaticStreamSerializationAllowed = 1; na++; }
    if (C > 1) { at[na].id = cudaLaunchAttributeClusterDimension; at[na].val.clusterDim.x = C; at[na].val.clusterDim.y = 1; at[na].val.clusterDim.z = 1; na++; }
    cfg.attrs = at; cfg.numAttrs = na;
    void* params[] = {&a, &S, &HB};
    return cudaLaunchKernelExC(&cfg, fn, params);
}
cudaError_t launch_band_rows(const BandArgs& a, int sm_count, cudaStream_t st) {
    // (gridDim.z is limited to 65535 rows: far above the rows of a pass)
    return launch_band(a, a.M, false, sm_count, st);
}
cudaError_t launch_band_decode(const BandArgs& a, int sm_count, cudaStream_t st) { return launch_band(a, 1, true, sm_count, st); }

}  // namespace lum
