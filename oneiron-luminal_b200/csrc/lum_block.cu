// Row-wise kernels of decoder layers whose sublayers share one norm, and their attention: norms, query / key preparation with the
// cache append, and attention over a window with learned per-head temperature and distance bias.
//
//   norm_rows     RMS or layer norm of rows of the residual stream -> operand of the next product
//   qkv_rows      queries and keys normalised over the whole projection, queries scaled (score factor x temperature), values mixed
//                 with the first mixing layer's; keys and values rounded to the cache type and appended
//   attn_band     attention of single rows over the cache: any head sizes, any number of query heads per K/V head, f32 or bf16
//                 cache.  FUSED: one row, with all of qkv_rows in the prologue (a decode step's attention is one kernel).
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
        float v = (nr_row[k] - mean) * inv * a.norm.gain[k];
        return a.norm.bias ? v + a.norm.bias[k] : v;
    };
    if (a.kind == WK_BF16) {
        for (int g = tid; g < a.out.chunks * 8; g += 256) {
            float f[8];
            if (vec && g * 8 + 8 <= W) {
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    const float4 v = ((const float4*)nr_row)[g * 2 + h], gn = ((const float4*)a.norm.gain)[g * 2 + h];
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

// ------------------------------------------------------------------------------------------------ attention, row by row
// One CTA = (split of the visible keys, K/V head and block of up to 8 of its query heads, row).  64 keys at a time:
//   scores   4 lanes per key, each a share of the head dimension for all 8 queries; two shuffles; distance bias; shared memory
//   softmax  one warp per query head: running maximum and sum
//   values   thread = two value dimensions and a share of the keys
// A tile's key and value loads are all issued before anything of the previous tile is waited for again: the next tile's keys are in
// flight during this tile's softmax, its values during its scores.
// The splits of a row are the CTAs of a thread-block cluster and fold their (maximum, sum, vector) through its shared memory.
namespace {
constexpr int kBdTK = 64, kBdR = 8, kBdMaxSplits = 16;
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
template <bool BF16, bool FUSED, int RB>
__global__ void __launch_bounds__(256, 2) attn_band(const BandArgs a, int S, int HB) {
    extern __shared__ __align__(16) float bd[];
    const QkvArgs& p = a.p;
    const BdSmem L = bd_layout(p.dkp, p.dvp);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int sp = blockIdx.x, kvh = blockIdx.y / HB, hb = blockIdx.y % HB, m = blockIdx.z;
    const int R = p.n_q / p.n_kv, r0 = hb * kBdR, nr = min(kBdR, R - r0), head0 = kvh * R + r0;
    float *q_s = bd + L.q, *sc = bd + L.sc, *red = bd + L.red, *o_s = bd + L.o, *m_s = bd + L.ml, *l_s = m_s + 8, *c_s = m_s + 16;
    if (FUSED) { pdl_launch_dependents(); pdl_grid_wait(); }
    const int pos = FUSED ? a.state->pos : a.row_pos[m];
    const int seq = FUSED ? 0 : (a.row_seq ? a.row_seq[m] : a.seq0);
    if (pos < 0 || pos >= a.max_seq || seq < 0 || seq >= a.max_batch) {          // (the same for every CTA of the cluster)
        if (FUSED && tid == 0 && sp == 0) atomicOr(a.status, LUM_ST_BAD_POS);
        return;
    }
    const size_t k_row = (size_t)p.n_kv * p.dkp, v_row = (size_t)p.n_kv * p.dvp;

    if (FUSED) {
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
            q_s[i] = r < nr ? a.q[((size_t)m * p.n_q + head0 + r) * p.dkp + (i - r * p.dkp)] : 0.0f;
        }
    }
    if (tid < 8) { m_s[tid] = -INFINITY; l_s[tid] = 0.0f; }
    const int lo = (a.window > 0 && pos + 1 > a.window) ? pos + 1 - a.window : 0;
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
        return (const char*)a.k_cache + (kv_phys_row(a.pg, seq, FUSED ? 0 : a.max_seq, j) * k_row + (size_t)kvh * p.dkp) * esz;
    };
    using VRaw = typename BandPair<BF16>::type;
    auto value_pair = [&](int j) -> VRaw {
        const char* vr = (const char*)(bd + L.vnew);
        if (!(FUSED && j == pos)) vr = (const char*)a.v_cache + (kv_phys_row(a.pg, seq, FUSED ? 0 : a.max_seq, j) * v_row + (size_t)kvh * p.dvp) * esz;
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
    const QkvArgs& p = a.p;
    if (!band_supported(p.n_q, p.n_kv, p.dkp, p.dvp) || rows <= 0) return cudaErrorInvalidValue;
    const int R = p.n_q / p.n_kv;
    int HB = (R + kBdR - 1) / kBdR;
    const size_t smem = (size_t)bd_layout(p.dkp, p.dvp).total * 4;
    static const void* const fns[2][2][2] = {
        {{(const void*)attn_band<false, false, 4>, (const void*)attn_band<false, false, 8>}, {(const void*)attn_band<false, true, 4>, (const void*)attn_band<false, true, 8>}},
        {{(const void*)attn_band<true, false, 4>, (const void*)attn_band<true, false, 8>}, {(const void*)attn_band<true, true, 4>, (const void*)attn_band<true, true, 8>}}};
    const void* fn = fns[a.kv_bf16 ? 1 : 0][fused ? 1 : 0][R > 4 ? 1 : 0];
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) return e;
    }
    // splits: enough CTAs for the SMs, none shorter than half a tile of keys at full reach
    const int reach = a.window > 0 && a.window < a.max_seq ? a.window : a.max_seq;
    static const int env_s = [] { const char* e = getenv("LUM_BAND_SPLITS"); return e ? atoi(e) : kBdMaxSplits; }();
    int S = 1;
    while (S < env_s && S < kBdMaxSplits && (long long)p.n_kv * HB * rows * S * 2 <= sm_count && reach >= S * 2 * kBdTK / 2) S *= 2;
    if (S > 8) {      // beyond the portable cluster size
        const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
        if (e != cudaSuccess) return e;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(S, p.n_kv * HB, rows); cfg.blockDim = dim3(256); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute at[2];
    int na = 0;
    if (a.use_pdl && fused) { at[na].id = cudaLaunchAttributeProgrammaticStreamSerialization; at[na].val.programmaticStreamSerializationAllowed = 1; na++; }
    if (S > 1) { at[na].id = cudaLaunchAttributeClusterDimension; at[na].val.clusterDim.x = S; at[na].val.clusterDim.y = 1; at[na].val.clusterDim.z = 1; na++; }
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
