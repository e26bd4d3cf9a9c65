// Gated linear recurrences behind a short convolution, and the convolution's memory.
//
//   conv_tail     after a pass of many rows of one sequence: the last projected values of every channel go to the sequence's ring
//   recur_step    rows of different sequences (a decode step: one): convolution, the gates' block-diagonal products, the recurrence and
//                 the multiplication with the other branch in one kernel
//   recur_conv    many rows of one sequence: the convolved values, also as the operand of the gates' product (dense_gemm, one group
//                 per block; two bf16 terms, so that the gates are as exact as their weights)
//   recur_scan    ... and the recurrence over those rows: the time axis is cut into pieces whose (decay, sum) pairs are combined by a
//                 scan, tile by tile
// Everything is computed in f32; the state is f32.  It starts at zero at position 0, whatever the slot held before.
#include <cuda_bf16.h>

#include "lum_gemv_dev.cuh"
#include "lum_dense.cuh"

namespace lum {

namespace {
__device__ __forceinline__ float softplus_exact(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
// Decay and input of one step; sp = softplus(lam), r and i before their sigmoids.  Decays are kept as e = a - 1: close to 1, a itself has
// lost the digits that decide how far back a channel remembers, and 1 - a^2 = -e (2 + e).
__device__ __forceinline__ void recur_gate(float r, float i, float u, float sp, float& e_out, float& b) {
    const float e = expm1f(-8.0f * sigmoid(r) * sp);
    float g;
    asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(g) : "f"(-e * (2.0f + e)));
    b = g * sigmoid(i) * u;
    e_out = e;
}
// a s + b
__device__ __forceinline__ float recur_next(float e, float s, float b) { return s + fmaf(e, s, b); }
__device__ __forceinline__ uint32_t pack_bf16(float x, float y) {
    const __nv_bfloat162 b = __floats2bfloat162_rn(x, y);
    return *(const uint32_t*)&b;
}
}  // namespace

// ------------------------------------------------------------------------------------------------ the convolution's memory
__global__ void __launch_bounds__(256) conv_tail(const ConvTailArgs a) {
    const int m = a.M - 1 - (int)blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
    if (m < 0 || c >= a.n_ch) return;
    a.conv.ring[((size_t)a.seq * a.conv.taps + a.row_pos[m] % a.conv.taps) * a.conv.ch + c] = a.src[(size_t)m * a.ld + c];
}
cudaError_t launch_conv_tail(const ConvTailArgs& a, cudaStream_t st) {
    if (a.conv.taps <= 0) return cudaSuccess;
    if (a.M <= 0 || a.n_ch <= 0) return cudaErrorInvalidValue;
    conv_tail<<<dim3((a.n_ch + 255) / 256, a.conv.taps < a.M ? a.conv.taps : a.M), 256, 0, st>>>(a);
    return cudaGetLastError();
}

// ------------------------------------------------------------------------------------------------ one step
// CTA = (block of the gates, 4 groups of 8 channels: a warp each) x 4 rows.  Lanes are 4 groups of K x 8 channels; the first chunks' weights
// are asked for before the projection's results are waited for.
namespace { constexpr int kRsRows = 4, kRsWarps = 4, kRsPre = 4, kRsConv = 4; }
template <int KIND>
__global__ void __launch_bounds__(kRsWarps * 32) recur_step(const RecurArgs a) {
    constexpr int E = KIND == WK_BF16 ? 8 : 4, CK = KIND == WK_BF16 ? 64 : 32;
    extern __shared__ __align__(16) float rs_u[];             // [rows][kc * CK]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int rgb = a.bwp / 8, per = (rgb + kRsWarps - 1) / kRsWarps;
    const int blk = blockIdx.x / per, part = blockIdx.x - blk * per, pg = part * kRsWarps + warp;      // pg: this warp's group of 8 channels
    const int m0 = blockIdx.y * kRsRows, nr = min(kRsRows, a.M - m0), KL = a.kc * CK;
    const bool has = pg < rgb;
    const int rg_r = blk * 2 * rgb + pg, rg_i = rg_r + rgb, RG = a.nt / 8;
    auto weights = [&](int c, uint4 (&w)[4]) {
        const uint4* base = (const uint4*)a.w_gate + (size_t)c * RG * 64 + lane;
        w[0] = __ldg(base + (size_t)rg_r * 64); w[1] = __ldg(base + (size_t)rg_r * 64 + 32);
        w[2] = __ldg(base + (size_t)rg_i * 64); w[3] = __ldg(base + (size_t)rg_i * 64 + 32);
    };
    uint4 pre[kRsPre][4];
    pdl_launch_dependents();
    if (has) {
#pragma unroll
        for (int c = 0; c < kRsPre; c++) if (c < a.kc) weights(c, pre[c]);
    }
    // what else does not depend on the step: this lane's channel (of row lane / 8) in the recurrence, the convolution's weights
    const int grp = lane >> 3, kb = pg * 8 + (lane & 7), c = blk * a.bw + kb, m = m0 + grp;
    const bool mine = has && grp < nr && kb < a.bw;
    const float rb = mine ? a.r_b[c] : 0.0f, ib = mine ? a.i_b[c] : 0.0f, lam = mine ? a.lam[c] : 0.0f;
    const bool four = a.conv.taps == 4 && KL <= kRsConv * kRsWarps * 32;
    float4 cw[kRsConv];
    float cb[kRsConv];
    if (four) {
#pragma unroll
        for (int i = 0; i < kRsConv; i++) {
            const int k = tid + i * kRsWarps * 32;
            cw[i] = k < a.bw ? __ldg((const float4*)a.conv.w + blk * a.bw + k) : make_float4(0.f, 0.f, 0.f, 0.f);
            cb[i] = k < a.bw && a.conv_b ? a.conv_b[blk * a.bw + k] : 0.0f;
        }
    }
    const float sp = softplus_exact(lam);
    pdl_grid_wait();

    int pos[kRsRows], seq[kRsRows];
    bool bad = false;
#pragma unroll
    for (int r = 0; r < kRsRows; r++) {
        pos[r] = r < nr ? (a.step ? a.step->pos : a.row_pos[m0 + r]) : 0;
        seq[r] = r < nr && a.row_seq ? a.row_seq[m0 + r] : a.seq0;
        bad = bad || pos[r] < 0 || pos[r] >= a.max_seq || seq[r] < 0 || seq[r] >= a.max_batch;
    }
    if (bad) {
        if (tid == 0) atomicOr(a.status, LUM_ST_BAD_POS);
        return;
    }
    int my_pos = pos[0], my_seq = seq[0];
#pragma unroll
    for (int r = 1; r < kRsRows; r++) if (grp == r) { my_pos = pos[r]; my_seq = seq[r]; }
    float* S = a.state + (size_t)my_seq * a.width + c;
    const float s_old = mine && my_pos > 0 ? *S : 0.0f, y = mine ? a.yx[(size_t)m * a.ld + c] : 0.0f;
    // ---- the block's inputs
    if (four) {
#pragma unroll
        for (int r = 0; r < kRsRows; r++) {
            if (r >= nr) continue;
            const float* src = a.yx + (size_t)(m0 + r) * a.ld + a.x_off + blk * a.bw;
            float* ring = a.conv.ring + (size_t)seq[r] * 4 * a.conv.ch + blk * a.bw;
            float x[kRsConv][4];
#pragma unroll
            for (int i = 0; i < kRsConv; i++) {
                const int k = tid + i * kRsWarps * 32;
#pragma unroll
                for (int d = 0; d < 4; d++) x[i][d] = k < a.bw && pos[r] >= d ? (d ? ring[(size_t)((pos[r] - d) & 3) * a.conv.ch + k] : src[k]) : 0.0f;
            }
#pragma unroll
            for (int i = 0; i < kRsConv; i++) {
                const int k = tid + i * kRsWarps * 32;
                if (k < KL) rs_u[r * KL + k] = fmaf(cw[i].w, x[i][0], fmaf(cw[i].z, x[i][1], fmaf(cw[i].y, x[i][2], cw[i].x * x[i][3]))) + cb[i];
                if (part == 0 && k < a.bw) ring[(size_t)(pos[r] & 3) * a.conv.ch + k] = x[i][0];       // (the row of the ring that no step of this position reads)
            }
        }
    } else
#pragma unroll
    for (int r = 0; r < kRsRows; r++) {
        if (r >= nr) continue;
        const float* src = a.yx + (size_t)(m0 + r) * a.ld + a.x_off;
        float* ring = a.conv.ring + (size_t)seq[r] * a.conv.taps * a.conv.ch;
        for (int k = tid; k < KL; k += kRsWarps * 32) {
            float u = 0.0f;
            if (k < a.bw) {
                const int ck = blk * a.bw + k;
                u = conv_at(a.conv, ring, src, 0, 0, pos[r], ck) + (a.conv_b ? a.conv_b[ck] : 0.0f);
                if (part == 0 && a.conv.taps > 0) ring[(size_t)(pos[r] % a.conv.taps) * a.conv.ch + ck] = src[ck];
            }
            rs_u[r * KL + k] = u;
        }
    }
    __syncthreads();
    if (!has) return;
    // ---- gates
    float ar[kRsRows], ai[kRsRows];
#pragma unroll
    for (int r = 0; r < kRsRows; r++) ar[r] = ai[r] = 0.0f;
    auto take = [&](int c, const uint4 (&w)[4]) {
#pragma unroll
        for (int h = 0; h < 2; h++) {
            float wr[E], wi[E];
            const uint32_t rv[4] = {w[h].x, w[h].y, w[h].z, w[h].w}, iv[4] = {w[2 + h].x, w[2 + h].y, w[2 + h].z, w[2 + h].w};
#pragma unroll
            for (int i = 0; i < 4; i++) {
                if (KIND == WK_BF16) {
                    wr[(2 * i) % E] = __uint_as_float(rv[i] << 16); wr[(2 * i + 1) % E] = __uint_as_float(rv[i] & 0xffff0000u);
                    wi[(2 * i) % E] = __uint_as_float(iv[i] << 16); wi[(2 * i + 1) % E] = __uint_as_float(iv[i] & 0xffff0000u);
                } else {
                    wr[i % E] = __uint_as_float(rv[i]); wi[i % E] = __uint_as_float(iv[i]);
                }
            }
#pragma unroll
            for (int r = 0; r < kRsRows; r++) {
                if (r < nr) {
                    const float* x = rs_u + r * KL + c * CK + h * 4 * E + grp * E;
#pragma unroll
                    for (int i = 0; i < E; i += 4) {
                        const float4 v = *(const float4*)(x + i);
                        ar[r] = fmaf(wr[i], v.x, ar[r]); ar[r] = fmaf(wr[i + 1], v.y, ar[r]); ar[r] = fmaf(wr[i + 2], v.z, ar[r]); ar[r] = fmaf(wr[i + 3], v.w, ar[r]);
                        ai[r] = fmaf(wi[i], v.x, ai[r]); ai[r] = fmaf(wi[i + 1], v.y, ai[r]); ai[r] = fmaf(wi[i + 2], v.z, ai[r]); ai[r] = fmaf(wi[i + 3], v.w, ai[r]);
                    }
                }
            }
        }
    };
#pragma unroll
    for (int c = 0; c < kRsPre; c++) if (c < a.kc) take(c, pre[c]);
    for (int c = kRsPre; c < a.kc; c++) {
        uint4 w[4];
        weights(c, w);
        take(c, w);
    }
    // ---- every lane has the sums of channel lane % 8 after two shuffles; lane group r finishes row r
    float vr = 0.0f, vi = 0.0f;
#pragma unroll
    for (int r = 0; r < kRsRows; r++) {
        ar[r] += __shfl_xor_sync(0xffffffffu, ar[r], 8); ar[r] += __shfl_xor_sync(0xffffffffu, ar[r], 16);
        ai[r] += __shfl_xor_sync(0xffffffffu, ai[r], 8); ai[r] += __shfl_xor_sync(0xffffffffu, ai[r], 16);
        if (grp == r) { vr = ar[r]; vi = ai[r]; }
    }
    if (!mine) return;
    float da, db;
    recur_gate(vr + rb, vi + ib, rs_u[grp * KL + kb], sp, da, db);
    const float s = recur_next(da, s_old, db);
    *S = s;
    const float v = s * y;
    if (a.out_x) { a.out_x[c] = v; return; }
    unsigned char* o = (unsigned char*)a.out.p + row_operand_off(a.out_kind, a.out.chunks, m, c);
    if (a.out_kind == WK_BF16) *(__nv_bfloat16*)o = __float2bfloat16_rn(v);
    else *(float*)o = v;
}
cudaError_t launch_recur_step(const RecurArgs& a_in, cudaStream_t st) {
    RecurArgs a = a_in;
    const int CK = chunk_elems(a.kind), per = (a.bwp / 8 + kRsWarps - 1) / kRsWarps;
    const size_t smem = (size_t)kRsRows * a.kc * CK * 4;
    if (a.M <= 0 || a.bwp % 8 || a.bw > a.bwp || a.bw > a.kc * CK || a.nt != a.blocks * 2 * a.bwp || smem > 200 * 1024) return cudaErrorInvalidValue;
    const void* fn = a.kind == WK_BF16 ? (const void*)recur_step<WK_BF16> : (const void*)recur_step<WK_F32>;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) return e;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.blocks * per, (a.M + kRsRows - 1) / kRsRows); cfg.blockDim = dim3(kRsWarps * 32); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization; at[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at; cfg.numAttrs = a.use_pdl ? 1 : 0;
    void* params[] = {&a};
    return cudaLaunchKernelExC(&cfg, fn, params);
}

// ------------------------------------------------------------------------------------------------ many rows of one sequence
// Thread = row x 8 channels of a block (16 bytes of a bf16 operand); lanes are 8 rows x 4 groups of channels.
template <int KIND>
__global__ void __launch_bounds__(256) recur_conv(const RecurArgs a) {
    const int gpb = a.bwp / 8, groups = a.blocks * gpb;
    const int lane = threadIdx.x & 31, g = (blockIdx.x * 8 + (threadIdx.x >> 5)) * 4 + (lane >> 3), m = blockIdx.y * 8 + (lane & 7);
    if (g >= groups || m >= a.M) return;
    const int blk = g / gpb, k0 = (g - blk * gpb) * 8, c0 = blk * a.bw + k0;
    const int pos = a.row_pos[m];
    const float* src = a.yx + (size_t)m * a.ld + a.x_off;
    float u[8];
    {
        const float* ring = a.conv.ring + (size_t)a.seq0 * a.conv.taps * a.conv.ch;
#pragma unroll
        for (int i = 0; i < 8; i++) u[i] = k0 + i < a.bw ? conv_at(a.conv, ring, src, a.ld, m, pos, c0 + i) + (a.conv_b ? a.conv_b[c0 + i] : 0.0f) : 0.0f;
    }
    float* uo = a.u + (size_t)m * a.ldu + c0;
    if (k0 + 8 <= a.bw && ((a.ldu | c0) & 3) == 0) {
        ((float4*)uo)[0] = make_float4(u[0], u[1], u[2], u[3]);
        ((float4*)uo)[1] = make_float4(u[4], u[5], u[6], u[7]);
    } else {
#pragma unroll
        for (int i = 0; i < 8; i++) if (k0 + i < a.bw) uo[i] = u[i];
    }
    const int kcol = blk * a.kc * (KIND == WK_BF16 ? 64 : 32) + k0;
    const size_t o = row_operand_off(KIND, a.hi.chunks, m, kcol);
    if (KIND == WK_BF16) {
        uint32_t h[4], l[4];
#pragma unroll
        for (int i = 0; i < 4; i++) {
            h[i] = pack_bf16(u[2 * i], u[2 * i + 1]);
            l[i] = pack_bf16(u[2 * i] - __uint_as_float(h[i] << 16), u[2 * i + 1] - __uint_as_float(h[i] & 0xffff0000u));
        }
        *(uint4*)((unsigned char*)a.hi.p + o) = make_uint4(h[0], h[1], h[2], h[3]);
        *(uint4*)((unsigned char*)a.lo.p + o) = make_uint4(l[0], l[1], l[2], l[3]);
    } else {
        float4* f = (float4*)((unsigned char*)a.hi.p + o);
        f[0] = make_float4(u[0], u[1], u[2], u[3]);
        f[1] = make_float4(u[4], u[5], u[6], u[7]);
    }
}
// The same for four taps and blocks of whole groups of 8 channels: thread = 4 channels x 8 rows, the window slides in registers.
template <int KIND>
__global__ void __launch_bounds__(256) recur_conv4(const RecurArgs a) {
    const int c0 = (blockIdx.x * 256 + threadIdx.x) * 4, m0 = blockIdx.y * 8, nr = min(8, a.M - m0);
    if (c0 >= a.width) return;
    const int blk = c0 / a.bw, k0 = blk * a.kc * (KIND == WK_BF16 ? 64 : 32) + (c0 - blk * a.bw), pos0 = a.row_pos[0];
    const float* src = a.yx + a.x_off + c0;
    const float* ring = a.conv.ring + (size_t)a.seq0 * 4 * a.conv.ch + c0;
    float4 w[4], x[11];
#pragma unroll
    for (int i = 0; i < 4; i++) w[i] = *(const float4*)(a.conv.w + (size_t)(c0 + i) * 4);
    const float4 b = a.conv_b ? *(const float4*)(a.conv_b + c0) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < 11; r++) {
        const int m = m0 + r - 3;
        x[r] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (m >= 0) { if (r - 3 < nr) x[r] = *(const float4*)(src + (size_t)m * a.ld); }
        else if (pos0 + m >= 0) x[r] = *(const float4*)(ring + (size_t)((pos0 + m) & 3) * a.conv.ch);
    }
#pragma unroll
    for (int r = 0; r < 8; r++) {
        if (r >= nr) continue;
        float4 u;
        u.x = fmaf(w[0].w, x[r + 3].x, fmaf(w[0].z, x[r + 2].x, fmaf(w[0].y, x[r + 1].x, w[0].x * x[r].x))) + b.x;
        u.y = fmaf(w[1].w, x[r + 3].y, fmaf(w[1].z, x[r + 2].y, fmaf(w[1].y, x[r + 1].y, w[1].x * x[r].y))) + b.y;
        u.z = fmaf(w[2].w, x[r + 3].z, fmaf(w[2].z, x[r + 2].z, fmaf(w[2].y, x[r + 1].z, w[2].x * x[r].z))) + b.z;
        u.w = fmaf(w[3].w, x[r + 3].w, fmaf(w[3].z, x[r + 2].w, fmaf(w[3].y, x[r + 1].w, w[3].x * x[r].w))) + b.w;
        *(float4*)(a.u + (size_t)(m0 + r) * a.ldu + c0) = u;
        const size_t o = row_operand_off(KIND, a.hi.chunks, m0 + r, k0);
        if (KIND == WK_BF16) {
            const uint32_t h0 = pack_bf16(u.x, u.y), h1 = pack_bf16(u.z, u.w);
            *(uint2*)((unsigned char*)a.hi.p + o) = make_uint2(h0, h1);
            *(uint2*)((unsigned char*)a.lo.p + o) = make_uint2(pack_bf16(u.x - __uint_as_float(h0 << 16), u.y - __uint_as_float(h0 & 0xffff0000u)),
                                                              pack_bf16(u.z - __uint_as_float(h1 << 16), u.w - __uint_as_float(h1 & 0xffff0000u)));
        } else {
            *(float4*)((unsigned char*)a.hi.p + o) = u;
        }
    }
}
cudaError_t launch_recur_conv(const RecurArgs& a, cudaStream_t st) {
    const int groups = a.blocks * a.bwp / 8;
    if (a.M <= 0 || a.row_seq || a.hi.chunks != a.blocks * a.kc || (a.kind == WK_BF16 && (!a.lo.p || a.lo.chunks != a.hi.chunks))) return cudaErrorInvalidValue;
    if (a.conv.taps == 4 && a.bw % 8 == 0 && ((a.ld | a.x_off | a.ldu | a.conv.ch) & 3) == 0) {
        const dim3 g4((a.width / 4 + 255) / 256, (a.M + 7) / 8);
        if (a.kind == WK_BF16) recur_conv4<WK_BF16><<<g4, 256, 0, st>>>(a);
        else recur_conv4<WK_F32><<<g4, 256, 0, st>>>(a);
        return cudaGetLastError();
    }
    const dim3 grid((groups + 31) / 32, (a.M + 7) / 8);
    if (a.kind == WK_BF16) recur_conv<WK_BF16><<<grid, 256, 0, st>>>(a);
    else recur_conv<WK_F32><<<grid, 256, 0, st>>>(a);
    return cudaGetLastError();
}

// CTA = 16 channels; thread = channel x 8 consecutive rows, 32 such pieces = a tile of 256 rows.  A piece is (product of decays, sum); one
// warp per channel scans the 32 pieces, then every thread goes through its rows again from the right start.
namespace { constexpr int kScCh = 16, kScSeg = 32, kScT = 8, kScThreads = kScCh * kScSeg, kScTile = kScSeg * kScT; }
__global__ void __launch_bounds__(kScThreads, 2) recur_scan(const RecurArgs a) {
    __shared__ float ag_a[kScCh][kScSeg + 1], ag_b[kScCh][kScSeg + 1], out[kScTile][kScCh + 1];
    const int tid = threadIdx.x, ch = tid % kScCh, seg = tid / kScCh, warp = tid >> 5, lane = tid & 31;
    const int c = blockIdx.x * kScCh + ch, cl = min(c, a.width - 1);
    const int blk = cl / a.bw, gr = blk * 2 * a.bwp + (cl - blk * a.bw), gi = gr + a.bwp;
    const float rb = a.r_b[cl], ib = a.i_b[cl], sp = softplus_exact(a.lam[cl]);
    const int pos0 = a.row_pos[0];
    float carry = 0.0f;                                        // of channel `warp`, in every lane of the warp
    const int cw = blockIdx.x * kScCh + warp;
    if (pos0 > 0 && cw < a.width) carry = a.state[(size_t)a.seq0 * a.width + cw];
    for (int t0 = 0; t0 < a.M; t0 += kScTile) {
        const int r0 = t0 + seg * kScT;
        float da[kScT], db[kScT], y[kScT];
        const bool whole = t0 + kScTile <= a.M;
        if (whole) {
            const float *pr = a.gates + (size_t)r0 * a.ldg + gr, *pi = a.gates + (size_t)r0 * a.ldg + gi, *pu = a.u + (size_t)r0 * a.ldu + cl;
#pragma unroll
            for (int k = 0; k < kScT; k++) { da[k] = pr[k * a.ldg]; db[k] = pi[k * a.ldg]; y[k] = pu[k * a.ldu]; }
        } else {
#pragma unroll
            for (int k = 0; k < kScT; k++) {
                const size_t m = min(r0 + k, a.M - 1);
                da[k] = a.gates[m * a.ldg + gr]; db[k] = a.gates[m * a.ldg + gi]; y[k] = a.u[m * a.ldu + cl];
            }
        }
#pragma unroll
        for (int k = 0; k < kScT; k++) recur_gate(da[k] + rb, db[k] + ib, y[k], sp, da[k], db[k]);
        if (!whole) {
#pragma unroll
            for (int k = 0; k < kScT; k++) if (r0 + k >= a.M) da[k] = db[k] = 0.0f;
        }
        float A = 0.0f, B = 0.0f;                              // product of the piece's decays, minus one, and its sum from zero
#pragma unroll
        for (int k = 0; k < kScT; k++) { A = recur_next(A, da[k], A); B = recur_next(da[k], B, db[k]); }
        ag_a[ch][seg] = A;
        ag_b[ch][seg] = B;
#pragma unroll
        for (int k = 0; k < kScT; k++) y[k] = a.yx[(size_t)(whole ? r0 + k : min(r0 + k, a.M - 1)) * a.ld + cl];
        __syncthreads();
        {
            float pa = ag_a[warp][lane], pb = ag_b[warp][lane];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float qa = __shfl_up_sync(0xffffffffu, pa, o), qb = __shfl_up_sync(0xffffffffu, pb, o);
                if (lane >= o) { pb = recur_next(pa, qb, pb); pa = recur_next(pa, qa, pa); }
            }
            const float end = recur_next(pa, carry, pb);             // state after piece `lane`
            const float before = __shfl_up_sync(0xffffffffu, end, 1);
            ag_b[warp][lane] = lane ? before : carry;
            carry = __shfl_sync(0xffffffffu, end, 31);
        }
        __syncthreads();
        float s = ag_b[ch][seg];
#pragma unroll
        for (int k = 0; k < kScT; k++) {
            s = recur_next(da[k], s, db[k]);
            out[seg * kScT + k][ch] = s * y[k];
        }
        __syncthreads();
        {   // 8 channels of a row per thread: 16 bytes of the operand
            const int m = tid % kScTile, h = tid / kScTile, k0 = blockIdx.x * kScCh + h * 8;
            if (t0 + m < a.M && k0 < a.width) {
                float f[8];
#pragma unroll
                for (int i = 0; i < 8; i++) f[i] = k0 + i < a.width ? out[m][h * 8 + i] : 0.0f;
                unsigned char* o = (unsigned char*)a.out.p + row_operand_off(a.out_kind, a.out.chunks, t0 + m, k0);
                if (a.out_kind == WK_BF16) *(uint4*)o = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
                else { ((float4*)o)[0] = make_float4(f[0], f[1], f[2], f[3]); ((float4*)o)[1] = make_float4(f[4], f[5], f[6], f[7]); }
            }
        }
    }
    if (lane == 0 && cw < a.width) a.state[(size_t)a.seq0 * a.width + cw] = carry;
}
cudaError_t launch_recur_scan(const RecurArgs& a, cudaStream_t st) {
    if (a.M <= 0 || a.row_seq) return cudaErrorInvalidValue;
    recur_scan<<<(a.width + kScCh - 1) / kScCh, kScThreads, 0, st>>>(a);
    return cudaGetLastError();
}

}  // namespace lum
