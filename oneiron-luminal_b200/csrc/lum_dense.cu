// Products with dense (bf16 / f32) weights in the chunked layout of lum_dense.cuh.
//
//   dense_gemv      one activation vector: HBM-bound, plain 16-byte loads straight from the layout (a warp's load is 512 contiguous
//                   bytes: 4 groups of K x 8 rows), norm in the prologue, residual / activation / greedy sample in the epilogue;
//                   a long K is split over the CTAs of a thread-block cluster, whose sums meet in shared memory
//   dense_gemm_tc   many rows, bf16: tcgen05.mma with both operands brought by one bulk copy per tile and chunk, accumulators
//                   double-buffered in tensor memory, the same epilogues per row
//   dense_gemm_f32  many rows, f32: CUDA cores, true 32-bit products and sums
#include <cuda_bf16.h>
#include <cstdlib>

#include "lum_gemv_dev.cuh"
#include "lum_dense.cuh"

namespace lum {

// ------------------------------------------------------------------------------------------------ layout
__device__ __forceinline__ float any_load(const void* p, uint32_t dtype, size_t i) {
    if (dtype == WK_BF16) return bf16_bits_to_f32(((const uint16_t*)p)[i]);
    if (dtype == 1u) return __half2float(((const __half*)p)[i]);
    return ((const float*)p)[i];
}
__global__ void __launch_bounds__(256) chunked_pack(const void* src, uint32_t src_dtype, size_t rows, size_t cols, unsigned char* dst, int kind, int nt, RowMap rm) {
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < rows * cols; i += (size_t)gridDim.x * 256) {
        const size_t n = i / cols, k = i - n * cols;
        unsigned char* o = dst + chunked_off(kind, nt, row_map(rm, n), k);
        if (kind == WK_BF16 && src_dtype == WK_BF16) *(uint16_t*)o = ((const uint16_t*)src)[i];
        else if (kind == WK_BF16) *(__nv_bfloat16*)o = __float2bfloat16_rn(any_load(src, src_dtype, i));
        else *(float*)o = any_load(src, src_dtype, i);
    }
}
__global__ void __launch_bounds__(256) chunked_unpack(const unsigned char* src, int kind, int nt, RowMap rm, size_t rows, size_t cols, float* f32, void* same) {
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < rows * cols; i += (size_t)gridDim.x * 256) {
        const size_t n = i / cols, k = i - n * cols;
        const unsigned char* o = src + chunked_off(kind, nt, row_map(rm, n), k);
        if (same) { if (kind == WK_BF16) ((uint16_t*)same)[i] = *(const uint16_t*)o; else ((float*)same)[i] = *(const float*)o; }
        else f32[i] = kind == WK_BF16 ? bf16_bits_to_f32(*(const uint16_t*)o) : *(const float*)o;
    }
}
static unsigned blocks_for(size_t n) { const size_t b = (n + 255) / 256; return (unsigned)(b < 1 ? 1 : b > 16384 ? 16384 : b); }
cudaError_t launch_chunked_pack(const void* src, uint32_t src_dtype, size_t rows, size_t cols, void* dst, int kind, int nt, RowMap rm, cudaStream_t st) {
    chunked_pack<<<blocks_for(rows * cols), 256, 0, st>>>(src, src_dtype, rows, cols, (unsigned char*)dst, kind, nt, rm);
    return cudaGetLastError();
}
cudaError_t launch_chunked_unpack(const void* src, int kind, int nt, RowMap rm, size_t rows, size_t cols, float* dst_f32, void* dst_same, cudaStream_t st) {
    chunked_unpack<<<blocks_for(rows * cols), 256, 0, st>>>((const unsigned char*)src, kind, nt, rm, rows, cols, dst_f32, dst_same);
    return cudaGetLastError();
}

// ------------------------------------------------------------------------------------------------ one vector
namespace {
constexpr int kDvThreads = 256, kDvWarps = 8, kDvRB = 4;      // row groups (of 8 rows) a warp carries at a time

template <int KIND> struct Elems;
template <> struct Elems<WK_BF16> { static constexpr int E = 8, CK = 64; };
template <> struct Elems<WK_F32> { static constexpr int E = 4, CK = 32; };

template <int KIND>
__device__ __forceinline__ float dot16(const uint4& w, const float* x, float acc) {
    if (KIND == WK_BF16) {
        const uint32_t v[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int i = 0; i < 4; i++) {
            acc = fmaf(__uint_as_float(v[i] << 16), x[2 * i], acc);
            acc = fmaf(__uint_as_float(v[i] & 0xffff0000u), x[2 * i + 1], acc);
        }
    } else {
        acc = fmaf(__uint_as_float(w.x), x[0], acc); acc = fmaf(__uint_as_float(w.y), x[1], acc);
        acc = fmaf(__uint_as_float(w.z), x[2], acc); acc = fmaf(__uint_as_float(w.w), x[3], acc);
    }
    return acc;
}
__device__ __forceinline__ uint4 ld_stream(const uint4* p) {      // weights are read once per step: do not keep them in L1
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
}  // namespace

// the residual streams of column n take in a sublayer's output
__device__ __forceinline__ void streams_take(const StreamArgs& h, int n, float y) {
    float old[kMaxStreams];
#pragma unroll
    for (int s = 0; s < kMaxStreams; s++) old[s] = s < h.n ? h.x[(size_t)s * h.ldx + n] : 0.0f;
    float u = 0.0f;
    for (int t = 0; t < h.n; t++) {
        float v = (h.out ? h.out[t] : 1.0f) * y;
        if (h.mix) {
#pragma unroll
            for (int s = 0; s < kMaxStreams; s++) if (s < h.n) v = fmaf(h.mix[s * h.n + t], old[s], v);
        } else {
            v += h.x[(size_t)t * h.ldx + n];
        }
        h.x[(size_t)t * h.ldx + n] = v;
        u = fmaf(h.next ? h.next[t] : 1.0f, v, u);
    }
    h.u[n] = u;
}

// grid = (row ranges) x (C CTAs of a cluster, each with a share of the chunks).  rl_max: row groups of the largest range.
template <int KIND, bool CL>
__global__ void __launch_bounds__(kDvThreads, 2) dense_gemv(const DenseArgs a, int C, int rl_max) {
    constexpr int E = Elems<KIND>::E, CK = Elems<KIND>::CK;
    extern __shared__ __align__(16) float dv_smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int cr = CL ? (int)(blockIdx.x % C) : 0, cq = CL ? (int)(blockIdx.x / C) : (int)blockIdx.x, Q = CL ? (int)(gridDim.x / C) : (int)gridDim.x;
    const int RG = a.nt / 8, gs = a.pair ? 2 : 1;             // pairs of row groups stay together
    const int rg0 = (int)((long long)cq * (RG / gs) / Q) * gs, rg1 = (int)((long long)(cq + 1) * (RG / gs) / Q) * gs;
    const int KC0 = a.seg[0].chunks, KC = KC0 + (a.nk > 1 ? a.seg[1].chunks : 0);
    const int c0 = (int)((long long)cr * KC / C), c1 = (int)((long long)(cr + 1) * KC / C);
    float* part = dv_smem;                                    // [8 warps][rl_max * 8]
    float* red = part + kDvWarps * rl_max * 8;                // [32]
    float* xs = red + 32;                                     // [(c1 - c0) * CK]

    pdl_launch_dependents();
    // items: (block of kDvRB row groups, chunk of this warp)
    const int nc = (c1 - c0 - warp + kDvWarps - 1) / kDvWarps, nrb = (rg1 - rg0 + kDvRB - 1) / kDvRB;
    const int n_items = nc > 0 ? nc * nrb : 0;
    auto load = [&](int item, uint4 (&v)[kDvRB][2]) {
        const int rb = item / nc, c = c0 + warp + (item - rb * nc) * kDvWarps;
        const bool second = c >= KC0;
        const unsigned char* base = (const unsigned char*)(second ? a.seg[1].w : a.seg[0].w) + (size_t)(second ? c - KC0 : c) * RG * 1024;
        const int g0 = rg0 + rb * kDvRB;
#pragma unroll
        for (int r = 0; r < kDvRB; r++) {
            if (g0 + r < rg1) {
                const uint4* p = (const uint4*)(base + (size_t)(g0 + r) * 1024) + lane;
                v[r][0] = ld_stream(p);
                v[r][1] = ld_stream(p + 32);
            } else {
                v[r][0] = v[r][1] = make_uint4(0u, 0u, 0u, 0u);
            }
        }
    };
    uint4 cur[kDvRB][2], nxt[kDvRB][2];
    if (n_items > 0) load(0, cur);                             // weights do not depend on the kernel before: ask for the first ones now
    pdl_grid_wait();

    // ---- activations of this CTA's chunks -> shared memory
    if (a.norm.mode != NORM_NONE) {                            // (one segment, C == 1)
        const int W = a.norm.width;
        const float* x = a.seg[0].x;
        float s = 0.0f;
        for (int i = tid; i < KC * CK; i += kDvThreads) { const float v = i < W ? x[i] : 0.0f; xs[i] = v; s += v; }
        float mean = 0.0f;
        if (a.norm.mode == NORM_LAYER) mean = block_sum(s, red, tid, kDvThreads, 1) / (float)W;
        s = 0.0f;
        for (int i = tid; i < W; i += kDvThreads) { const float d = xs[i] - mean; s = fmaf(d, d, s); }
        const float inv = 1.0f / sqrtf(block_sum(s, red, tid, kDvThreads, 1) / (float)W + a.norm.eps);
        for (int i = tid; i < W; i += kDvThreads) {
            float v = (xs[i] - mean) * inv * (a.norm.gain0 + a.norm.gain[i]);
            if (a.norm.bias) v += a.norm.bias[i];
            xs[i] = v;
        }
    } else {
        for (int i = tid; i < (c1 - c0) * (CK / 4); i += kDvThreads) {
            const int c = c0 + i / (CK / 4), o = i % (CK / 4);
            const float* src = c >= KC0 ? a.seg[1].x + (size_t)(c - KC0) * CK : a.seg[0].x + (size_t)c * CK;
            ((float4*)xs)[i] = *((const float4*)src + o);
        }
    }
    __syncthreads();

    // ---- weights
    float acc[kDvRB];
#pragma unroll
    for (int r = 0; r < kDvRB; r++) acc[r] = 0.0f;
    const int grp = lane >> 3;
    int ci = 0, rb = 0;
#pragma unroll 1
    for (int item = 0; item < n_items; item++) {
        if (item + 1 < n_items) load(item + 1, nxt);
        const float* xp = xs + (size_t)(warp + ci * kDvWarps) * CK + grp * E;
#pragma unroll
        for (int h = 0; h < 2; h++) {
            float x[E];
#pragma unroll
            for (int i = 0; i < E / 4; i++) *(float4*)&x[4 * i] = *(const float4*)(xp + h * 4 * E + 4 * i);
#pragma unroll
            for (int r = 0; r < kDvRB; r++) acc[r] = dot16<KIND>(cur[r][h], x, acc[r]);
        }
        if (++ci == nc) {
#pragma unroll
            for (int r = 0; r < kDvRB; r++) {
                float v = acc[r];
                v += __shfl_xor_sync(0xffffffffu, v, 8);
                v += __shfl_xor_sync(0xffffffffu, v, 16);
                if (lane < 8 && rg0 + rb * kDvRB + r < rg1) part[(size_t)warp * rl_max * 8 + (rb * kDvRB + r) * 8 + lane] = v;
                acc[r] = 0.0f;
            }
            ci = 0;
            rb++;
        }
#pragma unroll
        for (int r = 0; r < kDvRB; r++) { cur[r][0] = nxt[r][0]; cur[r][1] = nxt[r][1]; }
    }
    if (n_items == 0)
        for (int i = lane; i < (rg1 - rg0) * 8; i += 32) part[(size_t)warp * rl_max * 8 + i] = 0.0f;
    __syncthreads();

    // ---- sums of the warps (and of the cluster's CTAs), epilogue
    const int n_rows = (rg1 - rg0) * 8;
    if (CL) {
        for (int i = tid; i < n_rows; i += kDvThreads) {
            float v = 0.0f;
#pragma unroll
            for (int w = 0; w < kDvWarps; w++) v += part[(size_t)w * rl_max * 8 + i];
            part[i] = v;                                       // (slot i of warp 0: read and written by this thread only)
        }
        __syncthreads();
        cluster_arrive_release();
        cluster_wait_acquire();
    }
    if (a.pair) {                                              // (no cluster) gate rows i, up rows i + 8
        for (int j = tid; j < n_rows / 2; j += kDvThreads) {
            const int i = (j >> 3) * 16 + (j & 7);
            float g = 0.0f, u = 0.0f;
#pragma unroll
            for (int w = 0; w < kDvWarps; w++) { g += part[(size_t)w * rl_max * 8 + i]; u += part[(size_t)w * rl_max * 8 + i + 8]; }
            a.act_x[rg0 * 4 + j] = clamped_gate(g, u, a.limit);
        }
        return;
    }
    float sp = 0.0f, sq = 0.0f;
    if (a.act_row0 < a.nt) { sp = softplus(a.act_par[0]); sq = softplus(a.act_par[1]); }
    ArgBest best{-INFINITY, -1};
    for (int i = CL ? tid * C + cr : tid; i < n_rows; i += CL ? kDvThreads * C : kDvThreads) {
        float v = 0.0f;
        if (CL) {
            const uint32_t p = smem_u32(part + i);
            for (int r = 0; r < C; r++) v += cluster_ld_f32(cluster_map(p, (uint32_t)r));
        } else {
#pragma unroll
            for (int w = 0; w < kDvWarps; w++) v += part[(size_t)w * rl_max * 8 + i];
        }
        const int n = rg0 * 8 + i;
        if (a.bias) v += a.bias[n];
        if (n >= a.act_row0) a.act_x[n - a.act_row0] = xielu(v, sp, sq);
        else if (n < a.n_real) {
            if (a.epi == DENSE_STREAMS) streams_take(a.hc, n, v);
            else if (a.epi == DENSE_RESID) a.y[n] = a.y[n] + a.mult * v;
            else {
                v *= a.mult;
                if (n < a.gelu_rows) v = gelu_tanh(v);
                a.y[n] = v;
                if (a.epi == DENSE_ARGMAX) argbest_take(best, v, n);
            }
        }
    }
    if (CL) { cluster_arrive_release(); cluster_wait_acquire(); }      // another CTA may still be reading this one's sums
    if (a.epi == DENSE_ARGMAX) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best.v, o);
            const int oi = __shfl_xor_sync(0xffffffffu, best.i, o);
            argbest_take(best, ov, oi);
        }
        __syncthreads();
        if (lane == 0) { red[warp] = best.v; ((int*)red)[16 + warp] = best.i; }
        __syncthreads();
        if (tid == 0) for (int w = 1; w < kDvWarps; w++) argbest_take(best, red[w], ((int*)red)[16 + w]);
        argmax_finish(a.am, best, tid, kDvThreads, 1);
    }
}

cudaError_t launch_dense_gemv(const DenseArgs& a_in, int sm_count, cudaStream_t st) {
    DenseArgs a = a_in;
    if (a.nk < 1 || a.nk > 2 || a.nt <= 0 || a.nt % 8 || a.grp_rows || (a.kind != WK_BF16 && a.kind != WK_F32)) return cudaErrorInvalidValue;
    if (a.epi == DENSE_STREAMS && (a.hc.n < 1 || a.hc.n > kMaxStreams)) return cudaErrorInvalidValue;
    if (a.norm.mode != NORM_NONE && (a.nk != 1 || a.norm.width > a.seg[0].chunks * chunk_elems(a.kind))) return cudaErrorInvalidValue;
    const int RG = a.nt / 8, KC = a.seg[0].chunks + (a.nk > 1 ? a.seg[1].chunks : 0);
    // A long K: split over a cluster of two, so that a CTA has whole shares of both K and the rows and loads half of the vector
    // (measured on 4096 rows x K 25600: 39 us; a cluster of 8: 64 us; a whole decode step with 1 / 2 / 4 / 8: 1118 / 935 / 1124 / 1149 us)
    int C = 1;
    if (a.norm.mode == NORM_NONE && a.epi != DENSE_ARGMAX && !a.pair && KC >= 32) C = 2;
    static const int env_c = [] { const char* e = getenv("LUM_DENSE_CLUSTER"); return e ? atoi(e) : 0; }();
    if ((env_c == 1 || env_c == 2 || env_c == 4 || env_c == 8) && a.norm.mode == NORM_NONE && a.epi != DENSE_ARGMAX && !a.pair) C = env_c;
    int Q = 2 * sm_count / C;
    if (a.epi == DENSE_ARGMAX && Q > kArgmaxSlots) Q = kArgmaxSlots;
    // few rows: no more ranges than blocks of row groups a warp carries anyway would leave half of a warp's loads empty
    const int gs = a.pair ? 2 : 1;
    if (RG % gs || (a.pair && (a.epi != DENSE_STORE || C != 1))) return cudaErrorInvalidValue;
    if (Q > RG / gs) Q = RG / gs;
    if (Q < 1) Q = 1;
    const int rl = (RG / gs + Q - 1) / Q * gs, cl = (KC + C - 1) / C;
    const size_t smem = ((size_t)kDvWarps * rl * 8 + 32 + (size_t)cl * chunk_elems(a.kind)) * 4;
    if (smem > 220 * 1024) return cudaErrorInvalidValue;
    const void* fn = a.kind == WK_BF16 ? (C > 1 ? (const void*)dense_gemv<WK_BF16, true> : (const void*)dense_gemv<WK_BF16, false>)
                                       : (C > 1 ? (const void*)dense_gemv<WK_F32, true> : (const void*)dense_gemv<WK_F32, false>);
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
        if (e != cudaSuccess) return e;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(Q * C); cfg.blockDim = dim3(kDvThreads); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute at[2];
    int na = 0;
    if (a.use_pdl) { at[na].id = cudaLaunchAttributeProgrammaticStreamSerialization; at[na].val.programmaticStreamSerializationAllowed = 1; na++; }
    if (C > 1) { at[na].id = cudaLaunchAttributeClusterDimension; at[na].val.clusterDim.x = C; at[na].val.clusterDim.y = 1; at[na].val.clusterDim.z = 1; na++; }
    cfg.attrs = at; cfg.numAttrs = na;
    int c_arg = C, rl_arg = rl;
    void* params[] = {&a, &c_arg, &rl_arg};
    return cudaLaunchKernelExC(&cfg, fn, params);
}

// ------------------------------------------------------------------------------------------------ many rows
// 16 finished sums of row m: 8 gate rows and their 8 up rows, container rows n .. n + 15.
__device__ __forceinline__ void rows_epilogue_pair(const DenseArgs& a, int m, int n, const float (&g)[8], const float (&u)[8]) {
    float t[8];
#pragma unroll
    for (int i = 0; i < 8; i++) t[i] = clamped_gate(g[i], u[i], a.limit);
    unsigned char* o = (unsigned char*)a.act.p + row_operand_off(a.kind, a.act.chunks, m, n >> 1);
    if (a.kind == WK_BF16) {
        uint32_t w[4];
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(t[2 * i], t[2 * i + 1]);
            w[i] = *(const uint32_t*)&b;
        }
        *(uint4*)o = make_uint4(w[0], w[1], w[2], w[3]);
    } else {
        ((float4*)o)[0] = make_float4(t[0], t[1], t[2], t[3]);
        ((float4*)o)[1] = make_float4(t[4], t[5], t[6], t[7]);
    }
}
// Eight finished sums of row m, container rows n .. n + 7.
__device__ __forceinline__ void rows_epilogue8(const DenseArgs& a, int m, int n, float (&v)[8], float sp, float sq) {
    if (a.bias) {
#pragma unroll
        for (int i = 0; i < 8; i++) v[i] += a.bias[n + i];
    }
    if (n < a.gelu_rows) {                                    // (a multiple of 8; stored with factor 1)
#pragma unroll
        for (int i = 0; i < 8; i++) v[i] = gelu_tanh(v[i]);
    }
    if (n >= a.act_row0) {
        float t[8];
#pragma unroll
        for (int i = 0; i < 8; i++) t[i] = xielu(v[i], sp, sq);
        unsigned char* o = (unsigned char*)a.act.p + row_operand_off(a.kind, a.act.chunks, m, n - a.act_row0);
        if (a.kind == WK_BF16) {
            uint32_t w[4];
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const __nv_bfloat162 b = __floats2bfloat162_rn(t[2 * i], t[2 * i + 1]);
                w[i] = *(const uint32_t*)&b;
            }
            *(uint4*)o = make_uint4(w[0], w[1], w[2], w[3]);
        } else {
            ((float4*)o)[0] = make_float4(t[0], t[1], t[2], t[3]);
            ((float4*)o)[1] = make_float4(t[4], t[5], t[6], t[7]);
        }
        return;
    }
    float* y = a.y + (size_t)m * a.ldy + n;
    if (a.epi == DENSE_STORE && (a.ldy & 7) == 0 && n + 8 <= a.ldy && ((uintptr_t)y & 31) == 0) {      // a whole sector at once
        asm volatile("st.global.v8.f32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(y), "f"(a.mult * v[0]), "f"(a.mult * v[1]), "f"(a.mult * v[2]), "f"(a.mult * v[3]),
                     "f"(a.mult * v[4]), "f"(a.mult * v[5]), "f"(a.mult * v[6]), "f"(a.mult * v[7]) : "memory");
        return;
    }
    if ((a.ldy & 3) == 0 && n + 8 <= a.ldy) {                 // rows padded to whole 16-byte groups: columns beyond n_real receive zeros
        float4 r0 = make_float4(0.f, 0.f, 0.f, 0.f), r1 = r0;
        if (a.epi == DENSE_RESID) { r0 = ((const float4*)y)[0]; r1 = ((const float4*)y)[1]; }
        ((float4*)y)[0] = make_float4(r0.x + a.mult * v[0], r0.y + a.mult * v[1], r0.z + a.mult * v[2], r0.w + a.mult * v[3]);
        ((float4*)y)[1] = make_float4(r1.x + a.mult * v[4], r1.y + a.mult * v[5], r1.z + a.mult * v[6], r1.w + a.mult * v[7]);
        return;
    }
#pragma unroll
    for (int i = 0; i < 8; i++)
        if (n + i < a.n_real) y[i] = (a.epi == DENSE_RESID ? y[i] : 0.0f) + a.mult * v[i];
}

namespace {
constexpr int kDmThreads = 192;               // producer warp, tensor-core warp, four epilogue warps
constexpr int kDmMaxStages = 16;
constexpr int kDmABytes = 128 * 128;          // 128 rows x one chunk

__host__ __device__ constexpr uint32_t dm_idesc(int N) {      // kind::f16, bf16 x bf16 -> f32, both operands K-major, M = 128
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
}
__device__ __forceinline__ void dm_umma(uint32_t tmem_d, uint64_t da, uint64_t db, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(tmem_d), "l"(da), "l"(db), "r"(idesc), "r"(accumulate)
        : "memory");
}
}  // namespace

// Persistent CTAs over tiles of 128 rows x TN container rows (tile t: row tile t % mt, so that CTAs running together share weights).
__global__ void __launch_bounds__(kDmThreads, 1) dense_gemm_tc(const DenseArgs a, int TN, int stages) {
    extern __shared__ __align__(128) unsigned char dm_smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int stage_bytes = kDmABytes + TN * 128;
    const uint32_t s_base = smem_u32(dm_smem);
    const uint32_t bars = s_base + stages * stage_bytes;      // full[16], empty[16], acc_full[2], acc_empty[2], drained, the slot, the abort word
    auto full = [&](int s) { return bars + s * 8; };
    auto empty = [&](int s) { return bars + 128 + s * 8; };
    auto acc_full = [&](int b) { return bars + 256 + b * 8; };
    auto acc_empty = [&](int b) { return bars + 272 + b * 8; };
    const uint32_t drained = bars + 288, slot = bars + 296;
    volatile int* abort = (volatile int*)(dm_smem + stages * stage_bytes + 304);
    if (tid == 0) {
        for (int s = 0; s < stages; s++) { mbar_init(full(s), 1); mbar_init(empty(s), 1); }
        for (int b = 0; b < 2; b++) { mbar_init(acc_full(b), 1); mbar_init(acc_empty(b), 128); }
        mbar_init(drained, 1);
        mbar_fence_init();
        *abort = 0;
    }
    const uint32_t cols = TN >= 256 ? 512u : (uint32_t)(2 * TN);
    if (warp == 1) tmem_alloc(slot, cols);
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = *(volatile uint32_t*)(dm_smem + stages * stage_bytes + 296);

    // column tiles: a tile's rows of the container belong to one group
    const int grp = a.grp_rows ? a.grp_rows : a.nt, tpg = (grp + TN - 1) / TN;
    const int mt = (a.M + 127) / 128, ntile = tpg * (a.nt / grp), n_tiles = mt * ntile;
    const int KC0 = a.seg[0].chunks, KC = KC0 + (a.nk > 1 ? a.seg[1].chunks : 0);

    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < n_tiles && ok; t += gridDim.x) {
                const int tm = t % mt, gi = (t / mt) / tpg, ng = (t / mt - gi * tpg) * TN, n0 = gi * grp + ng, ca = gi * a.grp_chunks;
                const int rows = min(128, ((a.M - tm * 128) + 7) & ~7), wrows = min(TN, grp - ng);
                const uint32_t ab = (uint32_t)rows * 128, bb = (uint32_t)wrows * 128;
                for (int c = 0; c < KC; c++, it++) {
                    const int s = it % stages;
                    if (it >= (uint32_t)stages && !mbar_wait_abortable(empty(s), ((it / stages) - 1) & 1, abort)) { ok = false; break; }
                    mbar_arrive_expect_tx(full(s), ab + bb);
                    const bool second = c >= KC0;
                    const int cc = second ? c - KC0 : c;
                    const DenseK& g = second ? a.seg[1] : a.seg[0];
                    bulk_g2s(s_base + s * stage_bytes, (const unsigned char*)g.a + ((size_t)tm * (g.a_chunks ? g.a_chunks : g.chunks) + ca + cc) * kDmABytes, ab, full(s));
                    bulk_g2s(s_base + s * stage_bytes + kDmABytes, (const unsigned char*)g.w + (size_t)cc * a.nt * 128 + (size_t)n0 * 128, bb, full(s));
                }
            }
            if (!ok) {
                *abort = 1;
                atomicOr(a.status, LUM_ST_WAIT_EMPTY);
                // copies in flight must land before this CTA's shared memory goes away
                for (uint32_t j = it > (uint32_t)stages ? it - stages : 0; j < it; j++)
                    if (!mbar_wait(full(j % stages), (j / stages) & 1)) atomicOr(a.status, LUM_ST_WAIT_DRAIN);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            uint32_t it = 0;
            int ti = 0;
            bool ok = true;
            const uint32_t idesc = dm_idesc(TN);
            for (int t = blockIdx.x; t < n_tiles && ok; t += gridDim.x, ti++) {
                const int b = ti & 1;
                if (ti >= 2 && !mbar_wait_abortable(acc_empty(b), ((ti >> 1) - 1) & 1, abort)) { ok = false; break; }
                tc_fence_after_sync();
                const uint32_t d = tmem + b * TN;
                for (int c = 0; c < KC; c++, it++) {
                    const int s = it % stages;
                    if (!mbar_wait_abortable(full(s), (it / stages) & 1, abort)) { ok = false; break; }
                    tc_fence_after_sync();
                    const uint32_t sa = s_base + s * stage_bytes, sb = sa + kDmABytes;
#pragma unroll
                    for (int k = 0; k < 4; k++)               // 16 elements of K = two 16-byte groups
                        dm_umma(d, umma_smem_desc(sa + k * 256, 128, 1024), umma_smem_desc(sb + k * 256, 128, 1024), idesc, (c | k) ? 1u : 0u);
                    umma_commit(empty(s));
                }
                if (ok) umma_commit(acc_full(b));
            }
            if (!ok) { *abort = 1; atomicOr(a.status, LUM_ST_WAIT_FULL); }
            umma_commit(drained);
            if (!mbar_wait(drained, 0)) atomicOr(a.status, LUM_ST_WAIT_TMEM);
        }
        __syncwarp();
    } else {
        const int q = warp & 3;                               // tensor-memory lanes 32 q .. of this warp
        float sp = 0.0f, sq = 0.0f;
        if (a.act_row0 < a.nt) { sp = softplus(a.act_par[0]); sq = softplus(a.act_par[1]); }
        int ti = 0;
        for (int t = blockIdx.x; t < n_tiles; t += gridDim.x, ti++) {
            const int b = ti & 1, tm = t % mt, gi = (t / mt) / tpg, n0 = gi * grp + (t / mt - gi * tpg) * TN, n1 = (gi + 1) * grp;
            int ok = mbar_wait_abortable(acc_full(b), (ti >> 1) & 1, abort) ? 1 : 0;
            if (!__all_sync(0xffffffffu, ok)) { *abort = 1; if (lane == 0) atomicOr(a.status, LUM_ST_WAIT_TMEM); break; }
            tc_fence_after_sync();
            const int m = tm * 128 + q * 32 + lane;
            const uint32_t base = tmem + b * TN + ((uint32_t)(q * 32) << 16);
#pragma unroll 1
            for (int cb = 0; cb < TN; cb += 32) {
                uint32_t v0[16], v1[16];
                tmem_ld16(base + cb, v0);
                tmem_ld16(base + cb + 16, v1);
                tmem_ld_wait();
                if (cb + 32 >= TN) { tc_fence_before_sync(); mbar_arrive(acc_empty(b)); }     // the last columns are in registers
                if (m < a.M) {
                    if (a.pair) {
#pragma unroll
                        for (int h = 0; h < 2; h++) {
                            const int n = n0 + cb + h * 16;
                            if (n < n1) {
                                float g[8], u[8];
#pragma unroll
                                for (int i = 0; i < 8; i++) { g[i] = __uint_as_float(h ? v1[i] : v0[i]); u[i] = __uint_as_float(h ? v1[8 + i] : v0[8 + i]); }
                                rows_epilogue_pair(a, m, n, g, u);
                            }
                        }
                    } else
#pragma unroll
                    for (int h = 0; h < 4; h++) {
                        const int n = n0 + cb + h * 8;
                        if (n < n1) {
                            float f[8];
#pragma unroll
                            for (int i = 0; i < 8; i++) f[i] = __uint_as_float(h < 2 ? v0[(h & 1) * 8 + i] : v1[(h & 1) * 8 + i]);
                            rows_epilogue8(a, m, n, f, sp, sq);
                        }
                    }
                }
            }
        }
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, cols);
}

// f32: 64 x 64 tiles, 4 x 4 sums per thread, sequential over K.
__global__ void __launch_bounds__(256) dense_gemm_f32(const DenseArgs a) {
    __shared__ float As[32][68], Bs[32][68];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int grp = a.grp_rows ? a.grp_rows : a.nt, tpg = (grp + 63) / 64, gi = blockIdx.x / tpg;
    const int m0 = blockIdx.y * 64, n0 = gi * grp + (blockIdx.x - gi * tpg) * 64, n1 = (gi + 1) * grp, ka = gi * a.grp_chunks * 32;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.0f;
    for (int s = 0; s < a.nk; s++) {
        const DenseK& g = a.seg[s];
        const int lda = (g.a_chunks ? g.a_chunks : g.chunks) * 32;
        for (int c = 0; c < g.chunks; c++) {
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int idx = tid + i * 256;                // 512 groups of 4 floats per operand tile
                {
                    const int r = idx >> 3, k4 = idx & 7, m = m0 + r;
                    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (m < a.M) v = *(const float4*)((const float*)g.a + (size_t)m * lda + ka + c * 32 + k4 * 4);
                    As[k4 * 4][r] = v.x; As[k4 * 4 + 1][r] = v.y; As[k4 * 4 + 2][r] = v.z; As[k4 * 4 + 3][r] = v.w;
                }
                {
                    const int rg = idx >> 6, k4 = (idx >> 3) & 7, r = rg * 8 + (idx & 7), n = n0 + r;
                    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (n < n1) v = *(const float4*)((const unsigned char*)g.w + chunked_off(WK_F32, a.nt, n, (size_t)c * 32 + k4 * 4));
                    Bs[k4 * 4][r] = v.x; Bs[k4 * 4 + 1][r] = v.y; Bs[k4 * 4 + 2][r] = v.z; Bs[k4 * 4 + 3][r] = v.w;
                }
            }
            __syncthreads();
#pragma unroll
            for (int k = 0; k < 32; k++) {
                const float4 av = *(const float4*)&As[k][ty * 4], bv = *(const float4*)&Bs[k][tx * 4];
                const float x[4] = {av.x, av.y, av.z, av.w}, w[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++) acc[i][j] = fmaf(x[i], w[j], acc[i][j]);
            }
            __syncthreads();
        }
    }
    // eight neighbouring columns per thread for the shared epilogue: through shared memory, 32 rows at a time (As and Bs are free)
    float sp = 0.0f, sq = 0.0f;
    if (a.act_row0 < a.nt) { sp = softplus(a.act_par[0]); sq = softplus(a.act_par[1]); }
    for (int half = 0; half < 2; half++) {
        if ((ty >> 3) == half)
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) As[(ty & 7) * 4 + i][tx * 4 + j] = acc[i][j];
        __syncthreads();
        const int r = tid >> 3, n = n0 + (tid & 7) * 8, m = m0 + half * 32 + r;
        if (a.pair) {
            if (m < a.M && n < n1 && (tid & 1) == 0) {
                float g[8], u[8];
#pragma unroll
                for (int i = 0; i < 8; i++) { g[i] = As[r][(tid & 7) * 8 + i]; u[i] = As[r][(tid & 7) * 8 + 8 + i]; }
                rows_epilogue_pair(a, m, n, g, u);
            }
        } else if (m < a.M && n < n1) {
            float f[8];
#pragma unroll
            for (int i = 0; i < 8; i++) f[i] = As[r][(tid & 7) * 8 + i];
            rows_epilogue8(a, m, n, f, sp, sq);
        }
        __syncthreads();
    }
}

cudaError_t launch_dense_gemm(const DenseArgs& a_in, int sm_count, cudaStream_t st) {
    DenseArgs a = a_in;
    if (a.nk < 1 || a.nk > 2 || a.nt <= 0 || a.nt % 8 || a.M <= 0 || a.epi == DENSE_ARGMAX || a.epi == DENSE_STREAMS || (a.kind != WK_BF16 && a.kind != WK_F32)) return cudaErrorInvalidValue;
    if ((a.pair && a.nt % 16) || (a.grp_rows && (a.grp_rows % 8 || a.nt % a.grp_rows))) return cudaErrorInvalidValue;
    const int grp = a.grp_rows ? a.grp_rows : a.nt, groups = a.nt / grp;
    if (a.kind == WK_F32) {
        dense_gemm_f32<<<dim3((grp + 63) / 64 * groups, (a.M + 63) / 64), 256, 0, st>>>(a);
        return cudaGetLastError();
    }
    // tile width: the fewest (rounds over the SMs) x (time of a tile); a narrow tile does not fill the tensor pipe.  (With few rows a chunk
    // of K takes about 0.4 us whatever the tile's width, so that narrower tiles on more SMs gain nothing: 64 rows x 27648 x K 4096 took
    // 61 us with tiles of 256 and 84 us with tiles of 64.)
    const int mt = (a.M + 127) / 128;
    int TN = 256;
    double best = 1e30;
    for (int tn = 256; tn >= 64; tn >>= 1) {
        const long long tiles = (long long)mt * ((grp + tn - 1) / tn) * groups;
        const double cost = (double)((tiles + sm_count - 1) / sm_count) * (tn + (tn < 128 ? 64 : 48));
        if (cost < best) { best = cost; TN = tn; }
    }
    const int stage_bytes = kDmABytes + TN * 128;
    int stages = (220 * 1024) / stage_bytes;
    if (stages > kDmMaxStages) stages = kDmMaxStages;
    const size_t smem = (size_t)stages * stage_bytes + 512;
    static bool attr_set = false;
    if (!attr_set) {
        const cudaError_t e = cudaFuncSetAttribute((const void*)dense_gemm_tc, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
        if (e != cudaSuccess) return e;
        attr_set = true;
    }
    const int n_tiles = mt * ((grp + TN - 1) / TN) * groups;
    dense_gemm_tc<<<n_tiles < sm_count ? n_tiles : sm_count, kDmThreads, smem, st>>>(a, TN, stages);
    return cudaGetLastError();
}

}  // namespace lum
