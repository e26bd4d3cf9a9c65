// Causal attention of many rows of ONE sequence over its bf16 K/V cache, on the tensor cores: the attention of a prompt that
// is processed as rows (`LlamaAttention` / `QwenAttention` with s > 1, examples/llama/src/model.rs:415-488 — the reference's
// kernel walks the cache once per (KV head, query group, row); here 128 / G query rows times the G query heads of a KV head
// form the 128 rows of one tensor-core tile and share every K/V tile they read).
//
// One CTA = one KV head x one tile of QT = 128 / G query rows.  Per tile of 64 cached positions:
//     S = Q K^T          tcgen05.mma kind::f16, M = 128, N = 64, K = 128: 8 instructions per Q operand
//     online softmax     8 warps read S from tensor memory (thread = row, half of the keys), scale, mask, exponentiate
//     O_t = P V          M = 128, N = 128, K = 64: 4 instructions per P operand; V is read as stored (MN-major operand)
//     O = O * alpha + O_t   in registers (thread = row, half of the head dimension)
// K/V tiles arrive through cp.async, the next tile's copies in flight while the current one is computed.
//
// Accuracy.  The oracle computes this in f32 from f32 queries and bf16 cache values.  The cache values are bf16 already, so
// they enter the tensor core exactly.  The f32 operands — the queries and the softmax weights — are split into two bf16
// terms each (x = hi + lo, |x - hi - lo| <= 2^-17 |x|), and each product runs twice, once per term, accumulating in f32:
// the result differs from the f32 reference by the order of summation and by 2^-17 relative per operand, far inside the
// path's tolerance, at the cost of twice the tensor-core instructions (which are not what bounds this kernel).
#include <cuda_bf16.h>

#include "lum_common.cuh"
#include "lum_dense.cuh"
#include "lum_rows.cuh"

namespace lum {

namespace {

constexpr int kAtHD = 128;           // head dimension
constexpr int kAtKT = 64;            // cached positions per tile
constexpr int kAtThreads = 256;
// shared memory (bytes): operands in the tensor core's no-swizzle core-matrix order, [16-byte column group][row][16 bytes]
constexpr int kAtQBytes = 128 * kAtHD * 2;          // 32 KiB per Q term
constexpr int kAtKVBytes = kAtKT * kAtHD * 2;       // 16 KiB per K or V tile
constexpr int kAtPBytes = 128 * kAtKT * 2;          // 16 KiB per P term
constexpr int kAtOffQhi = 0, kAtOffQlo = kAtQBytes, kAtOffK = 2 * kAtQBytes, kAtOffV = kAtOffK + 2 * kAtKVBytes,
              kAtOffPhi = kAtOffV + 2 * kAtKVBytes, kAtOffPlo = kAtOffPhi + kAtPBytes, kAtOffMisc = kAtOffPlo + kAtPBytes;
constexpr int kAtMiscBytes = 2048;                  // 2 mbarriers, the tensor-memory slot, per-row exchange of maxima / sums
constexpr int kAtSmem = kAtOffMisc + kAtMiscBytes;
constexpr uint32_t kAtTmemCols = 256;               // S: columns 0..63, O_t: columns 64..191

// kind::f16, bf16 x bf16 -> f32; b_mn: the B operand is MN-major (V as stored: the head dimension contiguous)
__host__ __device__ constexpr uint32_t idesc_bf16(int M, int N, bool b_mn) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((b_mn ? 1u : 0u) << 16) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(M >> 4) << 24);
}
__device__ __forceinline__ void umma_bf16(uint32_t tmem_d, uint64_t da, uint64_t db, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(tmem_d), "l"(da), "l"(db), "r"(idesc), "r"(accumulate)
        : "memory");
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, uint32_t src_bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(src_bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// x = hi + lo in bf16; returns the two packed pairs for (x0, x1)
__device__ __forceinline__ void split2(float x0, float x1, uint32_t* hi, uint32_t* lo) {
    const __nv_bfloat16 h0 = __float2bfloat16_rn(x0), h1 = __float2bfloat16_rn(x1);
    const __nv_bfloat16 l0 = __float2bfloat16_rn(x0 - __bfloat162float(h0)), l1 = __float2bfloat16_rn(x1 - __bfloat162float(h1));
    *hi = (uint32_t)__bfloat16_as_ushort(h0) | ((uint32_t)__bfloat16_as_ushort(h1) << 16);
    *lo = (uint32_t)__bfloat16_as_ushort(l0) | ((uint32_t)__bfloat16_as_ushort(l1) << 16);
}

}  // namespace

// G = query heads per KV head (1, 2, 4 or 8): MMA row r = g * QT + qi is query row q0 + qi of head kvh * G + g.
__global__ void __launch_bounds__(kAtThreads, 1) attn_prompt_tc(const AttnRowsArgs a, int G, int lbo_sbo_swap) {
    extern __shared__ __align__(128) unsigned char smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kvh = blockIdx.x, QT = 128 / G, q0 = blockIdx.y * QT;
    const uint32_t s_base = smem_u32(smem);
    const uint32_t bar_s = s_base + kAtOffMisc, bar_o = bar_s + 8, tmem_slot = bar_s + 16;
    float* x_max = (float*)(smem + kAtOffMisc + 64);          // [2 halves][128 rows]
    int* s_flag = (int*)(smem + kAtOffMisc + 64 + 1024);      // [0]: largest position of the CTA's rows, [1]: a wait ran out

    if (tid == 0) { mbar_init(bar_s, 1); mbar_init(bar_o, 1); mbar_fence_init(); s_flag[0] = -1; s_flag[1] = 0; }
    if (warp == 0) tmem_alloc(tmem_slot, kAtTmemCols);
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = *(volatile uint32_t*)(smem + kAtOffMisc + 16);

    // this thread's row of the tile, for the softmax and the output
    const int row = (warp & 3) * 32 + lane, half = warp >> 2;
    const int g_row = row / QT, qi_row = row - g_row * QT, m_row = q0 + qi_row;
    const bool row_ok = m_row < a.M;
    int pos_row = row_ok ? a.row_pos[m_row] : -1;
    if (pos_row >= a.max_seq) pos_row = -1;                    // flagged by the kernel that appended the row
    {
        int pm = pos_row;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) pm = max(pm, __shfl_xor_sync(0xffffffffu, pm, o));
        if (lane == 0 && pm >= 0) atomicMax(&s_flag[0], pm);
    }

    // ---- Q tile -> two bf16 operands in shared memory
    const size_t qd = (size_t)a.n_q * kAtHD;
    for (int ch = tid; ch < 128 * 16; ch += kAtThreads) {
        const int r = ch >> 4, c = ch & 15;                    // 16 threads read one row's 512 bytes
        const int g = r / QT, qi = r - g * QT, m = q0 + qi;
        uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
        if (m < a.M) {
            const float4* src = (const float4*)(a.q_rot + (size_t)m * qd + ((size_t)kvh * G + g) * kAtHD + c * 8);
            const float4 v0 = src[0], v1 = src[1];
            split2(v0.x, v0.y, &hi.x, &lo.x); split2(v0.z, v0.w, &hi.y, &lo.y);
            split2(v1.x, v1.y, &hi.z, &lo.z); split2(v1.z, v1.w, &hi.w, &lo.w);
        }
        *(uint4*)(smem + kAtOffQhi + c * 2048 + r * 16) = hi;
        *(uint4*)(smem + kAtOffQlo + c * 2048 + r * 16) = lo;
    }
    __syncthreads();
    const int pos_max = s_flag[0];
    const int n_tiles = pos_max >= 0 ? pos_max / kAtKT + 1 : 0;

    const size_t row_elems = (size_t)a.n_kv * kAtHD;
    const __nv_bfloat16* kc = (const __nv_bfloat16*)a.k_cache + (size_t)kvh * kAtHD;
    const __nv_bfloat16* vc = (const __nv_bfloat16*)a.v_cache + (size_t)kvh * kAtHD;
    // one K and one V tile: 64 positions x 16 column groups = 1024 16-byte chunks each; a warp takes 8 positions x 4 groups
    auto load_tile = [&](int t, int buf) {
        const uint32_t kdst = s_base + kAtOffK + buf * kAtKVBytes, vdst = s_base + kAtOffV + buf * kAtKVBytes;
        // the tile's 64 positions start on a multiple of 64: one sequence slot or one page (of at least 64 rows) holds them all;
        // its first position is at most pos_max, so it is mapped
        const size_t tile_row = kv_phys_row(a.pg, a.seq0, a.max_seq, t * kAtKT);
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int ch = tid + i * kAtThreads;
            const int w = ch >> 5, l = ch & 31;                // 32 "warp slots" of 32 chunks
            const int key = (w >> 2) * 8 + (l >> 2), c = (w & 3) * 4 + (l & 3);
            const int j = t * kAtKT + key;
            const bool in = j <= pos_max;                      // rows never written (or beyond the capacity) read as zeros
            const size_t off = (tile_row + (size_t)(in ? key : 0)) * row_elems + c * 8;
            cp_async16(kdst + c * 1024 + key * 16, kc + off, in ? 16u : 0u);
            cp_async16(vdst + c * 1024 + key * 16, vc + off, in ? 16u : 0u);
        }
        cp_async_commit();
    };

    float o_acc[64];
#pragma unroll
    for (int i = 0; i < 64; i++) o_acc[i] = 0.0f;
    float m_run = -INFINITY, l_run = 0.0f;
    const float scale = 1.0f / sqrtf((float)kAtHD);
    constexpr uint32_t idesc_s = idesc_bf16(128, kAtKT, false), idesc_o = idesc_bf16(128, kAtHD, true);
    const uint32_t lane_base = tmem + ((uint32_t)((warp & 3) * 32) << 16);

    if (n_tiles > 0) load_tile(0, 0);
    uint32_t phase = 0;
    bool failed = false;
#pragma unroll 1
    for (int t = 0; t < n_tiles; t++) {
        const int buf = t & 1;
        if (t + 1 < n_tiles) { load_tile(t + 1, buf ^ 1); cp_async_wait<1>(); } else { cp_async_wait<0>(); }
        fence_proxy_async_smem();
        __syncthreads();
        if (tid == 0) {
            tc_fence_after_sync();
            const uint32_t kb = s_base + kAtOffK + buf * kAtKVBytes;
#pragma unroll
            for (int term = 0; term < 2; term++) {
                const uint32_t qb = s_base + (term ? kAtOffQlo : kAtOffQhi);
#pragma unroll
                for (int ks = 0; ks < kAtHD / 16; ks++)       // K = 16 elements = two 16-byte column groups per instruction
                    umma_bf16(tmem, umma_smem_desc(qb + ks * 2 * 2048, 2048, 128), umma_smem_desc(kb + ks * 2 * 1024, 1024, 128), idesc_s,
                              (term | ks) ? 1u : 0u);
            }
            umma_commit(bar_s);
        }
        if (!mbar_wait(bar_s, phase)) failed = true;
        tc_fence_after_sync();

        // ---- softmax of this thread's row over its 32 keys of the tile
        float s[32];
        {
            uint32_t v[16];
            tmem_ld16(lane_base + half * 32, v);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; i++) s[i] = __uint_as_float(v[i]);
            tmem_ld16(lane_base + half * 32 + 16, v);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; i++) s[16 + i] = __uint_as_float(v[i]);
        }
        const int j0 = t * kAtKT + half * 32;
        float mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < 32; i++) {
            s[i] = (j0 + i <= pos_row) ? s[i] * scale : -INFINITY;
            mx = fmaxf(mx, s[i]);
        }
        x_max[half * 128 + row] = mx;
        named_sync(1, kAtThreads);
        const float m_new = fmaxf(m_run, fmaxf(mx, x_max[(half ^ 1) * 128 + row]));
        const float alpha = (m_new == -INFINITY) ? 1.0f : expf(m_run - m_new);      // m_run = -inf: exp(-inf) = 0
        float psum = 0.0f;
        uint32_t ph[16], pl[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
            const float p0 = (s[i] == -INFINITY) ? 0.0f : expf(s[i] - m_new);
            const float p1 = (s[i + 1] == -INFINITY) ? 0.0f : expf(s[i + 1] - m_new);
            psum += p0 + p1;
            split2(p0, p1, &ph[i >> 1], &pl[i >> 1]);
        }
        l_run = l_run * alpha + psum;
        m_run = m_new;
#pragma unroll
        for (int c = 0; c < 4; c++) {                          // 4 column groups of 8 keys
            const int off = (half * 4 + c) * 2048 + row * 16;
            *(uint4*)(smem + kAtOffPhi + off) = make_uint4(ph[c * 4], ph[c * 4 + 1], ph[c * 4 + 2], ph[c * 4 + 3]);
            *(uint4*)(smem + kAtOffPlo + off) = make_uint4(pl[c * 4], pl[c * 4 + 1], pl[c * 4 + 2], pl[c * 4 + 3]);
        }
        fence_proxy_async_smem();
        tc_fence_before_sync();
        __syncthreads();
        if (tid == 0) {
            tc_fence_after_sync();
            const uint32_t vb = s_base + kAtOffV + buf * kAtKVBytes;
            // V as stored: 16-byte groups of 8 head dimensions, 1024 bytes apart along the head dimension (MN), 8 positions = 128
            // contiguous bytes along K
            const uint32_t v_lbo = lbo_sbo_swap ? 1024u : 128u, v_sbo = lbo_sbo_swap ? 128u : 1024u;
#pragma unroll
            for (int term = 0; term < 2; term++) {
                const uint32_t pb = s_base + (term ? kAtOffPlo : kAtOffPhi);
#pragma unroll
                for (int ks = 0; ks < kAtKT / 16; ks++)       // 16 positions per instruction
                    umma_bf16(tmem + 64, umma_smem_desc(pb + ks * 2 * 2048, 2048, 128), umma_smem_desc(vb + ks * 256, v_lbo, v_sbo), idesc_o,
                              (term | ks) ? 1u : 0u);
            }
            umma_commit(bar_o);
        }
        if (!mbar_wait(bar_o, phase)) failed = true;
        tc_fence_after_sync();
#pragma unroll
        for (int c = 0; c < 4; c++) {
            uint32_t v[16];
            tmem_ld16(lane_base + 64 + half * 64 + c * 16, v);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; i++) o_acc[c * 16 + i] = fmaf(o_acc[c * 16 + i], alpha, __uint_as_float(v[i]));
        }
        tc_fence_before_sync();
        phase ^= 1u;
        if (__syncthreads_or(failed ? 1 : 0)) { if (tid == 0) s_flag[1] = 1; break; }       // the tensor core never answered: give up, together
    }
    cp_async_wait<0>();
    __syncthreads();
    if (s_flag[1] && tid == 0 && a.status) atomicOr(a.status, LUM_ST_WAIT_TMEM);

    // ---- out = O / l, l = the two halves' sums
    x_max[half * 128 + row] = l_run;
    __syncthreads();
    const float l_tot = l_run + x_max[(half ^ 1) * 128 + row];
    if (row_ok) {
        const float inv = l_tot > 0.0f ? 1.0f / l_tot : 0.0f;
        float4* dst = (float4*)(a.out + (size_t)m_row * qd + ((size_t)kvh * G + g_row) * kAtHD + half * 64);
#pragma unroll
        for (int i = 0; i < 16; i++) dst[i] = make_float4(o_acc[4 * i] * inv, o_acc[4 * i + 1] * inv, o_acc[4 * i + 2] * inv, o_acc[4 * i + 3] * inv);
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 0) tmem_dealloc(tmem, kAtTmemCols);
}

bool attn_prompt_tc_supported(const AttnRowsArgs& a) {
    const int G = a.n_kv > 0 ? a.n_q / a.n_kv : 0;
    return a.hd == kAtHD && a.kv_bf16 && a.window == 0 && a.row_seq == nullptr && (G == 1 || G == 2 || G == 4 || G == 8) && a.n_q == G * a.n_kv &&
           (((uintptr_t)a.q_rot | (uintptr_t)a.out) & 15) == 0;
}

cudaError_t launch_attn_prompt_tc(const AttnRowsArgs& a, cudaStream_t st) {
    if (!attn_prompt_tc_supported(a)) return cudaErrorInvalidValue;
    static bool attr_set = false;
    if (!attr_set) {
        const cudaError_t e = cudaFuncSetAttribute((const void*)attn_prompt_tc, cudaFuncAttributeMaxDynamicSharedMemorySize, kAtSmem);
        if (e != cudaSuccess) return e;
        attr_set = true;
    }
    static const int swap = [] { const char* e = getenv("LUM_ATTN_TC_SWAP"); return e ? atoi(e) : 0; }();
    const int G = a.n_q / a.n_kv, QT = 128 / G;
    attn_prompt_tc<<<dim3(a.n_kv, (a.M + QT - 1) / QT), kAtThreads, kAtSmem, st>>>(a, G, swap);
    return cudaGetLastError();
}

// ---------------------------------------------------------------------------------------------------- band attention
// The same tiles for layers with their own head sizes, a window, and a distance bias: key size dkp (a multiple of 16) and value
// size dvp are run-time numbers, the query heads of a K/V head may be any number R <= 128 (QT = 128 / R query rows per CTA), tiles of keys
// start at the first key any row of the CTA still sees.  Queries arrive scaled (score factor and temperature).  The output goes
// straight to the operand of the next product.
//
// The tensor core works one tile ahead of the softmax: while tile t's scores are exponentiated, S(t + 1) is computed into the other
// score buffer, and O_t of tile t - 1 — issued at the end of the previous turn — is added up only when the new weights are ready to
// be stored.  The bias depends on the distance alone: r1 ln(1 + r2 d) is evaluated once per (head, distance) of a tile,
// R (QT + 63) values instead of 128 x 64, into shared memory (up to 16 heads per K/V head).  Rows are consecutive positions of one
// sequence.  Scores are kept in units of ln 2 (queries and bias carry the factor 1 / ln 2), so that a weight is one power of two.
//
// Two maps (differential attention): the CTAs of the two maps of a K/V head and the same rows are a cluster of two.  Each finishes its own
// softmax; the second hands lambda * its output over through the first one's shared memory, and the first subtracts, norms the head
// and stores.
//
// DVH: value dimensions a thread accumulates (half of the value size, rounded up to 16).
namespace {
__device__ __forceinline__ void cluster_st_f32x4(uint32_t addr, float4 v) {
    asm volatile("st.shared::cluster.v4.f32 [%0], {%1, %2, %3, %4};" ::"r"(addr), "f"(v.x), "f"(v.y), "f"(v.z), "f"(v.w) : "memory");
}
constexpr float kLog2e = 1.4426950408889634f;
__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
// x = hi + lo in bf16 with the high term cut off instead of rounded (no conversion instruction for it; |x - hi - lo| <= 2^-17 |x| all the same)
__device__ __forceinline__ void split2_cut(float x0, float x1, uint32_t* hi, uint32_t* lo) {
    const uint32_t b0 = __float_as_uint(x0), b1 = __float_as_uint(x1);
    *hi = __byte_perm(b0, b1, 0x7632);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x0 - __uint_as_float(b0 & 0xffff0000u), x1 - __uint_as_float(b1 & 0xffff0000u));
    *lo = *(const uint32_t*)&l;
}
constexpr int kBtTabMaxR = 16;                      // R (128 / R + 63) <= 1136 floats up to there
constexpr int kBtMiscBytes = 2048 + 4608;           // barriers, row exchange, flags; the bias table
struct BandSmem { int qlo, k, v, phi, plo, misc, total; };      // byte offsets; the high Q term is at 0
__host__ __device__ inline int band_xch_ld(int dvp) { return dvp + 4; }      // floats per row of the hand-over between two maps (from offset 0)
__host__ __device__ inline BandSmem band_smem(int dkp, int dvp, int maps) {
    BandSmem s;
    s.qlo = 128 * dkp * 2;
    s.k = 2 * s.qlo;
    s.v = s.k + 2 * kAtKT * dkp * 2;
    s.phi = s.v + 2 * kAtKT * dvp * 2;
    s.plo = s.phi + kAtPBytes;
    s.misc = s.plo + kAtPBytes;
    if (maps == 2 && s.misc < 128 * band_xch_ld(dvp) * 4) s.misc = 128 * band_xch_ld(dvp) * 4;
    s.total = s.misc + kBtMiscBytes;
    return s;
}
}  // namespace

template <int DVH>
__global__ void __launch_bounds__(kAtThreads, 1) attn_band_tc(const BandArgs a) {
    extern __shared__ __align__(128) unsigned char smem[];
    const QkvArgs& p = a.p;
    const int dkp = p.dkp, dvp = p.dvp, kgr = dkp / 8, vgr = dvp / 8;
    const BandSmem L = band_smem(dkp, dvp, p.maps);
    const int maps = p.maps, kh = blockIdx.x, map = kh % maps;                       // kh: this map's keys; kvh: the values of both
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int R = p.n_q / p.n_kv, kvh = kh / maps, QT = 128 / R;
    const int q0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * QT;      // later rows first: without a window they have the most keys
    const uint32_t s_base = smem_u32(smem);
    const uint32_t bar_s = s_base + L.misc, bar_o = bar_s + 8, tmem_slot = bar_s + 16;
    float* x_max = (float*)(smem + L.misc + 64);
    int* s_flag = (int*)(smem + L.misc + 64 + 1024);          // [0] largest, [2] smallest position of the CTA's rows, [1] a wait ran out
    float* tab = (float*)(smem + L.misc + 2048);
    constexpr uint32_t kCols = DVH > 64 ? 512u : 256u;        // S: columns 0..63 and 64..127 in turn, O_t from 128 on (2 DVH columns)
    constexpr uint32_t kOCol = 128;

    if (tid == 0) { mbar_init(bar_s, 1); mbar_init(bar_o, 1); mbar_fence_init(); s_flag[0] = -1; s_flag[1] = 0; s_flag[2] = 0x7fffffff; }
    if (warp == 0) tmem_alloc(tmem_slot, kCols);
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = *(volatile uint32_t*)(smem + L.misc + 16);

    const int row = (warp & 3) * 32 + lane, half = warp >> 2;
    const int g_row = row / QT, qi_row = row - g_row * QT, m_row = q0 + qi_row;
    const bool row_ok = g_row < R && m_row < a.M;
    int pos_row = row_ok ? a.row_pos[m_row] : -1;
    if (pos_row >= a.max_seq) pos_row = -1;                    // flagged by the kernel that appended the row
    {
        int pm = pos_row, pn = pos_row >= 0 ? pos_row : 0x7fffffff;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) { pm = max(pm, __shfl_xor_sync(0xffffffffu, pm, o)); pn = min(pn, __shfl_xor_sync(0xffffffffu, pn, o)); }
        if (lane == 0 && pm >= 0) { atomicMax(&s_flag[0], pm); atomicMin(&s_flag[2], pn); }
    }

    // ---- Q tile -> two bf16 operands in shared memory
    for (int ch = tid; ch < 128 * kgr; ch += kAtThreads) {
        const int r = ch / kgr, c = ch - r * kgr, g = r / QT, m = q0 + (r - g * QT);
        uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
        if (g < R && m < a.M) {
            const float4* src = (const float4*)(a.q + (((size_t)m * p.n_q + (size_t)kvh * R + g) * maps + map) * dkp + c * 8);
            const float4 v0 = src[0], v1 = src[1];
            split2_cut(v0.x * kLog2e, v0.y * kLog2e, &hi.x, &lo.x); split2_cut(v0.z * kLog2e, v0.w * kLog2e, &hi.y, &lo.y);
            split2_cut(v1.x * kLog2e, v1.y * kLog2e, &hi.z, &lo.z); split2_cut(v1.z * kLog2e, v1.w * kLog2e, &hi.w, &lo.w);
        }
        *(uint4*)(smem + c * 2048 + r * 16) = hi;
        *(uint4*)(smem + L.qlo + c * 2048 + r * 16) = lo;
    }
    __syncthreads();
    const int pos_max = s_flag[0], pos_min = s_flag[2];
    const int first = pos_max < 0 ? 0 : a.chunk > 0 ? pos_min / a.chunk * a.chunk : (a.window > 0 && pos_min + 1 > a.window) ? pos_min + 1 - a.window : 0;     // no row sees an earlier key
    const int t_lo = first / kAtKT, n_t = pos_max >= 0 ? pos_max / kAtKT + 1 - t_lo : 0;
    const int reach = a.chunk > 0 ? max(pos_row, 0) % a.chunk + 1 : a.window > 0 ? a.window : 0x7fffffff;    // this row sees distances 0 .. reach - 1
    const bool biased = a.r1 != nullptr, use_tab = biased && R <= kBtTabMaxR;
    const int TW = QT + kAtKT - 1, head = kvh * R + (row_ok ? g_row : 0);
    const float* my_tab = tab + (g_row < R ? g_row : 0) * TW + qi_row + kAtKT - 1 - half * 32;      // [-i]: key i of this thread's half tile

    const size_t k_row = (size_t)p.n_kv * maps * dkp, v_row = (size_t)p.n_kv * dvp;
    const __nv_bfloat16* kc = (const __nv_bfloat16*)a.k_cache + (size_t)kh * dkp;
    const __nv_bfloat16* vc = (const __nv_bfloat16*)a.v_cache + (size_t)kvh * dvp;
    // one operand tile (i-th of this CTA): 64 positions x `gr` 16-byte groups; a warp takes 8 positions x 4 groups at a time.  One copy
    // group per call, empty beyond the last tile.
    auto load_tile = [&](int i, uint32_t dst, const __nv_bfloat16* src, size_t row_elems, int gr) {
        if (i < n_t) {
            const int t = t_lo + i, gq = (gr + 3) / 4;
            // the tile's 64 positions start on a multiple of 64: one sequence slot or one page (of at least 64 rows) holds them all
            const size_t tile_row = kv_phys_row(a.pg, a.seq0, a.max_seq, t * kAtKT);
            for (int w = warp; w < 8 * gq; w += kAtThreads / 32) {
                const int kb = w / gq, key = kb * 8 + (lane >> 2), c = (w - kb * gq) * 4 + (lane & 3), j = t * kAtKT + key;
                const bool in = j <= pos_max;                  // rows never written read as zeros
                if (c < gr) cp_async16(dst + c * 1024 + key * 16, src + (tile_row + (size_t)(in ? key : 0)) * row_elems + c * 8, in ? 16u : 0u);
            }
        }
        cp_async_commit();
    };
    auto load_k = [&](int i) { load_tile(i, s_base + L.k + (i & 1) * kAtKT * dkp * 2, kc, k_row, kgr); };
    auto load_v = [&](int i) { load_tile(i, s_base + L.v + (i & 1) * kAtKT * dvp * 2, vc, v_row, vgr); };
    const uint32_t idesc_s = idesc_bf16(128, kAtKT, false), idesc_o = idesc_bf16(128, dvp, true);
    auto issue_s = [&](int i) {                                // thread 0: scores of tile i
        const uint32_t kb = s_base + L.k + (i & 1) * kAtKT * dkp * 2, d = tmem + (i & 1) * kAtKT;
        for (int term = 0; term < 2; term++) {
            const uint32_t qb = s_base + (term ? L.qlo : 0);
            for (int ks = 0; ks < dkp / 16; ks++)
                umma_bf16(d, umma_smem_desc(qb + ks * 2 * 2048, 2048, 128), umma_smem_desc(kb + ks * 2 * 1024, 1024, 128), idesc_s, (term | ks) ? 1u : 0u);
        }
        umma_commit(bar_s);
    };

    float o_acc[DVH];
#pragma unroll
    for (int i = 0; i < DVH; i++) o_acc[i] = 0.0f;
    float m_run = -INFINITY, l_run = 0.0f, alpha_prev = 1.0f;
    const uint32_t lane_base = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    auto add_o = [&]() {                                       // o_acc = alpha o_acc + O_t, of the tile whose alpha is alpha_prev
#pragma unroll
        for (int c = 0; c < DVH / 16; c++) {
            uint32_t v[16];
            tmem_ld16(lane_base + kOCol + half * DVH + c * 16, v);      // (columns beyond dvp: never written, never stored)
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; i++) o_acc[c * 16 + i] = fmaf(o_acc[c * 16 + i], alpha_prev, __uint_as_float(v[i]));
        }
    };

    bool failed = false;
    int done = 0;                                              // tiles whose O_t was issued
    if (n_t > 0) {
        load_k(0); load_k(1); load_v(0);
        cp_async_wait<2>();
        fence_proxy_async_smem();
        __syncthreads();
        if (tid == 0) { tc_fence_after_sync(); issue_s(0); }
    }
#pragma unroll 1
    for (int i = 0; i < n_t; i++) {
        const uint32_t par = (uint32_t)(i & 1);
        const int j0 = (t_lo + i) * kAtKT;
        if (use_tab) {
            const int d0 = pos_min - j0 - (kAtKT - 1);         // smallest distance in the tile: row 0, last key
            for (int x = tid; x < R * TW; x += kAtThreads) {
                const int g = x / TW;
                tab[x] = a.r1[kvh * R + g] * kLog2e * logf(fmaf(a.r2[kvh * R + g], (float)max(d0 + x - g * TW, 0), 1.0f));
            }
        }
        if (!mbar_wait(bar_s, par)) failed = true;             // S(i) is there, and K(i)'s buffer is free
        load_k(i + 2);
        cp_async_wait<2>();                                    // K(i + 1) has landed
        fence_proxy_async_smem();
        tc_fence_before_sync();
        if (__syncthreads_or(failed ? 1 : 0)) { failed = true; break; }      // the tensor core never answered: give up, together
        tc_fence_after_sync();
        if (tid == 0 && i + 1 < n_t) issue_s(i + 1);

        // ---- softmax of this thread's row over its 32 keys of the tile
        float s[32];
        {
            uint32_t v0[16], v1[16];
            tmem_ld16(lane_base + par * kAtKT + half * 32, v0);
            tmem_ld16(lane_base + par * kAtKT + half * 32 + 16, v1);
            tmem_ld_wait();
#pragma unroll
            for (int k = 0; k < 16; k++) { s[k] = __uint_as_float(v0[k]); s[16 + k] = __uint_as_float(v1[k]); }
        }
        const int dist0 = pos_row - (j0 + half * 32);          // distance of this thread's first key
        if (use_tab) {
#pragma unroll
            for (int k = 0; k < 32; k++) s[k] -= my_tab[-k];
        } else if (biased) {
            const float r1 = a.r1[head] * kLog2e, r2 = a.r2[head];
#pragma unroll
            for (int k = 0; k < 32; k++) s[k] -= r1 * logf(fmaf(r2, (float)max(dist0 - k, 0), 1.0f));
        }
        float mx = -INFINITY;
        if (__any_sync(0xffffffffu, dist0 < 31 || dist0 >= reach)) {       // some key of some row of the warp is out of sight
#pragma unroll
            for (int k = 0; k < 32; k++) s[k] = (dist0 - k >= 0 && dist0 - k < reach) ? s[k] : -INFINITY;
        }
#pragma unroll
        for (int k = 0; k < 32; k++) mx = fmaxf(mx, s[k]);
        x_max[half * 128 + row] = mx;
        named_sync(1, kAtThreads);
        const float m_new = fmaxf(m_run, fmaxf(mx, x_max[(half ^ 1) * 128 + row]));
        const float alpha = (m_new == -INFINITY) ? 1.0f : ex2(m_run - m_new);
        const float m_sub = (m_new == -INFINITY) ? 0.0f : m_new;           // nothing seen yet: 2^-inf = 0 below
        float psum = 0.0f;
        uint32_t ph[16], pl[16];
#pragma unroll
        for (int k = 0; k < 32; k += 2) {
            const float p0 = ex2(s[k] - m_sub), p1 = ex2(s[k + 1] - m_sub);
            psum += p0 + p1;
            split2_cut(p0, p1, &ph[k >> 1], &pl[k >> 1]);
        }
        l_run = l_run * alpha + psum;
        m_run = m_new;

        if (i > 0) {                                           // O_t of the tile before; P and V(i - 1) are free after that
            if (!mbar_wait(bar_o, par ^ 1u)) failed = true;
            tc_fence_after_sync();
            add_o();
        }
        alpha_prev = alpha;
        load_v(i + 1);
#pragma unroll
        for (int c = 0; c < 4; c++) {
            const int off = (half * 4 + c) * 2048 + row * 16;
            *(uint4*)(smem + L.phi + off) = make_uint4(ph[c * 4], ph[c * 4 + 1], ph[c * 4 + 2], ph[c * 4 + 3]);
            *(uint4*)(smem + L.plo + off) = make_uint4(pl[c * 4], pl[c * 4 + 1], pl[c * 4 + 2], pl[c * 4 + 3]);
        }
        cp_async_wait<2>();                                    // V(i) has landed
        fence_proxy_async_smem();
        tc_fence_before_sync();
        __syncthreads();
        if (tid == 0) {
            tc_fence_after_sync();
            const uint32_t vb = s_base + L.v + (i & 1) * kAtKT * dvp * 2;
#pragma unroll
            for (int term = 0; term < 2; term++) {
                const uint32_t pb = s_base + (term ? L.plo : L.phi);
#pragma unroll
                for (int ks = 0; ks < kAtKT / 16; ks++)
                    umma_bf16(tmem + kOCol, umma_smem_desc(pb + ks * 2 * 2048, 2048, 128), umma_smem_desc(vb + ks * 256, 128, 1024), idesc_o,
                              (term | ks) ? 1u : 0u);
            }
            umma_commit(bar_o);
        }
        done = i + 1;
    }
    if (done > 0 && !failed) {
        if (!mbar_wait(bar_o, (uint32_t)((done - 1) & 1))) failed = true;
        tc_fence_after_sync();
        add_o();
    }
    cp_async_wait<0>();
    if (failed) s_flag[1] = 1;
    __syncthreads();
    if (s_flag[1] && tid == 0 && a.status) atomicOr(a.status, LUM_ST_WAIT_TMEM);

    // ---- out = O / l, l = the two halves' sums, as bf16 in the operand of the next product
    x_max[half * 128 + row] = l_run;
    __syncthreads();
    const float l_tot = l_run + x_max[(half ^ 1) * 128 + row];
    float inv = l_tot > 0.0f ? 1.0f / l_tot : 0.0f;
    if (maps == 2) {
        const int ld = band_xch_ld(dvp), e0 = half * DVH;
        cluster_arrive_release();
        cluster_wait_acquire();                                // the first map's CTA is done with its tiles
        if (map == 1) {
            float d1 = 0.0f, d2 = 0.0f;
            for (int e = lane; e < p.dk; e += 32) { d1 = fmaf(a.lq1[e], a.lk1[e], d1); d2 = fmaf(a.lq2[e], a.lk2[e], d2); }
            d1 = warp_sum(d1); d2 = warp_sum(d2);
            const float f = inv * (expf(d1) - expf(d2) + a.diff);
            const uint32_t to = cluster_map(s_base + (uint32_t)(row * ld + e0) * 4, 0u);
#pragma unroll
            for (int i = 0; i < DVH; i += 4)
                if (e0 + i < dvp) cluster_st_f32x4(to + i * 4, make_float4(o_acc[i] * f, o_acc[i + 1] * f, o_acc[i + 2] * f, o_acc[i + 3] * f));
        }
        cluster_arrive_release();
        cluster_wait_acquire();
        if (map == 0) {
            const float* other = (const float*)smem + row * ld + e0;
            float ss = 0.0f;
#pragma unroll
            for (int i = 0; i < DVH; i += 4) {
                if (e0 + i < dvp) {
                    const float4 v = *(const float4*)(other + i);
                    const float w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                    for (int k = 0; k < 4; k++) {
                        const float t = fmaf(o_acc[i + k], inv, -w[k]);
                        o_acc[i + k] = t;
                        if (e0 + i + k < p.dv) ss = fmaf(t, t, ss);
                    }
                }
            }
            __syncthreads();                                   // every l_run has been read
            x_max[half * 128 + row] = ss;
            __syncthreads();
            inv = (1.0f - a.diff) / sqrtf((ss + x_max[(half ^ 1) * 128 + row]) / (float)p.dv + p.eps);
        }
    }
    if (row_ok && map == 0) {
        const int col0 = head * p.dv, e0 = half * DVH;
        unsigned char* out = (unsigned char*)a.out.p;
        if ((p.dv & 7) == 0) {
#pragma unroll
            for (int c = 0; c < DVH / 8; c++) {
                if (e0 + c * 8 < p.dv) {
                    uint32_t w[4];
#pragma unroll
                    for (int i = 0; i < 4; i++) {
                        const __nv_bfloat162 b = __floats2bfloat162_rn(o_acc[c * 8 + 2 * i] * inv, o_acc[c * 8 + 2 * i + 1] * inv);
                        w[i] = *(const uint32_t*)&b;
                    }
                    *(uint4*)(out + row_operand_off(WK_BF16, a.out.chunks, m_row, col0 + e0 + c * 8)) = make_uint4(w[0], w[1], w[2], w[3]);
                }
            }
        } else {
#pragma unroll
            for (int i = 0; i < DVH; i++)
                if (e0 + i < p.dv) *(__nv_bfloat16*)(out + row_operand_off(WK_BF16, a.out.chunks, m_row, col0 + e0 + i)) = __float2bfloat16_rn(o_acc[i] * inv);
        }
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 0) tmem_dealloc(tmem, kCols);
}

bool band_prompt_tc_supported(const BandArgs& a) {
    const QkvArgs& p = a.p;
    const int R = p.n_kv > 0 ? p.n_q / p.n_kv : 0;
    return a.kv_bf16 && a.out_kind == WK_BF16 && a.row_seq == nullptr && R >= 1 && R <= 128 && p.n_q == R * p.n_kv && p.dkp % 16 == 0 && p.dvp % 16 == 0 &&
           p.dvp <= 256 && p.maps <= 2 && band_smem(p.dkp, p.dvp, p.maps).total <= 226 * 1024;
}

cudaError_t launch_band_prompt_tc(const BandArgs& a, cudaStream_t st) {
    if (!band_prompt_tc_supported(a)) return cudaErrorInvalidValue;
    const int dvh = (a.p.dvp / 2 + 15) / 16 * 16;
    const void* fn = dvh <= 16 ? (const void*)attn_band_tc<16> : dvh <= 32 ? (const void*)attn_band_tc<32> : dvh <= 64 ? (const void*)attn_band_tc<64>
                     : dvh <= 96 ? (const void*)attn_band_tc<96> : (const void*)attn_band_tc<128>;
    BandArgs b = a;
    if (b.p.maps < 1) b.p.maps = 1;
    const int smem = band_smem(b.p.dkp, b.p.dvp, b.p.maps).total;
    const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
    if (e != cudaSuccess) return e;
    const int QT = 128 / (a.p.n_q / a.p.n_kv);
    void* params[] = {&b};
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(b.p.n_kv * b.p.maps, (a.M + QT - 1) / QT); cfg.blockDim = dim3(kAtThreads); cfg.dynamicSmemBytes = (size_t)smem; cfg.stream = st;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeClusterDimension; at[0].val.clusterDim.x = 2; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
    cfg.attrs = at; cfg.numAttrs = b.p.maps == 2 ? 1 : 0;
    return cudaLaunchKernelExC(&cfg, fn, params);
}

}  // namespace lum
