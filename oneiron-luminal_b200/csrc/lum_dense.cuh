// Dense (bf16 / f32) weights: the chunked layout and the argument blocks of the kernels that read it (lum_dense.cu), and of the
// row-wise kernels around them (lum_block.cu, lum_recur.cu).  Two schedules use them: decoder layers whose sublayers share one norm, and
// decoder layers with one sublayer after the other (lum_runtime.cu, "layers described one by one").
//
// Chunked layout of a [rows, K] matrix.  Rows are padded to a multiple of 8 and K to whole chunks of 128 bytes (64 bf16 or 32 f32
// elements), with zeros.  A chunk of K holds all rows: [chunk][row / 8][16-byte group 0..7][row % 8][16 bytes].  Hence
//   * any 8-aligned range of rows of one chunk is one contiguous run of 128 bytes per row: one bulk copy brings a tile of any height;
//   * the run is what tcgen05 reads as a K-major operand without swizzling (core matrices of 8 rows x 16 bytes; 128 bytes to the next
//     16-byte group of K, 1024 bytes to the next 8 rows);
//   * a warp's 16-byte loads of 4 groups x 8 rows are 512 contiguous bytes (the matrix-vector kernel).
// Several matrices with the same K share one container (their row ranges follow each other, each padded to 8 rows), so that one
// product computes q | k | v | up; a product over two inputs (o and down) walks the chunks of two containers.
#pragma once
#include "lum_kernels.cuh"

namespace lum {

constexpr int kLayoutChunked = -1;                     // value of Tensor::kc / WeightView::kc for the layout above
__host__ __device__ inline int chunk_elems(int kind) { return kind == WK_BF16 ? 64 : 32; }
__host__ __device__ inline size_t chunked_bytes(size_t padded_rows, size_t chunks) { return padded_rows * chunks * 128; }
// byte offset of element (n, k) in a container of nt (padded) rows
__host__ __device__ inline size_t chunked_off(int kind, int nt, size_t n, size_t k) {
    const size_t ck = chunk_elems(kind), e = kind == WK_BF16 ? 8 : 4, esz = 16 / e;
    const size_t c = k / ck, g = (k % ck) / e;
    return ((c * (nt / 8) + n / 8) * 8 + g) * 128 + (n % 8) * 16 + (k % e) * esz;
}
// row-major [rows, cols] of `src_kind` (WK_F32 / WK_BF16, or LUM_F16's code) -> the rows of a container that `rm` names (RowMap,
// lum_kernels.cuh), and back
cudaError_t launch_chunked_pack(const void* src, uint32_t src_dtype, size_t rows, size_t cols, void* dst, int kind, int nt, RowMap rm, cudaStream_t st);
cudaError_t launch_chunked_unpack(const void* src, int kind, int nt, RowMap rm, size_t rows, size_t cols, float* dst_f32, void* dst_same, cudaStream_t st);

// Rows of activations as the next product's operand.  bf16: tiles of 128 rows x one chunk, [row / 128][chunk][row % 128 / 8][group][row % 8]
// [16 bytes] — the layout above with the 128 rows of a tile for a container.  f32: row-major, chunks * 32 floats per row.
struct RowOperand { void* p; int chunks; };
__device__ __forceinline__ size_t row_operand_off(int kind, int chunks, int m, int k) {      // in bytes
    if (kind == WK_BF16)
        return (((size_t)(m >> 7) * chunks + (k >> 6)) * 16 + ((m & 127) >> 3)) * 1024 + ((k >> 3) & 7) * 128 + (m & 7) * 16 + (k & 7) * 2;
    return ((size_t)m * chunks * 32 + k) * 4;
}
inline size_t row_operand_bytes(int kind, int chunks, int rows) {
    return kind == WK_BF16 ? (size_t)((rows + 127) / 128) * chunks * 16384 : (size_t)rows * chunks * 128;
}

enum : int { NORM_NONE = -1, NORM_RMS = 0, NORM_LAYER = 1 };
struct NormArgs {
    int mode;                  // NORM_*
    const float* gain;         // [width]
    const float* bias;         // [width] (NORM_LAYER)
    float eps;
    int width;
    float gain0;               // added to every stored gain (1: gains stored around zero)
};

// What happens to a finished sum.  Rows of the container below act_row0 are stored (times mult); rows from act_row0 on are a
// feed-forward's inner vector: the activation is applied and the value goes to the operand of the next product.
// DENSE_STREAMS (one vector): the sum is a sublayer's output, and the residual streams take it in (see StreamArgs).
enum : int { DENSE_STORE = 0, DENSE_RESID = 1, DENSE_ARGMAX = 2, DENSE_STREAMS = 3 };   // RESID: y += mult * sum
// Residual streams x_1 .. x_n: a sublayer's output y leaves x_t = sum_s mix[s][t] x_s + out[t] y, and the next sublayer reads
// u = sum_t next[t] x_t.  Null mix: the identity; null out / next: ones.
constexpr int kMaxStreams = 8;
struct StreamArgs { int n; const float *mix, *out, *next; float* x; int ldx; float* u; };      // x: ldx floats from stream to stream
struct DenseK { const void* w; int chunks; const float* x; const void* a; int a_chunks; };   // x: one activation vector (f32); a: rows of activations (RowOperand) of a_chunks chunks (0: chunks)
struct DenseArgs {
    DenseK seg[2]; int nk;     // the product's K ranges, one container each
    int kind;                  // WK_BF16 or WK_F32
    int nt, n_real;            // padded rows of the containers; rows that exist
    int epi;
    float mult;
    float* y; int ldy;         // rows: ldy floats per row
    int act_row0;              // == nt: no activation rows
    const float* act_par;      // the two numbers of xIELU
    float* act_x;              // one vector: activated values, f32
    RowOperand act;            // rows: activated values as an operand
    const float* bias;         // [nt] added to the sums (null: none)
    int gelu_rows;             // rows of the container below it: gelu (tanh form) of the stored value
    // pair 1: the whole container is groups of 8 gate rows, each followed by 8 up rows; the operand of the next product receives
    // clamped_gate(gate, up, limit), half as many values (as act_x / act above; act_row0 is not used)
    int pair; float limit;
    int grp_rows, grp_chunks;  // rows, not one vector: container rows [g * grp_rows, ..) multiply chunks [g * grp_chunks, ..) of the activations (0: all the same)
    StreamArgs hc;             // DENSE_STREAMS
    NormArgs norm;             // one vector only: norm of seg[0].x in the prologue
    int M;
    GemvArgs am;               // DENSE_ARGMAX: part_val, part_idx, counter, state, tokens_out, advance, pair_out
    uint32_t* status;
    int use_pdl;
};
cudaError_t launch_dense_gemv(const DenseArgs& a, int sm_count, cudaStream_t st);
cudaError_t launch_dense_gemm(const DenseArgs& a, int sm_count, cudaStream_t st);     // bf16: tensor cores; f32: CUDA cores

// ---- row-wise kernels (lum_block.cu)
struct NormRowsArgs {
    const float* x; int ldx;
    const int* row_index;      // optional: row m of the output is row row_index[m] of x
    int M;
    NormArgs norm;
    int kind; RowOperand out;
};
cudaError_t launch_norm_rows(const NormRowsArgs& a, cudaStream_t st);

// A causal convolution per channel over the last `taps` tokens.  Values before this pass come from the sequence's ring: the value of
// position p lies in row p % taps, so that a step of one token reads taps - 1 rows and writes the one that is left.
struct ConvArgs {
    const float* w; int taps;          // [channels][taps], the last tap is the current token's; taps 0: none
    float* ring; int ch;               // [sequence][taps][ch]
};
// channel c of the row at `src` (rows ld floats apart); in_pass: rows before it that belong to the same sequence and pass
__device__ __forceinline__ float conv_at(const ConvArgs& cv, const float* ring, const float* src, int ld, int in_pass, int pos, int c) {
    if (cv.taps == 0) return src[c];
    if (cv.taps == 4) {                                        // all loads at once
        float v[4];
#pragma unroll
        for (int d = 0; d < 4; d++) v[d] = d <= in_pass ? src[c - (ptrdiff_t)d * ld] : pos >= d ? ring[(size_t)((pos - d) & 3) * cv.ch + c] : 0.0f;
        const float4 w = *(const float4*)(cv.w + (size_t)c * 4);
        return fmaf(w.w, v[0], fmaf(w.z, v[1], fmaf(w.y, v[2], w.x * v[3])));
    }
    const float* w = cv.w + (size_t)c * cv.taps;
    float s = 0.0f;
    for (int d = cv.taps - 1; d >= 0; d--) {
        float v = 0.0f;
        if (d <= in_pass) v = src[c - (ptrdiff_t)d * ld];
        else if (pos >= d) v = ring[(size_t)((pos - d) % cv.taps) * cv.ch + c];
        s = fmaf(w[cv.taps - 1 - d], v, s);
    }
    return s;
}
// After a pass of M > 1 rows of one sequence: its last `taps` values of every channel go to the ring.
struct ConvTailArgs { ConvArgs conv; const float* src; int ld, n_ch, M; const int* row_pos; int seq; };
cudaError_t launch_conv_tail(const ConvTailArgs& a, cudaStream_t st);

// q | k | v rows as the projection left them -> queries ready for the scores, and this step's cache rows
struct QkvArgs {
    const float* qkv; int ld, q_off, k_off, v_off;
    const float *q_gain, *k_gain;      // norm over the whole projection (null: none)
    float eps;
    float scale; const float* temp;    // q is multiplied by scale * temp[head] (temp null: scale)
    int n_q, n_kv, dk, dv, dkp, dvp;   // dkp / dvp: head sizes of the cache rows (padded with zeros)
    int mix;                           // 0: none, 1: this layer's values are kept in v_first, 2: v = (1 - lambda) v + lambda v_first
    const float* lambda; float* v_first; int ld_vfirst;
    // Preparation head by head (per_head): short convolution, RMS norm of each head with one gain [dk] for all (q_gain, k_gain; null:
    // none), rotation of the first rot_dims dimensions.  maps: queries and keys per head and value (rows [head][map][dk]).
    int per_head, maps;
    ConvArgs conv;                     // columns of qkv as the projection left them
    const float2* rot; int rot_dims;   // [position][rot_dims / 2] (cosine, sine)
};
struct BandArgs {
    QkvArgs p;
    const float* q;                    // rows: [M][n_q * dkp] prepared queries
    void *k_cache, *v_cache; int kv_bf16;
    KvPages pg;
    const int *row_pos, *row_seq; int seq0;
    const DecodeState* state;          // one vector: position comes from here; the cache pointers and pages are the sequence's own
    int M, window, max_seq, max_batch;
    int chunk;                         // > 0: keys of the query's own chunk of positions only
    // two maps: o = a1 - lambda a2, lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff, then RMS norm over the head's dv values, times 1 - diff
    const float *lq1, *lk1, *lq2, *lk2; float diff;
    const float *r1, *r2;              // distance bias r1[h] * ln(1 + r2[h] * distance), taken off the score (null: none)
    float* out_x;                      // one vector: [n_q * dv]
    int out_kind; RowOperand out;      // rows
    float* q_out;                      // launch_qkv_rows: [M][n_q * dkp]
    uint32_t* status;
    int use_pdl;
};
cudaError_t launch_qkv_rows(const BandArgs& a, cudaStream_t st);             // prepare M rows, append k / v
cudaError_t launch_band_rows(const BandArgs& a, int sm_count, cudaStream_t st);      // attention of M prepared rows (any sizes, any cache type)
cudaError_t launch_band_decode(const BandArgs& a, int sm_count, cudaStream_t st);    // one row, preparation and append included
bool band_supported(int n_q, int n_kv, int dkp, int dvp);
cudaError_t launch_qkv_head_rows(const BandArgs& a, cudaStream_t st);        // the same with QkvArgs::per_head

// Residual streams row by row: takes in a sublayer's output (or starts the streams from the embedding), and leaves the next sublayer's
// input — normalised, as an operand, or the plain sum u.
struct StreamRowsArgs {
    StreamArgs hc;                     // x: rows of n streams, [row][stream][ldx]; u: null, or rows ldx floats apart (then no norm)
    const float* y; int ldy;           // the sublayer's output rows; null: x_t = embedding row * scale for every t
    const void* table; int table_kind, vocab; const int* row_tok; const DecodeState* state; float scale;     // state: one vector, token and position from it
    const int* row_pos; int max_seq;
    int M, width;
    NormArgs norm; int kind; RowOperand out;
    uint32_t* status; int use_pdl;
};
cudaError_t launch_stream_rows(const StreamRowsArgs& a, cudaStream_t st);

// ---- gated linear recurrence (lum_recur.cu): u = conv(x) + bias; r, i = sigmoid(block-diagonal products of u + bias);
// ln a = -8 r softplus(lam); S = a S + sqrt(1 - a^2) i u; output S * y, y and x side by side as the projection left them (y activated)
struct RecurArgs {
    const float* yx; int ld, x_off;
    int width, blocks, bw, bwp;        // bwp: rows of a block's r (and of its i) in the gates' container, bw rounded up to 8
    const void* w_gate; int kind, kc, nt;      // container [kc chunks][blocks * (r: bwp | i: bwp)]
    const float *conv_b, *r_b, *i_b, *lam;
    ConvArgs conv;
    float* state; int max_batch;       // [sequence][width]
    const int *row_pos, *row_seq; int seq0; const DecodeState* step;      // step: one vector, position from it
    int M, max_seq;
    float* u; int ldu;                 // rows: u (launch_recur_conv), [width]
    RowOperand hi, lo;                 // rows: u as the gates' operand, two bf16 terms (f32: hi alone), block b at chunks b * kc
    const float* gates; int ldg;       // rows: products without bias, laid out as the container's rows
    int out_kind; RowOperand out;      // rows
    float* out_x;                      // one vector
    uint32_t* status; int use_pdl;
};
cudaError_t launch_recur_step(const RecurArgs& a, cudaStream_t st);          // rows of different sequences, or one row: everything in one kernel
cudaError_t launch_recur_conv(const RecurArgs& a, cudaStream_t st);          // many rows of one sequence: u and the gates' operand ...
cudaError_t launch_recur_scan(const RecurArgs& a, cudaStream_t st);          // ... and, after the gates' product, the recurrence
bool band_prompt_tc_supported(const BandArgs& a);                            // lum_attn_tc.cu: many rows of one sequence, bf16 cache
cudaError_t launch_band_prompt_tc(const BandArgs& a, cudaStream_t st);
inline int head_pad(int d) { return (d + 15) / 16 * 16; }

__device__ __forceinline__ float softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
// sp = softplus(p), sq = softplus(q) of the two learned numbers
__device__ __forceinline__ float xielu(float z, float sp, float sq) {
    return z > 0.0f ? fmaf(sp * z, z, 0.5f * z) : fmaf(0.5f + sq, expm1f(z) - z, 0.5f * z);
}
__device__ __forceinline__ float gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z))); }
__device__ __forceinline__ float sigmoid(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
__device__ __forceinline__ float clamped_gate(float g, float u, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * sigmoid(1.702f * g) * (u + 1.0f);
}
// score correction of a key `d` positions back
__device__ __forceinline__ float distance_bias(float r1, float r2, float d) { return r1 * log1pf(r2 * d); }

}  // namespace lum
