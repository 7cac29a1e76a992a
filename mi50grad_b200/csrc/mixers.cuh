// Parameter blocks and launchers of the dense-weight decoder path: projections with bf16 or fp32 weights,
// windowed attention, linear recurrences (Mamba-2 / state-space duality, lightning attention), residual adds
// of normalised sublayer outputs (post-norm), and residual streams joined by hyper-connections (pre-norm).
//
// Every kernel exists for two element types of weights, activations and caches, selected by `dt`:
// bf16 (what serving uses) and fp32 (everything in 32 bits).  Positions, angles, scores, norms, the
// residual stream and the recurrence are fp32 in both.
#pragma once
#include <cuda_bf16.h>
#include "common.cuh"

#define DT_BF16 0
#define DT_F32 1

typedef __nv_bfloat16 bf16;

template <typename T> __device__ __forceinline__ float ld_f(const T* p);
template <> __device__ __forceinline__ float ld_f<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ld_f<bf16>(const bf16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ T to_t(float v);
template <> __device__ __forceinline__ float to_t<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 to_t<bf16>(float v) { return __float2bfloat16(v); }
// SiLU with the precise exponential (the 16-bit paths keep silu_f)
__device__ __forceinline__ float silu_p(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid_p(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_p(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// ---------------------------------------------------------------------------
// A residual update that its consumer performs: x = h + m * rsqrt(sum(ss) / H + eps) * w, where m is the
// raw output of the sublayer before it and ss its partial sums of squares.  The consumer also stores x
// to hout (a buffer other than h: other CTAs still read h).  m == null: x = h, nothing is stored.
// h == null: x = m * rsqrt(sum(ss) / H + eps) * w, the plain norm of m (pre-norm decoders); nothing is stored.
// ---------------------------------------------------------------------------
struct PostNorm {
    const float* h;          // [rows][H]
    const float* m;          // [rows][H]
    const float* w;          // [H]
    const float* ss;         // [rows][np]
    float* hout;             // [rows][H]
    int np, H;
    float eps;
    int pad;
};

// ---------------------------------------------------------------------------
// Hyper-connections: a row has `n` residual streams x_0 .. x_(n-1).  Between two sublayers
//     X' = Mix^T X + Out y^T,   u = In^T X'     (X: the streams as rows; y: output of the sublayer before, u: input
// of the next one, before its norm).  coef: Mix [n][n] | Out [n] | In [n].
// ---------------------------------------------------------------------------
struct StreamMix {
    float* x;                // [rows][n][H], updated in place
    float* u;                // [rows][H]
    const float* coef;
    int n, pad;
};
#define STREAMS_MAX 16

// W adjacent columns of one row (x: the row's first stream at the column): updates the streams, y -> u.
template <int N, int W>
__device__ __forceinline__ void stream_mix_n(float* x, const float* coef, int H, float (&y)[W]) {
    float v[N][W], u[W];
#pragma unroll
    for (int s = 0; s < N; ++s) {
        if constexpr (W == 4) *(float4*)v[s] = *(const float4*)(x + (size_t)s * H);
        else
#pragma unroll
            for (int e = 0; e < W; ++e) v[s][e] = x[(size_t)s * H + e];
    }
#pragma unroll
    for (int e = 0; e < W; ++e) u[e] = 0.f;
#pragma unroll
    for (int t = 0; t < N; ++t) {
        float o[W];
#pragma unroll
        for (int e = 0; e < W; ++e) {
            o[e] = coef[N * N + t] * y[e];
#pragma unroll
            for (int s = 0; s < N; ++s) o[e] = fmaf(coef[s * N + t], v[s][e], o[e]);
            u[e] = fmaf(coef[N * N + N + t], o[e], u[e]);
        }
        if constexpr (W == 4) *(float4*)(x + (size_t)t * H) = *(const float4*)o;
        else
#pragma unroll
            for (int e = 0; e < W; ++e) x[(size_t)t * H + e] = o[e];
    }
#pragma unroll
    for (int e = 0; e < W; ++e) y[e] = u[e];
}
template <int W>
__device__ __forceinline__ void stream_mix(int n, float* x, const float* coef, int H, float (&y)[W]) {
    switch (n) {
        case 1: stream_mix_n<1, W>(x, coef, H, y); return;
        case 2: stream_mix_n<2, W>(x, coef, H, y); return;
        case 3: stream_mix_n<3, W>(x, coef, H, y); return;
        case 4: stream_mix_n<4, W>(x, coef, H, y); return;
    }
#pragma unroll
    for (int e = 0; e < W; ++e) {
        float v[STREAMS_MAX], u = 0.f;
#pragma unroll 1
        for (int s = 0; s < n; ++s) v[s] = x[(size_t)s * H + e];
#pragma unroll 1
        for (int t = 0; t < n; ++t) {
            float o = coef[n * n + t] * y[e];
#pragma unroll 1
            for (int s = 0; s < n; ++s) o = fmaf(coef[s * n + t], v[s], o);
            x[(size_t)t * H + e] = o;
            u = fmaf(coef[n * n + n + t], o, u);
        }
        y[e] = u;
    }
}

// ---- decode projection (csrc/gemv_dense.cu), 1..8 rows
#define DG_STORE 0           // out (element type) = y; SiLU on the first act_cols outputs
#define DG_GATE_PAIR 1       // out (element type) = act(gate) * up, weight rows interleaved by 8
#define DG_STORE_F32 2       // out (fp32) = y, or softcap * tanh(y / softcap); ss_out: partial sums of y^2
#define DG_STREAMS 3         // hyper-connections: y goes into the streams `sm`, u of the next sublayer comes out;
                             // ss_out: partial sums of u^2
#define ACT_SILU 0
#define ACT_RELU 1
struct DenseGemvParams {
    const void* w;           // [N][ldw], columns K .. ldw-1 zero, ldw a multiple of 8
    const void* x;           // [rows][ldx] activations (null: the input is pn)
    PostNorm pn;
    void* out;
    float* ss_out;           // DG_STORE_F32, optional: [rows][ss_np], entry of CTA i = sum over its outputs
    int ldw, ldx, K, N, rows, ldo, mode, dt;
    int rpc;                 // outputs per CTA, see b2_gemv_dense
    int ss_np;
    float softcap;
    int mma;                 // 1: tensor-core kernel for any number of bf16 rows
    int act, act_cols;       // DG_GATE_PAIR: ACT_*; DG_STORE: outputs that get SiLU
    StreamMix sm;            // DG_STREAMS
};
#define DG_FMA_ROWS 2        // bf16 rows up to which the FMA kernel serves

// ---- many-row projection in fp32 (csrc/gemm_f32.cu); same epilogues
struct GemmF32Params {
    const float* w; const float* x; void* out;
    int ldw, ldx, K, N, T, ldo, mode, act;
    float softcap; int act_cols;
};

// ---- one mixer: windowed attention and / or a linear recurrence (csrc/attention_window.cu, csrc/ssd.cu).
// They read columns of a projection row ([q | k | z | x | B | C | dt] of a parallel mixer, [q | k | v] of an
// attention, [q | k | v | g] of a lightning attention) and write columns of one row, the input of the output
// projection.
struct MixLayer {
    // attention: H query heads over G key/value heads of size d (values: dv); dp, vp: d, dv rounded up to 8,
    // the head lengths of the padded q buffer and of the caches
    int H, G, d, dp, rot, window;            // window <= 0: unlimited
    float attn_scale, left_scale, right_scale, eps;       // left_scale, right_scale multiply the columns written
    const float* q_norm; const float* k_norm;             // [H*d], [G*d], or with head_norm [d]
    const float* cos_tab; const float* sin_tab;           // [max_seq][rot/2]
    void* kcache; void* vcache;                           // [slot][max_seq][G][dp], [..][vp]
    const float* sink;                                    // [H] one more term exp(sink) in the soft-max's denominator, or null
    int dv, vp, off_v;                                    // off_v < 0: the values are the keys as projected
    int head_norm;                                        // 0: norms over the whole projection, 1: per head
    int keep_first;                                       // slots [0, keep_first) stay visible beyond the window
    float softcap;                                        // > 0: scores become softcap * tanh(score / softcap)
    // recurrence: heads of size P, state N, groups of heads sharing B and C.  Decay and step size per token
    // (dt, A_log) or, with `decay`, constant per head with step size one.
    int heads, P, N, groups, ngroups, taps;
    const float* conv_w; const float* conv_b;             // [C][taps], [C]; C = heads*P + 2*groups*N
    const float* dt_bias; const float* A_log; const float* D; const float* norm_w;      // D null: no direct term
    const float* decay; const float* log_decay;           // [heads], or null
    float* state;                                         // [slot][heads][N][P]
    void* conv_state;                                     // [slot][taps-1][C] raw inputs, oldest first
    int off_q, off_k, off_z, off_x, off_dt, max_seq;      // columns of the projection row
    int rx, rB, rC;                                       // columns of x, B and C in a row of MixRun::xbc
    int gate;                                             // REC_GATE_*
    int out_col;                                          // column of the output row where the recurrence starts
    int exact_weights;                                    // prompt attention: 1 = soft-max weights keep all 24 bits in the
                                                          // product with V (always so with a softcap), 0 = rounded to bf16
};
#define REC_GATE_SILU_NORM 0   // norm(y * silu(z)) in ngroups equal parts
#define REC_NORM_SIGMOID 1     // norm(y) * sigmoid(z)

static inline bool attn_valid(const MixLayer* l) {
    return l->H >= 1 && l->G >= 1 && l->H % l->G == 0 && l->d >= 1 && l->dp >= l->d && l->dp <= 256 && !(l->dp & 7) && l->dv >= 1 &&
           l->vp >= l->dv && l->vp <= 256 && !(l->vp & 7) && l->rot <= l->d && !(l->rot & 1) && l->keep_first >= 0;
}

struct MixRun {
    const void* proj; int ld_proj; int dt;
    const RowMeta* rows; const int* seq_rows;             // rows of one sequence are consecutive
    int n_rows, n_seqs;
    void* qbuf;              // [rows][H][dp] normalised, rotated queries
    void* xbc; int ld_xbc; int pad;                   // [rows][ld_xbc] x | B | C after convolution and SiLU (lightning: the projection rows)
    float* dtb; int ld_dt; int splits;                    // [rows][ld_dt] step sizes; cache slices per attention row
    float* ubuf; int ld_u; int fuse_norm;                 // [rows][ld_u] what the recurrence's norm is taken of
    void* out; int ldo; int commit;                       // [rows][ldo]; commit 0: leave recurrent state alone
    float* attn_scratch; int* attn_counters; int* ssd_counters;     // counters are zero between launches
    // chunked scan
    float* chunk_state;      // [chunks][heads][N][P] local states
    void* chunk_prev;        // [chunks][heads][3][N][Pp] bf16 planes of the state before each chunk
    float* chunk_decay;      // [chunks][heads] total log decay
};

B2_API int b2_gemv_dense(const DenseGemvParams* p, cudaStream_t s);
B2_API int b2_gemm_f32(const GemmF32Params* p, cudaStream_t s);
B2_API int b2_embed_rows(const void* embed, const int* row_tokens, const void* rows, const void* seqs, float* h, void* xb,
                         int ldx, int n_rows, int H, int vocab, int dt, cudaStream_t s);
B2_API int b2_post_norm(float* h, const float* m, const float* w, const float* final_w, void* xb, int ldx, int n_rows, int H,
                        float eps, int dt, int planes, long long plane_stride, cudaStream_t s);
// Embedding rows (row_tokens: a token or < 0 for the sequence's own; null: rows of h) times scale into every
// stream; then u, its norm as xb (element type) and, optionally, u itself.
struct StreamRows {
    StreamMix sm;
    const float* y; long long plane_stride; int planes, pad0;    // sublayer output [rows][H], as a sum of planes (or null)
    const float* w;          // norm weight [H]
    void* xb; int ldx, rows, H, dt;
    float eps, scale;
    // embedding
    const void* embed; int ld_embed, vocab;
    const int* row_tokens; const RowMeta* meta; const SeqState* seqs; const float* h;    // embed null: rows of h [rows][H]
    int from_embedding, pad;
};
B2_API int b2_stream_rows(const StreamRows* p, cudaStream_t s);
B2_API int b2_mix_prepare(const MixLayer* l, const MixRun* r, cudaStream_t s);
B2_API int b2_head_prepare(const MixLayer* l, const MixRun* r, cudaStream_t s);
B2_API int b2_window_attn_decode(const MixLayer* l, const MixRun* r, cudaStream_t s);
B2_API int b2_window_attn_rows(const MixLayer* l, const MixRun* r, cudaStream_t s);
B2_API int b2_ssd_step(const MixLayer* l, const MixRun* r, cudaStream_t s);
B2_API int b2_ssd_chunk(const MixLayer* l, const MixRun* r, cudaStream_t s);
#define SSD_CHUNK 64
