// Parameter blocks and launchers of the dense-weight, post-norm decoder path: projections with bf16 or
// fp32 weights, windowed attention whose queries and keys are normalised over the whole projection, a
// Mamba-2 (state-space duality) recurrence, and residual adds of normalised sublayer outputs.
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
__device__ __forceinline__ float softplus_p(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// ---------------------------------------------------------------------------
// A residual update that its consumer performs: x = h + m * rsqrt(sum(ss) / H + eps) * w, where m is the
// raw output of the sublayer before it and ss its partial sums of squares.  The consumer also stores x
// to hout (a buffer other than h: other CTAs still read h).  m == null: x = h, nothing is stored.
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

// ---- decode projection (csrc/gemv_dense.cu), 1..8 rows
#define DG_STORE 0           // out (element type) = y
#define DG_SILU_PAIR 1       // out (element type) = silu(gate) * up, weight rows interleaved by 8
#define DG_STORE_F32 2       // out (fp32) = y, or softcap * tanh(y / softcap); ss_out: partial sums of y^2
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
};
#define DG_FMA_ROWS 2        // bf16 rows up to which the FMA kernel serves

// ---- many-row projection in fp32 (csrc/gemm_f32.cu); same epilogues
struct GemmF32Params {
    const float* w; const float* x; void* out;
    int ldw, ldx, K, N, T, ldo, mode, pad;
    float softcap; int pad1;
};

// ---- one parallel mixer: windowed attention beside a state-space recurrence (csrc/attention_window.cu,
// csrc/ssd.cu).  Both read columns of the same projection row [q | k | z | x | B | C | dt] and write
// columns [attention | recurrence] of one row, the input of a common output projection.
struct MixLayer {
    // attention: H query heads over G key/value heads of size d (dp: d rounded up to 8, the row length
    // of the padded q buffer and of the caches); the values are the keys as projected
    int H, G, d, dp, rot, window;            // window <= 0: unlimited
    float attn_scale, left_scale, right_scale, eps;
    const float* q_norm; const float* k_norm;             // [H*d], [G*d]
    const float* cos_tab; const float* sin_tab;           // [max_seq][rot/2]
    void* kcache; void* vcache;                           // [slot][max_seq][G][dp]
    // recurrence: heads of size P, state N, groups of heads sharing B and C, norm over ngroups parts
    int heads, P, N, groups, ngroups, taps;
    const float* conv_w; const float* conv_b;             // [C][taps], [C]; C = heads*P + 2*groups*N
    const float* dt_bias; const float* A_log; const float* D; const float* norm_w;
    float* state;                                         // [slot][heads][N][P]
    void* conv_state;                                     // [slot][taps-1][C] raw inputs, oldest first
    int off_q, off_k, off_z, off_x, off_dt, max_seq;      // columns of the projection row
};

struct MixRun {
    const void* proj; int ld_proj; int dt;
    const RowMeta* rows; const int* seq_rows;             // rows of one sequence are consecutive
    int n_rows, n_seqs;
    void* qbuf;              // [rows][H][dp] normalised, rotated queries
    void* xbc; int ld_xbc; int pad;                   // [rows][ld_xbc] x | B | C after convolution and SiLU
    float* dtb; int ld_dt; int splits;                    // [rows][ld_dt] step sizes; cache slices per attention row
    float* ubuf; int ld_u; int fuse_norm;                 // [rows][ld_u] recurrence output times SiLU(z), before the norm
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
B2_API int b2_mix_prepare(const MixLayer* l, const MixRun* r, cudaStream_t s);
B2_API int b2_window_attn_decode(const MixLayer* l, const MixRun* r, cudaStream_t s);
B2_API int b2_window_attn_rows(const MixLayer* l, const MixRun* r, cudaStream_t s);
B2_API int b2_ssd_step(const MixLayer* l, const MixRun* r, cudaStream_t s);
B2_API int b2_ssd_chunk(const MixLayer* l, const MixRun* r, cudaStream_t s);
#define SSD_CHUNK 64
