// Many-row projection in true fp32 (no reduced-precision matrix mode): out[t][n] = sum_k x[t][k] w[n][k].
// It serves models that run entirely in 32 bits; 64 x 64 tiles on the FMA pipes, K in steps of 16, each
// output summed by one thread in ascending k.
#include "mixers.cuh"

#define GF_T 64
#define GF_K 16

__global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32Params p) {
    __shared__ float xs[GF_K][GF_T + 4], ws[GF_K][GF_T + 4];
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int t0 = blockIdx.y * GF_T, n0 = blockIdx.x * GF_T;
    // columns of a thread: (tx & 7) and (tx & 7) + 8 of two 16-wide groups, so that it holds gate and up
    // of the rows interleaved by 8
    int nl[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) nl[j] = ((tx >> 3) * 2 + (j >> 1)) * 16 + (tx & 7) + 8 * (j & 1);
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < p.K; k0 += GF_K) {
        for (int i = tid; i < GF_T * GF_K; i += 256) {
            const int r = i / GF_K, c = i % GF_K;
            xs[c][r] = (t0 + r < p.T && k0 + c < p.K) ? p.x[(size_t)(t0 + r) * p.ldx + k0 + c] : 0.f;
            ws[c][r] = (n0 + r < p.N && k0 + c < p.K) ? p.w[(size_t)(n0 + r) * p.ldw + k0 + c] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < GF_K; ++c) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = xs[c][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = ws[c][nl[j]];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = t0 + ty * 4 + i;
        if (t >= p.T) continue;
        if (p.mode == DG_GATE_PAIR) {
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int n = n0 + nl[j], o = (n >> 4) * 8 + (n & 7);
                if (n + 8 < p.N) ((float*)p.out)[(size_t)t * p.ldo + o] = (p.act == ACT_RELU ? fmaxf(acc[i][j], 0.f) : silu_p(acc[i][j])) * acc[i][j + 1];
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int n = n0 + nl[j];
                if (n < p.N) {
                    const float v = acc[i][j];
                    ((float*)p.out)[(size_t)t * p.ldo + n] =
                        (p.mode == DG_STORE_F32 && p.softcap > 0.f) ? p.softcap * tanhf(v / p.softcap)
                                                                    : (p.mode == DG_STORE && n < p.act_cols ? silu_p(v) : v);
                }
            }
        }
    }
}

B2_API int b2_gemm_f32(const GemmF32Params* p, cudaStream_t s) {
    if (p->T < 1 || p->N < 1 || p->K < 1 || p->ldx < p->K || p->ldw < p->K) return cudaErrorInvalidValue;
    if (p->mode == DG_GATE_PAIR && (p->N & 15)) return cudaErrorInvalidValue;
    dim3 grid((p->N + GF_T - 1) / GF_T, (p->T + GF_T - 1) / GF_T);
    return launch_pdl(gemm_f32_kernel, grid, dim3(256), 0, s, *p);
}
B2_API int b2_sizeof_gemm_f32_params() { return (int)sizeof(GemmF32Params); }
