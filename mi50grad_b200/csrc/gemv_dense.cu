// Decode projection with dense bf16 or fp32 weights, 1..8 token rows, fp32 accumulation.
//
// A CTA of eight warps owns rpc = 8, 16 or 32 outputs; a warp holds four output rows and a slice of K, so
// that small matrices still give every SM a CTA and no reduction leaves the CTA (bitwise the same sum
// whatever runs beside it).  The first weight blocks are requested before the dependency wait: with
// programmatic dependent launch they travel while the kernel before this one finishes.
//
// The input is either an activation row, or the residual stream together with the raw output of the
// sublayer before it (PostNorm): every CTA forms x = h + norm(m) * w while it stages its input, and the
// CTAs share out storing the updated stream.  That removes the serial "normalise and add" launch of a
// post-norm block.
#include "mixers.cuh"

#define DG_THREADS 256
#define DG_WARPS 8
#define DG_U 2                   // weight blocks per row and lane in flight, twice (current and next)

template <typename T> struct DgVec;
template <> struct DgVec<bf16> {
    static constexpr int V = 8;
    static __device__ __forceinline__ void unpack(const uint4& u, float (&f)[8]) {
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(w[i] << 16); f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u); }
    }
};
template <> struct DgVec<float> {
    static constexpr int V = 4;
    static __device__ __forceinline__ void unpack(const uint4& u, float (&f)[4]) {
        f[0] = __uint_as_float(u.x); f[1] = __uint_as_float(u.y); f[2] = __uint_as_float(u.z); f[3] = __uint_as_float(u.w);
    }
};

template <typename T, int MR>
__global__ void __launch_bounds__(DG_THREADS) gemv_dense_kernel(const DenseGemvParams p, int KC) {
    constexpr int V = DgVec<T>::V;
    extern __shared__ __align__(16) unsigned char dg_smem[];
    T* xs = (T*)dg_smem;                                    // [MR][KC]
    __shared__ float red[DG_WARPS][4][MR];
    __shared__ float y_s[32][MR];
    __shared__ float inv_s[B2_MAX_ROWS];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int WN = p.rpc >> 2, WK = DG_WARPS / WN;
    const int wn = warp % WN, wk = warp / WN;
    const int STRIDE = WK * 32 * V;
    const int Kp = (p.K + V - 1) / V * V;                   // (weights are zero-padded up to ldw >= Kp)
    const int n0 = blockIdx.x * p.rpc;
    const T* wr[4];
#pragma unroll
    for (int r = 0; r < 4; ++r) wr[r] = (const T*)p.w + (size_t)min(n0 + wn * 4 + r, p.N - 1) * p.ldw;
    float acc[4][MR];
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int m = 0; m < MR; ++m) acc[r][m] = 0.f;
    int k = (wk * 32 + lane) * V;
    uint4 cur[DG_U][4], nxt[DG_U][4];
    auto load = [&](uint4 (&dst)[DG_U][4], int kk) {
#pragma unroll
        for (int u = 0; u < DG_U; ++u)
#pragma unroll
            for (int r = 0; r < 4; ++r)
                dst[u][r] = kk + u * STRIDE < Kp ? ldg_nc_v4(wr[r] + kk + u * STRIDE) : make_uint4(0u, 0u, 0u, 0u);
    };
    load(cur, k);
    pdl_wait();                                             // from here on: what earlier kernels of the step wrote
    if (!p.x && p.pn.m) {
        if (warp < p.rows) {
            float s = 0.f;
            for (int i0 = lane; i0 < p.pn.np; i0 += 128) {
                float v[4];
#pragma unroll
                for (int u = 0; u < 4; ++u) v[u] = i0 + 32 * u < p.pn.np ? p.pn.ss[(size_t)warp * p.pn.np + i0 + 32 * u] : 0.f;
                s += (v[0] + v[1]) + (v[2] + v[3]);
            }
            s = warp_sum(s);
            if (lane == 0) inv_s[warp] = rsqrtf(s / (float)p.pn.H + p.pn.eps);
        }
        __syncthreads();
    }
    for (int c0 = 0; c0 < Kp; c0 += KC) {
        const int cl = min(KC, Kp - c0);
        // ---- stage the input of this K chunk
        if (p.x) {
            const bool vec = (p.ldx % V) == 0;
            for (int i = tid * V; i < p.rows * KC; i += DG_THREADS * V) {
                const int m = i / KC, kk = i % KC;
                if (kk >= cl) continue;
                const T* src = (const T*)p.x + (size_t)m * p.ldx + c0 + kk;
                if (vec && c0 + kk + V <= p.K) *(uint4*)(xs + i) = *(const uint4*)src;
                else
                    for (int e = 0; e < V; ++e) xs[i + e] = c0 + kk + e < p.K ? src[e] : to_t<T>(0.f);
            }
        } else {
            const PostNorm& n = p.pn;
            const bool vec = (n.H & 3) == 0;
#pragma unroll 2
            for (int i = tid * 4; i < p.rows * KC; i += DG_THREADS * 4) {
                const int m = i / KC, kk = i % KC, kg = c0 + kk;
                if (kk >= cl) continue;
                float v[4];
                const size_t o = (size_t)m * n.H + kg;
                if (vec && kg + 4 <= p.K) {
                    const float4 h4 = *(const float4*)(n.h + o);
                    v[0] = h4.x; v[1] = h4.y; v[2] = h4.z; v[3] = h4.w;
                    if (n.m) {
                        const float4 m4 = *(const float4*)(n.m + o), w4 = *(const float4*)(n.w + kg);
                        const float inv = inv_s[m];
                        v[0] += m4.x * inv * w4.x; v[1] += m4.y * inv * w4.y; v[2] += m4.z * inv * w4.z; v[3] += m4.w * inv * w4.w;
                        if ((kg >> 2) % (int)gridDim.x == (int)blockIdx.x) *(float4*)(n.hout + o) = make_float4(v[0], v[1], v[2], v[3]);
                    }
                } else {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        v[e] = 0.f;
                        if (kg + e < p.K) {
                            v[e] = n.h[o + e];
                            if (n.m) {
                                v[e] += n.m[o + e] * inv_s[m] * n.w[kg + e];
                                if ((kg >> 2) % (int)gridDim.x == (int)blockIdx.x) n.hout[o + e] = v[e];
                            }
                        }
                    }
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) xs[i + e] = to_t<T>(v[e]);
            }
        }
        __syncthreads();
        // ---- multiply; KC is a multiple of DG_U * STRIDE, so a lane's blocks never straddle two chunks
        for (; k < c0 + cl; k += DG_U * STRIDE) {
            load(nxt, k + DG_U * STRIDE);
#pragma unroll
            for (int u = 0; u < DG_U; ++u) {
                const int kk = k + u * STRIDE;
                if (kk < Kp) {
                    float wf[4][V];
#pragma unroll
                    for (int r = 0; r < 4; ++r) DgVec<T>::unpack(cur[u][r], wf[r]);
#pragma unroll
                    for (int m = 0; m < MR; ++m) {
                        if (m < p.rows) {
                            float xf[V];
                            DgVec<T>::unpack(*(const uint4*)(xs + (size_t)m * KC + kk - c0), xf);
#pragma unroll
                            for (int r = 0; r < 4; ++r)
#pragma unroll
                                for (int e = 0; e < V; ++e) acc[r][m] = fmaf(wf[r][e], xf[e], acc[r][m]);
                        }
                    }
                }
            }
#pragma unroll
            for (int u = 0; u < DG_U; ++u)
#pragma unroll
                for (int r = 0; r < 4; ++r) cur[u][r] = nxt[u][r];
        }
        __syncthreads();
    }
    // ---- sums over lanes, then over the K slices, in a fixed order
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int m = 0; m < MR; ++m) {
            const float v = warp_sum(acc[r][m]);
            if (lane == 0) red[warp][r][m] = v;
        }
    __syncthreads();
    if (tid < p.rpc * MR) {
        const int nl = tid / MR, m = tid % MR;
        float v = 0.f;
        for (int q = 0; q < WK; ++q) v += red[q * WN + (nl >> 2)][nl & 3][m];
        y_s[nl][m] = v;
    }
    __syncthreads();
    if (p.mode == DG_SILU_PAIR) {
        const int half = p.rpc >> 1;
        if (tid < half * MR) {
            const int j = tid / MR, m = tid % MR, nl = (j >> 3) * 16 + (j & 7);
            const int o = blockIdx.x * half + j;
            if (m < p.rows && 2 * o < p.N) ((T*)p.out)[(size_t)m * p.ldo + o] = to_t<T>(silu_p(y_s[nl][m]) * y_s[nl + 8][m]);
        }
        return;
    }
    if (tid < p.rpc * MR) {
        const int m = tid / p.rpc, nl = tid % p.rpc, n = n0 + nl;
        if (m < p.rows && n < p.N) {
            const float v = y_s[nl][m];
            if (p.mode == DG_STORE) ((T*)p.out)[(size_t)m * p.ldo + n] = to_t<T>(v);
            else ((float*)p.out)[(size_t)m * p.ldo + n] = p.softcap > 0.f ? p.softcap * tanhf(v / p.softcap) : v;
        }
    }
    if (p.mode == DG_STORE_F32 && p.ss_out && warp < p.rows) {
        float v = (lane < p.rpc && n0 + lane < p.N) ? y_s[lane][warp % MR] : 0.f;
        v = warp_sum(v * v);
        if (lane == 0) p.ss_out[(size_t)warp * p.ss_np + blockIdx.x] = v;
    }
}

template <typename T, int MR>
static int launch_dg(const DenseGemvParams* p, cudaStream_t s) {
    const int WK = DG_WARPS / (p->rpc >> 2);
    const int unit = DG_U * WK * 32 * DgVec<T>::V;
    const int cap = 65536 * (int)sizeof(T) / 2 / (MR * (int)sizeof(T));
    int KC = (p->K + unit - 1) / unit * unit;
    if (KC > cap) KC = cap / unit * unit;
    const size_t smem = (size_t)MR * KC * sizeof(T);
    static SmemOptIn opt;
    if (int e = opt.ensure((const void*)gemv_dense_kernel<T, MR>, smem)) return e;
    return launch_pdl(gemv_dense_kernel<T, MR>, dim3((p->N + p->rpc - 1) / p->rpc), dim3(DG_THREADS), smem, s, *p, KC);
}
template <typename T>
static int launch_dg_rows(const DenseGemvParams* p, cudaStream_t s) {
    if (p->rows == 1) return launch_dg<T, 1>(p, s);
    if (p->rows == 2) return launch_dg<T, 2>(p, s);
    if (p->rows <= 4) return launch_dg<T, 4>(p, s);
    return launch_dg<T, 8>(p, s);
}

B2_API int b2_gemv_dense(const DenseGemvParams* p, cudaStream_t s) {
    if (p->rows < 1 || p->rows > B2_MAX_ROWS || p->K < 1 || p->N < 1 || (p->ldw & 7) || p->ldw < p->K || ((uintptr_t)p->w & 15))
        return cudaErrorInvalidValue;
    if (p->rpc != 8 && p->rpc != 16 && p->rpc != 32) return cudaErrorInvalidValue;
    if (p->mode == DG_SILU_PAIR && (p->rpc < 16 || (p->N & 15))) return cudaErrorInvalidValue;
    if (p->x ? (p->ldx < p->K || ((uintptr_t)p->x & 15)) : (!p->pn.h || p->pn.H != p->K)) return cudaErrorInvalidValue;
    if (p->ss_out && (p->N + p->rpc - 1) / p->rpc > p->ss_np) return cudaErrorInvalidValue;
    if (p->dt == DT_BF16) return launch_dg_rows<bf16>(p, s);
    if (p->dt == DT_F32) return launch_dg_rows<float>(p, s);
    return cudaErrorInvalidValue;
}
B2_API int b2_sizeof_dense_gemv_params() { return (int)sizeof(DenseGemvParams); }
