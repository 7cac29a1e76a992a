// Decode projection with dense bf16 or fp32 weights, 1..8 token rows, fp32 accumulation.
//
// bf16: the tensor core as an fp32-accumulating dot-product engine.  A warp owns 16 outputs and a slice of K;
// a lane's 16-byte weight loads hold eight consecutive k of one output row, and because the order of k inside
// a product is free, those bytes ARE the A fragments of two m16n8k16 steps, no re-packing needed, as long as
// the activations (B, token rows in the 8-wide dimension) are read with the same permutation: one 16-byte
// shared-memory load.  Per 32 k: two global loads, one shared load, two MMAs, whatever the number of rows.
// One or two rows, and fp32, run on the FMA pipes instead: there a warp's load covers 512 contiguous bytes of a
// weight row, which HBM answers faster than the eight 64-byte pieces of a fragment load.
//
// All reductions stay inside a CTA (bitwise the same sum whatever runs beside it).  The first weight blocks
// are requested before the dependency wait: with programmatic dependent launch they travel while the kernel
// before this one finishes.
//
// The input is either an activation row, or the residual stream together with the raw output of the
// sublayer before it (PostNorm): every CTA forms x = h + norm(m) * w while it stages its input, and the
// CTAs share out storing the updated stream.  That removes the serial "normalise and add" launch of a
// post-norm block.  In a pre-norm block with several residual streams the projection that ends a sublayer updates
// the streams in its epilogue and leaves the next sublayer's input with partial sums of squares; the next
// projection normalises it while it stages (PostNorm without h).
#include "mixers.cuh"

#define DG_THREADS 256
#define DG_WARPS 8
#define DG_U 2                   // weight blocks per row and lane in flight, twice (current and next)


// ---------------------------------------------------------------------------
// bf16
// ---------------------------------------------------------------------------
#define DM_D 4                   // 64-k weight blocks of a warp in flight
#define DM_PAD 32                // elements of padding per staged row: eight lanes' 16-byte reads cover all banks

__device__ __forceinline__ void dm_mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t dm_pack(float a, float b) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    return *(const uint32_t*)&h;
}

// 1 / rms of every row of a PostNorm input (warp r takes row r) into inv[]
__device__ __forceinline__ void pn_inverse(const PostNorm& n, int rows, float* inv, int warp, int lane) {
    if (warp >= rows) return;
    float s = 0.f;
    for (int i0 = lane; i0 < n.np; i0 += 256) {
        float v[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) v[u] = i0 + 32 * u < n.np ? n.ss[(size_t)warp * n.np + i0 + 32 * u] : 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u) s += v[u];
    }
    s = warp_sum(s);
    if (lane == 0) inv[warp] = rsqrtf(s / (float)n.H + n.eps);
}
// Four columns [k, k + 4) of row m of the updated stream; CTA (k / 4) mod gridDim stores them.  (EXT: see dg_extended)
template <bool EXT>
__device__ __forceinline__ void pn_load4(const PostNorm& n, int m, int k, const float* inv, float (&v)[4]) {
    const size_t o = (size_t)m * n.H + k;
    const bool mine = (k >> 2) % (int)gridDim.x == (int)blockIdx.x;
    if ((n.H & 3) == 0) {
        if (EXT && !n.h) {
            const float4 m4 = *(const float4*)(n.m + o), w4 = *(const float4*)(n.w + k);
            const float iv = inv[m];
            v[0] = m4.x * iv * w4.x; v[1] = m4.y * iv * w4.y; v[2] = m4.z * iv * w4.z; v[3] = m4.w * iv * w4.w;
            return;
        }
        const float4 h4 = *(const float4*)(n.h + o);
        v[0] = h4.x; v[1] = h4.y; v[2] = h4.z; v[3] = h4.w;
        if (n.m) {
            const float4 m4 = *(const float4*)(n.m + o), w4 = *(const float4*)(n.w + k);
            const float iv = inv[m];
            v[0] += m4.x * iv * w4.x; v[1] += m4.y * iv * w4.y; v[2] += m4.z * iv * w4.z; v[3] += m4.w * iv * w4.w;
            if (mine) *(float4*)(n.hout + o) = make_float4(v[0], v[1], v[2], v[3]);
        }
    } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            v[e] = 0.f;
            if (k + e < n.H) {
                if (EXT && !n.h) { v[e] = n.m[o + e] * inv[m] * n.w[k + e]; continue; }
                v[e] = n.h[o + e];
                if (n.m) { v[e] += n.m[o + e] * inv[m] * n.w[k + e]; if (mine) n.hout[o + e] = v[e]; }
            }
        }
    }
}

// Launches that need what only decoders over residual streams use (the plain norm of the input, the update of the
// streams, activations other than the SiLU pair) run instantiations of their own, so that the others stay lean.
static bool dg_extended(const DenseGemvParams& p) { return p.mode == DG_STREAMS || p.act || p.act_cols > 0 || (!p.x && !p.pn.h); }

// Finished [rpc][8] tile in y_s -> output (both element types).
template <typename T, bool EXT>
__device__ __forceinline__ void dg_epilogue(const DenseGemvParams& p, float (*y_s)[8], int tid, int lane, int warp) {
    const int n0 = blockIdx.x * p.rpc;
    if (p.mode == DG_GATE_PAIR) {
        const int half = p.rpc >> 1;
        for (int i = tid; i < half * p.rows; i += DG_THREADS) {
            const int m = i / half, j = i % half, nl = (j >> 3) * 16 + (j & 7), o = blockIdx.x * half + j;
            const float g = y_s[nl][m];
            if (2 * o < p.N) ((T*)p.out)[(size_t)m * p.ldo + o] = to_t<T>((EXT && p.act == ACT_RELU ? fmaxf(g, 0.f) : silu_p(g)) * y_s[nl + 8][m]);
        }
        return;
    }
    for (int i = tid; i < p.rpc * p.rows; i += DG_THREADS) {
        const int m = i / p.rpc, nl = i % p.rpc, n = n0 + nl;
        if (n >= p.N) continue;
        const float v = y_s[nl][m];
        if (p.mode == DG_STORE) ((T*)p.out)[(size_t)m * p.ldo + n] = to_t<T>(EXT && n < p.act_cols ? silu_p(v) : v);
        else if (EXT && p.mode == DG_STREAMS) {
            float y[1] = {v};
            stream_mix<1>(p.sm.n, p.sm.x + (size_t)m * p.sm.n * p.N + n, p.sm.coef, p.N, y);
            p.sm.u[(size_t)m * p.N + n] = y_s[nl][m] = y[0];
        } else ((float*)p.out)[(size_t)m * p.ldo + n] = p.softcap > 0.f ? p.softcap * tanhf(v / p.softcap) : v;
    }
    if (EXT && p.mode == DG_STREAMS) __syncthreads();
    if ((p.mode == DG_STORE_F32 || (EXT && p.mode == DG_STREAMS)) && p.ss_out && warp < p.rows) {
        float s = 0.f;
        for (int nl = lane; nl < p.rpc; nl += 32) if (n0 + nl < p.N) s += y_s[nl][warp] * y_s[nl][warp];
        s = warp_sum(s);
        if (lane == 0) p.ss_out[(size_t)warp * p.ss_np + blockIdx.x] = s;
    }
}

template <bool EXT>
__global__ void __launch_bounds__(DG_THREADS, 2) gemv_bf16_kernel(const DenseGemvParams p, int KC) {
    extern __shared__ __align__(16) unsigned char dg_smem[];
    bf16* xs = (bf16*)dg_smem;                              // [1 or 2][rows][KC + DM_PAD]
    __shared__ float red[DG_WARPS][16][8];
    __shared__ float y_s[128][8];
    __shared__ float inv_s[B2_MAX_ROWS];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int WN = p.rpc >> 4, WK = DG_WARPS / WN, wn = warp % WN, wk = warp / WN;
    const int Kp = (p.K + 7) & ~7, nb = (Kp + 63) >> 6;      // 64-k blocks; this warp's are wk, wk + WK, ...
    const int n0 = blockIdx.x * p.rpc + wn * 16;
    const bf16* w_lo = (const bf16*)p.w + (size_t)min(n0 + g, p.N - 1) * p.ldw + t * 8;
    const bf16* w_hi = (const bf16*)p.w + (size_t)min(n0 + g + 8, p.N - 1) * p.ldw + t * 8;
    uint4 buf[DM_D][4];
    auto load = [&](uint4 (&b)[4], int blk) {
        const int k = blk * 64;
        const bool a = k + t * 8 < Kp, c = k + 32 + t * 8 < Kp;
        const uint4 z = make_uint4(0u, 0u, 0u, 0u);
        b[0] = a ? ldg_nc_v4(w_lo + k) : z; b[1] = a ? ldg_nc_v4(w_hi + k) : z;
        b[2] = c ? ldg_nc_v4(w_lo + k + 32) : z; b[3] = c ? ldg_nc_v4(w_hi + k + 32) : z;
    };
#pragma unroll
    for (int d = 0; d < DM_D; ++d) load(buf[d], wk + WK * d);
    pdl_wait();                                             // from here on: what earlier kernels of the step wrote
    const int LDX = KC + DM_PAD;
    const int chunks = (Kp + KC - 1) / KC;
    auto stage = [&](int c) {                               // activations of K chunk c by cp.async, zero beyond K
        bf16* dst = xs + (size_t)(c & 1) * p.rows * LDX;
        const int c0 = c * KC, cl = min(KC, ((Kp - c0) + 63) & ~63);
        for (int i = tid; i < p.rows * (cl >> 3); i += DG_THREADS) {
            const int m = i / (cl >> 3), kk = (i % (cl >> 3)) * 8, k = c0 + kk;
            const bf16* src = (const bf16*)p.x + (size_t)m * p.ldx + k;
            bf16* d = dst + (size_t)m * LDX + kk;
            if (k + 8 <= p.K && (p.ldx & 7) == 0) cp_async16(d, src);
            else
                for (int e = 0; e < 8; ++e) d[e] = k + e < p.K ? src[e] : __float2bfloat16(0.f);
        }
        cp_async_commit();
    };
    if (p.x) stage(0);
    else {
        // (the launcher gives a PostNorm input one chunk)
        if (p.pn.m) { pn_inverse(p.pn, p.rows, inv_s, warp, lane); __syncthreads(); }
        const int kl = nb * 64;
#pragma unroll 4
        for (int i = tid * 4; i < p.rows * kl; i += DG_THREADS * 4) {
            const int m = i / kl, k = i % kl;
            float v[4] = {0.f, 0.f, 0.f, 0.f};
            if (k < p.K) pn_load4<EXT>(p.pn, m, k, inv_s, v);
            uint2 pk; pk.x = dm_pack(v[0], v[1]); pk.y = dm_pack(v[2], v[3]);
            *(uint2*)(xs + (size_t)m * LDX + k) = pk;
        }
    }
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    const bool live = g < p.rows;
    int blk = wk;                                           // (KC is a multiple of 64 * WK * DM_D)
    for (int c = 0; c < chunks; ++c) {
        if (c + 1 < chunks) { stage(c + 1); cp_async_wait<1>(); } else cp_async_wait<0>();
        __syncthreads();
        const bf16* xr = xs + ((size_t)(c & 1) * p.rows + (live ? g : 0)) * LDX + t * 8 - (size_t)c * KC;
        const int end = min(nb, (c + 1) * (KC >> 6));
        for (; blk < end; blk += WK * DM_D) {
#pragma unroll
            for (int d = 0; d < DM_D; ++d) {
                const int b = blk + WK * d;
                if (b < end) {
                    uint4 x0 = *(const uint4*)(xr + b * 64), x1 = *(const uint4*)(xr + b * 64 + 32);
                    if (!live) { x0 = make_uint4(0u, 0u, 0u, 0u); x1 = x0; }
                    dm_mma(acc, buf[d][0].x, buf[d][1].x, buf[d][0].y, buf[d][1].y, x0.x, x0.y);
                    dm_mma(acc, buf[d][0].z, buf[d][1].z, buf[d][0].w, buf[d][1].w, x0.z, x0.w);
                    dm_mma(acc, buf[d][2].x, buf[d][3].x, buf[d][2].y, buf[d][3].y, x1.x, x1.y);
                    dm_mma(acc, buf[d][2].z, buf[d][3].z, buf[d][2].w, buf[d][3].w, x1.z, x1.w);
                    load(buf[d], b + WK * DM_D);
                }
            }
        }
        if (c + 1 < chunks) __syncthreads();
    }
    *(float2*)&red[warp][g][2 * t] = make_float2(acc[0], acc[1]);
    *(float2*)&red[warp][g + 8][2 * t] = make_float2(acc[2], acc[3]);
    __syncthreads();
    for (int i = tid; i < p.rpc * 8; i += DG_THREADS) {
        const int nl = i >> 3, m = i & 7;
        float v = 0.f;
        for (int q = 0; q < WK; ++q) v += red[q * WN + (nl >> 4)][nl & 15][m];
        y_s[nl][m] = v;
    }
    __syncthreads();
    dg_epilogue<bf16, EXT>(p, y_s, tid, lane, warp);
}

template <bool EXT>
static int launch_dm(const DenseGemvParams* p, cudaStream_t s) {
    const int WK = DG_WARPS / (p->rpc >> 4), unit = 64 * WK * DM_D, Kr = (p->K + unit - 1) / unit * unit;
    int KC = Kr;
    const size_t cap = 64 << 10;
    bool two = false;
    if (p->x && (size_t)p->rows * Kr * 2 > cap) {           // K in double-buffered chunks
        two = true;
        KC = (int)(cap / 2 / ((size_t)p->rows * 2)) / unit * unit;
        if (KC < unit) KC = unit;
        if (KC >= Kr) { KC = Kr; two = false; }
    }
    const size_t smem = (size_t)(two ? 2 : 1) * p->rows * (KC + DM_PAD) * 2;
    if (smem > 200 << 10) return cudaErrorInvalidValue;     // (a PostNorm input wider than shared memory)
    static SmemOptIn opt;
    if (int e = opt.ensure((const void*)gemv_bf16_kernel<EXT>, smem)) return e;
    return launch_pdl(gemv_bf16_kernel<EXT>, dim3((p->N + p->rpc - 1) / p->rpc), dim3(DG_THREADS), smem, s, *p, KC);
}

// ---------------------------------------------------------------------------
// FMA pipes: fp32, and one or two bf16 rows
// ---------------------------------------------------------------------------
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

template <typename T, int MR, bool EXT>
__global__ void __launch_bounds__(DG_THREADS) gemv_fma_kernel(const DenseGemvParams p, int KC) {
    constexpr int V = DgVec<T>::V;
    extern __shared__ __align__(16) unsigned char dg_smem[];
    T* xs = (T*)dg_smem;                                 // [MR][KC]
    __shared__ float red[DG_WARPS][4][MR];
    __shared__ float y_s[32][8];
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
    if (!p.x && p.pn.m) { pn_inverse(p.pn, p.rows, inv_s, warp, lane); __syncthreads(); }
    for (int c0 = 0; c0 < Kp; c0 += KC) {
        const int cl = min(KC, Kp - c0);
        // ---- stage the input of this K chunk
        if (p.x && (p.ldx & 7) == 0) {
            for (int i = tid * V; i < p.rows * KC; i += DG_THREADS * V) {
                const int m = i / KC, kk = i % KC, kg = c0 + kk;
                if (kk >= cl) continue;
                const T* src = (const T*)p.x + (size_t)m * p.ldx + kg;
                if (kg + V <= p.K) *(uint4*)(xs + i) = *(const uint4*)src;
                else
                    for (int e = 0; e < V; ++e) xs[i + e] = kg + e < p.K ? src[e] : to_t<T>(0.f);
            }
        } else {
#pragma unroll 4
            for (int i = tid * 4; i < p.rows * KC; i += DG_THREADS * 4) {
                const int m = i / KC, kk = i % KC, kg = c0 + kk;
                if (kk >= cl) continue;
                float v[4] = {0.f, 0.f, 0.f, 0.f};
                if (!p.x) { if (kg < p.K) pn_load4<EXT>(p.pn, m, kg, inv_s, v); }
                else
#pragma unroll
                    for (int e = 0; e < 4; ++e) if (kg + e < p.K) v[e] = ld_f((const T*)p.x + (size_t)m * p.ldx + kg + e);
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
    dg_epilogue<T, EXT>(p, y_s, tid, lane, warp);
}

template <typename T, int MR, bool EXT>
static int launch_dg(const DenseGemvParams* p, cudaStream_t s) {
    const int WK = DG_WARPS / (p->rpc >> 2), unit = DG_U * WK * 32 * DgVec<T>::V, cap = 32768 / MR;
    int KC = (p->K + unit - 1) / unit * unit;
    if (KC > cap) KC = cap / unit * unit;
    const size_t smem = (size_t)MR * KC * sizeof(T);
    static SmemOptIn opt;
    if (int e = opt.ensure((const void*)gemv_fma_kernel<T, MR, EXT>, smem)) return e;
    return launch_pdl(gemv_fma_kernel<T, MR, EXT>, dim3((p->N + p->rpc - 1) / p->rpc), dim3(DG_THREADS), smem, s, *p, KC);
}

template <bool EXT>
static int launch_dg_rows(const DenseGemvParams* p, cudaStream_t s) {
    if (p->dt == DT_BF16) return p->rows == 1 ? launch_dg<bf16, 1, EXT>(p, s) : launch_dg<bf16, 2, EXT>(p, s);
    if (p->rows == 1) return launch_dg<float, 1, EXT>(p, s);
    if (p->rows == 2) return launch_dg<float, 2, EXT>(p, s);
    if (p->rows <= 4) return launch_dg<float, 4, EXT>(p, s);
    return launch_dg<float, 8, EXT>(p, s);
}

// rpc (outputs per CTA): 8, 16 or 32 in fp32 and for one or two bf16 rows, 16, 32, 64 or 128 for more bf16 rows
// (a gate / up pair needs at least 16).  mma: take the tensor-core kernel for one or two rows as well.
B2_API int b2_gemv_dense(const DenseGemvParams* p, cudaStream_t s) {
    if (p->rows < 1 || p->rows > B2_MAX_ROWS || p->K < 1 || p->N < 1 || (p->ldw & 7) || p->ldw < p->K || ((uintptr_t)p->w & 15))
        return cudaErrorInvalidValue;
    if (p->mode == DG_GATE_PAIR && (p->rpc < 16 || (p->N & 15))) return cudaErrorInvalidValue;
    if (p->x ? (p->ldx < p->K || ((uintptr_t)p->x & 15)) : ((!p->pn.h && !p->pn.m) || p->pn.H != p->K)) return cudaErrorInvalidValue;
    if (p->mode == DG_STREAMS && (p->sm.n < 1 || p->sm.n > STREAMS_MAX || !p->sm.x || !p->sm.u || !p->sm.coef)) return cudaErrorInvalidValue;
    if (p->ss_out && (p->N + p->rpc - 1) / p->rpc > p->ss_np) return cudaErrorInvalidValue;
    const bool ext = dg_extended(*p);
    const bool tc = p->dt == DT_BF16 && (p->mma || p->rows > DG_FMA_ROWS);
    if (tc) {
        if (p->rpc != 16 && p->rpc != 32 && p->rpc != 64 && p->rpc != 128) return cudaErrorInvalidValue;
        return ext ? launch_dm<true>(p, s) : launch_dm<false>(p, s);
    }
    if (p->rpc != 8 && p->rpc != 16 && p->rpc != 32) return cudaErrorInvalidValue;
    if (p->dt != DT_BF16 && p->dt != DT_F32) return cudaErrorInvalidValue;
    return ext ? launch_dg_rows<true>(p, s) : launch_dg_rows<false>(p, s);
}
B2_API int b2_sizeof_dense_gemv_params() { return (int)sizeof(DenseGemvParams); }
