// Row kernel of decoders with several residual streams joined by hyper-connections (pre-norm).  One launch
// does everything between two sublayers: the streams take the output of the sublayer before (a sum of
// planes when its projection was split over K), the next sublayer's input is formed from them and
// normalised.  In front of the first sublayer the streams are filled from the embedding instead; behind
// the last one the input weights are all one and the norm is the final norm.  The streams are fp32.
#include "mixers.cuh"

template <typename T>
__device__ __forceinline__ void store4(T* d, const float (&o)[4]) {
    if constexpr (sizeof(T) == 2) {
        const __nv_bfloat162 p0 = __floats2bfloat162_rn(o[0], o[1]), p1 = __floats2bfloat162_rn(o[2], o[3]);
        uint2 pk; pk.x = *(const uint32_t*)&p0; pk.y = *(const uint32_t*)&p1;
        *(uint2*)d = pk;
    } else *(float4*)d = make_float4(o[0], o[1], o[2], o[3]);
}
template <typename T, int W>
__device__ __forceinline__ void load_e(const T* p, float (&v)[W]) {
    if constexpr (W == 4 && sizeof(T) == 2) {
        const uint2 w = *(const uint2*)p;
        v[0] = __uint_as_float(w.x << 16); v[1] = __uint_as_float(w.x & 0xffff0000u);
        v[2] = __uint_as_float(w.y << 16); v[3] = __uint_as_float(w.y & 0xffff0000u);
    } else if constexpr (W == 4) *(float4*)v = *(const float4*)p;
    else
#pragma unroll
        for (int e = 0; e < W; ++e) v[e] = ld_f(p + e);
}

// W = 4 (PER > 0): H % 4 == 0, at most PER * NT * 4 columns, and a row's u stays in registers between the passes
template <typename T, int W, int PER, int NT>
__global__ void __launch_bounds__(NT) stream_rows_kernel(const StreamRows p) {
    __shared__ float red[32], coef[STREAMS_MAX * (STREAMS_MAX + 2)];
    pdl_launch_dependents();
    const int r = blockIdx.x, tid = threadIdx.x, n = p.sm.n, H = p.H;
    for (int i = tid; i < n * (n + 2); i += NT) coef[i] = p.sm.coef[i];
    __syncthreads();
    pdl_wait();
    float* x = p.sm.x + (size_t)r * n * H;
    const T* emb = nullptr;
    float in_sum = 0.f;
    if (p.from_embedding) {
        if (p.embed) {
            int tok = p.row_tokens ? p.row_tokens[r] : -1;
            if (tok < 0) tok = p.seqs[p.meta[r].seq].token;
            emb = (const T*)p.embed + (size_t)min(max(tok, 0), p.vocab - 1) * p.ld_embed;
        }
        for (int s = 0; s < n; ++s) in_sum += coef[n * n + n + s];
    }
    auto column = [&](int c, float (&u)[W]) {                    // columns [c, c + W): streams updated, u formed
        if (p.from_embedding) {
            if (emb) load_e<T, W>(emb + c, u);
            else load_e<float, W>(p.h + (size_t)r * H + c, u);
#pragma unroll
            for (int e = 0; e < W; ++e) u[e] *= p.scale;
            for (int s = 0; s < n; ++s) {
                if constexpr (W == 4) *(float4*)(x + (size_t)s * H + c) = make_float4(u[0], u[1], u[2], u[3]);
                else x[(size_t)s * H + c] = u[0];
            }
#pragma unroll
            for (int e = 0; e < W; ++e) u[e] *= in_sum;
        } else {
            const float* y = p.y + (size_t)r * H + c;
            load_e<float, W>(y, u);
            for (int q = 1; q < p.planes; ++q) {
                float v[W];
                load_e<float, W>(y + q * p.plane_stride, v);
#pragma unroll
                for (int e = 0; e < W; ++e) u[e] += v[e];
            }
            stream_mix<W>(n, x + c, coef, H, u);
        }
        if (p.sm.u) {
            float* d = p.sm.u + (size_t)r * H + c;
            if constexpr (W == 4) *(float4*)d = make_float4(u[0], u[1], u[2], u[3]);
            else d[0] = u[0];
        }
    };
    T* xb = (T*)p.xb + (size_t)r * p.ldx;
    float ss = 0.f;
    if constexpr (PER > 0) {
        float u[PER][4];
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int c = (tid + k * NT) * 4;
#pragma unroll
            for (int e = 0; e < 4; ++e) u[k][e] = 0.f;
            if (c < H) column(c, u[k]);
#pragma unroll
            for (int e = 0; e < 4; ++e) ss += u[k][e] * u[k][e];
        }
        const float inv = rsqrtf(block_sum(ss, red) / (float)H + p.eps);
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int c = (tid + k * NT) * 4;
            if (c >= H) continue;
            float w[4];
            load_e<float, 4>(p.w + c, w);
#pragma unroll
            for (int e = 0; e < 4; ++e) w[e] *= u[k][e] * inv;
            store4<T>(xb + c, w);
        }
    } else {
        for (int c = tid; c < H; c += NT) {
            float u[1];
            column(c, u);
            ss += u[0] * u[0];
        }
        const float inv = rsqrtf(block_sum(ss, red) / (float)H + p.eps);
        for (int c = tid; c < H; c += NT) {              // (a thread re-reads only what it wrote)
            float v = 0.f;
            for (int s = 0; s < n; ++s) v = fmaf(coef[n * n + n + s], x[(size_t)s * H + c], v);
            xb[c] = to_t<T>(v * inv * p.w[c]);
        }
    }
}

template <typename T>
static int launch_sr(const StreamRows* p, cudaStream_t s) {
    const bool vec = (p->H & 3) == 0 && p->H <= 8192 && (p->ldx & 3) == 0 && (p->plane_stride & 3) == 0 && (p->ld_embed & 3) == 0;
    auto go = [&](auto kern, int threads) -> int {
        const dim3 g(p->rows), b(threads);
        // the embedding is a plain launch: whatever follows in the step may rely on prepare_rows (which precedes it) being complete
        if (p->from_embedding) { kern<<<g, b, 0, s>>>(*p); return cudaGetLastError(); }
        return launch_pdl(kern, g, b, 0, s, *p);
    };
    if (!vec) return go(stream_rows_kernel<T, 1, 0, 256>, 256);
    // A thread's groups of four columns go one after another, so few per thread are fast as long as the CTAs that
    // leaves on an SM still cover each other's barriers: 1024 threads up to 64 rows, 512 beyond.  (512 rows of 4096
    // columns, four streams: 17.3 us, with 256 threads 22.0; one row 3.8, 4.4 and 6.0.)
    const int nt = p->rows <= 64 ? 1024 : 512, per = (p->H + 4 * nt - 1) / (4 * nt);
    if (nt == 1024) return per <= 1 ? go(stream_rows_kernel<T, 4, 1, 1024>, 1024) : go(stream_rows_kernel<T, 4, 2, 1024>, 1024);
    if (per <= 1) return go(stream_rows_kernel<T, 4, 1, 512>, 512);
    return per <= 2 ? go(stream_rows_kernel<T, 4, 2, 512>, 512) : go(stream_rows_kernel<T, 4, 4, 512>, 512);
}
B2_API int b2_stream_rows(const StreamRows* p, cudaStream_t s) {
    if (p->rows < 1 || p->H < 1 || p->sm.n < 1 || p->sm.n > STREAMS_MAX || !p->sm.x || !p->sm.coef || !p->w || !p->xb || p->ldx < p->H ||
        (p->from_embedding ? (p->embed ? p->ld_embed < p->H || !p->meta || !p->seqs : !p->h) : (!p->y || p->planes < 1)))
        return cudaErrorInvalidValue;
    return p->dt == DT_BF16 ? launch_sr<bf16>(p, s) : launch_sr<float>(p, s);
}
B2_API int b2_sizeof_stream_rows() { return (int)sizeof(StreamRows); }
