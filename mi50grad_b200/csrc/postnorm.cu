// Row kernels of post-norm decoders: embedding gather, and the residual update x += rmsnorm(m) * w with an
// optional norm of the result.  The residual stream is fp32; xb is its copy in the element type of the
// projections (or, with final_w, the normalised stream that the output head reads).
#include "mixers.cuh"

template <typename T>
__global__ void __launch_bounds__(256) embed_rows_kernel(const T* __restrict__ embed, const int* __restrict__ row_tokens,
                                                         const RowMeta* __restrict__ rows, const SeqState* __restrict__ seqs,
                                                         float* __restrict__ h, T* __restrict__ xb, int ldx, int H, int vocab) {
    pdl_launch_dependents();
    const int r = blockIdx.x;
    int tok = row_tokens ? row_tokens[r] : -1;
    if (tok < 0) tok = seqs[rows[r].seq].token;
    tok = min(max(tok, 0), vocab - 1);
    const T* e = embed + (size_t)tok * H;
    for (int i = threadIdx.x; i < H; i += 256) {
        h[(size_t)r * H + i] = ld_f(e + i);
        if (xb) xb[(size_t)r * ldx + i] = e[i];
    }
}
B2_API int b2_embed_rows(const void* embed, const int* row_tokens, const void* rows, const void* seqs, float* h, void* xb,
                         int ldx, int n_rows, int H, int vocab, int dt, cudaStream_t s) {
    // a plain launch: whatever follows in the step may rely on prepare_rows (which precedes it) being complete
    if (dt == DT_BF16)
        embed_rows_kernel<bf16><<<n_rows, 256, 0, s>>>((const bf16*)embed, row_tokens, (const RowMeta*)rows, (const SeqState*)seqs, h, (bf16*)xb, ldx, H, vocab);
    else
        embed_rows_kernel<float><<<n_rows, 256, 0, s>>>((const float*)embed, row_tokens, (const RowMeta*)rows, (const SeqState*)seqs, h, (float*)xb, ldx, H, vocab);
    return cudaGetLastError();
}

// VEC: H % 4 == 0, H <= 8192 and ldx % 4 == 0, the row stays in registers between its passes
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) post_norm_kernel(float* __restrict__ h, const float* __restrict__ m, const float* __restrict__ w,
                                                        const float* __restrict__ fw, T* __restrict__ xb, int ldx, int H, float eps, int planes,
                                                        size_t plane_stride) {
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x, tid = threadIdx.x;
    float* hr = h + (size_t)r * H;
    const float* mr = m ? m + (size_t)r * H : nullptr;
    if constexpr (VEC) {
        const int n4 = H >> 2;
        float4 a[8], x[8];
        float ss = 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int i = tid + 256 * u;
            a[u] = make_float4(0.f, 0.f, 0.f, 0.f); x[u] = a[u];
            if (i < n4) { x[u] = ((const float4*)hr)[i]; if (mr) a[u] = ((const float4*)mr)[i]; }
            for (int q = 1; q < planes; ++q)
                if (i < n4) { const float4 b = *(const float4*)(mr + q * plane_stride + 4 * i); a[u].x += b.x; a[u].y += b.y; a[u].z += b.z; a[u].w += b.w; }
            ss += a[u].x * a[u].x + a[u].y * a[u].y + a[u].z * a[u].z + a[u].w * a[u].w;
        }
        if (mr) {
            const float inv = rsqrtf(block_sum(ss, red) / (float)H + eps);
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int i = tid + 256 * u;
                if (i < n4) {
                    const float4 w4 = ((const float4*)w)[i];
                    x[u].x += a[u].x * inv * w4.x; x[u].y += a[u].y * inv * w4.y; x[u].z += a[u].z * inv * w4.z; x[u].w += a[u].w * inv * w4.w;
                    ((float4*)hr)[i] = x[u];
                }
            }
        }
        float fin = 1.f;
        if (fw) {
            ss = 0.f;
#pragma unroll
            for (int u = 0; u < 8; ++u) ss += x[u].x * x[u].x + x[u].y * x[u].y + x[u].z * x[u].z + x[u].w * x[u].w;
            fin = rsqrtf(block_sum(ss, red) / (float)H + eps);
        }
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int i = tid + 256 * u;
            if (i < n4) {
                float4 o = x[u];
                if (fw) { const float4 f4 = ((const float4*)fw)[i]; o.x *= fin * f4.x; o.y *= fin * f4.y; o.z *= fin * f4.z; o.w *= fin * f4.w; }
                T* d = xb + (size_t)r * ldx + 4 * i;
                if constexpr (sizeof(T) == 2) {
                    const __nv_bfloat162 p0 = __floats2bfloat162_rn(o.x, o.y), p1 = __floats2bfloat162_rn(o.z, o.w);
                    uint2 pk; pk.x = *(const uint32_t*)&p0; pk.y = *(const uint32_t*)&p1;
                    *(uint2*)d = pk;
                } else *(float4*)d = o;
            }
        }
    } else {
        auto sum = [&](int i) { float v = mr[i]; for (int q = 1; q < planes; ++q) v += mr[q * plane_stride + i]; return v; };
        float inv = 0.f;
        if (mr) {
            float ss = 0.f;
            for (int i = tid; i < H; i += 256) { const float v = sum(i); ss += v * v; }
            inv = rsqrtf(block_sum(ss, red) / (float)H + eps);
        }
        float ss = 0.f;
        for (int i = tid; i < H; i += 256) {                 // (a thread re-reads only what it wrote)
            float v = hr[i];
            if (mr) { v += sum(i) * inv * w[i]; hr[i] = v; }
            ss += v * v;
        }
        float fin = 1.f;
        if (fw) fin = rsqrtf(block_sum(ss, red) / (float)H + eps);
        for (int i = tid; i < H; i += 256) xb[(size_t)r * ldx + i] = to_t<T>(fw ? hr[i] * fin * fw[i] : hr[i]);
    }
}

// h += rmsnorm(m) * w (m null: h as it is), then xb = h, or with final_w xb = rmsnorm(h) * final_w.  m is the sum
// of `planes` arrays plane_stride floats apart (the splits of a projection over K).
B2_API int b2_post_norm(float* h, const float* m, const float* w, const float* final_w, void* xb, int ldx, int n_rows, int H,
                        float eps, int dt, int planes, long long plane_stride, cudaStream_t s) {
    if (!m) planes = 1;
    const bool vec = (H & 3) == 0 && H <= 8192 && (ldx & 3) == 0 && (plane_stride & 3) == 0;
    if (dt == DT_BF16) {
        if (vec) return launch_pdl(post_norm_kernel<bf16, true>, dim3(n_rows), dim3(256), 0, s, h, m, w, final_w, (bf16*)xb, ldx, H, eps, planes, (size_t)plane_stride);
        return launch_pdl(post_norm_kernel<bf16, false>, dim3(n_rows), dim3(256), 0, s, h, m, w, final_w, (bf16*)xb, ldx, H, eps, planes, (size_t)plane_stride);
    }
    if (vec) return launch_pdl(post_norm_kernel<float, true>, dim3(n_rows), dim3(256), 0, s, h, m, w, final_w, (float*)xb, ldx, H, eps, planes, (size_t)plane_stride);
    return launch_pdl(post_norm_kernel<float, false>, dim3(n_rows), dim3(256), 0, s, h, m, w, final_w, (float*)xb, ldx, H, eps, planes, (size_t)plane_stride);
}
