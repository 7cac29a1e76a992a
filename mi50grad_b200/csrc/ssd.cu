// Linear recurrences with a scalar decay per head and token:
//     S_t = a_t S_(t-1) + dt_t B_t x_t^T,     y_t = S_t^T C_t + D x_t
// with S [N x P] fp32 per head, B and C shared by the heads of a group.
//   Mamba-2 (state-space duality): a_t = exp(-exp(A_log) dt_t); then an RMSNorm of y * silu(z) in ngroups parts.
//   Lightning attention: a constant per head, dt = 1, no D, q / k / v in the places of C / B / x, every head its own
//   group; then an RMSNorm of y times sigmoid(z).
//
//   ssd_step    token by token: one CTA per (head, 32 columns of P, sequence), the state in registers
//               (requested before the dependency wait); the last CTA of a norm part normalises it.
//   ssd_chunk   prompts in bf16: chunks of 64 tokens.  (1) local end state of every chunk, (2) the pass over
//               the chunks, (3) outputs.  The products run on bf16 tensor cores; every operand that is not
//               exactly bf16 (weighted inputs, masked scores, states) enters as the sum of three bf16 terms
//               (24 bits), so the recurrence keeps fp32 accuracy.
#include "mixers.cuh"

// The last taps-1 raw inputs of the channels [c0, c1) after this launch's rows [r0, r1) of one sequence.
// Ascending in place: entry i takes the old entry i + n (n rows) or a row of the projection.
template <typename T>
__device__ __forceinline__ void conv_history(const MixLayer& L, const MixRun& R, int seq, int r0, int r1, int c0, int c1,
                                             int tid, int nthr) {
    const int C = L.heads * L.P + 2 * L.groups * L.N, K = L.taps - 1, n = r1 - r0;
    if (K == 0) return;
    T* hist = (T*)L.conv_state + (size_t)seq * K * C;
    for (int c = c0 + tid; c < c1; c += nthr)
        for (int i = 0; i < K; ++i) {
            const int back = n - K + i;                     // row index of the input that lands in entry i
            hist[(size_t)i * C + c] = back >= 0 ? ((const T*)R.proj)[(size_t)(r0 + back) * R.ld_proj + L.off_x + c]
                                                : hist[(size_t)(i + n) * C + c];
        }
}
// Channels a CTA (head h, column block of width pw at p0) carries over: its own x columns, and for the
// first head of a group and the first block also the group's B and C.
template <typename T>
__device__ __forceinline__ void conv_history_of(const MixLayer& L, const MixRun& R, int seq, int r0, int r1, int h, int p0, int pw,
                                                int tid, int nthr) {
    const int I = L.heads * L.P, rep = L.heads / L.groups;
    conv_history<T>(L, R, seq, r0, r1, h * L.P + p0, h * L.P + min(L.P, p0 + pw), tid, nthr);
    if (p0 == 0 && h % rep == 0) {
        const int g = h / rep;
        conv_history<T>(L, R, seq, r0, r1, I + g * L.N, I + (g + 1) * L.N, tid, nthr);
        conv_history<T>(L, R, seq, r0, r1, I + (L.groups + g) * L.N, I + (L.groups + g + 1) * L.N, tid, nthr);
    }
}

__device__ __forceinline__ uint32_t sc_pack(bf16 a, bf16 b) {
    return (uint32_t)__bfloat16_as_ushort(a) | ((uint32_t)__bfloat16_as_ushort(b) << 16);
}
// log decay and step size of the token in row r
__device__ __forceinline__ float rec_rate(const MixLayer& L, int h) { return L.decay ? L.log_decay[h] : -expf(L.A_log[h]); }
__device__ __forceinline__ float rec_dt(const MixLayer& L, const MixRun& R, int r, int h) {
    return L.decay ? 1.f : R.dtb[(size_t)r * R.ld_dt + h];
}

// RMSNorm of one part of one row: out = u / rms(u) * w * right_scale (* sigmoid(z)), from column out_col on.
#define NP_REGS 4                // float4s per thread that stay in registers between the passes
template <typename T>
__device__ __forceinline__ void norm_part(const MixLayer& L, const MixRun& R, int r, int part, float* red) {
    const int I = L.heads * L.P, w = I / L.ngroups, c0 = part * w, tid = threadIdx.x, nt = blockDim.x;
    const float* u = R.ubuf + (size_t)r * R.ld_u + c0;
    const float* nw = L.norm_w + c0;
    T* out = (T*)R.out + (size_t)r * R.ldo + L.out_col + c0;
    const T* z = (const T*)R.proj + (size_t)r * R.ld_proj + L.off_z + c0;
    const bool gate = L.gate == REC_NORM_SIGMOID;
    auto one = [&](int i, float v, float inv) {
        v *= inv * nw[i] * L.right_scale;
        out[i] = to_t<T>(gate ? v * sigmoid_p(ld_f(z + i)) : v);
    };
    float ss = 0.f;
    if (((w | c0 | R.ld_u) & 3) == 0) {
        float4 v[NP_REGS];
        const int w4 = w >> 2;
#pragma unroll
        for (int j = 0; j < NP_REGS; ++j) {
            const int i = tid + j * nt;
            v[j] = i < w4 ? __ldcg((const float4*)u + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int j = 0; j < NP_REGS; ++j) ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
        for (int i = tid + NP_REGS * nt; i < w4; i += nt) {
            const float4 q = __ldcg((const float4*)u + i);
            ss += q.x * q.x + q.y * q.y + q.z * q.z + q.w * q.w;
        }
        const float inv = rsqrtf(block_sum(ss, red) / (float)w + L.eps);
        const bool packed = sizeof(T) == 2 && (((int)R.ldo | L.out_col | R.ld_proj | L.off_z) & 3) == 0;
        auto four = [&](int i, const float4& q) {
            if (packed) {
                const float4 w = ((const float4*)nw)[i];
                const float f = inv * L.right_scale;
                float o[4] = {q.x * f * w.x, q.y * f * w.y, q.z * f * w.z, q.w * f * w.w};
                if (gate) {
                    const uint2 g = *(const uint2*)(z + 4 * i);
                    o[0] *= sigmoid_p(__uint_as_float(g.x << 16)); o[1] *= sigmoid_p(__uint_as_float(g.x & 0xffff0000u));
                    o[2] *= sigmoid_p(__uint_as_float(g.y << 16)); o[3] *= sigmoid_p(__uint_as_float(g.y & 0xffff0000u));
                }
                uint2 pk; pk.x = sc_pack(__float2bfloat16(o[0]), __float2bfloat16(o[1])); pk.y = sc_pack(__float2bfloat16(o[2]), __float2bfloat16(o[3]));
                *(uint2*)(out + 4 * i) = pk;
            } else { one(4 * i, q.x, inv); one(4 * i + 1, q.y, inv); one(4 * i + 2, q.z, inv); one(4 * i + 3, q.w, inv); }
        };
#pragma unroll
        for (int j = 0; j < NP_REGS; ++j) if (tid + j * nt < w4) four(tid + j * nt, v[j]);
        for (int i = tid + NP_REGS * nt; i < w4; i += nt) four(i, __ldcg((const float4*)u + i));
        return;
    }
    for (int i = tid; i < w; i += nt) { const float x = __ldcg(u + i); ss += x * x; }
    const float inv = rsqrtf(block_sum(ss, red) / (float)w + L.eps);
    for (int i = tid; i < w; i += nt) one(i, __ldcg(u + i), inv);
}

template <typename T>
__global__ void __launch_bounds__(256) ssd_norm_kernel(const MixLayer L, const MixRun R) {
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    norm_part<T>(L, R, blockIdx.x, blockIdx.y, red);
}

// ---------------------------------------------------------------------------
// token by token: grid (heads, ceil(P / 32), sequences); lane = column of P, warp = slice of N
// ---------------------------------------------------------------------------
#define SS_WARPS 8
#define SS_THREADS (SS_WARPS * 32)

template <typename T, int NB>                    // NB: state rows per warp
__global__ void __launch_bounds__(SS_THREADS) ssd_step_kernel(const MixLayer L, const MixRun R) {
    __shared__ float Bs[SS_WARPS * NB], Cs[SS_WARPS * NB], part[SS_WARPS][32], red[32];
    __shared__ int s_last;
    pdl_launch_dependents();
    const int h = blockIdx.x, p0 = blockIdx.y * 32, sq = blockIdx.z;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int grp = h / (L.heads / L.groups), p = p0 + lane;
    const bool pv = p < L.P;
    const int r0 = R.seq_rows[sq], r1 = R.seq_rows[sq + 1];
    const int seq = R.rows[r0].seq;
    float* S = L.state + ((size_t)seq * L.heads + h) * L.N * L.P + p;
    // the state was last written in an earlier step
    float st[NB];
#pragma unroll
    for (int i = 0; i < NB; ++i) { const int n = warp + SS_WARPS * i; st[i] = (pv && n < L.N) ? S[(size_t)n * L.P] : 0.f; }
    const float A = rec_rate(L, h), Dh = L.D ? L.D[h] : 0.f, a_const = L.decay ? L.decay[h] : 0.f;
    const bool gated = L.gate == REC_GATE_SILU_NORM;
    pdl_wait();
    for (int r = r0; r < r1; ++r) {
        const T* xbc = (const T*)R.xbc + (size_t)r * R.ld_xbc;
        for (int n = tid; n < SS_WARPS * NB; n += SS_THREADS) {
            Bs[n] = n < L.N ? ld_f(xbc + L.rB + grp * L.N + n) : 0.f;
            Cs[n] = n < L.N ? ld_f(xbc + L.rC + grp * L.N + n) : 0.f;
        }
        const float x = pv ? ld_f(xbc + L.rx + h * L.P + p) : 0.f;
        const float dt = rec_dt(L, R, r, h);
        const float z = (gated && warp == 0 && pv) ? ld_f((const T*)R.proj + (size_t)r * R.ld_proj + L.off_z + h * L.P + p) : 0.f;
        const float a = L.decay ? a_const : expf(A * dt), dx = dt * x;
        __syncthreads();
        float y = 0.f;
#pragma unroll
        for (int i = 0; i < NB; ++i) {
            const int n = warp + SS_WARPS * i;
            st[i] = fmaf(a, st[i], Bs[n] * dx);
            y = fmaf(st[i], Cs[n], y);
        }
        part[warp][lane] = y;
        __syncthreads();
        if (warp == 0 && pv) {
            float s = 0.f;
#pragma unroll
            for (int w = 0; w < SS_WARPS; ++w) s += part[w][lane];
            R.ubuf[(size_t)r * R.ld_u + h * L.P + p] = (s + Dh * x) * (gated ? silu_p(z) : 1.f);
        }
    }
    if (R.commit) {
#pragma unroll
        for (int i = 0; i < NB; ++i) { const int n = warp + SS_WARPS * i; if (pv && n < L.N) S[(size_t)n * L.P] = st[i]; }
        conv_history_of<T>(L, R, seq, r0, r1, h, p0, 32, tid, SS_THREADS);
    }
    if (!R.fuse_norm) return;
    // ---- the last CTA of a norm part (of the whole row when parts cut through heads) normalises it
    const bool whole = L.heads % L.ngroups != 0;
    const int units = whole ? 1 : L.ngroups, hpu = L.heads / units, unit = h / hpu;
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        int* cnt = R.ssd_counters + sq * units + unit;
        s_last = atomicAdd(cnt, 1) == hpu * (int)gridDim.y - 1;
        if (s_last) *cnt = 0;
        __threadfence();
    }
    __syncthreads();
    if (!s_last) return;
    for (int r = r0; r < r1; ++r)
        for (int q = 0; q < (whole ? L.ngroups : 1); ++q) norm_part<T>(L, R, r, whole ? q : unit, red);
}

static bool ssd_valid(const MixLayer* l) {
    return l->heads >= 1 && l->P >= 1 && l->N >= 1 && l->N <= 256 && l->groups >= 1 && l->heads % l->groups == 0 &&
           l->ngroups >= 1 && (l->heads * l->P) % l->ngroups == 0 && l->taps >= 1 && (l->decay ? l->log_decay != nullptr : l->A_log != nullptr);
}

// one CTA per part of a row, with a thread for every four columns of it
template <typename T>
static int launch_ssd_norm(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    const int w4 = (l->heads * l->P / l->ngroups + 3) / 4, nt = w4 >= 256 ? 256 : (w4 + 31) / 32 * 32;
    return launch_pdl(ssd_norm_kernel<T>, dim3(r->n_rows, l->ngroups), dim3(nt), 0, s, *l, *r);
}
template <typename T>
static int launch_ssd_step(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    dim3 grid(l->heads, (l->P + 31) / 32, r->n_seqs);
    int e;
    if (l->N <= 64) e = launch_pdl(ssd_step_kernel<T, 8>, grid, dim3(SS_THREADS), 0, s, *l, *r);
    else if (l->N <= 128) e = launch_pdl(ssd_step_kernel<T, 16>, grid, dim3(SS_THREADS), 0, s, *l, *r);
    else e = launch_pdl(ssd_step_kernel<T, 32>, grid, dim3(SS_THREADS), 0, s, *l, *r);
    if (e || r->fuse_norm) return e;
    return launch_ssd_norm<T>(l, r, s);
}
// Any mix of sequences; fuse_norm = 0 adds a launch for the norm (many rows per sequence).
B2_API int b2_ssd_step(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    if (!ssd_valid(l) || r->n_seqs < 1) return cudaErrorInvalidValue;
    return r->dt == DT_BF16 ? launch_ssd_step<bf16>(l, r, s) : launch_ssd_step<float>(l, r, s);
}
B2_API int b2_ssd_units(const MixLayer* l, int n_seqs) { return n_seqs * (l->heads % l->ngroups ? 1 : l->ngroups); }

// ---------------------------------------------------------------------------
// chunked scan: one sequence, bf16
// ---------------------------------------------------------------------------
#define SC_T SSD_CHUNK
#define SC_P 64                  // columns of P per CTA
#define SC_LDP (SC_P + 8)
#define SC_TERMS 3

__device__ __forceinline__ void sc_ldsm4(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void sc_ldsm4_t(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void sc_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// v = t[0] + t[1] + t[2] with bf16 terms (exact to 24 bits)
__device__ __forceinline__ void sc_split(float v, bf16 (&t)[SC_TERMS]) {
#pragma unroll
    for (int i = 0; i < SC_TERMS; ++i) { t[i] = __float2bfloat16(v); v -= __bfloat162float(t[i]); }
}

// cumulative log decay of a chunk (one warp; two tokens per lane)
__device__ __forceinline__ void sc_cumsum(const MixLayer& L, const MixRun& R, int t0, int n, int h, float A, float* la, float* dts, int lane) {
    const float d0 = 2 * lane < n ? rec_dt(L, R, t0 + 2 * lane, h) : 0.f;
    const float d1 = 2 * lane + 1 < n ? rec_dt(L, R, t0 + 2 * lane + 1, h) : 0.f;
    const float a0 = A * d0, a1 = A * d1;
    float s = a0 + a1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const float v = __shfl_up_sync(0xffffffffu, s, o); if (lane >= o) s += v; }
    const float before = s - (a0 + a1);
    la[2 * lane] = before + a0; la[2 * lane + 1] = s;
    dts[2 * lane] = d0; dts[2 * lane + 1] = d1;
}
// rows [t0, t0 + n) x columns [c0, c0 + w) of xbc into smem [64][ld], zero-padded to wp columns (wp % 8 == 0)
__device__ __forceinline__ void sc_stage(const MixRun& R, int t0, int n, int c0, int w, int wp, bf16* dst, int ld, int tid, int nthr) {
    const bf16* src = (const bf16*)R.xbc + c0;
    const bool vec = ((R.ld_xbc | c0) & 7) == 0;
    const int ppr = wp >> 3;
    for (int i = tid; i < SC_T * ppr; i += nthr) {
        const int r = i / ppr, c = (i % ppr) * 8;
        bf16* d = dst + r * ld + c;
        if (vec && r < n && c + 8 <= w) cp_async16(d, src + (size_t)(t0 + r) * R.ld_xbc + c);
        else
#pragma unroll
            for (int e = 0; e < 8; ++e) d[e] = (r < n && c + e < w) ? src[(size_t)(t0 + r) * R.ld_xbc + c + e] : __float2bfloat16(0.f);
    }
    cp_async_commit();
}

// (1) local end states: grid (chunks, heads, ceil(P / 64)), four warps over the rows of N
__global__ void __launch_bounds__(128) ssd_chunk_state_kernel(const MixLayer L, const MixRun R) {
    extern __shared__ __align__(16) unsigned char sc_smem[];
    const int Np = (L.N + 15) & ~15, LDN = Np + 8;
    bf16* Bs = (bf16*)sc_smem;                               // [64][LDN]
    bf16* W = Bs + SC_T * LDN;                               // [3][64][SC_LDP]
    __shared__ float la[SC_T], dts[SC_T];
    pdl_launch_dependents();
    const int c = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * SC_P;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int grp = h / (L.heads / L.groups), pw = min(SC_P, L.P - p0);
    const int t0 = c * SC_T, n = min(SC_T, R.n_rows - t0);
    const float A = rec_rate(L, h);
    pdl_wait();
    sc_stage(R, t0, n, L.rB + grp * L.N, L.N, Np, Bs, LDN, tid, 128);
    if (warp == 0) sc_cumsum(L, R, t0, n, h, A, la, dts, lane);
    __syncthreads();
    const float end = la[SC_T - 1];
    for (int i = tid; i < SC_T * SC_P; i += 128) {
        const int s = i / SC_P, p = i % SC_P;
        float v = 0.f;
        if (s < n && p < pw) v = ld_f((const bf16*)R.xbc + (size_t)(t0 + s) * R.ld_xbc + L.rx + h * L.P + p0 + p) * (dts[s] * expf(end - la[s]));
        bf16 q[SC_TERMS];
        sc_split(v, q);
#pragma unroll
        for (int k = 0; k < SC_TERMS; ++k) W[(k * SC_T + s) * SC_LDP + p] = q[k];
    }
    cp_async_wait<0>();
    __syncthreads();
    const int g = lane >> 2, t = lane & 3;
    const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_col = (lane >> 4) * 8;
    float* out = R.chunk_state + ((size_t)c * L.heads + h) * L.N * L.P + p0;
    for (int mt = warp; mt < Np / 16; mt += 4) {
        float acc[SC_P / 8][4];
#pragma unroll
        for (int j = 0; j < SC_P / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
        for (int k0 = 0; k0 < SC_T; k0 += 16) {
            uint32_t a[4];                                   // A = B^T: (m = state row, k = token) from [token][state row]
            sc_ldsm4_t(a, Bs + (k0 + (lane & 7) + (lane >> 4) * 8) * LDN + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int q = 0; q < SC_TERMS; ++q)
#pragma unroll
                for (int np = 0; np < SC_P / 16; ++np) {
                    if (np * 16 >= pw) break;
                    uint32_t b[4];
                    sc_ldsm4_t(b, W + (q * SC_T + k0 + v_row) * SC_LDP + np * 16 + v_col);
                    sc_mma(acc[2 * np], a, b[0], b[1]);
                    sc_mma(acc[2 * np + 1], a, b[2], b[3]);
                }
        }
#pragma unroll
        for (int j = 0; j < SC_P / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int nn = mt * 16 + g + 8 * (e >> 1), p = 8 * j + 2 * t + (e & 1);
                if (nn < L.N && p < pw) out[(size_t)nn * L.P + p] = acc[j][e];
            }
    }
    if (tid == 0 && blockIdx.z == 0) R.chunk_decay[c * L.heads + h] = end;
    // nothing of this launch reads the convolution history: carry it over here
    if (c == 0 && R.commit) conv_history_of<bf16>(L, R, R.rows[0].seq, 0, R.n_rows, h, p0, SC_P, tid, 128);
}

// (2) the pass over the chunks: grid (ceil(N * Pp / 256), heads); leaves the state before every chunk as bf16 planes
__global__ void __launch_bounds__(256) ssd_chunk_pass_kernel(const MixLayer L, const MixRun R, int chunks) {
    pdl_launch_dependents();
    const int Pp = (L.P + 7) & ~7, h = blockIdx.y;
    const int i = blockIdx.x * 256 + threadIdx.x, n = i / Pp, p = i % Pp;
    const bool in = n < L.N, ok = in && p < L.P;
    float* S = L.state + (((size_t)R.rows[0].seq * L.heads + h) * L.N + n) * L.P + p;
    float s = ok ? *S : 0.f;
    pdl_wait();
    if (!in) return;
    const float* cs = R.chunk_state + ((size_t)h * L.N + n) * L.P + p;
    const size_t cst = (size_t)L.heads * L.N * L.P;
    bf16* prev = (bf16*)R.chunk_prev + ((size_t)h * SC_TERMS * L.N + n) * Pp + p;
    const size_t pst = (size_t)L.heads * SC_TERMS * L.N * Pp;
    for (int c0 = 0; c0 < chunks; c0 += 4) {
        float v[4], d[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            v[u] = (ok && c0 + u < chunks) ? cs[(c0 + u) * cst] : 0.f;
            d[u] = c0 + u < chunks ? R.chunk_decay[(c0 + u) * L.heads + h] : 0.f;
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            if (c0 + u >= chunks) break;
            bf16 q[SC_TERMS];
            sc_split(s, q);
#pragma unroll
            for (int k = 0; k < SC_TERMS; ++k) prev[(c0 + u) * pst + (size_t)k * L.N * Pp] = q[k];
            s = fmaf(expf(d[u]), s, v[u]);
        }
    }
    if (ok && R.commit) *S = s;
}

// (3) outputs: grid (chunks, heads, ceil(P / 64)), four warps of 16 tokens
__global__ void __launch_bounds__(128) ssd_chunk_out_kernel(const MixLayer L, const MixRun R) {
    extern __shared__ __align__(16) unsigned char sc_smem[];
    const int Np = (L.N + 15) & ~15, LDN = Np + 8, Pp = (L.P + 7) & ~7;
    bf16* Cs = (bf16*)sc_smem;                               // [64][LDN]
    bf16* Bs = Cs + SC_T * LDN;                              // [64][LDN]
    bf16* Xs = Bs + SC_T * LDN;                              // [64][SC_LDP]
    bf16* Sp = Xs + SC_T * SC_LDP;                           // [3][Np][SC_LDP]
    __shared__ float la[SC_T], dts[SC_T];
    pdl_launch_dependents();
    const int c = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * SC_P;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int grp = h / (L.heads / L.groups), pw = min(SC_P, L.P - p0), pwp = (pw + 7) & ~7;
    const int t0 = c * SC_T, n = min(SC_T, R.n_rows - t0);
    const float A = rec_rate(L, h), Dh = L.D ? L.D[h] : 0.f;
    const bool gated = L.gate == REC_GATE_SILU_NORM;
    pdl_wait();
    sc_stage(R, t0, n, L.rC + grp * L.N, L.N, Np, Cs, LDN, tid, 128);
    sc_stage(R, t0, n, L.rB + grp * L.N, L.N, Np, Bs, LDN, tid, 128);
    sc_stage(R, t0, n, L.rx + h * L.P + p0, pw, SC_P, Xs, SC_LDP, tid, 128);
    {
        const bf16* src = (const bf16*)R.chunk_prev + ((size_t)c * L.heads + h) * SC_TERMS * L.N * Pp + p0;
        const int ppr = SC_P / 8;
        for (int i = tid; i < SC_TERMS * Np * ppr; i += 128) {
            const int col = (i % ppr) * 8, nn = (i / ppr) % Np, q = i / (ppr * Np);
            bf16* d = Sp + (q * Np + nn) * SC_LDP + col;
            if (nn < L.N && col < pwp) cp_async16(d, src + ((size_t)q * L.N + nn) * Pp + col);
            else *(uint4*)d = make_uint4(0u, 0u, 0u, 0u);
        }
        cp_async_commit();
    }
    if (warp == 0) sc_cumsum(L, R, t0, n, h, A, la, dts, lane);
    cp_async_wait<0>();
    __syncthreads();
    if (warp * 16 >= n) return;
    const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8;
    const int b_row = (lane & 7) + (lane >> 4) * 8, b_col = ((lane >> 3) & 1) * 8;
    const bf16* Cw = Cs + warp * 16 * LDN;
    float o[SC_P / 8][4], s[SC_T / 8][4];
#pragma unroll
    for (int j = 0; j < SC_P / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
    for (int j = 0; j < SC_T / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
    for (int k0 = 0; k0 < Np; k0 += 16) {
        uint32_t a[4];
        sc_ldsm4(a, Cw + a_row * LDN + k0 + a_col);
        // scores C B^T of the tokens up to this warp's own
#pragma unroll
        for (int np = 0; np < SC_T / 16; ++np) {
            if (np > warp) break;
            uint32_t b[4];
            sc_ldsm4(b, Bs + (np * 16 + b_row) * LDN + k0 + b_col);
            sc_mma(s[2 * np], a, b[0], b[1]);
            sc_mma(s[2 * np + 1], a, b[2], b[3]);
        }
        // C times the state before the chunk
#pragma unroll
        for (int q = 0; q < SC_TERMS; ++q)
#pragma unroll
            for (int np = 0; np < SC_P / 16; ++np) {
                if (np * 16 >= pw) break;
                uint32_t b[4];
                sc_ldsm4_t(b, Sp + (q * Np + k0 + a_row) * SC_LDP + np * 16 + a_col);
                sc_mma(o[2 * np], a, b[0], b[1]);
                sc_mma(o[2 * np + 1], a, b[2], b[3]);
            }
    }
    const int r_lo = warp * 16 + g, r_hi = r_lo + 8;
    const float la_lo = la[r_lo], la_hi = la[r_hi], e_lo = expf(la_lo), e_hi = expf(la_hi);
#pragma unroll
    for (int j = 0; j < SC_P / 8; ++j) { o[j][0] *= e_lo; o[j][1] *= e_lo; o[j][2] *= e_hi; o[j][3] *= e_hi; }
#pragma unroll
    for (int k16 = 0; k16 < SC_T / 16; ++k16) {
        if (k16 > warp) break;
        uint32_t pa[SC_TERMS][4];
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
            const int j = 2 * k16 + hf, s0 = 8 * j + 2 * t;
            bf16 q0[SC_TERMS], q1[SC_TERMS], q2[SC_TERMS], q3[SC_TERMS];
            sc_split(s0 <= r_lo ? s[j][0] * expf(la_lo - la[s0]) * dts[s0] : 0.f, q0);
            sc_split(s0 + 1 <= r_lo ? s[j][1] * expf(la_lo - la[s0 + 1]) * dts[s0 + 1] : 0.f, q1);
            sc_split(s0 <= r_hi ? s[j][2] * expf(la_hi - la[s0]) * dts[s0] : 0.f, q2);
            sc_split(s0 + 1 <= r_hi ? s[j][3] * expf(la_hi - la[s0 + 1]) * dts[s0 + 1] : 0.f, q3);
#pragma unroll
            for (int q = 0; q < SC_TERMS; ++q) { pa[q][hf * 2] = sc_pack(q0[q], q1[q]); pa[q][hf * 2 + 1] = sc_pack(q2[q], q3[q]); }
        }
#pragma unroll
        for (int np = 0; np < SC_P / 16; ++np) {
            if (np * 16 >= pw) break;
            uint32_t b[4];
            sc_ldsm4_t(b, Xs + (k16 * 16 + a_row) * SC_LDP + np * 16 + a_col);
#pragma unroll
            for (int q = 0; q < SC_TERMS; ++q) {
                sc_mma(o[2 * np], pa[q], b[0], b[1]);
                sc_mma(o[2 * np + 1], pa[q], b[2], b[3]);
            }
        }
    }
#pragma unroll
    for (int j = 0; j < SC_P / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = e >= 2 ? r_hi : r_lo, p = 8 * j + 2 * t + (e & 1);
            if (r < n && p < pw) {
                float u = o[j][e] + Dh * ld_f(Xs + r * SC_LDP + p);
                if (gated) u *= silu_p(ld_f((const bf16*)R.proj + (size_t)(t0 + r) * R.ld_proj + L.off_z + h * L.P + p0 + p));
                R.ubuf[(size_t)(t0 + r) * R.ld_u + h * L.P + p0 + p] = u;
            }
        }
}

// All rows belong to one sequence, bf16 only (b2_ssd_step takes everything else).
B2_API int b2_ssd_chunk(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    if (!ssd_valid(l) || r->dt != DT_BF16 || r->n_seqs != 1 || !r->chunk_state || !r->chunk_prev || !r->chunk_decay)
        return cudaErrorInvalidValue;
    const int chunks = (r->n_rows + SC_T - 1) / SC_T, Np = (l->N + 15) & ~15, Pp = (l->P + 7) & ~7, pb = (l->P + SC_P - 1) / SC_P;
    const size_t sm1 = ((size_t)SC_T * (Np + 8) + SC_TERMS * SC_T * SC_LDP) * sizeof(bf16);
    const size_t sm3 = ((size_t)2 * SC_T * (Np + 8) + SC_T * SC_LDP + (size_t)SC_TERMS * Np * SC_LDP) * sizeof(bf16);
    static SmemOptIn o1, o3;
    if (int e = o1.ensure((const void*)ssd_chunk_state_kernel, sm1)) return e;
    if (int e = o3.ensure((const void*)ssd_chunk_out_kernel, sm3)) return e;
    if (int e = launch_pdl(ssd_chunk_state_kernel, dim3(chunks, l->heads, pb), dim3(128), sm1, s, *l, *r)) return e;
    if (int e = launch_pdl(ssd_chunk_pass_kernel, dim3((l->N * Pp + 255) / 256, l->heads), dim3(256), 0, s, *l, *r, chunks)) return e;
    if (int e = launch_pdl(ssd_chunk_out_kernel, dim3(chunks, l->heads, pb), dim3(128), sm3, s, *l, *r)) return e;
    return launch_ssd_norm<bf16>(l, r, s);
}
B2_API long long b2_ssd_chunk_state_floats(const MixLayer* l, int rows) {
    return (long long)((rows + SC_T - 1) / SC_T) * l->heads * l->N * l->P;
}
B2_API long long b2_ssd_chunk_prev_bytes(const MixLayer* l, int rows) {
    return (long long)((rows + SC_T - 1) / SC_T) * l->heads * SC_TERMS * l->N * ((l->P + 7) & ~7) * (long long)sizeof(bf16);
}
