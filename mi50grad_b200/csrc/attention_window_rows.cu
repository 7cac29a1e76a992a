// Sliding-window attention of many query rows of one sequence (visibility, cap and sink as in
// csrc/attention_window.cu): 64-row tiles on bf16 tensor cores (mma.sync) that walk only the key blocks their
// windows and the kept first keys reach.
#include "mixers.cuh"

// ---------------------------------------------------------------------------
// many rows of ONE sequence, bf16: grid (H, 64-row tiles), four warps of 16 rows
// ---------------------------------------------------------------------------
#define WR_ROWS 64
#define WR_KEYS 64
#define WR_PAD 8

__device__ __forceinline__ void wr_ldsm4(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void wr_ldsm4_t(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void wr_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t wr_pack(float x, float y) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    return *(const uint32_t*)&h;
}

// v = t[0] + .. + t[TERMS - 1] with bf16 terms of two values each
template <int TERMS>
__device__ __forceinline__ void wr_split(float a, float b, uint32_t (&t)[TERMS]) {
#pragma unroll
    for (int i = 0; i < TERMS; ++i) {
        t[i] = wr_pack(a, b);
        if (i + 1 < TERMS) { a -= __uint_as_float(t[i] << 16); b -= __uint_as_float(t[i] & 0xffff0000u); }
    }
}
// cap * tanh(x / cap) = cap - 2 cap / (1 + exp(2 x / cap)); e = 2 log2(e) / cap
__device__ __forceinline__ float wr_cap(float x, float cap, float e) { return cap - __fdividef(2.f * cap, 1.f + exp2f(x * e)); }

// TERMS: bf16 terms of a soft-max weight in the product with V (1: the weight rounded to bf16, 3: all of its 24 bits)
// CAP: capped scores.
template <int DP, int TERMS, bool CAP>
__global__ void __launch_bounds__(128, 1) window_rows_kernel(const MixLayer L, const MixRun R) {
    constexpr int LD = DP + WR_PAD, NT_O = DP / 8, PPR = DP / 8;
    extern __shared__ __align__(16) unsigned char wrs[];
    bf16* Qs = (bf16*)wrs;                       // [64][LD]
    bf16* Kb = Qs + WR_ROWS * LD;                // [2][64][LD]
    bf16* Vb = Kb + 2 * WR_KEYS * LD;            // [2][64][LD]
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    // (the tiles that see most keys start first)
    const int row0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * WR_ROWS, nrows = min(WR_ROWS, R.n_rows - row0), head = blockIdx.x;
    const int kvh = head / (L.H / L.G);
    const RowMeta rm = R.rows[row0];
    const int p0 = rm.pos;                       // positions of the tile: p0 .. p0 + nrows - 1
    const int k_lo = L.window > 0 ? max(0, p0 - L.window + 1) : 0, k_hi = p0 + nrows;
    const int b0 = k_lo / WR_KEYS, b1 = (k_hi + WR_KEYS - 1) / WR_KEYS;
    // blocks walked: those of the kept first keys in front of b0, then b0 .. b1 - 1
    const int kept = min(b0, (L.keep_first + WR_KEYS - 1) / WR_KEYS), n_blk = kept + b1 - b0;
    const size_t kv_base = (size_t)rm.seq * L.max_seq * L.G + kvh;
    pdl_wait();
    for (int i = tid; i < WR_ROWS * PPR; i += 128) {
        const int pc = i % PPR, r = i / PPR;
        bf16* dst = Qs + r * LD + pc * 8;
        if (r < nrows && pc * 8 < L.dp) cp_async16(dst, (const bf16*)R.qbuf + ((size_t)(row0 + r) * L.H + head) * L.dp + pc * 8);
        else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
    }
    auto stage = [&](int blk, int buf) {
        for (int i = tid; i < WR_KEYS * PPR; i += 128) {
            const int pc = i % PPR, r = i / PPR, slot = blk * WR_KEYS + r;
            bf16* kd = Kb + (buf * WR_KEYS + r) * LD + pc * 8;
            bf16* vd = Vb + (buf * WR_KEYS + r) * LD + pc * 8;
            if (slot < k_hi && pc * 8 < L.dp) cp_async16(kd, (const bf16*)L.kcache + (kv_base + (size_t)slot * L.G) * L.dp + pc * 8);
            else *(uint4*)kd = make_uint4(0u, 0u, 0u, 0u);
            if (slot < k_hi && pc * 8 < L.vp) cp_async16(vd, (const bf16*)L.vcache + (kv_base + (size_t)slot * L.G) * L.vp + pc * 8);
            else *(uint4*)vd = make_uint4(0u, 0u, 0u, 0u);
        }
    };
    stage(kept > 0 ? 0 : b0, 0);
    cp_async_commit();
    float o[NT_O][4];
#pragma unroll
    for (int n = 0; n < NT_O; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    const bf16* qw = Qs + warp * 16 * LD;
    const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8;
    const int b_row = (lane & 7) + (lane >> 4) * 8, b_col = ((lane >> 3) & 1) * 8;
    constexpr float LOG2E = 1.44269504f;                     // scores end up in the log2 domain
    const float cap = CAP ? L.softcap : 0.f, cap_e = CAP ? 2.f * LOG2E / cap : 0.f;
    const float sc = CAP ? L.attn_scale : L.attn_scale * LOG2E;
    const int q_lo = p0 + warp * 16 + g, q_hi = q_lo + 8;    // positions of this thread's two rows
    const int w_lo = L.window > 0 ? q_lo - L.window : -1, w_hi = L.window > 0 ? q_hi - L.window : -1;     // last invisible slots
    const int wp0 = p0 + warp * 16;                          // the warp's positions: wp0 .. wp0 + 15
    for (int it = 0; it < n_blk; ++it) {
        auto block_of = [&](int i) { return i < kept ? i : i - kept + b0; };
        const int buf = it & 1, s_base = block_of(it) * WR_KEYS;
        cp_async_wait<0>();
        __syncthreads();
        if (it + 1 < n_blk) stage(block_of(it + 1), buf ^ 1);
        cp_async_commit();
        // nothing of this block is visible to the warp's rows
        if (s_base > wp0 + 15 || (L.window > 0 && s_base + WR_KEYS - 1 <= wp0 - L.window && s_base >= L.keep_first) || warp * 16 >= nrows) continue;
        const bf16* Kt = Kb + buf * WR_KEYS * LD;
        const bf16* Vt = Vb + buf * WR_KEYS * LD;
        float s[WR_KEYS / 8][4];
#pragma unroll
        for (int n = 0; n < WR_KEYS / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll 4
        for (int k0 = 0; k0 < DP; k0 += 16) {
            uint32_t a[4];
            wr_ldsm4(a, qw + a_row * LD + k0 + a_col);
#pragma unroll
            for (int np = 0; np < WR_KEYS / 16; ++np) {
                uint32_t b[4];
                wr_ldsm4(b, Kt + (np * 16 + b_row) * LD + k0 + b_col);
                wr_mma(s[2 * np], a, b[0], b[1]);
                wr_mma(s[2 * np + 1], a, b[2], b[3]);
            }
        }
        float mx_lo = -INFINITY, mx_hi = -INFINITY;
        const bool whole = s_base + WR_KEYS - 1 <= wp0 && (L.window <= 0 || s_base > wp0 + 15 - L.window || s_base + WR_KEYS <= L.keep_first);
#pragma unroll
        for (int n = 0; n < WR_KEYS / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float v = s[n][e] * sc;
                if constexpr (CAP) v = wr_cap(v, cap, cap_e) * LOG2E;
                if (!whole) {
                    const int slot = s_base + 8 * n + 2 * t + (e & 1);
                    const bool vis = e >= 2 ? (slot <= q_hi && (slot > w_hi || slot < L.keep_first))
                                            : (slot <= q_lo && (slot > w_lo || slot < L.keep_first));
                    if (!vis) v = -INFINITY;
                }
                s[n][e] = v;
                if (e >= 2) mx_hi = fmaxf(mx_hi, v); else mx_lo = fmaxf(mx_lo, v);
            }
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1)); mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1)); mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
        const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);
        const float rf_lo = mn_lo == -INFINITY ? 0.f : mn_lo, rf_hi = mn_hi == -INFINITY ? 0.f : mn_hi;
        const float c_lo = exp2f(m_lo - rf_lo), c_hi = exp2f(m_hi - rf_hi);
        m_lo = mn_lo; m_hi = mn_hi;
        float rs_lo = 0.f, rs_hi = 0.f;
#pragma unroll
        for (int n = 0; n < WR_KEYS / 8; ++n) {
            s[n][0] = exp2f(s[n][0] - rf_lo); s[n][1] = exp2f(s[n][1] - rf_lo);
            s[n][2] = exp2f(s[n][2] - rf_hi); s[n][3] = exp2f(s[n][3] - rf_hi);
            rs_lo += s[n][0] + s[n][1]; rs_hi += s[n][2] + s[n][3];
        }
        l_lo = l_lo * c_lo + rs_lo; l_hi = l_hi * c_hi + rs_hi;
#pragma unroll
        for (int n = 0; n < NT_O; ++n) { o[n][0] *= c_lo; o[n][1] *= c_lo; o[n][2] *= c_hi; o[n][3] *= c_hi; }
#pragma unroll
        for (int k16 = 0; k16 < WR_KEYS / 16; ++k16) {
            uint32_t t0[TERMS], t1[TERMS], t2[TERMS], t3[TERMS];
            wr_split<TERMS>(s[2 * k16][0], s[2 * k16][1], t0);
            wr_split<TERMS>(s[2 * k16][2], s[2 * k16][3], t1);
            wr_split<TERMS>(s[2 * k16 + 1][0], s[2 * k16 + 1][1], t2);
            wr_split<TERMS>(s[2 * k16 + 1][2], s[2 * k16 + 1][3], t3);
#pragma unroll
            for (int np = 0; np < NT_O / 2; ++np) {
                uint32_t b[4];
                wr_ldsm4_t(b, Vt + (k16 * 16 + a_row) * LD + np * 16 + a_col);
#pragma unroll
                for (int i = 0; i < TERMS; ++i) {
                    const uint32_t pa[4] = {t0[i], t1[i], t2[i], t3[i]};
                    wr_mma(o[2 * np], pa, b[0], b[1]);
                    wr_mma(o[2 * np + 1], pa, b[2], b[3]);
                }
            }
        }
    }
    cp_async_wait<0>();
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1); l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1); l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
    if (L.sink) {
        const float sk = L.sink[head] * LOG2E;
        l_lo += exp2f(sk - m_lo); l_hi += exp2f(sk - m_hi);
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int rr = warp * 16 + g + 8 * half;
        if (rr >= nrows) continue;
        const float f = L.left_scale / (half ? l_hi : l_lo);
        bf16* dst = (bf16*)R.out + (size_t)(row0 + rr) * R.ldo + (size_t)head * L.dv;
#pragma unroll
        for (int n = 0; n < NT_O; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int c = 8 * n + 2 * t + e;
                if (c < L.dv) dst[c] = __float2bfloat16(o[n][2 * half + e] * f);
            }
    }
}

template <int DP, int TERMS, bool CAP>
static int launch_wr(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    const size_t smem = (size_t)(WR_ROWS + 4 * WR_KEYS) * (DP + WR_PAD) * sizeof(bf16);
    static SmemOptIn opt;
    if (int e = opt.ensure((const void*)window_rows_kernel<DP, TERMS, CAP>, smem)) return e;
    return launch_pdl(window_rows_kernel<DP, TERMS, CAP>, dim3(l->H, (r->n_rows + WR_ROWS - 1) / WR_ROWS), dim3(128), smem, s, *l, *r);
}
template <int TERMS, bool CAP>
static int launch_wr_t(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    const int m = l->dp > l->vp ? l->dp : l->vp;
    if (m <= 32) return launch_wr<32, TERMS, CAP>(l, r, s);
    if (m <= 64) return launch_wr<64, TERMS, CAP>(l, r, s);
    if (m <= 96) return launch_wr<96, TERMS, CAP>(l, r, s);
    if (m <= 128) return launch_wr<128, TERMS, CAP>(l, r, s);
    return launch_wr<256, TERMS, CAP>(l, r, s);
}
// All rows belong to one sequence, bf16 only (b2_window_attn_decode takes everything else).
B2_API int b2_window_attn_rows(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    if (r->dt != DT_BF16 || r->n_seqs != 1 || !attn_valid(l)) return cudaErrorInvalidValue;
    if (l->softcap > 0.f) return launch_wr_t<3, true>(l, r, s);
    return l->exact_weights ? launch_wr_t<3, false>(l, r, s) : launch_wr_t<1, false>(l, r, s);
}
