// Sliding-window attention, and the preparation pass in front of a mixer.
//
//   mix_prepare       parallel mixer: RMSNorm of Q and of K over the WHOLE projection (all heads at once), rotation
//                     of the first `rot` dimensions of every head in (i, i + rot/2) pairs, K and the values into the
//                     cache, causal convolution + SiLU of the recurrence's inputs, its step sizes.
//   head_prepare      attention alone: RMSNorm of every Q and K head with one weight for all heads, optional
//                     rotation, K and the values into the cache.
//   window decode     split-KV flash decoding, any head size up to 256, bf16 or fp32 cache.
//   (many query rows of one sequence: csrc/attention_window_rows.cu)
//
// Visibility: the row at position p sees slots max(0, p - window + 1) .. p of its sequence and its first
// keep_first slots (slot = position: rows of a sequence are consecutive tokens, no draft trees).  Scores may be
// capped (softcap * tanh(score / softcap)), and a learned sink per head may join the soft-max's denominator: it
// is neither scaled nor capped and has no value.
#include "mixers.cuh"

// ---------------------------------------------------------------------------
// prepare: one-dimensional grid.  First (q_slices + 1) CTAs per row: slices of the query heads, then the keys;
// every one of them sums the squares of its whole projection.  Then the convolution: column blocks of 512
// channels times tiles of conv_rows rows.
// ---------------------------------------------------------------------------
#define MP_THREADS 256
#define MP_COLS (2 * MP_THREADS)
#define MP_MAX_ROWS 8            // rows of a convolution tile
#define MP_TAPS 4                // taps whose weights stay in registers

template <typename T>
__device__ __forceinline__ void mp_heads(const MixLayer& L, const MixRun& R, int r, int slice, int q_slices, float* sv, float* red) {
    const int tid = threadIdx.x;
    const bool is_q = slice < q_slices;
    const RowMeta rm = R.rows[r];
    const int heads = is_q ? L.H : L.G, n = heads * L.d, off = is_q ? L.off_q : L.off_k;
    const int per = is_q ? (heads + q_slices - 1) / q_slices : heads;
    const int h0 = is_q ? slice * per : 0, h1 = min(heads, h0 + per), i0 = h0 * L.d, i1 = h1 * L.d;
    const T* src = (const T*)R.proj + (size_t)r * R.ld_proj + off;
    const float* nw = is_q ? L.q_norm : L.k_norm;
    const size_t slot = ((size_t)rm.seq * L.max_seq + rm.slot) * L.G * L.dp;
    T* dst = is_q ? (T*)R.qbuf + (size_t)r * L.H * L.dp : (T*)L.kcache + slot;
    T* vdst = (T*)L.vcache + slot;                         // (values = keys as projected: vp == dp)
    constexpr int V = 16 / sizeof(T);
    const bool vec = ((off | R.ld_proj | n) & (V - 1)) == 0;
    pdl_wait();
    float ss = 0.f;
    if (vec) {
#pragma unroll 2
        for (int i = tid * V; i < n; i += MP_THREADS * V) {
            const uint4 u = *(const uint4*)(src + i);
            const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
            for (int e = 0; e < V; ++e) {
                const float v = sizeof(T) == 4 ? __uint_as_float(w[e & 3])
                                               : __uint_as_float((e & 1) ? (w[(e >> 1) & 3] & 0xffff0000u) : (w[(e >> 1) & 3] << 16));
                ss += v * v;
                if (i + e >= i0 && i + e < i1) sv[i + e - i0] = v;
            }
        }
    } else
        for (int i = tid; i < n; i += MP_THREADS) {
            const float v = ld_f(src + i);
            ss += v * v;
            if (i >= i0 && i < i1) sv[i - i0] = v;
        }
    const float inv = rsqrtf(block_sum(ss, red) / (float)n + L.eps);      // (its barriers also publish sv)
    const int half = L.rot >> 1;
    const float* ct = L.cos_tab + (size_t)rm.pos * half;
    const float* st = L.sin_tab + (size_t)rm.pos * half;
#pragma unroll 2
    for (int i = tid; i < (h1 - h0) * L.dp; i += MP_THREADS) {
        const int hd = i / L.dp, e = i - hd * L.dp, j = hd * L.d + e;
        float o = 0.f, raw = 0.f;
        if (e < L.d) {
            raw = sv[j];
            o = raw * inv * nw[i0 + j];
            if (e < L.rot) {
                const bool first = e < half;
                const int a = first ? e : e - half, jo = first ? j + half : j - half;
                const float other = sv[jo] * inv * nw[i0 + jo];
                o = first ? o * ct[a] - other * st[a] : o * ct[a] + other * st[a];
            }
        }
        dst[h0 * L.dp + i] = to_t<T>(o);
        if (!is_q) vdst[i] = to_t<T>(raw);
    }
}

// two adjacent elements (one 2 x sizeof(T) load when `pair`: the address is aligned to it)
template <typename T>
__device__ __forceinline__ float2 mp_ld2(const T* p, bool pair, bool second) {
    if (pair) {
        if constexpr (sizeof(T) == 4) return *(const float2*)p;
        else return __bfloat1622float2(*(const __nv_bfloat162*)p);
    }
    return make_float2(ld_f(p), second ? ld_f(p + 1) : 0.f);
}

template <typename T>
__device__ __forceinline__ void mp_conv(const MixLayer& L, const MixRun& R, int blk, int r0, int rows) {
    __shared__ int s_local[MP_MAX_ROWS], s_seq[MP_MAX_ROWS];
    const int tid = threadIdx.x, C = L.heads * L.P + 2 * L.groups * L.N, c = blk * MP_COLS + 2 * tid, K = L.taps - 1;
    if (tid < rows) {
        // rows of the same sequence in front of this one in the launch, as far as the taps reach
        const int r = r0 + tid, seq = R.rows[r].seq;
        int local = 0;
        while (local < K && r - local - 1 >= 0 && R.rows[r - local - 1].seq == seq) ++local;
        s_local[tid] = local; s_seq[tid] = seq;
    }
    const bool in = c < C, second = c + 1 < C;
    const bool pair = second && ((L.off_x | R.ld_proj | C) & 1) == 0, pair_out = second && (R.ld_xbc & 1) == 0;
    float b0 = 0.f, b1 = 0.f, w0[MP_TAPS], w1[MP_TAPS];
    const bool regs = L.taps <= MP_TAPS;
    if (in) {
        b0 = L.conv_b[c]; b1 = second ? L.conv_b[c + 1] : 0.f;
#pragma unroll
        for (int j = 0; j < MP_TAPS; ++j) {
            w0[j] = (regs && j < L.taps) ? L.conv_w[(size_t)c * L.taps + j] : 0.f;
            w1[j] = (regs && j < L.taps && second) ? L.conv_w[(size_t)(c + 1) * L.taps + j] : 0.f;
        }
    }
    pdl_wait();
    __syncthreads();
    if (blk == 0)
        for (int i = tid; i < rows * L.heads; i += MP_THREADS) {
            const int r = r0 + i / L.heads, h = i % L.heads;
            R.dtb[(size_t)r * R.ld_dt + h] = softplus_p(ld_f((const T*)R.proj + (size_t)r * R.ld_proj + L.off_dt + h) + L.dt_bias[h]);
        }
    if (!in) return;
    for (int i = 0; i < rows; ++i) {
        const int r = r0 + i, local = s_local[i];
        const T* row = (const T*)R.proj + (size_t)r * R.ld_proj + L.off_x + c;
        const T* hist = (const T*)L.conv_state + (size_t)s_seq[i] * K * C + c;
        auto tap = [&](int j) {                              // weight j belongs to the input K - j tokens back
            const int back = K - j;
            return back <= local ? mp_ld2(row - (size_t)back * R.ld_proj, pair, second)
                                 : mp_ld2(hist + (size_t)(K - (back - local)) * C, pair, second);
        };
        float a0 = b0, a1 = b1;
        if (regs) {
            float2 v[MP_TAPS];
#pragma unroll
            for (int j = 0; j < MP_TAPS; ++j) v[j] = j < L.taps ? tap(j) : make_float2(0.f, 0.f);
#pragma unroll
            for (int j = 0; j < MP_TAPS; ++j) { a0 = fmaf(w0[j], v[j].x, a0); a1 = fmaf(w1[j], v[j].y, a1); }
        } else
            for (int j = 0; j < L.taps; ++j) {
                const float2 v = tap(j);
                a0 = fmaf(L.conv_w[(size_t)c * L.taps + j], v.x, a0);
                if (second) a1 = fmaf(L.conv_w[(size_t)(c + 1) * L.taps + j], v.y, a1);
            }
        T* out = (T*)R.xbc + (size_t)r * R.ld_xbc + c;
        const T o0 = to_t<T>(silu_p(a0)), o1 = to_t<T>(silu_p(a1));
        if (pair_out) {
            if constexpr (sizeof(T) == 4) *(float2*)out = make_float2(o0, o1);
            else { __nv_bfloat162 h; h.x = o0; h.y = o1; *(__nv_bfloat162*)out = h; }
        } else { out[0] = o0; if (second) out[1] = o1; }
    }
}

template <typename T>
__global__ void __launch_bounds__(MP_THREADS) mix_prepare_kernel(const MixLayer L, const MixRun R, int q_slices, int col_blocks, int conv_rows) {
    extern __shared__ float mp_v[];              // the heads a CTA rotates
    __shared__ float red[32];
    pdl_launch_dependents();
    const int nh = R.n_rows * (q_slices + 1);
    int b = blockIdx.x;
    if (b < nh) { mp_heads<T>(L, R, b / (q_slices + 1), b % (q_slices + 1), q_slices, mp_v, red); return; }
    b -= nh;
    const int r0 = (b / col_blocks) * conv_rows;
    mp_conv<T>(L, R, b % col_blocks, r0, min(conv_rows, R.n_rows - r0));
}

// ---------------------------------------------------------------------------
// head_prepare: one warp per (row, query head | key head | value head)
// ---------------------------------------------------------------------------
template <typename T, int EPL>
__global__ void __launch_bounds__(256) head_prepare_kernel(const MixLayer L, const MixRun R) {
    __shared__ float sv[8][32 * EPL];
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int per = L.H + L.G + (L.off_v >= 0 ? L.G : 0), unit = blockIdx.x * 8 + warp;
    if (unit >= R.n_rows * per) return;
    const int r = unit / per, j = unit % per;
    const RowMeta rm = R.rows[r];
    const bool is_q = j < L.H, is_v = j >= L.H + L.G;
    const int hd = is_q ? j : (is_v ? j - L.H - L.G : j - L.H), n = is_v ? L.dv : L.d, np = is_v ? L.vp : L.dp;
    const int off = (is_q ? L.off_q : (is_v ? L.off_v : L.off_k)) + hd * n, c0 = lane * EPL;
    const T* src = (const T*)R.proj + (size_t)r * R.ld_proj + off + c0;
    const size_t slot = ((size_t)rm.seq * L.max_seq + rm.slot) * L.G + hd;
    T* dst = is_q ? (T*)R.qbuf + ((size_t)r * L.H + hd) * L.dp : (is_v ? (T*)L.vcache + slot * L.vp : (T*)L.kcache + slot * L.dp);
    const float* nw = is_q ? L.q_norm : L.k_norm;
    const bool vec = ((off | n | R.ld_proj) & (EPL - 1)) == 0;
    float w[EPL], v[EPL], ss = 0.f;
#pragma unroll
    for (int e = 0; e < EPL; ++e) w[e] = (!is_v && c0 + e < n) ? nw[c0 + e] : 0.f;
    pdl_wait();
#pragma unroll
    for (int e = 0; e < EPL; ++e) v[e] = 0.f;
    if (vec && c0 < n) {
        T raw[EPL];
        if constexpr (EPL * sizeof(T) == 4) *(uint32_t*)raw = *(const uint32_t*)src;
        else if constexpr (EPL * sizeof(T) == 8) *(uint2*)raw = *(const uint2*)src;
        else
#pragma unroll
            for (int i = 0; i < (int)(EPL * sizeof(T) / 16); ++i) ((uint4*)raw)[i] = ((const uint4*)src)[i];
#pragma unroll
        for (int e = 0; e < EPL; ++e) v[e] = ld_f(raw + e);
    } else
#pragma unroll
        for (int e = 0; e < EPL; ++e) if (c0 + e < n) v[e] = ld_f(src + e);
    auto put = [&](T* d, int len, const float (&o)[EPL]) {          // (len is a multiple of 8)
        if (c0 >= len) return;
        T raw[EPL];
#pragma unroll
        for (int e = 0; e < EPL; ++e) raw[e] = to_t<T>(o[e]);
        if constexpr (EPL * sizeof(T) == 4) *(uint32_t*)(d + c0) = *(const uint32_t*)raw;
        else if constexpr (EPL * sizeof(T) == 8) *(uint2*)(d + c0) = *(const uint2*)raw;
        else
#pragma unroll
            for (int i = 0; i < (int)(EPL * sizeof(T) / 16); ++i) ((uint4*)(d + c0))[i] = ((const uint4*)raw)[i];
    };
    if (is_v) { put(dst, np, v); return; }
    if (!is_q && L.off_v < 0) put((T*)L.vcache + slot * L.vp, L.vp, v);
#pragma unroll
    for (int e = 0; e < EPL; ++e) ss += v[e] * v[e];
    const float inv = rsqrtf(warp_sum(ss) / (float)n + L.eps);
#pragma unroll
    for (int e = 0; e < EPL; ++e) v[e] *= inv * w[e];
    if (L.rot > 0) {
        const int half = L.rot >> 1;
        const float* ct = L.cos_tab + (size_t)rm.pos * half;
        const float* st = L.sin_tab + (size_t)rm.pos * half;
#pragma unroll
        for (int e = 0; e < EPL; ++e) sv[warp][c0 + e] = v[e];
        __syncwarp();
#pragma unroll
        for (int e = 0; e < EPL; ++e) {
            const int i = c0 + e;
            if (i >= L.rot) continue;
            const bool first = i < half;
            const int a = first ? i : i - half;
            const float other = sv[warp][first ? i + half : a];
            v[e] = first ? v[e] * ct[a] - other * st[a] : v[e] * ct[a] + other * st[a];
        }
    }
    put(dst, np, v);
}
template <typename T>
static int launch_hp(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    const int per = l->H + l->G + (l->off_v >= 0 ? l->G : 0), m = l->dp > l->vp ? l->dp : l->vp;
    const dim3 grid((r->n_rows * per + 7) / 8), block(256);
    if (m <= 64) return launch_pdl(head_prepare_kernel<T, 2>, grid, block, 0, s, *l, *r);
    if (m <= 128) return launch_pdl(head_prepare_kernel<T, 4>, grid, block, 0, s, *l, *r);
    return launch_pdl(head_prepare_kernel<T, 8>, grid, block, 0, s, *l, *r);
}

B2_API int b2_head_prepare(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    if (!attn_valid(l) || !l->head_norm || !l->q_norm || !l->k_norm || (l->off_v < 0 && l->dv != l->d) || (l->rot > 0 && !l->cos_tab))
        return cudaErrorInvalidValue;
    return r->dt == DT_BF16 ? launch_hp<bf16>(l, r, s) : launch_hp<float>(l, r, s);
}

B2_API int b2_mix_prepare(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    if (!attn_valid(l) || l->head_norm || l->off_v >= 0 || l->dv != l->d) return cudaErrorInvalidValue;
    if (l->H < 1 || l->G < 1 || l->H % l->G || l->d > 256 || l->dp < l->d || (l->dp & 7) || l->rot > l->d || (l->rot & 1) ||
        l->taps < 1 || l->groups < 1 || l->heads % l->groups)
        return cudaErrorInvalidValue;
    const int C = l->heads * l->P + 2 * l->groups * l->N;
    // few rows: cut the query heads so that a slice is one pass of a CTA; many rows fill the GPU as they are
    int qs = r->n_rows <= B2_MAX_ROWS ? (l->H * l->d + 511) / 512 : 1;
    if (qs > l->H) qs = l->H;
    const int per = (l->H + qs - 1) / qs;
    qs = (l->H + per - 1) / per;
    const int cb = (C + MP_COLS - 1) / MP_COLS, cr = r->n_rows <= B2_MAX_ROWS ? 1 : MP_MAX_ROWS;
    const dim3 grid(r->n_rows * (qs + 1) + cb * ((r->n_rows + cr - 1) / cr));
    const size_t smem = (size_t)(per > l->G ? per : l->G) * l->d * sizeof(float);
    static SmemOptIn opt[2];
    if (r->dt == DT_BF16) {
        if (int e = opt[0].ensure((const void*)mix_prepare_kernel<bf16>, smem)) return e;
        return launch_pdl(mix_prepare_kernel<bf16>, grid, dim3(MP_THREADS), smem, s, *l, *r, qs, cb, cr);
    }
    if (int e = opt[1].ensure((const void*)mix_prepare_kernel<float>, smem)) return e;
    return launch_pdl(mix_prepare_kernel<float>, grid, dim3(MP_THREADS), smem, s, *l, *r, qs, cb, cr);
}

// ---------------------------------------------------------------------------
// decode: grid (G * head blocks, rows, splits)
// ---------------------------------------------------------------------------
#define WD_WARPS 8
#define WD_THREADS (WD_WARPS * 32)
#define WD_GT 8                  // query heads per CTA
#define WD_KEYS 4                // keys of a warp per soft-max update (and as many on their way)
#define WD_MIN_SPLIT 64          // keys that are worth a CTA of their own
#define WD_MAX_SPLITS 32

// EPL consecutive elements of a cache row, as loaded
template <typename T, int EPL> struct WRaw { uint32_t w[EPL * sizeof(T) / 4]; };
template <typename T, int EPL>
__device__ __forceinline__ void wr_load(WRaw<T, EPL>& v, const T* p, bool ok) {
    constexpr int NW = EPL * sizeof(T) / 4;
#pragma unroll
    for (int i = 0; i < NW; ++i) v.w[i] = 0u;
    if (!ok) return;
    if constexpr (NW % 4 == 0) {
#pragma unroll
        for (int i = 0; i < NW / 4; ++i) {
            const uint4 u = ((const uint4*)p)[i];
            v.w[4 * i] = u.x; v.w[4 * i + 1] = u.y; v.w[4 * i + 2] = u.z; v.w[4 * i + 3] = u.w;
        }
    } else if constexpr (NW == 2) { const uint2 u = *(const uint2*)p; v.w[0] = u.x; v.w[1] = u.y; }
    else v.w[0] = *(const uint32_t*)p;
}
template <typename T, int EPL>
__device__ __forceinline__ float wr_get(const WRaw<T, EPL>& v, int e) {
    if constexpr (sizeof(T) == 4) return __uint_as_float(v.w[e]);
    else return __uint_as_float((e & 1) ? (v.w[e >> 1] & 0xffff0000u) : (v.w[e >> 1] << 16));
}

// EXT: kept first keys, capped scores, a sink, values of another size than the keys
template <typename T, int EPL, int GT, bool EXT>
__global__ void __launch_bounds__(WD_THREADS) window_decode_kernel(const MixLayer L, const MixRun R) {
    const int Gq = L.H / L.G, nhb = (Gq + GT - 1) / GT;
    const int kvh = blockIdx.x / nhb, hb = (blockIdx.x % nhb) * GT, nh = min(GT, Gq - hb);
    const int r = blockIdx.y, sp = blockIdx.z;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    pdl_launch_dependents();
    const RowMeta rm = R.rows[r];
    const int k1 = rm.pos + 1;                                               // keys [k0, k1)
    const int k0 = L.window > 0 ? max(0, k1 - L.window) : 0;
    // the keys a row sees, in order: kf kept first ones, then its window
    const int kf = EXT ? min(L.keep_first, k0) : 0, total = kf + k1 - k0, jump = k0 - kf;
    const int nsplit = max(1, min(R.splits, (total + WD_MIN_SPLIT - 1) / WD_MIN_SPLIT));
    if (sp >= nsplit) return;
    const int per = (total + nsplit - 1) / nsplit;
    const int a0 = sp * per, a1 = min(total, a0 + per);
    __shared__ float sm_m[WD_WARPS][GT], sm_l[WD_WARPS][GT], sm_f[WD_MAX_SPLITS][GT], sm_li[GT];
    __shared__ float sm_acc[WD_WARPS][32 * EPL];
    __shared__ int s_last;
    pdl_wait();
    const int col = lane * EPL;
    const bool in = col < L.dp, in_v = EXT ? col < L.vp : in;           // multiples of EPL (<= 8): lanes are in or out as a whole
    // Scores of WD_KEYS keys x GT heads are summed over the lanes by recursive halving: every step a lane hands
    // half of its values to its partner and keeps the other half, so afterwards each lane holds ONE finished
    // score (the value with index lane >> SH) and the soft-max costs one exponential per lane.  The running
    // maximum and sum of a head live in the lanes of its scores.
    constexpr int NV = WD_KEYS * GT, SH = NV == 32 ? 0 : NV == 16 ? 1 : NV == 8 ? 2 : 3;
    const int mykey = (lane >> SH) & (WD_KEYS - 1);
    float q[GT][EPL], acc[GT][EPL], m_l = -INFINITY, l_l = 0.f;
#pragma unroll
    for (int h = 0; h < GT; ++h) {
        WRaw<T, EPL> qv;
        wr_load(qv, (const T*)R.qbuf + ((size_t)r * L.H + kvh * Gq + hb + h) * L.dp + col, in && h < nh);
#pragma unroll
        for (int e = 0; e < EPL; ++e) { q[h][e] = wr_get(qv, e) * L.attn_scale; acc[h][e] = 0.f; }
    }
    const size_t base = (size_t)rm.seq * L.max_seq * L.G + kvh, stride = (size_t)L.G * L.dp, vstride = EXT ? (size_t)L.G * L.vp : stride;
    const T* kc = (const T*)L.kcache + base * L.dp + col;
    const T* vc = (const T*)L.vcache + base * (EXT ? L.vp : L.dp) + col;
    const int dv = EXT ? L.dv : L.d;
    WRaw<T, EPL> kn[WD_KEYS], vn[WD_KEYS];
    auto fetch = [&](int s) {
#pragma unroll
        for (int i = 0; i < WD_KEYS; ++i) {
            const int idx = s + i * WD_WARPS + warp, key = EXT && idx < kf ? idx : idx + jump;
            const bool ok = idx < a1;
            wr_load(kn[i], kc + (size_t)key * stride, in && ok);
            wr_load(vn[i], vc + (size_t)key * vstride, in_v && ok);
        }
    };
    if (a0 < a1) fetch(a0);
    for (int s = a0; s + warp < a1; s += WD_WARPS * WD_KEYS) {
        WRaw<T, EPL> kk[WD_KEYS], vv[WD_KEYS];
#pragma unroll
        for (int i = 0; i < WD_KEYS; ++i) { kk[i] = kn[i]; vv[i] = vn[i]; }
        if (s + WD_WARPS * WD_KEYS < a1) fetch(s + WD_WARPS * WD_KEYS);
        float d[NV];                                         // [head][key]
#pragma unroll
        for (int h = 0; h < GT; ++h)
#pragma unroll
            for (int i = 0; i < WD_KEYS; ++i) {
                float x = 0.f;
                if (h < nh)
#pragma unroll
                    for (int e = 0; e < EPL; ++e) x = fmaf(q[h][e], wr_get(kk[i], e), x);
                d[h * WD_KEYS + i] = x;
            }
        int off = 16;
#pragma unroll
        for (int n = NV; n > 1; n >>= 1, off >>= 1) {
            const bool up = lane & off;
#pragma unroll
            for (int i = 0; i < n / 2; ++i) {
                const float give = up ? d[i] : d[i + n / 2], keep = up ? d[i + n / 2] : d[i];
                d[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
            }
        }
#pragma unroll
        for (int o = 16 / NV; o > 0; o >>= 1) d[0] += __shfl_xor_sync(0xffffffffu, d[0], o);
        if (EXT && L.softcap > 0.f) d[0] = L.softcap * tanhf(d[0] / L.softcap);
        const float sc = s + mykey * WD_WARPS + warp < a1 ? d[0] : -INFINITY;
        float mn = sc;
#pragma unroll
        for (int o = 1; o < WD_KEYS; o <<= 1) mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, o << SH));
        mn = fmaxf(mn, m_l);                                 // (the first key of the pass is always inside: finite)
        const float corr_l = expf(m_l - mn), p_l = expf(sc - mn);
        float ps = p_l;
#pragma unroll
        for (int o = 1; o < WD_KEYS; o <<= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o << SH);
        l_l = l_l * corr_l + ps;
        m_l = mn;
#pragma unroll
        for (int h = 0; h < GT; ++h) {
            if (h >= nh) break;
            const float corr = __shfl_sync(0xffffffffu, corr_l, (h * WD_KEYS) << SH);
            float pw[WD_KEYS];
#pragma unroll
            for (int i = 0; i < WD_KEYS; ++i) pw[i] = __shfl_sync(0xffffffffu, p_l, (h * WD_KEYS + i) << SH);
#pragma unroll
            for (int e = 0; e < EPL; ++e) {
                float a = acc[h][e] * corr;
#pragma unroll
                for (int i = 0; i < WD_KEYS; ++i) a = fmaf(pw[i], wr_get(vv[i], e), a);
                acc[h][e] = a;
            }
        }
    }
    // ---- merge the warps, one head at a time
    if ((lane & ((WD_KEYS << SH) - 1)) == 0) { sm_m[warp][lane / (WD_KEYS << SH)] = m_l; sm_l[warp][lane / (WD_KEYS << SH)] = l_l; }
    const int unit = (r * L.G + kvh) * nhb + (blockIdx.x % nhb);
    float* my = R.attn_scratch + ((size_t)unit * R.splits + sp) * GT * (32 * EPL + 4);
#pragma unroll
    for (int h = 0; h < GT; ++h) {
        if (h >= nh) break;
        __syncthreads();
#pragma unroll
        for (int e = 0; e < EPL; ++e) sm_acc[warp][col + e] = acc[h][e];
        __syncthreads();
        float mm = -INFINITY;
#pragma unroll
        for (int w = 0; w < WD_WARPS; ++w) mm = fmaxf(mm, sm_m[w][h]);
        const int head = kvh * Gq + hb + h;
        const bool sink = EXT && L.sink && nsplit == 1;             // (slices: the merge below counts it)
        if (sink) mm = fmaxf(mm, L.sink[head]);
        float ll = sink ? expf(L.sink[head] - mm) : 0.f, f[WD_WARPS];
#pragma unroll
        for (int w = 0; w < WD_WARPS; ++w) { f[w] = sm_m[w][h] == -INFINITY ? 0.f : expf(sm_m[w][h] - mm); ll += sm_l[w][h] * f[w]; }
        for (int c = tid; c < dv; c += WD_THREADS) {
            float a = 0.f;
#pragma unroll
            for (int w = 0; w < WD_WARPS; ++w) a += sm_acc[w][c] * f[w];
            if (nsplit == 1) ((T*)R.out)[(size_t)r * R.ldo + head * dv + c] = to_t<T>(a / ll * L.left_scale);
            else {
                my[h * (32 * EPL + 4) + c] = a;
                if (c == 0) { my[h * (32 * EPL + 4) + 32 * EPL] = mm; my[h * (32 * EPL + 4) + 32 * EPL + 1] = ll; }
            }
        }
    }
    if (nsplit == 1) return;
    // ---- merge the slices: the last CTA of this (row, key head, head block)
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        const int old = atomicAdd(&R.attn_counters[unit], 1);
        s_last = old == nsplit - 1;
        if (s_last) R.attn_counters[unit] = 0;
        __threadfence();
    }
    __syncthreads();
    if (!s_last) return;
    const float* all = R.attn_scratch + (size_t)unit * R.splits * GT * (32 * EPL + 4);
    if (tid < nh) {
        const float* e0 = all + tid * (32 * EPL + 4) + 32 * EPL;
        const size_t st = (size_t)GT * (32 * EPL + 4);
        float mv[WD_MAX_SPLITS], lv[WD_MAX_SPLITS], mm = -INFINITY, ll = 0.f;
#pragma unroll
        for (int x = 0; x < WD_MAX_SPLITS; ++x) {
            mv[x] = x < nsplit ? __ldcg(e0 + x * st) : -INFINITY;
            lv[x] = x < nsplit ? __ldcg(e0 + x * st + 1) : 0.f;
        }
#pragma unroll
        for (int x = 0; x < WD_MAX_SPLITS; ++x) mm = fmaxf(mm, mv[x]);
        if (EXT && L.sink) { const float sk = L.sink[kvh * Gq + hb + tid]; mm = fmaxf(mm, sk); ll = expf(sk - mm); }
#pragma unroll
        for (int x = 0; x < WD_MAX_SPLITS; ++x) {
            const float f = mv[x] == -INFINITY ? 0.f : expf(mv[x] - mm);
            ll += lv[x] * f;
            sm_f[x][tid] = f;
        }
        sm_li[tid] = 1.f / ll;
    }
    __syncthreads();
    for (int i = tid; i < nh * dv; i += WD_THREADS) {
        const int h = i / dv, c = i % dv;
        float a = 0.f;
        for (int x0 = 0; x0 < nsplit; x0 += 8) {
            float v[8];
#pragma unroll
            for (int u = 0; u < 8; ++u)
                v[u] = x0 + u < nsplit ? __ldcg(all + ((size_t)(x0 + u) * GT + h) * (32 * EPL + 4) + c) : 0.f;
#pragma unroll
            for (int u = 0; u < 8; ++u) if (x0 + u < nsplit) a = fmaf(v[u], sm_f[x0 + u][h], a);
        }
        ((T*)R.out)[(size_t)r * R.ldo + (kvh * Gq + hb + h) * dv + c] = to_t<T>(a * sm_li[h] * L.left_scale);
    }
}

// floats of scratch for `rows` rows, dp: the larger of MixLayer's dp and vp (attn_counters: rows * G * ceil(H / G / WD_GT) ints)
B2_API long long b2_window_attn_scratch(int H, int G, int dp, int rows, int splits) {
    const int nhb = (H / G + WD_GT - 1) / WD_GT, epl = dp <= 64 ? 2 : dp <= 128 ? 4 : 8;
    return (long long)rows * G * nhb * splits * WD_GT * (32 * epl + 4);
}
B2_API int b2_window_attn_units(int H, int G, int rows) { return rows * G * ((H / G + WD_GT - 1) / WD_GT); }

template <typename T, int EPL, bool EXT>
static int launch_wd(const MixLayer* l, const MixRun* run, cudaStream_t s) {
    const int Gq = l->H / l->G;
    // cache slices beyond what is resident at once would only add a second wave
    MixRun one = *run;
    const int units = l->G * ((Gq + WD_GT - 1) / WD_GT) * run->n_rows, slots = 148 * (Gq > 4 || EPL > 4 ? 1 : 2);
    if (units * one.splits > slots) one.splits = units >= slots ? 1 : slots / units;
    const MixRun* r = &one;
    // (a smaller head block keeps fewer registers; scratch is laid out for at most WD_GT heads per block)
    if (Gq <= 1) return launch_pdl(window_decode_kernel<T, EPL, 1, EXT>, dim3(l->G, r->n_rows, r->splits), dim3(WD_THREADS), 0, s, *l, *r);
    if (Gq <= 2) return launch_pdl(window_decode_kernel<T, EPL, 2, EXT>, dim3(l->G, r->n_rows, r->splits), dim3(WD_THREADS), 0, s, *l, *r);
    if (Gq <= 4) return launch_pdl(window_decode_kernel<T, EPL, 4, EXT>, dim3(l->G, r->n_rows, r->splits), dim3(WD_THREADS), 0, s, *l, *r);
    const int nhb = (Gq + WD_GT - 1) / WD_GT;
    return launch_pdl(window_decode_kernel<T, EPL, WD_GT, EXT>, dim3(l->G * nhb, r->n_rows, r->splits), dim3(WD_THREADS), 0, s, *l, *r);
}
template <typename T, bool EXT>
static int launch_wd_t(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    const int m = l->dp > l->vp ? l->dp : l->vp;
    if (m <= 64) return launch_wd<T, 2, EXT>(l, r, s);
    if (m <= 128) return launch_wd<T, 4, EXT>(l, r, s);
    return launch_wd<T, 8, EXT>(l, r, s);
}
B2_API int b2_window_attn_decode(const MixLayer* l, const MixRun* r, cudaStream_t s) {
    if (!attn_valid(l) || r->splits < 1 || r->splits > WD_MAX_SPLITS) return cudaErrorInvalidValue;
    const bool ext = l->keep_first > 0 || l->softcap > 0.f || l->sink || l->dv != l->d;
    if (r->dt == DT_BF16) return ext ? launch_wd_t<bf16, true>(l, r, s) : launch_wd_t<bf16, false>(l, r, s);
    return ext ? launch_wd_t<float, true>(l, r, s) : launch_wd_t<float, false>(l, r, s);
}

B2_API int b2_sizeof_mix_layer() { return (int)sizeof(MixLayer); }
B2_API int b2_sizeof_mix_run() { return (int)sizeof(MixRun); }
