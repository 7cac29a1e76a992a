"""Every mechanism of the Degedra decoder alone: the CUDA kernels against the plain functions of
degedra_oracle."""
import ctypes as C
from types import SimpleNamespace

import pytest
import torch

import degedra_oracle as O

pytestmark = pytest.mark.gpu
DTS = {"bf16": (torch.bfloat16, 0, 2e-2), "f32": (torch.float32, 1, 2e-5)}


def _close(got, ref, tol):
    got, ref = got.double().cpu(), ref.double().cpu()
    err = float((got - ref).abs().max() / (ref.abs().max() + 1e-9))
    assert err < tol, err


def _rnd(*sh, seed=0, std=1.0):
    return torch.randn(*sh, generator=torch.Generator().manual_seed(seed + sum(sh))) * std


def _lin(w, dtype, rpc):
    N, K = w.shape
    d = torch.zeros(N, -(-K // 8) * 8, dtype=dtype, device="cuda")
    d[:, :K] = w
    few = min(rpc, 32)
    return SimpleNamespace(w=d, N=N, K=K, rpc=max(16, rpc) if dtype == torch.bfloat16 else few, rpc_few=few)


# ------------------------------------------------------------------ projections
@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("mma", [False, True])
@pytest.mark.parametrize("N,K,rows,rpc", [(37, 90, 1, 8), (333, 5000, 2, 128), (64, 200, 3, 16), (301, 2056, 8, 32), (1000, 5000, 2, 8),
                                          (40, 17000, 8, 16), (129, 4096, 5, 32), (700, 1500, 7, 64)])
def test_gemv_dense(dt, N, K, rows, rpc, mma):
    from mi50grad_b200.ops import kernels as K_
    from mi50grad_b200.ops import lib as L
    T, _, tol = DTS[dt]
    w, x = _rnd(N, K, std=K ** -0.5).to(T), _rnd(rows, K, seed=1).to(T)
    lin = _lin(w, T, rpc)
    ref = x.double() @ w.double().T
    xs = torch.zeros(rows, -(-K // 8) * 8, dtype=T, device="cuda")
    xs[:, :K] = x
    xin = xs[:, :K]
    out = torch.full((rows, N), 7.0, device="cuda")
    ss = torch.zeros(rows, -(-N // 8), device="cuda")
    K_.gemv_dense(lin, xin, out, L.DG_STORE_F32, ss_out=ss, mma=mma)
    _close(out, ref, 2e-5)
    assert torch.allclose(ss.sum(1), out.pow(2).sum(1), rtol=1e-4)
    K_.gemv_dense(lin, xin, out, L.DG_STORE_F32, softcap=1.5, mma=mma)
    _close(out, 1.5 * torch.tanh(ref / 1.5), 2e-5)
    o16 = torch.zeros(rows, N, dtype=T, device="cuda")
    K_.gemv_dense(lin, xin, o16, L.DG_STORE, mma=mma)
    _close(o16, ref, tol)


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("mma", [False, True])
@pytest.mark.parametrize("H,rows", [(90, 3), (256, 8), (5000, 1), (168, 2)])
def test_gemv_dense_forms_the_residual_update(dt, H, rows, mma):
    from mi50grad_b200.ops import kernels as K_
    from mi50grad_b200.ops import lib as L
    T, _, tol = DTS[dt]
    h, m, nw = _rnd(rows, H), _rnd(rows, H, seed=2, std=3.0), 1 + _rnd(H, seed=3, std=0.2)
    w = _rnd(48, H, std=H ** -0.5).to(T)
    x = h.double() + O.rms(m.double(), 1e-5) * nw.double()
    hd, md, wd = h.cuda(), m.cuda(), nw.cuda()
    hout = torch.zeros_like(hd)
    parts = 11
    ss = torch.stack([c.pow(2).sum(1) for c in md.split(-(-H // parts), dim=1)], 1).contiguous()
    out = torch.zeros(rows, 48, device="cuda")
    pn = K_.post_norm_input(hd, md, wd, ss, hout, 1e-5)
    K_.gemv_dense(_lin(w, T, 16), None, out, L.DG_STORE_F32, pn=pn, rows=rows, mma=mma)
    _close(hout, x, 2e-6)
    assert torch.equal(hd.cpu(), h)
    _close(out, x.to(T).double() @ w.double().T, tol)
    K_.gemv_dense(_lin(w, T, 8), None, out, L.DG_STORE_F32, pn=K_.post_norm_input(hd), rows=rows, mma=mma)
    _close(out, h.to(T).double() @ w.double().T, tol)


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("F,K,rows", [(33, 90, 1), (200, 168, 8), (3000, 512, 4)])
def test_gate_up_pair(dt, F, K, rows):
    from mi50grad_b200.engine.mixer_engine import interleave_dense_gate_up
    from mi50grad_b200.ops import kernels as K_
    from mi50grad_b200.ops import lib as L
    T, _, tol = DTS[dt]
    g, u, x = _rnd(F, K, std=K ** -0.5).to(T), _rnd(F, K, seed=1, std=K ** -0.5).to(T), _rnd(rows, K, seed=2).to(T)
    ref = O.silu(x.double() @ g.double().T) * (x.double() @ u.double().T)
    both = interleave_dense_gate_up(g, u)
    xs = torch.zeros(rows, -(-K // 8) * 8, dtype=T, device="cuda")
    xs[:, :K] = x
    out = torch.zeros(rows, -(-F // 8) * 8, dtype=T, device="cuda")
    for rpc in (16, 32):
        out.fill_(3.0)
        K_.gemv_dense(_lin(both, T, rpc), xs[:, :K], out, L.DG_GATE_PAIR)
        _close(out[:, :F], ref, tol)
        assert float(out[:, F:].abs().sum()) == 0
    out.fill_(3.0)
    lin = _lin(both, T, 16)
    if dt == "bf16":
        K_.gemm_bf16_tc(lin.w[:, :K], xs[:, :K], out, L.TC_EPI_SILU_PAIR)
    else:
        K_.gemm_f32(lin.w[:, :K], xs[:, :K], out, L.DG_GATE_PAIR)
    _close(out[:, :F], ref, tol)


@pytest.mark.parametrize("N,K,T_", [(37, 90, 9), (300, 200, 64), (640, 1032, 130), (129, 4096, 511)])
def test_many_row_gemms(N, K, T_):
    from mi50grad_b200.ops import kernels as K_
    from mi50grad_b200.ops import lib as L
    w, x = _rnd(N, K, std=K ** -0.5), _rnd(T_, K, seed=1)
    out = torch.zeros(T_, N, device="cuda")
    K_.gemm_f32(w.cuda(), x.cuda(), out, softcap=0.0)
    _close(out, x.double() @ w.double().T, 1e-5)
    K_.gemm_f32(w.cuda(), x.cuda(), out, L.DG_STORE_F32, softcap=2.0)
    _close(out, 2 * torch.tanh(x.double() @ w.double().T / 2), 1e-5)
    wb, xb = _lin(w, torch.bfloat16, 8).w, _lin(x, torch.bfloat16, 8).w
    ref = x.bfloat16().double() @ w.bfloat16().double().T
    K_.gemm_bf16_tc(wb[:, :K], xb[:, :K], out)
    _close(out, ref, 1e-5)
    K_.gemm_bf16_tc(wb[:, :K], xb[:, :K], out, softcap=2.0)
    _close(out, 2 * torch.tanh(ref / 2), 1e-5)
    o16 = torch.zeros(T_, N, dtype=torch.bfloat16, device="cuda")
    K_.gemm_bf16_tc(wb[:, :K], xb[:, :K], o16, L.TC_EPI_STORE_F16)
    _close(o16, ref, 1e-2)
    K_.gemm_tc_check_status()


@pytest.mark.parametrize("N,K,T_,t", [(640, 1032, 130, 256), (129, 4096, 511, 512), (900, 512, 512, 512), (384, 640, 300, 256)])
def test_gemm_cta_pairs_and_k_splits(N, K, T_, t):
    """Two-CTA tiles (odd tile counts and ragged token counts too), and products left as planes to be summed."""
    from mi50grad_b200.ops import kernels as K_
    from mi50grad_b200.ops import lib as L
    w, x = _lin(_rnd(N, K, std=K ** -0.5), torch.bfloat16, 8).w, _lin(_rnd(T_, K, seed=1), torch.bfloat16, 8).w
    w, x = w[:, :K], x[:, :K]
    ref = x.double().cpu() @ w.double().cpu().T
    out = torch.zeros(T_, N, device="cuda")
    K_.gemm_bf16_tc(w, x, out, t_tile=t, cta_pair=True)
    _close(out, ref, 1e-5)
    if N % 16 == 0:
        o16 = torch.zeros(T_, N // 2, dtype=torch.bfloat16, device="cuda")
        K_.gemm_bf16_tc(w, x, o16, L.TC_EPI_SILU_PAIR, t_tile=t, cta_pair=True)
        r = ref.reshape(T_, N // 16, 2, 8)
        _close(o16, (O.silu(r[:, :, 0]) * r[:, :, 1]).reshape(T_, N // 2), 1e-2)
    for pair in (True, False):
        for ks in (2, 3):
            planes = torch.zeros(ks, T_, N, device="cuda")
            K_.gemm_bf16_tc(w, x, planes, t_tile=t if pair else 128, cta_pair=pair, k_splits=ks)
            _close(planes.sum(0), ref, 1e-5)
            assert float(planes[-1].abs().max()) > 0
    K_.gemm_tc_check_status()


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("H", [90, 168, 4096])
def test_post_norm(dt, H):
    from mi50grad_b200.ops import kernels as K_
    T, _, tol = DTS[dt]
    h, m, w, f = _rnd(5, H), _rnd(5, H, seed=1, std=0.01), 1 + _rnd(H, seed=2, std=0.3), 1 + _rnd(H, seed=3, std=0.3)
    x = h.double() + O.rms(m.double(), 1e-4) * w.double()
    for fw in (None, f):
        hd = h.cuda()
        xb = torch.zeros(5, -(-H // 8) * 8, dtype=T, device="cuda")
        K_.post_norm_(hd, m.cuda(), w.cuda(), xb, 1e-4, None if fw is None else fw.cuda())
        _close(hd, x, 2e-6)
        _close(xb[:, :H], x if fw is None else O.rms(x, 1e-4) * f.double(), tol)
        hd = h.cuda()
        parts = torch.stack([0.25 * m, 0.5 * m, 0.25 * m]).cuda()
        K_.post_norm_(hd, parts, w.cuda(), xb, 1e-4, None if fw is None else fw.cuda())
        _close(hd, x, 2e-6)


# ------------------------------------------------------------------ the mixer's kernels
class Mix:
    """One parallel layer with random tensors, its caches and its work buffers."""

    def __init__(self, dt, H=4, G=2, d=40, rot=24, window=11, heads=6, P=20, N=24, groups=3, ngroups=4, taps=4, slots=3,
                 max_seq=512, scale=0.3, seed=0, rows=400):
        from mi50grad_b200.ops import lib as L
        self.T, code, self.tol = DTS[dt]
        self.H, self.G, self.d, self.rot, self.window, self.scale = H, G, d, rot, window, scale
        self.heads, self.P, self.N, self.groups, self.ngroups, self.taps = heads, P, N, groups, ngroups, taps
        self.I, self.C, self.dp = heads * P, heads * P + 2 * groups * N, -(-d // 8) * 8
        self.eps, self.base, self.ls, self.rs = 1e-5, 700.0, 0.6, 1.7
        c = lambda t: t.float().cuda().contiguous()
        rt = lambda t: t.to(self.T).float()
        self.q_norm, self.k_norm = 1 + _rnd(H * d, seed=seed, std=0.2), 1 + _rnd(G * d, seed=seed + 1, std=0.2)
        self.conv, self.conv_b = _rnd(self.C, taps, seed=seed + 2, std=taps ** -0.5), _rnd(self.C, seed=seed + 3, std=0.2)
        self.dt_bias, self.A_log = _rnd(heads, seed=seed + 4) - 1.0, _rnd(heads, seed=seed + 5)
        self.D, self.norm_w = _rnd(heads, seed=seed + 6), 1 + _rnd(self.I, seed=seed + 7, std=0.2)
        self.dev = {n: c(getattr(self, n)) for n in ("q_norm", "k_norm", "conv", "conv_b", "dt_bias", "A_log", "D", "norm_w")}
        f = torch.tensor([self.base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
        ang = torch.arange(max_seq, dtype=torch.float64)[:, None] * f[None]
        z = lambda *s, dtype=self.T: torch.zeros(*s, dtype=dtype, device="cuda")
        self.k, self.v = z(slots, max_seq, G, self.dp), z(slots, max_seq, G, self.dp)
        self.S = z(slots, heads, N, P, dtype=torch.float32)
        self.hist = z(slots, taps - 1, self.C)
        self.keep = [c(torch.cos(ang)), c(torch.sin(ang))]
        m = self.m = L.MixLayer()
        m.H, m.G, m.d, m.dp, m.rot, m.window = H, G, d, self.dp, rot, window
        m.attn_scale, m.left_scale, m.right_scale, m.eps = scale, self.ls, self.rs, self.eps
        for n in ("q_norm", "k_norm", "conv_b", "dt_bias", "A_log", "D", "norm_w"):
            setattr(m, n, self.dev[n].data_ptr())
        m.conv_w, m.cos_tab, m.sin_tab = self.dev["conv"].data_ptr(), self.keep[0].data_ptr(), self.keep[1].data_ptr()
        m.kcache, m.vcache, m.state, m.conv_state = self.k.data_ptr(), self.v.data_ptr(), self.S.data_ptr(), self.hist.data_ptr()
        m.heads, m.P, m.N, m.groups, m.ngroups, m.taps = heads, P, N, groups, ngroups, taps
        m.off_q, m.off_k, m.off_z = 0, H * d, H * d + G * d
        m.off_x, m.off_dt, m.max_seq = m.off_z + self.I, m.off_z + self.I + self.C, max_seq
        m.dv, m.vp, m.off_v, m.rx, m.rB, m.rC, m.out_col = d, self.dp, -1, 0, self.I, self.I + groups * N, H * d
        self.ld = -(-(m.off_dt + heads) // 8) * 8
        self.ld_xbc, self.ldo = -(-self.C // 8) * 8, -(-(H * d + self.I) // 8) * 8
        lib = L.lib()
        self.splits, R = 5, rows
        self.b = dict(proj=z(R, self.ld), qbuf=z(R, H * self.dp), xbc=z(R, self.ld_xbc), dtb=z(R, heads, dtype=torch.float32),
                      ubuf=z(R, self.I, dtype=torch.float32), out=z(R, self.ldo),
                      attn_scratch=z(lib.b2_window_attn_scratch(H, G, self.dp, R, self.splits), dtype=torch.float32),
                      attn_counters=z(lib.b2_window_attn_units(H, G, R), dtype=torch.int32),
                      ssd_counters=z(lib.b2_ssd_units(C.byref(m), R), dtype=torch.int32),
                      chunk_state=z(lib.b2_ssd_chunk_state_floats(C.byref(m), R), dtype=torch.float32),
                      chunk_prev=torch.zeros(lib.b2_ssd_chunk_prev_bytes(C.byref(m), R), dtype=torch.uint8, device="cuda"),
                      chunk_decay=z(-(-R // 64) * heads, dtype=torch.float32))
        r = self.r = L.MixRun()
        for n, t in self.b.items():
            setattr(r, n, t.data_ptr())
        r.dt, r.ld_proj, r.ld_xbc, r.ld_dt, r.ld_u, r.ldo = code, self.ld, self.ld_xbc, heads, self.I, self.ldo
        r.splits, r.commit = self.splits, 1

    def rows(self, parts):
        """parts: [(slot, first position, count)] -> sets the row tables, returns the row count."""
        ent, sr = [], [0]
        for s, p0, n in parts:
            ent += [(s, p0 + i, p0 + i, p0 + i + 1, 0) for i in range(n)]
            sr.append(sr[-1] + n)
        from mi50grad_b200.ops.kernels import make_rows
        self.keep_rows = (make_rows(ent, "cuda"), torch.tensor(sr, dtype=torch.int32, device="cuda"))
        self.r.rows, self.r.seq_rows = self.keep_rows[0].data_ptr(), self.keep_rows[1].data_ptr()
        self.r.n_rows, self.r.n_seqs = sr[-1], len(parts)
        self.r.fuse_norm = int(sr[-1] == len(parts) or sr[-1] <= 8)
        return sr[-1]

    def op(self, name):
        from mi50grad_b200.ops.kernels import mix_op
        mix_op(name, self.m, self.r)

    # plain counterparts, from the projection rows of one sequence
    def ref_qkv(self, proj, p0=0):
        p, H, G, d = proj.double(), self.H, self.G, self.d
        pos = torch.arange(p0, p0 + p.shape[0])
        q = O.rms(p[:, :H * d], self.eps) * self.q_norm.double()
        kr = p[:, H * d:H * d + G * d]
        k = O.rms(kr, self.eps) * self.k_norm.double()
        rot = lambda t, h: O.rotate_half(t.reshape(-1, h, d), pos, self.rot, self.base)
        return rot(q, H), rot(k, G), kr.reshape(-1, G, d)

    def ref_ssd(self, proj, S=None, hist=None):
        """-> (normalised output, state, history, u before the norm, conv outputs, dt)"""
        p = proj.double()
        o = self.m.off_z
        z, xbc, dt = p[:, o:o + self.I], p[:, o + self.I:o + self.I + self.C], p[:, self.m.off_dt:self.m.off_dt + self.heads]
        S = torch.zeros(self.heads, self.N, self.P, dtype=torch.float64) if S is None else S
        hist = torch.zeros(self.taps - 1, self.C, dtype=torch.float64) if hist is None else hist
        y, hist = O.causal_conv_silu(xbc, self.conv.double(), self.conv_b.double(), hist)
        yc = y.to(self.T).double()                               # the kernels hand the convolution on in the element type
        dt = O.softplus(dt + self.dt_bias.double())
        n, I, GN = p.shape[0], self.I, self.groups * self.N
        o_, S = O.ssd_recurrence(yc[:, :I].reshape(n, self.heads, self.P), yc[:, I:I + GN].reshape(n, self.groups, self.N),
                                 yc[:, I + GN:].reshape(n, self.groups, self.N), dt, self.A_log, self.D, S)
        out = O.gated_group_norm(o_.reshape(n, I), z, self.norm_w.double(), self.ngroups, self.eps)
        return out * self.rs, S, hist, o_.reshape(n, I) * O.silu(z), y, dt


SHAPES = [dict(), dict(H=12, G=1, d=32, rot=32, heads=5, P=33, N=17, groups=1, ngroups=5, taps=2),
          dict(H=3, G=3, d=100, rot=64, heads=2, P=72, N=130, groups=2, ngroups=1, taps=5),
          dict(H=8, G=2, d=64, rot=64, heads=8, P=64, N=128, groups=1, ngroups=2, taps=4),
          dict(H=10, G=2, d=128, rot=96, heads=6, P=24, N=48, groups=3, ngroups=2, taps=3),
          dict(H=2, G=1, d=256, rot=128, heads=1, P=128, N=256, groups=1, ngroups=1, taps=1)]


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("shape", range(len(SHAPES)))
def test_prepare(dt, shape):
    x = Mix(dt, **SHAPES[shape])
    n = x.rows([(1, 5, 4), (0, 0, 1), (2, 100, 7)])
    proj = _rnd(n, x.ld).to(x.T)
    hist = _rnd(3, x.taps - 1, x.C, seed=9).to(x.T)
    x.b["proj"][:n] = proj.cuda()
    x.hist.copy_(hist)
    x.op("mix_prepare")
    row = 0
    for slot, p0, cnt in ((1, 5, 4), (0, 0, 1), (2, 100, 7)):
        pr = proj[row:row + cnt]
        q, k, v = x.ref_qkv(pr, p0)
        got = x.b["qbuf"][row:row + cnt].reshape(cnt, x.H, x.dp)
        _close(got[..., :x.d], q, x.tol)
        assert float(got[..., x.d:].abs().sum()) == 0
        _close(x.k[slot, p0:p0 + cnt, :, :x.d], k, x.tol)
        assert torch.equal(x.v[slot, p0:p0 + cnt, :, :x.d].cpu().double(), v)
        _, _, _, _, y, dts = x.ref_ssd(pr, hist=hist[slot].double())
        _close(x.b["xbc"][row:row + cnt, :x.C], y, x.tol)
        _close(x.b["dtb"][row:row + cnt], dts, 1e-5)
        row += cnt


def _fill_cache(x, slot, n, seed=3):
    k, v = _rnd(n, x.G, x.d, seed=seed).to(x.T), _rnd(n, x.G, x.d, seed=seed + 1).to(x.T)
    x.k[slot, :n, :, :x.d] = k.cuda()
    x.v[slot, :n, :, :x.d] = v.cuda()
    return k, v


def _set_q(x, q):
    x.b["qbuf"][:q.shape[0]].zero_()
    x.b["qbuf"][:q.shape[0]].reshape(-1, x.H, x.dp)[..., :x.d] = q.cuda()


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("shape", range(len(SHAPES)))
@pytest.mark.parametrize("window", [1, 11, 64, 200, 0])
def test_window_attention_decode(dt, shape, window):
    x = Mix(dt, window=window, **SHAPES[shape])
    parts = [(0, 0, 1), (2, 299, 1), (1, 150, 3), (0, 1, 2)]
    n = x.rows(parts)
    q = _rnd(n, x.H, x.d).to(x.T)
    _set_q(x, q)
    kv = {s: _fill_cache(x, s, 300, seed=10 * s) for s in range(3)}
    for splits in (1, x.splits):
        x.r.splits = splits
        x.b["out"].fill_(9.0)
        x.op("window_attn_decode")
        row = 0
        for s, p0, cnt in parts:
            k, v = kv[s]
            ref = O.window_attention(q[row:row + cnt].double(), k.double(), v.double(), x.scale, window or 10 ** 9, p0) * x.ls
            _close(x.b["out"][row:row + cnt, :x.H * x.d].reshape(cnt, x.H, x.d), ref, x.tol)
            row += cnt
        assert int(x.b["attn_counters"].abs().sum()) == 0
        assert torch.all(x.b["out"][:, x.H * x.d:] == 9.0)


@pytest.mark.parametrize("shape", range(len(SHAPES)))
@pytest.mark.parametrize("p0,n,window", [(0, 16, 11), (0, 130, 1), (37, 100, 64), (191, 65, 63), (5, 200, 0), (128, 64, 65)])
def test_window_attention_rows(shape, p0, n, window):
    x = Mix("bf16", window=window, **SHAPES[shape])
    x.rows([(1, p0, n)])
    q = _rnd(n, x.H, x.d).to(x.T)
    _set_q(x, q)
    k, v = _fill_cache(x, 1, p0 + n)
    x.op("window_attn_rows")
    ref = O.window_attention(q.double(), k.double(), v.double(), x.scale, window or 10 ** 9, p0) * x.ls
    _close(x.b["out"][:n, :x.H * x.d].reshape(n, x.H, x.d), ref, x.tol)


@pytest.mark.parametrize("dt,rows_path", [("bf16", True), ("bf16", False), ("f32", False)])
@pytest.mark.parametrize("window", [3, 32, 64, 96, 129])
def test_window_edges_stand_out(dt, rows_path, window):
    """Every query's score with the keys just inside and just outside its window dwarfs all others, and the
    values differ: a window one token off changes the output completely."""
    x = Mix(dt, H=2, G=1, d=64, rot=32, window=window, scale=1.0)
    n = 2 * window + 70
    k = torch.zeros(n, 1, 64)
    v = _rnd(n, 1, 64)
    # key j carries bit pattern j; the query at i matches keys i - window (outside) and i - window + 1 (inside)
    code = torch.sign(_rnd(n + 1, 64, seed=5)) * 0.5
    k[:, 0] = code[:n]
    q = torch.zeros(n, 2, 64)
    for i in range(n):
        q[i, 0] = 2.0 * code[max(0, i - window + 1)]
        q[i, 1] = 2.0 * code[max(0, i - window)]
    q, k, v = q.to(x.T), k.to(x.T), v.to(x.T)
    x.k[0, :n, :, :64], x.v[0, :n, :, :64] = k.cuda(), v.cuda()
    x.rows([(0, 0, n)])
    _set_q(x, q)
    x.op("window_attn_rows" if rows_path else "window_attn_decode")
    got = x.b["out"][:n, :128].reshape(n, 2, 64).double().cpu() / x.ls
    ref = O.window_attention(q.double(), k.double(), v.double(), 1.0, window)
    assert float((got - ref).abs().max()) < (3e-2 if dt == "bf16" else 1e-4)
    # the first query whose far key has just left the window must differ from the one that still sees it
    wrong = O.window_attention(q.double(), k.double(), v.double(), 1.0, window + 1)
    assert float((ref - wrong)[window:, 1].abs().mean()) > 0.1
    inside = O.window_attention(q.double(), k.double(), v.double(), 1.0, max(1, window - 1))
    assert float((ref - inside)[window:, 0].abs().mean()) > 0.1


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("shape", range(len(SHAPES)))
def test_recurrence_step(dt, shape):
    x = Mix(dt, **SHAPES[shape])
    parts = [(1, 5, 3), (0, 0, 1), (2, 9, 4)]
    n = x.rows(parts)
    proj = _rnd(n, x.ld).to(x.T)
    S0, h0 = _rnd(3, x.heads, x.N, x.P, seed=4), _rnd(3, x.taps - 1, x.C, seed=9).to(x.T)
    x.b["proj"][:n] = proj.cuda()
    refs, row = [], 0
    for s, _, cnt in parts:
        refs.append(x.ref_ssd(proj[row:row + cnt], S0[s].double(), h0[s].double()))
        row += cnt
    for fuse, commit in ((1, 0), (1, 1), (0, 1)):
        x.S.copy_(S0); x.hist.copy_(h0)
        x.r.fuse_norm, x.r.commit = fuse, commit
        x.b["out"].fill_(9.0)
        x.op("mix_prepare")
        x.op("ssd_step")
        row = 0
        for (s, _, cnt), (out, S, hist, u, _, _) in zip(parts, refs):
            _close(x.b["ubuf"][row:row + cnt], u, 4e-3 if dt == "bf16" else 2e-5)
            _close(x.b["out"][row:row + cnt, x.H * x.d:x.H * x.d + x.I], out, x.tol)
            _close(x.S[s], S if commit else S0[s], 4e-3 if dt == "bf16" else 2e-5)
            assert torch.equal(x.hist[s].double().cpu(), hist if commit else h0[s].double())
            row += cnt
        assert int(x.b["ssd_counters"].abs().sum()) == 0


@pytest.mark.parametrize("shape", range(len(SHAPES)))
@pytest.mark.parametrize("n", [3, 64, 65, 200])
def test_recurrence_chunked(shape, n):
    x = Mix("bf16", **SHAPES[shape])
    x.rows([(2, 7, n)])
    x.r.fuse_norm = 0
    proj = _rnd(n, x.ld).to(x.T)
    S0, h0 = _rnd(3, x.heads, x.N, x.P, seed=4), _rnd(3, x.taps - 1, x.C, seed=9).to(x.T)
    x.b["proj"][:n] = proj.cuda()
    x.S.copy_(S0); x.hist.copy_(h0)
    x.op("mix_prepare")
    # the recurrence itself from exactly the kernel's inputs: nothing but fp32 rounding may be left
    xbc, dts = x.b["xbc"][:n, :x.C].double().cpu(), x.b["dtb"][:n].double().cpu()
    I, GN = x.I, x.groups * x.N
    y, S = O.ssd_recurrence(xbc[:, :I].reshape(n, x.heads, x.P), xbc[:, I:I + GN].reshape(n, x.groups, x.N),
                            xbc[:, I + GN:].reshape(n, x.groups, x.N), dts, x.A_log, x.D, S0[2].double())
    x.op("ssd_chunk")
    z = proj.double()[:, x.m.off_z:x.m.off_z + I]
    _close(x.b["ubuf"][:n], y.reshape(n, I) * O.silu(z), 1e-5)
    _close(x.S[2], S, 1e-5)
    _close(x.b["out"][:n, x.H * x.d:x.H * x.d + I],
           O.gated_group_norm(y.reshape(n, I), z, x.norm_w.double(), x.ngroups, x.eps) * x.rs, x.tol)
    _, _, hist, _, _, _ = x.ref_ssd(proj, S0[2].double(), h0[2].double())
    assert torch.equal(x.hist[2].double().cpu(), hist)
    assert torch.equal(x.S[0].cpu(), S0[0]) and torch.equal(x.hist[1].cpu(), h0[1])


def test_recurrence_keeps_a_distant_token():
    """Decay close to one: a single large input must still be in the output hundreds of tokens and several
    chunks later."""
    x = Mix("bf16", heads=2, P=16, N=16, groups=1, ngroups=1, taps=2, rows=512)
    x.A_log.fill_(-9.0); x.dev["A_log"].fill_(-9.0)
    n = 500
    x.rows([(0, 0, n)])
    x.r.fuse_norm = 0
    proj = _rnd(n, x.ld, std=0.05).to(x.T)
    proj[3] *= 200
    x.b["proj"][:n] = proj.cuda()
    x.op("mix_prepare"); x.op("ssd_chunk")
    out = x.ref_ssd(proj)[0]
    _close(x.b["out"][:n, x.H * x.d:x.H * x.d + x.I], out, 3e-2)
    other = proj.clone()
    other[3] = 0
    assert float((x.ref_ssd(other)[0] - out)[-50:].abs().mean()) > 0.1
