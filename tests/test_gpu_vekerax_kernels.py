"""Every mechanism of the Vekerax decoder alone: the CUDA kernels against the plain functions of
vekerax_oracle."""
import ctypes as C

import pytest
import torch

import vekerax_oracle as O
from test_gpu_degedra_kernels import DTS, _close, _lin, _rnd

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ projections and streams
def _coef(n, seed=0):
    """(mix, out, in) and the device array of all three"""
    M, b, a = _rnd(n, n, seed=seed + 1), _rnd(n, seed=seed + 2), _rnd(n, seed=seed + 3)
    return M, b, a, torch.cat([M.reshape(-1), b, a]).cuda()


def _ref_streams(x, M, b, a, y):
    """x [rows, n, H] -> (new x, u) in float64"""
    new = O.streams_out(x.double().transpose(0, 1), M.double(), b.double(), 1.0, y.double())
    return new.transpose(0, 1), O.streams_in(new, a.double())


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("mma", [False, True])
@pytest.mark.parametrize("n,H,K,rows", [(1, 90, 40, 1), (2, 256, 300, 2), (3, 168, 64, 8), (4, 1000, 500, 1), (6, 64, 72, 5), (16, 40, 24, 1)])
def test_projection_into_the_streams(dt, mma, n, H, K, rows):
    """The projection that ends a sublayer updates the streams and leaves the next input with its sums of
    squares; the next projection normalises that input itself."""
    from mi50grad_b200.ops import kernels as K_
    from mi50grad_b200.ops import lib as L
    T, _, tol = DTS[dt]
    w, v = _rnd(H, K, std=K ** -0.5).to(T), _rnd(rows, K, seed=1).to(T)
    x = _rnd(rows, n, H, seed=2)
    M, b, a, coef = _coef(n)
    y = v.double() @ w.double().T
    rx, ru = _ref_streams(x, M, b, a, y)
    xs = torch.zeros(rows, -(-K // 8) * 8, dtype=T, device="cuda")
    xs[:, :K] = v
    lin = _lin(w, T, 16)
    xd, u, ss = x.cuda(), torch.zeros(rows, H, device="cuda"), torch.zeros(rows, -(-H // 8), device="cuda")
    K_.gemv_dense(lin, xs[:, :K], None, L.DG_STREAMS, ss_out=ss, mma=mma, sm=K_.stream_mix(xd, u, coef))
    _close(xd, rx, 1e-5)
    _close(u, ru, 1e-5)
    assert torch.allclose(ss.sum(1).double().cpu(), ru.pow(2).sum(1), rtol=1e-4)
    w2, nw, out = _rnd(48, H, seed=7, std=H ** -0.5).to(T), 1 + _rnd(H, seed=4, std=0.2), torch.zeros(rows, 48, device="cuda")
    nd = nw.cuda()
    K_.gemv_dense(_lin(w2, T, 16), None, out, L.DG_STORE_F32, pn=K_.norm_input(u, nd, ss, 1e-5), rows=rows, mma=mma)
    _close(out, (O.rms(ru, 1e-5) * nw.double()).to(T).double() @ w2.double().T, tol)


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("n,H,rows,planes", [(1, 90, 3, 1), (2, 320, 9, 3), (3, 168, 1, 2), (4, 4096, 5, 1), (5, 72, 4, 2), (4, 9000, 2, 1), (2, 2052, 3, 4),
                                             (16, 64, 2, 1)])
def test_stream_rows(dt, n, H, rows, planes):
    from mi50grad_b200.ops import kernels as K_
    T, _, tol = DTS[dt]
    x, y, w = _rnd(rows, n, H), _rnd(planes, rows + 2, H, seed=1), 1 + _rnd(H, seed=2, std=0.3)
    M, b, a, coef = _coef(n)
    wd, yd = w.cuda(), y.cuda()[:, :rows]
    rx, ru = _ref_streams(x, M, b, a, y[:, :rows].sum(0))
    for keep_u in (True, False):
        xd, u = x.cuda(), torch.zeros(rows, H, device="cuda")
        xb = torch.zeros(rows, -(-H // 8) * 8, dtype=T, device="cuda")
        K_.stream_rows(xd, coef, wd, xb, 1e-4, y=yd, u=u if keep_u else None)
        _close(xd, rx, 1e-5)
        _close(xb[:, :H], O.rms(ru, 1e-4) * w.double(), tol)
        if keep_u:
            _close(u, ru, 1e-5)


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("n,H", [(1, 90), (3, 168), (4, 256), (6, 64)])
def test_embedding_into_the_streams(dt, n, H):
    from mi50grad_b200.ops import kernels as K_
    T, _, tol = DTS[dt]
    V, rows, scale = 31, 4, 2.5
    table = torch.zeros(V, -(-H // 8) * 8, dtype=T)
    table[:, :H] = _rnd(V, H).to(T)
    w = 1 + _rnd(H, seed=2, std=0.3)
    M, b, a, coef = _coef(n)
    toks = [5, -1, 30, -1]
    seqs = torch.tensor([[7, 11, 0, 0], [9, 12, 0, 0]], dtype=torch.int32, device="cuda")
    meta = K_.make_rows([(0, 0, 0, 0, 0), (1, 0, 0, 0, 0), (0, 0, 0, 0, 0), (0, 0, 0, 0, 0)], "cuda")
    e = table[[5, 12, 30, 11], :H].double() * scale
    ref = O.rms(e * a.double().sum(), 1e-5) * w.double()
    wd, td = w.cuda(), table.cuda()
    tok = torch.tensor(toks, dtype=torch.int32, device="cuda")
    for from_rows in (False, True):
        x, xb = torch.zeros(rows, n, H, device="cuda"), torch.zeros(rows, -(-H // 8) * 8, dtype=T, device="cuda")
        if from_rows:
            K_.stream_rows(x, coef, wd, xb, 1e-5, h=(e / scale).float().cuda(), scale=scale)
        else:
            K_.stream_rows(x, coef, wd, xb, 1e-5, embed=td, tokens=tok, rows_meta=meta, seqs=seqs, scale=scale)
        _close(x, e[:, None].expand(rows, n, H), 1e-6)
        _close(xb[:, :H], ref, tol)


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("F,K,rows", [(33, 90, 1), (200, 168, 8), (1000, 512, 4)])
def test_relu_gate_pair(dt, F, K, rows):
    from mi50grad_b200.engine.mixer_engine import interleave_dense_gate_up
    from mi50grad_b200.ops import kernels as K_
    from mi50grad_b200.ops import lib as L
    T, _, tol = DTS[dt]
    g, u, x = _rnd(F, K, std=K ** -0.5).to(T), _rnd(F, K, seed=1, std=K ** -0.5).to(T), _rnd(rows, K, seed=2).to(T)
    eye = torch.eye(F, dtype=torch.float64)
    ref = O.relu_mlp({"gate": g.double(), "up": u.double(), "down": eye}, "", x.double())
    both = interleave_dense_gate_up(g, u)
    xs = torch.zeros(rows, -(-K // 8) * 8, dtype=T, device="cuda")
    xs[:, :K] = x
    lin = _lin(both, T, 16)
    out = torch.zeros(rows, -(-F // 8) * 8, dtype=T, device="cuda")
    for mma in (False, True):
        K_.gemv_dense(lin, xs[:, :K], out.fill_(3.0), L.DG_GATE_PAIR, act=L.ACT_RELU, mma=mma)
        _close(out[:, :F], ref, tol)
        assert float(out[:, F:].abs().sum()) == 0
    out.fill_(3.0)
    if dt == "bf16":
        K_.gemm_bf16_tc(lin.w[:, :K], xs[:, :K], out, L.TC_EPI_SILU_PAIR, act=L.ACT_RELU)
    else:
        K_.gemm_f32(lin.w[:, :K], xs[:, :K], out, L.DG_GATE_PAIR, act=L.ACT_RELU)
    _close(out[:, :F], ref, tol)


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("N,K,rows,cols", [(100, 90, 1, 37), (300, 256, 5, 299), (64, 128, 8, 64)])
def test_silu_on_the_first_outputs(dt, N, K, rows, cols):
    from mi50grad_b200.ops import kernels as K_
    from mi50grad_b200.ops import lib as L
    T, _, tol = DTS[dt]
    w, x = _rnd(N, K, std=K ** -0.5).to(T), _rnd(rows, K, seed=1).to(T)
    y = x.double() @ w.double().T
    ref = torch.cat([O.silu(y[:, :cols]), y[:, cols:]], 1)
    xs = torch.zeros(rows, -(-K // 8) * 8, dtype=T, device="cuda")
    xs[:, :K] = x
    lin = _lin(w, T, 16)
    out = torch.zeros(rows, N, dtype=T, device="cuda")
    for mma in (False, True):
        K_.gemv_dense(lin, xs[:, :K], out.zero_(), L.DG_STORE, act_cols=cols, mma=mma)
        _close(out, ref, tol)
    out.zero_()
    if dt == "bf16":
        K_.gemm_bf16_tc(lin.w[:, :K], xs[:, :K], out, L.TC_EPI_STORE_F16, act_cols=cols)
    else:
        K_.gemm_f32(lin.w[:, :K], xs[:, :K], out, act_cols=cols)
    _close(out, ref, tol)


# ------------------------------------------------------------------ attention
class Att:
    """One attention with random tensors, its caches and its work buffers."""

    def __init__(self, dt, H=4, G=2, d=40, e=24, window=11, keep=0, cap=0.0, sink=True, scale=0.3, rot=0, shared_values=False, slots=3,
                 max_seq=512, rows=400, splits=5):
        from mi50grad_b200.ops import lib as L
        self.T, code, self.tol = DTS[dt]
        self.H, self.G, self.d, self.e, self.window, self.keep, self.cap, self.scale, self.rot = H, G, d, e, window, keep, cap, scale, rot
        self.dp, self.vp, self.eps, self.base, self.splits = -(-d // 8) * 8, -(-e // 8) * 8, 1e-5, 300.0, splits
        self.sink = _rnd(H, seed=3) if sink else None
        self.q_norm, self.k_norm = 1 + _rnd(d, seed=1, std=0.2), 1 + _rnd(d, seed=2, std=0.2)
        z = lambda *s, dtype=self.T: torch.zeros(*s, dtype=dtype, device="cuda")
        self.k, self.v = z(slots, max_seq, G, self.dp), z(slots, max_seq, G, self.vp)
        self.dev = [self.q_norm.cuda(), self.k_norm.cuda(), self.sink.cuda() if sink else None]
        m = self.m = L.MixLayer()
        m.H, m.G, m.d, m.dp, m.dv, m.vp, m.window, m.keep_first, m.softcap = H, G, d, self.dp, e, self.vp, window, keep, cap
        m.attn_scale, m.left_scale, m.eps, m.head_norm, m.max_seq, m.exact_weights, m.rot = scale, 1.0, self.eps, 1, max_seq, 1, rot
        m.q_norm, m.k_norm, m.sink = self.dev[0].data_ptr(), self.dev[1].data_ptr(), L.ptr(self.dev[2])
        m.kcache, m.vcache = self.k.data_ptr(), self.v.data_ptr()
        m.off_q, m.off_k, m.off_v = 0, H * d, -1 if shared_values else H * d + G * d
        if rot:
            f = torch.tensor([self.base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
            ang = torch.arange(max_seq, dtype=torch.float64)[:, None] * f[None]
            self.tabs = [torch.cos(ang).float().cuda(), torch.sin(ang).float().cuda()]
            m.cos_tab, m.sin_tab = self.tabs[0].data_ptr(), self.tabs[1].data_ptr()
        self.ld = -(-(H * d + G * d + G * e) // 8) * 8
        self.ldo = -(-(H * e) // 8) * 8
        lib = L.lib()
        m_ = max(self.dp, self.vp)
        self.b = dict(proj=z(rows, self.ld), qbuf=z(rows, H * self.dp), out=z(rows, self.ldo),
                      attn_scratch=z(lib.b2_window_attn_scratch(H, G, m_, rows, splits), dtype=torch.float32),
                      attn_counters=z(lib.b2_window_attn_units(H, G, rows), dtype=torch.int32))
        r = self.r = L.MixRun()
        for n, t in self.b.items():
            setattr(r, n, t.data_ptr())
        r.dt, r.ld_proj, r.ldo, r.splits, r.commit = code, self.ld, self.ldo, splits, 1

    def rows(self, parts):
        """parts: [(slot, first position, count)]"""
        from mi50grad_b200.ops.kernels import make_rows
        ent, sr = [], [0]
        for s, p0, n in parts:
            ent += [(s, p0 + i, p0 + i, p0 + i + 1, 0) for i in range(n)]
            sr.append(sr[-1] + n)
        self.keep_rows = (make_rows(ent, "cuda"), torch.tensor(sr, dtype=torch.int32, device="cuda"))
        self.r.rows, self.r.seq_rows = self.keep_rows[0].data_ptr(), self.keep_rows[1].data_ptr()
        self.r.n_rows, self.r.n_seqs = sr[-1], len(parts)
        return sr[-1]

    def op(self, name):
        from mi50grad_b200.ops.kernels import mix_op
        mix_op(name, self.m, self.r)

    def fill(self, slot, k, v):
        n = k.shape[0]
        self.k[slot, :n, :, :self.d], self.v[slot, :n, :, :self.e] = k.cuda(), v.cuda()

    def set_q(self, q):
        self.b["qbuf"].zero_()
        self.b["qbuf"][:q.shape[0]].reshape(-1, self.H, self.dp)[..., :self.d] = q.cuda()

    def out(self, n):
        return self.b["out"][:n, :self.H * self.e].reshape(n, self.H, self.e)

    def ref(self, q, k, v, p0, **kw):
        a = dict(softcap=self.cap, window=self.window or None, keep=self.keep, sink=self.sink)
        a.update(kw)
        return O.sink_attention(q.double(), k.double(), v.double(), self.scale, q0=p0, **a)


SHAPES = [dict(), dict(H=12, G=1, d=32, e=72), dict(H=3, G=3, d=100, e=100), dict(H=8, G=2, d=64, e=64), dict(H=10, G=2, d=128, e=40),
          dict(H=2, G=1, d=18, e=256), dict(H=2, G=2, d=200, e=20), dict(H=1, G=1, d=8, e=1)]


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("shape", range(len(SHAPES)))
@pytest.mark.parametrize("rot,shared", [(0, False), (8, False), (0, True)])
def test_head_prepare(dt, shape, rot, shared):
    kw = dict(SHAPES[shape])
    if shared:
        kw["e"] = kw.get("d", 40)
    x = Att(dt, rot=rot, shared_values=shared, **kw)
    n = x.rows([(1, 5, 4), (0, 0, 1), (2, 100, 7)])
    proj = _rnd(n, x.ld).to(x.T)
    x.b["proj"][:n] = proj.cuda()
    x.op("head_prepare")
    from degedra_oracle import rotate_half
    row, p = 0, proj.double()
    for slot, p0, c in ((1, 5, 4), (0, 0, 1), (2, 100, 7)):
        pr = p[row:row + c]
        o1, o2 = x.H * x.d, x.H * x.d + x.G * x.d
        q = O.head_norm(pr[:, :o1].reshape(c, x.H, x.d), x.q_norm, x.eps)
        k = O.head_norm(pr[:, o1:o2].reshape(c, x.G, x.d), x.k_norm, x.eps)
        v = pr[:, o1:o2].reshape(c, x.G, x.d) if shared else pr[:, o2:o2 + x.G * x.e].reshape(c, x.G, x.e)
        if rot:
            pos = torch.arange(p0, p0 + c)
            q, k = rotate_half(q, pos, rot, x.base), rotate_half(k, pos, rot, x.base)
        got = x.b["qbuf"][row:row + c].reshape(c, x.H, x.dp)
        _close(got[..., :x.d], q, x.tol)
        assert float(got[..., x.d:].abs().sum()) == 0
        _close(x.k[slot, p0:p0 + c, :, :x.d], k, x.tol)
        assert torch.equal(x.v[slot, p0:p0 + c, :, :x.e].double().cpu(), v)
        assert float(x.v[slot, p0:p0 + c, :, x.e:].abs().sum()) == 0
        row += c


MASKS = [(1, 0), (11, 4), (64, 1), (64, 64), (200, 70), (0, 0), (5, 130)]


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("shape", range(len(SHAPES)))
@pytest.mark.parametrize("window,keep", MASKS)
def test_attention_decode(dt, shape, window, keep):
    x = Att(dt, window=window, keep=keep, cap=3.0 if shape % 2 else 0.0, sink=shape != 3, **SHAPES[shape])
    parts = [(0, 0, 1), (2, 299, 1), (1, 150, 3), (0, 1, 2), (1, window + keep, 2)]
    n = x.rows(parts)
    q = _rnd(n, x.H, x.d).to(x.T)
    x.set_q(q)
    kv = {s: (_rnd(300, x.G, x.d, seed=10 * s).to(x.T), _rnd(300, x.G, x.e, seed=10 * s + 1).to(x.T)) for s in range(3)}
    for s in kv:
        x.fill(s, *kv[s])
    refs, row = [], 0
    for s, p0, c in parts:
        refs.append(x.ref(q[row:row + c], *kv[s], p0))
        row += c
    for splits in (1, x.splits):
        x.r.splits = splits
        x.b["out"].fill_(9.0)
        x.op("window_attn_decode")
        _close(x.out(n), torch.cat(refs), x.tol)
        assert int(x.b["attn_counters"].abs().sum()) == 0
        assert torch.all(x.b["out"][:, x.H * x.e:] == 9.0)


@pytest.mark.parametrize("shape", range(len(SHAPES)))
@pytest.mark.parametrize("p0,n,window,keep", [(0, 16, 11, 4), (0, 130, 1, 0), (37, 100, 64, 65), (191, 65, 63, 3), (5, 200, 0, 0), (128, 64, 65, 64),
                                              (300, 70, 20, 130)])
def test_attention_rows(shape, p0, n, window, keep):
    x = Att("bf16", window=window, keep=keep, cap=0.0 if shape % 2 else 4.0, sink=shape != 3, **SHAPES[shape])
    x.rows([(1, p0, n)])
    q, k, v = _rnd(n, x.H, x.d).to(x.T), _rnd(p0 + n, x.G, x.d, seed=3).to(x.T), _rnd(p0 + n, x.G, x.e, seed=4).to(x.T)
    x.set_q(q)
    x.fill(1, k, v)
    x.op("window_attn_rows")
    ref = x.ref(q, k, v, p0)
    _close(x.out(n), ref, x.tol)
    # weights that keep all their bits against weights rounded to bf16 (both are forms of the kernel)
    a = x.out(n).double().cpu()
    x.m.exact_weights = 0
    x.op("window_attn_rows")
    b = x.out(n).double().cpu()
    assert float((a - ref).pow(2).mean()) <= float((b - ref).pow(2).mean()) * 1.01 + 1e-12


@pytest.mark.parametrize("dt,rows_path", [("bf16", True), ("bf16", False), ("f32", False)])
@pytest.mark.parametrize("window,keep", [(3, 1), (32, 4), (64, 63), (96, 65), (20, 128)])
def test_edges_of_the_mask_stand_out(dt, rows_path, window, keep):
    """Four query heads whose score with one key dwarfs all others: the key just inside the window, the one just
    outside, the last kept one and the first that is not kept.  A mask one token off changes the output."""
    x = Att(dt, H=4, G=1, d=64, e=32, window=window, keep=keep, scale=1.0, sink=False)
    n = 2 * window + keep + 70
    code = torch.sign(_rnd(n, 64, seed=5)) * 0.5
    k, v = code[:, None].clone(), _rnd(n, 1, 32)
    q = torch.zeros(n, 4, 64)
    for i in range(n):
        for h, j in enumerate((max(0, i - window + 1), max(0, i - window), keep - 1, keep)):
            q[i, h] = 2.0 * code[j]
    q, k, v = q.to(x.T), k.to(x.T), v.to(x.T)
    x.fill(0, k, v)
    x.rows([(0, 0, n)])
    x.set_q(q)
    x.op("window_attn_rows" if rows_path else "window_attn_decode")
    got = x.out(n).double().cpu()
    ref = x.ref(q, k, v, 0)
    assert float((got - ref).abs().max()) < (3e-2 if dt == "bf16" else 1e-4)
    far = slice(window + keep + 1, None)
    for h, wrong in ((0, dict(window=window - 1)), (1, dict(window=window + 1)), (2, dict(keep=keep - 1)), (3, dict(keep=keep + 1))):
        assert float((ref - x.ref(q, k, v, 0, **wrong))[far, h].abs().mean()) > 0.1


@pytest.mark.parametrize("dt,rows_path", [("bf16", True), ("bf16", False), ("f32", False)])
def test_sink_and_cap_stand_out(dt, rows_path):
    """Sinks from negligible to dominant, scores far beyond the cap."""
    x = Att(dt, H=4, G=1, d=16, e=16, window=40, keep=2, cap=5.0, scale=1.0)
    x.sink.copy_(torch.tensor([-20.0, 0.0, 4.0, 9.0]))
    x.dev[2].copy_(x.sink)
    n = 100
    q, k, v = (3 * _rnd(n, 4, 16)).to(x.T), (2 * _rnd(n, 1, 16, seed=1)).to(x.T), _rnd(n, 1, 16, seed=2).to(x.T)
    x.fill(0, k, v)
    x.rows([(0, 0, n)])
    x.set_q(q)
    for splits in (1, 5):
        x.r.splits = splits
        x.op("window_attn_rows" if rows_path else "window_attn_decode")
        ref = x.ref(q, k, v, 0)
        assert float((x.out(n).double().cpu() - ref).abs().max()) < (2e-2 if dt == "bf16" else 2e-5)
    for wrong, heads in ((dict(sink=None), (2, 3)), (dict(sink=x.sink * x.scale / 5), (3,)), (dict(softcap=None), (0, 1, 2, 3))):
        for h in heads:
            assert float((ref - x.ref(q, k, v, 0, **wrong))[:, h].abs().mean()) > 0.02


# ------------------------------------------------------------------ lightning attention
class Rec:
    def __init__(self, dt, heads=6, N=24, P=20, decay=None, slots=3, rows=520):
        from mi50grad_b200.engine.vekerax_engine import LOG_ZERO
        from mi50grad_b200.ops import lib as L
        import math
        self.T, code, self.tol = DTS[dt]
        self.heads, self.N, self.P, self.I, self.eps = heads, N, P, heads * P, 1e-5
        self.decay = list(decay) if decay else [1.0, 0.0, 0.5, 0.9, 0.99, 0.999, 0.3, 0.97][:heads]
        assert len(self.decay) == heads
        z = lambda *s, dtype=self.T: torch.zeros(*s, dtype=dtype, device="cuda")
        self.nw = 1 + _rnd(self.I, seed=1, std=0.2)
        self.S = z(slots, heads, N, P, dtype=torch.float32)
        self.dev = [torch.tensor(self.decay).cuda(), torch.tensor([math.log(d) if d else LOG_ZERO for d in self.decay]).cuda(), self.nw.cuda()]
        m = self.m = L.MixLayer()
        m.heads, m.P, m.N, m.groups, m.ngroups, m.taps, m.right_scale, m.eps, m.gate = heads, P, N, heads, 1, 1, 1.0, self.eps, L.REC_NORM_SIGMOID
        m.decay, m.log_decay, m.norm_w, m.state = *(t.data_ptr() for t in self.dev), self.S.data_ptr()
        m.rC, m.rB, m.rx, m.off_z = 0, heads * N, 2 * heads * N, 2 * heads * N + self.I
        self.ld = -(-(2 * heads * N + 2 * self.I) // 8) * 8
        lib = L.lib()
        self.b = dict(proj=z(rows, self.ld), ubuf=z(rows, self.I, dtype=torch.float32), out=z(rows, -(-self.I // 8) * 8),
                      ssd_counters=z(lib.b2_ssd_units(C.byref(m), rows), dtype=torch.int32),
                      chunk_state=z(lib.b2_ssd_chunk_state_floats(C.byref(m), rows), dtype=torch.float32),
                      chunk_prev=torch.zeros(lib.b2_ssd_chunk_prev_bytes(C.byref(m), rows), dtype=torch.uint8, device="cuda"),
                      chunk_decay=z(-(-rows // 64) * heads, dtype=torch.float32))
        r = self.r = L.MixRun()
        for n, t in self.b.items():
            setattr(r, n, t.data_ptr())
        r.dt, r.ld_proj, r.ld_u, r.ldo, r.commit = code, self.ld, self.I, self.b["out"].shape[1], 1
        r.xbc, r.ld_xbc = r.proj, r.ld_proj

    rows, op = Att.rows, Att.op

    def ref(self, proj, S=None):
        """-> (output, state, o before the norm) from projection rows whose q, k, v already have their SiLU"""
        p, n, a = proj.double(), proj.shape[0], self.heads * self.N
        S = torch.zeros(self.heads, self.N, self.P, dtype=torch.float64) if S is None else S.double()
        cut = lambda o, w: p[:, o:o + self.heads * w].reshape(n, self.heads, w)
        o, S = O.decayed_outer_recurrence(cut(0, self.N), cut(a, self.N), cut(2 * a, self.P), torch.tensor(self.decay).double(), S)
        o = o.reshape(n, self.I)
        return O.norm_then_gate(o, p[:, self.m.off_z:self.m.off_z + self.I], self.nw, self.eps), S, o


REC_SHAPES = [dict(), dict(heads=5, N=17, P=33), dict(heads=2, N=130, P=72), dict(heads=8, N=128, P=64), dict(heads=1, N=256, P=128),
              dict(heads=3, N=8, P=9)]


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("shape", range(len(REC_SHAPES)))
def test_lightning_step(dt, shape):
    x = Rec(dt, **REC_SHAPES[shape])
    parts = [(1, 5, 3), (0, 0, 1), (2, 9, 4)]
    n = x.rows(parts)
    proj, S0 = _rnd(n, x.ld).to(x.T), _rnd(3, x.heads, x.N, x.P, seed=4)
    x.b["proj"][:n] = proj.cuda()
    for fuse, commit in ((1, 0), (1, 1), (0, 1)):
        x.S.copy_(S0)
        x.r.fuse_norm, x.r.commit = fuse, commit
        x.op("ssd_step")
        row = 0
        for s, _, c in parts:
            out, S, o = x.ref(proj[row:row + c], S0[s])
            _close(x.b["ubuf"][row:row + c], o, 2e-5)
            _close(x.b["out"][row:row + c, :x.I], out, x.tol)
            _close(x.S[s], S if commit else S0[s], 2e-5)
            row += c
        assert int(x.b["ssd_counters"].abs().sum()) == 0


@pytest.mark.parametrize("shape", range(len(REC_SHAPES)))
@pytest.mark.parametrize("n", [3, 64, 65, 200])
def test_lightning_chunked(shape, n):
    x = Rec("bf16", **REC_SHAPES[shape])
    x.rows([(2, 7, n)])
    proj, S0 = _rnd(n, x.ld).to(x.T), _rnd(3, x.heads, x.N, x.P, seed=4)
    x.b["proj"][:n] = proj.cuda()
    x.S.copy_(S0)
    x.op("ssd_chunk")
    out, S, o = x.ref(proj, S0[2])
    _close(x.b["ubuf"][:n], o, 1e-5)
    _close(x.S[2], S, 1e-5)
    _close(x.b["out"][:n, :x.I], out, x.tol)
    assert torch.equal(x.S[0].cpu(), S0[0])


def test_lightning_keeps_a_distant_token():
    """Decay close to one: a single large input must still be in the output several chunks later."""
    x = Rec("bf16", heads=2, N=16, P=16, decay=(0.9995, 1.0))
    n = 500
    x.rows([(0, 0, n)])
    proj = _rnd(n, x.ld, std=0.05).to(x.T)
    proj[3] *= 200
    proj[:, x.m.rC:x.m.rC + 32] += proj[3, x.m.rB:x.m.rB + 32] * 0.05
    x.b["proj"][:n] = proj.cuda()
    x.op("ssd_chunk")
    out = x.ref(proj)[0]
    _close(x.b["out"][:n, :x.I], out, 2e-2)
    other = proj.clone()
    other[3, x.m.rx:x.m.rx + 32] = 0
    assert float((x.ref(other)[0] - out)[-50:].abs().mean()) > 0.1
