"""The kernels of the Zidepel model one mechanism at a time, through the C ABI, against the plain float64 restatement
(oracle/hybrid_oracle.py). fp32: a few units of fp32 rounding. bfloat16: inputs are given bfloat16 values where a kernel
stores or multiplies them in that type, so that only what it rounds itself is compared at bfloat16's rounding."""
import ctypes as C

import numpy as np
import pytest

import _hybrid as T

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
o = T.o

BF16, F32 = 2, 3
TYPES = [pytest.param(BF16, id="bf16"), pytest.param(F32, id="f32")]


def up8(n):
    return (n + 7) // 8 * 8


def rng(seed):
    return np.random.default_rng(seed)


def dev(a):
    return torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).cuda()


def zeros(*shape, dtype=torch.float32):
    return torch.zeros(*shape, dtype=dtype, device="cuda")


def ttype(wtype):
    return torch.bfloat16 if wtype == BF16 else torch.float32


def host(t):
    torch.cuda.synchronize()
    return t.float().cpu().numpy().astype(np.float64)


def padded(v, n):
    return np.concatenate([v, np.zeros(v.shape[:-1] + (n - v.shape[-1],))], axis=-1)


def close(got, want, tol, size=None):
    err = np.abs(got - want).max() / (size or np.abs(want).max())
    assert err <= tol, err


def connect(g, n):
    c = {"mix": g.standard_normal((n, n)), "out": g.standard_normal(n), "in": g.standard_normal(n)}
    return c, dev(np.concatenate([c["mix"].ravel(), c["out"], c["in"]]))


# ------------------------------------------------------------------ one token: products

def pack(lib, w, wtype, cols):
    stride = lib.b200_packed_row_stride(wtype, cols)
    d = zeros(w.shape[0], stride, dtype=torch.uint8)
    src = dev(w)
    assert lib.b200_cast_pack(wtype, src.data_ptr(), w.shape[1], w.shape[0], w.shape[1], d.data_ptr(), stride, 0, 1, None) == 0
    torch.cuda.synchronize()
    return d, stride


def matvec(lib, pkg, w, wtype, **kw):
    cols = up8(w.shape[1])
    d, stride = pack(lib, w, wtype, cols)
    a = pkg.MatvecArgs()
    a.d_w, a.row_stride, a.rows, a.cols, a.wtype, a.n_out = d.data_ptr(), stride, w.shape[0], cols, wtype, 1
    for k, v in kw.items():
        if k == "d_out":
            a.d_out[0] = v.data_ptr()
        else:
            setattr(a, k, v.data_ptr() if isinstance(v, torch.Tensor) else v)
    rc = lib.b200_matvec(C.byref(a), None)
    torch.cuda.synchronize()
    return rc


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("dim", [5, 64, 101, 320, 2560, 3001, 5120])
def test_layer_norm_input(lib, pkg, wtype, dim):
    g, n = rng(1), up8(dim)
    w, x, gamma, beta, out = o.bf16(g.standard_normal((40, dim))), g.standard_normal(dim) * 3 + 11, g.standard_normal(dim), g.standard_normal(dim), zeros(40)
    assert matvec(lib, pkg, w, wtype, d_in_vec=dev(padded(x, n)), d_norm_gamma=dev(padded(gamma, n)), d_norm_beta=dev(padded(beta, n)), norm_dim=dim,
                  eps=1e-3, d_out=out) == 0
    close(host(out), w @ o.layer_norm(x.astype(np.float32).astype(float), gamma, beta, 1e-3), 4e-6)


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("dim", [24, 101, 2048, 4104])
def test_first_reader(lib, pkg, wtype, dim):
    """Embedding row plus position row, their norm kept, then what the first sublayer reads."""
    g, n, pos = rng(2), up8(dim), 6
    w, emb, ptab = o.bf16(g.standard_normal((33, dim))), g.standard_normal((9, dim)), g.standard_normal((7, dim))
    ew, eb, nw, nb = (g.standard_normal(dim) for _ in range(4))
    toks, take, x0, out = [1, 8, 3, 0, 2, 2, 5, 7], -1.3, zeros(n), zeros(33)
    assert matvec(lib, pkg, w, wtype, in_mode=pkg.B200_IN_EMBED, d_emb=dev(padded(emb, n)), emb_rows=9, emb_scale=1.0,
                  d_tokens=torch.tensor(toks, dtype=torch.int32, device="cuda"), d_pos=torch.tensor([pos], dtype=torch.int32, device="cuda"),
                  d_emb_pos=dev(padded(ptab, n)), emb_pos_rows=7, d_slot_norm_gamma=dev(padded(ew, n)), d_slot_norm_beta=dev(padded(eb, n)),
                  d_resid_out=x0, d_mix_coef=dev(np.array([take])), d_norm_gamma=dev(padded(nw, n)), d_norm_beta=dev(padded(nb, n)), norm_dim=dim, eps=1e-4,
                  d_out=out) == 0
    x = o.embedding([0] * pos + [toks[pos]], emb, ptab, ew, eb, 1e-4)[pos]
    close(host(x0), padded(x, n), 2e-6)
    close(host(out), w @ o.layer_norm(take * x, nw, nb, 1e-4), 6e-6)


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("n,rows,cols,same", [(1, 40, 64, False), (2, 101, 72, False), (3, 9, 8, True), (4, 256, 2560, False), (5, 33, 512, False), (7, 640, 100, False),
                                              (8, 2048, 5000, False), (8, 3, 9000, True)])
def test_product_joins_the_streams(lib, pkg, wtype, n, rows, cols, same):
    """Rows of every length, i.e. one to eight rows at a time in the kernel."""
    g, D = rng(3), up8(rows)
    w, x, c = o.bf16(g.standard_normal((rows, cols))), g.standard_normal(cols), connect(g, n)
    old = g.standard_normal((1 if same else n, rows))
    new, u = zeros(n, D), zeros(D)
    assert matvec(lib, pkg, w, wtype, d_in_vec=dev(padded(x, up8(cols))), out_mode=pkg.B200_OUT_STREAMS, d_out=u, d_streams_in=dev(padded(old, D)),
                  streams_in_stride=0 if same else D, d_streams_out=new, streams_out_stride=D, d_connect=c[1], n_streams=n) == 0
    want = o.connect((np.repeat(old, n, axis=0) if same else old)[:, None], c[0], lambda u: u, lambda u: (w @ x)[None])[:, 0]
    close(host(new)[:, :rows], want, 4e-6)
    close(host(u)[:rows], c[0]["in"] @ want, 6e-6)
    assert not host(new)[:, rows:].any() and not host(u)[rows:].any()


@pytest.mark.parametrize("wtype", TYPES)
def test_squared_relu_of_a_product(lib, pkg, wtype):
    g = rng(4)
    w, x, out = o.bf16(g.standard_normal((77, 136))), g.standard_normal(136), zeros(77)
    assert matvec(lib, pkg, w, wtype, d_in_vec=dev(x), act=pkg.B200_ACT_RELU2, d_out=out) == 0
    close(host(out), np.maximum(w @ x, 0) ** 2, 4e-6)


def test_parts_of_two_families_are_refused(lib, pkg):
    w, x, out, v = np.ones((8, 8)), zeros(8), zeros(8), zeros(8)
    base = dict(d_in_vec=x, d_out=out)
    streams = dict(base, out_mode=pkg.B200_OUT_STREAMS, d_streams_in=v, streams_in_stride=8, d_streams_out=zeros(9, 8), streams_out_stride=8, d_connect=zeros(99))
    for bad in (dict(streams, n_streams=0), dict(streams, n_streams=9), dict(streams, n_streams=2, d_connect=None), dict(base, d_norm_beta=v),
                dict(base, d_norm_gamma=v, d_norm_beta=v, norm_groups=2), dict(base, d_slot_norm_gamma=v, d_slot_norm_beta=v), dict(base, d_emb_pos=v, emb_pos_rows=1),
                dict(base, d_norm_gamma=v, d_norm_beta=v, softcap=3.0), dict(streams, n_streams=1, d_norm_gamma=v)):
        assert matvec(lib, pkg, w, BF16, **bad) < 0, bad
    a = pkg.MatvecArgs()                                              # binary16 weights
    a.d_w, a.row_stride, a.rows, a.cols, a.wtype, a.n_out = zeros(64).data_ptr(), 16, 8, 8, 1, 1
    a.d_in_vec, a.d_norm_gamma, a.d_norm_beta, a.d_out[0] = x.data_ptr(), v.data_ptr(), v.data_ptr(), out.data_ptr()
    assert lib.b200_matvec(C.byref(a), None) < 0


# ------------------------------------------------------------------ rows: streams, norms, products

@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("n,dim,rows", [(1, 24, 3), (3, 101, 70), (4, 2048, 9), (8, 1032, 5)])
def test_rows_join_the_streams(lib, pkg, wtype, n, dim, rows):
    g, ld = rng(5), up8(dim)
    c = connect(g, n)
    for same in (False, True):
        old, y, gamma, beta = g.standard_normal((1 if same else n, rows, dim)), g.standard_normal((rows, dim)), g.standard_normal(dim), g.standard_normal(dim)
        new, u, out = zeros(n, rows, ld), zeros(rows, ld), zeros(rows, ld, dtype=ttype(wtype))
        keep = [dev(padded(old, ld)), dev(padded(y, ld + 8)), dev(padded(gamma, ld)), dev(padded(beta, ld))]
        a = pkg.RowsStreamsArgs()
        a.streams_in, a.streams_in_stride, a.y, a.y_ld, a.connect, a.n_streams = keep[0].data_ptr(), 0 if same else rows * ld, keep[1].data_ptr(), ld + 8, c[1].data_ptr(), n
        a.gamma, a.beta, a.eps, a.rows, a.dim, a.ld, a.wtype = keep[2].data_ptr(), keep[3].data_ptr(), 1e-3, rows, dim, ld, wtype
        a.streams_out, a.streams_out_stride, a.u_out, a.out = new.data_ptr(), rows * ld, u.data_ptr(), out.data_ptr()
        assert lib.b200_rows_streams(C.byref(a), None) == 0
        want = o.connect(np.repeat(old, n, axis=0) if same else old, c[0], lambda x: x, lambda x: y)
        wu = np.tensordot(c[0]["in"], want, axes=(0, 0))
        close(host(new)[..., :dim], want, 2e-6)
        close(host(u)[:, :dim], wu, 4e-6)
        close(host(out), padded(o.layer_norm(wu, gamma, beta, 1e-3), ld), 5e-3 if wtype == BF16 else 2e-5)
        a.out, a.streams_out, new2 = None, None, host(new)
        assert lib.b200_rows_streams(C.byref(a), None) == 0 and np.array_equal(host(new), new2)
        a.n_streams = 9
        assert lib.b200_rows_streams(C.byref(a), None) < 0


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("dim", [24, 101, 2048])
def test_rows_start_and_end(lib, pkg, wtype, dim):
    g, ld, rows, pos0 = rng(6), up8(dim), 12, 5
    emb, ptab = g.standard_normal((31, dim)), g.standard_normal((17, dim))
    v = [g.standard_normal(dim) for _ in range(4)]
    toks, take = g.integers(0, 31, rows), 0.8
    x, out = zeros(rows, ld), zeros(rows, ld, dtype=ttype(wtype))
    keep = [dev(padded(emb, ld)), dev(padded(ptab, ld)), torch.from_numpy(toks.astype(np.int32)).cuda(), dev(np.array([take]))] + [dev(padded(k, ld)) for k in v]
    a = pkg.RowsStartArgs()
    a.emb, a.emb_pos, a.tokens, a.vocab, a.pos_rows, a.pos0 = keep[0].data_ptr(), keep[1].data_ptr(), keep[2].data_ptr(), 31, 17, pos0
    a.take, a.emb_gamma, a.emb_beta, a.gamma, a.beta = (k.data_ptr() for k in keep[3:])
    a.eps, a.rows, a.dim, a.ld, a.wtype, a.x, a.out = 1e-4, rows, dim, ld, wtype, x.data_ptr(), out.data_ptr()
    assert lib.b200_rows_start(C.byref(a), None) == 0
    want = o.layer_norm(emb[toks] + ptab[pos0:pos0 + rows], v[0], v[1], 1e-4)
    close(host(x), padded(want, ld), 3e-6)
    close(host(out), padded(o.layer_norm(take * want, v[2], v[3], 1e-4), ld), 5e-3 if wtype == BF16 else 2e-5)
    index = torch.tensor([11, 0, 7], dtype=torch.int32, device="cuda")
    last = zeros(3, ld, dtype=ttype(wtype))
    assert lib.b200_rows_layer_norm(x.data_ptr(), index.data_ptr(), 3, dim, ld, 1e-2, keep[6].data_ptr(), keep[7].data_ptr(), wtype, last.data_ptr(), None) == 0
    close(host(last), padded(o.layer_norm(host(x)[[11, 0, 7], :dim], v[2], v[3], 1e-2), ld), 5e-3 if wtype == BF16 else 2e-5)


@pytest.mark.parametrize("M,N,K", [(3, 64, 24), (130, 200, 72), (300, 1032, 256)])
def test_squared_relu_of_row_products(lib, pkg, M, N, K):
    g = rng(7)
    a, b = o.bf16(g.standard_normal((M, K))), o.bf16(g.standard_normal((N, K)))
    want = np.maximum(a @ b.T, 0) ** 2
    for fn, t in ((lib.b200_gemm_bf16, torch.bfloat16), (lib.b200_gemm_f32, torch.float32)):
        da, db, out = dev(a).to(t), dev(b).to(t), zeros(M, N, dtype=t)
        p = pkg.GemmArgs()
        p.A, p.a_row, p.a_col, p.B, p.b_row, p.b_col, p.M, p.N, p.K, p.alpha, p.relu2 = da.data_ptr(), K, 1, db.data_ptr(), 1, K, M, N, K, 1.0, 1
        if t == torch.bfloat16:
            p.Ch, p.ldch = out.data_ptr(), N
        else:
            p.C, p.ldc = out.data_ptr(), N
        assert fn(C.byref(p), None) == 0
        close(host(out), want, 5e-3 if t == torch.bfloat16 else 1e-5)
    f = zeros(M, N)
    p.C, p.ldc, p.Ch = f.data_ptr(), N, None
    p.A, p.B = dev(a).bfloat16().data_ptr(), dev(b).bfloat16().data_ptr()
    assert lib.b200_gemm_bf16(C.byref(p), None) < 0                   # an fp32 result keeps its sign


# ------------------------------------------------------------------ attention

_soil = None


def soil(lib, pkg):
    """Leaves NaN in the shared memory of every SM: a kernel that reads what it has not written shows it."""
    global _soil
    if _soil is None:
        w = torch.full((2368, 3072), float("nan"), device="cuda")
        a = pkg.MatvecArgs()
        keep = [w, zeros(3072), zeros(2368)]
        a.d_w, a.row_stride, a.rows, a.cols, a.wtype, a.n_out, a.d_in_vec = w.data_ptr(), 3072 * 4, 2368, 3072, F32, 1, keep[1].data_ptr()
        a.d_out[0] = keep[2].data_ptr()
        _soil = (a, keep)
    assert lib.b200_matvec(C.byref(_soil[0]), None) == 0


class Attn:
    """Projections of n tokens, and a kernel state that has not seen any of them. Cache rows not written yet hold NaN."""

    def __init__(self, lib, pkg, wtype, H, G, d, dv, n, cap, temp, seed, max_seq=None, far=None, eps=1e-3):
        self.lib, self.pkg, self.wtype, self.n, self.H, self.G, self.d, self.dv = lib, pkg, wtype, n, H, G, d, dv
        g, self.scale, self.cap, self.max_seq = rng(seed), 0.9 * d ** -0.5, cap, max_seq or n
        q, k, v = g.standard_normal((n, H, d)), g.standard_normal((n, G, d)), g.standard_normal((n, G, dv))
        if far:                                                       # (query position, key position): that key outweighs the rest
            for i, j in far:
                q[i] = np.repeat(k[j], H // G, axis=0)
                v[j] *= 5.0
        self.gq, self.gk = 1.8 + 0.3 * g.standard_normal(d), 1.8 + 0.3 * g.standard_normal(d)
        self.temp = temp
        f = o.query_temperature(self.max_seq, temp)
        self.want = o.attend(o.rms_norm(q, self.gq, eps) * f[:n, None, None], o.rms_norm(k, self.gk, eps), v, self.scale, cap)
        self.size = np.abs(self.want).max()
        self.ld = H * d + G * d + G * dv + 3                          # rows that start anywhere
        self.proj = dev(np.concatenate([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1), np.full((n, 3), np.nan)], axis=1))
        self.keep = [dev(self.gq), dev(self.gk), dev(f)]
        self.kc = torch.full((G, self.max_seq, up8(d)), float("nan"), dtype=ttype(wtype), device="cuda")
        self.vc = torch.full((G, self.max_seq, up8(dv)), float("nan"), dtype=ttype(wtype), device="cuda")
        self.splits = lib.b200_gqa_splits(wtype, H, G, d, dv, self.max_seq)
        self.part, self.out = torch.full((H * self.splits * (up8(dv) + 8),), float("nan"), device="cuda"), zeros(H * dv)
        self.tickets, self.pos = zeros(H * G, dtype=torch.int32), zeros(1, dtype=torch.int32)
        a = self.a = pkg.GqaArgs()
        a.wtype, a.heads, a.kv_heads, a.dim, a.vdim, a.max_seq, a.scale, a.softcap, a.eps = wtype, H, G, d, dv, self.max_seq, self.scale, cap or 0.0, eps
        a.d_q_gamma, a.d_k_gamma, a.d_q_scale = (t.data_ptr() for t in self.keep)
        if not temp:
            a.d_q_scale = None
        a.d_k_cache, a.d_v_cache, a.d_part, a.d_tickets, a.d_out, a.d_pos = (t.data_ptr() for t in (self.kc, self.vc, self.part, self.tickets, self.out, self.pos))
        a.n_split = self.splits

    def at(self, row):
        base = self.proj.data_ptr() + 4 * row * self.ld
        self.a.d_q, self.a.d_k, self.a.d_v = base, base + 4 * self.H * self.d, base + 4 * (self.H + self.G) * self.d

    def rows(self, pos0, m):
        a, H, dv = self.a, self.H, self.dv
        self.at(pos0)
        q = torch.full((m, H, up8(self.d)), float("nan"), dtype=ttype(self.wtype), device="cuda")
        out = zeros(m, H * dv + 5, dtype=ttype(self.wtype))
        a.n_rows, a.pos0, a.proj_ld, a.d_q_rows, a.d_out_rows, a.out_ld = m, pos0, self.ld, q.data_ptr(), out.data_ptr(), H * dv + 5
        assert self.lib.b200_gqa_rows_prep(C.byref(a), None) == 0
        soil(self.lib, self.pkg)
        assert self.lib.b200_gqa_rows_attend(C.byref(a), None) == 0
        got = host(out)
        assert not got[:, H * dv:].any()
        return got[:, :H * dv].reshape(m, H, dv)

    def one(self, pos):
        self.at(pos)
        self.pos.fill_(pos)
        self.out.fill_(float("nan"))
        soil(self.lib, self.pkg)
        assert self.lib.b200_gqa_decode(C.byref(self.a), None) == 0
        got = host(self.out).reshape(self.H, self.dv)
        assert not host(self.tickets).any()
        return got


SHAPES = [(4, 2, 24, 16), (5, 1, 33, 41), (2, 2, 128, 128), (12, 2, 160, 264), (9, 3, 4, 72), (1, 1, 2, 1), (16, 4, 80, 112), (2, 1, 256, 64), (3, 1, 300, 500)]


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("H,G,d,dv", SHAPES)
def test_attention_rows_then_single_tokens(lib, pkg, wtype, H, G, d, dv):
    """Portions down to two tokens, then one by one: every way leaves the same cache. One key far back outweighs the rest,
    for queries in a portion, in a later portion and alone, with keys at the borders of tiles and splits."""
    n, far = 340, [(140, 3), (150, 64), (151, 63), (220, 0), (300, 127), (301, 128), (330, 5), (331, 191), (332, 192), (333, 332), (339, 0)]
    t = Attn(lib, pkg, wtype, H, G, d, dv, n, 20.0, {"coef": 0.4, "every": 7}, 11, far=far)
    tol = 2e-2 if wtype == BF16 else 2e-5
    at = 0
    for m in (1, 2, 13, 130, 64, 2, 88):
        got = t.rows(at, m) if m > 1 else t.one(at)[None]
        close(got, t.want[at:at + m], tol, t.size)
        at += m
    assert at == 300
    for i in range(at, n):
        close(t.one(i)[None], t.want[i:i + 1], tol, t.size)
    assert torch.isfinite(t.kc).all() and torch.isfinite(t.vc).all()
    assert not host(t.kc)[..., d:].any() and not host(t.vc)[..., dv:].any()


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("cap,temp", [(None, None), (3.0, None), (None, {"coef": 0.3, "every": 1}), (40.0, {"coef": -0.1, "every": 2.5})])
def test_attention_options(lib, pkg, wtype, cap, temp):
    t = Attn(lib, pkg, wtype, 6, 3, 40, 24, 100, cap, temp, 12)
    tol = 2e-2 if wtype == BF16 else 2e-5
    close(t.rows(0, 70), t.want[:70], tol, t.size)
    for i in range(70, 75):
        close(t.one(i)[None], t.want[i:i + 1], tol, t.size)


@pytest.mark.parametrize("wtype", TYPES)
def test_attention_over_clusters_of_blocks(lib, pkg, wtype):
    """Positions around every border of the decode kernel's shares of a long sequence (a block's, a cluster's), a far key each."""
    n, lone = 4200, [2047, 2048, 2049, 2050, 2303, 2304, 3000, 4095, 4096, 4097, 4098, 4199]
    t = Attn(lib, pkg, wtype, 2, 2, 64, 32, n, 28.0, {"coef": 0.25, "every": 300}, 13, far=[(i, (i * 37) % (i - 1)) for i in lone])
    assert t.splits == 2
    got = t.rows(0, n)
    tol = 2e-2 if wtype == BF16 else 3e-5
    close(got, t.want, tol, t.size)
    for i in [0, 1, 7, 8, 9, 15, 16, 17, 62, 63, 64, 65, 127, 128, 129, 511, 512, 513, 1000] + lone:
        close(t.one(i)[None], t.want[i:i + 1], tol, t.size)
    one = [t.one(4199) for _ in range(3)]
    assert np.array_equal(one[0], one[1]) and np.array_equal(one[0], one[2])


def test_attention_ignores_positions_outside_the_cache(lib, pkg):
    t = Attn(lib, pkg, F32, 4, 2, 24, 16, 20, None, None, 14)
    t.rows(0, 20)
    before = host(t.kc)
    for pos in (-1, 20, 1 << 20):
        t.at(0)
        t.pos.fill_(pos)
        t.out.fill_(7.0)
        assert lib.b200_gqa_decode(C.byref(t.a), None) == 0
        assert (host(t.out) == 7.0).all() and np.array_equal(host(t.kc), before)
    t.a.n_split = 0
    assert lib.b200_gqa_decode(C.byref(t.a), None) < 0
    t.a.kv_heads = 3
    assert lib.b200_gqa_rows_prep(C.byref(t.a), None) < 0


# ------------------------------------------------------------------ linear attention

class Gla:
    def __init__(self, lib, pkg, H, d, dv, rank, tau, n, seed, slots=3, bias=(2.0, 2.0), wtype=F32, eps=1e-4):
        g = rng(seed)
        self.lib, self.pkg, self.H, self.dv, self.n, self.wtype, self.slots, self.d = lib, pkg, H, dv, n, wtype, slots, d
        q, k, v, gate, f = (g.standard_normal((n, s)) for s in (H * d, H * d, H * dv, H * dv, rank))
        a2, b, gamma = g.standard_normal((H * d, rank)) * rank ** -0.5, bias[0] + bias[1] * g.standard_normal(H * d), 1 + 0.3 * g.standard_normal(dv)
        a = o.decay(f @ a2.T + b, tau).reshape(n, H, d)
        qs = q.reshape(n, H, d) * d ** -0.5
        runs = [o.recurrence(qs[:, h], k.reshape(n, H, d)[:, h], v.reshape(n, H, dv)[:, h], a[:, h]) for h in range(H)]
        self.state = np.stack([r[1] for r in runs])
        self.want = o.rms_norm(np.stack([r[0] for r in runs], axis=1), gamma, eps).reshape(n, -1) * o.silu(gate)
        self.size = np.abs(self.want).max()
        r8 = up8(rank)
        self.sections = np.cumsum([0, up8(H * d), up8(H * d), up8(H * dv), up8(H * dv), r8])
        self.ld = int(self.sections[-1])
        self.proj = dev(np.concatenate([padded(x, up8(x.shape[1])) for x in (q, k, v, gate, f)], axis=1))
        R4 = (rank + 3) // 4 * 4
        nc = (n + 63) // 64
        self.keep = [dev(padded(a2, R4)), dev(b), dev(gamma)]
        nan = lambda *s: torch.full(s, float("nan"), device="cuda")
        self.st, self.out, self.pos = nan(slots, H, d, up8(dv)), zeros(H * dv), zeros(1, dtype=torch.int32)
        planes = lambda *s: nan(nc, H, 3, *s).bfloat16()
        d16 = (d + 15) // 16 * 16
        self.scratch = [planes(64, d16), planes(64, d16), planes(64, up8(dv)), planes(64, 64), planes(d, up8(dv)), nan(nc, H, up8(d)), nan(n, H * dv)]
        p = self.p = pkg.GlaArgs()
        p.wtype, p.heads, p.dim, p.vdim, p.rank, p.n_slots, p.tau, p.q_scale, p.eps = wtype, H, d, dv, rank, slots, tau, d ** -0.5, eps
        p.d_a2, p.d_a2_bias, p.d_norm_gamma = (t.data_ptr() for t in self.keep)
        p.d_state, p.d_out, p.d_pos = self.st.data_ptr(), self.out.data_ptr(), self.pos.data_ptr()
        p.d_qd, p.d_kd, p.d_values, p.d_scores, p.d_chunk_state, p.d_decay, p.d_o = (t.data_ptr() for t in self.scratch)

    def at(self, row):
        base = self.proj.data_ptr() + 4 * row * self.ld
        self.p.d_q, self.p.d_k, self.p.d_v, self.p.d_gate, self.p.d_f = (base + 4 * int(s) for s in self.sections[:5])

    def rows(self, pos0, m):
        self.at(pos0)
        out = zeros(m, self.H * self.dv + 3, dtype=ttype(self.wtype))
        self.p.n_rows, self.p.pos0, self.p.proj_ld, self.p.d_out_rows, self.p.out_ld = m, pos0, self.ld, out.data_ptr(), self.H * self.dv + 3
        soil(self.lib, self.pkg)
        assert self.lib.b200_gla_rows(C.byref(self.p), None) == 0
        got = host(out)
        assert not got[:, self.H * self.dv:].any()
        return got[:, :self.H * self.dv]

    def one(self, pos):
        self.at(pos)
        self.pos.fill_(pos)
        self.out.fill_(float("nan"))
        soil(self.lib, self.pkg)
        assert self.lib.b200_gla_decode(C.byref(self.p), None) == 0
        return host(self.out)

    def last_state(self):
        s = host(self.st)[self.n % self.slots]
        assert not s[..., self.dv:].any()
        return s[..., :self.dv]


GLA_SHAPES = [(3, 20, 18, 5), (2, 37, 70, 9), (1, 3, 2, 1), (2, 64, 136, 16), (4, 48, 32, 12), (1, 256, 512, 64), (20, 16, 8, 40), (2, 300, 1000, 4)]


@pytest.mark.parametrize("H,d,dv,rank", GLA_SHAPES)
def test_recurrence_in_portions_and_token_by_token(lib, pkg, H, d, dv, rank):
    n = 210
    t = Gla(lib, pkg, H, d, dv, rank, 6.0, n, 21)
    at = 0
    for m in (1, 2, 15, 16, 17, 1, 63, 2, 64):                        # across sixteens and chunks, single tokens in between
        got = t.rows(at, m) if m > 1 else t.one(at)[None]
        close(got, t.want[at:at + m], 2e-5)
        at += m
    for i in range(at, n):
        close(t.one(i)[None], t.want[i:i + 1], 2e-5)
    close(t.last_state(), t.state, 1e-5)


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("n", [1, 2, 16, 63, 64, 65, 128, 129, 700])
def test_recurrence_of_whole_portions(lib, pkg, wtype, n):
    for H, d, dv in ((3, 40, 48), (2, 24, 200)):
        t = Gla(lib, pkg, H, d, dv, 7, 16.0, n, 22, wtype=wtype)
        close(t.rows(0, n), t.want, 5e-3 if wtype == BF16 else 2e-5)
        close(t.last_state(), t.state, 1e-5)


@pytest.mark.parametrize("tau,bias", [(1.0, (-6.0, 12.0)), (0.25, (0.0, 30.0)), (500.0, (3.0, 1.0)), (1.0, (60.0, 0.0)), (1.0, (-200.0, 0.0))])
def test_recurrence_with_extreme_decays(lib, pkg, tau, bias):
    """Channels that forget everything at once beside channels that forget nothing: nothing overflows, nothing is lost."""
    t = Gla(lib, pkg, 2, 24, 20, 6, tau, 200, 23, bias=bias)
    close(t.rows(0, 150), t.want[:150], 5e-5)
    for i in range(150, 200):
        close(t.one(i)[None], t.want[i:i + 1], 5e-5)


def test_an_early_token_is_kept_for_hundreds_of_tokens(lib, pkg):
    """One large token at the start, decays near one: it dominates the outputs to the end, through chunks and single tokens."""
    t = Gla(lib, pkg, 2, 16, 16, 4, 4000.0, 600, 24, bias=(4.0, 0.5))
    before = host(t.proj)
    big = before.copy()
    s = t.sections
    big[2, s[2]:s[3]] *= 300.0
    t.proj.copy_(dev(big))
    q, k, v, g, f = (big[:, s[i]:s[i + 1]] for i in range(5))
    a = o.decay(f[:, :4] @ host(t.keep[0])[:, :4].T + host(t.keep[1]), 4000.0)
    gamma = host(t.keep[2])
    outs = [o.recurrence(q[:, h * 16:h * 16 + 16] / 4, k[:, h * 16:h * 16 + 16], v[:, h * 16:h * 16 + 16], a[:, h * 16:h * 16 + 16])[0] for h in range(2)]
    want = o.rms_norm(np.stack(outs, axis=1), gamma, 1e-4).reshape(600, -1) * o.silu(g)
    close(t.rows(0, 100), want[:100], 2e-5)
    close(t.rows(100, 480), want[100:580], 2e-5)
    for i in range(580, 600):
        close(t.one(i)[None], want[i:i + 1], 2e-5)
    assert np.abs(want - t.want)[400:].max() > 0.5


def test_slow_channels_keep_their_precision_token_by_token(lib, pkg):
    """Decays within 1e-4 of one, each rounded the same way at every token: a thousand single tokens must not add that up."""
    t = Gla(lib, pkg, 1, 12, 8, 2, 40.0, 1000, 27, bias=(5.0, 0.3))
    t.out.fill_(0.0)
    for i in range(990):
        t.at(i)
        t.pos.fill_(i)
        assert lib.b200_gla_decode(C.byref(t.p), None) == 0
    for i in range(990, 1000):
        close(t.one(i)[None], t.want[i:i + 1], 5e-6, t.size)
    close(t.last_state(), t.state, 2e-6)


def test_a_position_can_be_run_again(lib, pkg):
    """States are kept per position: running ahead and coming back, as far as the slots reach, changes nothing."""
    t = Gla(lib, pkg, 2, 24, 20, 6, 8.0, 100, 25, slots=5)
    t.rows(0, 50)
    first = [t.one(i) for i in range(50, 54)]
    again = [t.one(i) for i in range(50, 54)]
    assert all(np.array_equal(a, b) for a, b in zip(first, again))
    close(np.stack(first), t.want[50:54], 2e-5)
    close(t.rows(50, 50), t.want[50:], 2e-5)                          # and from there as one portion
    close(t.rows(0, 3), t.want[:3], 2e-5)                             # a new sequence starts from nothing
    close(t.one(3)[None], t.want[3:4], 2e-5)
    close(t.one(0)[None], t.want[:1], 2e-5)


def test_bad_recurrences_are_refused(lib, pkg):
    t = Gla(lib, pkg, 2, 24, 200, 6, 8.0, 10, 26)
    for field, value in (("tau", 0.0), ("n_slots", 1), ("rank", 0), ("d_a2", None), ("d_state", None)):
        old = getattr(t.p, field)
        t.at(0)
        setattr(t.p, field, value)
        assert lib.b200_gla_decode(C.byref(t.p), None) < 0, field
        setattr(t.p, field, old)
    t.p.n_rows, t.p.pos0, t.p.proj_ld, t.p.d_out_rows, t.p.out_ld = 4, 0, t.ld, t.out.data_ptr(), 400
    t.p.d_o = None                                                    # heads wider than a block need it
    assert lib.b200_gla_rows(C.byref(t.p), None) < 0
