"""The kernels of the latent-attention model one mechanism at a time, through the C ABI, against the plain float64
restatement (oracle/latent_oracle.py). fp32 inputs and weights: a few units of fp32 rounding; bfloat16 weights are given
bfloat16 values, so that the decode kernels (fp32 activations) meet the same bar and only stored bfloat16 results and
tensor-core operands are compared at bfloat16's rounding."""
import ctypes as C

import numpy as np
import pytest

import _latent as T

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


def zeros(*shape):
    return torch.zeros(*shape, dtype=torch.float32, device="cuda")


def host(t):
    torch.cuda.synchronize()
    return t.float().cpu().numpy().astype(np.float64)


def padded(v, n):
    return np.concatenate([v, np.zeros(v.shape[:-1] + (n - v.shape[-1],))], axis=-1)


def typed(a, wtype):
    t = torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).cuda()
    return t.bfloat16() if wtype == BF16 else t


def close(got, want, tol):
    err = np.abs(got - want).max() / np.abs(want).max()
    assert err <= tol, err


def pack(lib, w, wtype, cols, row0=0, step=1, rows=None):
    """w [r, k] -> packed rows of `cols` columns."""
    rows = rows or w.shape[0]
    stride = lib.b200_packed_row_stride(wtype, cols)
    d = torch.full((rows, stride), 0x7f, dtype=torch.uint8, device="cuda")
    src = dev(w)
    assert lib.b200_cast_pack(wtype, src.data_ptr(), w.shape[1], w.shape[0], w.shape[1], d.data_ptr(), stride, row0, step, None) == 0
    torch.cuda.synchronize()
    return d, stride


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("rows,cols", [(3, 8), (5, 37), (40, 256), (7, 1003)])
def test_cast_pack_rounds_to_nearest_and_pads(lib, wtype, rows, cols):
    w = rng(1).standard_normal((rows, cols)).astype(np.float32)
    w[0, 0], w[1, 1] = 1.00390625, 3e38                               # a tie (to even), near the top of the range
    d, stride = pack(lib, w, wtype, up8(cols), row0=1, step=2, rows=2 * rows + 1)
    raw = d.cpu().numpy()
    got = raw.view(np.float32).astype(np.float64) if wtype == F32 else \
        (raw.view(np.uint16).astype(np.uint32) << 16).view(np.float32).astype(np.float64)
    assert np.array_equal(got[1::2][:rows, :cols], o.bf16(w) if wtype == BF16 else w)
    assert not got[1::2][:rows, cols:].any()
    assert (raw[0] == 0x7f).all()                                     # rows in between are left alone


def matvec(lib, pkg, w, wtype, cols, rows, **kw):
    d, stride = pack(lib, w, wtype, cols)
    a = pkg.MatvecArgs()
    a.d_w, a.row_stride, a.rows, a.cols, a.wtype = d.data_ptr(), stride, rows, cols, wtype
    a.n_out = 1
    for k, v in kw.items():
        if k == "d_out":
            a.d_out[0] = v.data_ptr()
        else:
            setattr(a, k, v.data_ptr() if isinstance(v, torch.Tensor) else v)
    rc = lib.b200_matvec(C.byref(a), None)
    torch.cuda.synchronize()
    return rc


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("rows,cols", [(1, 8), (9, 40), (203, 104), (640, 2560), (97, 5000), (40, 8000), (16, 15360)])
def test_matvec(lib, pkg, wtype, rows, cols):
    w, x, out = o.bf16(rng(2).standard_normal((rows, cols))), rng(3).standard_normal(cols), zeros(rows)
    assert matvec(lib, pkg, w, wtype, cols, rows, d_in_vec=dev(x), d_out=out) == 0
    close(host(out), w @ x.astype(np.float32), 2e-6)


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("dim,groups,mix", [(64, 1, False), (102, 3, True), (320, 5, True), (2560, 2, True), (3000, 4, False), (5120, 8, True)])
def test_postnorm_input(lib, pkg, wtype, dim, groups, mix):
    """h = norm(z) (parts apart), x = mix + c h, both kept; then a second norm before the product."""
    g, n = rng(4), up8(dim)
    w, z, gamma, final, older = (g.standard_normal(s) for s in ((24, dim), dim, dim, dim, dim))
    w, c, eps = o.bf16(w), 0.7, 1e-3
    z[: dim // groups] *= 30.0                                        # parts of very different size
    h = o.group_rms(z, gamma, groups, eps)
    x = older + c * h if mix else h
    for norm2 in (False, True):
        out, kept, post = zeros(24), zeros(n), zeros(n)
        kw = dict(in_mode=pkg.B200_IN_POSTNORM, d_in_vec=dev(padded(z, n)), d_slot_norm_gamma=dev(padded(gamma, n)), eps=eps, norm_dim=dim,
                  norm_groups=groups, d_resid_out=kept, d_post_copy=post, d_out=out)
        if mix:
            kw.update(d_mix_in=dev(padded(older, n)), d_mix_coef=dev(np.array([c])))
        if norm2:
            kw.update(d_norm_gamma=dev(padded(final, n)))
        assert matvec(lib, pkg, padded(w, n), wtype, n, 24, **kw) == 0
        close(host(post), padded(h, n), 2e-6)
        close(host(kept), padded(x, n), 2e-6)
        close(host(out), w @ (o.group_rms(x, final, groups, eps) if norm2 else x), 4e-6)


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("rows,cols,hist", [(102, 72, 1), (256, 256, 7), (2560, 512, 36)])
def test_gated_output_and_depth_sum(lib, pkg, wtype, rows, cols, hist):
    g = rng(5)
    w, x, res, gate, bias = (g.standard_normal(s) for s in ((rows, cols), cols, rows, rows, rows))
    w, hs, n = o.bf16(w), g.standard_normal((hist, rows)), up8(rows)
    coef, gate = g.standard_normal(hist), gate * 4
    out, mix = zeros(n), zeros(n)
    assert matvec(lib, pkg, w, wtype, cols, rows, d_in_vec=dev(x), out_mode=pkg.B200_OUT_GATED, d_out_resid=dev(res), d_out_gate=dev(gate),
                  d_out_gate_bias=dev(bias), resid_alpha=2.5, d_out=out, d_hist=dev(padded(hs, n)), hist_n=hist, hist_stride=n,
                  d_hist_coef=dev(coef), d_hist_out=mix) == 0
    close(host(out)[:rows], 2.5 * res + o.logistic(gate + bias) * (w @ x), 4e-6)
    close(host(mix)[:rows], o.depth_average(hs, coef), 4e-6)
    assert not host(out)[rows:].any()


@pytest.mark.parametrize("wtype", TYPES)
def test_pairs_then_plain_rows_and_softcap(lib, pkg, wtype):
    g = rng(6)
    w, x = o.bf16(g.standard_normal((2 * 88 + 40, 104))), g.standard_normal(104)
    y = w @ x
    act, rest = zeros(88), zeros(40)
    assert matvec(lib, pkg, w, wtype, 104, len(w), d_in_vec=dev(x), out_mode=pkg.B200_OUT_GLU, act=1, glu_rows=176, d_out=act, d_out2=rest) == 0
    close(host(act), o.gelu(y[0:176:2]) * y[1:176:2], 4e-6)
    close(host(rest), y[176:], 4e-6)
    out = zeros(len(w))
    assert matvec(lib, pkg, w, wtype, 104, len(w), d_in_vec=dev(x), softcap=3.0, d_out=out) == 0
    close(host(out), o.softcap(y, 3.0), 4e-6)


def test_matvec_refuses_what_it_does_not_do(lib, pkg):
    w = np.ones((8, 16))
    bad = [dict(out_mode=pkg.B200_OUT_GATED), dict(in_mode=pkg.B200_IN_POSTNORM), dict(norm_groups=3, norm_dim=16), dict(norm_dim=17),
           dict(hist_n=2), dict(out_mode=pkg.B200_OUT_GLU, glu_rows=3)]
    for kw in bad:
        assert matvec(lib, pkg, w, F32, 16, 8, d_in_vec=dev(np.ones(16)), d_out=zeros(8), **kw) == -1, kw


@pytest.mark.parametrize("M,N,K", [(1, 64, 8), (130, 203, 104), (300, 96, 1000), (64, 2560, 320), (257, 520, 2568)])
def test_bf16_product(lib, pkg, M, N, K):
    a, b = o.bf16(rng(7).standard_normal((M, K))), o.bf16(rng(8).standard_normal((N, K)))
    da, db = typed(a, BF16), typed(b, BF16)
    c, ld = zeros(M, N), up8(N)
    ch = torch.zeros(M, ld, dtype=torch.bfloat16, device="cuda")
    for half in (False, True):
        g = pkg.GemmArgs()
        g.A, g.a_row, g.a_col, g.B, g.b_row, g.b_col = da.data_ptr(), K, 1, db.data_ptr(), 1, K
        g.C, g.ldc, g.M, g.N, g.K, g.alpha = c.data_ptr(), N, M, N, K, 1.0
        if half:
            g.C, g.Ch, g.ldch = None, ch.data_ptr(), ld
        assert lib.b200_gemm_bf16(C.byref(g), None) == 0
    close(host(c), a @ b.T, 1e-5)
    close(host(ch)[:, :N], a @ b.T, 4.1e-3)
    assert not host(ch)[:, N:].any()


# ------------------------------------------------------------------ row kernels

@pytest.mark.parametrize("dim,groups,hist", [(102, 3, 0), (102, 1, 2), (320, 5, 6), (2560, 2, 3)])
def test_rows_postnorm(lib, pkg, dim, groups, hist):
    g, M, ld = rng(9), 5, up8(dim)
    x, y, gate = (g.standard_normal((M, dim)) for _ in range(3))
    bias, gamma, coef, hs = g.standard_normal(dim), g.standard_normal(dim), g.standard_normal(hist + 1), g.standard_normal((hist, M, dim))
    h = o.gated_postnorm(x, y, gate, bias, 2.5, gamma, groups, 1e-4)
    want = o.depth_average(list(hs) + [h], coef) if hist else h
    post, out, half = zeros(M, ld), zeros(M, ld), torch.ones(M, ld, dtype=torch.bfloat16, device="cuda")
    keep = [dev(padded(x, ld)), dev(padded(y, dim + 3)), dev(padded(gate, dim + 9)), dev(bias), dev(gamma), dev(padded(hs, ld)), dev(coef)]
    a = pkg.RowsPostnormArgs()
    a.x, a.y, a.y_ld, a.gate, a.gate_ld, a.gate_bias, a.gamma = (keep[0].data_ptr(), keep[1].data_ptr(), dim + 3, keep[2].data_ptr(), dim + 9,
                                                                 keep[3].data_ptr(), keep[4].data_ptr())
    a.alpha, a.eps, a.rows, a.dim, a.ld, a.groups, a.norm_out = 2.5, 1e-4, M, dim, ld, groups, post.data_ptr()
    a.hist, a.hist_n, a.hist_stride, a.coef, a.out, a.out_h = keep[5].data_ptr(), hist, M * ld, keep[6].data_ptr(), out.data_ptr(), half.data_ptr()
    assert lib.b200_rows_postnorm(C.byref(a), None) == 0
    close(host(post), padded(h, ld), 3e-6)
    close(host(out), padded(want, ld), 3e-6)
    close(host(half), padded(want, ld), 4.1e-3)


@pytest.mark.parametrize("wtype", TYPES)
def test_small_row_steps(lib, wtype):
    g = rng(10)
    half = torch.bfloat16 if wtype == BF16 else torch.float32
    tol = 4.1e-3 if wtype == BF16 else 3e-6
    x, gamma = g.standard_normal((6, 102)), g.standard_normal(102)
    index = torch.tensor([4, 0, 5], dtype=torch.int32, device="cuda")
    out = torch.ones(3, 104, dtype=half, device="cuda")
    assert lib.b200_rows_norm(dev(padded(x, 104)).data_ptr(), index.data_ptr(), 3, 102, 104, 3, 1e-3, dev(gamma).data_ptr(), wtype, out.data_ptr(), None) == 0
    close(host(out), padded(o.group_rms(x[[4, 0, 5]], gamma, 3, 1e-3), 104), tol)

    gu = 2.0 * g.standard_normal((5, 150))
    out = torch.ones(5, 72, dtype=half, device="cuda")
    assert lib.b200_rows_gelu_mul(dev(gu).data_ptr(), 150, 5, 72, wtype, out.data_ptr(), None) == 0
    close(host(out), o.gelu(gu[:, 0:144:2]) * gu[:, 1:144:2], tol)

    emb, ids = g.standard_normal((30, 104)), [3, 29, 0, 3]
    tok, x0, xh = torch.tensor(ids, dtype=torch.int32, device="cuda"), zeros(4, 104), torch.zeros(4, 104, dtype=torch.bfloat16, device="cuda")
    assert lib.b200_rows_embed(dev(emb).data_ptr(), tok.data_ptr(), 4, 30, 104, 5.0, x0.data_ptr(), xh.data_ptr(), None) == 0
    close(host(x0), 5.0 * emb[ids], 1e-6)
    close(host(xh), 5.0 * emb[ids], 4.1e-3)

    z = dev(20.0 * g.standard_normal((3, 50)))
    want = host(z)
    want[:, :41] = o.softcap(want[:, :41], 7.0)
    assert lib.b200_rows_softcap(z.data_ptr(), 3, 41, 50, 7.0, None) == 0
    close(host(z), want, 1e-6)


# ------------------------------------------------------------------ latent attention

class Attention:
    """One latent-attention layer's inputs for n tokens, and both forms of the kernels over them."""

    def __init__(self, lib, pkg, wtype, mix, n, seed, rot_dims=None, max_seq=None):
        self.lib, self.pkg, self.wtype, self.mix, self.n = lib, pkg, wtype, mix, n
        g = rng(seed)
        H, d, r, v, R = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
        self.q, self.dkv, self.gate = g.standard_normal((n, H, d + r)), 2.0 * g.standard_normal((n, R + r)), g.standard_normal((n, H * v))
        self.gamma = 1.0 + 0.3 * g.standard_normal(R)
        self.uk, self.uv = o.bf16(g.standard_normal((H * d, R)) * R ** -0.5), o.bf16(g.standard_normal((H * v, R)) * R ** -0.5)
        self.eps, self.max_seq = 1e-4, max_seq or n
        if rot_dims is not None:
            mix["rot"]["dims"] = rot_dims
        self.R8, self.r8, self.d8, self.v8 = up8(R), up8(r), up8(d), up8(v)

    def expected(self):
        c, kr = o.rms(self.dkv[:, :self.mix["kv_rank"]], self.gamma, self.eps), self.dkv[:, self.mix["kv_rank"]:]
        kr = o.rotate(kr, np.arange(self.n), self.mix["rot"]["base"], self.mix["rot"]["dims"])
        self.c, self.kr = c, kr
        return o.attend(self.q, c, kr, self.mix, self.uk, self.uv).reshape(self.n, -1) * o.logistic(self.gate)

    def args(self):
        m, dims = self.mix, self.mix["rot"]["dims"]
        H, d, v, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        pos, i = np.arange(self.max_seq)[:, None], np.arange(dims // 2)[None, :]
        ang = pos * m["rot"]["base"] ** (-2.0 * i / max(dims, 1))
        ukt = padded(np.concatenate([self.uk[h * d:(h + 1) * d].T for h in range(H)]), self.d8)
        kv = np.zeros((H * (self.d8 + self.v8), self.R8))
        for h in range(H):
            at = h * (self.d8 + self.v8)
            kv[at:at + d, :R] = self.uk[h * d:(h + 1) * d]
            kv[at + self.d8:at + self.d8 + v, :R] = self.uv[h * v:(h + 1) * v]
        self.kvmat = kv
        self.keep = dict(rope=dev(np.stack([np.cos(ang), np.sin(ang)], axis=-1)) if dims else zeros(2), gamma=dev(padded(self.gamma, self.R8)),
                         cache=torch.full((self.max_seq, self.R8 + self.r8), 1e30, device="cuda").to(torch.bfloat16 if self.wtype == BF16 else torch.float32),
                         ukt=typed(ukt, self.wtype), kv=typed(kv, self.wtype))
        a = self.pkg.LatentArgs()
        a.wtype, a.heads, a.dim, a.rot_dim, a.rot_dims, a.vdim, a.kv_rank = self.wtype, H, d, m["rot_dim"], dims, v, R
        a.window, a.max_seq = (m["mask"]["size"] if m.get("mask") else 0), self.max_seq
        a.scale, a.eps = m["scale"], self.eps
        a.d_rope, a.d_dkv_gamma, a.d_cache = (self.keep[k].data_ptr() for k in ("rope", "gamma", "cache"))
        a.d_w_uk_t, a.d_w_kv = self.keep["ukt"].data_ptr(), self.keep["kv"].data_ptr()
        return a

    def decode(self, positions=None):
        """All tokens one at a time; the output of every one (or of `positions`)."""
        m, a = self.mix, self.args()
        H = m["heads"]
        a.n_split = self.lib.b200_latent_splits(H, a.window, self.max_seq)
        q, dkv, gate = dev(self.q.reshape(self.n, -1)), dev(self.dkv), dev(self.gate)
        pos = torch.arange(self.n, dtype=torch.int32, device="cuda")
        out, qlat, part = zeros(self.n, H * m["vdim"]), zeros(H * (self.R8 + self.r8)), zeros(H * a.n_split * (self.R8 + 8))
        a.d_qlat, a.d_part = qlat.data_ptr(), part.data_ptr()
        for i in range(self.n):
            a.d_q, a.d_dkv, a.d_gate = q[i].data_ptr(), dkv[i].data_ptr(), gate[i].data_ptr()
            a.d_out, a.d_pos = out[i].data_ptr(), pos[i:].data_ptr()
            assert self.lib.b200_latent_decode(C.byref(a), None) == 0
        return host(out)

    def rows(self, portions):
        """The same tokens in portions."""
        m, a = self.mix, self.args()
        H, dims = m["heads"], torch.bfloat16 if self.wtype == BF16 else torch.float32
        proj = dev(np.concatenate([self.q.reshape(self.n, -1), self.dkv, self.gate], axis=1))
        ld, oq = proj.shape[1], m["heads"] * (m["dim"] + m["rot_dim"])
        out = torch.zeros(self.n, up8(H * m["vdim"]), dtype=dims, device="cuda")
        q_rows = torch.zeros(self.n, H * (self.d8 + self.r8), dtype=dims, device="cuda")
        kvw, p = self.keep["kv"].double(), 0
        for k in portions:
            row0 = max(0, p - a.window + 1) if a.window else 0
            a.d_q = proj[p].data_ptr()
            a.d_dkv, a.d_gate, a.proj_ld = a.d_q + 4 * oq, a.d_q + 4 * (oq + self.dkv.shape[1]), ld
            a.n_rows, a.pos0, a.kv_row0, a.d_q_rows = k, p, row0, q_rows.data_ptr()
            a.d_out_rows, a.out_ld = out[p].data_ptr(), out.shape[1]
            assert self.lib.b200_latent_rows_prep(C.byref(a), None) == 0
            torch.cuda.synchronize()
            kv = (self.keep["cache"][row0:p + k, :self.R8].double() @ kvw.T).to(dims).contiguous()
            a.d_kv, a.kv_ld = kv.data_ptr(), kv.shape[1]
            assert self.lib.b200_latent_rows_attend(C.byref(a), None) == 0
            torch.cuda.synchronize()
            p += k
        assert p == self.n
        return host(out)[:, :H * m["vdim"]]


SHAPES = [  # heads, dim, rot_dim, vdim, kv_rank, window
    (3, 20, 12, 18, 37, 21), (1, 8, 2, 1, 8, 1), (18, 40, 24, 72, 300, 33), (2, 136, 64, 130, 520, 96), (5, 9, 6, 7, 50, 300), (9, 64, 32, 128, 96, 65),
    (1, 260, 10, 24, 40, 50)]


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("shape", SHAPES)
def test_decode_attention(lib, pkg, wtype, shape):
    n = 150
    t = Attention(lib, pkg, wtype, T.L(*shape, None, base=300.0)["mixer"], n, 11)
    want = t.expected()
    close(t.decode(), want, 2e-2 if wtype == BF16 else 5e-6)


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("portions", [[150], [64, 1, 2, 83], [2] * 10 + [63, 65, 2]])
def test_rows_attention(lib, pkg, wtype, shape, portions):
    t = Attention(lib, pkg, wtype, T.L(*shape, None, base=300.0)["mixer"], 150, 12)
    want = t.expected()
    close(t.rows(portions), want, 2.5e-2 if wtype == BF16 else 5e-6)


@pytest.mark.parametrize("wtype", TYPES)
def test_no_window_and_partly_rotated_parts(lib, pkg, wtype):
    mix = T.L(4, 16, 12, 20, 40, 1, None, base=200.0)["mixer"]
    mix["mask"] = None
    t = Attention(lib, pkg, wtype, mix, 140, 13, rot_dims=8, max_seq=200)
    want, tol = t.expected(), 2.5e-2 if wtype == BF16 else 5e-6
    close(t.decode(), want, tol)
    close(t.rows([100, 40]), want, tol)


@pytest.mark.parametrize("wtype", TYPES)
@pytest.mark.parametrize("window", [2, 31, 32, 33, 64, 96, 100])
def test_one_loud_key_just_inside_and_just_outside_the_window(lib, pkg, wtype, window):
    """One position's key answers every query far louder than the others: the output is its value while it is in
    the window and nothing like it one position later."""
    n, loud = 170, 40
    t = Attention(lib, pkg, wtype, T.L(2, 16, 8, 16, 24, window, None, scale=1.5)["mixer"], n, 14)
    t.q[:, :, :16] = t.q[loud, :, :16]                               # every query asks for the same thing
    t.q[:, :, 16:] *= 0.1
    keys = np.stack([t.uk[h * 16:(h + 1) * 16].T @ t.q[loud, h, :16] for h in range(2)])
    others = t.dkv[:, :24] * t.gamma                                 # nothing in the others' keys answers it
    others -= others @ np.linalg.pinv(keys) @ keys
    t.dkv[:, :24] = others / t.gamma
    t.dkv[loud, :24] = (keys[0] / np.linalg.norm(keys[0]) + keys[1] / np.linalg.norm(keys[1])) / t.gamma
    want = t.expected()
    value = (t.uv @ t.c[loud]).reshape(1, -1) * o.logistic(t.gate)
    for got in (t.decode(), t.rows([n]), t.rows([50, 2, 30, 88])):
        close(got, want, 6e-2 if wtype == BF16 else 5e-6)    # scores of 30 and more, rounded operands
        inside, outside = loud + window - 1, loud + window
        near = np.abs(got - value).max(axis=1) / np.abs(value).max()
        assert near[inside] < 0.2 and (near[loud:inside + 1] < 0.3).all() and near[outside] > 0.3, (near[inside], near[outside])


def test_a_position_outside_the_cache_is_ignored(lib, pkg):
    t = Attention(lib, pkg, F32, T.L(2, 16, 8, 16, 24, 9, None)["mixer"], 4, 15)
    a = t.args()
    a.n_split = 1
    q, dkv, gate, out, qlat, part = dev(t.q[0]), dev(t.dkv[0]), dev(t.gate[0]), zeros(32), zeros(64), zeros(2 * 32)
    a.d_q, a.d_dkv, a.d_gate, a.d_out, a.d_qlat, a.d_part = (x.data_ptr() for x in (q, dkv, gate, out, qlat, part))
    before = t.keep["cache"].clone()
    for p in (-1, 4, 1 << 30):
        pos = torch.tensor([p], dtype=torch.int32, device="cuda")
        a.d_pos = pos.data_ptr()
        assert lib.b200_latent_decode(C.byref(a), None) == 0
        torch.cuda.synchronize()
    assert torch.equal(before, t.keep["cache"]) and not host(out).any()
    a.n_split = 0
    assert lib.b200_latent_decode(C.byref(a), None) == -1
