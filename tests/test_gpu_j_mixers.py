"""Kernels behind the mixers of a layer against the float64 restatement (oracle/pimezen_oracle.py):
sliding-window attention with kept first tokens, distance bias and head mixing; gated linear
attention; the fp32-stream pieces around them.  Storage bf16 and fp32; prompts whole, in portions
and token by token."""
import numpy as np
import pytest
import torch

from oracle import pimezen_oracle as po

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


def _round(a, dtype):
    return torch.tensor(a).to(dtype).double().numpy()


def _pad(a, heads, padded):
    """[T, heads * d] -> [T, heads * padded]"""
    t = torch.tensor(a)
    out = torch.zeros(t.shape[0], heads, padded, dtype=torch.float64)
    d = t.shape[1] // heads
    out[:, :, :d] = t.view(-1, heads, d)
    return out.view(t.shape[0], -1)


def _up(n):
    return -(-n // 16) * 16


def _rel(got, want):
    """rms error of every row relative to the rms of the row or of the whole reference, whichever is
    larger; the worst row"""
    rows = np.sqrt((want ** 2).mean(-1))
    d = np.sqrt(((got - want) ** 2).mean(-1)) / np.maximum(rows, np.sqrt((want ** 2).mean()))
    return float(d.max())


class Window:
    """One window-attention problem: raw projections of B sequences and the mixer's weights."""

    def __init__(self, dtype, T, H, G, dim, vdim, size, keep, B=1, seed=0, scale=None):
        self.__dict__.update(dtype=dtype, T=T, H=H, G=G, dim=dim, vdim=vdim, size=size, keep=keep, B=B)
        rng = np.random.default_rng(seed)
        r = lambda *s: _round(rng.standard_normal(s), dtype)
        self.scale = dim ** -0.5 if scale is None else scale
        self.eps = 1e-5
        self.q, self.k, self.v = r(B, T, H * dim), r(B, T, G * dim), r(B, T, G * vdim)
        self.qn, self.kn = _round(1 + 0.2 * rng.standard_normal(dim), dtype), _round(1 + 0.2 * rng.standard_normal(dim), dtype)
        self.r1, self.r2 = _round(rng.uniform(0.0, 1.0, H), dtype), _round(rng.uniform(0.01, 1.0, H), dtype)
        self.talk = _round(np.eye(H) + 0.3 * rng.standard_normal((H, H)), dtype)

    def reference(self):
        out = []
        for b in range(self.B):
            q = po.head_norm(self.q[b], self.qn, self.H, self.eps)
            k = po.head_norm(self.k[b], self.kn, self.G, self.eps)
            w = po.softmax_weights(q, k, self.scale, self.r1, self.r2, self.size, self.keep)
            w = po.mix_heads(w, self.talk)
            v = self.v[b].reshape(self.T, self.G, self.vdim)
            rep = self.H // self.G
            out.append(np.stack([w[h] @ v[:, h // rep] for h in range(self.H)], 1).reshape(self.T, -1))
        return 1.25 * np.stack(out)

    def rings(self):
        z = dict(dtype=self.dtype, device="cuda")
        slots = self.size + self.keep
        return (torch.full((self.B, slots, self.G, _up(self.dim)), 3.0, **z),
                torch.full((self.B, slots, self.G, _up(self.vdim)), 3.0, **z))   # stale contents

    def run(self, portions, rings=None, on_device=False):
        from complexity_deep_b200 import ops
        dev = dict(dtype=self.dtype, device="cuda")
        dp, vp = _up(self.dim), _up(self.vdim)
        rk, rv = rings or self.rings()
        w = {"q_norm": torch.tensor(self.qn), "k_norm": torch.tensor(self.kn), "r1": torch.tensor(self.r1),
             "r2": torch.tensor(self.r2), "talk": torch.tensor(self.talk)}
        for n in ("q_norm", "k_norm"):
            w[n] = torch.nn.functional.pad(w[n], (0, dp - self.dim))
        w = {k: v.to(**dev).contiguous() for k, v in w.items()}
        at, outs = 0, []
        for n in portions:
            rows = [torch.cat([_pad(self.q[b, at:at + n], self.H, dp), _pad(self.k[b, at:at + n], self.G, dp),
                               _pad(self.v[b, at:at + n], self.G, vp)], 1) for b in range(self.B)]
            buf = torch.cat(rows, 0).to(**dev).contiguous()
            a, c = self.H * dp, self.H * dp + self.G * dp
            wide = torch.zeros(self.B * n, self.H * vp + 16, **dev)
            out = wide[:, 8:8 + self.H * vp]                # columns of a wider buffer
            pos = torch.tensor([at], dtype=torch.int32, device="cuda") if on_device else None
            ops.window_attention_({"q": buf[:, :a], "k": buf[:, a:c], "v": buf[:, c:]}, out, w, rk, rv,
                                  batch=self.B, seq_len=n, heads=self.H, kv_heads=self.G, dim=self.dim,
                                  vdim=self.vdim, window=self.size, keep=self.keep, scale=self.scale,
                                  eps=self.eps, out_scale=1.25, pos0=0 if on_device else at, pos_dev=pos)
            o = out.double().cpu().view(self.B, n, self.H, vp)
            assert float(o[..., self.vdim:].abs().max() if vp > self.vdim else 0) == 0
            outs.append(o[..., :self.vdim].reshape(self.B, n, -1))
            at += n
        ops.status_fetch()
        return torch.cat(outs, 1).numpy()


TOL = {BF: 2.5e-2, F32: 3e-5}
SHAPES = [  # T, H, G, dim, vdim, size, keep, B
    (70, 4, 2, 32, 48, 20, 3, 2),
    (130, 8, 2, 64, 112, 50, 7, 1),
    (96, 8, 8, 128, 128, 40, 3, 1),
    (83, 16, 8, 128, 128, 37, 2, 2),
    (101, 6, 3, 24, 40, 33, 0, 1),
    (90, 16, 4, 128, 128, 64, 5, 1),
    (75, 5, 1, 40, 112, 19, 40, 1),
    (60, 12, 12, 16, 64, 200, 2, 1),
    (66, 24, 8, 48, 64, 17, 1, 1),
    (64, 3, 3, 72, 136, 16, 16, 1),
    (50, 8, 8, 96, 256, 1, 4, 1),
    (40, 40, 4, 16, 16, 9, 2, 1),
]


def _cuts(T, seed):
    rng, out = np.random.default_rng(seed), []
    while sum(out) < T:
        out.append(int(min(rng.choice([1, 2, 3, 7, 16, 17, 33, 40]), T - sum(out))))
    return out


@pytest.mark.parametrize("dtype", [BF, F32], ids=["bf16", "fp32"])
@pytest.mark.parametrize("shape", SHAPES)
def test_window_attention_whole_portions_and_decode(shape, dtype):
    T, H, G, dim, vdim, size, keep, B = shape
    w = Window(dtype, T, H, G, dim, vdim, size, keep, B, seed=T)
    ref = w.reference()
    for portions in ([T], _cuts(T, 1), [2] * (T // 2) + [1] * (T % 2), [T - 9] + [1] * 9, [1] * T):
        assert _rel(w.run(portions), ref) <= TOL[dtype], portions
    assert _rel(w.run([1] * T, on_device=True), ref) <= TOL[dtype]


@pytest.mark.parametrize("dtype", [BF, F32], ids=["bf16", "fp32"])
@pytest.mark.parametrize("H,G,dim,vdim,size,keep", [(8, 2, 64, 112, 50, 7), (3, 1, 48, 32, 32, 4), (16, 4, 128, 128, 45, 5)])
def test_window_edges_show(dtype, H, G, dim, vdim, size, keep):
    """One query looks for one key that stands out by far: just inside and just outside the window,
    the last kept token and the one after it, and the query's own token; as part of a prompt, as a
    decoded token and in a portion of two."""
    T, i = 2 * size + keep + 9, 2 * size + keep + 5
    for j in (i, i - 1, i - size + 1, i - size, keep - 1, keep, 0):
        w = Window(dtype, T, H, G, dim, vdim, size, keep, seed=j, scale=28.0 / dim)
        w.q *= 0.1
        w.k *= 0.1
        u = np.sign(np.random.default_rng(5).standard_normal(dim))
        w.q[0, i] = np.tile(u, H)
        w.k[0, j] = np.tile(u, G)
        w.v[0, j] *= 8
        ref = w.reference()
        seen = po.window_visible(i, j, size, keep)
        big = np.abs(ref[0, i]).mean() > 3.0
        assert big == seen                                   # the reference itself shows it
        for portions in ([T], [i] + [1] * (T - i), [i - 1, 2] + [T - i - 1], [j + 1, T - j - 1] if j + 1 < T else [T]):
            got = w.run(portions)
            assert _rel(got, ref) <= TOL[dtype], (j, portions)
            assert _rel(got[:, i], ref[:, i]) <= TOL[dtype], (j, portions)


def test_window_ring_is_reused_without_traces():
    w1 = Window(BF, 90, 4, 2, 32, 32, 20, 3, seed=1)
    w2 = Window(BF, 47, 4, 2, 32, 32, 20, 3, seed=2)
    rings = w1.rings()
    w1.run([50] + [1] * 40, rings)
    used = w2.run([2, 13] + [1] * 32, rings)
    fresh = w2.run([2, 13] + [1] * 32)
    assert np.array_equal(used, fresh)


def test_window_long_decode_passes_the_window_many_times():
    w = Window(F32, 400, 2, 1, 16, 16, 12, 3, seed=4)
    assert _rel(w.run([1] * 400), w.reference()) <= TOL[F32]


class Linear:
    def __init__(self, dtype, T, H, dk, dv, rank, tau, B=1, seed=0, bias=(-1.0, 4.0)):
        self.__dict__.update(dtype=dtype, T=T, H=H, dk=dk, dv=dv, rank=rank, tau=tau, B=B)
        rng = np.random.default_rng(seed)
        r = lambda *s: _round(rng.standard_normal(s), dtype)
        self.q, self.k, self.v, self.g = r(B, T, H * dk), r(B, T, H * dk), r(B, T, H * dv), r(B, T, H * dv)
        self.u = r(B, T, rank)
        self.a2 = _round(rng.standard_normal((H * dk, rank)) / rank ** 0.5, dtype)
        self.a2_b = _round(rng.uniform(*bias, H * dk), dtype)
        self.norm = _round(1 + 0.2 * rng.standard_normal(dv), dtype)
        self.eps = 1e-5

    def reference(self):
        outs, states = [], []
        for b in range(self.B):
            h = lambda a, d: a[b].reshape(self.T, self.H, d)
            z = self.u[b] @ self.a2.T + self.a2_b
            alpha = po.sigmoid(z) ** (1.0 / self.tau)
            o, S = po.linear_recurrence(h(self.q, self.dk) * self.dk ** -0.5, h(self.k, self.dk), h(self.v, self.dv),
                                        alpha.reshape(self.T, self.H, self.dk))
            y = po.rms(o, self.eps) * self.norm * h(self.g, self.dv) * po.sigmoid(h(self.g, self.dv))
            outs.append(0.75 * y.reshape(self.T, -1))
            states.append(S)
        return np.stack(outs), np.stack(states)

    def run(self, portions, state=None):
        from complexity_deep_b200 import ops
        dev = dict(dtype=self.dtype, device="cuda")
        kp, vp, rp = _up(self.dk), _up(self.dv), _up(self.rank)
        if state is None:
            state = torch.zeros(self.B, self.H, kp, vp, dtype=F32, device="cuda")
        a2 = torch.zeros(self.H, kp, rp)
        a2[:, :self.dk, :self.rank] = torch.tensor(self.a2).view(self.H, self.dk, self.rank)
        w = {"a2": a2.view(-1, rp).to(**dev), "a2_b": _pad(self.a2_b[None], self.H, kp)[0].to(**dev),
             "norm": torch.nn.functional.pad(torch.tensor(self.norm), (0, vp - self.dv)).to(**dev)}
        at, outs = 0, []
        for n in portions:
            rows = [torch.cat([_pad(self.q[b, at:at + n], self.H, kp), _pad(self.k[b, at:at + n], self.H, kp),
                               _pad(self.v[b, at:at + n], self.H, vp), _pad(self.g[b, at:at + n], self.H, vp),
                               _pad(self.u[b, at:at + n], 1, rp)], 1) for b in range(self.B)]
            buf = torch.cat(rows, 0).to(**dev).contiguous()
            cut = np.cumsum([0, self.H * kp, self.H * kp, self.H * vp, self.H * vp, rp])
            proj = {name: buf[:, cut[x]:cut[x + 1]] for x, name in enumerate(("q", "k", "v", "gate", "inner"))}
            out = torch.zeros(self.B * n, self.H * vp, **dev)
            ops.linear_attention_(proj, out, w, state, batch=self.B, seq_len=n, heads=self.H, dim=self.dk,
                                  vdim=self.dv, tau=self.tau, eps=self.eps, out_scale=0.75)
            o = out.double().cpu().view(self.B, n, self.H, vp)
            outs.append(o[..., :self.dv].reshape(self.B, n, -1))
            at += n
        ops.status_fetch()
        return torch.cat(outs, 1).numpy(), state[:, :, :self.dk, :self.dv].double().cpu().numpy()


LINEAR_TOL = {BF: 1e-2, F32: 1e-4}
LINEAR_SHAPES = [  # T, H, dk, dv, rank, tau, B
    (150, 6, 48, 64, 16, 12.0, 1),
    (97, 3, 24, 40, 5, 2.0, 2),
    (200, 2, 128, 128, 16, 16.0, 1),
    (130, 5, 16, 96, 24, 1.0, 1),
    (64, 2, 80, 48, 8, 7.0, 1),
    (129, 1, 256, 256, 32, 16.0, 1),
    (66, 3, 136, 24, 12, 16.0, 1),
    (70, 1, 320, 264, 16, 16.0, 1),
]


@pytest.mark.parametrize("dtype", [BF, F32], ids=["bf16", "fp32"])
@pytest.mark.parametrize("shape", LINEAR_SHAPES)
def test_linear_attention_whole_portions_and_decode(shape, dtype):
    m = Linear(dtype, *shape[:6], B=shape[6], seed=shape[0])
    T = shape[0]
    ref, state = m.reference()
    for portions in ([T], _cuts(T, 3), [2] * (T // 2) + [1] * (T % 2), [63, T - 63], [T - 20] + [1] * 20, [1] * T):
        got, s = m.run(portions)
        assert _rel(got, ref) <= LINEAR_TOL[dtype], portions
        assert _rel(s.reshape(1, -1), state.reshape(1, -1)) <= (1e-4 if dtype == BF else 1e-5), portions


@pytest.mark.parametrize("dtype", [BF, F32], ids=["bf16", "fp32"])
def test_linear_attention_fast_and_mixed_decays(dtype):
    """Decays from almost none to so fast that the cumulative one leaves the fp32 range within a
    chunk, side by side in one head."""
    m = Linear(dtype, 190, 2, 48, 32, 8, 0.5, seed=9)
    m.a2_b = _round(np.linspace(-12.0, 30.0, 2 * 48), dtype)
    ref, state = m.reference()
    for portions in ([190], [100, 90], [17, 40, 133], [1] * 190):
        got, s = m.run(portions)
        assert np.isfinite(got).all() and np.isfinite(s).all()
        assert _rel(got, ref) <= LINEAR_TOL[dtype], portions
        assert _rel(s.reshape(1, -1), state.reshape(1, -1)) <= 1e-4


def test_linear_attention_remembers_a_far_key():
    """Almost no decay and one strong key: queries hundreds of tokens later find it, whatever the
    cut; without the carried state they would not."""
    m = Linear(BF, 500, 2, 32, 32, 8, 16.0, seed=11, bias=(12.0, 14.0))
    u = np.sign(np.random.default_rng(1).standard_normal(64)) * 4
    m.k *= 0.02
    m.k[0, 3] = u
    m.q[0, 480:] = u / 4
    ref, _ = m.reference()
    lost = Linear(BF, 500, 2, 32, 32, 8, 16.0, seed=11, bias=(12.0, 14.0))
    lost.__dict__.update(k=np.where(np.arange(500)[None, :, None] == 3, 0, m.k), q=m.q)
    assert _rel(lost.reference()[0][:, 480:], ref[:, 480:]) > 0.3
    for portions in ([500], [2, 2, 496], [400, 64, 16] + [1] * 20, [100] * 5):
        assert _rel(m.run(portions)[0][:, 480:], ref[:, 480:]) <= LINEAR_TOL[BF], portions


# ------------------------------------------------------------------------------ fp32 stream
@pytest.mark.parametrize("T,K,N", [(1, 64, 40), (33, 312, 72), (130, 200, 328), (300, 64, 1000), (2300, 512, 768),
                                   (40, 4096, 2048)])
def test_linear_into_fp32_stream(T, K, N):
    from complexity_deep_b200 import ops
    g = torch.Generator().manual_seed(T + N)
    x = torch.randn(T, K, generator=g).to(BF)
    w = (torch.randn(N, K, generator=g) / K ** 0.5).to(BF)
    s = torch.randn(N, generator=g).to(BF)
    r = torch.randn(T, N, generator=g) * 10
    want = r.double() + s.double() * (x.double() @ w.double().t())
    stream = r.cuda()
    out = ops.linear_to_f32(x.cuda(), w.cuda(), residual=stream, col_scale=s.cuda(), inplace=True)
    assert out.data_ptr() == stream.data_ptr()
    assert float((out.double().cpu() - want).abs().max()) <= 2e-5 * float(want.abs().max())
    plain = ops.linear_to_f32(x.cuda(), w.cuda())
    assert float((plain.double().cpu() - x.double() @ w.double().t()).abs().max()) <= 2e-5
    full = ops.linear_to_f32(x.float().cuda(), w.float().cuda(), residual=r.cuda(), col_scale=s.float().cuda())
    assert float((full.double().cpu() - want).abs().max()) <= 2e-5 * float(want.abs().max())
    ops.status_fetch()


@pytest.mark.parametrize("T,H,I", [(5, 64, 40), (300, 296, 392), (2100, 256, 704)])
@pytest.mark.parametrize("limit", [0.5, 3.0, 1e30])
def test_clamped_glu(T, H, I, limit):
    from complexity_deep_b200.core.mlp import ClampedGLU
    from complexity_deep_b200 import ops
    g = torch.Generator().manual_seed(T)
    mlp = ClampedGLU(H, I, limit)
    for p in mlp.parameters():
        p.data = (torch.randn(p.shape, generator=g) * 2 / p.shape[1] ** 0.5).to(BF).float()
    x = torch.randn(T, H, generator=g).to(BF)
    W = {k: v.detach().double().numpy() for k, v in mlp.named_parameters()}
    want = po.clamped_glu(x.double().numpy(), W["gate_proj.weight"], W["up_proj.weight"], W["down_proj.weight"], limit)
    for dtype in (F32, BF):
        m = mlp.to(device="cuda", dtype=dtype)
        got = m.run(x.to(device="cuda", dtype=dtype), torch.zeros(T, H, device="cuda")).double().cpu().numpy()
        assert _rel(got, want) <= (3e-5 if dtype == F32 else 1.5e-2)
    ops.status_fetch()


@pytest.mark.parametrize("T,W", [(1, 20), (37, 328), (5, 1500), (9, 2304)])
def test_stream_norm_and_embedding(T, W):
    from complexity_deep_b200 import ops
    from complexity_deep_b200.core.normalization import StreamNorm
    from complexity_deep_b200.core.padding import pad_rows
    g = torch.Generator().manual_seed(W)
    ldx = -(-W // 8) * 8
    table = torch.randn(50, W, generator=g).to(BF)
    ids = torch.randint(0, 50, (T,), generator=g)
    for dtype in (BF, F32):
        x = ops.embed_rows(ids.cuda(), pad_rows(table, 56, ldx).to(dtype).cuda(), W, ldx)
        assert torch.equal(x[:, :W].cpu(), table[ids].float()) and float(x[:, W:].abs().sum()) == 0
        norm = StreamNorm(W, 1e-3, offset=1.0)
        norm.weight.data = (torch.randn(W, generator=g) * 0.3).to(BF).float()
        want = po.norm(table[ids].double().numpy(), norm.weight.detach().double().numpy(), 1e-3)
        got = norm.to(device="cuda", dtype=dtype)(x)
        assert got.dtype == dtype and float(got[:, W:].float().abs().sum()) == 0
        assert _rel(got[:, :W].double().cpu().numpy(), want) <= (3e-3 if dtype == BF else 1e-6)
