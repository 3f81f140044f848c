"""Kernels behind the Rugedra layers against the float64 restatement (oracle/rugedra_oracle.py): latent
attention, the delta rule with per-channel decay, learned routing with experts, and the fp32-stream
pieces around them.  Storage bf16 and fp32; prompts whole, in portions and token by token."""
import numpy as np
import pytest
import torch

from oracle import rugedra_oracle as ro

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


def _round(a, dtype):
    return torch.tensor(a).to(dtype).double().numpy()


def _pad(a, heads, padded):
    """[T, heads * d] -> [T, heads * padded]"""
    t = torch.tensor(a)
    out = torch.zeros(t.shape[0], heads, padded, dtype=torch.float64)
    d = t.shape[1] // heads
    out[:, :, :d] = t.reshape(-1, heads, d)
    return out.view(t.shape[0], -1)


def _up(n):
    return -(-n // 16) * 16


def _rel(got, want):
    """rms error of every row relative to the rms of the row or of the whole reference, whichever is
    larger; the worst row"""
    rows = np.sqrt((want ** 2).mean(-1))
    d = np.sqrt(((got - want) ** 2).mean(-1)) / np.maximum(rows, np.sqrt((want ** 2).mean()))
    return float(d.max())


def _cuts(T, seed):
    rng, out = np.random.default_rng(seed), []
    while sum(out) < T:
        out.append(int(min(rng.choice([1, 2, 3, 7, 16, 17, 33, 40, 65]), T - sum(out))))
    return out


# ------------------------------------------------------------------------------ latent attention
class Latent:
    """One problem: projections of B sequences and the mixer's weights."""

    def __init__(self, dtype, T, H, dim, rot, vdim, rank, B=1, seed=0, scale=None, base=1000.0, rot_dims=None):
        self.__dict__.update(dtype=dtype, T=T, H=H, dim=dim, rot=rot, vdim=vdim, rank=rank, B=B)
        rng = np.random.default_rng(seed)
        r = lambda *s: _round(rng.standard_normal(s), dtype)
        self.scale = (dim + rot) ** -0.5 if scale is None else scale
        self.eps, self.base, self.rot_dims = 1e-5, base, rot_dims or rot
        self.q, self.kv, self.gate = r(B, T, H, dim + rot), r(B, T, rank + rot), r(B, T, H)
        self.norm = _round(1 + 0.2 * rng.standard_normal(rank), dtype)
        self.uk = _round(rng.standard_normal((H, dim, rank)) * rank ** -0.5, dtype)
        self.uv = _round(rng.standard_normal((H, vdim, rank)) * rank ** -0.5, dtype)

    def reference(self):
        c = {"heads": self.H, "dim": self.dim, "vdim": self.vdim, "kv_rank": self.rank, "scale": self.scale,
             "rot": {"dims": self.rot_dims, "base": self.base}}
        out = []
        for b in range(self.B):
            lat, key = ro.latent_split(self.kv[b], {"dkv": np.eye(self.rank + self.rot), "dkv.norm": self.norm}, c, self.eps)
            o = ro.latent_heads(self.q[b], lat, key, self.uk, self.uv, c) * ro.sigmoid(self.gate[b])[:, :, None]
            out.append(0.75 * o.reshape(self.T, -1))
        return np.stack(out)

    def weights(self):
        from complexity_deep_b200.core.rotary import interleaved_tables
        dp, kp, vp, rp = _up(self.dim), _up(self.rank), _up(self.vdim), _up(self.rot)
        uk, uv = torch.zeros(self.H, dp, kp), torch.zeros(self.H, vp, kp)
        uk[:, :self.dim, :self.rank], uv[:, :self.vdim, :self.rank] = torch.tensor(self.uk), torch.tensor(self.uv)
        d64 = -(-self.dim // 64) * 64
        dev = dict(dtype=self.dtype, device="cuda")
        expand = torch.cat([torch.nn.functional.pad(uk, (0, 0, 0, d64 - dp)).view(-1, kp), uv.view(-1, kp)]).to(**dev)
        cos, sin = interleaved_tables(self.T + 3, self.rot_dims, rp, self.base, "cuda")
        return {"norm": torch.nn.functional.pad(torch.tensor(self.norm), (0, kp - self.rank)).to(**dev),
                "expand": expand, "uk": uk.to(**dev), "uv": uv.to(**dev), "uk_t": uk.transpose(1, 2).contiguous().to(**dev),
                "cos": cos, "sin": sin}

    def new_cache(self, capacity=None):
        return torch.full((self.B, capacity or self.T + 5, _up(self.rank) + _up(self.rot)), 9.0, dtype=self.dtype,
                          device="cuda")                                        # stale contents

    def run(self, portions, cache=None, on_device=False):
        from complexity_deep_b200 import ops
        dp, kp, vp, rp = _up(self.dim), _up(self.rank), _up(self.vdim), _up(self.rot)
        cache = self.new_cache() if cache is None else cache
        w, at, outs = self.weights(), 0, []
        for n in portions:
            rows = []
            for b in range(self.B):
                q = self.q[b, at:at + n]
                q = torch.cat([_pad(q[:, :, :self.dim].reshape(n * self.H, -1), 1, dp),
                               _pad(q[:, :, self.dim:].reshape(n * self.H, -1), 1, rp)], 1).view(n, -1)
                kv = self.kv[b, at:at + n]
                rows.append(torch.cat([q, _pad(kv[:, :self.rank], 1, kp), _pad(kv[:, self.rank:], 1, rp),
                                       _pad(self.gate[b, at:at + n], 1, _up(self.H))], 1))
            buf = torch.cat(rows, 0).to(dtype=self.dtype, device="cuda").contiguous()
            a = self.H * (dp + rp)
            wide = torch.zeros(self.B * n, self.H * vp + 16, dtype=self.dtype, device="cuda")
            out = wide[:, 8:8 + self.H * vp]                # columns of a wider buffer
            pos = torch.tensor([at], dtype=torch.int32, device="cuda") if on_device else None
            ops.latent_attention_({"q": buf[:, :a], "kv": buf[:, a:a + kp + rp], "gate": buf[:, a + kp + rp:]}, out, w,
                                  cache, batch=self.B, seq_len=n, heads=self.H, dim=self.dim, rot=self.rot,
                                  rank=self.rank, vdim=self.vdim, scale=self.scale, eps=self.eps, out_scale=0.75,
                                  pos0=0 if on_device else at, pos_dev=pos)
            o = out.double().cpu().view(self.B, n, self.H, vp)
            assert vp == self.vdim or float(o[..., self.vdim:].abs().max()) == 0
            outs.append(o[..., :self.vdim].reshape(self.B, n, -1))
            at += n
        ops.status_fetch()
        return torch.cat(outs, 1).numpy()


LATENT_TOL = {BF: 2.5e-2, F32: 3e-5}
LATENT_SHAPES = [  # T, H, dim, rot, vdim, rank, B
    (150, 4, 24, 16, 40, 48, 2),
    (70, 3, 10, 6, 9, 21, 1),
    (290, 6, 128, 64, 128, 256, 1),
    (131, 5, 64, 32, 96, 160, 2),
    (200, 16, 64, 64, 64, 512, 1),
    (140, 2, 48, 20, 112, 72, 3),
    (90, 24, 16, 16, 16, 32, 1),
    (80, 1, 200, 72, 144, 40, 1),
    (84, 2, 24, 24, 24, 680, 1),
    (100, 40, 32, 32, 64, 128, 1),
]


@pytest.mark.parametrize("dtype", [BF, F32], ids=["bf16", "fp32"])
@pytest.mark.parametrize("shape", LATENT_SHAPES)
def test_latent_attention_whole_portions_and_decode(shape, dtype):
    m = Latent(dtype, *shape[:6], B=shape[6], seed=shape[0])
    T, ref = shape[0], m.reference()
    for portions in ([T], _cuts(T, 1), [2] * (T // 2) + [1] * (T % 2), [T - 9] + [1] * 9, [T - 66, 66], [64, T - 64]):
        assert _rel(m.run(portions), ref) <= LATENT_TOL[dtype], portions
    if T <= 100:
        assert _rel(m.run([1] * T), ref) <= LATENT_TOL[dtype]
    assert _rel(m.run([1] * 40 + [T - 40]), ref) <= LATENT_TOL[dtype]
    got = m.run([1] * 60, on_device=True)
    assert _rel(got, ref[:, :60]) <= LATENT_TOL[dtype]


def test_part_of_the_rotated_elements_turns():
    m = Latent(F32, 60, 2, 16, 24, 16, 32, rot_dims=10, seed=3)
    assert _rel(m.run([37] + [1] * 23), m.reference()) <= LATENT_TOL[F32]


@pytest.mark.parametrize("dtype", [BF, F32], ids=["bf16", "fp32"])
@pytest.mark.parametrize("part", ["latent", "rotated"])
def test_one_key_stands_out(part, dtype):
    """A query finds one key among hundreds by its latent or by its rotated part: the first token, tile
    borders, its own token and the one before; as part of a prompt, of a portion, and decoded."""
    T, i, H, dim, rot, rank = 420, 400, 3, 64, 32, 96
    for j in (0, 1, 63, 64, 127, 128, 255, 256, i - 1, i):
        m = Latent(dtype, T, H, dim, rot, 48, rank, seed=j, scale=0.05)
        m.q *= 0.1
        rng = np.random.default_rng(7)
        if part == "latent":
            m.kv[0, :, rank:] *= 0.1
            u = rng.standard_normal(rank)
            m.kv[0, j, :rank] = _round(u, dtype)
            lat = ro.rms(m.kv[0, j, :rank], m.eps) * m.norm
            m.q[0, i, :, :dim] = _round(np.einsum("hdr,r->hd", m.uk, lat) * 6, dtype)
        else:
            m.kv[0, :, rank:] *= 0.1
            u = np.sign(rng.standard_normal(rot)) * 4
            m.kv[0, j, rank:] = u
            # the query's rotated part is chosen so that after its rotation it points at the rotated key
            back = ro.rotate(ro.rotate(u, j, rot, m.base), -i, rot, m.base)
            m.q[0, i, :, dim:] = _round(np.tile(back, (H, 1)), dtype)
        ref = m.reference()
        lost = Latent(dtype, T, H, dim, rot, 48, rank, seed=j, scale=0.05)
        lost.__dict__.update(q=m.q, kv=np.where(np.arange(T)[None, :, None] == j, -0.5 * m.kv, m.kv))
        assert _rel(lost.reference()[:, i], ref[:, i]) > 0.3            # the reference itself shows the key
        cuts = ([T], [i] + [1] * (T - i), [i - 1, 2, T - i - 1], [i - 70, T - i + 70])
        if j + 1 < T:
            cuts += ([j + 1, T - j - 1],)
        for portions in cuts:
            got = m.run(portions)
            assert _rel(got[:, i], ref[:, i]) <= LATENT_TOL[dtype], (j, portions)
            assert _rel(got, ref) <= LATENT_TOL[dtype], (j, portions)


def test_latent_cache_is_reused_without_traces():
    a, b = Latent(BF, 150, 4, 64, 32, 64, 128, seed=1), Latent(BF, 90, 4, 64, 32, 64, 128, seed=2)
    cache = a.new_cache(160)
    a.run([100] + [1] * 50, cache)
    used = b.run([2, 13, 65] + [1] * 10, cache)
    assert np.array_equal(used, b.run([2, 13, 65] + [1] * 10, b.new_cache(160)))


def test_long_latent_decoding():
    m = Latent(BF, 700, 8, 32, 16, 32, 64, seed=4)
    assert _rel(m.run([5] + [1] * 695), m.reference()) <= LATENT_TOL[BF]


def test_latent_attention_refuses_what_does_not_fit():
    m = Latent(F32, 20, 2, 16, 16, 16, 16)
    with pytest.raises(RuntimeError):
        m.run([20], m.new_cache(19))


# ------------------------------------------------------------------------------ delta rule
class Delta:
    def __init__(self, dtype, T, H, G, dk, dv, taps, rank, B=1, seed=0, bias=(-5.0, 1.0), a_log=(-2.0, 1.0)):
        self.__dict__.update(dtype=dtype, T=T, H=H, G=G, dk=dk, dv=dv, taps=taps, rank=rank, B=B)
        rng = np.random.default_rng(seed)
        r = lambda *s: _round(rng.standard_normal(s), dtype)
        self.q, self.k, self.v, self.b = r(B, T, G * dk), r(B, T, G * dk), r(B, T, H * dv), r(B, T, H)
        self.conv = {n: _round(rng.standard_normal((ch, taps)) * 0.6, dtype)
                     for n, ch in (("q", G * dk), ("k", G * dk), ("v", H * dv))}
        self.ia, self.ig = r(B, T, rank), r(B, T, rank)
        self.a2 = _round(rng.standard_normal((H * dk, rank)) * rank ** -0.5, dtype)
        self.g2 = _round(rng.standard_normal((H * dv, rank)) * rank ** -0.5, dtype)
        self.A_log, self.dt_bias = rng.uniform(*a_log, H), rng.uniform(*bias, H * dk)
        self.norm = _round(1 + 0.2 * rng.standard_normal(dv), dtype)
        self.eps = 1e-5

    def reference(self):
        outs, states = [], []
        for b in range(self.B):
            T, H, G, dk, dv = self.T, self.H, self.G, self.dk, self.dv
            q, k, v = (ro.silu(ro.short_conv(getattr(self, n)[b], self.conv[n])) for n in "qkv")
            q, k = ro.unit(q.reshape(T, G, dk)) * dk ** -0.5, ro.unit(k.reshape(T, G, dk))
            q, k = np.repeat(q, H // G, axis=1), np.repeat(k, H // G, axis=1)
            g = ro.channel_decay(self.ia[b], {"a1": np.eye(self.rank), "a2": self.a2, "dt_bias": self.dt_bias,
                                              "A_log": self.A_log}, H)
            o, S = ro.delta_recurrence(q, k, v.reshape(T, H, dv), g, ro.sigmoid(self.b[b]))
            y = (ro.rms(o, self.eps) * self.norm).reshape(T, -1) * ro.sigmoid(self.ig[b] @ self.g2.T)
            outs.append(0.75 * y)
            states.append(S)
        return np.stack(outs), np.stack(states)

    def carried(self):
        kp, vp = _up(self.dk), _up(self.dv)
        C = 2 * self.G * kp + self.H * vp
        return (torch.full((self.B, self.taps, C), 5.0, dtype=self.dtype, device="cuda"),       # stale contents
                torch.zeros(self.B, self.H, kp, vp, dtype=F32, device="cuda"))

    def run(self, portions, carried=None, on_device=False):
        from complexity_deep_b200 import ops
        dev = dict(dtype=self.dtype, device="cuda")
        kp, vp, rp = _up(self.dk), _up(self.dv), _up(self.rank)
        ring, state = carried or self.carried()
        inner = torch.zeros(self.H * (kp + vp), 2 * rp, dtype=torch.float64)
        inner[:self.H * kp].view(self.H, kp, -1)[:, :self.dk, :self.rank] = torch.tensor(self.a2).view(self.H, self.dk, -1)
        inner[self.H * kp:].view(self.H, vp, -1)[:, :self.dv, rp:rp + self.rank] = torch.tensor(self.g2).view(self.H, self.dv, -1)
        taps = torch.cat([_pad(self.conv["q"].T, self.G, kp), _pad(self.conv["k"].T, self.G, kp),
                          _pad(self.conv["v"].T, self.H, vp)], 1)
        w = {"inner": inner.to(**dev), "taps": taps.to(**dev).contiguous(),
             "rate": torch.tensor(np.exp(self.A_log), dtype=F32, device="cuda"),
             "dt_bias": _pad(self.dt_bias[None], self.H, kp)[0].to(dtype=F32, device="cuda"),
             "norm": torch.nn.functional.pad(torch.tensor(self.norm), (0, vp - self.dv)).to(**dev)}
        at, outs = 0, []
        for n in portions:
            s = slice(at, at + n)
            rows = [torch.cat([_pad(self.q[b, s], self.G, kp), _pad(self.k[b, s], self.G, kp),
                               _pad(self.v[b, s], self.H, vp), _pad(self.b[b, s], 1, _up(self.H)),
                               _pad(self.ia[b, s], 1, rp), _pad(self.ig[b, s], 1, rp)], 1) for b in range(self.B)]
            buf = torch.cat(rows, 0).to(**dev).contiguous()
            cut = np.cumsum([0, self.G * kp, self.G * kp, self.H * vp, _up(self.H), 2 * rp])
            proj = {name: buf[:, cut[x]:cut[x + 1]] for x, name in enumerate(("q", "k", "v", "b", "inner"))}
            wide = torch.zeros(self.B * n, self.H * vp + 16, **dev)
            out = wide[:, 8:8 + self.H * vp]
            pos = torch.tensor([at], dtype=torch.int32, device="cuda") if on_device else None
            ops.delta_attention_(proj, out, w, ring, state, batch=self.B, seq_len=n, heads=self.H, kv_heads=self.G,
                                 dim=self.dk, vdim=self.dv, eps=self.eps, out_scale=0.75, pos0=0 if on_device else at,
                                 pos_dev=pos)
            o = out.double().cpu().view(self.B, n, self.H, vp)
            assert vp == self.dv or float(o[..., self.dv:].abs().max()) == 0
            outs.append(o[..., :self.dv].reshape(self.B, n, -1))
            at += n
        ops.status_fetch()
        return torch.cat(outs, 1).numpy(), state[:, :, :self.dk, :self.dv].double().cpu().numpy()


# bf16: the results of convolution and silu are stored in bf16; a head whose output is small before its
# norm amplifies that
DELTA_TOL = {BF: 4e-2, F32: 1e-4}
STATE_TOL = {BF: 1e-2, F32: 2e-5}
DELTA_SHAPES = [  # T, H, G, dk, dv, taps, rank, B
    (150, 4, 2, 24, 40, 3, 8, 2),
    (97, 3, 1, 7, 9, 1, 5, 1),
    (200, 4, 4, 128, 128, 4, 32, 1),
    (130, 6, 3, 64, 80, 2, 24, 2),
    (193, 2, 2, 32, 64, 4, 16, 1),
    (70, 2, 1, 96, 200, 6, 16, 1),
    (90, 1, 1, 200, 48, 4, 16, 1),
    (66, 2, 2, 128, 32, 12, 16, 1),
    (65, 2, 1, 16, 16, 4, 130, 1),
    (48, 1, 1, 320, 264, 4, 16, 1),
]


@pytest.mark.parametrize("dtype", [BF, F32], ids=["bf16", "fp32"])
@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_delta_rule_whole_portions_and_decode(shape, dtype):
    m = Delta(dtype, *shape[:7], B=shape[7], seed=shape[0])
    T = shape[0]
    ref, state = m.reference()
    for portions in ([T], _cuts(T, 3), [2] * (T // 2) + [1] * (T % 2), [T - 20] + [1] * 20, [17, T - 17], [1] * T):
        got, s = m.run(portions)
        assert _rel(got, ref) <= DELTA_TOL[dtype], portions
        assert _rel(s.reshape(1, -1), state.reshape(1, -1)) <= STATE_TOL[dtype], portions
    got, s = m.run([1] * T, on_device=True)
    assert _rel(got, ref) <= DELTA_TOL[dtype]


@pytest.mark.parametrize("dtype", [BF, F32], ids=["bf16", "fp32"])
def test_delta_rule_with_fast_and_mixed_decays(dtype):
    """Decays from almost none to so fast that the cumulative one leaves the fp32 range within a few
    tokens, side by side in one head; and every channel fast."""
    for bias in (np.linspace(-14.0, 60.0, 2 * 48), np.full(2 * 48, 70.0), np.full(2 * 48, -14.0)):
        m = Delta(dtype, 190, 2, 2, 48, 32, 4, 8, seed=9, a_log=(1.0, 2.5))
        m.dt_bias = bias
        ref, state = m.reference()
        for portions in ([190], [100, 90], [17, 40, 133], [1] * 190):
            got, s = m.run(portions)
            assert np.isfinite(got).all() and np.isfinite(s).all()
            assert _rel(got, ref) <= DELTA_TOL[dtype], portions
            assert _rel(s.reshape(1, -1), state.reshape(1, -1)) <= STATE_TOL[dtype]


@pytest.mark.parametrize("dtype", [BF, F32], ids=["bf16", "fp32"])
def test_delta_rule_remembers_a_far_key(dtype):
    """Almost no decay, and keys in a subspace that leaves one written direction alone: queries hundreds
    of tokens later find it, whatever the cut; without the carried state they would not."""
    T, dk, dv = 500, 64, 32
    m = Delta(dtype, T, 2, 2, dk, dv, 1, 8, seed=11, bias=(-14.0, -12.0))
    m.conv = {n: np.ones_like(v) for n, v in m.conv.items()}
    half = np.arange(2 * dk) % dk < dk // 2
    m.k = np.where(half[None, None], -30.0, m.k)                 # silu(-30) = 0: the first half stays unwritten
    m.k[0, 3] = np.where(half, 4.0, -30.0)
    m.b[0, 3] = 4.0
    m.q[0, 480:] = np.where(half, 4.0, -30.0)
    m.v[0, 3] = _round(3 * np.sign(np.random.default_rng(2).standard_normal(2 * dv)), dtype)
    ref, _ = m.reference()
    lost = Delta(dtype, T, 2, 2, dk, dv, 1, 8, seed=11, bias=(-14.0, -12.0))
    lost.__dict__.update(m.__dict__, v=np.where(np.arange(T)[None, :, None] == 3, -m.v, m.v))
    assert _rel(lost.reference()[0][:, 480:], ref[:, 480:]) > 0.3
    for portions in ([T], [2, 2, T - 4], [400, 64, 16] + [1] * 20, [100] * 5):
        assert _rel(m.run(portions)[0][:, 480:], ref[:, 480:]) <= DELTA_TOL[dtype], portions


def test_delta_state_overwrites_a_repeated_key():
    """Writing the same key again replaces its value: the read-out is the last value alone."""
    m = Delta(F32, 40, 1, 1, 16, 16, 1, 8, seed=1, bias=(-20.0, -19.0))
    m.conv = {n: np.ones_like(v) for n, v in m.conv.items()}
    m.k[:] = m.k[0, 0]
    m.b[:] = 30.0                                                # beta = 1
    m.q[:] = m.k
    got, s = m.run([11, 29])
    ref, state = m.reference()
    v = ro.silu(m.v[0, -1])
    read = np.einsum("hcd,c->hd", s[0], ro.unit(ro.silu(m.k[0, 0])))[0]
    assert np.abs(read - v).max() <= 1e-4 and _rel(got, ref) <= DELTA_TOL[F32]


def test_delta_ring_and_state_are_reused_without_traces():
    a, b = Delta(BF, 100, 4, 2, 32, 48, 4, 8, seed=1), Delta(BF, 47, 4, 2, 32, 48, 4, 8, seed=2)
    used = a.carried()
    a.run([60] + [1] * 40, used)
    used[1].zero_()
    got, s = b.run([2, 20] + [1] * 25, used)
    want, s2 = b.run([2, 20] + [1] * 25)
    assert np.array_equal(got, want) and np.array_equal(s, s2)


def test_long_delta_decoding():
    m = Delta(F32, 400, 2, 1, 16, 16, 4, 8, seed=4)
    assert _rel(m.run([3] + [1] * 397)[0], m.reference()[0]) <= DELTA_TOL[F32]


# ------------------------------------------------------------------------------ routing and experts
@pytest.mark.parametrize("E,top,groups,keep", [(6, 3, 3, 2), (5, 1, 1, 1), (128, 8, 8, 3), (64, 6, 64, 9), (33, 33, 1, 1),
                                               (40, 4, 2, 1), (96, 10, 4, 4)])
def test_choice_of_experts(E, top, groups, keep):
    from complexity_deep_b200 import ops
    rng = np.random.default_rng(E)
    ld = -(-E // 8) * 8
    logits = np.full((301, ld), 50.0, dtype=np.float32)                # the padding must not be chosen
    logits[:, :E] = rng.standard_normal((301, E)) * 3
    logits[0, :E] = 0.0                                                # ties: the lower index first
    ids, weights = ops.route_top(torch.tensor(logits, device="cuda"), E, top, groups, keep)
    for t in range(301):
        want, w = ro.choose_experts(logits[t, :E].astype(np.float64), top, groups, keep)
        assert ids[t].tolist() == list(want), t
        assert np.abs(weights[t].cpu().numpy() - w).max() <= 1e-6


@pytest.mark.parametrize("T,width,ff,E,top,groups,keep", [(1, 72, 20, 6, 3, 3, 2), (37, 40, 29, 5, 1, 1, 1),
                                                         (300, 128, 64, 16, 4, 4, 2), (33, 264, 136, 64, 8, 8, 4),
                                                         (2500, 64, 32, 8, 2, 2, 1)])
def test_routed_experts(T, width, ff, E, top, groups, keep):
    from complexity_deep_b200 import ops
    from complexity_deep_b200.core.padding import pad_rows
    from complexity_deep_b200.core.routed_experts import RoutedExperts
    g = torch.Generator().manual_seed(T)
    mlp = RoutedExperts(width, ff, E, top, 1.3, groups, keep)
    for p in mlp.parameters():
        p.data = (torch.randn(p.shape, generator=g) * 2 / p.shape[-1] ** 0.5).to(BF).float()
    x = torch.randn(T, width, generator=g).to(BF)
    W = {"router": mlp.router.weight.detach().double().numpy()}
    for e in range(E):
        for n in ("gate", "up", "down"):
            W[f"e{e}.{n}"] = getattr(mlp, n + "_proj")[e].detach().double().numpy()
    router = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}}
    want = 0.6 * ro.mixture(x.double().numpy(), W, {"router": router, "expert": {"limit": 1.3}})
    ldx = -(-width // 8) * 8
    start = torch.randn(T, ldx, generator=g)
    for dtype in (F32, BF):
        m = mlp.to(device="cuda", dtype=dtype)
        out = m.run(pad_rows(x, T, ldx).to(device="cuda", dtype=dtype), start.cuda(), scale=0.6).cpu()
        got = (out - start)[:, :width].double().numpy()
        assert _rel(got, want) <= (5e-5 if dtype == F32 else 2e-2)
    ops.status_fetch()


# ------------------------------------------------------------------------------ fp32 stream
@pytest.mark.parametrize("T,width,ff", [(1, 40, 24), (65, 264, 100), (2100, 128, 512)])
def test_squared_relu(T, width, ff):
    from complexity_deep_b200.core.mlp import SquaredReLU
    g = torch.Generator().manual_seed(T)
    mlp = SquaredReLU(width, ff)
    for p in mlp.parameters():
        p.data = (torch.randn(p.shape, generator=g) / p.shape[1] ** 0.5).to(BF).float()
    x = torch.randn(T, width, generator=g).to(BF)
    W = [p.detach().double().numpy() for p in (mlp.up_proj.weight, mlp.down_proj.weight)]
    want = 1.7 * ro.squared_relu(x.double().numpy(), *W)
    for dtype in (F32, BF):
        m = mlp.to(device="cuda", dtype=dtype)
        got = m.run(x.to(device="cuda", dtype=dtype), torch.zeros(T, width, device="cuda"), scale=1.7).double().cpu().numpy()
        assert _rel(got, want) <= (3e-5 if dtype == F32 else 1.5e-2)


@pytest.mark.parametrize("T,W", [(1, 20), (37, 328), (5, 1500), (9, 2300)])
def test_layer_norm_and_positions(T, W):
    from complexity_deep_b200 import ops
    from complexity_deep_b200.core.normalization import StreamNorm
    from complexity_deep_b200.core.padding import pad_rows
    g = torch.Generator().manual_seed(W)
    ldx = -(-W // 8) * 8
    table, pos = torch.randn(50, W, generator=g).to(BF), (torch.randn(90, W, generator=g) + 3.0).to(BF)
    ids = torch.randint(0, 50, (2, T), generator=g)
    want = np.concatenate([ro.embed(i.numpy(), table.double().numpy(), pos.double().numpy()[11:]) for i in ids])
    for dtype in (BF, F32):
        t, p = (pad_rows(a, -(-a.shape[0] // 8) * 8, ldx).to(dtype).cuda() for a in (table, pos))
        x = ops.embed_positions(ids.cuda(), t, p, W, ldx, T, 11)
        on_dev = ops.embed_positions(ids.cuda(), t, p, W, ldx, T, 0, torch.tensor([11], dtype=torch.int32, device="cuda"))
        assert torch.equal(x, on_dev) and float(x[:, W:].abs().sum()) == 0
        assert np.abs(x[:, :W].double().cpu().numpy() - want).max() <= 1e-6
        norm = StreamNorm(W, 1e-3, centred=True)
        norm.weight.data = (1 + torch.randn(W, generator=g) * 0.3).to(BF).float()
        ref = ro.layer_norm(want, norm.weight.detach().double().numpy(), 1e-3)
        got = norm.to(device="cuda", dtype=dtype)(x)
        assert got.dtype == dtype and float(got[:, W:].float().abs().sum()) == 0
        assert _rel(got[:, :W].double().cpu().numpy(), ref) <= (3e-3 if dtype == BF else 2e-6)
    with pytest.raises(RuntimeError):
        ops.embed_positions(ids.cuda(), t, p, W, ldx, T, p.shape[0] - T + 1)


@pytest.mark.parametrize("T,K,N", [(3, 64, 40), (130, 24, 328), (2300, 128, 768)])
def test_products_of_columns_with_scale(T, K, N):
    """x is a column slice of a wider buffer; the result scaled, added to the stream, or squared relu."""
    from complexity_deep_b200 import ops
    g = torch.Generator().manual_seed(T + N)
    wide = torch.randn(T, K + 48, generator=g).to(BF)
    w = (torch.randn(N, K, generator=g) / K ** 0.5).to(BF)
    r = torch.randn(T, N, generator=g)
    x = wide[:, 16:16 + K]
    y = x.double() @ w.double().t()
    for dtype in (BF, F32):
        xs = wide.to(device="cuda", dtype=dtype)[:, 16:16 + K]
        ws = w.to(device="cuda", dtype=dtype)
        got = ops.linear_to_f32(xs, ws, residual=r.cuda(), scale=-0.3)
        assert float((got.double().cpu() - (r.double() - 0.3 * y)).abs().max()) <= 2e-5
        sq = ops.project(xs, ws, act="relu2").double().cpu()
        assert float((sq - y.clamp(min=0) ** 2).abs().max()) <= (5e-3 if dtype == BF else 2e-5) * float((y ** 2).max())
    ops.status_fetch()
