"""Host side of the Rugedra model: configuration, checkpoint names and files, registry, states, command
line; and properties of the float64 restatement that the GPU tests rely on."""
import json

import numpy as np
import pytest
import torch

from oracle import rugedra_oracle as ro
from rugedra_cases import CASES, bf16_weights, tokens, write_checkpoint


@pytest.mark.parametrize("name", sorted(CASES))
def test_config_and_checkpoint_round_trip(name, tmp_path):
    from complexity_deep_b200.models import RugedraConfig, RugedraModel, model_class
    cfg, rank = CASES[name]
    assert RugedraConfig.from_dict(cfg).to_dict() == cfg
    assert model_class(cfg) is RugedraModel
    w = bf16_weights(cfg, rank)
    model = RugedraModel.from_pretrained(write_checkpoint(tmp_path / "a", cfg, w))
    params = dict(model.named_parameters())
    names = model.checkpoint_names()
    assert set(names) == set(params)
    for k, v in names.items():
        want = w[v] if isinstance(v, str) else np.stack([w[n] for n in v])
        assert np.array_equal(params[k].double().numpy(), want), v
    model.save_pretrained(tmp_path / "b")
    assert json.loads((tmp_path / "b" / "config.json").read_text()) == cfg
    again = RugedraModel.from_pretrained(str(tmp_path / "b"), dtype=torch.float32)
    for k, p in again.named_parameters():
        assert p.dtype == torch.float32 and torch.equal(p, params[k].float())


def test_wrong_checkpoints_and_configs_are_refused(tmp_path):
    from complexity_deep_b200.models import RugedraConfig, RugedraModel
    cfg, rank = CASES["odd"]
    w = bf16_weights(cfg, rank)
    for change in (lambda d: d.pop("l0.mlp.e5.up"), lambda d: d.update(extra=np.zeros(3)), lambda d: d.pop("l0.mix.a1"),
                   lambda d: d.update({"l1.mix.dkv": np.ones((51, 72))}), lambda d: d.update({"l0.mlp.e1.gate": np.ones((21, 72))})):
        bad = dict(w)
        change(bad)
        with pytest.raises(ValueError):
            RugedraModel.from_pretrained(write_checkpoint(tmp_path, cfg, bad))
    for layer, path, value in ((0, ("type",), "serial"), (0, ("mlp", "kind"), "routed")):
        broken = json.loads(json.dumps(cfg))
        d = broken["layers"][layer]
        for p in path[:-1]:
            d = d[p]
        d[path[-1]] = value
        with pytest.raises(ValueError):
            RugedraConfig.from_dict(broken)
    for layer, path, value in ((0, ("mixer", "kv_heads"), 3), (0, ("mlp", "router", "top"), 5), (1, ("mixer", "rot", "dims"), 14),
                               (4, ("mlp", "router", "groups", "count"), 4)):
        broken = json.loads(json.dumps(cfg))
        d = broken["layers"][layer]
        for p in path[:-1]:
            d = d[p]
        d[path[-1]] = value
        with pytest.raises(ValueError):
            with torch.device("meta"):
                RugedraModel(RugedraConfig.from_dict(broken))


def test_latent_state_grows_and_copies():
    from complexity_deep_b200.core.state import DecoderState, LatentState
    s = LatentState(2, 16, 1000, "cpu", torch.float32)
    s.rows[:, :256] = 7.0
    assert s.reserve(256) is s.rows and s.reserve(257).shape[1] == 512 and float(s.rows[:, :256].mean()) == 7.0
    assert s.reserve(1000).shape[1] == 1000
    with pytest.raises(RuntimeError):
        s.reserve(1001)
    fixed = LatentState(2, 16, 1000, "cpu", torch.float32, capacity=40)
    with pytest.raises(RuntimeError):
        fixed.reserve(41)
    a = DecoderState([{"mix": fixed}], 2, "cpu", 40)
    b = DecoderState([{"mix": s}], 2, "cpu")
    b.advance(30)
    address = fixed.rows.data_ptr()
    a.load(b)
    assert fixed.rows.data_ptr() == address and a.length == 30 and float(fixed.rows[:, :30].mean()) == 7.0
    b.advance(11)
    with pytest.raises(ValueError):
        a.load(b)


def test_padded_projections_keep_their_rows():
    from complexity_deep_b200.core.mixers import DeltaRule, LatentAttention
    m = LatentAttention(24, 3, 10, 6, 9, 21, 0.3, 6, 100.0, 50, 1e-5)
    q = dict(m.projections())["q"].view(3, 32, 24)
    w = m.q_proj.weight.detach().view(3, 16, 24)
    assert torch.equal(q[:, :10], w[:, :10]) and torch.equal(q[:, 16:22], w[:, 10:])
    assert float(q[:, 10:16].abs().sum()) == 0 and float(q[:, 22:].abs().sum()) == 0
    kv = dict(m.projections())["kv"]
    assert torch.equal(kv[:21], m.kv_proj.weight[:21]) and torch.equal(kv[32:38], m.kv_proj.weight[21:])
    k = m._weights()
    assert torch.equal(k["uk"], k["uk_t"].transpose(1, 2)) and k["cos"].shape == (50, 8)
    assert float(k["cos"][:, 3:].min()) == 1 and float(k["sin"][:, 3:].abs().max()) == 0
    d = DeltaRule(24, 4, 2, 7, 5, 3, 13, 9, 1e-5)
    torch.nn.init.normal_(d.q_conv)
    inner = d._weights()["inner"]
    x, y = torch.randn(13), torch.randn(9)
    both = torch.zeros(32)
    both[:13], both[16:25] = x, y
    z = inner @ both
    assert torch.allclose(z[:64].view(4, 16)[:, :7].reshape(-1), d.a2_proj.weight @ x, atol=1e-5)
    assert torch.allclose(z[64:].view(4, 16)[:, :5].reshape(-1), d.g2_proj.weight @ y, atol=1e-5)
    assert torch.equal(d._weights()["taps"][:, :7].t(), d.q_conv[:7])


def test_command_line_info(tmp_path, capsys):
    from complexity_deep_b200 import cli
    cfg, rank = CASES["ragged"]
    w = bf16_weights(cfg, rank)
    assert cli.main(["info", "--model", write_checkpoint(tmp_path, cfg, w)]) == 0
    info = json.loads(capsys.readouterr().out)
    assert info["architecture"] == "Rugedra" and info["layers"] == 3 and info["class"] == "RugedraModel"


# ------------------------------------------------------------------------------ the restatement
def test_restatement_rotation_depends_on_distances_only():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal(12), rng.standard_normal(12)
    a = ro.rotate(q, 9, 12, 100.0) @ ro.rotate(k, 4, 12, 100.0)
    assert np.allclose(a, ro.rotate(q, 105, 12, 100.0) @ ro.rotate(k, 100, 12, 100.0))
    assert np.allclose(ro.rotate(ro.rotate(q, 5, 12, 100.0), -5, 12, 100.0), q)
    part = ro.rotate(q, 9, 4, 100.0)
    assert np.array_equal(part[4:], q[4:]) and not np.allclose(part[:4], q[:4])


def test_restatement_of_the_absorbed_scores():
    """(uk c) . q = (uk^T q) . c: the form that never expands the latent gives the same result."""
    rng = np.random.default_rng(1)
    T, H, d, r, dv, R = 9, 2, 4, 4, 3, 6
    q, lat, key = rng.standard_normal((T, H, d + r)), rng.standard_normal((T, R)), rng.standard_normal((T, r))
    uk, uv = rng.standard_normal((H, d, R)), rng.standard_normal((H, dv, R))
    c = {"heads": H, "dim": d, "vdim": dv, "scale": 0.4, "rot": {"dims": r, "base": 50.0}}
    out = ro.latent_heads(q, lat, key, uk.reshape(-1, R), uv.reshape(-1, R), c)
    qr = np.stack([ro.rotate(q[p, :, d:], p, r, 50.0) for p in range(T)])
    for n in range(H):
        s = (q[:, n, :d] @ uk[n] @ lat.T + qr[:, n] @ key.T) * 0.4
        assert np.allclose(out[:, n], (ro.causal_softmax(s) @ lat) @ uv[n].T)


def test_restatement_recurrence_splits_anywhere_and_solves_for_its_keys():
    rng = np.random.default_rng(2)
    q, k, v = rng.standard_normal((12, 2, 6)), ro.unit(rng.standard_normal((12, 2, 6))), rng.standard_normal((12, 2, 5))
    g, beta = rng.uniform(0.3, 1.0, (12, 2, 6)), rng.uniform(0.0, 1.0, (12, 2))
    o, S = ro.delta_recurrence(q, k, v, g, beta)
    o1, S1 = ro.delta_recurrence(q[:5], k[:5], v[:5], g[:5], beta[:5])
    o2, S2 = ro.delta_recurrence(q[5:], k[5:], v[5:], g[5:], beta[5:], S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    # without decay and with beta 1, reading with the last key gives the last value
    o, S = ro.delta_recurrence(k, k, v, np.ones_like(g), np.ones_like(beta))
    assert np.allclose(o, v, atol=1e-5)


def test_restatement_convolution_and_routing():
    x = np.arange(1.0, 6.0)[:, None]
    assert np.allclose(ro.short_conv(x, np.array([[2.0, 3.0]]))[:, 0], [3, 8, 13, 18, 23])
    assert np.allclose(ro.short_conv(x, np.array([[5.0]]))[:, 0], 5 * x[:, 0])
    logits = np.array([5.0, 0.0, 4.0, 4.5, 0.1, 0.2])
    ids, w = ro.choose_experts(logits, 2, 3, 1)
    assert list(ids) == [0, 1] and np.isclose(w.sum(), 1)                 # the best group holds the best expert
    ids, w = ro.choose_experts(logits, 2, 1, 1)
    assert list(ids) == [0, 3] and np.isclose(w[0] / w[1], np.exp(0.5))
    assert list(ro.choose_experts(logits, 3, 3, 2)[0]) == [0, 3, 2]


def test_restatement_is_causal_and_every_tensor_counts():
    cfg, rank = CASES["odd"]
    w = bf16_weights(cfg, rank)
    ids = tokens(cfg, 40)
    base = ro.forward(w, cfg, ids)
    changed = ids.copy()
    changed[30] = (changed[30] + 1) % cfg["vocab"]
    assert np.allclose(ro.forward(w, cfg, changed)[:30], base[:30])
    scale = base.std()
    for name in w:
        if name.startswith(("l0.mix", "l1")) or "." not in name or name == "final.norm":
            other = dict(w)
            other[name] = w[name] * 1.5 + 0.05
            assert np.abs(ro.forward(other, cfg, ids) - base).max() > 1e-3 * scale, name
