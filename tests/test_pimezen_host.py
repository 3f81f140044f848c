"""Host side of the Pimezen model: configuration, checkpoint names and files, registry, states,
sampling, command line; and properties of the float64 restatement that the GPU tests rely on."""
import json

import numpy as np
import pytest
import torch

from oracle import pimezen_oracle as po
from pimezen_cases import CASES, bf16_weights, tokens, write_checkpoint


@pytest.mark.parametrize("name", sorted(CASES))
def test_config_and_checkpoint_round_trip(name, tmp_path):
    from complexity_deep_b200.models import PimezenConfig, PimezenModel, model_class
    cfg, rank = CASES[name]
    assert PimezenConfig.from_dict(cfg).to_dict() == cfg
    assert model_class(cfg) is PimezenModel
    w = bf16_weights(cfg, rank)
    model = PimezenModel.from_pretrained(write_checkpoint(tmp_path / "a", cfg, w))
    names = model.checkpoint_names()
    params = dict(model.named_parameters())
    assert set(names) == set(params) and set(names.values()) == set(w)
    for k, v in names.items():
        assert np.array_equal(params[k].double().numpy(), w[v]), v
    model.save_pretrained(tmp_path / "b")
    again = PimezenModel.from_pretrained(str(tmp_path / "b"), dtype=torch.float32)
    assert json.loads((tmp_path / "b" / "config.json").read_text()) == cfg
    for k, p in again.named_parameters():
        assert p.dtype == torch.float32 and torch.equal(p, params[k].float())


def test_wrong_checkpoints_and_configs_are_refused(tmp_path):
    from complexity_deep_b200.models import PimezenConfig, PimezenModel, model_class
    cfg, rank = CASES["odd"]
    w = bf16_weights(cfg, rank)
    for change in (lambda d: d.pop("l1.mix.left.talk"), lambda d: d.update(extra=np.zeros(3)),
                   lambda d: d.update({"l0.ls1": np.ones(8)})):
        bad = dict(w)
        change(bad)
        with pytest.raises(ValueError):
            PimezenModel.from_pretrained(write_checkpoint(tmp_path, cfg, bad))
    for path, value in ((("type",), "serial"), (("mlp", "kind"), "routed")):
        broken = json.loads(json.dumps(cfg))
        d = broken["layers"][0]
        for p in path[:-1]:
            d = d[p]
        d[path[-1]] = value
        with pytest.raises(ValueError):
            PimezenConfig.from_dict(broken)
    with pytest.raises(ValueError):
        model_class({"architecture": "Unknown"})


def test_registry_defaults_to_the_reference_model():
    from complexity_deep_b200.models import ComplexityModel, model_class
    assert model_class({"hidden_size": 64}) is ComplexityModel


def test_safetensors_files(tmp_path):
    from complexity_deep_b200.models.weights import read_safetensors, write_safetensors
    t = {"a": torch.randn(3, 5).to(torch.bfloat16), "b": torch.arange(7, dtype=torch.int32),
         "c": torch.randn(2, 2, 3), "d": torch.zeros(0, 4), "e": torch.arange(3, dtype=torch.uint8),
         "f": torch.randn(3)}
    write_safetensors(tmp_path / "x", t)
    back = read_safetensors(tmp_path / "x")
    assert set(back) == set(t) and all(torch.equal(back[k], v) and back[k].dtype == v.dtype for k, v in t.items())
    data = (tmp_path / "x").read_bytes()
    (tmp_path / "cut").write_bytes(data[:-4])
    with pytest.raises(ValueError):
        read_safetensors(tmp_path / "cut")


def test_padded_heads_keep_their_rows():
    from complexity_deep_b200.core.padding import pad_heads, pad_rows, pad_vector
    w = torch.randn(3 * 5, 7)
    p = pad_heads(w, 3, 8).view(3, 8, 7)
    assert torch.equal(p[:, :5].reshape(15, 7), w) and float(p[:, 5:].abs().sum()) == 0
    assert pad_heads(w, 3, 5) is w and pad_rows(w, 15) is w
    assert pad_vector(torch.ones(3), 8).tolist() == [1, 1, 1, 0, 0, 0, 0, 0]


def test_state_pool_reuses_states():
    from complexity_deep_b200.core.state import DecoderState, RecurrentState, StatePool, WindowState
    made = []

    def make():
        s = DecoderState([{"left": WindowState(1, 4, 2, 1, 16, 16, "cpu", torch.float32),
                           "right": RecurrentState(1, 1, 16, 16, "cpu")}], 1, "cpu")
        made.append(s)
        return s

    pool = StatePool(make)
    a = pool.get("a")
    assert pool.get("a") is a and len(pool) == 1
    a.layers[0]["right"].s.fill_(3.0)
    a.advance(5)
    b = pool.get("b")
    assert b is not a and b.length == 0
    pool.release("a")
    pool.release("never")
    c = pool.get("c")
    assert c is a and c.length == 0 and float(c.layers[0]["right"].s.abs().sum()) == 0 and len(made) == 2
    d = make()
    b.advance(3)
    b.layers[0]["right"].s.fill_(2.0)
    d.load(b)
    assert d.length == 3 and int(d.position) == 3 and float(d.layers[0]["right"].s.mean()) == 2.0
    with pytest.raises(ValueError):
        d.set_length(1)


def test_sampling_rules():
    from complexity_deep_b200.models.generation import sample_next
    logits = torch.tensor([[1.0, 4.0, 3.0, -2.0], [9.0, 0.0, 0.0, 0.0]])
    assert sample_next(logits, do_sample=False).tolist() == [[1], [0]]
    torch.manual_seed(0)
    seen = {tuple(sample_next(logits, top_k=2, top_p=1.0).flatten().tolist()) for _ in range(200)}
    assert seen <= {(1, 0), (2, 0), (1, 1), (1, 2), (1, 3), (2, 1), (2, 2), (2, 3)} and {(1, 0), (2, 0)} <= seen
    assert {tuple(sample_next(logits, top_k=0, top_p=0.5).flatten().tolist()) for _ in range(50)} == {(1, 0)}
    sample_next(logits, top_k=50)                     # more than the vocabulary holds


def test_command_line_parsing(tmp_path, capsys):
    from complexity_deep_b200 import cli
    from complexity_deep_b200.trace import _parser
    assert cli.parse_prompts(["1,2,3", "4,5,6"]) == [[1, 2, 3], [4, 5, 6]]
    with pytest.raises(SystemExit):
        cli.parse_prompts(["1,2", "3"])
    cfg, rank = CASES["ragged"]
    path = write_checkpoint(tmp_path, cfg, bf16_weights(cfg, rank))
    assert cli.main(["info", "--model", path]) == 0
    info = json.loads(capsys.readouterr().out)
    assert info["architecture"] == "Pimezen" and info["layers"] == 2
    a = _parser().parse_args(["--model", "m", "--dtype", "float32", "--out", "o", "--max-tokens", "9"])
    assert a.max_tokens == 9
    with pytest.raises(SystemExit):
        _parser().parse_args(["--model", "m", "--dtype", "float16", "--out", "o"])


# ------------------------------------------------------------------------------ the restatement
def test_restatement_window_and_softmax():
    assert [po.window_visible(10, j, 4, 2) for j in (0, 1, 2, 6, 7, 10, 11)] == [True, True, False, False, True, True,
                                                                               False]
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 1, 4))
    w = po.softmax_weights(q, k, 0.5, np.zeros(2), np.ones(2), 3, 1)
    assert np.allclose(w.sum(-1), 1) and w[0, 8, 0] > 0 and w[0, 8, 5] == 0 and w[0, 8, 6] > 0
    # without a bias and with everything visible this is ordinary causal softmax attention
    full = po.softmax_weights(q, k, 0.5, np.zeros(2), np.ones(2), 99, 0)
    s = np.einsum("ihd,jd->hij", q, k[:, 0]) * 0.5
    s = np.where(np.tri(9, dtype=bool), s, -np.inf)
    e = np.exp(s - s.max(-1, keepdims=True))
    assert np.allclose(full, e / e.sum(-1, keepdims=True))
    # the bias weakens far keys
    far = po.softmax_weights(q, k, 0.5, np.array([2.0, 2.0]), np.ones(2), 99, 0)
    assert far[0, 8, 0] < full[0, 8, 0]


def test_restatement_recurrence_splits_anywhere():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((12, 2, 3)), rng.standard_normal((12, 2, 3)), rng.standard_normal((12, 2, 5))
    alpha = rng.uniform(0.2, 1.0, (12, 2, 3))
    o, S = po.linear_recurrence(q, k, v, alpha)
    o1, S1 = po.linear_recurrence(q[:5], k[:5], v[:5], alpha[:5])
    o2, S2 = po.linear_recurrence(q[5:], k[5:], v[5:], alpha[5:], S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    # closed form of the last output
    cum = np.cumprod(alpha[::-1], axis=0)[::-1]
    decay = np.concatenate([cum[1:], np.ones((1, 2, 3))])
    want = np.einsum("hc,thc,thd->hd", q[-1], k * decay, v)
    assert np.allclose(o[-1], want)


def test_restatement_is_causal_and_every_mechanism_counts():
    cfg, rank = CASES["odd"]
    w = bf16_weights(cfg, rank)
    ids = tokens(cfg, 40)
    base = po.forward(w, cfg, ids)
    changed = ids.copy()
    changed[30] = (changed[30] + 1) % cfg["vocab"]
    assert np.array_equal(po.forward(w, cfg, changed)[:30], base[:30])
    scale = base.std()
    for name in w:
        if name.startswith("l1") or name in ("final.norm", "embed"):
            other = dict(w)
            other[name] = w[name] * 1.5 + 0.05
            assert np.abs(po.forward(other, cfg, ids) - base).max() > 1e-3 * scale, name
