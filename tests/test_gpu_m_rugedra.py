"""The Rugedra model through the framework's own entry points (loading, forward with a carried
state, generate, DecodeGraph, PrefillGraph, trace replay) against the float64 restatement, in fp32
and bf16, on small models of several sizes."""
import json
import subprocess

import numpy as np
import pytest
import torch

from conftest import ROOT
from oracle import rugedra_oracle as ro
from rugedra_cases import CASES, bf16_weights, tokens, write_checkpoint

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
# rms error of a position's logits relative to their overall rms.  bf16: a token whose router scores are
# close may take another expert, and a head whose output is small before its norm amplifies rounding;
# the bulk is far below.
TOL = {F32: 1e-4, BF: 0.6}
BULK = {F32: 1e-5, BF: 0.04}

_cache = {}


def _model(name, dtype, tmp_path_factory):
    if (name, dtype) not in _cache:
        from complexity_deep_b200 import load_model
        cfg, rank = CASES[name]
        w = bf16_weights(cfg, rank, seed=3)
        path = write_checkpoint(tmp_path_factory.mktemp(name), cfg, w)
        _cache[name, dtype] = (cfg, w, path, load_model(path, "cuda", dtype))
    return _cache[name, dtype]


def _reference(name, cfg, w, ids):
    key = (name, tuple(int(t) for t in ids))
    if key not in _cache:
        _cache[key] = ro.forward(w, cfg, ids)
    return _cache[key]


def _check(got, want, dtype, what=""):
    d = got - want
    d = np.sqrt(((d - d.mean(-1, keepdims=True)) ** 2).mean(-1)) / want.std()
    assert np.isfinite(got).all()
    assert d.max() <= TOL[dtype] and np.median(d) <= BULK[dtype], (what, d.max(), np.median(d))


def _run(model, ids, portions):
    """Logits of all positions, the tokens given in portions from a carried state."""
    state, at, out = None, 0, []
    for n in portions:
        r = model(torch.tensor(ids[None, at:at + n], device="cuda"), past_key_values=state, use_cache=True)
        state = r.past_key_values
        out.append(r.logits[0].double().cpu().numpy())
        at += n
    assert state.length == len(ids)
    from complexity_deep_b200 import ops
    ops.status_fetch()
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", [F32, BF], ids=["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(CASES))
def test_logits_whole_portions_and_token_by_token(name, dtype, tmp_path_factory):
    cfg, w, _, model = _model(name, dtype, tmp_path_factory)
    T = 153
    ids = tokens(cfg, T)
    want = _reference(name, cfg, w, ids)
    for portions in ([T], [2] * 76 + [1], [1] * T, [T - 11] + [1] * 11, [3, 20, 2, 17, 1, 110], [64, 89], [70, 83]):
        _check(_run(model, ids, portions), want, dtype, portions)


@pytest.mark.parametrize("dtype", [F32, BF], ids=["fp32", "bf16"])
@pytest.mark.parametrize("n", [1, 2, 3])
def test_first_tokens(n, dtype, tmp_path_factory):
    cfg, w, _, model = _model("odd", dtype, tmp_path_factory)
    ids = tokens(cfg, n, seed=n)
    _check(_run(model, ids, [n]), _reference("odd", cfg, w, ids), dtype)


def test_batch_equals_each_sequence_alone(tmp_path_factory):
    cfg, w, _, model = _model("odd", BF, tmp_path_factory)
    ids = np.stack([tokens(cfg, 50, seed=s) for s in range(3)])
    out = model(torch.tensor(ids[:, :45], device="cuda"), use_cache=True)
    state, parts = out.past_key_values, [out.logits]
    for t in range(45, 50):
        parts.append(model(torch.tensor(ids[:, t:t + 1], device="cuda"), past_key_values=state, use_cache=True).logits)
    got = torch.cat(parts, 1).double().cpu().numpy()
    for b in range(3):
        _check(got[b], _reference("odd", cfg, w, ids[b]), BF)
        alone = _run(model, ids[b], [45] + [1] * 5)
        assert np.median(np.abs(alone - got[b])) <= 0.02 * got[b].std()


def test_states_are_reused_without_traces(tmp_path_factory):
    cfg, w, _, model = _model("odd", F32, tmp_path_factory)
    pool = model.state_pool()
    long, short = tokens(cfg, 70, seed=1), tokens(cfg, 29, seed=2)
    model(torch.tensor(long[None], device="cuda"), past_key_values=pool.get("a"), use_cache=True)
    first = pool.get("a")
    pool.release("a")
    state = pool.get("b")
    assert state is first
    got = [model(torch.tensor(short[None, a:b], device="cuda"), past_key_values=state, use_cache=True).logits[0]
           for a, b in ((0, 2), (2, 20), (20, 21), (21, 29))]
    _check(torch.cat(got).double().cpu().numpy(), _reference("odd", cfg, w, short), F32)


def test_long_decoding(tmp_path_factory):
    cfg, w, _, model = _model("ragged", F32, tmp_path_factory)
    ids = tokens(cfg, 300, seed=5)
    _check(_run(model, ids, [4] + [1] * 296), _reference("ragged", cfg, w, ids), F32)


def test_logit_rows(tmp_path_factory):
    cfg, w, _, model = _model("odd", F32, tmp_path_factory)
    ids = torch.tensor(tokens(cfg, 20)[None], device="cuda")
    full = model(ids).logits[0]
    some = model(ids, logit_rows=torch.tensor([3, 19], device="cuda")).logits
    assert torch.equal(some, full[[3, 19]])
    assert model(ids, logit_rows=torch.empty(0, dtype=torch.int64, device="cuda")).logits.shape == (0, cfg["vocab"])


def _greedy(w, cfg, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(np.argmax(ro.forward(w, cfg, np.array(ids))[-1])))
    return ids


def test_greedy_generation_and_command_line(tmp_path_factory, capsys):
    from complexity_deep_b200 import cli
    cfg, w, path, model = _model("odd", F32, tmp_path_factory)
    prompts = np.stack([tokens(cfg, 9, seed=s) for s in (0, 1)])
    want = [_greedy(w, cfg, p, 24) for p in prompts]
    got = model.generate(torch.tensor(prompts, device="cuda"), max_new_tokens=24, do_sample=False)
    assert got.tolist() == want
    args = [x for p in prompts for x in ("--prompt", ",".join(map(str, p)))]
    assert cli.main(["generate", "--model", path, "--dtype", "float32", "--greedy", "--max-new-tokens", "24"] + args) == 0
    assert [[int(t) for t in line.split(",")] for line in capsys.readouterr().out.split()] == want
    stop = want[0][14]
    one = model.generate(torch.tensor(prompts[:1], device="cuda"), max_new_tokens=24, do_sample=False, eos_token_id=stop)
    assert one[0].tolist() == want[0][:want[0].index(stop, 9) + 1]


@pytest.mark.parametrize("name", ["odd", "wide"])
def test_graphs_equal_eager(name, tmp_path_factory):
    from complexity_deep_b200.models import DecodeGraph, PrefillGraph
    cfg, w, _, model = _model(name, BF, tmp_path_factory)
    ids = torch.tensor(np.stack([tokens(cfg, 120, seed=s) for s in range(2)]), device="cuda")
    graph = DecodeGraph(model, batch=2, capacity=124)
    for _ in range(2):                                   # the second run starts from a used state
        out = model(ids[:, :80], use_cache=True)
        assert torch.equal(graph.prefill(ids[:, :80]), out.logits)
        for t in range(80, 120):
            step = model(ids[:, t:t + 1], past_key_values=out.past_key_values, use_cache=True).logits
            got = graph.step(ids[:, t:t + 1])
            assert float((got - step).abs().max()) <= 0.05 * float(step.std()), t
    pre = PrefillGraph(model, 2, 70)
    for a in (0, 40):
        assert torch.equal(pre(ids[:, a:a + 70]), model(ids[:, a:a + 70]).logits)
    with pytest.raises(RuntimeError):
        for t in range(10):
            graph.step(ids[:, :1])


def test_more_tokens_than_positions_are_refused(tmp_path_factory):
    cfg, w, _, model = _model("ragged", F32, tmp_path_factory)
    limit = cfg["max_positions"]
    out = model(torch.tensor(tokens(cfg, limit)[None], device="cuda"), use_cache=True)
    with pytest.raises(RuntimeError):
        model(torch.zeros(1, 1, dtype=torch.int64, device="cuda"), past_key_values=out.past_key_values)
    with pytest.raises(ValueError):
        model.make_decode_cache(1, limit + 1)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(dtype, tmp_path_factory, tmp_path):
    cfg, w, path, _ = _model("odd", F32, tmp_path_factory)
    ids = {n: tokens(cfg, 40, seed=s) for s, n in enumerate("ab")}
    steps = [{"entries": [("a", 0, 17, [0, 16])], "end": []},
             {"entries": [("b", 0, 3, [])], "end": []},
             {"entries": [("a", 17, 19, [1]), ("b", 3, 39, [35])], "end": []},
             {"entries": [("b", 39, 40, [0])], "end": ["b"]},
             {"entries": [("a", 19, 40, [20])], "end": ["a"]}]
    lines = [json.dumps({"step": i, "entries": [{"id": n, "tokens": ids[n][lo:hi].tolist(), "want": want}
                                                for n, lo, hi, want in s["entries"]], "end": s["end"]})
             for i, s in enumerate(steps)]
    run = subprocess.run([f"{ROOT}/bin/trace_run", "--model", path, "--dtype", dtype, "--out", str(tmp_path),
                          "--max-tokens", "80"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [x for x in run.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(5)]
    for i, s in enumerate(steps):
        want = [_reference("odd", cfg, w, ids[n])[lo + k] for n, lo, hi, ks in s["entries"] for k in ks]
        if not want:
            assert not (tmp_path / f"{i}.f32").exists()
            continue
        got = np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]).astype(np.float64)
        _check(got, np.stack(want), getattr(torch, dtype), i)
