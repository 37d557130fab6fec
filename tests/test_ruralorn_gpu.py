"""Ruralorn models on the engine against the plain restatement: prompts, portions, decoding, batches,
reused slots, generation through the public entry points."""
import json

import pytest
import torch

import ruralorn_models as M
import ruralorn_oracle as O
from test_entrypoints_cpu import _sentence, workspace  # noqa: F401  (fixture)

pytestmark = pytest.mark.gpu
DT = {"bf16": torch.bfloat16, "fp32": torch.float32}
TOL = {"bf16": 2e-2, "fp32": 1e-4}


def _ok():
    from easy_to_hard_b200.ops import _lib
    torch.cuda.synchronize()
    assert _lib.read_status() == 0


def _run(eng, key, ids, cuts, close=True):
    """Logits of every position, the tokens entering in the portions that ``cuts`` bounds."""
    eng.open(key)
    out = [eng.step([(key, ids[a:b], range(b - a))]) for a, b in zip(cuts, cuts[1:])]
    if close:
        eng.close(key)
    return torch.cat(out)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("name", sorted(M.ZOO))
def test_prompts_portions_and_decoding(dt, name):
    cfg = M.settled(M.ZOO[name], dt)
    W = M.weights(cfg, 1)
    T = 150
    ids = M.tokens(cfg, T)
    want = O.forward(cfg, W, ids)
    eng = M.build(cfg, W, DT[dt], 2, 160)
    for cuts in ([0, T], list(range(T + 1)), list(range(0, T, 2)) + [T], list(range(0, T, 7)) + [T],
                 list(range(0, T, 25)) + [T], [0, 1, 66, 131, 133, T],
                 [0, 100] + list(range(101, T + 1))):
        got = _run(eng, "s", ids, cuts)
        assert M.error(got, want) < TOL[dt], cuts[:3]
    _ok()


@pytest.mark.parametrize("name", sorted(M.ZOO))
def test_bf16_with_a_choice_of_experts(name):
    """Rounding may swap experts of nearly equal score at a few positions; most are not touched."""
    cfg = M.ZOO[name]
    W = M.weights(cfg, 1)
    ids = M.tokens(cfg, 150)
    got = _run(M.build(cfg, W, torch.bfloat16, 1, 152), "s", ids, [0, 70, 90, 91, 150])
    assert M.error(got, O.forward(cfg, W, ids), 0.5) < TOL["bf16"]


@pytest.mark.parametrize("dt", DT)
def test_residual_stream_layer_by_layer(dt):
    for name in ("mixed", "odd", "plain"):
        cfg = M.settled(M.ZOO[name], dt)
        W = M.weights(cfg, 2)
        ids = M.tokens(cfg, 40)
        want = []
        O.forward(cfg, W, ids, trace=want)
        eng = M.build(cfg, W, DT[dt], 1, 48)
        eng.layer_trace = []
        _run(eng, "s", ids, [0, 40])
        assert len(eng.layer_trace) == len(want)
        for got, w in zip(eng.layer_trace, want):
            assert M.error(got, w) < TOL[dt]


@pytest.mark.parametrize("dt", DT)
def test_unequal_requests_in_one_step_match_each_alone(dt):
    """Prompts, portions of prompts and decode steps of different sequences in one step."""
    cfg = M.settled(M.ZOO["mixed"], dt)
    W = M.weights(cfg, 4)
    lens = {"a": 70, "b": 9, "c": 131, "d": 33}
    ids = {k: M.tokens(cfg, n, ord(k)) for k, n in lens.items()}
    eng = M.build(cfg, W, DT[dt], 4, 136)
    plan = [{"b": 3, "a": 60}, {"a": 1, "c": 100}, {"a": 1, "b": 2, "c": 1, "d": 30},
            {"a": 1, "b": 1, "c": 1, "d": 1}, {"a": 7, "b": 1, "c": 29, "d": 2}, {"b": 2}]
    at = dict.fromkeys(lens, 0)
    got = {k: [] for k in lens}
    for k in lens:
        eng.open(k)
    for step in plan:
        out = eng.step([(k, ids[k][at[k]: at[k] + n], range(n)) for k, n in step.items()])
        for k, x in zip(step, out.split(list(step.values()))):
            got[k].append(x)
            at[k] += step[k]
    for k in lens:
        x = torch.cat(got[k])
        assert len(x) == lens[k]
        assert M.error(x, O.forward(cfg, W, ids[k])) < TOL[dt], k
    _ok()


def test_slots_are_used_again():
    """A slot's former owner leaves no trace, whatever its length was."""
    cfg = M.ZOO["mixed"]
    W = M.weights(cfg, 5)
    eng = M.build(cfg, W, torch.float32, 2, 128)
    eng.open("stays")
    ids = {i: M.tokens(cfg, n, i) for i, n in enumerate((120, 5, 64, 2, 90))}
    stay = M.tokens(cfg, 40, 77)
    kept = [eng.step([("stays", stay[:11], range(11))])]
    for i, t in ids.items():
        got = _run(eng, i, t, [0, len(t) // 2, len(t)] if i % 2 else [0, len(t)])
        assert M.error(got, O.forward(cfg, W, t)) < TOL["fp32"]
        kept.append(eng.step([("stays", stay[11 + 5 * i: 16 + 5 * i], range(5))]))
    x = torch.cat(kept)
    assert M.error(x, O.forward(cfg, W, stay[: len(x)])) < TOL["fp32"]


def test_steps_larger_than_one_forward_are_cut(monkeypatch):
    from easy_to_hard_b200.models import hybrid_engine
    cfg = M.ZOO["mixed"]
    W = M.weights(cfg, 6)
    a, b = M.tokens(cfg, 100, 1), M.tokens(cfg, 77, 2)
    eng = M.build(cfg, W, torch.float32, 2, 104)
    monkeypatch.setattr(hybrid_engine, "MAX_FORWARD_TOKENS", 48)
    eng.open("a"), eng.open("b")
    got = eng.step([("a", a, [99, 3, 50]), ("b", b, [0, 76])])
    want = torch.cat([O.forward(cfg, W, a)[[99, 3, 50]], O.forward(cfg, W, b)[[0, 76]]])
    assert M.error(got, want) < TOL["fp32"]


@pytest.mark.parametrize("dt", DT)
def test_long_decoding_past_every_window(dt):
    """Hundreds of single tokens, far past every window, some of them right behind a portion."""
    cfg = M.settled(M.ZOO["mixed"], dt)
    W = M.weights(cfg, 7)
    T = 420
    ids = M.tokens(cfg, T, 5)
    eng = M.build(cfg, W, DT[dt], 1, T)
    got = _run(eng, "s", ids, [0, 40] + list(range(41, 300)) + [330] + list(range(331, T + 1)))
    assert M.error(got, O.forward(cfg, W, ids)) < TOL[dt]
    _ok()


def test_one_key_outside_the_window_changes_nothing():
    """Replacing a token moves exactly the positions whose window (through the layers) it is in."""
    cfg = M.config([M.layer(3, 24, 16, 24, 56, window=9, mlp=M.moe(3, 1, 32))], width=72)
    W = M.weights(cfg, 13)
    ids = M.tokens(cfg, 60, 3)
    other = list(ids)
    other[20] = (ids[20] + 1) % cfg["vocab"]
    for dt in DT:
        eng = M.build(cfg, W, DT[dt], 1, 64)
        for cuts in ([0, 60], [0, 23] + list(range(24, 61)), list(range(0, 61, 2))):
            a, b = (_run(eng, "s", x, cuts) for x in (ids, other))
            moved = ((a - b).abs().amax(1) > 1e-3 * float(a.std())).tolist()
            assert moved == [20 <= i < 29 for i in range(60)], (dt, cuts[:3])
    _ok()


def test_bad_steps_are_refused():
    cfg = M.ZOO["mixed"]
    eng = M.build(cfg, M.weights(cfg), torch.bfloat16, 1, 32)
    eng.open("a")
    with pytest.raises(ValueError, match="vocabulary"):
        eng.step([("a", [cfg["vocab"]], [])])
    eng.close("a"), eng.open("a")
    with pytest.raises(ValueError, match="place"):
        eng.step([("a", [1, 2], [2])])
    eng.close("a"), eng.open("a")
    with pytest.raises(RuntimeError, match="positions"):
        eng.step([("a", [1] * 40, [])])
    with pytest.raises(RuntimeError, match="slots"):
        eng.open("b")
    _ok()


def _greedy(cfg, W, ids, n):
    ids = list(ids)
    for _ in range(n):
        ids.append(int(O.forward(cfg, W, ids)[-1].argmax()))
    return ids


def test_greedy_generation_of_unequal_rows():
    """The public generate(): left-padded prompts, captured decode step, long past every window;
    twice, so that the graph and the slots are used again."""
    import inference_generate as api
    cfg = M.config([M.layer(6, 40, 24, 24, 72, window=12, mlp=M.moe(5, 2, 44)),
                    M.layer(3, 24, 8, 40, 56, window=None, mlp=M.moe(4, 1, 32, None))], width=96,
                   vocab=120)
    W = M.weights(cfg, 8)
    from easy_to_hard_b200.models.hybrid import HybridLM, hybrid_config
    model = HybridLM.from_tensors(hybrid_config(cfg), W, dtype=torch.float32)
    for lens, new in (((5, 17, 1), 45), ((30, 2, 11), 12)):
        rows = [M.tokens(cfg, n, n) for n in lens]
        T = max(lens)
        prompt = torch.zeros(3, T, dtype=torch.int32)
        for b, r in enumerate(rows):
            prompt[b, T - len(r):] = torch.tensor(r)
        pad = torch.tensor([T - n for n in lens]).cuda()
        seq, steps = api.generate(model, prompt.cuda(), pad, new, temperature=0.0)
        assert seq.shape == (3, T + new) and steps == new - 1
        for b, r in enumerate(rows):
            assert seq[b, T - len(r):].tolist() == _greedy(cfg, W, r, new)
    assert model._decode_engine._graphs                    # the captured step is what ran
    _ok()


def test_prompts_larger_than_one_forward_in_generate(monkeypatch):
    from easy_to_hard_b200.models import hybrid_engine
    cfg = M.ZOO["mixed"]
    W = M.weights(cfg, 9)
    monkeypatch.setattr(hybrid_engine, "MAX_FORWARD_TOKENS", 40)
    rows = [M.tokens(cfg, n, n) for n in (61, 7, 30)]
    prompt = torch.zeros(3, 61, dtype=torch.int32)
    for b, r in enumerate(rows):
        prompt[b, 61 - len(r):] = torch.tensor(r)
    eng = M.build(cfg, W, torch.float32, 3, 80)
    seq, _ = eng.generate(prompt.cuda(), torch.tensor([61 - len(r) for r in rows]), 4, 0.0)
    for b, r in enumerate(rows):
        assert seq[b, 61 - len(r): 65].tolist() == _greedy(cfg, W, r, 4)


def test_sampled_generation_in_bf16_is_reproducible():
    cfg = M.config(M.ZOO["wide"]["layers"], width=192, vocab=257, cap=3.0)
    eng = M.build(cfg, M.weights(cfg, 10), torch.bfloat16, 4, 96, use_graph=True)
    prompt = torch.randint(0, cfg["vocab"], (4, 40), device="cuda", dtype=torch.int32)
    runs = [eng.generate(prompt, None, 50, 0.8, 20, seed=s)[0].clone() for s in (1, 1, 2)]
    assert torch.equal(runs[0], runs[1]) and not torch.equal(runs[0], runs[2])
    assert int(runs[0].min()) >= 0 and int(runs[0].max()) < cfg["vocab"]
    _ok()


def _save(folder, cfg, W):
    from easy_to_hard_b200.utils.safetensors_io import save_safetensors
    folder.mkdir(exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_safetensors(folder / "model.safetensors", W)


def test_command_line_generation(workspace, tmp_path):  # noqa: F811
    """inference_generate.main on a checkpoint folder of the design, and the interactive one."""
    import inference_generate as ig
    import interactive
    cfg = M.config(M.ZOO["mixed"]["layers"], width=120, vocab=400)
    folder = tmp_path / "model"
    _save(folder, cfg, M.weights(cfg, 11))
    (folder / "tokenizer.model").write_bytes(
        (workspace / "tiny-llama" / "tokenizer.model").read_bytes())
    g = torch.Generator().manual_seed(4)
    (tmp_path / "p.json").write_text(json.dumps([{"prompt": _sentence(g, 3 + i)}
                                                 for i in range(5)]))
    out = tmp_path / "out.jsonl"
    ig.main(1, tmp_path / "p.json", out, batch_size=2, num_samples=1, max_new_tokens=12, top_k=10,
            temperature=0.7, checkpoint_path=folder / "model.safetensors")
    rows = [json.loads(x) for x in out.read_text().splitlines()]
    assert {r["idx"] for r in rows} == set(range(5))
    assert all(isinstance(r["output"], str) for r in rows)
    stats = interactive.main("two three", num_samples=1, max_new_tokens=9, top_k=5,
                             checkpoint_path=folder / "model.safetensors")
    assert len(stats["tokens_per_sec"]) == 1
    with pytest.raises(ValueError, match="8-bit"):
        ig.main(1, tmp_path / "p.json", out, checkpoint_path=folder / "model.safetensors",
                on_the_fly_8bit_quantization=True)
    _ok()


@pytest.mark.parametrize("dt", ["bfloat16", "float32"])
def test_trace_replay(dt, tmp_path, capsys):
    import numpy as np
    from easy_to_hard_b200 import trace_run
    cfg = M.ZOO["plain"]
    W = M.weights(cfg, 12)
    _save(tmp_path / "m", cfg, W)
    a, b = M.tokens(cfg, 50, 1), M.tokens(cfg, 20, 2)
    steps = [dict(step=0, entries=[dict(id="x", tokens=a[:40], want=[])], end=[]),
             dict(step=1, entries=[dict(id="x", tokens=a[40:], want=[9, 0])], end=["x"]),
             dict(step=2, entries=[dict(id="x", tokens=b[:19], want=[18])], end=[]),
             dict(step=3, entries=[dict(id="x", tokens=b[19:], want=[0])], end=["x"])]
    (tmp_path / "o").mkdir()
    rc = trace_run.main(["--model", str(tmp_path / "m"), "--dtype", dt, "--out",
                         str(tmp_path / "o"), "--max-tokens", "50"],
                        [json.dumps(s) for s in steps])
    assert rc == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == \
        [f"done {i}" for i in range(4)]
    assert sorted(p.name for p in (tmp_path / "o").iterdir()) == ["1.f32", "2.f32", "3.f32"]
    got = [torch.from_numpy(np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4"))
           .view(-1, cfg["vocab"]) for i in (1, 2, 3)]
    wa, wb = O.forward(cfg, W, a), O.forward(cfg, W, b)
    tol = TOL["bf16" if dt == "bfloat16" else "fp32"]
    assert M.error(got[0], wa[[49, 40]]) < tol
    assert M.error(torch.cat(got[1:]), wb[[18, 19]]) < tol
