"""Sigisun through the framework on CPU tensors: configuration and checkpoint round trips, the engine's ragged steps,
scheduler and sampling against the plain restatement in ``sigisun_oracle.py``."""
import json

import pytest
import torch

import sigisun_oracle as O
from sigisun_helpers import CONFIGS, feed, make_engine, rel_rms, tokens, write_checkpoint


@pytest.fixture(autouse=True)
def _invariant_checks(monkeypatch):
    import openrlhf_b200.rollout.engine as E

    monkeypatch.setattr(E, "_DEBUG", True)
    threads = torch.get_num_threads()
    torch.set_num_threads(1)              # thousands of tiny operations
    yield
    torch.set_num_threads(threads)


@pytest.fixture(scope="module", params=sorted(CONFIGS))
def case(request, tmp_path_factory):
    cfg = CONFIGS[request.param]
    path = tmp_path_factory.mktemp(request.param)
    return cfg, write_checkpoint(path, cfg, seed=len(request.param)), path


def test_whole_prompt_portions_and_single_tokens_give_the_same_logits(case):
    cfg, w, path = case
    toks = tokens(cfg, 160)
    want = O.forward(cfg, w, toks)
    eng = make_engine(path, "cpu", torch.float32)
    for cuts in ([160], [1], [2], [7, 3, 50, 2], [129, 1]):
        assert rel_rms(feed(eng, toks, cuts), want) < 2e-5, cuts
    assert eng.blocks.num_free() == eng.num_pages - 1


def test_mixed_batches_and_reused_rows(case):
    cfg, w, path = case
    seqs = {f"q{i}": tokens(cfg, n, i) for i, n in enumerate((9, 140, 3, 31, 1, 70))}
    want = {k: O.forward(cfg, w, t) for k, t in seqs.items()}
    eng = make_engine(path, "cpu", torch.float32, rows=3, pages=7)
    g = torch.Generator().manual_seed(5)
    at, live, todo = {}, [], list(seqs)
    while todo or live:
        while todo and len(live) < 3:
            live.append(todo.pop(0))
        entries = []
        for k in live:
            if int(torch.randint(0, 4, (1,), generator=g)) == 0 and len(live) > 1:
                continue                                       # sits this step out
            n = int(torch.randint(1, 40, (1,), generator=g)) if int(torch.randint(0, 2, (1,), generator=g)) else 1
            part = seqs[k][at.get(k, 0):at.get(k, 0) + n]
            entries.append((k, part, [0, len(part) - 1] if len(part) > 1 else [0]))
        if not entries:
            continue
        lg, o = eng.extend(entries), 0
        for k, part, wanted in entries:
            ref = want[k][[at.get(k, 0) + j for j in wanted]]
            assert rel_rms(lg[o:o + len(wanted)], ref) < 2e-5 * float(want[k].std() / ref.std()) + 1e-5, (k, at.get(k, 0))
            o += len(wanted)
            at[k] = at.get(k, 0) + len(part)
            if at[k] == len(seqs[k]):
                eng.finish(k)
                live.remove(k)
    assert eng.blocks.num_free() == eng.num_pages - 1


def test_checkpoint_and_config_round_trip(case, tmp_path):
    from openrlhf_b200.models.hf_io import _open_shards, load_pretrained, save_pretrained
    from openrlhf_b200.models.registry import read_config

    cfg, w, path = case
    m = load_pretrained(str(path), device="cpu")
    assert m.cfg.num_params() == sum(t.numel() for t in w.values())
    save_pretrained(m, str(tmp_path))
    names, handles = _open_shards(str(tmp_path))
    assert set(names) == set(w)
    for k, fn in names.items():
        assert torch.equal(handles[fn].get_tensor(k), w[k]), k
    assert read_config(str(tmp_path)) == m.cfg
    back = json.load(open(tmp_path / "config.json"))
    assert back == json.load(open(path / "config.json"))


def _greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(O.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_the_scheduler(tmp_path):
    from openrlhf_b200.rollout.engine import SamplingParams

    cfg = CONFIGS["mix"]
    w = write_checkpoint(tmp_path, cfg, seed=3)
    prompts = [tokens(cfg, n, i) for i, n in enumerate((5, 61, 127, 2, 30))]
    want = [_greedy(cfg, w, p, 12) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    eng = make_engine(tmp_path, "cpu", torch.float32, rows=3, check_interval=4)
    out = eng.generate(prompts, sp)
    assert [o.outputs[0].token_ids for o in out] == want
    lp = torch.log_softmax(O.forward(cfg, w, prompts[0] + want[0]), -1)
    got = torch.tensor(out[0].outputs[0].logprob_values)
    ref = torch.stack([lp[len(prompts[0]) - 1 + k, t] for k, t in enumerate(want[0])])
    assert (got - ref).abs().max() < 1e-3
    # chunked prefill beside decoding rows, several samples of one prompt, a pool that forces preemption
    small = make_engine(tmp_path, "cpu", torch.float32, rows=4, pages=6, max_prefill_tokens=128, check_interval=4)
    sp2 = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True, n=2)
    out2 = small.generate([prompts[2], prompts[1], prompts[0]], sp2)
    for o, k in zip(out2, (2, 1, 0)):
        assert [c.token_ids for c in o.outputs] == [want[k]] * 2
    assert small.blocks.num_free() == 6 - 1


def test_preemption_recomputes_the_state(tmp_path):
    from openrlhf_b200.rollout.engine import SamplingParams

    cfg = CONFIGS["ssm"]
    write_checkpoint(tmp_path, cfg, seed=4)
    prompts = [tokens(cfg, 120, i) for i in range(3)]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True, n=2)
    ref = make_engine(tmp_path, "cpu", torch.float32, rows=6).generate(prompts, sp)
    tight = make_engine(tmp_path, "cpu", torch.float32, rows=6, pages=8, check_interval=4)
    out = tight.generate(prompts, sp)
    assert tight.stats["preemptions"] >= 1
    assert [[c.token_ids for c in o.outputs] for o in out] == [[c.token_ids for c in o.outputs] for o in ref]


def test_sleep_drops_the_caches_and_a_fresh_sequence_is_right_afterwards(case):
    cfg, w, path = case
    toks = tokens(cfg, 50)
    eng = make_engine(path, "cpu", torch.float32)
    feed(eng, toks, [20, 1])
    eng.sleep()
    assert rel_rms(feed(eng, toks, [20, 1]), O.forward(cfg, w, toks)) < 2e-5


def test_trace_replay_writes_the_wanted_logits(case, tmp_path, capsys):
    import numpy as np

    from openrlhf_b200.cli.trace_run import make_engine as trace_engine
    from openrlhf_b200.cli.trace_run import replay

    cfg, w, path = case
    a, b = tokens(cfg, 20, 1), tokens(cfg, 6, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:15], "want": [14, 3]}, {"id": "b", "tokens": b[:5], "want": []}],
              "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[5:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[15:], "want": []}], "end": ["a"]}]
    replay(trace_engine(str(path), "float32", 128, device="cpu"), [json.dumps(s) for s in steps], str(tmp_path))
    assert capsys.readouterr().out.split("\n")[:3] == ["done 0", "done 1", "done 2"]
    got0 = torch.from_numpy(np.fromfile(tmp_path / "0.f32", dtype="<f4")).view(2, -1)
    assert rel_rms(got0, O.forward(cfg, w, a)[[14, 3]]) < 1e-4
    got1 = torch.from_numpy(np.fromfile(tmp_path / "1.f32", dtype="<f4")).view(1, -1)
    assert rel_rms(got1, O.forward(cfg, w, b)[[5]]) < 1e-4
    assert not (tmp_path / "2.f32").exists()


def test_what_the_design_does_not_have_is_refused(tmp_path):
    from openrlhf_b200.models.actor import Actor
    from openrlhf_b200.models.hybrid_config import HybridConfig
    from openrlhf_b200.models.registry import architecture_of

    cfg = CONFIGS["mix"]
    write_checkpoint(tmp_path, cfg)
    with pytest.raises(ValueError, match="prefix caching"):
        make_engine(tmp_path, "cpu", torch.float32, enable_prefix_caching=True)
    with pytest.raises(NotImplementedError):
        Actor(str(tmp_path), device="cpu")
    with pytest.raises(ValueError, match="unknown architecture"):
        architecture_of({"architecture": "none-such"})
    bad = json.loads(json.dumps(cfg))
    bad["layers"][3]["mixer"]["kv_from"] = 0
    with pytest.raises(ValueError, match="cannot read"):
        HybridConfig.from_dict(bad)
    eng = make_engine(tmp_path, "cpu", torch.float32, rows=1, max_len=128, pages=2)
    eng.extend([("a", [1] * 100, [])])
    with pytest.raises(RuntimeError, match="no free row"):
        eng.extend([("b", [1], [])])
    with pytest.raises(ValueError, match="max_model_len"):
        eng.extend([("a", [1] * 29, [])])
    eng.finish("a")


@pytest.mark.parametrize("mistake", ["window", "keep", "sink", "state", "taps", "gate", "scale"])
def test_the_comparison_notices_a_wrong_mechanism(case, mistake, monkeypatch):
    """A mistake planted in the restatement must exceed the tolerance the engine is held to."""
    cfg, w, _ = case
    kinds = {layer["type"] for layer in cfg["layers"]}
    if ("attention" if mistake in ("window", "keep", "sink", "scale") else "mamba2") not in kinds:
        pytest.skip("no such layer")
    if mistake == "keep" and not any(layer["mixer"].get("mask", {}).get("keep_first", 0) for layer in cfg["layers"]):
        pytest.skip("nothing is kept")
    toks = tokens(cfg, 160)
    right = O.forward(cfg, w, toks)
    if mistake in ("window", "keep"):
        vis = O.visible
        monkeypatch.setattr(O, "visible", (lambda i, j, s, k: vis(i, j, s + 1, k)) if mistake == "window" else
                            (lambda i, j, s, k: vis(i, j, s, max(k - 1, 0))))
    elif mistake == "sink":
        monkeypatch.setattr(O, "sink_softmax", lambda s: torch.softmax(s, -1))
    elif mistake == "scale":
        f = O.windowed_attention
        monkeypatch.setattr(O, "windowed_attention", lambda q, k, v, sc, *a: f(q, k, v, sc * 1.01, *a))
    elif mistake == "state":
        f = O.ssd_recurrence
        monkeypatch.setattr(O, "ssd_recurrence", lambda x, b, c, dt, a, d: (
            torch.cat([f(x[:64], b[:64], c[:64], dt[:64], a, d)[0], f(x[64:], b[64:], c[64:], dt[64:], a, d)[0]]), None))
    elif mistake == "taps":
        f = O.causal_conv
        monkeypatch.setattr(O, "causal_conv", lambda u, wt, b: f(u, wt, b * 1.01))
    else:
        f = O.group_rms_norm
        monkeypatch.setattr(O, "group_rms_norm", lambda x, wt, g, e: f(x, wt, g, e * 1000))
    assert rel_rms(O.forward(cfg, w, toks), right) > 2e-4


def test_generate_command_line(tmp_path, capsys):
    from openrlhf_b200.cli.generate import main

    cfg = CONFIGS["ssm"]
    w = write_checkpoint(tmp_path / "model", cfg, seed=6)
    prompts = [tokens(cfg, 9, 1), tokens(cfg, 30, 2)]
    (tmp_path / "in.jsonl").write_text(json.dumps(prompts[0]) + "\n" + json.dumps({"tokens": prompts[1]}) + "\n")
    assert main(["--model", str(tmp_path / "model"), "--input", str(tmp_path / "in.jsonl"), "--device", "cpu", "--dtype",
                 "float32", "--max_new_tokens", "5", "--n_samples", "2"]) == 0
    rows = [json.loads(x) for x in capsys.readouterr().out.splitlines()]
    assert [(r["prompt"], r["sample"]) for r in rows] == [(0, 0), (0, 1), (1, 0), (1, 1)]
    for r in rows:
        assert r["tokens"] == _greedy(cfg, w, prompts[r["prompt"]], 5) and r["finish_reason"] == "length"
    assert main(["--model", "tiny-sigisun", "--input", str(tmp_path / "in.jsonl"), "--device", "cpu",
                 "--max_new_tokens", "2"]) == 0


def test_component_build_lists_existing_sources():
    import os

    from openrlhf_b200.csrc import build

    for name in build.COMPONENTS:
        assert all(os.path.exists(p) for p in build.sources(name))
    assert build.PRECISE <= {os.path.basename(p) for p in build.sources()}
