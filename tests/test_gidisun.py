"""Gidisun on the CPU definitions: configuration, mechanisms, engine schedules, scheduler, tensor parallelism and trace replay
against the plain implementation in `gidisun_oracle.py`."""
import io
import json

import pytest
import torch

import gidisun_oracle as O
from gidisun_util import configs, feed, make_engine, portions, random_ids, row_error
from mp_util import run_ranks
from slopllm_b200.models.gidisun import GidisunConfig, GidisunModel
from slopllm_b200.ops.rotary import YarnScaling, rotary_table

CONFIGS = configs()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_portions(name):
    raw, low = CONFIGS[name]
    t = O.random_tensors(raw, 1, low)
    ids = random_ids(raw, 90, 2)
    want = O.forward(raw, t, ids)
    eng = make_engine(raw, t)
    for cuts in ([90], portions(90, [2, 31, 3]), portions(90, [64], tail=5)):
        assert row_error(feed(eng, ids, cuts), want).max() < 1e-5, cuts


def test_every_mechanism_shows_in_the_logits():
    """The checks above mean something only if a lost mechanism moves the logits: each is changed in the plain implementation."""
    raw = CONFIGS["tiled"][0]
    t = O.random_tensors(raw, 1)
    ids = random_ids(raw, 90, 2)
    want = O.forward(raw, t, ids)

    def moved(changed_raw=None, changed_t=None):
        return row_error(O.forward(changed_raw or raw, {**t, **(changed_t or {})}, ids), want)[-1].item()

    def mixer(i, **kw):
        r = json.loads(json.dumps(raw))
        r["layers"][i]["mixer"].update(kw)
        return r

    rot = lambda **kw: {**raw["layers"][0]["mixer"]["rot"], **kw}
    assert moved(mixer(0, mask={"size": 69})) > 1e-4 and moved(mixer(3, mask={"size": 18})) > 1e-4
    assert moved(mixer(0, rot=rot(scaling=None))) > 1e-3 and moved(mixer(0, rot=rot(base=1e4))) > 1e-3
    assert moved(changed_t={"l0.mix.sink": torch.full((5,), -40.0)}) > 1e-3
    assert moved(mixer(1, gate_cap=4.0)) > 1e-3 and moved(mixer(2, tau=3.0)) > 1e-3
    for n in ("l0.norm1b", "l1.mix.norm", "l2.mix.norm", "l0.mix.dkv.norm", "final.norm", "l1.mix.i.b", "l1.mix.f.b", "l2.mix.a2.b"):
        assert moved(changed_t={n: t[n] + 0.5 * (1 + torch.arange(t[n].numel()) % 3)}) > 1e-3, n


def test_rotary_tables():
    for dims, base, sc in ((16, 1e4, None), (64, 1e6, dict(factor=2.0, original=1024, fast=32.0, slow=1.0)),
                           (32, 1e4, dict(factor=8.0, original=128, fast=16.0, slow=2.0)), (8, 100.0, dict(factor=1.0, original=64, fast=4.0, slow=1.0)),
                           (4, 1e4, dict(factor=4.0, original=8, fast=64.0, slow=32.0))):
        f, gain = O.yarn_frequencies(dims, base, sc)
        tab = rotary_table(dims, base, YarnScaling(**sc) if sc else None)
        assert torch.allclose(tab.freq.double(), f, rtol=1e-6) and abs(tab.gain - gain) < 1e-12
    x = torch.randn(5, 3, 24, generator=torch.Generator().manual_seed(0))
    pos = torch.tensor([0, 1, 7, 300, 4000])
    rot = {"dims": 16, "base": 1e4, "scaling": dict(factor=4.0, original=256, fast=32.0, slow=1.0)}
    got = rotary_table(16, 1e4, YarnScaling(4.0, 256, 32.0, 1.0)).apply(x, pos)
    assert torch.allclose(got, O.rotate_half(x, pos, rot), atol=2e-3) and torch.equal(got[..., 16:], x[..., 16:])


def test_batches_of_unequal_requests_and_reused_slots():
    """Requests of several lengths interleaved in mixed steps, finished and replaced by others in the same pages and state
    slots: every request's logits equal its own."""
    raw, low = CONFIGS["tiled"]
    t = O.random_tensors(raw, 3, low)
    eng = make_engine(raw, t, num_pages=6, max_states=2)
    lens = [100, 40, 129, 7, 64, 90]
    ids = [random_ids(raw, n, 10 + i) for i, n in enumerate(lens)]
    got = [[] for _ in lens]
    live, waiting, turn = {}, list(range(len(lens))), 0
    while live or waiting:
        while waiting and len(live) < 2:
            live[waiting.pop(0)] = eng.kv.new_sequence()
        step = []
        for j, (i, s) in enumerate(live.items()):
            n = [17, 1, 2, 33, 1, 64][(turn + j * 2) % 6]
            step.append((i, s, ids[i][s.length:s.length + n]))
        out = eng.step([s for _, s, _ in step], [x for _, _, x in step], [range(len(x)) for _, _, x in step])
        at = 0
        for i, s, x in step:
            got[i].append(out[at:at + len(x)])
            at += len(x)
            if s.length == lens[i]:
                eng.finish(live.pop(i))
        turn += 1
    eng.kv.assert_clear()
    for i in range(len(lens)):
        assert row_error(torch.cat(got[i]), O.forward(raw, t, ids[i])).max() < 1e-5, i


def test_a_request_may_pause():
    raw, low = CONFIGS["odd"]
    t = O.random_tensors(raw, 5, low)
    eng = make_engine(raw, t)
    a, b = random_ids(raw, 30, 1), random_ids(raw, 25, 2)
    sa, sb = eng.kv.new_sequence(), eng.kv.new_sequence()
    out = [eng.step([sa], [a[:10]], [range(10)])]
    for k in range(5):
        eng.step([sb], [b[k * 5:k * 5 + 5]], [[]])
    out += [eng.step([sb, sa], [b[:1], a[10:]], [[], range(20)])]
    assert row_error(torch.cat(out), O.forward(raw, t, a)).max() < 1e-5


def test_state_slots_run_out_with_an_error():
    raw, low = CONFIGS["ones"]
    eng = make_engine(raw, O.random_tensors(raw, 0, low), max_states=2)
    seqs = [eng.kv.new_sequence() for _ in range(3)]
    eng.step(seqs[:2], [[1, 2], [3]])
    with pytest.raises(RuntimeError, match="state slots"):
        eng.step(seqs[2:], [[4]])
    eng.finish(seqs[0])
    eng.finish(seqs[2])
    s = eng.kv.new_sequence()
    eng.step([s], [[4, 5]])


def _oracle_greedy(raw, t, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(O.forward(raw, t, ids)[-1].argmax()))
    return ids[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    """Seven requests over two rows and two state slots, prompts longer than the chunk budget."""
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.scheduler.scheduler import GenerationRequest, GenerationScheduler
    raw, low = CONFIGS["tiled"]
    t = O.random_tensors(raw, 7, low)
    eng = make_engine(raw, t, num_pages=10, max_batch=2, max_states=2)
    sched = GenerationScheduler(eng, max_batch=2, chunk_size=24)
    reqs = [GenerationRequest(id=str(i), input_ids=random_ids(raw, n, 20 + i), max_tokens=5, sampling=SamplingParams(temperature=0.0))
            for i, n in enumerate((70, 3, 25, 49, 1, 30, 12))]
    for r in reqs:
        sched.submit(r)
    for _ in range(200):
        sched.step()
        if all(r.retired for r in reqs):
            break
    for r in reqs:
        assert r.error is None and r.finish_reason == "length"
        assert r.generated == _oracle_greedy(raw, t, r.input_ids, 5), r.id
    assert eng.model.states.free == 2 and not eng.kv.sequences


def _tp_logits(rank, world):
    from slopllm_b200.parallel.dist import init_from_env
    raw = O.config([O.attention_layer(heads=4, dim=16, vdim=8, kv_rank=24, window=12, ff=64), O.gla_layer(heads=2), O.mlstm_layer(heads=4, ff=32)],
                   width=48, vocab=96)
    t = O.random_tensors(raw, 9)
    ctx = init_from_env("gloo")
    eng = make_engine(raw, t, ctx=ctx)
    ids = random_ids(raw, 40, 4)
    got = feed(eng, ids, portions(40, [15], tail=3))
    return row_error(got, O.forward(raw, t, ids)).max().item()


def test_tensor_parallel_ranks_match():
    assert max(run_ranks(_tp_logits, 2)) < 1e-5


def test_configuration_errors():
    raw, _ = CONFIGS["odd"]
    bad = json.loads(json.dumps(raw))
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        GidisunConfig.from_dict(bad)
    bad = json.loads(json.dumps(raw))
    del bad["layers"][1]["mixer"]["kv_rank"]
    with pytest.raises(ValueError, match="kv_rank"):
        GidisunConfig.from_dict(bad)
    bad = json.loads(json.dumps(raw))
    bad["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(ValueError, match="feed-forward"):
        GidisunConfig.from_dict(bad)
    t = O.random_tensors(raw, 0, 5)
    t["l1.mix.uk"] = t["l1.mix.uk"][:-1]
    with pytest.raises(ValueError, match="l1.mix.uk"):
        GidisunModel.from_tensors(GidisunConfig.from_dict(raw), t)


def write_checkpoint(path, raw, t):
    from slopllm_b200.checkpoint.safetensors_io import save_file
    path.mkdir(exist_ok=True)
    (path / "config.json").write_text(json.dumps(raw))
    save_file(t, str(path / "model.safetensors"))
    return str(path)


def test_registry_and_trace_replay(tmp_path, monkeypatch, capsys):
    import numpy as np
    from slopllm_b200.cli import trace_run
    from slopllm_b200.models.registry import inspect_model, load_any
    raw, low = CONFIGS["odd"]
    t = O.random_tensors(raw, 2, low)
    model_dir = write_checkpoint(tmp_path / "m", raw, t)
    assert inspect_model(model_dir)[0] == "gidisun"
    cfg, model = load_any(model_dir)
    assert cfg.vocab_size == raw["vocab"] and not model.supports_prefix_sharing
    with pytest.raises(ValueError):
        inspect_model(model_dir, mtp=1)
    a, b = random_ids(raw, 70, 1), random_ids(raw, 12, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:11], "want": []}, {"id": "a", "tokens": a[66:69], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[69:], "want": [0]}, {"id": "b", "tokens": b[11:], "want": [0]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": a, "want": [69]}], "end": ["c"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert trace_run.main(["--model", model_dir, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "192", "--cpu"]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = O.forward(raw, t, a), O.forward(raw, t, b)
    read = lambda i: torch.from_numpy(np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4")).view(-1, raw["vocab"])
    assert row_error(read(0), wa[[0, 65]]).max() < 1e-5
    assert not (tmp_path / "o" / "1.f32").exists()
    assert row_error(read(2), torch.stack([wa[69], wb[11]])).max() < 1e-5
    assert row_error(read(3), wa[69:70]).max() < 1e-5


def _tensor_bytes(obj) -> int:
    seen, total, stack = set(), 0, [obj]
    while stack:
        x = stack.pop()
        if isinstance(x, torch.Tensor):
            if x.data_ptr() not in seen:
                seen.add(x.data_ptr())
                total += x.numel() * x.element_size()
        elif isinstance(x, (list, tuple)):
            stack += x
        elif hasattr(x, "__dataclass_fields__"):
            stack += [getattr(x, f) for f in x.__dataclass_fields__]
    return total


@pytest.mark.parametrize("world", [1, 2])
def test_memory_plan_matches_the_built_model(world, capsys):
    from slopllm_b200.cli import plan as plan_cli
    from slopllm_b200.models.gidisun import assemble_gidisun_weights, random_gidisun_tensors
    from slopllm_b200.utils.sizing import gidisun_cache_bytes, gidisun_weight_bytes
    cfg = GidisunConfig.tiny()
    w = assemble_gidisun_weights(cfg, random_gidisun_tensors(cfg), "cpu", torch.float32, 0, world)
    table = sum(t.numel() * 4 for t in {id(m.rot.freq): m.rot.freq for m in w.mixers if hasattr(m, "rot")}.values())
    assert _tensor_bytes(w) == gidisun_weight_bytes(cfg, world, 4) + table
    page, state = gidisun_cache_bytes(cfg, world, 4)
    assert page == sum(m.spec.row_values() for m in w.mixers) * 4 * 64 and state == sum(m.spec.state_values() for m in w.mixers) * 4
    assert plan_cli.main(["--random-init", "gidisun", "--max-pages", "64"]) == 0
    capsys.readouterr()


def test_command_line_runtime():
    """The shared entry-point code builds the family, and a request runs through its scheduler with sampling."""
    import argparse
    from slopllm_b200.cli.model_cli import add_model_args, build_runtime
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.scheduler.scheduler import GenerationRequest
    ap = argparse.ArgumentParser()
    add_model_args(ap)
    rt = build_runtime(ap.parse_args(["--cpu", "--random-init", "gidisun-tiny", "--no-cuda-graph", "--batch-size", "2", "--chunk-size", "32",
                                      "--max-pages", "16"]))
    assert rt.model_type == "gidisun"
    reqs = [GenerationRequest(id=str(i), input_ids=[5 + i] * 40, max_tokens=4, sampling=SamplingParams(temperature=0.8)) for i in range(3)]
    for r in reqs:
        rt.scheduler.submit(r)
    for _ in range(40):
        rt.scheduler.step()
    assert all(r.retired and r.error is None and len(r.generated) == 4 for r in reqs)
