"""Pulunex on the CPU definitions: configuration, mechanisms, engine schedules, scheduler, tensor parallelism and trace replay
against the plain implementation in `pulunex_oracle.py`."""
import io
import json
import types

import pytest
import torch

import pulunex_oracle as O
from mp_util import run_ranks
from pulunex_util import configs, feed, make_engine, portions, random_ids, row_error, same, sharp_model
from slopllm_b200.models.pulunex import PulunexConfig, PulunexModel
from slopllm_b200.models.weights import ExpertWeights
from slopllm_b200.ops import RefOps
from slopllm_b200.ops import experts as EX
from slopllm_b200.ops import shift as SH
from slopllm_b200.ops import talking as TK

CONFIGS = configs()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_portions(name):
    raw = CONFIGS[name]
    t = O.random_tensors(raw, 1)
    ids = random_ids(raw, 90, 2)
    want = O.forward(raw, t, ids)
    eng = make_engine(raw, t)
    for cuts in ([90], portions(90, [2, 31, 3]), portions(90, [64], tail=5)):
        assert same(feed(eng, ids, cuts), want), cuts


def test_every_mechanism_shows_in_the_logits():
    """The checks mean something only if a lost mechanism moves the logits: each is changed in the plain implementation."""
    raw = CONFIGS["tiled"]
    t = O.random_tensors(raw, 1)
    ids = random_ids(raw, 110, 2)
    want = O.forward(raw, t, ids)

    def moved(changed_raw=None, changed_t=None):
        return row_error(O.forward(changed_raw or raw, t if changed_t is None else {**t, **changed_t}, ids), want).max().item()

    def changed(f):
        r = json.loads(json.dumps(raw))
        f(r)
        return r

    for i, l in enumerate(raw["layers"]):
        size = (l["mixer"].get("mask") or {}).get("size", 0)
        assert moved(changed(lambda r: r["layers"][i]["mixer"].update(scale=l["mixer"]["scale"] * 1.3))) > 1e-3, i
        for d in ((-1, 1) if size else ()):                       # a chunk one position longer or shorter
            assert moved(changed(lambda r: r["layers"][i]["mixer"].update(mask={"size": size + d}))) > 1e-3, (i, d)
    assert moved(changed(lambda r: r["layers"][3]["mixer"].update(mask={"size": 64}))) > 1e-3
    assert moved(changed(lambda r: r["embedding"].update(scale=1.0))) > 1e-3 and moved(changed(lambda r: r.update(logit_scale=0.4))) > 1e-3
    for i, n in ((0, 2), (3, 4)):                                 # identity experts that are left out
        z = t[f"l{i}.mlp.router"].clone()
        z[-n:] = 0
        assert moved(changed_t={f"l{i}.mlp.router": z}) > 1e-3
    for n in sorted(t):
        if t[n].dim() < 2 or n.endswith((".talk", ".sg", "pos")):
            assert moved(changed_t={n: t[n] + 0.5 * (1 + torch.arange(t[n].numel()) % 3).view(t[n].shape)}) > 1e-3, n


def test_token_shift_carries_its_state():
    """Portions of several sequences in shuffled slots against the whole sequences."""
    g = torch.Generator().manual_seed(1)
    H, total, slots = 7, [20, 9, 1], [2, 0, 3]
    y, r = ([torch.randn(n, H, generator=g) for n in total] for _ in range(2))
    w, mix = torch.full((H,), 1.3), torch.randn(H, generator=g)
    want = [O.token_shift(O.scalar_norm(a + b, torch.tensor(1.3), 1e-3), mix) for a, b in zip(y, r)]
    state, done, got = torch.zeros(4, H), [0, 0, 0], [[], [], []]
    for cut in ([5, 1, 0], [2, 3, 1], [13, 5, 0]):
        live = [b for b in range(3) if cut[b]]
        part = lambda x: torch.cat([x[b][done[b]:done[b] + cut[b]] for b in live])
        ind = torch.tensor([0] + [cut[b] for b in live]).cumsum(0)
        out, res = SH.add_shift_norm(None, part(y), part(r), w, 1e-3, SH.Shift(mix, state, ind, torch.tensor([slots[b] for b in live]), None), torch.float32)
        assert torch.equal(res, part(y) + part(r))
        for j, b in enumerate(live):
            got[b].append(out[ind[j]:ind[j + 1]])
            done[b] += cut[b]
    for b in range(3):
        assert torch.allclose(torch.cat(got[b]), want[b], atol=1e-6)
    assert not state[1].any()


def test_corrected_routing_and_identity_experts():
    g = torch.Generator().manual_seed(0)
    z, c = torch.randn(40, 9, generator=g), torch.randn(9, generator=g)
    ids, w = EX.route_softmax(z, 4, correction=c)
    want, ww = O.choose(z, c, 4)
    assert torch.equal(ids.long(), want) and torch.allclose(w, ww)
    assert not torch.equal(ids, EX.route_softmax(z, 4)[0])
    ex = ExpertWeights(torch.randn(6, 10, 12, generator=g), torch.randn(6, 12, 5, generator=g))     # router outputs 6 to 8: identity
    x = torch.randn(40, 12, generator=g)
    a, b = torch.zeros(40, 12), torch.zeros(40, 12)
    EX.add_experts(x, ex, ids, w, a, None, identity=True)
    EX.add_experts(x, ex, ids, w, b, None)
    assert torch.allclose(a - b, x * (w * (ids >= 6)).sum(-1, keepdim=True), atol=1e-4) and (ids >= 6).any()


def test_activations():
    x, gate = torch.randn(5, 12, generator=torch.Generator().manual_seed(0)) * 4, torch.tensor([0.0, 1.0, -2.0, 30.0, -30.0])
    ops, out = RefOps(None), torch.empty(5, 6)
    ops.gated_act(x, out, "silu", row_gate=gate)
    assert torch.allclose(out, O.silu(x[:, :6]) * x[:, 6:] * torch.sigmoid(gate)[:, None], atol=1e-6)
    ops.plain_act(x[:, :6], out, "gelu_tanh")
    assert torch.allclose(out, O.gelu_tanh(x[:, :6]), atol=1e-6)


def test_chunks_count_from_the_start_of_the_sequence():
    assert [TK.first_visible(p, 5) for p in (0, 4, 5, 9, 10)] == [0, 0, 5, 5, 10] and TK.first_visible(99, 0) == 0 and TK.first_visible(7, 1) == 7
    at = torch.arange(12)
    for size in (0, 1, 5, 12, 40):
        mask = O.chunk_mask(at, at, size)
        for p in range(12):
            assert mask[p].nonzero().flatten().tolist() == list(range(TK.first_visible(p, size), p + 1))
    st = types.SimpleNamespace(extra={"spans": [[3, 20], [64, 1]]}, input_ids=torch.zeros(21))
    plan = TK.TalkingPlan.of(st, 8, 10)
    assert plan is TK.TalkingPlan.of(st, 8, 10) and plan.count == 4
    # (a tile's keys start at its first query's chunk)
    assert sorted(plan.tiles.tolist()) == [[0, 8, 3, 0], [8, 8, 11, 0], [16, 4, 19, 0], [20, 1, 64, 1]] and plan.longest == 13
    for work in (1, 3, 147, 148, 149, 5000):
        for keys in (1, 31, 32, 33, 4096):
            assert 1 <= TK.key_splits(work, keys, 32) <= min(64, -(-keys // 32))


def test_batches_of_unequal_requests_and_reused_slots():
    """Requests of several lengths interleaved in mixed steps, finished and replaced by others in the same pages and state
    slots: every request's logits equal its own."""
    raw = CONFIGS["tiled"]
    t = O.random_tensors(raw, 3)
    eng = make_engine(raw, t, num_pages=6, max_states=2)
    lens = [100, 40, 129, 7, 64, 90]
    ids = [random_ids(raw, n, 10 + i) for i, n in enumerate(lens)]
    got = [[] for _ in lens]
    live, waiting, turn = {}, list(range(len(lens))), 0
    while live or waiting:
        while waiting and len(live) < 2:
            live[waiting.pop(0)] = eng.kv.new_sequence()
        step = [(i, s, ids[i][s.length:s.length + [17, 1, 2, 33, 1, 64][(turn + j * 2) % 6]]) for j, (i, s) in enumerate(live.items())]
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
        assert same(torch.cat(got[i]), O.forward(raw, t, ids[i])), i


def test_far_tokens_reach_the_logits_through_the_caches():
    raw, t = sharp_model()
    ids = random_ids(raw, 230, 6)
    want = O.forward(raw, t, ids)
    for place in (0, 1, 63, 64, 199, 200):                        # around page and chunk borders too
        changed = list(ids)
        changed[place] = (ids[place] + 1) % raw["vocab"]
        assert row_error(O.forward(raw, t, changed), want)[-1] > 1e-3
    assert same(feed(make_engine(raw, t), ids, [70] + [1] * 160), want)


def _oracle_greedy(raw, t, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(O.forward(raw, t, ids)[-1].argmax()))
    return ids[len(prompt):]


def _generate(raw, t, prompts, max_tokens):
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.scheduler.scheduler import GenerationRequest, GenerationScheduler
    eng = make_engine(raw, t, num_pages=10, max_batch=2, max_states=2)
    sched = GenerationScheduler(eng, max_batch=2, chunk_size=24)
    reqs = [GenerationRequest(id=str(i), input_ids=p, max_tokens=max_tokens, sampling=SamplingParams(temperature=0.0)) for i, p in enumerate(prompts)]
    for r in reqs:
        sched.submit(r)
    for _ in range(200):
        sched.step()
        if all(r.retired for r in reqs):
            break
    assert eng.model.states.free == 2 and not eng.kv.sequences
    return reqs


def test_greedy_generation_through_the_scheduler():
    """Seven requests over two rows and two state slots, prompts longer than the chunk budget."""
    raw = CONFIGS["tiled"]
    t = O.random_tensors(raw, 7)
    for r in _generate(raw, t, [random_ids(raw, n, 20 + i) for i, n in enumerate((70, 3, 25, 49, 1, 30, 12))], 5):
        assert r.error is None and r.finish_reason == "length"
        assert r.generated == _oracle_greedy(raw, t, r.input_ids, 5), r.id


def test_no_sequence_passes_the_last_position():
    raw = O.config([O.layer(2, 1, 8, mlp=O.dense(8))], width=16, positions=40)
    t = O.random_tensors(raw, 7)
    short, full, over = _generate(raw, t, [random_ids(raw, n, n) for n in (36, 40, 41)], 9)
    assert short.error is None and short.generated == _oracle_greedy(raw, t, short.input_ids, 5)
    assert full.error is None and full.generated == _oracle_greedy(raw, t, full.input_ids, 1)
    assert "40 positions" in over.error and over.finish_reason == "error"
    eng = make_engine(raw, t)
    s = eng.kv.new_sequence()
    eng.step([s], [random_ids(raw, 39, 1)])
    with pytest.raises(ValueError, match="40 positions"):
        eng.step([s], [[1, 2]])
    eng.step([s], [[1]])
    with pytest.raises(ValueError, match="40 positions"):
        eng.step([s], [[1]])
    assert s.length == 40


def _tp_logits(rank, world):
    from slopllm_b200.parallel.dist import init_from_env
    raw = O.config([O.layer(4, 2, 16, 12, size=17, mlp=O.dense(64)), O.layer(8, 4, 8, 10, mlp=O.moe(5, 3, 12, identity=3, shared=20)),
                    O.layer(4, 4, 8, 10, size=30, kv_from=1, mlp=O.moe(3, 2, 8))], width=48, vocab=96)
    t = O.random_tensors(raw, 9)
    ctx = init_from_env("gloo")
    eng = make_engine(raw, t, ctx=ctx)
    ids = random_ids(raw, 40, 4)
    got = feed(eng, ids, portions(40, [15], tail=3))
    return same(got, O.forward(raw, t, ids))


def test_tensor_parallel_ranks_match():
    assert all(run_ranks(_tp_logits, 2))


def test_configuration_errors():
    raw = CONFIGS["odd"]

    def bad(match, change):
        r = json.loads(json.dumps(raw))
        change(r["layers"])
        with pytest.raises(ValueError, match=match):
            PulunexConfig.from_dict(r)

    bad("unknown mixer", lambda l: l[2].update(type="other"))
    bad("scale", lambda l: l[1]["mixer"].pop("scale"))
    bad("vdim", lambda l: l[0]["mixer"].pop("vdim"))
    bad("feed-forward", lambda l: l[0]["mlp"].update(kind="sparse"))
    bad("evenly", lambda l: l[0]["mixer"].update(kv_heads=4))
    bad("negative", lambda l: l[0]["mixer"].update(mask={"size": -1}))
    bad("kv_from", lambda l: l[2]["mixer"].update(kv_from=2))
    bad("kv_from", lambda l: l[2]["mixer"].update(kv_from=3))
    bad("kv_from", lambda l: l[3]["mixer"].update(kv_from=2))
    bad("key heads", lambda l: l[2]["mixer"].update(kv_from=0))
    bad("chosen", lambda l: l[3]["mlp"]["router"].update(top=4))
    with pytest.raises(ValueError, match="no layers"):
        PulunexConfig.from_dict({**raw, "layers": []})
    t = O.random_tensors(raw, 0)
    t["l0.mix.v.b"] = t["l0.mix.v.b"][:-1]
    with pytest.raises(ValueError, match="l0.mix.v.b"):
        PulunexModel.from_tensors(PulunexConfig.from_dict(raw), t)
    del t["l0.mix.v.b"]
    with pytest.raises(KeyError, match="l0.mix.v.b"):
        PulunexModel.from_tensors(PulunexConfig.from_dict(raw), t)


def test_shared_keys_are_stored_once():
    raw = CONFIGS["tiled"]
    model = PulunexModel.from_tensors(PulunexConfig.from_dict(raw), O.random_tensors(raw, 0))
    cache = model.allocate_cache(2, 1)
    assert [bool(r) for r in cache.rows] == [True, True, False, False, True] and all("shift" in s for s in cache.state)


def test_registry_and_trace_replay(tmp_path, monkeypatch, capsys):
    import numpy as np
    from slopllm_b200.cli import trace_run
    from slopllm_b200.models.registry import hybrid_family, inspect_model, load_any
    from test_gidisun import write_checkpoint
    raw = CONFIGS["odd"]
    t = O.random_tensors(raw, 2)
    model_dir = write_checkpoint(tmp_path / "m", raw, t)
    assert inspect_model(model_dir)[0] == "pulunex" and hybrid_family("pulunex-tiny").config is PulunexConfig
    cfg, model = load_any(model_dir)
    assert cfg.vocab_size == raw["vocab"] and not model.supports_prefix_sharing
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
    assert same(read(0), wa[[0, 65]])
    assert not (tmp_path / "o" / "1.f32").exists()
    assert same(read(2), torch.stack([wa[69], wb[11]]))
    assert same(read(3), wa[69:70])


@pytest.mark.parametrize("world", [1, 2])
def test_memory_plan_matches_the_built_model(world, capsys):
    from slopllm_b200.cli import plan as plan_cli
    from slopllm_b200.models.pulunex import assemble_pulunex_weights, random_pulunex_tensors
    from slopllm_b200.utils.sizing import pulunex_cache_bytes, pulunex_weight_bytes
    from test_gidisun import _tensor_bytes
    cfg = PulunexConfig.tiny()
    t = random_pulunex_tensors(cfg)
    w = assemble_pulunex_weights(cfg, t, "cpu", torch.float32, 0, world)
    assert _tensor_bytes(w) == pulunex_weight_bytes(cfg, world, 4)
    page, state = pulunex_cache_bytes(cfg, world, 4)
    specs = PulunexModel(cfg, w).specs
    assert page == sum(s.row_values() for s in specs) * 4 * 64 and state == sum(s.state_values() for s in specs) * 4
    assert plan_cli.main(["--random-init", "pulunex", "--max-pages", "64"]) == 0
    capsys.readouterr()


def test_command_line_runtime():
    """The shared entry-point code builds the family, and requests run through its scheduler with sampling."""
    import argparse
    from slopllm_b200.cli.model_cli import add_model_args, build_runtime
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.scheduler.scheduler import GenerationRequest
    ap = argparse.ArgumentParser()
    add_model_args(ap)
    args = ap.parse_args(["--cpu", "--random-init", "pulunex-tiny", "--no-cuda-graph", "--batch-size", "2", "--chunk-size", "32", "--max-pages", "16"])
    args.max_model_len = None
    rt = build_runtime(args)
    assert rt.model_type == "pulunex" and args.max_model_len == rt.cfg.max_positions == rt.engine.max_positions
    reqs = [GenerationRequest(id=str(i), input_ids=[5 + i] * 40, max_tokens=4, sampling=SamplingParams(temperature=0.8)) for i in range(3)]
    for r in reqs:
        rt.scheduler.submit(r)
    for _ in range(40):
        rt.scheduler.step()
    assert all(r.retired and r.error is None and len(r.generated) == 4 for r in reqs)
