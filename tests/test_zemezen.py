"""Zemezen on the CPU definitions: configuration, mechanisms, engine schedules, scheduler, tensor parallelism and trace replay
against the plain implementation in `zemezen_oracle.py`."""
import io
import json

import pytest
import torch

import zemezen_oracle as O
from mp_util import run_ranks
from slopllm_b200.models.zemezen import ZemezenConfig, ZemezenModel
from slopllm_b200.ops import delta as D
from slopllm_b200.ops import experts as EX
from zemezen_util import configs, feed, make_engine, portions, random_ids, row_error

CONFIGS = configs()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_portions(name):
    raw, ranks = CONFIGS[name]
    t = O.random_tensors(raw, 1, ranks)
    ids = random_ids(raw, 90, 2)
    want = O.forward(raw, t, ids)
    eng = make_engine(raw, t)
    for cuts in ([90], portions(90, [2, 31, 3]), portions(90, [64], tail=5)):
        assert row_error(feed(eng, ids, cuts), want).max() < 1e-5, cuts


def test_every_mechanism_shows_in_the_logits():
    """The checks mean something only if a lost mechanism moves the logits: each is changed in the plain implementation."""
    raw, ranks = CONFIGS["tiled"]
    t = O.random_tensors(raw, 1, ranks)
    ids = random_ids(raw, 90, 2)
    want = O.forward(raw, t, ids)

    def moved(changed_raw=None, changed_t=None):
        return row_error(O.forward(changed_raw or raw, {**t, **(changed_t or {})}, ids), want)[-1].item()

    def layer(i, part, **kw):
        r = json.loads(json.dumps(raw))
        for l in r["layers"]:
            if l is r["layers"][i] or l.get("weights_of") == i:
                l[part].update(kw)
        return r

    rot = lambda **kw: {**raw["layers"][0]["mixer"]["rot"], **kw}
    router = lambda **kw: {**raw["layers"][0]["mlp"]["router"], **kw}
    for mask in ({"size": 69, "keep_first": 5}, {"size": 71, "keep_first": 5}, {"size": 70, "keep_first": 4}, {"size": 70, "keep_first": 6}):
        assert moved(layer(0, "mixer", mask=mask)) > 1e-4, mask
    assert moved(layer(0, "mixer", rot=rot(base=1e4))) > 1e-3 and moved(layer(0, "mixer", rot=rot(dims=40))) > 1e-3
    assert moved(layer(0, "mlp", router=router(top=2))) > 1e-3 and moved(layer(0, "mlp", router=router(groups={"count": 5, "keep": 2}))) > 1e-4
    assert moved(layer(2, "mixer", scale=0.1)) > 1e-3 and moved(layer(0, "mixer", scale=0.1)) > 1e-3
    assert moved(changed_t={"l0.mix.sink": torch.full((6,), -40.0)}) > 1e-3
    for n in sorted(t):
        if n.endswith(("norm", "norm1", "dt_bias", "A_log", ".conv", ".b", "g2", "a2")):
            assert moved(changed_t={n: t[n] + 0.5 * (1 + torch.arange(t[n].numel()).view_as(t[n]) % 3)}) > 1e-3, n


def test_short_convolution_ring():
    g = torch.Generator().manual_seed(0)
    for taps in (1, 2, 4):
        x, w = torch.randn(30, 6, generator=g), torch.randn(6, taps, generator=g)
        ring, got, at = torch.zeros(2, taps, 6), [], 0
        for n in (1, 2, 9, 1, 1, 16):
            got.append(D.short_conv(x[at:at + n], w.t().contiguous(), ring, torch.arange(at, at + n), torch.tensor([0, n]), torch.tensor([1]), n, torch.float32))
            at += n
        assert torch.allclose(torch.cat(got), O.short_conv(x, w), atol=1e-6) and not ring[0].any()


@pytest.mark.parametrize("E,top,groups,keep", [(15, 4, 5, 3), (1, 1, 1, 1), (40, 6, 8, 3), (9, 4, 3, 2), (8, 8, 1, 1)])
def test_routing(E, top, groups, keep):
    z = torch.randn(50, E, generator=torch.Generator().manual_seed(E)) * 2
    ids, w = EX.route_softmax(z, top, groups, keep)
    want = O.choose_experts(z, top, groups, keep)
    assert torch.allclose(torch.zeros(50, E).scatter(1, ids.long(), w), want, atol=1e-6)
    if groups > 1 and keep < groups:
        assert not torch.allclose(want, O.choose_experts(z, top), atol=1e-6)      # (the groups do limit the choice)


def test_batches_of_unequal_requests_and_reused_slots():
    """Requests of several lengths interleaved in mixed steps, finished and replaced by others in the same pages and state
    slots: every request's logits equal its own."""
    raw, ranks = CONFIGS["tiled"]
    t = O.random_tensors(raw, 3, ranks)
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
        assert row_error(torch.cat(got[i]), O.forward(raw, t, ids[i])).max() < 1e-5, i


def test_layers_that_share_weights_keep_their_own_caches():
    raw, ranks = CONFIGS["odd"]
    eng = make_engine(raw, O.random_tensors(raw, 1, ranks))
    w, c = eng.model.w, eng.cache
    assert w.blocks[3].w_in is w.blocks[0].w_in and w.blocks[5].w_out is w.blocks[1].w_out and w.norms[3] is w.norms[0]
    assert c.state[3]["S"].data_ptr() != c.state[0]["S"].data_ptr() and c.rows[5]["k"].data_ptr() != c.rows[1]["k"].data_ptr()


def _oracle_greedy(raw, t, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(O.forward(raw, t, ids)[-1].argmax()))
    return ids[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    """Seven requests over two rows and two state slots, prompts longer than the chunk budget."""
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.scheduler.scheduler import GenerationRequest, GenerationScheduler
    raw, ranks = CONFIGS["tiled"]
    t = O.random_tensors(raw, 7, ranks)
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
    raw = O.config([O.attention_layer(heads=4, kv_heads=2, dim=16, window=12, keep=2, mlp=O.dense(64)),
                    O.delta_layer(heads=4, kv_heads=2, dim=12, vdim=8, mlp=O.moe(6, 2, 32, 3, 2)), O.latent_layer(heads=2, mlp=O.moe(4, 1, 8)), 1],
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
    raw, ranks = CONFIGS["odd"]

    def bad(match, change):
        r = json.loads(json.dumps(raw))
        change(r["layers"])
        with pytest.raises(ValueError, match=match):
            ZemezenConfig.from_dict(r)

    bad("unknown mixer", lambda l: l[2].update(type="other"))
    bad("kv_rank", lambda l: l[2]["mixer"].pop("kv_rank"))
    bad("feed-forward", lambda l: l[1]["mlp"].update(kind="sparse"))
    bad("evenly", lambda l: l[1]["mixer"].update(kv_heads=4))
    bad("vdim", lambda l: l[1]["mixer"].update(vdim=8))
    bad("even and at most", lambda l: l[1]["mixer"]["rot"].update(dims=5))
    bad("cannot be chosen", lambda l: l[0]["mlp"]["router"].update(top=7))
    bad("differs", lambda l: l[3]["mixer"].update(conv=3))
    bad("no layer", lambda l: l[0].update(weights_of=3))
    t = O.random_tensors(raw, 0, ranks)
    t["l2.mix.uk"] = t["l2.mix.uk"][:-1]
    with pytest.raises(ValueError, match="l2.mix.uk"):
        ZemezenModel.from_tensors(ZemezenConfig.from_dict(raw), t)


def test_registry_and_trace_replay(tmp_path, monkeypatch, capsys):
    import numpy as np
    from slopllm_b200.cli import trace_run
    from slopllm_b200.models.registry import inspect_model, load_any
    from test_gidisun import write_checkpoint
    raw, ranks = CONFIGS["odd"]
    t = O.random_tensors(raw, 2, ranks)
    model_dir = write_checkpoint(tmp_path / "m", raw, t)
    assert inspect_model(model_dir)[0] == "zemezen"
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
    assert row_error(read(0), wa[[0, 65]]).max() < 1e-5
    assert not (tmp_path / "o" / "1.f32").exists()
    assert row_error(read(2), torch.stack([wa[69], wb[11]])).max() < 1e-5
    assert row_error(read(3), wa[69:70]).max() < 1e-5


@pytest.mark.parametrize("world", [1, 2])
def test_memory_plan_matches_the_built_model(world, capsys):
    from slopllm_b200.cli import plan as plan_cli
    from slopllm_b200.models.zemezen import assemble_zemezen_weights, random_zemezen_tensors
    from slopllm_b200.utils.sizing import zemezen_cache_bytes, zemezen_weight_bytes
    from test_gidisun import _tensor_bytes
    cfg = ZemezenConfig.tiny()
    w = assemble_zemezen_weights(cfg, random_zemezen_tensors(cfg), "cpu", torch.float32, 0, world)
    tables = sum(b.mixer.rot.freq.numel() * 4 for b in w.blocks if hasattr(b.mixer, "rot"))
    assert _tensor_bytes(w) == zemezen_weight_bytes(cfg, world, 4) + tables
    page, state = zemezen_cache_bytes(cfg, world, 4)
    assert page == sum(b.spec.row_values() for b in w.blocks) * 4 * 64 and state == sum(b.spec.state_values() for b in w.blocks) * 4
    assert plan_cli.main(["--random-init", "zemezen", "--max-pages", "64"]) == 0
    capsys.readouterr()


def test_command_line_runtime():
    """The shared entry-point code builds the family, and requests run through its scheduler with sampling."""
    import argparse
    from slopllm_b200.cli.model_cli import add_model_args, build_runtime
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.scheduler.scheduler import GenerationRequest
    ap = argparse.ArgumentParser()
    add_model_args(ap)
    rt = build_runtime(ap.parse_args(["--cpu", "--random-init", "zemezen-tiny", "--no-cuda-graph", "--batch-size", "2", "--chunk-size", "32",
                                      "--max-pages", "16"]))
    assert rt.model_type == "zemezen"
    reqs = [GenerationRequest(id=str(i), input_ids=[5 + i] * 40, max_tokens=4, sampling=SamplingParams(temperature=0.8)) for i in range(3)]
    for r in reqs:
        rt.scheduler.submit(r)
    for _ in range(40):
        rt.scheduler.step()
    assert all(r.retired and r.error is None and len(r.generated) == 4 for r in reqs)
