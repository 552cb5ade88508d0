"""Vononex on the CPU definitions: configuration, mechanisms, engine schedules, scheduler, tensor parallelism and trace replay
against the plain implementation in `vononex_oracle.py`."""
import io
import json
import math

import pytest
import torch

import vononex_oracle as O
from mp_util import run_ranks
from slopllm_b200.models.vononex import VononexConfig, VononexModel
from slopllm_b200.ops import recurrent as RC
from slopllm_b200.ops import reference as R
from slopllm_b200.ops.rotary import AngleTable, adjacent_order
from vononex_util import configs, far_key_model, feed, make_engine, portions, random_ids, row_error, same

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
    ids = random_ids(raw, 90, 2)
    want = O.forward(raw, t, ids)

    def moved(changed_raw=None, changed_t=None):
        return row_error(O.forward(changed_raw or raw, t if changed_t is None else {**t, **changed_t}, ids), want)[-1].item()

    def layer(i, side=None, **kw):
        r = json.loads(json.dumps(raw))
        m = r["layers"][i]["mixer"]
        (m if side is None else m[side]).update(kw)
        return r

    for i in (1, 2):
        c = raw["layers"][i]["mixer"]
        for side in ("left", "right"):
            rot = c[side]["rot"]
            assert moved(layer(i, side, rot={**rot, "base": rot["base"] * 3})) > 1e-3, (i, side)
            assert moved(layer(i, side, rot={**rot, "dims": rot["dims"] - 2})) > 1e-3, (i, side)
        assert moved(layer(i, "left", scale=c["left"]["scale"] * 1.3)) > 1e-3
        assert moved(layer(i, left_scale=c["left_scale"] + 0.2)) > 1e-3 and moved(layer(i, right_scale=c["right_scale"] + 0.2)) > 1e-3
        for h in range(c["right"]["heads"]):
            decay = list(c["right"]["decay"])
            decay[h] *= 0.9
            assert moved(layer(i, "right", decay=decay)) > 1e-3, (i, h)
    other = json.loads(json.dumps(raw))
    other["postln_alpha"] *= 1.1
    assert moved(other) > 1e-3
    for n in sorted(t):
        if t[n].dim() == 1:
            assert moved(changed_t={n: t[n] + 0.5 * (1 + torch.arange(t[n].numel()) % 3)}) > 1e-3, n


def test_adjacent_order_and_angles():
    """Turning adjacent pairs of reordered values is the rotate-half rotation; equal rotations share their columns."""
    table = AngleTable()
    a, b = table.turn(6, 500.0), table.turn(10, 500.0)
    assert table.turn(6, 500.0) is a and table.turn(6, 501.0) is not a and b.at == 3
    pos = torch.tensor([0, 1, 63, 64, 100000], dtype=torch.int32)
    x = torch.randn(5, 3, 10, generator=torch.Generator().manual_seed(0))
    angles = table.at(pos)
    for turn in (a, b):
        order = adjacent_order(10, turn.dims)
        assert sorted(order.tolist()) == list(range(10))
        want = O.rotate(x.double(), pos, turn.dims, 500.0)[..., order]
        assert torch.allclose(turn.apply(x[..., order], angles).double(), want, atol=1e-6)
        assert torch.allclose(turn.apply(turn.apply(x, angles), angles, back=True), x, atol=1e-6)
    with pytest.raises(ValueError):
        table.turn(5, 10.0)


def test_min_gru_and_activation():
    g = torch.Generator().manual_seed(0)
    z, u = torch.randn(40, 7, generator=g) * 3, torch.randn(40, 7, generator=g) * 3
    u[0, 0], u[0, 1] = 0.0, -0.0                                  # the candidate is 1/2 from either side
    S = torch.randn(7, generator=g)
    want = O.min_gru(torch.sigmoid(z), u, S)
    state = S.clone()
    assert torch.allclose(R.min_gru_scan(z, u, state), want, atol=1e-6) and torch.allclose(state, want[-1], atol=1e-6)
    x = torch.randn(9, 12, generator=g) * 4
    assert torch.allclose(R.gated_act(x, "gelu_tanh"), O.gelu_tanh(x[:, :6]) * x[:, 6:], atol=1e-6)


def test_retention_carries_its_state():
    """Portions of several sequences in shuffled slots against the token-by-token definition."""
    g = torch.Generator().manual_seed(1)
    h, dk, dv, decay = 3, 6, 5, [0.9, 1.0, 0.0]
    table = AngleTable()
    turn = table.turn(4, 100.0)
    total, slots = [20, 9, 1], [2, 0, 3]
    rows = [torch.randn(n, h * (2 * dk + 2 * dv), generator=g) for n in total]
    order = adjacent_order(dk, 4)

    def want(x):
        n = x.shape[0]
        q, k, v, gate = torch.split(x, [h * dk, h * dk, h * dv, h * dv], 1)
        turned = lambda y: O.rotate(y.view(n, h, dk), torch.arange(n), 4, 100.0)
        o, S = O.retain(turned(q), turned(k) * dk ** -0.5, v.view(n, h, dv), torch.tensor(decay), torch.zeros(h, dk, dv))
        return O.rms(o, 1e-3).reshape(n, -1) * O.silu(gate) * 0.7

    def stored(x):
        y = x.clone()
        for i in range(2 * h):
            y[:, i * dk:(i + 1) * dk] = x[:, i * dk:(i + 1) * dk][:, order]
        return y

    state, done, got = torch.zeros(4, h, dk, dv), [0, 0, 0], [[], [], []]
    for cut in ([5, 1, 0], [2, 3, 1], [13, 5, 0]):
        live = [b for b in range(3) if cut[b]]
        x = torch.cat([stored(rows[b])[done[b]:done[b] + cut[b]] for b in live])
        pos = torch.cat([torch.arange(done[b], done[b] + cut[b]) for b in live])
        ind = torch.tensor([0] + [cut[b] for b in live]).cumsum(0)
        out = torch.empty(x.shape[0], h * dv)
        RC.retention_mix(x, RC.retention_decays(decay), turn, table.at(pos), 1e-3, state, ind, torch.tensor([slots[b] for b in live]), h, dk, dv, out, 0.7)
        for j, b in enumerate(live):
            got[b].append(out[ind[j]:ind[j + 1]])
            done[b] += cut[b]
    for b in range(3):
        assert torch.allclose(torch.cat(got[b]), want(rows[b]), atol=1e-5)
    assert not state[1].any()
    assert RC.retention_decays([0.5, 0.0])[1].tolist() == [-1.0, -200.0]
    with pytest.raises(ValueError):
        RC.retention_decays([-0.1])


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
    raw, t = far_key_model()
    ids = random_ids(raw, 200, 6)
    want = O.forward(raw, t, ids)
    for place in (0, 1, 63, 64):                                  # around a page border too
        changed = list(ids)
        changed[place] = (ids[place] + 1) % raw["vocab"]
        assert row_error(O.forward(raw, t, changed), want)[-1] > 2e-3
    assert same(feed(make_engine(raw, t), ids, [70] + [1] * 130), want)


def _oracle_greedy(raw, t, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(O.forward(raw, t, ids)[-1].argmax()))
    return ids[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    """Seven requests over two rows and two state slots, prompts longer than the chunk budget."""
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.scheduler.scheduler import GenerationRequest, GenerationScheduler
    raw = CONFIGS["tiled"]
    t = O.random_tensors(raw, 7)
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
    raw = O.config([O.parallel_layer(heads=4, kv_heads=2, dim=16, vdim=12, dims=8, left_scale=0.6, right_scale=1.4, r_heads=4, r_dim=12, r_vdim=8, ff=64),
                    O.mingru_layer(width=40, ff=20), O.parallel_layer(heads=2, kv_heads=2, r_heads=2)], width=48, vocab=96)
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
            VononexConfig.from_dict(r)

    bad("unknown mixer", lambda l: l[2].update(type="other"))
    bad("width", lambda l: l[1]["mixer"].pop("width"))
    bad("right_scale", lambda l: l[0]["mixer"].pop("right_scale"))
    bad("kv_heads", lambda l: l[0]["mixer"]["left"].pop("kv_heads"))
    bad("decay", lambda l: l[0]["mixer"]["right"].pop("decay"))
    bad("feed-forward", lambda l: l[0]["mlp"].update(kind="sparse"))
    bad("evenly", lambda l: l[0]["mixer"]["left"].update(kv_heads=4))
    bad("vdim", lambda l: l[0]["mixer"]["left"].update(vdim=9))
    bad("even and at most", lambda l: l[0]["mixer"]["left"]["rot"].update(dims=5))
    bad("even and at most", lambda l: l[0]["mixer"]["right"]["rot"].update(dims=12))
    bad("decays for", lambda l: l[0]["mixer"]["right"]["decay"].pop())
    with pytest.raises(ValueError, match="no layers"):
        VononexConfig.from_dict({**raw, "layers": []})
    t = O.random_tensors(raw, 0)
    t["l0.mix.left.v.b"] = t["l0.mix.left.v.b"][:-1]
    with pytest.raises(ValueError, match="l0.mix.left.v.b"):
        VononexModel.from_tensors(VononexConfig.from_dict(raw), t)
    del t["l0.mix.left.v.b"]
    with pytest.raises(KeyError, match="l0.mix.left.v.b"):
        VononexModel.from_tensors(VononexConfig.from_dict(raw), t)


def test_registry_and_trace_replay(tmp_path, monkeypatch, capsys):
    import numpy as np
    from slopllm_b200.cli import trace_run
    from slopllm_b200.models.registry import hybrid_family, inspect_model, load_any
    from test_gidisun import write_checkpoint
    raw = CONFIGS["odd"]
    t = O.random_tensors(raw, 2)
    model_dir = write_checkpoint(tmp_path / "m", raw, t)
    assert inspect_model(model_dir)[0] == "vononex" and hybrid_family("vononex-tiny").config is VononexConfig and hybrid_family("qwen3") is None
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
    from slopllm_b200.models.vononex import assemble_vononex_weights, random_vononex_tensors
    from slopllm_b200.utils.sizing import vononex_cache_bytes, vononex_weight_bytes
    from test_gidisun import _tensor_bytes
    cfg = VononexConfig.tiny()
    w = assemble_vononex_weights(cfg, random_vononex_tensors(cfg), "cpu", torch.float32, 0, world)
    assert _tensor_bytes(w) == vononex_weight_bytes(cfg, world, 4)
    page, state = vononex_cache_bytes(cfg, world, 4)
    assert page == sum(m.spec.row_values() for m in w.mixers) * 4 * 64 and state == sum(m.spec.state_values() for m in w.mixers) * 4
    assert plan_cli.main(["--random-init", "vononex", "--max-pages", "64"]) == 0
    capsys.readouterr()


def test_command_line_runtime():
    """The shared entry-point code builds the family, and requests run through its scheduler with sampling."""
    import argparse
    from slopllm_b200.cli.model_cli import add_model_args, build_runtime
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.scheduler.scheduler import GenerationRequest
    ap = argparse.ArgumentParser()
    add_model_args(ap)
    rt = build_runtime(ap.parse_args(["--cpu", "--random-init", "vononex-tiny", "--no-cuda-graph", "--batch-size", "2", "--chunk-size", "32",
                                      "--max-pages", "16"]))
    assert rt.model_type == "vononex"
    reqs = [GenerationRequest(id=str(i), input_ids=[5 + i] * 40, max_tokens=4, sampling=SamplingParams(temperature=0.8)) for i in range(3)]
    for r in reqs:
        rt.scheduler.submit(r)
    for _ in range(40):
        rt.scheduler.step()
    assert all(r.retired and r.error is None and len(r.generated) == 4 for r in reqs)


def test_norm_over_whole_rows_is_not_per_head():
    """One head's large queries damp the others': the oracle's norm spans the heads (as the framework's, by the tests above)."""
    x = torch.ones(1, 4)
    x[:, 2:] = 7.0
    assert O.norm(x, torch.ones(4), 0.0)[0, 0].item() == pytest.approx(1 / math.sqrt((2 + 2 * 49) / 4))
