"""Latent-attention stacks without a GPU: configuration, snapshot reading, planning, the oracle's mechanisms against direct formulas, the
scheduler's context limit and the trace replay's bookkeeping."""
import json
import math

import pytest
import torch

from latent_stack_models import CONFIGS, MIXED, make_tensors, masters_of, variant, write_snapshot

from cuteafd_b200.config import from_hf_config, spec_by_name, spec_from_json, spec_to_json
from cuteafd_b200.ref import latent_stack as oracle


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_config_and_spec_round_trip(name):
    cfg = CONFIGS[name]
    spec = from_hf_config(cfg)
    assert spec.family == "bedovik" and spec.n_layers == len(cfg["layers"]) and spec.learned_positions == cfg["max_positions"] and spec.rms_eps == cfg["norm"]["eps"]
    for b, layer in zip(spec.blocks, cfg["layers"]):
        m = layer["mixer"]
        assert (b.attn.n_heads, b.attn.head_dim, b.attn.v_head_dim, b.attn.kv_lora_rank, b.attn.softmax_scale) == (m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["scale"])
        assert b.attn.out_gate == (layer["type"] == "latent_attention") and (b.moe is None) == (layer["mlp"] is None)
    assert spec_from_json(json.loads(json.dumps(spec_to_json(spec)))) == spec


def test_layer_runs_of_a_loop():
    assert from_hf_config(MIXED).layer_runs() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert from_hf_config(variant(MIXED, loop=None)).layer_runs() == [(i, None) for i in range(4)]
    assert from_hf_config(variant(MIXED, loop={"start": 3, "stop": 4, "times": 2})).layer_runs() == [(0, None), (1, None), (2, None), (3, 0), (3, 1)]


def test_bad_configurations_are_refused():
    for change in ({"loop": {"start": 2, "stop": 5, "times": 1}}, {"loop": {"start": 2, "stop": 2, "times": 1}}, {"layers": [dict(MIXED["layers"][0], type="other")]},
                   {"layers": [dict(MIXED["layers"][0], mlp=dict(MIXED["layers"][0]["mlp"], kind="dense"))]}):
        with pytest.raises(ValueError):
            from_hf_config(variant(MIXED, **change))
    bad = json.loads(json.dumps(MIXED))
    bad["layers"][0]["mlp"]["router"].update(top=9)             # only 8 experts can be left after the groups
    with pytest.raises(ValueError):
        from_hf_config(bad)


def test_snapshot_reader_checks_names_and_shapes(tmp_path):
    from cuteafd_b200.loader.stack_checkpoint import read_stack_masters
    t = make_tensors(MIXED)
    spec, m = masters_of(MIXED, t, tmp_path / "a")
    assert torch.equal(m["layers"][0]["w_up"][3].float(), t["l0.mlp.e3.up"]) and "w_g" not in m["layers"][1] and "router" not in m["layers"][1]
    assert m["layers"][2]["norm"][2] == float(t["l2.norm1.alpha"]) and torch.equal(m["loop_step"].float(), t["loop.step"])
    with pytest.raises(KeyError):
        read_stack_masters(write_snapshot(MIXED, {k: v for k, v in t.items() if k != "l2.mix.g"}, tmp_path / "b"), spec)
    with pytest.raises(ValueError):
        read_stack_masters(write_snapshot(MIXED, dict(t, **{"l1.mix.uk": t["l1.mix.uk"][:-1]}), tmp_path / "c"), spec)


def test_plan_reads_the_family(tmp_path):
    from cuteafd_b200.loader.plan import plan
    p = write_snapshot(MIXED, make_tensors(MIXED), tmp_path / "m")
    rep = plan(str(p), world=1, layout=True)
    assert rep.supported and rep.family == "bedovik" and rep.layout.pool_tokens > 0
    assert not plan(str(p), world=4, layout=True).supported
    spec = from_hf_config(MIXED)
    assert spec.kv_bytes_per_token() == len(spec.layer_runs()) * 256 * 2        # widest latent (200) in whole 64-element chunks, one row per run
    assert plan("bedovik", world=1, layout=True).supported and spec_by_name("bedovik").blocks


# ------------------------------------------------------------------ the oracle, mechanism by mechanism
def test_oracle_norms_and_embedding():
    x = torch.tensor([[0.5, -2.0, 30.0]])
    w, b = torch.tensor([2.0, 1.0, 3.0]), torch.tensor([0.1, 0.2, -0.3])
    want = [math.tanh(0.7 * v) * a + c for v, a, c in zip(x[0].tolist(), w.tolist(), b.tolist())]
    assert torch.allclose(oracle.dyt_norm(x, 0.7, w, b)[0], torch.tensor(want))
    y = oracle.rms_norm(torch.tensor([[3.0, 4.0]]), torch.tensor([1.0, 2.0]), 0.5)
    assert torch.allclose(y, torch.tensor([[3.0, 8.0]]) / math.sqrt(12.5 + 0.5))
    e = oracle.embed(torch.tensor([2, 0]), torch.arange(6.0).reshape(3, 2), torch.tensor([[10.0, 20.0], [30.0, 40.0], [0.0, 0.0]]))
    assert e.tolist() == [[14.0, 25.0], [30.0, 41.0]]


def test_oracle_attention_finds_a_planted_key_and_never_looks_ahead():
    torch.manual_seed(0)
    T, H, d, dv, r = 9, 2, 4, 3, 5
    q, c, uk, uv = torch.randn(T, H, d), torch.randn(T, r), torch.randn(H, d, r), torch.randn(H, dv, r)
    base = oracle.latent_attention(q, c, uk, uv, 0.5)
    later = c.clone()
    later[5:] += 3.0
    assert torch.allclose(oracle.latent_attention(q, later, uk, uv, 0.5)[:5], base[:5])
    basis = torch.eye(T)[:, :8]                                                  # rank 8, dim 8: key j of head 1 is basis row j
    q2, uk2, uv2 = torch.zeros(T, H, 8), torch.stack([torch.zeros(8, 8), torch.eye(8)]), torch.randn(H, dv, 8)
    q2[7, 1, 2] = 40.0                                                           # row 7 of head 1 points at key 2, head 0 at nothing
    o = oracle.latent_attention(q2, basis, uk2, uv2, 1.0)
    assert torch.allclose(o[7, 1], uv2[1][:, 2], atol=1e-5) and torch.allclose(o[7, 0], (uv2[0] @ basis[:8].mean(0)), atol=1e-5)
    assert torch.allclose(base[0], torch.stack([uv[h] @ c[0] for h in range(H)]), atol=1e-5)
    g = oracle.head_gate(base, torch.ones(T, 2), torch.tensor([[0.0, 0.0], [100.0, 0.0]]))
    assert torch.allclose(g[:, 0], base[:, 0] * 0.5) and torch.allclose(g[:, 1], base[:, 1])


def test_oracle_routing_keeps_groups_by_their_best_member():
    # group 0 has the best expert, group 1 the best pair, group 2 the second best single: ranked by best members, groups 0 and 2 stay
    z = torch.tensor([[5.0, -9.0, 3.0, 3.0, 4.0, -9.0]])
    picks = oracle.route(z, torch.eye(6), {"experts": 6, "top": 3, "scale": 2.0, "groups": {"count": 3, "keep": 2}})[0]
    s = torch.softmax(z[0], 0)
    assert [e for e, _ in picks] == [0, 4, 1] and abs(sum(w for _, w in picks) - 2.0) < 1e-6
    assert abs(picks[0][1] - 2.0 * float(s[0] / (s[0] + s[4] + s[1]))) < 1e-6
    assert [e for e, _ in oracle.route(z, torch.eye(6), {"experts": 6, "top": 3})[0]] == [0, 4, 2]


def test_oracle_expert_and_pass_entry():
    up, down = torch.tensor([[1.0, 0.0], [0.0, -1.0]]), torch.tensor([[1.0, 2.0]])
    assert oracle.expert(torch.tensor([3.0, 2.0]), up, down).tolist() == [9.0]
    assert oracle.expert(torch.tensor([-3.0, -2.0]), up, down).tolist() == [8.0]
    x = oracle.enter_pass(torch.tensor([[1.0]]), torch.tensor([[10.0]]), torch.tensor([[2.0, 3.0]]), torch.tensor([0.5]))
    assert x.tolist() == [[32.5]]


def test_oracle_stack_is_causal_and_uses_every_tensor():
    t = make_tensors(MIXED, 3)
    toks = torch.randint(0, MIXED["vocab"], (12,), generator=torch.Generator().manual_seed(1)).tolist()
    full, part = oracle.logits(MIXED, t, toks), oracle.logits(MIXED, t, toks[:7])
    assert torch.allclose(full[:7], part, atol=1e-4)
    for name in ("pos", "loop.in", "loop.step", "l0.norm1.b", "l0.norm1.alpha", "l0.mix.g", "l1.mix.uk", "l2.ls2", "l3.ls1", "final.norm.b"):
        assert not torch.allclose(oracle.logits(MIXED, dict(t, **{name: t[name] * 0.5}), toks), full, atol=1e-3), name


# ------------------------------------------------------------------ scheduler limit
def test_scheduler_respects_the_model_context():
    from cuteafd_b200.engine.kv import PagePool
    from cuteafd_b200.serving.runner import FakeRunner
    from cuteafd_b200.serving.scheduler import NgramDrafter, Request, Scheduler
    done = {}
    runner = FakeRunner()
    top, run = [], runner.run
    runner.run = lambda rows: (top.append(max(r.start_pos + len(r.tokens) for r in rows)), run(rows))[1]
    sched = Scheduler(runner, PagePool(64), max_context=40, drafter=NgramDrafter())
    cb = lambda rid: lambda toks, fin, why: done.setdefault(rid, []).append((list(toks), fin, why))
    assert not sched.submit(Request("long", list(range(41)), on_token=cb("long")))
    assert sched.submit(Request("fits", [1, 2] * 15, max_tokens=1000, on_token=cb("fits")))
    assert sched.submit(Request("edge", list(range(40)), max_tokens=9, on_token=cb("edge")))
    sched.run_until_idle()
    assert done["long"][0][2].startswith("error: prompt")
    assert sum(len(t) for t, _, _ in done["fits"]) == 11 and sum(len(t) for t, _, _ in done["edge"]) == 1 and max(top) <= 40


# ------------------------------------------------------------------ trace replay bookkeeping (no engine)
def test_trace_replay_tracks_requests_and_frees_pages(tmp_path, capsys):
    from types import SimpleNamespace

    from cuteafd_b200.engine.kv import PagePool
    from cuteafd_b200.serving import trace

    class Runner:
        def __init__(self):
            self.seen, self.forgot = [], []

        def run(self, rows):
            self.seen.append([(r.state.req.rid, r.start_pos, list(r.tokens), list(r.want_logits)) for r in rows])
            for r in rows:
                r.state.seq.ensure(rep.pool, r.start_pos + len(r.tokens))
            n = sum(len(r.want_logits) for r in rows)
            self.last_lane = SimpleNamespace(logits=torch.arange(64.0).reshape(16, 4)[:max(n, 1)])

        def forget(self, st):
            self.forgot.append(st.req.rid)

    rep = trace.TraceReplay.__new__(trace.TraceReplay)
    rep.pool, rep.runner, rep.live = PagePool(4), Runner(), {}
    assert rep.step([{"id": "a", "tokens": [1, 2, 3], "want": []}, {"id": "b", "tokens": [4], "want": [0]}], []).shape == (1, 4)
    assert rep.step([{"id": "b", "tokens": [5, 6], "want": []}], []) is None
    assert rep.step([{"id": "a", "tokens": [7] * 62, "want": [0, 61]}], ["a"]).shape == (2, 4)
    assert rep.runner.seen[2] == [("a", 3, [7] * 62, [0, 61])] and rep.runner.seen[1] == [("b", 1, [5, 6], [])]
    assert rep.runner.forgot == ["a"] and rep.pool.n_free == 2
    rep.step([{"id": "a", "tokens": [9], "want": []}], ["a", "b"])
    assert rep.runner.seen[3] == [("a", 0, [9], [])] and rep.pool.n_free == 3 and not rep.live


def test_subset_build_follows_sources():
    from cuteafd_b200 import build
    stems, extra = build.SUBSETS["latent_stack"]
    assert all((build.CSRC / f"{s}.cu").exists() for s in stems)
    assert build.source_hash(stems, extra) != build.source_hash(stems) != build.source_hash()
