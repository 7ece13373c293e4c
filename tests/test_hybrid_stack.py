"""Hybrid recurrent / windowed-attention stacks without a GPU: configuration, snapshot reading, planning, the oracle's mechanisms against direct
formulas, state slots that step back."""
import json
import math
from types import SimpleNamespace

import pytest
import torch

from hybrid_stack_models import CONFIGS, MIXED, ODD, RECURRENT, make_tensors, masters_of, variant, write_snapshot

from cuteafd_b200.config import from_hf_config, spec_by_name, spec_from_json, spec_to_json
from cuteafd_b200.ref import hybrid_stack as oracle


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_config_and_spec_round_trip(name):
    cfg = CONFIGS[name]
    spec = from_hf_config(cfg)
    assert (spec.family, spec.stack, spec.n_layers, spec.rms_eps) == ("tudilix", "hybrid", len(cfg["layers"]), cfg["norm"]["eps"])
    assert (spec.residual_mult, spec.logit_softcap) == (cfg["residual_mult"], cfg["logit_softcap"])
    for b, layer in zip(spec.blocks, cfg["layers"]):
        m = layer["mixer"]
        if layer["type"] == "rglru":
            assert b.attn is None and (b.rec.width, b.rec.blocks, b.rec.conv_taps) == (m["width"], m["blocks"], m["conv"])
        else:
            a = b.attn
            assert b.rec is None and (a.n_heads, a.n_kv_heads, a.head_dim, a.v_head_dim, a.window, a.conv_taps, a.softmax_scale, a.rope_dims, a.rope_theta) == \
                (m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"], m["conv"], m["scale"], m["rot"]["dims"], m["rot"]["base"])
            assert a.kv_from == m.get("kv_from", -1) and (a.rope_scaling is None) == (m["rot"]["scaling"] is None)
        assert (b.ffn is None) == (layer["mlp"] is None) and (b.ffn is None or (b.ffn.intermediate, b.ffn.limit) == (layer["mlp"]["ff"], layer["mlp"]["limit"]))
    assert spec_from_json(json.loads(json.dumps(spec_to_json(spec)))) == spec


def test_bad_configurations_are_refused():
    bad = []
    for layer, key, value in ((1, "kv_heads", 4), (1, "kv_from", 3), (4, "kv_from", 1), (0, "blocks", 7), (3, "kv_from", 0), (1, "kv_from", 1)):
        c = json.loads(json.dumps(MIXED))
        c["layers"][layer]["mixer"][key] = value
        bad.append(c)
    c = json.loads(json.dumps(MIXED))
    c["layers"][4]["mixer"]["rot"]["dims"] = 74
    bad += [c, variant(MIXED, layers=[dict(MIXED["layers"][0], type="other")]), variant(MIXED, layers=[dict(MIXED["layers"][0], mlp={"kind": "moe", "ff": 8, "limit": 1.0})])]
    for c in bad:
        with pytest.raises(ValueError):
            from_hf_config(c)


def test_snapshot_reader_checks_names_and_shapes(tmp_path):
    from cuteafd_b200.loader.stack_checkpoint import read_hybrid_masters
    t = make_tensors(MIXED)
    spec, m = masters_of(MIXED, t, tmp_path / "a")
    assert torch.equal(m["layers"][1]["k_conv"].float(), t["l1.mix.k.conv"]) and "wk" not in m["layers"][3] and "w_up" not in m["layers"][2]
    assert torch.equal(m["layers"][0]["ra"].float(), t["l0.mix.ra"]) and torch.equal(m["final_norm"].float(), t["final.norm"])
    with pytest.raises(KeyError):
        read_hybrid_masters(write_snapshot(MIXED, {k: v for k, v in t.items() if k != "l2.mix.lam"}, tmp_path / "b"), spec)
    with pytest.raises(ValueError):
        read_hybrid_masters(write_snapshot(MIXED, dict(t, **{"l1.mix.v.conv": t["l1.mix.v.conv"][:, 1:]}), tmp_path / "c"), spec)


def test_plan_reads_the_family(tmp_path):
    from cuteafd_b200.loader.plan import plan
    p = write_snapshot(MIXED, make_tensors(MIXED), tmp_path / "m")
    rep = plan(str(p), world=1, layout=True)
    assert rep.supported and rep.family == "tudilix" and rep.layout.pool_tokens > 0 and not plan(str(p), world=4, layout=True).supported
    spec = from_hf_config(MIXED)
    # layers 1 and 4 keep keys and values, in rows of the wider one: layer 4 (one head of 128 + 192 padded elements); layer 3 reads layer 1's
    assert spec.kv_layers() == [1, 4] and spec.kv_bytes_per_token() == 2 * 320 * 2
    assert spec.state_bytes_per_seq(8) == (120 * (10 * 2 + 9 * 4) + 96 * (11 * 2 + 9 * 4)) + (6 * 40 + 2 * 64) * 11 * 2 + 160 * 9 * 2 + (3 * 72 + 208) * 10 * 2
    assert plan("tudilix", world=1, layout=True).supported and spec_by_name("tudilix").stack == "hybrid"
    r = write_snapshot(RECURRENT, make_tensors(RECURRENT), tmp_path / "r")
    assert plan(str(r), world=1, layout=True).supported and from_hf_config(RECURRENT).kv_bytes_per_token() == 0


# ------------------------------------------------------------------ the oracle, mechanism by mechanism
def test_oracle_norm_weights_are_distances_from_one():
    y = oracle.centred_norm(torch.tensor([[3.0, 4.0]]), torch.tensor([0.0, 1.0]), 0.5)
    assert torch.allclose(y, torch.tensor([[3.0, 8.0]]) / math.sqrt(12.5 + 0.5))


def test_oracle_convolution():
    u, w = torch.tensor([[1.0], [10.0], [100.0]]), torch.tensor([[0.5, 2.0, 3.0]])
    assert oracle.causal_conv(u, w).flatten().tolist() == [3.0, 2.0 + 30.0, 0.5 + 20.0 + 300.0]
    assert oracle.causal_conv(u, torch.tensor([[4.0]]), torch.tensor([1.0])).flatten().tolist() == [5.0, 41.0, 401.0]


def test_oracle_rotation_and_yarn():
    rot = {"dims": 4, "base": 100.0, "scaling": None}
    x = torch.zeros(3, 1, 5)
    x[:, 0, 0], x[:, 0, 3], x[:, 0, 4] = 1.0, 2.0, 7.0
    y = oracle.rotate(x, rot)
    for p in range(3):
        assert torch.allclose(y[p, 0], torch.tensor([math.cos(p), math.sin(p), -2 * math.sin(p * 0.1), 2 * math.cos(p * 0.1), 7.0]), atol=1e-6)
    sc = {"factor": 4.0, "original": 128, "fast": 8.0, "slow": 2.0}
    freq, amp = oracle.rope_frequencies({"dims": 16, "base": 50.0, "scaling": sc})
    edge = lambda turns: 16 * math.log(128 / (2 * math.pi * turns)) / (2 * math.log(50.0))
    lo, hi = math.floor(edge(8.0)), math.ceil(edge(2.0))
    assert 0 < lo < hi < 8 and amp == 0.1 * math.log(4.0) + 1
    assert freq[:lo + 1] == [50.0 ** (-i / 8) for i in range(lo + 1)]                                  # fast turns stay
    assert all(abs(freq[i] - 50.0 ** (-i / 8) / 4) < 1e-12 for i in range(hi, 8))                       # slow ones are stretched
    mid = (lo + hi) // 2
    ramp = (mid - lo) / (hi - lo)
    assert abs(freq[mid] - 50.0 ** (-mid / 8) * (1 - ramp + ramp / 4)) < 1e-12
    none, _ = oracle.rope_frequencies({"dims": 4, "base": 10.0, "scaling": dict(sc, original=7.0, fast=1.2, slow=1.1)})      # both edges fall into one pair
    assert none[0] == 1.0 and abs(none[1] - 10.0 ** -0.5 / 4) < 1e-12


def test_oracle_window_and_groups():
    torch.manual_seed(0)
    see = oracle.visible(6, 3)
    assert [see[i].nonzero().flatten().tolist() for i in (0, 1, 2, 5)] == [[0], [0, 1], [0, 1, 2], [3, 4, 5]]
    assert oracle.visible(4, None).equal(torch.ones(4, 4, dtype=torch.bool).tril())
    q, k, v = torch.zeros(9, 4, 9), torch.eye(9)[:, None].repeat(1, 2, 1), torch.randn(9, 2, 3)
    q[8, 2, 4] = q[8, 1, 3] = 60.0                                  # the window of 5 keys behind row 8 starts at key 4
    o = oracle.attend(q, k, v, 1.0, 5)
    assert torch.allclose(o[8, 2], v[4, 1], atol=1e-5) and torch.allclose(o[8, 1], v[4:, 0].mean(0), atol=1e-5)
    assert torch.allclose(o[0], v[0].repeat_interleave(2, 0), atol=1e-6)


def test_oracle_recurrence():
    u, r, i = torch.tensor([[1.0, 2.0], [3.0, -1.0]]), torch.tensor([[0.5, 0.25], [1.0, 0.0]]), torch.tensor([[1.0, 0.5], [0.25, 1.0]])
    lam = torch.tensor([-2.0, 0.3])
    s = oracle.lru(u, r, i, lam)
    want = [0.0, 0.0]
    for t in range(2):
        for c in range(2):
            a = math.exp(-8.0 * float(r[t, c]) * math.log(1 + math.exp(float(lam[c]))))
            want[c] = a * want[c] + math.sqrt(1 - a * a) * float(i[t, c] * u[t, c])
        assert torch.allclose(s[t], torch.tensor(want))
    w, b = torch.tensor([[[1.0, 2.0], [0.0, 1.0]], [[3.0, 0.0], [0.0, 0.0]]]), torch.tensor([[0.0, 1.0], [0.0, -1.0]])
    g = oracle.block_gate(torch.tensor([[1.0, 2.0, 0.5, 9.0]]), w, b)
    assert torch.allclose(g, torch.sigmoid(torch.tensor([[5.0, 3.0, 1.5, -1.0]])))


def test_oracle_glu_and_softcap():
    y = oracle.clamped_glu(torch.tensor([3.0, -5.0, 0.5]), torch.tensor([-4.0, 9.0, 0.25]), 2.0)
    sg = lambda z: 1 / (1 + math.exp(-z))
    assert torch.allclose(y, torch.tensor([2 * sg(3.404) * -1.0, -5 * sg(-8.51) * 3.0, 0.5 * sg(0.851) * 1.25]))
    assert torch.allclose(oracle.softcap(torch.tensor([100.0, 1.0]), 4.0), torch.tensor([4.0 * math.tanh(25.0), 4.0 * math.tanh(0.25)]))
    assert torch.allclose(oracle.gelu_tanh(torch.tensor([1.3, -0.4])), torch.nn.functional.gelu(torch.tensor([1.3, -0.4]), approximate="tanh"))


def test_oracle_stack_is_causal_and_uses_every_tensor():
    for cfg in (MIXED, ODD):
        t = make_tensors(cfg, 3)
        toks = torch.randint(0, cfg["vocab"], (12,), generator=torch.Generator().manual_seed(1)).tolist()
        full, part = oracle.logits(cfg, t, toks), oracle.logits(cfg, t, toks[:7])
        assert torch.allclose(full[:7], part, atol=1e-4)
        for name in t:
            if cfg is ODD and name.startswith(("l2.mix.q", "l2.mix.k")):      # a window of one token: whatever the scores, it sees itself
                continue
            assert not torch.allclose(oracle.logits(cfg, dict(t, **{name: t[name] * 0.5 - 0.1}), toks), full, atol=1e-3), name


# ------------------------------------------------------------------ weights and state slots
def test_rope_tables_keep_what_fp32_rounds_off():
    from cuteafd_b200.models.hybrid_stack import rope_key, rope_tables
    spec = from_hf_config(MIXED)
    tables = rope_tables(spec, "cpu")
    assert len(tables) == 2
    for i in (1, 4):
        f, amp = tables[rope_key(spec.blocks[i].attn)]
        want, wamp = oracle.rope_frequencies(MIXED["layers"][i]["mixer"]["rot"])
        assert torch.allclose(f[0].double() + f[1].double(), torch.tensor(want, dtype=torch.float64), rtol=1e-13) and abs(amp - wamp) < 1e-12


def test_runner_lets_position_addressed_states_step_back():
    from cuteafd_b200.serving.runner import EngineRunner
    r = EngineRunner(SimpleNamespace(state_depth=4, max_seqs=2, reset_state_slots=lambda s: None), max_rows=64)
    a, b = object(), object()
    row = lambda st, pos, n: SimpleNamespace(state=st, start_pos=pos, tokens=[1] * n)
    s = r._slots_of([row(a, 0, 20), row(b, 0, 3)])
    assert sorted(s) == [0, 1]
    with pytest.raises(RuntimeError, match="step back"):
        r._slots_of([row(a, 19, 1)])                  # a long run keeps its last state only
    assert r._slots_of([row(a, 20, 4)]) == s[:1]
    assert r._slots_of([row(a, 22, 3)]) == s[:1]      # two of four drafted rows were rejected
    assert r._slots_of([row(a, 22, 1)]) == s[:1]
    with pytest.raises(RuntimeError, match="step back"):
        r._slots_of([row(a, 21, 1)])                  # only the last step's rows can be taken back
    r.forget(b)
    with pytest.raises(RuntimeError, match="cached pages"):
        r._slots_of([row(object(), 64, 1)])
    assert r._slots_of([row(object(), 0, 1)]) == s[1:]


def test_subset_build_names_existing_sources():
    from cuteafd_b200 import build
    stems, _ = build.SUBSETS["hybrid_stack"]
    assert all((build.CSRC / f"{s}.cu").exists() for s in stems)
