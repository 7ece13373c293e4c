"""Hyper-connected stacks without a GPU: configuration, snapshot reading, weight layout, planning, the oracle's mechanisms against direct formulas."""
import json
import math

import pytest
import torch

from hyper_stack_models import CONFIGS, MIXED, ODD, PLAIN, RANK, make_tensors, masters_of, variant, write_snapshot

from cuteafd_b200.config import from_hf_config, spec_by_name, spec_from_json, spec_to_json
from cuteafd_b200.ref import hyper_stack as oracle


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_config_and_spec_round_trip(name):
    cfg = CONFIGS[name]
    spec = from_hf_config(cfg)
    assert (spec.family, spec.stack, spec.n_layers, spec.rms_eps, spec.streams) == ("vozetar", "hyper", len(cfg["layers"]), cfg["norm"]["eps"], cfg["streams"])
    pairs = (cfg.get("embedding") or {}).get("bigram")
    assert (spec.pair_table is None) == (pairs is None) and (pairs is None or vars(spec.pair_table) == pairs)
    for b, layer in zip(spec.blocks, cfg["layers"]):
        m, mlp, a, r = layer["mixer"], layer["mlp"], b.attn, b.rec
        am = m if layer["type"] == "attention" else m["left"]
        mask = am.get("mask") or {"size": 0, "keep_first": 0}
        assert (a.n_heads, a.n_kv_heads, a.head_dim, a.v_head_dim, a.softmax_scale, a.rope_dims, a.rope_theta, a.conv_taps, a.window, a.keep_first) == \
            (am["heads"], am["kv_heads"], am["dim"], am["vdim"], am["scale"], am["rot"]["dims"], am["rot"]["base"], am.get("conv", 0), mask["size"], mask["keep_first"])
        assert (a.rope_interleaved, a.qkv_bias, a.out_bias, a.sink, a.qk_norm_whole, a.values_are_keys, a.gate_width) == {
            "attention": (False, True, True, True, False, False, am["heads"] * am["vdim"]), "parallel": (True, True, False, True, False, False, 0),
            "parallel_2": (True, False, False, False, True, True, am["heads"])}[layer["type"]]
        if layer["type"] == "attention":
            assert r is None
        else:
            rm = m["right"]
            assert (r.heads, r.dim, r.vdim) == (rm["heads"], rm["dim"], rm["vdim"])
            assert (r.kind, b.merge_norm, b.merge_scales) == (("retention", False, (m["left_scale"], m["right_scale"])) if layer["type"] == "parallel" else ("gla", True, (0.5, 0.5)))
            assert (list(r.decay), r.rope_dims, r.rope_theta) == (rm["decay"], rm["rot"]["dims"], rm["rot"]["base"]) if r.kind == "retention" else r.tau == rm["tau"]
        if mlp is None:
            assert b.ffn is None and b.moe is None
        elif mlp["kind"] == "dense":
            assert b.moe is None and (b.ffn.intermediate, b.ffn.activation) == (mlp["ff"], "silu_glu")
        else:
            e, g = b.moe, mlp["router"].get("groups") or {"count": 1, "keep": 1}
            assert (e.n_experts, e.top_k, e.intermediate, e.n_group, e.topk_group, e.scoring, e.normalize) == \
                (mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"], g["count"], g["keep"], "sigmoid", False)
            assert (e.n_shared, e.shared_inter if e.n_shared else 0) == ((1, mlp["shared"]["ff"]) if mlp.get("shared") else (0, 0))
    assert spec_from_json(json.loads(json.dumps(spec_to_json(spec)))) == spec


def test_bad_configurations_are_refused():
    bad = []
    for layer, path, value in ((1, ("mixer", "kv_heads"), 3), (0, ("mixer", "right", "decay"), [0.5]), (0, ("mixer", "left", "rot", "dims"), 42), (2, ("mixer", "left", "vdim"), 40),
                               (0, ("mixer", "right", "rot", "dims"), 26), (0, ("type",), "other"), (1, ("mlp", "kind"), "other"), (1, ("mlp", "router", "groups", "count"), 5),
                               (1, ("mlp", "router", "top"), 7)):
        c = json.loads(json.dumps(MIXED))
        at = c["layers"][layer]
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        bad.append(c)
    for c in bad + [variant(MIXED, streams=0)]:
        with pytest.raises(ValueError):
            from_hf_config(c)


def test_snapshot_reader_checks_names_and_shapes(tmp_path):
    from cuteafd_b200.loader.stack_checkpoint import read_hyper_masters
    t = make_tensors(MIXED)
    spec, m = masters_of(MIXED, t, tmp_path / "a")
    L = m["layers"]
    assert torch.equal(L[1]["k_conv"].float(), t["l1.mix.k.conv"]) and torch.equal(L[1]["o_b"].float(), t["l1.mix.o.b"]) and "q_conv" not in L[0] and "wv" not in L[2]
    assert torch.equal(L[2]["a2"].float(), t["l2.mix.right.a2"]) and torch.equal(L[2]["merge_norms"][1].float(), t["l2.mix.right.out"]) and "ws_gate" not in L[2]
    assert torch.equal(L[1]["w_down"][7].float(), t["l1.mlp.e7.down"]) and torch.equal(L[0]["hc2"][2].float(), t["l0.hc2.mix"]) and "hc2" not in L[3]
    assert torch.equal(m["pairs"].float(), t["bigram"])
    with pytest.raises(KeyError):
        read_hyper_masters(write_snapshot(MIXED, {k: v for k, v in t.items() if k != "l0.mix.left.sink"}, tmp_path / "b"), spec)
    for name, bad in (("l2.mix.left.q.norm", t["l2.mix.left.q.norm"][1:]), ("l2.mix.right.a2", t["l2.mix.right.a2"][:, 1:]), ("bigram", t["bigram"][1:])):
        with pytest.raises(ValueError):
            read_hyper_masters(write_snapshot(MIXED, dict(t, **{name: bad}), tmp_path / name), spec)


def test_plan_reads_the_family(tmp_path):
    from cuteafd_b200.loader.plan import plan
    p = write_snapshot(MIXED, make_tensors(MIXED), tmp_path / "m")
    rep = plan(str(p), world=1, layout=True)
    assert rep.supported and rep.family == "vozetar" and rep.layout.pool_tokens > 0 and not plan(str(p), world=4, layout=True).supported
    spec = from_hf_config(MIXED)
    # every layer keeps keys and values, in rows of the widest: layer 2 (three heads of 64 + 64 padded elements)
    assert spec.kv_layers() == [0, 1, 2, 3] and spec.kv_bytes_per_token() == 4 * 384 * 2
    vp = lambda n: -(-n // 4) * 4
    rec = lambda H, d, v: H * (4 * (2 * d * vp(v) + 8 * (2 * d + vp(v))) + 8)
    assert spec.state_bytes_per_seq(8) == (9 * 4 + rec(3, 24, 40) + rec(4, 20, 36) + (4 * 40 + 2 * 96) * 10 * 2 + (6 + 3) * 48 * 11 * 2 + (4 * 72 + 136) * 9 * 2)
    assert plan("vozetar", world=1, layout=True).supported and spec_by_name("vozetar", experts=64).stack == "hyper"


def test_weights_stack_what_reads_one_row(tmp_path):
    """The input projection's segments start on multiples of 8 and hold the stored rows; added mixers share an output projection."""
    from cuteafd_b200.models.hyper_stack import input_segments, place
    for cfg in (MIXED, ODD):
        spec = from_hf_config(cfg)
        for b, layer in zip(spec.blocks, cfg["layers"]):
            segs = input_segments(b, 5)
            cols, rows = place(segs)
            assert all(at % 8 == 0 for at, _ in cols.values()) and rows % 8 == 0 and rows >= sum(n for _, n in segs)
            ends = sorted((at, at + n) for at, n in cols.values())
            assert all(x[1] <= y[0] for x, y in zip(ends, ends[1:]))
            assert ("gate" in cols) == (layer["type"] != "parallel") and ("a1" in cols) == (layer["type"] == "parallel_2") and ("rv" in cols) == (layer["type"] != "attention")


# ------------------------------------------------------------------ the oracle, mechanism by mechanism
def test_oracle_pair_rows():
    assert oracle.bigram_rows([4, 9, 9], {"buckets": 10, "mul_prev": 3, "mul_cur": 5}) == [10, (12 + 45) % 10, (27 + 45) % 10]


def test_oracle_streams():
    x = [torch.tensor([[1.0]]), torch.tensor([[10.0]]), torch.tensor([[100.0]])]
    assert float(oracle.collapse(x, torch.tensor([1.0, 2.0, 3.0]))) == 321.0
    mix = torch.tensor([[1.0, 2.0, 0.0], [0.0, 1.0, 0.0], [3.0, 0.0, 1.0]])             # [from, to]
    out = oracle.spread(x, mix, torch.tensor([0.5, 0.0, -1.0]), torch.tensor([[4.0]]))
    assert [float(v) for v in out] == [1 + 300 + 2, 2 + 10, 100 - 4]


def test_oracle_rotations():
    x = torch.zeros(3, 1, 5)
    x[:, 0] = torch.tensor([1.0, 2.0, 3.0, 4.0, 7.0])
    for p in range(3):
        c, s = (math.cos(p), math.cos(p * 0.1)), (math.sin(p), math.sin(p * 0.1))
        inter = [c[0] - 2 * s[0], 2 * c[0] + s[0], 3 * c[1] - 4 * s[1], 4 * c[1] + 3 * s[1], 7.0]
        half = [c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + s[0], 4 * c[1] + 2 * s[1], 7.0]
        assert torch.allclose(oracle.rotate(x, 4, 100.0, True)[p, 0], torch.tensor(inter), atol=1e-6)
        assert torch.allclose(oracle.rotate(x, 4, 100.0, False)[p, 0], torch.tensor(half), atol=1e-6)


def test_oracle_window_sink_and_groups():
    see = oracle.visible(7, 2, 3)
    assert [see[i].nonzero().flatten().tolist() for i in (0, 2, 3, 6)] == [[0], [0, 1, 2], [0, 1, 2, 3], [0, 1, 2, 5, 6]]
    assert oracle.visible(4, None, 0).equal(torch.ones(4, 4, dtype=torch.bool).tril())
    torch.manual_seed(0)
    q, k, v = torch.zeros(4, 4, 3), torch.randn(4, 2, 3), torch.randn(4, 2, 5)
    o = oracle.attend(q, k, v, 1.0, oracle.visible(4, None, 0), torch.tensor([0.0, 1.0, -50.0, math.log(4.0)]))
    assert torch.allclose(o[3, 0], v[:, 0].sum(0) / 5) and torch.allclose(o[3, 1], v[:, 0].sum(0) / (4 + math.e))
    assert torch.allclose(o[3, 2], v[:, 1].mean(0)) and torch.allclose(o[3, 3], v[:, 1].sum(0) / 8) and torch.allclose(o[0, 3], v[0, 1] / 5)


def test_oracle_linear_attention():
    torch.manual_seed(1)
    T, H, d, dv = 5, 2, 3, 4
    q, k, v, a = torch.randn(T, H, d), torch.randn(T, H, d), torch.randn(T, H, dv), torch.rand(T, H, d)
    o = oracle.linear_attention(q, k, v, a)
    for t in range(T):
        for h in range(H):
            want = sum(float((q[t, h] * k[j, h] * a[j + 1:t + 1, h].prod(0)).sum()) * v[j, h] for j in range(t + 1))
            assert torch.allclose(o[t, h], want, atol=1e-5)


def test_oracle_routing():
    s = torch.tensor([0.9, 0.1, 0.2, 0.6, 0.55, 0.3])                     # groups of two: 1.0, 0.8, 0.85
    assert oracle.choose_experts(s, 3, {"count": 3, "keep": 2}) == [0, 4, 5]
    assert oracle.choose_experts(s, 2, {"count": 6, "keep": 3}) == [0, 3] and oracle.choose_experts(s, 3, None) == [0, 3, 4]
    t = {"m.router": torch.tensor([[2.0], [1.0], [-1.0]])}
    for e in range(3):
        t[f"m.e{e}.gate"] = t[f"m.e{e}.up"] = t[f"m.e{e}.down"] = torch.tensor([[float(e + 1)]])
    y = oracle.feed_forward(torch.tensor([[0.5]]), t, "m", {"kind": "moe", "router": {"experts": 3, "top": 2}, "expert": {"ff": 1}})
    sg, ex = (lambda z: 1 / (1 + math.exp(-z))), (lambda w: (0.5 * w) ** 2 * (1 / (1 + math.exp(-0.5 * w))) * w)
    assert abs(float(y) - (sg(1.0) * ex(1) + sg(0.5) * ex(2))) < 1e-6


def test_oracle_stack_is_causal_and_uses_every_tensor():
    for name, cfg in (("mixed", MIXED), ("odd", ODD), ("plain", PLAIN)):
        t = {k: v.double() for k, v in make_tensors(cfg, 3, RANK[name]).items()}
        toks = torch.randint(0, cfg["vocab"], (12,), generator=torch.Generator().manual_seed(1)).tolist()
        full, part = oracle.logits(cfg, t, toks), oracle.logits(cfg, t, toks[:7])
        assert torch.allclose(full[:7], part, atol=1e-9)
        for n in t:
            if ".mlp.e" in n:                                             # not every expert is chosen by twelve tokens
                continue
            changed = t[n] * 0.5 - 0.1 * torch.arange(t[n].numel()).reshape(t[n].shape).remainder(3)
            assert not torch.allclose(oracle.logits(cfg, dict(t, **{n: changed}), toks), full, atol=1e-6), n


def test_subset_build_names_existing_sources():
    from cuteafd_b200 import build
    stems, _ = build.SUBSETS["hyper_stack"]
    assert all((build.CSRC / f"{s}.cu").exists() for s in stems)
