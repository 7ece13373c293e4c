"""Mixed stacks without a GPU: configuration, snapshot reading, weight layout, planning, pooled rows on pages, the oracle's mechanisms against direct
formulas."""
import json
import math

import pytest
import torch

from mixed_stack_models import BLEND, CONFIGS, ODD, PLAIN, make_tensors, masters_of, write_snapshot

from cuteafd_b200.config import AttentionSpec, from_hf_config, spec_by_name, spec_from_json, spec_to_json
from cuteafd_b200.ref import mixed_stack as oracle


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_config_and_spec_round_trip(name):
    cfg = CONFIGS[name]
    spec = from_hf_config(cfg)
    assert (spec.family, spec.stack, spec.n_layers, spec.rms_eps, spec.embed_scale, spec.side_dim) == \
        ("sikazen", "mixed", len(cfg["layers"]), cfg["norm"]["eps"], cfg["embedding"]["scale"], (cfg.get("token_side") or {}).get("dim", 0))
    for b, layer in zip(spec.blocks, cfg["layers"]):
        m, a, r = layer["mixer"], b.attn, b.rec
        if layer["type"] == "hgrn2":
            assert a is None and (r.kind, r.heads, r.dim, r.vdim) == ("hgrn2", m["heads"], m["dim"], m["vdim"])
        elif layer["type"] == "attention":
            mask = m.get("mask") or {"size": 0, "pool": 0}
            assert (a.kind, a.n_heads, a.n_kv_heads, a.head_dim, a.v_head_dim, a.softmax_scale, a.window, a.pool) == \
                ("conv_gqa", m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], mask["size"], mask["pool"])
            assert (a.rope_dims, a.rope_theta, a.rope_divisor, a.rope_interleaved, a.qk_norm_unit, a.qkv_bias, a.conv_taps) == \
                (m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling", {"factor": 1.0})["factor"], False, True, True, 0)
        else:
            assert (a.kind, a.n_heads, a.head_dim, a.rope_dims, a.v_head_dim, a.kv_lora_rank, a.q_lora_rank, a.softmax_scale, a.sink, a.rope_theta) == \
                ("latent", m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"], m["scale"], True, m["rot"]["base"])
        assert (b.ffn is None) == (layer["mlp"] is None) and (b.ffn is None or (b.ffn.intermediate, b.ffn.activation) == (layer["mlp"]["ff"], "silu_glu"))
    lp = cfg.get("loop")
    order = [i for i, _ in oracle.layer_order(len(cfg["layers"]), lp)]
    assert [i for i, _ in spec.layer_runs()] == order and [bool(t) for _, t in spec.layer_runs()] == [x for _, x in oracle.layer_order(len(cfg["layers"]), lp)]
    assert spec_from_json(json.loads(json.dumps(spec_to_json(spec)))) == spec


def test_bad_configurations_are_refused():
    for layer, path, value in ((1, ("mixer", "kv_heads"), 4), (1, ("mixer", "rot", "dims"), 42), (2, ("mixer", "rot", "dims"), 8), (0, ("type",), "other"), (0, ("mlp", "kind"), "other"),
                               (1, ("mixer", "mask", "pool"), -1)):
        c = json.loads(json.dumps(BLEND))
        at = c["layers"][layer]
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            from_hf_config(c)
    for loop in ({"start": 2, "stop": 2, "times": 2}, {"start": 0, "stop": 9, "times": 2}, {"start": 0, "stop": 1, "times": 0}):
        with pytest.raises(ValueError):
            from_hf_config(dict(BLEND, loop=loop))


def test_snapshot_reader_checks_names_and_shapes(tmp_path):
    from cuteafd_b200.loader.stack_checkpoint import read_mixed_masters
    t = make_tensors(BLEND)
    spec, m = masters_of(BLEND, t, tmp_path / "a")
    L = m["layers"]
    assert L[0]["norm1"] == float(t["l0.norm1"]) and m["final_norm"] == float(t["final.norm"]) and "norm2" not in L[3] and torch.equal(m["side"].float(), t["side.embed"])
    assert torch.equal(L[1]["k_b"].float(), t["l1.mix.k.b"]) and torch.equal(L[2]["dkv"].float(), t["l2.mix.dkv"]) and torch.equal(L[4]["lower"].float(), t["l4.mix.lower"])
    with pytest.raises(KeyError):
        read_mixed_masters(write_snapshot(BLEND, {k: v for k, v in t.items() if k != "l2.mix.sink"}, tmp_path / "b"), spec)
    for name, bad in (("l0.mix.lower", t["l0.mix.lower"][1:]), ("side.embed", t["side.embed"][:, 1:]), ("l2.mix.uq", t["l2.mix.uq"][:, 1:]), ("l1.norm1", torch.ones(2))):
        with pytest.raises(ValueError):
            read_mixed_masters(write_snapshot(BLEND, dict(t, **{name: bad}), tmp_path / name), spec)


def test_plan_reads_the_family(tmp_path):
    from cuteafd_b200.loader.plan import plan
    p = write_snapshot(BLEND, make_tensors(BLEND), tmp_path / "m")
    rep = plan(str(p), world=1, layout=True)
    assert rep.supported and rep.family == "sikazen" and rep.layout.pool_tokens > 0 and not plan(str(p), world=4, layout=True).supported
    spec = from_hf_config(BLEND)
    # runs: 0, 1, 2, 1, 2, 3, 4 - three planes of keys and values (4 heads of 128 + 192), two of latents (128 + 64); blocks of 6 in strips of 16 rows
    # a page (2 heads of 64 + 64), blocks of 20 in strips of 8
    assert spec.attention_runs("conv_gqa") == [1, 3, 5] and spec.attention_runs("latent") == [2, 4]
    assert spec.kv_bytes_per_token() == 2 * (3 * 4 * 320 + 2 * 192 + 2 * 16 / 64 * 256 + 8 / 64 * 4 * 320)
    rec = lambda H, d, v: H * (4 * (2 * d * v + 8 * (2 * d + v)) + 8)
    assert spec.state_bytes_per_seq(8) == rec(3, 24, 40) + rec(2, 64, 72)
    assert plan("sikazen", world=1, layout=True).supported and spec_by_name("sikazen", loop=(1, 3, 2)).stack == "mixed"


def test_weights_stack_what_reads_one_row():
    from cuteafd_b200.models.hyper_stack import place
    from cuteafd_b200.models.mixed_stack import input_segments, mixer_width
    for cfg in (BLEND, ODD):
        for b, layer in zip(from_hf_config(cfg).blocks, cfg["layers"]):
            cols, rows = place(input_segments(b))
            assert all(at % 8 == 0 for at, _ in cols.values()) and rows % 8 == 0
            ends = sorted((at, at + n) for at, n in cols.values())
            assert all(x[1] <= y[0] for x, y in zip(ends, ends[1:]))
            assert set(cols) == {"attention": {"qkv"}, "latent_attention": {"dq", "dkv"}, "hgrn2": {"rq", "rf", "rv"}}[layer["type"]]
            assert mixer_width(b) == layer["mixer"]["heads"] * layer["mixer"]["vdim"]


@pytest.mark.parametrize("pool", [1, 2, 3, 4, 5, 6, 7, 8, 9, 12, 16, 20, 63, 64, 65, 100, 500])
def test_pooled_rows_stand_with_the_pages_of_their_tokens(pool):
    """A block's row belongs to a page the sequence holds by the time the block is complete, no two blocks share a row, and strips of eight are whole."""
    from cuteafd_b200.ops import pooled_page_rows
    rows = pooled_page_rows(pool)
    assert rows == AttentionSpec(kind="conv_gqa", pool=pool).pooled_page_rows and rows % 8 == 0
    seen = set()
    for b in range(4000 // pool):
        s = b >> 3
        j = (s * pool) >> 3
        at = (s - (8 * j + pool - 1) // pool) * 8 + (b & 7)
        assert 0 <= at < rows and j <= (b * pool + pool - 1) // 64 and (j, at) not in seen
        seen.add((j, at))


# ------------------------------------------------------------------ the oracle, mechanism by mechanism
def test_oracle_norms_and_gelu():
    x = torch.tensor([[3.0, 4.0]])
    assert torch.allclose(oracle.unit_norm(x, 0.5), x / math.sqrt(13.0))
    z = 0.7
    assert abs(float(oracle.gelu_tanh(torch.tensor(z))) - 0.5 * z * (1 + math.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))) < 1e-6


def test_oracle_rotations():
    x = torch.zeros(3, 1, 5)
    x[:, 0] = torch.tensor([1.0, 2.0, 3.0, 4.0, 7.0])
    for p in range(3):
        c, s = (math.cos(p / 4), math.cos(p * 0.1 / 4)), (math.sin(p / 4), math.sin(p * 0.1 / 4))
        inter = [c[0] - 2 * s[0], 2 * c[0] + s[0], 3 * c[1] - 4 * s[1], 4 * c[1] + 3 * s[1], 7.0]
        half = [c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + s[0], 4 * c[1] + 2 * s[1], 7.0]
        rot = {"dims": 4, "base": 100.0, "scaling": {"factor": 4.0}}
        assert torch.allclose(oracle.turn(x, rot, True)[p, 0], torch.tensor(inter), atol=1e-6)
        assert torch.allclose(oracle.turn(x, rot, False)[p, 0], torch.tensor(half), atol=1e-6)
    assert torch.equal(oracle.turn(x, None, True), x)


def test_oracle_window_and_blocks():
    assert [oracle.window_tokens(i, 3) for i in (0, 2, 5)] == [[0], [0, 1, 2], [3, 4, 5]] and oracle.window_tokens(3, None) == [0, 1, 2, 3]
    # blocks of four, a window of three: block 0 ends at 3, position 5 still has it in front of its window's edge at 3, position 6 sees it
    assert [oracle.pooled_blocks(i, 3, 4) for i in (4, 5, 6, 9, 10)] == [[], [], [0], [0], [0, 1]]
    assert oracle.pooled_blocks(9, 1, 1) == list(range(9)) and oracle.pooled_blocks(9, None, 4) == []
    torch.manual_seed(0)
    q, k, v = torch.randn(12, 2, 3), torch.randn(12, 1, 3), torch.randn(12, 1, 5)
    o = oracle.pooled_attention(q, k, v, 0.7, 3, 4)
    keys = torch.cat([k[:4, 0].mean(0, True), k[4:8, 0].mean(0, True), k[9:, 0]])
    vals = torch.cat([v[:4, 0].mean(0, True), v[4:8, 0].mean(0, True), v[9:, 0]])
    for h in range(2):
        assert torch.allclose(o[11, h], torch.softmax(keys @ q[11, h] * 0.7, 0) @ vals, atol=1e-6)
        # position 5: token 2 has left the window, its block is not seen yet
        assert torch.allclose(o[5, h], torch.softmax(k[3:6, 0] @ q[5, h] * 0.7, 0) @ v[3:6, 0], atol=1e-6)


def test_oracle_sink_and_forget_gate():
    p = oracle.sink_softmax(torch.zeros(1, 3), torch.tensor(math.log(2.0)))
    assert torch.allclose(p, torch.full((1, 3), 0.2))
    f = oracle.forget_gate(torch.tensor([0.0, 50.0, -50.0]), torch.tensor([0.5, 0.25, 0.25]))
    assert torch.allclose(f, torch.tensor([0.75, 1.0, 0.25]))
    # one channel, one value: a state that forgets a quarter a step and takes what it gives up
    t = {"m.q": torch.tensor([[2.0, 0.0]]), "m.f": torch.zeros(1, 2), "m.f.b": torch.zeros(1), "m.lower": torch.tensor([0.5]), "m.v": torch.tensor([[0.0, 1.0]]), "m.norm": torch.tensor([3.0]),
         "m.o": torch.tensor([[1.0], [0.0]])}
    h = torch.tensor([[1.0, 4.0], [1.0, -8.0]])
    y = oracle.hgrn2_mixer(h, t, "m", {"heads": 1, "dim": 1, "vdim": 1}, 1.0)
    q = 2.0 / (1 + math.exp(-2.0))
    o = [q * 1.0, q * (0.75 * 1.0 - 2.0)]
    assert torch.allclose(y[:, 0], torch.tensor([3.0 * x / math.sqrt(x * x + 1.0) for x in o]), atol=1e-6)


def test_oracle_latent_attention_is_attention_over_expanded_rows():
    torch.manual_seed(1)
    T, W, H, d, dr, dv, r, rq = 6, 10, 2, 4, 2, 3, 5, 7
    m = {"heads": H, "dim": d, "rot_dim": dr, "vdim": dv, "kv_rank": r, "q_rank": rq, "scale": 0.3, "rot": {"dims": dr, "base": 10.0}}
    t = {f"m.{n}": torch.randn(*s) for n, s in {"dq": (rq, W), "dq.norm": (rq,), "uq": (H * (d + dr), rq), "dkv": (r + dr, W), "dkv.norm": (r,), "uk": (H * d, r), "uv": (H * dv, r), "sink": (H,),
                                                "o": (W, H * dv)}.items()}
    h = torch.randn(T, W)
    got = oracle.latent_mixer(h, t, "m", m, 1e-5)
    rms = lambda x, g: x / torch.sqrt((x * x).mean(-1, keepdim=True) + 1e-5) * g
    q = (rms(h @ t["m.dq"].T, t["m.dq.norm"]) @ t["m.uq"].T).view(T, H, d + dr)
    kv = h @ t["m.dkv"].T
    c = rms(kv[:, :r], t["m.dkv.norm"])
    out = torch.zeros(T, H, dv)
    for i in range(T):
        for hd in range(H):
            w = [math.exp(float(t["m.sink"][hd]))]
            for j in range(i + 1):
                a, b = (complex(float(x[0]), float(x[1])) * complex(math.cos(p), math.sin(p)) for x, p in ((q[i, hd, d:], i), (kv[j, r:], j)))
                w.append(math.exp(0.3 * (float(q[i, hd, :d] @ (t["m.uk"][hd * d:(hd + 1) * d] @ c[j])) + (a * b.conjugate()).real)))
            for j in range(i + 1):
                out[i, hd] += w[j + 1] / sum(w) * (t["m.uv"][hd * dv:(hd + 1) * dv] @ c[j])
    assert torch.allclose(got, out.reshape(T, -1) @ t["m.o"].T, atol=1e-4)


def test_oracle_order_of_layers_and_side_input():
    assert oracle.layer_order(4, {"start": 1, "stop": 3, "times": 3}) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    t = {"side.embed": torch.tensor([[9.0, 9.0, 1.0, 2.0], [9.0, 9.0, 3.0, 4.0]]), "l1.side.gate": torch.eye(2), "l1.side.proj": torch.eye(2), "l1.side.norm": torch.tensor([1.0, 10.0])}
    x, g = torch.tensor([[0.5, -1.0]]), oracle.gelu_tanh(torch.tensor([0.5, -1.0]))
    y = g * torch.tensor([3.0, 4.0])
    assert torch.allclose(oracle.side_input(x, torch.tensor([1]), 1, t, 2, 0.0)[0], y / y.pow(2).mean().sqrt() * torch.tensor([1.0, 10.0]), atol=1e-6)


def test_oracle_stack_is_causal_and_uses_every_tensor():
    for cfg in (BLEND, ODD, PLAIN):
        t = {k: v.double() for k, v in make_tensors(cfg, 3).items()}
        toks = torch.randint(0, cfg["vocab"], (12,), generator=torch.Generator().manual_seed(1)).tolist()
        full, part = oracle.logits(cfg, t, toks), oracle.logits(cfg, t, toks[:7])
        assert torch.allclose(full[:7], part, atol=1e-9)
        for n in t:
            changed = t[n] * 0.5 - 0.1 * torch.arange(t[n].numel()).reshape(t[n].shape).remainder(3)
            assert not torch.allclose(oracle.logits(cfg, dict(t, **{n: changed}), toks), full, atol=1e-6), n


def test_subset_build_names_existing_sources():
    from cuteafd_b200 import build
    stems, _ = build.SUBSETS["mixed_stack"]
    assert all((build.CSRC / f"{s}.cu").exists() for s in stems)
