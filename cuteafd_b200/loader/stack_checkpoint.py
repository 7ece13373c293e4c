"""Snapshots of layer stacks: tensor names <-> the masters `models.latent_stack`, `models.hybrid_stack`, `models.hyper_stack` and `models.mixed_stack` pack.  Matrices are [out, in].

Latent-attention stacks (the Bedovik design): layer i's tensors start with `l<i>.`: `norm1` (+ `.b`, `.alpha`), `mix.{q,dkv,dkv.norm,uk,uv,g,o}`, `mlp.router`, `mlp.e<j>.{up,down}`,
`ls1`, `ls2`; the stack has `embed`, `pos`, `loop.in`, `loop.step`, `final.norm` (+ `.b`, `.alpha`) and `head`.

Hybrid recurrent / windowed-attention stacks (the Tudilix design): `l<i>.norm1`, `norm1b` and, with a feed-forward, `norm2`, `norm2b`,
`mlp.{gate,up,down}` (+ `.b`); attention has `mix.{q,k,v,o}`, `mix.{q,k,v}.conv`, `mix.{q,k}.norm` (no `k` and `v` where the layer uses
another layer's); the recurrence has `mix.{y,x}` (+ `.b`), `mix.conv` (+ `.b`), `mix.{ra,ri}` (+ `.b`), `mix.lam`, `mix.o`; the stack has
`embed`, `final.norm` and `head`.

Hyper-connected stacks (the Vozetar design): `l<i>.norm1`, `hc1.{in,out,mix}` and, with a feed-forward, `norm2`, `hc2.*`, `mlp.{gate,up,down}` or
`mlp.router`, `mlp.e<j>.{gate,up,down}`, `mlp.shared.{gate,up,down}`; attention has `{q,k,v,o}` (+ `.b`, `.conv`, `.norm`), `sink` and `g` as its kind
has them, under `mix.` or - beside a linear mixer with `right.{q,k,v,g,o}`, `right.{a1,a2,a2.b,norm}` - under `mix.left.`; normalised mixers have
`mix.{left,right}.out`; the stack has `embed`, `bigram`, `final.norm` and `head`.

Mixed stacks (the Sikazen design): `l<i>.norm1` and, with a feed-forward, `norm2` (a number each), `mlp.{gate,up,down}`, with a side input
`side.{gate,proj,norm}`; under `mix.` attention has `{q,k,v}` (+ `.b`) and `o`, latent attention `dq` (+ `.norm`), `uq`, `dkv` (+ `.norm`), `uk`, `uv`,
`sink`, `o`, HGRN2 `q`, `f` (+ `.b`), `lower`, `v`, `norm`, `o`; the stack has `embed`, `side.embed`, `final.norm` (a number) and `head`.
"""
from __future__ import annotations

from pathlib import Path

import torch

from ..config import ModelSpec
from .safetensors_io import catalog, read_tensor


def _reader(snapshot: str | Path):
    """get(name, *shape): a tensor of the snapshot in its stored dtype, refused when its shape is not the one the configuration implies (0: a size
    that only the tensor tells)."""
    cat = catalog(snapshot)

    def get(name: str, *shape: int) -> torch.Tensor:
        if name not in cat:
            raise KeyError(f"tensor {name} missing from the snapshot")
        t = read_tensor(cat[name])
        if t.dim() == len(shape):
            shape = tuple(n or m for n, m in zip(shape, t.shape))
        if t.numel() != torch.Size(shape).numel() or (t.dim() > 1 and tuple(t.shape) != shape):
            raise ValueError(f"tensor {name}: shape {tuple(t.shape)}, the configuration implies {shape}")
        return t.reshape(shape)
    return get


def read_stack_masters(snapshot: str | Path, spec: ModelSpec) -> dict:
    """Weights of a snapshot in their stored dtype, checked against the shapes the configuration implies."""
    get = _reader(snapshot)
    W = spec.hidden

    def norm(name: str) -> tuple:
        return get(name, W), get(f"{name}.b", W), float(get(f"{name}.alpha"))

    def layer(i: int, b) -> dict:
        a, m, p = b.attn, b.moe, f"l{i}"
        H, d, dv, r = a.n_heads, a.head_dim, a.v_head_dim, a.kv_lora_rank
        lw = {"norm": norm(f"{p}.norm1"), "wq": get(f"{p}.mix.q", H * d, W), "w_dkv": get(f"{p}.mix.dkv", r, W), "kv_norm": get(f"{p}.mix.dkv.norm", r),
              "w_uk": get(f"{p}.mix.uk", H * d, r), "w_uv": get(f"{p}.mix.uv", H * dv, r), "wo": get(f"{p}.mix.o", W, H * dv), "ls1": get(f"{p}.ls1", W)}
        if a.out_gate:
            lw["w_g"] = get(f"{p}.mix.g", H, W)
        if m is not None:
            E, ff = m.n_experts, m.intermediate
            lw["router"], lw["ls2"] = get(f"{p}.mlp.router", E, W), get(f"{p}.ls2", W)
            lw["w_up"] = torch.stack([get(f"{p}.mlp.e{j}.up", ff, W) for j in range(E)])
            lw["w_down"] = torch.stack([get(f"{p}.mlp.e{j}.down", W, ff) for j in range(E)])
        return lw

    w = {"embed": get("embed", spec.vocab, W), "lm_head": get("head", spec.vocab, W), "final_norm": norm("final.norm")}
    if spec.learned_positions:
        w["pos"] = get("pos", spec.learned_positions, W)
    if spec.loop is not None:
        w["loop_in"], w["loop_step"] = get("loop.in", W, 2 * W), get("loop.step", spec.loop.times, W)
    w["layers"] = [layer(i, b) for i, b in enumerate(spec.blocks)]
    return w


def read_hybrid_masters(snapshot: str | Path, spec: ModelSpec) -> dict:
    """Weights of a hybrid stack's snapshot in their stored dtype, checked against the shapes the configuration implies."""
    get, W = _reader(snapshot), spec.hidden

    def layer(i: int, b) -> dict:
        p = f"l{i}"
        lw = {"norm1": get(f"{p}.norm1", W), "norm1b": get(f"{p}.norm1b", W)}
        if b.rec is not None:
            n, nb, sq = b.rec.width, b.rec.blocks, b.rec.width // b.rec.blocks
            for k in ("y", "x"):
                lw[f"w{k}"], lw[f"{k}_b"] = get(f"{p}.mix.{k}", n, W), get(f"{p}.mix.{k}.b", n)
            lw["conv"], lw["conv_b"], lw["lam"] = get(f"{p}.mix.conv", n, b.rec.conv_taps), get(f"{p}.mix.conv.b", n), get(f"{p}.mix.lam", n)
            for k in ("ra", "ri"):
                lw[k], lw[f"{k}_b"] = get(f"{p}.mix.{k}", nb, sq, sq), get(f"{p}.mix.{k}.b", nb, sq)
            lw["wo"] = get(f"{p}.mix.o", W, n)
        else:
            a = b.attn
            sizes = {"q": a.n_heads * a.head_dim, "k": a.n_kv_heads * a.head_dim, "v": a.n_kv_heads * a.v_head_dim}
            for k in ("q", "k", "v") if a.kv_from < 0 else ("q",):
                lw[f"w{k}"], lw[f"{k}_conv"] = get(f"{p}.mix.{k}", sizes[k], W), get(f"{p}.mix.{k}.conv", sizes[k], a.conv_taps)
                if k != "v":
                    lw[f"{k}_norm"] = get(f"{p}.mix.{k}.norm", a.head_dim)
            lw["wo"] = get(f"{p}.mix.o", W, a.n_heads * a.v_head_dim)
        if b.ffn is not None:
            ff = b.ffn.intermediate
            lw["norm2"], lw["norm2b"] = get(f"{p}.norm2", W), get(f"{p}.norm2b", W)
            for k, n, d in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
                lw[f"w_{k}"], lw[f"{k}_b"] = get(f"{p}.mlp.{k}", n, d), get(f"{p}.mlp.{k}.b", n)
        return lw

    return {"embed": get("embed", spec.vocab, W), "lm_head": get("head", spec.vocab, W), "final_norm": get("final.norm", W),
            "layers": [layer(i, b) for i, b in enumerate(spec.blocks)]}


def read_hyper_masters(snapshot: str | Path, spec: ModelSpec) -> dict:
    """Weights of a hyper-connected stack's snapshot in their stored dtype, checked against the shapes the configuration implies."""
    get, W, S = _reader(snapshot), spec.hidden, spec.streams

    def layer(i: int, b) -> dict:
        a, r, m = b.attn, b.rec, b.moe
        p = f"l{i}.mix" + (".left" if r is not None else "")
        hc = lambda q: (get(f"l{i}.hc{q}.in", S), get(f"l{i}.hc{q}.out", S), get(f"l{i}.hc{q}.mix", S, S))
        lw = {"norm1": get(f"l{i}.norm1", W), "hc1": hc(1), "wo": get(f"{p}.o", W, a.n_heads * a.v_head_dim)}
        sizes = {"q": a.n_heads * a.head_dim, "k": a.n_kv_heads * a.head_dim, "v": a.n_kv_heads * a.v_head_dim}
        for k in ("q", "k") if a.values_are_keys else ("q", "k", "v"):
            lw[f"w{k}"] = get(f"{p}.{k}", sizes[k], W)
            if a.qkv_bias:
                lw[f"{k}_b"] = get(f"{p}.{k}.b", sizes[k])
            if a.conv_taps:
                lw[f"{k}_conv"] = get(f"{p}.{k}.conv", sizes[k], a.conv_taps)
            if a.qk_norm_whole and k != "v":
                lw[f"{k}_norm"] = get(f"{p}.{k}.norm", sizes[k])
        if a.out_bias:
            lw["o_b"] = get(f"{p}.o.b", W)
        if a.sink:
            lw["sink"] = get(f"{p}.sink", a.n_heads)
        if a.out_gate:
            lw["wg"] = get(f"{p}.g", a.gate_width, W)
        if r is not None:
            p, hk, hv = f"l{i}.mix.right", r.heads * r.dim, r.heads * r.vdim
            lw.update(rq=get(f"{p}.q", hk, W), rk=get(f"{p}.k", hk, W), rv=get(f"{p}.v", hv, W), rg=get(f"{p}.g", hv, W), r_o=get(f"{p}.o", W, hv))
            if r.kind == "gla":
                lw["a1"] = get(f"{p}.a1", r.rank, W)
                lw["a2"], lw["a2_b"], lw["r_norm"] = get(f"{p}.a2", hk, lw["a1"].shape[0]), get(f"{p}.a2.b", hk), get(f"{p}.norm", r.vdim)
        if b.merge_norm:
            lw["merge_norms"] = (get(f"l{i}.mix.left.out", W), get(f"l{i}.mix.right.out", W))
        if m is None and b.ffn is None:
            return lw
        p, glu = f"l{i}.mlp", lambda p, ff: (get(f"{p}.gate", ff, W), get(f"{p}.up", ff, W), get(f"{p}.down", W, ff))
        lw["norm2"], lw["hc2"] = get(f"l{i}.norm2", W), hc(2)
        if b.ffn is not None:
            lw["ws_gate"], lw["ws_up"], lw["ws_down"] = glu(p, b.ffn.intermediate)
            return lw
        lw["router"] = get(f"{p}.router", m.n_experts, W)
        lw["w_gate"], lw["w_up"], lw["w_down"] = (torch.stack(ts) for ts in zip(*[glu(f"{p}.e{j}", m.intermediate) for j in range(m.n_experts)]))
        if m.n_shared:
            lw["ws_gate"], lw["ws_up"], lw["ws_down"] = glu(f"{p}.shared", m.shared_inter)
        return lw

    w = {"embed": get("embed", spec.vocab, W), "lm_head": get("head", spec.vocab, W), "final_norm": get("final.norm", W)}
    if spec.pair_table is not None:
        w["pairs"] = get("bigram", spec.pair_table.buckets + 1, W)
    w["layers"] = [layer(i, b) for i, b in enumerate(spec.blocks)]
    return w


def read_mixed_masters(snapshot: str | Path, spec: ModelSpec) -> dict:
    """Weights of a mixed stack's snapshot in their stored dtype, checked against the shapes the configuration implies."""
    get, W, sd = _reader(snapshot), spec.hidden, spec.side_dim

    def layer(i: int, b) -> dict:
        a, r, p = b.attn, b.rec, f"l{i}.mix"
        lw = {"norm1": float(get(f"l{i}.norm1"))}
        if r is not None:
            hk, hv = r.heads * r.dim, r.heads * r.vdim
            lw.update(rq=get(f"{p}.q", hk, W), rf=get(f"{p}.f", hk, W), f_b=get(f"{p}.f.b", hk), lower=get(f"{p}.lower", hk), rv=get(f"{p}.v", hv, W), r_norm=get(f"{p}.norm", r.vdim),
                      wo=get(f"{p}.o", W, hv))
        elif a.kind == "latent":
            H, d, dv, rk, dr = a.n_heads, a.head_dim, a.v_head_dim, a.kv_lora_rank, a.rope_dims
            lw.update(dq=get(f"{p}.dq", a.q_lora_rank, W), dq_norm=get(f"{p}.dq.norm", a.q_lora_rank), uq=get(f"{p}.uq", H * (d + dr), a.q_lora_rank), dkv=get(f"{p}.dkv", rk + dr, W),
                      dkv_norm=get(f"{p}.dkv.norm", rk), w_uk=get(f"{p}.uk", H * d, rk), w_uv=get(f"{p}.uv", H * dv, rk), sink=get(f"{p}.sink", H), wo=get(f"{p}.o", W, H * dv))
        else:
            for k, n in (("q", a.n_heads * a.head_dim), ("k", a.n_kv_heads * a.head_dim), ("v", a.n_kv_heads * a.v_head_dim)):
                lw[f"w{k}"], lw[f"{k}_b"] = get(f"{p}.{k}", n, W), get(f"{p}.{k}.b", n)
            lw["wo"] = get(f"{p}.o", W, a.n_heads * a.v_head_dim)
        if b.ffn is not None:
            ff, p = b.ffn.intermediate, f"l{i}.mlp"
            lw.update(norm2=float(get(f"l{i}.norm2")), ws_gate=get(f"{p}.gate", ff, W), ws_up=get(f"{p}.up", ff, W), ws_down=get(f"{p}.down", W, ff))
        if sd:
            p = f"l{i}.side"
            lw.update(side_gate=get(f"{p}.gate", sd, W), side_proj=get(f"{p}.proj", W, sd), side_norm=get(f"{p}.norm", W))
        return lw

    w = {"embed": get("embed", spec.vocab, W), "lm_head": get("head", spec.vocab, W), "final_norm": float(get("final.norm")),
         "layers": [layer(i, b) for i, b in enumerate(spec.blocks)]}
    if sd:
        w["side"] = get("side.embed", spec.vocab, spec.n_layers * sd)
    return w
