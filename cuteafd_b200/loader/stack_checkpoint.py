"""Snapshots of latent-attention layer stacks (the Bedovik design): tensor names <-> the masters `models.latent_stack` packs.

Layer i's tensors start with `l<i>.`: `norm1` (+ `.b`, `.alpha`), `mix.{q,dkv,dkv.norm,uk,uv,g,o}`, `mlp.router`, `mlp.e<j>.{up,down}`,
`ls1`, `ls2`; the stack has `embed`, `pos`, `loop.in`, `loop.step`, `final.norm` (+ `.b`, `.alpha`) and `head`.  Matrices are [out, in].
"""
from __future__ import annotations

from pathlib import Path

import torch

from ..config import ModelSpec
from .safetensors_io import catalog, read_tensor


def read_stack_masters(snapshot: str | Path, spec: ModelSpec) -> dict:
    """Weights of a snapshot in their stored dtype, checked against the shapes the configuration implies."""
    cat = catalog(snapshot)

    def get(name: str, *shape: int) -> torch.Tensor:
        if name not in cat:
            raise KeyError(f"tensor {name} missing from the snapshot")
        t = read_tensor(cat[name])
        if t.numel() != torch.Size(shape).numel() or (t.dim() > 1 and tuple(t.shape) != shape):
            raise ValueError(f"tensor {name}: shape {tuple(t.shape)}, the configuration implies {shape}")
        return t.reshape(shape)

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
