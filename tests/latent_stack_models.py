"""Small Bedovik configurations and random weights for the tests, written out as snapshots."""
import copy
import json

import torch

from cuteafd_b200.config import from_hf_config
from cuteafd_b200.loader.safetensors_io import write_file


def mixer(kind, heads, dim, vdim, rank, scale):
    return {"type": kind, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale}}


def experts(n, top, ff, count, keep, scale):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}


# unequal layers, a loop over the middle, a layer without feed-forward; nothing a multiple of 64
MIXED = {"architecture": "Bedovik", "vocab": 301, "width": 200, "max_positions": 900, "norm": {"eps": 1e-4},
         "loop": {"start": 1, "stop": 3, "times": 3},
         "layers": [{**mixer("latent_attention", 3, 40, 24, 72, 0.3), "mlp": experts(12, 3, 40, 3, 2, 1.7)},
                    {**mixer("latent_attention_2", 5, 72, 136, 136, 0.2), "mlp": None},
                    {**mixer("latent_attention", 2, 100, 56, 40, 0.15), "mlp": experts(10, 2, 56, 5, 3, 0.8)},
                    {**mixer("latent_attention_2", 8, 16, 16, 200, 0.45), "mlp": experts(6, 6, 24, 1, 1, 1.0)}]}
# odd widths everywhere (operand rows that are not multiples of 16 bytes), no loop, one expert per token, ungrouped
ODD = {"architecture": "Bedovik", "vocab": 97, "width": 90, "max_positions": 500, "norm": {"eps": 1e-5},
       "layers": [{**mixer("latent_attention_2", 7, 20, 12, 50, 0.4), "mlp": experts(5, 1, 36, 1, 1, 2.0)},
                  {**mixer("latent_attention", 1, 33, 45, 33, 0.3), "mlp": experts(8, 4, 27, 2, 1, 1.3)}]}
# wide latents: all eight chunk counts of the attention kernel's upper half, and one beyond it; the loop ends the stack
WIDE = {"architecture": "Bedovik", "vocab": 203, "width": 136, "max_positions": 700, "norm": {"eps": 1e-6},
        "loop": {"start": 1, "stop": 4, "times": 2},
        "layers": [{**mixer("latent_attention", 4, 64, 64, 320, 0.2), "mlp": experts(9, 2, 48, 3, 1, 1.1)},
                   {**mixer("latent_attention_2", 6, 128, 96, 448, 0.15), "mlp": None},
                   {**mixer("latent_attention", 16, 192, 128, 512, 0.1), "mlp": experts(8, 3, 64, 4, 3, 2.5)},
                   {**mixer("latent_attention_2", 2, 200, 64, 600, 0.1), "mlp": experts(4, 2, 32, 2, 2, 0.9)}]}
# the whole stack is one pass: a loop of one
ONCE = {"architecture": "Bedovik", "vocab": 130, "width": 72, "max_positions": 300, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 2, "times": 1},
        "layers": [{**mixer("latent_attention", 2, 8, 8, 16, 0.5), "mlp": experts(4, 2, 16, 2, 1, 1.0)},
                   {**mixer("latent_attention", 12, 24, 40, 64, 0.3), "mlp": experts(16, 5, 40, 4, 3, 1.5)}]}
CONFIGS = {"mixed": MIXED, "odd": ODD, "wide": WIDE, "once": ONCE}


def make_tensors(cfg: dict, seed: int = 0) -> dict:
    """Random weights by stored name, rounded to bf16 (fp32 tensors).  Norm gains, offsets, scales and step vectors are all away from 1 and
    0; queries are strong enough that single keys stand out of the softmax."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    r = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean).to(torch.bfloat16).float()
    mat = lambda n, k, gain=1.0: r(n, k, std=gain * k ** -0.5)
    t = {"embed": r(V, W), "pos": r(cfg["max_positions"], W, std=0.5), "head": mat(V, W)}

    def norm(name):
        t[name], t[f"{name}.b"], t[f"{name}.alpha"] = r(W, std=0.2, mean=1.0), r(W, std=0.2), torch.tensor(0.3 + 0.4 * float(torch.rand((), generator=g))).to(torch.bfloat16).float()

    if cfg.get("loop"):
        t["loop.in"], t["loop.step"] = mat(W, 2 * W, 1.2), r(cfg["loop"]["times"], W, std=0.5)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}"
        H, d, dv, rank = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        norm(f"{p}.norm1")
        t.update({f"{p}.mix.q": mat(H * d, W, 4.0), f"{p}.mix.dkv": mat(rank, W), f"{p}.mix.dkv.norm": r(rank, std=0.2, mean=1.0), f"{p}.mix.uk": mat(H * d, rank),
                  f"{p}.mix.uv": mat(H * dv, rank), f"{p}.mix.o": mat(W, H * dv), f"{p}.ls1": r(W, std=0.2, mean=0.8)})
        if layer["type"] == "latent_attention":
            t[f"{p}.mix.g"] = mat(H, W, 2.0)
        if layer.get("mlp") is not None:
            E, ff = layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"]
            t[f"{p}.mlp.router"], t[f"{p}.ls2"] = mat(E, W, 3.0), r(W, std=0.2, mean=0.7)
            for e in range(E):
                t[f"{p}.mlp.e{e}.up"], t[f"{p}.mlp.e{e}.down"] = mat(ff, W), mat(W, ff)
    norm("final.norm")
    return t


def write_snapshot(cfg: dict, tensors: dict, path):
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_file(path / "model.safetensors", {k: v.to(torch.bfloat16) for k, v in tensors.items()})
    return path


def masters_of(cfg: dict, tensors: dict, tmp_path):
    """(spec, masters) through the snapshot reader."""
    from cuteafd_b200.loader.stack_checkpoint import read_stack_masters
    p = write_snapshot(cfg, tensors, tmp_path)
    spec = from_hf_config(p)
    return spec, read_stack_masters(p, spec)


def variant(cfg: dict, **changes) -> dict:
    out = copy.deepcopy(cfg)
    out.update(changes)
    return out
