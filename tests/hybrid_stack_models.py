"""Small Tudilix configurations and random weights for the tests, written out as snapshots."""
import copy
import json

import torch

from cuteafd_b200.config import from_hf_config
from cuteafd_b200.loader.safetensors_io import write_file


def yarn(factor, original, fast=16.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attention(heads, kv_heads, dim, vdim, window, conv, rot_dims, scale, base=10000.0, scaling=None, ff=0, limit=1.0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": window}, "scale": scale,
         "rot": {"base": base, "dims": rot_dims, "scaling": scaling}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def rglru(width, blocks, conv, ff=0, limit=1.0):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


# unequal layers of both kinds, feed-forwards on some of either, shared keys across a recurrent layer, two rotations
MIXED = {"architecture": "Tudilix", "vocab": 301, "width": 200, "norm": {"eps": 1e-4}, "residual_mult": 0.7, "logit_softcap": 12.0,
         "layers": [rglru(120, 3, 3, ff=72, limit=0.8), attention(6, 2, 40, 24, 70, 4, 12, 0.3, scaling=yarn(4.0, 64)), rglru(96, 2, 4),
                    attention(4, 2, 40, 24, 33, 2, 12, 0.25, scaling=yarn(4.0, 64), ff=100, limit=1.3, kv_from=1), attention(3, 1, 72, 136, 128, 3, 72, 0.2, base=500.0)]}
# odd widths everywhere (rows and heads that do not start on 16 bytes), one tap and many, windows of one token and of whole pages
ODD = {"architecture": "Tudilix", "vocab": 97, "width": 90, "norm": {"eps": 1e-5}, "residual_mult": 1.0, "logit_softcap": 26.0,
       "layers": [attention(7, 7, 33, 45, 64, 5, 10, 0.4, scaling=yarn(2.0, 32, fast=4.0), ff=27, limit=2.0), rglru(45, 3, 1), attention(5, 1, 20, 13, 1, 1, 20, 0.3),
                  rglru(35, 1, 6, ff=36), attention(14, 7, 33, 45, 65, 2, 10, 0.3, scaling=yarn(2.0, 32, fast=4.0), kv_from=0)]}
# every width class of the attention kernels, groups that do not divide a tile of rows
WIDE = {"architecture": "Tudilix", "vocab": 203, "width": 136, "norm": {"eps": 1e-6}, "residual_mult": 0.4, "logit_softcap": 50.0,
        "layers": [attention(9, 1, 256, 256, 100, 4, 64, 0.06), rglru(256, 1, 4), attention(12, 4, 192, 64, 200, 3, 32, 0.08, scaling=yarn(16.0, 48), ff=264, limit=7.0),
                   attention(8, 4, 64, 192, 129, 2, 64, 0.12), attention(40, 1, 128, 128, 77, 4, 128, 0.09, base=1e6, ff=64)]}
# one layer of each kind in their simplest shape; the window is longer than any text
PLAIN = {"architecture": "Tudilix", "vocab": 130, "width": 72, "norm": {"eps": 1e-6}, "residual_mult": 0.5, "logit_softcap": 5.0,
         "layers": [attention(4, 4, 16, 16, 4096, 2, 16, 0.5, ff=48, limit=0.5), rglru(64, 8, 2, ff=40, limit=3.0)]}
# no attention at all
RECURRENT = {"architecture": "Tudilix", "vocab": 110, "width": 64, "norm": {"eps": 1e-5}, "residual_mult": 0.6, "logit_softcap": 20.0,
             "layers": [rglru(64, 2, 4), rglru(160, 5, 2, ff=56, limit=1.0)]}
CONFIGS = {"mixed": MIXED, "odd": ODD, "wide": WIDE, "plain": PLAIN, "recurrent": RECURRENT}


def make_tensors(cfg: dict, seed: int = 0) -> dict:
    """Random weights by stored name, rounded to bf16 (fp32 tensors).  Gains and biases are away from 1 and 0, a part of the recurrent channels
    remembers for hundreds of tokens, and queries are strong enough that single keys stand out of the softmax."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    r = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean).to(torch.bfloat16).float()
    mat = lambda n, k, gain=1.0: r(n, k, std=gain * k ** -0.5)
    norm = lambda n: r(n, std=0.25)
    t = {"embed": r(V, W), "head": mat(V, W, 3.0), "final.norm": norm(W)}

    def conv(n, taps):
        w = r(n, taps, std=0.5)
        w[:, -1] += 0.7
        return w.to(torch.bfloat16).float()

    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}"
        t[f"{p}.norm1"], t[f"{p}.norm1b"] = norm(W), norm(W)
        if layer["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for k, n in (("q", H * d), ("k", G * d), ("v", G * dv)):
                if k != "q" and m.get("kv_from") is not None:
                    continue
                t[f"{p}.mix.{k}"], t[f"{p}.mix.{k}.conv"] = mat(n, W), conv(n, m["conv"])
                if k != "v":
                    t[f"{p}.mix.{k}.norm"] = r(d, std=0.3, mean=1.2)
            t[f"{p}.mix.o"] = mat(W, H * dv)
        else:
            n, nb = m["width"], m["blocks"]
            sq = n // nb
            for k in ("y", "x"):
                t[f"{p}.mix.{k}"], t[f"{p}.mix.{k}.b"] = mat(n, W), r(n, std=0.2)
            t[f"{p}.mix.conv"], t[f"{p}.mix.conv.b"] = conv(n, m["conv"]), r(n, std=0.2)
            t[f"{p}.mix.ra"], t[f"{p}.mix.ra.b"] = r(nb, sq, sq, std=2.0 * sq ** -0.5), r(nb, sq, std=2.0, mean=-2.0)
            t[f"{p}.mix.ri"], t[f"{p}.mix.ri.b"] = r(nb, sq, sq, std=2.0 * sq ** -0.5), r(nb, sq)
            t[f"{p}.mix.lam"], t[f"{p}.mix.o"] = r(n, std=1.5, mean=-3.0), mat(W, n)
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            t[f"{p}.norm2"], t[f"{p}.norm2b"] = norm(W), norm(W)
            for k, n, d in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
                t[f"{p}.mlp.{k}"], t[f"{p}.mlp.{k}.b"] = mat(n, d, 1.3), r(n, std=0.3)
    return t


def write_snapshot(cfg: dict, tensors: dict, path):
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_file(path / "model.safetensors", {k: v.to(torch.bfloat16) for k, v in tensors.items()})
    return path


def masters_of(cfg: dict, tensors: dict, tmp_path):
    """(spec, masters) through the snapshot reader."""
    from cuteafd_b200.loader.stack_checkpoint import read_hybrid_masters
    p = write_snapshot(cfg, tensors, tmp_path)
    spec = from_hf_config(p)
    return spec, read_hybrid_masters(p, spec)


def variant(cfg: dict, **changes) -> dict:
    out = copy.deepcopy(cfg)
    out.update(changes)
    return out
