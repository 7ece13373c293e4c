"""Small Sikazen configurations and random weights for the tests, written out as snapshots."""
import copy
import json

import torch

from cuteafd_b200.config import from_hf_config
from cuteafd_b200.loader.safetensors_io import write_file


def attention(heads, kv_heads, dim, vdim, scale, rot, window, pool, mlp=None, base=10000.0, factor=2.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}, "mask": {"size": window, "pool": pool}}
    if factor is not None:
        m["rot"]["scaling"] = {"factor": factor}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot, vdim, rank, q_rank, scale, mlp=None, base=10000.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale, "rot": {"base": base, "dims": rot}}}


def hgrn2(heads, dim, vdim, mlp=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def model(vocab, width, layers, *, eps=1e-5, scale=1.5, side=20, loop=None):
    cfg = {"architecture": "Sikazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if side:
        cfg["token_side"] = {"dim": side}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


# every kind of layer, unequal sizes, two of three layers twice
BLEND = model(301, 200, [hgrn2(3, 24, 40, dense(72)), attention(6, 2, 40, 24, 0.6, 12, 70, 6, dense(56)), latent(5, 40, 16, 24, 72, 88, 0.25, dense(80)),
                         attention(4, 4, 72, 136, 0.3, 72, 33, 20, None, factor=1.0), hgrn2(2, 64, 72, None)], eps=1e-4, side=28, loop=(1, 3, 2))
# odd widths everywhere (rows and heads that do not start on 16 bytes), blocks of one token and longer than a page, a window of one token, a loop
# over the whole stack, no feed-forward or no other part
ODD = model(97, 90, [attention(7, 7, 33, 45, 0.4, 22, 1, 1, dense(35)), latent(3, 13, 6, 7, 21, 19, 0.4), hgrn2(1, 13, 7, dense(27)), attention(5, 1, 20, 13, 0.9, 20, 64, 70, None, factor=8.0),
                     latent(1, 33, 2, 45, 65, 9, 0.2, dense(13)), hgrn2(3, 9, 17, None)], scale=0.25, side=7, loop=(0, 6, 2))
# every width class of the attention kernels, latents beyond the tensor-core form's, rotated parts of a chunk and more, groups that do not divide a
# tile of rows, recurrent heads of unequal sides
WIDE = model(203, 136, [attention(9, 1, 256, 256, 0.08, 64, 100, 8, dense(264)), latent(12, 128, 64, 128, 512, 200, 0.08), hgrn2(2, 128, 256, dense(64)), attention(12, 4, 192, 64, 0.1, 32, 129, 4),
                        latent(3, 192, 32, 64, 320, 72, 0.1, dense(40)), attention(40, 1, 64, 192, 0.2, 64, 64, 16, dense(32)), hgrn2(2, 256, 64)], eps=1e-6, side=64, loop=(5, 6, 3))
# no loop, no side table, windows longer than any text or none, many heads, a latent wider than the tensor-core form takes
PLAIN = model(130, 72, [latent(2, 24, 72, 24, 600, 33, 0.2, dense(48)), attention(4, 2, 16, 24, 0.9, 8, 4096, 4, dense(40), factor=None), hgrn2(4, 16, 16, dense(40)), latent(130, 8, 8, 8, 16, 24, 0.4)],
              scale=1.0, side=0)
PLAIN["layers"].append({**copy.deepcopy(PLAIN["layers"][1]), "mlp": None})
del PLAIN["layers"][-1]["mixer"]["mask"]
CONFIGS = {"blend": BLEND, "odd": ODD, "wide": WIDE, "plain": PLAIN}


def make_tensors(cfg: dict, seed: int = 0) -> dict:
    """Random weights by stored name, rounded to bf16 (fp32 tensors).  Numbers, gains and biases are away from 0 and 1, sinks take a share, part of the
    forget gates remember for hundreds of tokens, and queries are strong enough that single keys stand out of the softmax."""
    g = torch.Generator().manual_seed(seed)
    W, V, n = cfg["width"], cfg["vocab"], len(cfg["layers"])
    r = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean).to(torch.bfloat16).float()
    mat = lambda n, k, gain=1.0: r(n, k, std=gain * k ** -0.5)
    gain = lambda n: r(n, std=0.25, mean=1.1)
    number = lambda: r(1, std=0.2, mean=1.2).reshape(())
    t = {"embed": r(V, W), "head": mat(V, W, 3.0), "final.norm": number()}
    sd = (cfg.get("token_side") or {}).get("dim", 0)
    if sd:
        t["side.embed"] = r(V, n * sd)
    for i, layer in enumerate(cfg["layers"]):
        m, p, mlp = layer["mixer"], f"l{i}", layer.get("mlp")
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        t[f"{p}.norm1"] = number()
        if layer["type"] == "attention":
            G = m["kv_heads"]
            for k, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                t[f"{p}.mix.{k}"], t[f"{p}.mix.{k}.b"] = mat(rows, W), r(rows, std=0.4)
        elif layer["type"] == "latent_attention":
            rk, qk, dr = m["kv_rank"], m["q_rank"], m["rot_dim"]
            t.update({f"{p}.mix.dq": mat(qk, W), f"{p}.mix.dq.norm": gain(qk), f"{p}.mix.uq": mat(H * (d + dr), qk, 1.7), f"{p}.mix.dkv": mat(rk + dr, W, 1.5), f"{p}.mix.dkv.norm": gain(rk),
                      f"{p}.mix.uk": mat(H * d, rk, 1.5), f"{p}.mix.uv": mat(H * dv, rk), f"{p}.mix.sink": r(H, std=1.0, mean=1.0)})
        else:
            t.update({f"{p}.mix.q": mat(H * d, W), f"{p}.mix.f": mat(H * d, W), f"{p}.mix.f.b": r(H * d, std=2.5, mean=2.0),
                      f"{p}.mix.lower": torch.rand(H * d, generator=g).mul(0.9 if i else 0.0).to(torch.bfloat16).float(), f"{p}.mix.v": mat(H * dv, W), f"{p}.mix.norm": gain(dv)})
        t[f"{p}.mix.o"] = mat(W, H * dv, 1.5)
        if mlp is not None:
            ff = mlp["ff"]
            t[f"{p}.norm2"] = number()
            t[f"{p}.mlp.gate"], t[f"{p}.mlp.up"], t[f"{p}.mlp.down"] = mat(ff, W, 1.3), mat(ff, W, 1.3), mat(W, ff, 1.5)
        if sd:
            t[f"{p}.side.gate"], t[f"{p}.side.proj"], t[f"{p}.side.norm"] = mat(sd, W, 0.6), mat(W, sd), r(W, std=0.3, mean=0.5)
    return t


def write_snapshot(cfg: dict, tensors: dict, path):
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_file(path / "model.safetensors", {k: v.to(torch.bfloat16) for k, v in tensors.items()})
    return path


def masters_of(cfg: dict, tensors: dict, tmp_path):
    """(spec, masters) through the snapshot reader."""
    from cuteafd_b200.loader.stack_checkpoint import read_mixed_masters
    p = write_snapshot(cfg, tensors, tmp_path)
    spec = from_hf_config(p)
    return spec, read_mixed_masters(p, spec)
