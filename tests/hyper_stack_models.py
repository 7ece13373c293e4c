"""Small Vozetar configurations and random weights for the tests, written out as snapshots."""
import copy
import json

import torch

from cuteafd_b200.config import from_hf_config
from cuteafd_b200.loader.safetensors_io import write_file


def attn(heads, kv_heads, dim, vdim, scale, rot=0, base=10000.0, window=None, keep=0, conv=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}}
    if window is not None:
        m["mask"] = {"size": window, "keep_first": keep}
    if conv is not None:
        m["conv"] = conv
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def retention(heads, dim, vdim, rot, base=10000.0, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot}, "decay": decay or [1.0 - 2.0 ** -(3 + 2 * h) for h in range(heads)]}


def gla(heads, dim, vdim, tau):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def plain(m, mlp):
    return {"type": "attention", "mixer": m, "mlp": mlp}


def parallel(left, right, scales, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def parallel2(left, right, mlp):
    return {"type": "parallel_2", "mixer": {"left": left, "right": right}, "mlp": mlp}


# every kind of mixer and of feed-forward, in unequal sizes, two streams
MIXED = {"architecture": "Vozetar", "vocab": 301, "width": 200, "norm": {"eps": 1e-4}, "streams": 2, "embedding": {"bigram": {"buckets": 97, "mul_prev": 13, "mul_cur": 7}},
         "layers": [parallel(attn(6, 2, 40, 24, 0.3, 12, window=70, keep=5), retention(3, 24, 40, 16, decay=[0.5, 0.96875, 0.99951171875]), (0.8, 1.4), dense(72)),
                    plain(attn(4, 2, 40, 56, 0.25, 24, base=500.0, conv=3), moe(12, 3, 40, groups=(4, 2), shared=56)),
                    parallel2(attn(6, 3, 48, 48, 0.2, 32, window=33, keep=70, conv=4), gla(4, 20, 36, 8.0), moe(6, 2, 24)),
                    plain(attn(3, 1, 72, 136, 0.2, 72, conv=2), None)]}
# odd widths everywhere (rows and heads that do not start on 16 bytes), one tap and many, windows of one token and of whole pages, groups of one
# expert, as many experts as are chosen, half rotations that do not fall on whole vectors
ODD = {"architecture": "Vozetar", "vocab": 97, "width": 90, "norm": {"eps": 1e-5}, "streams": 4, "embedding": {"bigram": {"buckets": 61, "mul_prev": 1000003, "mul_cur": 999983}},
       "layers": [plain(attn(7, 7, 33, 45, 0.4, 22, conv=1), moe(5, 2, 27, groups=(5, 3), shared=13)),
                  parallel(attn(5, 1, 20, 13, 0.3, 20, window=1), retention(1, 13, 7, 6, base=100.0), (1.0, 0.5), dense(35)),
                  parallel2(attn(5, 5, 27, 27, 0.3, 2, window=64, keep=1, conv=6), gla(3, 9, 17, 1.0), dense(27)),
                  parallel(attn(14, 7, 33, 45, 0.3, 10, window=65, keep=64), retention(2, 5, 66, 0), (0.3, 2.0), moe(4, 4, 19))]}
# every width class of the attention kernels, groups that do not divide a tile of rows, recurrent heads of unequal sides; one stream
WIDE = {"architecture": "Vozetar", "vocab": 203, "width": 136, "norm": {"eps": 1e-6}, "streams": 1, "embedding": {"bigram": {"buckets": 40, "mul_prev": 3, "mul_cur": 1}},
        "layers": [parallel(attn(9, 1, 256, 256, 0.06, 64, window=100, keep=130), retention(2, 128, 256, 128, decay=[0.875, 0.998046875]), (1.0, 1.0), dense(264)),
                   plain(attn(12, 4, 192, 64, 0.08, 32, conv=3), dense(64)),
                   parallel2(attn(8, 4, 128, 128, 0.12, 128, window=129, keep=3, conv=2), gla(2, 256, 64, 16.0), moe(16, 4, 64, groups=(2, 1), shared=128)),
                   plain(attn(40, 1, 64, 192, 0.09, 64, base=1e6, conv=4), dense(32))]}
# no pair table, windows longer than any text, five streams
PLAIN = {"architecture": "Vozetar", "vocab": 130, "width": 72, "norm": {"eps": 1e-6}, "streams": 5,
         "layers": [parallel2(attn(4, 4, 16, 16, 0.5, 16, window=4096, keep=2, conv=2), gla(4, 16, 16, 16.0), dense(48)), plain(attn(2, 2, 24, 24, 0.4, 24, conv=4), dense(40)),
                    parallel(attn(4, 2, 16, 24, 0.5, 8, window=4096, keep=4), retention(4, 16, 32, 8), (0.9, 1.1), dense(40))]}
CONFIGS = {"mixed": MIXED, "odd": ODD, "wide": WIDE, "plain": PLAIN}
RANK = {"mixed": 6, "odd": 5, "wide": 16, "plain": 8}


def make_tensors(cfg: dict, seed: int = 0, rank: int = 6) -> dict:
    """Random weights by stored name, rounded to bf16 (fp32 tensors).  Gains, biases and stream constants are away from 0 and 1, sinks take a share,
    part of the decays remember for hundreds of tokens, and queries are strong enough that single keys stand out of the softmax."""
    g = torch.Generator().manual_seed(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    r = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean).to(torch.bfloat16).float()
    mat = lambda n, k, gain=1.0: r(n, k, std=gain * k ** -0.5)
    norm = lambda n: r(n, std=0.25, mean=1.1)
    t = {"embed": r(V, W), "head": mat(V, W, 3.0), "final.norm": norm(W)}
    pairs = (cfg.get("embedding") or {}).get("bigram")
    if pairs:
        t["bigram"] = r(pairs["buckets"] + 1, W, std=0.7)

    def conv(n, taps):
        w = r(n, taps, std=0.5)
        w[:, -1] += 0.7
        return w.to(torch.bfloat16).float()

    def attention(p, m, *, bias, out_bias=False, sink=False, gate="", whole=False, values=True):
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for k, n in (("q", H * d), ("k", G * d), ("v", G * dv)):
            if k == "v" and not values:
                continue
            t[f"{p}.{k}"] = mat(n, W, 1.5 if k != "v" else 1.0)
            if bias:
                t[f"{p}.{k}.b"] = r(n, std=0.4)
            if m.get("conv"):
                t[f"{p}.{k}.conv"] = conv(n, m["conv"])
            if whole and k != "v":
                t[f"{p}.{k}.norm"] = r(n, std=0.3, mean=1.3)
        if sink:
            t[f"{p}.sink"] = r(H, std=1.0, mean=1.0)
        if gate:
            t[f"{p}.g"] = mat(H if gate == "head" else H * dv, W, 1.5)
        t[f"{p}.o"] = mat(W, H * dv, 1.5)
        if out_bias:
            t[f"{p}.o.b"] = r(W, std=0.3)

    def linear(p, m, kind):
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        for k, n in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
            t[f"{p}.{k}"] = mat(n, W)
        t[f"{p}.o"] = mat(W, H * dv, 1.5)
        if kind == "gla":
            t[f"{p}.a1"], t[f"{p}.a2"], t[f"{p}.a2.b"], t[f"{p}.norm"] = mat(rank, W), mat(H * d, rank, 2.0), r(H * d, std=2.0, mean=2.0), norm(dv)

    def glu(p, ff):
        t[f"{p}.gate"], t[f"{p}.up"], t[f"{p}.down"] = mat(ff, W, 1.3), mat(ff, W, 1.3), mat(W, ff, 1.5)

    for i, layer in enumerate(cfg["layers"]):
        m, p, mlp = layer["mixer"], f"l{i}", layer.get("mlp")
        for q in (1, 2) if mlp is not None else (1,):
            t[f"{p}.norm{q}"] = norm(W)
            t[f"{p}.hc{q}.in"], t[f"{p}.hc{q}.out"] = r(S, std=0.3, mean=1.0 / S), r(S, std=0.3, mean=0.8)
            t[f"{p}.hc{q}.mix"] = (0.8 * torch.eye(S) + r(S, S, std=0.3) / S).to(torch.bfloat16).float()
        if layer["type"] == "attention":
            attention(f"{p}.mix", m, bias=True, out_bias=True, sink=True, gate="value")
        elif layer["type"] == "parallel":
            attention(f"{p}.mix.left", m["left"], bias=True, sink=True)
            linear(f"{p}.mix.right", m["right"], "retention")
        else:
            attention(f"{p}.mix.left", m["left"], bias=False, gate="head", whole=True, values=False)
            linear(f"{p}.mix.right", m["right"], "gla")
            t[f"{p}.mix.left.out"], t[f"{p}.mix.right.out"] = norm(W), norm(W)
        if mlp is not None and mlp["kind"] == "dense":
            glu(f"{p}.mlp", mlp["ff"])
        elif mlp is not None:
            t[f"{p}.mlp.router"] = mat(mlp["router"]["experts"], W, 2.0)
            for j in range(mlp["router"]["experts"]):
                glu(f"{p}.mlp.e{j}", mlp["expert"]["ff"])
            if mlp.get("shared"):
                glu(f"{p}.mlp.shared", mlp["shared"]["ff"])
    return t


def write_snapshot(cfg: dict, tensors: dict, path):
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_file(path / "model.safetensors", {k: v.to(torch.bfloat16) for k, v in tensors.items()})
    return path


def masters_of(cfg: dict, tensors: dict, tmp_path):
    """(spec, masters) through the snapshot reader."""
    from cuteafd_b200.loader.stack_checkpoint import read_hyper_masters
    p = write_snapshot(cfg, tensors, tmp_path)
    spec = from_hf_config(p)
    return spec, read_hyper_masters(p, spec)


def variant(cfg: dict, **changes) -> dict:
    out = copy.deepcopy(cfg)
    out.update(changes)
    return out
