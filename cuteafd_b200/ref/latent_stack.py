"""Plain fp32 oracle of latent-attention layer stacks (the Bedovik design): one function per mechanism, whole sequences, no cache.

Works on the raw material of a snapshot - the `config.json` dictionary and a dictionary of tensors by their stored names - so it shares
neither the model description nor the weight preparation of the engine it is compared with.  Everything is evaluated in the dtype of
the tensors it is given (tests pass float32 or float64).  Slow on purpose: loops over heads and over tokens where a loop is clearest.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------ single mechanisms
def embed(tokens: torch.Tensor, table: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
    """Token row plus the learned row of its position (`tokens` [T] starts at position 0)."""
    return torch.stack([table[int(t)] + positions[p] for p, t in enumerate(tokens)])


def dyt_norm(x: torch.Tensor, alpha: float, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """Dynamic Tanh: an element-wise squashing in the place of a normalisation."""
    return torch.tanh(x * alpha) * w + b


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def latent_rows(h: torch.Tensor, w_dkv: torch.Tensor, w_norm: torch.Tensor, eps: float) -> torch.Tensor:
    """What a token leaves in the cache."""
    return rms_norm(h @ w_dkv.T, w_norm, eps)


def latent_attention(q: torch.Tensor, c: torch.Tensor, w_uk: torch.Tensor, w_uv: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, heads, dim]; c [T, rank]; w_uk [heads, dim, rank]; w_uv [heads, vdim, rank] -> [T, heads, vdim].  Causal softmax attention
    over keys and values expanded from the latents, without positions."""
    T, H, _ = q.shape
    out = []
    see = torch.ones(T, T, dtype=torch.bool).tril()
    for h in range(H):
        k, v = c @ w_uk[h].T, c @ w_uv[h].T
        s = (q[:, h] @ k.T * scale).masked_fill(~see, -math.inf)
        out.append(torch.softmax(s, -1) @ v)
    return torch.stack(out, 1)


def head_gate(o: torch.Tensor, h: torch.Tensor, w_g: torch.Tensor) -> torch.Tensor:
    """One sigmoid per head, from the mixer's input."""
    return o * torch.sigmoid(h @ w_g.T)[:, :, None]


def route(h: torch.Tensor, w_router: torch.Tensor, r: dict) -> list[list[tuple[int, float]]]:
    """[(expert, weight)] per token: softmax over all experts, groups of neighbours ranked by their best member, the best experts of
    the kept groups, weights renormalised over the chosen ones and scaled."""
    z = h @ w_router.T
    scores = torch.softmax(z, -1)
    n, groups = int(r["experts"]), r.get("groups") or {"count": 1, "keep": 1}
    per = n // int(groups["count"])
    picks = []
    for s in scores.tolist():
        best = sorted(range(int(groups["count"])), key=lambda g: -max(s[g * per:(g + 1) * per]))[:int(groups["keep"])]
        allowed = [e for e in range(n) if e // per in best]
        chosen = sorted(allowed, key=lambda e: -s[e])[:int(r["top"])]
        total = sum(s[e] for e in chosen) + 1e-20
        picks.append([(e, s[e] / total * float(r.get("scale", 1.0))) for e in chosen])
    return picks


def expert(h: torch.Tensor, w_up: torch.Tensor, w_down: torch.Tensor) -> torch.Tensor:
    return torch.relu(h @ w_up.T).square() @ w_down.T


def moe(h: torch.Tensor, tensors: dict, stem: str, cfg: dict) -> torch.Tensor:
    out = torch.zeros_like(h)
    for t, picks in enumerate(route(h, tensors[f"{stem}.router"], cfg["router"])):
        for e, w in picks:
            out[t] += w * expert(h[t], tensors[f"{stem}.e{e}.up"], tensors[f"{stem}.e{e}.down"])
    return out


def enter_pass(x: torch.Tensor, x0: torch.Tensor, w_in: torch.Tensor, step: torch.Tensor) -> torch.Tensor:
    """Start of one pass of the loop: merge with the embedding output, add the pass's vector."""
    return torch.cat([x, x0], -1) @ w_in.T + step


# ------------------------------------------------------------------ stack
def mixer(h: torch.Tensor, tensors: dict, stem: str, layer: dict, eps: float) -> torch.Tensor:
    m = layer["mixer"]
    H, d, dv, rank, T = int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["kv_rank"]), h.shape[0]
    q = (h @ tensors[f"{stem}.q"].T).reshape(T, H, d)
    c = latent_rows(h, tensors[f"{stem}.dkv"], tensors[f"{stem}.dkv.norm"], eps)
    o = latent_attention(q, c, tensors[f"{stem}.uk"].reshape(H, d, rank), tensors[f"{stem}.uv"].reshape(H, dv, rank), float(m["scale"]))
    if layer["type"] == "latent_attention":
        o = head_gate(o, h, tensors[f"{stem}.g"])
    return o.reshape(T, H * dv) @ tensors[f"{stem}.o"].T


def block(x: torch.Tensor, tensors: dict, i: int, layer: dict, eps: float) -> torch.Tensor:
    """Parallel layer: one norm, both sub-layers read it, both results are scaled per channel and added."""
    h = named_norm(x, tensors, f"l{i}.norm1")
    out = x + mixer(h, tensors, f"l{i}.mix", layer, eps) * tensors[f"l{i}.ls1"]
    if layer.get("mlp") is not None:
        out = out + moe(h, tensors, f"l{i}.mlp", layer["mlp"]) * tensors[f"l{i}.ls2"]
    return out


def named_norm(x: torch.Tensor, tensors: dict, name: str) -> torch.Tensor:
    return dyt_norm(x, float(tensors[f"{name}.alpha"]), tensors[name], tensors[f"{name}.b"])


def hidden_states(cfg: dict, tensors: dict, tokens) -> list[torch.Tensor]:
    """Residual rows [T, width] after every layer run, in the order they run."""
    eps = float(cfg["norm"]["eps"])
    x = x0 = embed(torch.as_tensor(tokens), tensors["embed"], tensors["pos"])
    layers, loop = cfg["layers"], cfg.get("loop")
    start, stop, times = (int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else (0, 0, 0)
    taps = []

    def run(i):
        nonlocal x
        x = block(x, tensors, i, layers[i], eps)
        taps.append(x)

    for i in range(start):
        run(i)
    for t in range(times):
        x = enter_pass(x, x0, tensors["loop.in"], tensors["loop.step"][t])
        for i in range(start, stop):
            run(i)
    for i in range(stop, len(layers)):
        run(i)
    return taps


def logits(cfg: dict, tensors: dict, tokens) -> torch.Tensor:
    """[T, vocab] of a whole sequence."""
    return named_norm(hidden_states(cfg, tensors, tokens)[-1], tensors, "final.norm") @ tensors["head"].T


def greedy(cfg: dict, tensors: dict, prompt: list[int], n: int) -> tuple[list[int], list[torch.Tensor]]:
    """Greedy continuation by re-running the whole sequence for every token: (tokens, the logits row each was chosen from)."""
    toks, out, rows = list(prompt), [], []
    for _ in range(n):
        row = logits(cfg, tensors, toks)[-1]
        rows.append(row)
        out.append(int(row.argmax()))
        toks.append(out[-1])
    return out, rows
