"""Plain oracle of mixed stacks (the Sikazen design): one function per mechanism, whole sequences, no cache.

Works on the raw material of a snapshot - the `config.json` dictionary and a dictionary of tensors by their stored names - so it shares
neither the model description nor the weight preparation of the engine it is compared with.  Everything is evaluated in the dtype of
the tensors it is given (tests pass float32 or float64).  Slow on purpose: loops over heads, blocks and tokens where a loop is clearest.
"""
from __future__ import annotations

import math

import torch

from .hybrid_stack import rms_norm
from .hyper_stack import glu, linear_attention, rotate, silu


# ------------------------------------------------------------------ single mechanisms
def unit_norm(x: torch.Tensor, eps: float) -> torch.Tensor:
    """Rows over their root mean square."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def turn(x: torch.Tensor, rot: dict | None, interleaved: bool) -> torch.Tensor:
    """x [T, heads, dim], row t at position t; linear scaling divides every angle by the factor."""
    if not rot or not int(rot["dims"]):
        return x
    f = float((rot.get("scaling") or {}).get("factor", 1.0))
    if f == 1.0:
        return rotate(x, int(rot["dims"]), float(rot["base"]), interleaved)
    T, dims, out = x.shape[0], int(rot["dims"]), x.clone()
    for i in range(dims // 2):
        a = torch.arange(T, dtype=torch.float64) * (float(rot["base"]) ** (-2.0 * i / dims) / f)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        j, k = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        u, v = x[:, :, j], x[:, :, k]
        out[:, :, j], out[:, :, k] = u * c - v * s, v * c + u * s
    return out


def window_tokens(i: int, size: int | None) -> list[int]:
    """Tokens that position i sees one by one."""
    return [j for j in range(i + 1) if size is None or i - j < size]


def pooled_blocks(i: int, size: int | None, pool: int) -> list[int]:
    """Blocks of `pool` tokens that position i sees as one key each: those that lie wholly in front of its window."""
    out, b = [], 0
    while size is not None and pool and b * pool + pool - 1 <= i - size:
        out.append(b)
        b += 1
    return out


def pooled_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, size: int | None, pool: int) -> torch.Tensor:
    """q [T, heads, dim], k [T, kv heads, dim], v [T, kv heads, vdim] -> [T, heads, vdim]: tokens of the window and means of the blocks in front
    of it under one softmax."""
    T, H = q.shape[:2]
    group, n = H // k.shape[1], T // pool if pool else 0
    kb = torch.stack([k[b * pool:(b + 1) * pool].mean(0) for b in range(n)]) if n else None
    vb = torch.stack([v[b * pool:(b + 1) * pool].mean(0) for b in range(n)]) if n else None
    out = torch.zeros(T, H, v.shape[2], dtype=v.dtype)
    for i in range(T):
        toks, blocks = window_tokens(i, size), pooled_blocks(i, size, pool)
        keys, vals = k[toks], v[toks]
        if blocks:
            keys, vals = torch.cat([kb[blocks], keys]), torch.cat([vb[blocks], vals])
        for h in range(H):
            p = torch.softmax(keys[:, h // group] @ q[i, h] * scale, 0)
            out[i, h] = p @ vals[:, h // group]
    return out


def sink_softmax(s: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """Weights of the scores s [., keys] with one more logit in the denominator."""
    return torch.softmax(torch.cat([s, sink.expand(s.shape[0], 1)], 1), -1)[:, :-1]


def forget_gate(z: torch.Tensor, lower: torch.Tensor) -> torch.Tensor:
    return lower + (1.0 - lower) * torch.sigmoid(z)


# ------------------------------------------------------------------ sub-layers
def attention_mixer(h: torch.Tensor, t: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    row = lambda x, n, w: (h @ t[f"{p}.{x}"].T + t[f"{p}.{x}.b"]).reshape(T, n, w)
    q, k, v = row("q", H, d), row("k", G, d), row("v", G, dv)
    q, k = unit_norm(turn(q, m.get("rot"), False), eps), unit_norm(turn(k, m.get("rot"), False), eps)
    mask = m.get("mask") or {}
    o = pooled_attention(q, k, v, float(m["scale"]), int(mask["size"]) if mask.get("size") else None, int(mask.get("pool") or 0))
    return o.reshape(T, -1) @ t[f"{p}.o"].T


def latent_mixer(h: torch.Tensor, t: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, d, dr, dv, r = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    q = (rms_norm(h @ t[f"{p}.dq"].T, t[f"{p}.dq.norm"], eps) @ t[f"{p}.uq"].T).reshape(T, H, d + dr)
    down = h @ t[f"{p}.dkv"].T
    c, kr = rms_norm(down[:, :r], t[f"{p}.dkv.norm"], eps), turn(down[:, r:].reshape(T, 1, dr), m.get("rot"), True)[:, 0]
    qr, k, v = turn(q[:, :, d:], m.get("rot"), True), (c @ t[f"{p}.uk"].T).reshape(T, H, d), (c @ t[f"{p}.uv"].T).reshape(T, H, dv)
    see, out = torch.ones(T, T, dtype=torch.bool).tril(), []
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + qr[:, i] @ kr.T) * float(m["scale"])
        out.append(sink_softmax(s.masked_fill(~see, -math.inf), t[f"{p}.sink"][i]) @ v[:, i])
    return torch.stack(out, 1).reshape(T, -1) @ t[f"{p}.o"].T


def hgrn2_mixer(h: torch.Tensor, t: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    f = forget_gate(h @ t[f"{p}.f"].T + t[f"{p}.f.b"], t[f"{p}.lower"]).reshape(T, H, d)
    o = linear_attention(silu(h @ t[f"{p}.q"].T).reshape(T, H, d), 1.0 - f, (h @ t[f"{p}.v"].T).reshape(T, H, dv), f)
    return rms_norm(o, t[f"{p}.norm"], eps).reshape(T, -1) @ t[f"{p}.o"].T


MIXERS = {"attention": attention_mixer, "latent_attention": latent_mixer, "hgrn2": hgrn2_mixer}


def side_input(x: torch.Tensor, tokens: torch.Tensor, layer: int, t: dict, dim: int, eps: float) -> torch.Tensor:
    """What the token adds to the residual rows behind a layer: its part of the table, gated by the rows."""
    p, e = f"l{layer}.side", t["side.embed"][tokens][:, layer * dim:(layer + 1) * dim]
    return rms_norm((gelu_tanh(x @ t[f"{p}.gate"].T) * e) @ t[f"{p}.proj"].T, t[f"{p}.norm"], eps)


# ------------------------------------------------------------------ stack
def layer_order(n: int, loop: dict | None) -> list[tuple[int, bool]]:
    """(layer, whether the embedding output is added in front of it), in the order the layers run."""
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    body = [(i, i == a and k > 0) for k in range(times) for i in range(a, b)]
    return [(i, False) for i in range(a)] + body + [(i, False) for i in range(b, n)]


def hidden_states(cfg: dict, t: dict, tokens) -> list[torch.Tensor]:
    """The residual rows [T, width] after every layer run."""
    eps, tokens, taps = float(cfg["norm"]["eps"]), torch.as_tensor(tokens), []
    x0 = t["embed"][tokens] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    x, side = x0, cfg.get("token_side")
    for i, again in layer_order(len(cfg["layers"]), cfg.get("loop")):
        p, layer = f"l{i}", cfg["layers"][i]
        if again:
            x = x + x0
        n = unit_norm(x, eps)
        y = MIXERS[layer["type"]](n * t[f"{p}.norm1"], t, f"{p}.mix", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + glu(n * t[f"{p}.norm2"], t[f"{p}.mlp.gate"], t[f"{p}.mlp.up"], t[f"{p}.mlp.down"])
        x = x + y
        if side:
            x = x + side_input(x, tokens, i, t, int(side["dim"]), eps)
        taps.append(x)
    return taps


def logits(cfg: dict, t: dict, tokens) -> torch.Tensor:
    """[T, vocab] of a whole sequence."""
    return (unit_norm(hidden_states(cfg, t, tokens)[-1], float(cfg["norm"]["eps"])) * t["final.norm"]) @ t["head"].T


def greedy(cfg: dict, t: dict, prompt: list[int], n: int) -> tuple[list[int], list[torch.Tensor]]:
    """Greedy continuation by re-running the whole sequence for every token: (tokens, the logits row each was chosen from)."""
    toks, out, rows = list(prompt), [], []
    for _ in range(n):
        row = logits(cfg, t, toks)[-1]
        rows.append(row)
        out.append(int(row.argmax()))
        toks.append(out[-1])
    return out, rows
