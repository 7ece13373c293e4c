"""Plain oracle of hyper-connected stacks with side-by-side mixers (the Vozetar design): one function per mechanism, whole sequences, no cache.

Works on the raw material of a snapshot - the `config.json` dictionary and a dictionary of tensors by their stored names - so it shares
neither the model description nor the weight preparation of the engine it is compared with.  Everything is evaluated in the dtype of
the tensors it is given (tests pass float32 or float64).  Slow on purpose: loops over heads, streams, experts and tokens where a loop is
clearest.
"""
from __future__ import annotations

import math

import torch

from .hybrid_stack import causal_conv, rms_norm


# ------------------------------------------------------------------ single mechanisms
def bigram_rows(tokens, spec: dict) -> list[int]:
    """Row of the pair table for every token of a sequence; the first one has a row of its own, behind the others."""
    b, mp, mc = int(spec["buckets"]), int(spec["mul_prev"]), int(spec["mul_cur"])
    return [b if i == 0 else (int(tokens[i - 1]) * mp + int(t) * mc) % b for i, t in enumerate(tokens)]


def collapse(streams: list[torch.Tensor], w: torch.Tensor) -> torch.Tensor:
    """The streams' weighted sum: what a sub-layer reads."""
    out = torch.zeros_like(streams[0])
    for s, x in enumerate(streams):
        out = out + w[s] * x
    return out


def spread(streams: list[torch.Tensor], mix: torch.Tensor, out: torch.Tensor, y: torch.Tensor) -> list[torch.Tensor]:
    """Every stream anew from all old ones (mix is indexed [from, to]) and its share of the sub-layer's result."""
    n = len(streams)
    return [sum(mix[s, t] * streams[s] for s in range(n)) + out[t] * y for t in range(n)]


def rotate(x: torch.Tensor, dims: int, base: float, interleaved: bool) -> torch.Tensor:
    """x [T, heads, dim], row t at position t.  Pair i: dimensions 2i and 2i + 1, or i and i + dims / 2; dimensions past `dims` pass."""
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    out = x.clone()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        j, k = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        u, v = x[:, :, j], x[:, :, k]
        out[:, :, j], out[:, :, k] = u * c - v * s, v * c + u * s
    return out


def visible(T: int, size: int | None, keep_first: int) -> torch.Tensor:
    """[query, key]: not later than the query, and fewer than `size` tokens behind it or one of the first `keep_first` tokens."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    return see if size is None else see & ((i - j < size) | (j < keep_first))


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, see: torch.Tensor, sink: torch.Tensor | None) -> torch.Tensor:
    """q [T, heads, dim], k [T, kv heads, dim], v [T, kv heads, vdim] -> [T, heads, vdim]; `sink`: one more logit per head without a value."""
    H = q.shape[1]
    group, out = H // k.shape[1], []
    for h in range(H):
        s = (q[:, h] @ k[:, h // group].T * scale).masked_fill(~see, -math.inf)
        if sink is not None:
            s = torch.cat([s, sink[h].expand(s.shape[0], 1)], 1)
        out.append(torch.softmax(s, -1)[:, :q.shape[0]] @ v[:, h // group])
    return torch.stack(out, 1)


def linear_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor) -> torch.Tensor:
    """q, k [T, heads, dim], v [T, heads, vdim], decay [T, heads, dim]: S_t = diag(decay_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, d = q.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=v.dtype)
        for t in range(T):
            S = decay[t, h][:, None] * S + k[t, h][:, None] * v[t, h][None, :]
            out[t, h] = S.T @ q[t, h]
    return out


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def glu(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def choose_experts(scores: torch.Tensor, top: int, groups: dict | None) -> list[int]:
    """The best experts of one token, out of the best groups of neighbours (a group counts as the sum of its two best scores)."""
    E = scores.numel()
    n, keep = (int(groups["count"]), int(groups["keep"])) if groups else (1, 1)
    per = E // n
    worth = [sum(sorted(scores[g * per:(g + 1) * per].tolist(), reverse=True)[:2]) for g in range(n)]
    best = sorted(range(n), key=lambda g: -worth[g])[:keep]
    allowed = [e for e in range(E) if e // per in best]
    return sorted(allowed, key=lambda e: -float(scores[e]))[:top]


# ------------------------------------------------------------------ sub-layers
def project(h: torch.Tensor, t: dict, name: str) -> torch.Tensor:
    y = h @ t[name].T
    return y + t[f"{name}.b"] if f"{name}.b" in t else y


def attention_mixer(h: torch.Tensor, t: dict, p: str, m: dict, eps: float, *, interleaved: bool, values_are_keys: bool = False) -> torch.Tensor:
    """Which of the optional parts a layer has (biases, convolutions, norms, sink, gate) shows in its tensors."""
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])

    def row(x):
        y = project(h, t, f"{p}.{x}")
        return causal_conv(y, t[f"{p}.{x}.conv"]) if f"{p}.{x}.conv" in t else y

    q, k = row("q"), row("k")
    v = k if values_are_keys else row("v")
    if f"{p}.q.norm" in t:
        q, k = rms_norm(q, t[f"{p}.q.norm"], eps), rms_norm(k, t[f"{p}.k.norm"], eps)
    turn = lambda x: rotate(x, int(m["rot"]["dims"]), float(m["rot"]["base"]), interleaved)
    mask = m.get("mask") or {}
    see = visible(T, int(mask["size"]) if mask.get("size") else None, int(mask.get("keep_first") or 0))
    o = attend(turn(q.reshape(T, H, d)), turn(k.reshape(T, G, d)), v.reshape(T, G, dv), float(m["scale"]), see, t.get(f"{p}.sink"))
    if f"{p}.g" in t:
        g = torch.sigmoid(h @ t[f"{p}.g"].T)
        o = o * g[:, :, None] if g.shape[1] == H and H * dv != H else o * g.reshape(T, H, dv)
    return project(o.reshape(T, -1), t, f"{p}.o")


def retention_mixer(h: torch.Tensor, t: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    turn = lambda x: rotate(x.reshape(T, H, d), int(m["rot"]["dims"]), float(m["rot"]["base"]), False)
    decay = torch.tensor([float(x) for x in m["decay"]], dtype=h.dtype)[None, :, None].expand(T, H, d)
    o = linear_attention(turn(h @ t[f"{p}.q"].T), turn(h @ t[f"{p}.k"].T) * d ** -0.5, (h @ t[f"{p}.v"].T).reshape(T, H, dv), decay)
    o = rms_norm(o, torch.ones(dv, dtype=h.dtype), eps).reshape(T, -1)
    return (o * silu(h @ t[f"{p}.g"].T)) @ t[f"{p}.o"].T


def gla_mixer(h: torch.Tensor, t: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    z = (h @ t[f"{p}.a1"].T) @ t[f"{p}.a2"].T + t[f"{p}.a2.b"]
    decay = torch.exp(-torch.log1p(torch.exp(-z)) / float(m["tau"])).reshape(T, H, d)
    o = linear_attention((h @ t[f"{p}.q"].T).reshape(T, H, d) * d ** -0.5, (h @ t[f"{p}.k"].T).reshape(T, H, d), (h @ t[f"{p}.v"].T).reshape(T, H, dv), decay)
    o = rms_norm(o, t[f"{p}.norm"], eps).reshape(T, -1)
    return (o * silu(h @ t[f"{p}.g"].T)) @ t[f"{p}.o"].T


def mixer(h: torch.Tensor, t: dict, p: str, kind: str, m: dict, eps: float) -> torch.Tensor:
    if kind == "attention":
        return attention_mixer(h, t, p, m, eps, interleaved=False)
    if kind == "parallel":
        left = attention_mixer(h, t, f"{p}.left", m["left"], eps, interleaved=True)
        return float(m["left_scale"]) * left + float(m["right_scale"]) * retention_mixer(h, t, f"{p}.right", m["right"], eps)
    if kind == "parallel_2":
        left = attention_mixer(h, t, f"{p}.left", m["left"], eps, interleaved=True, values_are_keys=True)
        right = gla_mixer(h, t, f"{p}.right", m["right"], eps)
        return 0.5 * (rms_norm(left, t[f"{p}.left.out"], eps) + rms_norm(right, t[f"{p}.right.out"], eps))
    raise ValueError(kind)


def feed_forward(h: torch.Tensor, t: dict, p: str, m: dict) -> torch.Tensor:
    if m["kind"] == "dense":
        return glu(h, t[f"{p}.gate"], t[f"{p}.up"], t[f"{p}.down"])
    r, out = m["router"], []
    for row in h:
        s = torch.sigmoid(row @ t[f"{p}.router"].T)
        out.append(sum(s[e] * glu(row, t[f"{p}.e{e}.gate"], t[f"{p}.e{e}.up"], t[f"{p}.e{e}.down"]) for e in choose_experts(s, int(r["top"]), r.get("groups"))))
    y = torch.stack(out)
    return y + glu(h, t[f"{p}.shared.gate"], t[f"{p}.shared.up"], t[f"{p}.shared.down"]) if m.get("shared") else y


# ------------------------------------------------------------------ stack
def hidden_states(cfg: dict, t: dict, tokens) -> list[torch.Tensor]:
    """The sum of the streams [T, width] after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = t["embed"][torch.as_tensor(tokens)]
    pairs = (cfg.get("embedding") or {}).get("bigram")
    if pairs:
        x = x + t["bigram"][torch.as_tensor(bigram_rows(tokens, pairs))]
    streams, taps = [x] * int(cfg["streams"]), []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        subs = [lambda h: mixer(h, t, f"{p}.mix", layer["type"], layer["mixer"], eps)]
        if layer.get("mlp") is not None:
            subs.append(lambda h: feed_forward(h, t, f"{p}.mlp", layer["mlp"]))
        for q, sub in enumerate(subs, 1):
            hc = f"{p}.hc{q}"
            y = sub(rms_norm(collapse(streams, t[f"{hc}.in"]), t[f"{p}.norm{q}"], eps))
            streams = spread(streams, t[f"{hc}.mix"], t[f"{hc}.out"], y)
        taps.append(sum(streams))
    return taps


def logits(cfg: dict, t: dict, tokens) -> torch.Tensor:
    """[T, vocab] of a whole sequence."""
    return rms_norm(hidden_states(cfg, t, tokens)[-1], t["final.norm"], float(cfg["norm"]["eps"])) @ t["head"].T


def greedy(cfg: dict, t: dict, prompt: list[int], n: int) -> tuple[list[int], list[torch.Tensor]]:
    """Greedy continuation by re-running the whole sequence for every token: (tokens, the logits row each was chosen from)."""
    toks, out, rows = list(prompt), [], []
    for _ in range(n):
        row = logits(cfg, t, toks)[-1]
        rows.append(row)
        out.append(int(row.argmax()))
        toks.append(out[-1])
    return out, rows
