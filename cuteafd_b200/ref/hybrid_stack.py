"""Plain oracle of hybrid recurrent / windowed-attention stacks (the Tudilix design): one function per mechanism, whole sequences, no cache.

Works on the raw material of a snapshot - the `config.json` dictionary and a dictionary of tensors by their stored names - so it shares
neither the model description nor the weight preparation of the engine it is compared with.  Everything is evaluated in the dtype of
the tensors it is given (tests pass float32 or float64).  Slow on purpose: loops over heads, channels' blocks and tokens where a loop is
clearest.
"""
from __future__ import annotations

import math

import torch

GLU_SLOPE = 1.702           # steepness of the sigmoid in the feed-forward's gate
DECAY_SHARPNESS = 8.0       # the recurrence's log decay is -8 * gate * softplus(lambda)


# ------------------------------------------------------------------ single mechanisms
def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose stored weight is the gain's distance from one."""
    return rms_norm(x, 1.0 + w, eps)


def causal_conv(u: torch.Tensor, w: torch.Tensor, bias: torch.Tensor | None = None) -> torch.Tensor:
    """u [T, channels], w [channels, taps]: each channel's last `taps` inputs, the last column weighing the current one; zeros in front."""
    T, taps = u.shape[0], w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                out[t] += w[:, j] * u[src]
    return out if bias is None else out + bias


def rope_frequencies(rot: dict) -> tuple[list[float], float]:
    """(angle per position of every rotated pair, factor on cosine and sine) with YaRN scaling where the configuration has it."""
    n, base = int(rot["dims"]), float(rot["base"])
    freq = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return freq, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_of(turns: float) -> float:
        return n * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(pair_of(float(sc["fast"]))), 0), min(math.ceil(pair_of(float(sc["slow"]))), n - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, dim], row t at position t: neighbouring dimensions (2i, 2i + 1) turn together, dimensions past rot.dims pass."""
    freq, amp = rope_frequencies(rot)
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    out = x.clone()
    for i, f in enumerate(freq):
        a = pos * f
        c, s = (torch.cos(a) * amp).to(x.dtype)[:, None], (torch.sin(a) * amp).to(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def visible(T: int, window: int | None) -> torch.Tensor:
    """[query, key]: the key is not later than the query and fewer than `window` tokens behind it."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < (window or T))


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int | None) -> torch.Tensor:
    """q [T, heads, dim], k [T, kv heads, dim], v [T, kv heads, vdim] -> [T, heads, vdim]."""
    T, H, _ = q.shape
    group, see = H // k.shape[1], visible(T, window)
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // group].T * scale).masked_fill(~see, -math.inf)
        out.append(torch.softmax(s, -1) @ v[:, h // group])
    return torch.stack(out, 1)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def block_gate(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, width]; w [blocks, n, n] and b [blocks, n]: every block of channels has its own sigmoid gate."""
    n = w.shape[1]
    return torch.cat([torch.sigmoid(u[:, i * n:(i + 1) * n] @ w[i].T + b[i]) for i in range(w.shape[0])], -1)


def lru(u: torch.Tensor, r: torch.Tensor, i: torch.Tensor, lam: torch.Tensor) -> torch.Tensor:
    """Real-gated linear recurrence over the rows, from a zero state; every row's state is returned."""
    decay = -DECAY_SHARPNESS * r * torch.log1p(torch.exp(lam))
    state, out = torch.zeros_like(u[0]), []
    for t in range(u.shape[0]):
        a = torch.exp(decay[t])
        state = a * state + torch.sqrt(1.0 - a * a) * i[t] * u[t]
        out.append(state)
    return torch.stack(out)


def clamped_glu(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    """Gate bounded from above, linear half bounded on both sides and shifted by one."""
    g, u = gate.clamp(max=limit), up.clamp(-limit, limit)
    return g * torch.sigmoid(GLU_SLOPE * g) * (u + 1.0)


def softcap(z: torch.Tensor, cap: float | None) -> torch.Tensor:
    return cap * torch.tanh(z / cap) if cap else z


# ------------------------------------------------------------------ sub-layers
def keys_values(h: torch.Tensor, t: dict, p: str, m: dict, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    T, G = h.shape[0], int(m["kv_heads"])
    k = causal_conv(h @ t[f"{p}.k"].T, t[f"{p}.k.conv"]).reshape(T, G, int(m["dim"]))
    v = causal_conv(h @ t[f"{p}.v"].T, t[f"{p}.v.conv"]).reshape(T, G, int(m["vdim"]))
    return rotate(rms_norm(k, t[f"{p}.k.norm"], eps), m["rot"]), v


def attention_mixer(h: torch.Tensor, t: dict, p: str, m: dict, eps: float, shared: tuple | None) -> tuple[torch.Tensor, tuple]:
    """(output, (keys, values) of this layer); `shared`: another layer's keys and values, used instead of own ones."""
    T, H = h.shape[0], int(m["heads"])
    q = causal_conv(h @ t[f"{p}.q"].T, t[f"{p}.q.conv"]).reshape(T, H, int(m["dim"]))
    q = rotate(rms_norm(q, t[f"{p}.q.norm"], eps), m["rot"])
    kv = shared if shared is not None else keys_values(h, t, p, m, eps)
    o = attend(q, *kv, float(m["scale"]), (m.get("mask") or {}).get("size"))
    return o.reshape(T, -1) @ t[f"{p}.o"].T, kv


def recurrent_mixer(h: torch.Tensor, t: dict, p: str) -> torch.Tensor:
    y = gelu_tanh(h @ t[f"{p}.y"].T + t[f"{p}.y.b"])
    u = causal_conv(h @ t[f"{p}.x"].T + t[f"{p}.x.b"], t[f"{p}.conv"], t[f"{p}.conv.b"])
    s = lru(u, block_gate(u, t[f"{p}.ra"], t[f"{p}.ra.b"]), block_gate(u, t[f"{p}.ri"], t[f"{p}.ri.b"]), t[f"{p}.lam"])
    return (s * y) @ t[f"{p}.o"].T


def feed_forward(h: torch.Tensor, t: dict, p: str, m: dict) -> torch.Tensor:
    g, u = h @ t[f"{p}.gate"].T + t[f"{p}.gate.b"], h @ t[f"{p}.up"].T + t[f"{p}.up.b"]
    return clamped_glu(g, u, float(m["limit"])) @ t[f"{p}.down"].T + t[f"{p}.down.b"]


# ------------------------------------------------------------------ stack
def hidden_states(cfg: dict, t: dict, tokens) -> list[torch.Tensor]:
    """Residual rows [T, width] after every layer."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = t["embed"][torch.as_tensor(tokens)]
    taps, cache = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        h = centred_norm(x, t[f"{p}.norm1"], eps)
        if layer["type"] == "attention":
            out, cache[i] = attention_mixer(h, t, f"{p}.mix", m, eps, cache[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            out = recurrent_mixer(h, t, f"{p}.mix")
        x = x + mult * centred_norm(out, t[f"{p}.norm1b"], eps)
        if layer.get("mlp") is not None:
            out = feed_forward(centred_norm(x, t[f"{p}.norm2"], eps), t, f"{p}.mlp", layer["mlp"])
            x = x + mult * centred_norm(out, t[f"{p}.norm2b"], eps)
        taps.append(x)
    return taps


def logits(cfg: dict, t: dict, tokens) -> torch.Tensor:
    """[T, vocab] of a whole sequence."""
    z = centred_norm(hidden_states(cfg, t, tokens)[-1], t["final.norm"], float(cfg["norm"]["eps"])) @ t["head"].T
    return softcap(z, cfg.get("logit_softcap"))


def greedy(cfg: dict, t: dict, prompt: list[int], n: int) -> tuple[list[int], list[torch.Tensor]]:
    """Greedy continuation by re-running the whole sequence for every token: (tokens, the logits row each was chosen from)."""
    toks, out, rows = list(prompt), [], []
    for _ in range(n):
        row = logits(cfg, t, toks)[-1]
        rows.append(row)
        out.append(int(row.argmax()))
        toks.append(out[-1])
    return out, rows
