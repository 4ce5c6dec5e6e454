"""The Nesisun decoder written out plainly: float64, whole sequences, one function per mechanism.

Shares no code with the package; the package is tested against this.  ``cfg`` is the nested
dictionary of a config.json, ``W`` a dictionary name -> tensor (any element type; promoted here).

Notation: h input of both sub-layers [T, width]; positions 0..T-1; H query heads, G key/value heads, d head
size, n window size, c kept first positions.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w.to(F)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def lin(h, W, name):
    y = h @ W[name].to(F).T
    return y + W[name + ".b"].to(F) if name + ".b" in W else y


# ----------------------------------------------------------------------------- the stream's start
def bigram_rows(tokens: List[int], buckets: int, mul_prev: int, mul_cur: int) -> List[int]:
    """Row of the pair table for every token: a hash of the token before and the token; ``buckets`` for the first."""
    rows = [buckets]
    for before, now in zip(tokens, tokens[1:]):
        rows.append((before * mul_prev + now * mul_cur) % buckets)
    return rows[:len(tokens)]


def embed(cfg: dict, W, tokens: List[int]) -> torch.Tensor:
    e = cfg["embedding"]
    x = W["embed"].to(F)[torch.tensor(tokens, dtype=torch.long)] * float(e["scale"])
    b = e.get("bigram")
    if b:
        x = x + W["bigram"].to(F)[torch.tensor(bigram_rows(tokens, int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])))]
    return x


# ----------------------------------------------------------------------------- attention
def rotate_neighbours(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, d]: entries 2i and 2i + 1 of the first ``dims`` of a head turned by position * base^(-2i/dims)."""
    if not rot:
        return x
    n, base = int(rot["dims"]), float(rot["base"])
    out = x.clone()
    for i in range(n // 2):
        a = torch.arange(x.shape[0], dtype=F) * base ** (-2.0 * i / n)
        c, s = a.cos()[:, None], a.sin()[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def visible(i: int, size: int, keep: int) -> List[int]:
    """Keys that query i sees: the window's and the first ``keep`` (size 0: every earlier one)."""
    return [j for j in range(i + 1) if not size or i - j < size or j < keep]


def softmax_with_sink(s: torch.Tensor, sink: Optional[float]) -> torch.Tensor:
    """Weights of the scores s; the denominator holds exp(sink) besides."""
    m = float(s.max()) if sink is None else max(float(s.max()), sink)
    e = torch.exp(s - m)
    return e / (e.sum() + (0.0 if sink is None else math.exp(sink - m)))


def sink_attention(q, k, v, scale: float, size: int, keep: int, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for i in range(T):
        keys = torch.tensor(visible(i, size, keep))
        for a in range(H):
            g = a // (H // G)
            w = softmax_with_sink((k[keys, g] @ q[i, a]) * scale, None if sink is None else float(sink[a]))
            out[i, a] = w @ v[keys, g]
    return out


def attention_mixer(h, m: dict, W, p: str) -> torch.Tensor:
    """The values are the keys as projected (bias included), before they are turned."""
    T = h.shape[0]
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = lin(h, W, p + "q").view(T, H, d)
    k = lin(h, W, p + "k").view(T, G, d)
    mask = m.get("mask") or {}
    o = sink_attention(rotate_neighbours(q, m.get("rot")), rotate_neighbours(k, m.get("rot")), k, float(m["scale"]),
                       int(mask.get("size") or 0), int(mask.get("keep_first") or 0), W[p + "sink"].to(F))
    return o.reshape(T, H * d) @ W[p + "o"].to(F).T


# ----------------------------------------------------------------------------- feed-forward
def dense_feed_forward(h, W, p: str) -> torch.Tensor:
    return lin(gelu_tanh(lin(h, W, p + "gate")) * lin(h, W, p + "up"), W, p + "down")


def clamped_expert(h, W, p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(lin(h, W, p + "gate"), max=limit)
    u = torch.clamp(lin(h, W, p + "up"), -limit, limit)
    return lin(g * torch.sigmoid(1.702 * g) * (u + 1.0), W, p + "down")


def route(scores: torch.Tensor, correction: torch.Tensor, top: int, scale: float):
    """scores [E] -> (chosen experts, their weights): chosen by score + correction, weighted by the scores over their sum."""
    chosen = torch.topk(scores + correction, top).indices
    w = scores[chosen]
    return chosen, w / (w.sum() + 1e-20) * scale


def moe_feed_forward(h, mlp: dict, W, p: str) -> torch.Tensor:
    r = mlp["router"]
    real = int(r["experts"])
    scores = torch.softmax(lin(h, W, p + "router"), dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, w = route(scores[t], W[p + "correction"].to(F), int(r["top"]), float(r.get("scale", 1.0)))
        for e, w_e in zip(chosen.tolist(), w):
            out[t] += w_e * (h[t] if e >= real else clamped_expert(h[t:t + 1], W, f"{p}e{e}.", float(mlp["expert"]["limit"]))[0])
    return out


def feed_forward(h, mlp: dict, W, p: str) -> torch.Tensor:
    return dense_feed_forward(h, W, p) if mlp["kind"] == "dense" else moe_feed_forward(h, mlp, W, p)


# ----------------------------------------------------------------------------- the model
def run_layer(x, L: dict, W, p: str, eps: float) -> torch.Tensor:
    """One norm, both sub-layers on its output."""
    h = rms_norm(x, W[p + "norm1"], eps)
    y = attention_mixer(h, L["mixer"], W, p + "mix.")
    if L.get("mlp"):
        y = y + feed_forward(h, L["mlp"], W, p + "mlp.")
    return x + y


def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int], return_layers: bool = False):
    """Logits [T, vocab] (float64) of one sequence.  ``return_layers``: also the stream after every layer, [layers, T, width]."""
    eps = float(cfg["norm"]["eps"])
    x = embed(cfg, W, tokens)
    after = []
    for i, L in enumerate(cfg["layers"]):
        x = run_layer(x, L, W, f"l{L.get('weights_of', i)}.", eps)
        after.append(x)
    logits = lin(rms_norm(x, W["final.norm"], eps), W, "head")
    return (logits, torch.stack(after)) if return_layers else logits


def load_model_folder(folder, dtype=F):
    """(config dictionary, name -> tensor) of a folder with config.json and model.safetensors, read with nothing but
    the standard library and torch."""
    import json
    import struct
    from pathlib import Path
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    header = json.loads(raw[8:8 + n])
    types = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "F64": torch.float64, "I32": torch.int32}
    W = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        t = torch.frombuffer(bytearray(raw[8 + n + lo:8 + n + hi]), dtype=types[info["dtype"]]).reshape(info["shape"])
        W[name] = t.to(dtype) if t.dtype.is_floating_point else t
    return cfg, W
