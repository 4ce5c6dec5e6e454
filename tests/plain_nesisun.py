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


# ----------------------------------------------------------------------------- random models for the tests
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Name -> shape of every tensor of a model."""
    W = int(cfg["width"])
    out = {"embed": (int(cfg["vocab"]), W), "final.norm": (W,), "head": (int(cfg["vocab"]), W)}
    if cfg["embedding"].get("bigram"):
        out["bigram"] = (int(cfg["embedding"]["bigram"]["buckets"]) + 1, W)
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", L["mixer"]
        H, G, d = m["heads"], m["kv_heads"], m["dim"]
        out.update({p + "norm1": (W,), p + "mix.q": (H * d, W), p + "mix.q.b": (H * d,), p + "mix.k": (G * d, W), p + "mix.k.b": (G * d,),
                    p + "mix.sink": (H,), p + "mix.o": (W, H * d)})
        mlp = L.get("mlp")
        if not mlp:
            continue
        p += "mlp."
        if mlp["kind"] == "dense":
            out.update({p + "gate": (mlp["ff"], W), p + "up": (mlp["ff"], W), p + "down": (W, mlp["ff"])})
            continue
        r, ff = mlp["router"], mlp["expert"]["ff"]
        E = r["experts"] + r.get("identity", 0)
        out.update({p + "router": (E, W), p + "correction": (E,)})
        for x in range(r["experts"]):
            out.update({f"{p}e{x}.gate": (ff, W), f"{p}e{x}.up": (ff, W), f"{p}e{x}.down": (W, ff)})
    return out


def random_weights(cfg: dict, seed: int, dtype=torch.float32) -> Dict[str, torch.Tensor]:
    """Weights drawn so that no mechanism drowns: matrices N(0, 1.5^2 / fan_in), norm weights around one, biases and sinks
    of the size of what they join, corrections that move choices.  In 16 bits queries and keys are smaller: a score s
    carries a rounding error of about |s| * 2^-8."""
    gentle = dtype != torch.float32
    gen = torch.Generator().manual_seed(seed)
    rand = lambda *s: torch.randn(*s, generator=gen, dtype=torch.float32)
    out = {}
    for name, shape in sorted(tensor_shapes(cfg).items()):
        last = name.split(".")[-1]
        if name in ("embed", "bigram"):
            t = rand(*shape) * 0.8
        elif last in ("norm1", "norm"):
            t = 1 + 0.2 * rand(*shape)
        elif last == "sink":
            t = 1.5 * rand(*shape)
        elif last == "correction":
            t = 0.1 * rand(*shape)
        elif last == "b":
            t = (0.4 if gentle else 0.7) * rand(*shape)
        elif last == "router":
            t = rand(*shape) * (3.0 / math.sqrt(shape[-1]))
        elif last in ("q", "k"):
            t = rand(*shape) * ((1.0 if gentle else 2.0) / math.sqrt(shape[-1]))
        else:
            t = rand(*shape) * (1.5 / math.sqrt(shape[-1]))
        out[name] = t.to(dtype)
    return out


def write_model(folder, cfg: dict, seed: int, dtype=torch.float32, weights=None):
    """A model folder (config.json, model.safetensors); returns the weights as stored."""
    import json
    from pathlib import Path
    from pytriton_llama_b200.weights import write_file      # only the file format comes from the package
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    W = weights if weights is not None else random_weights(cfg, seed, dtype)
    (folder / "config.json").write_text(json.dumps(cfg))
    write_file(folder / "model.safetensors", W)
    return W


def attention(heads, kv_heads, dim, scale, size=0, keep=0, dims=0, base=1000.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if size:
        m["mask"] = {"size": size, "keep_first": keep}
    if dims:
        m["rot"] = {"dims": dims, "base": base}
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, identity=0, scale=1.0, limit=1.0):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "identity": identity, "top": top, "scale": scale}}


def layer(mixer, mlp=None, weights_of=None):
    L = {"type": "attention", "mixer": mixer, "mlp": mlp}
    if weights_of is not None:
        L["weights_of"] = weights_of
    return L


def again(layers, j):
    """One more layer that uses the tensors of ``layers[j]``."""
    return dict(layers[j], weights_of=j)


def config(vocab, width, layers, eps=1e-5, scale=0.7, buckets=61, mul_prev=13, mul_cur=5):
    emb = {"scale": scale}
    if buckets:
        emb["bigram"] = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
    return {"architecture": "Nesisun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": emb, "layers": layers}


# Windows and kept positions of different sizes from layer to layer, part of a head or all of it turned, layers with and
# without a feed-forward, experts of both kinds, and layers run again right away and later.
_A = [layer(attention(4, 2, 16, 0.3, size=11, keep=6, dims=8), dense(40)),
      layer(attention(6, 2, 24, 0.2, size=7, keep=3, dims=24, base=50.0), moe(24, 5, 3, identity=2, scale=1.7, limit=0.8)),
      layer(attention(3, 3, 8, 0.4, size=5, keep=9, dims=4, base=10.0))]
TINY_A = config(97, 48, [_A[0], _A[1], again(_A, 1), _A[2], again(_A, 0)], scale=0.6)
# An expert layer first; one query head per key head; a window of one; no kept position; every expert chosen; identity
# experts in the majority; a pair table of one row and one more.
TINY_B = config(70, 64, [
    layer(attention(2, 1, 32, 0.25, size=1, keep=2, dims=32, base=300.0), moe(16, 2, 3, identity=4, scale=2.0, limit=0.5)),
    layer(attention(4, 4, 16, 0.35, size=9, keep=0, dims=2, base=1.0e6), dense(24)),
    layer(attention(8, 2, 8, 0.3, size=20, keep=17, dims=6), moe(8, 4, 4, scale=0.9, limit=2.0)),
], eps=3e-4, scale=1.0, buckets=1)
# Everything seen, nothing turned, widths that are no multiple of eight, one expert and one identity expert, multipliers
# whose products pass 32 bits.
TINY_C = config(50, 36, [
    layer(attention(3, 1, 12, 0.3), dense(19)),
    layer(attention(1, 1, 20, 0.25, size=8, keep=40, dims=10, base=77.0), moe(10, 1, 1, identity=1, limit=0.6)),
    layer(attention(2, 2, 9, 0.5, size=4, keep=1, dims=4, base=5.0), dense(8)),
], scale=1.3, buckets=1009, mul_prev=3_000_000_019, mul_cur=1_000_003)
TINY = {"A": TINY_A, "B": TINY_B, "C": TINY_C}
