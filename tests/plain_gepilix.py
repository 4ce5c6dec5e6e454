"""The Gepilix decoder written out plainly: float64, whole sequences, one function per mechanism.

Shares no code with the package; the package is tested against this.  ``cfg`` is the nested
dictionary of a config.json, ``W`` a dictionary name -> tensor (any element type; promoted here).

Notation: h input of a sub-layer [T, width]; positions 0..T-1; H query heads, G key/value heads,
d query/key head size, e value head size.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def lin(h, W, name, bias=False):
    y = h @ W[name].to(F).T
    return y + W[name + ".b"].to(F) if bias else y


def tanh_norm(x, W, name):
    """tanh(alpha x) w + b, entry by entry: no statistic of the row."""
    return torch.tanh(W[name + ".alpha"].to(F) * x) * W[name].to(F) + W[name + ".b"].to(F)


# ----------------------------------------------------------------------------- softmax attention
def pair_frequencies(rot: dict) -> torch.Tensor:
    """Frequency of pair i: base^(-2i/dims), slowed by ``factor`` where the wavelength exceeds original/low, kept where
    it is below original/high, and mixed linearly in original/wavelength between the two."""
    n, base = int(rot["dims"]), float(rot["base"])
    out = []
    s = rot.get("scaling")
    for i in range(n // 2):
        f = base ** (-2.0 * i / n)
        if s:
            turns = float(s["original"]) * f / (2 * math.pi)
            if turns < float(s["low"]):
                f = f / float(s["factor"])
            elif turns <= float(s["high"]):
                m = (turns - float(s["low"])) / (float(s["high"]) - float(s["low"]))
                f = (1 - m) * f / float(s["factor"]) + m * f
        out.append(f)
    return torch.tensor(out, dtype=F)


def rotate_halves(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, d]: entry i of the first ``dims`` of a head is paired with entry i + dims/2."""
    if not rot:
        return x
    n = int(rot["dims"])
    half = n // 2
    a = torch.arange(x.shape[0], dtype=F)[:, None] * pair_frequencies(rot)[None, :]
    c, s = a.cos()[:, None, :], a.sin()[:, None, :]
    out = x.clone()
    u, v = x[..., :half], x[..., half:n]
    out[..., :half] = u * c - v * s
    out[..., half:n] = v * c + u * s
    return out


def capped_attention(q, k, v, scale: float, cap: float, first_key) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; query i sees keys first_key(i) .. i; a score s becomes
    cap tanh(s / cap)."""
    T, H, _ = q.shape
    G, e = k.shape[1], v.shape[2]
    out = torch.zeros(T, H, e, dtype=F)
    for i in range(T):
        lo = first_key(i)
        for a in range(H):
            g = a // (H // G)
            s = (k[lo:i + 1, g] @ q[i, a]) * scale
            out[i, a] = torch.softmax(cap * torch.tanh(s / cap), dim=0) @ v[lo:i + 1, g]
    return out


def _heads(h, m, W, p, bias):
    T = h.shape[0]
    H, G, d, e = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    return (lin(h, W, p + "q", bias).view(T, H, d), lin(h, W, p + "k", bias).view(T, G, d), lin(h, W, p + "v", bias).view(T, G, e))


def chunk_attention_mixer(h, m: dict, W, p: str) -> torch.Tensor:
    """Biases, no rotation, keys of the query's own chunk only, one gate per head."""
    q, k, v = _heads(h, m, W, p, True)
    n = int(m["mask"]["size"])
    o = capped_attention(q, k, v, float(m["scale"]), float(m["softcap"]), lambda i: i // n * n)
    o = o * torch.sigmoid(lin(h, W, p + "g"))[:, :, None]
    return lin(o.reshape(h.shape[0], -1), W, p + "o")


def window_attention_mixer(h, m: dict, W, p: str) -> torch.Tensor:
    """No biases, rotated halves, a sliding window."""
    q, k, v = _heads(h, m, W, p, False)
    q, k = rotate_halves(q, m.get("rot")), rotate_halves(k, m.get("rot"))
    n = int(m["mask"]["size"])
    o = capped_attention(q, k, v, float(m["scale"]), float(m["softcap"]), lambda i: max(0, i - n + 1))
    return lin(o.reshape(h.shape[0], -1), W, p + "o")


# ----------------------------------------------------------------------------- recurrences
def causal_conv(x, w, b) -> torch.Tensor:
    """x [T, C], w [C, taps]: y_t = b + sum_j w[:, j] x_(t - taps + 1 + j), with x_s = 0 for s < 0."""
    T, C = x.shape
    n = w.shape[1]
    padded = torch.cat([torch.zeros(n - 1, C, dtype=F), x])
    y = b.to(F).expand(T, C).clone()
    for j in range(n):
        y += padded[j:j + T] * w[:, j].to(F)
    return y


def linear_unit_mixer(h, m: dict, W, p: str) -> torch.Tensor:
    """Two branches; the second passes a short convolution and a gated linear recurrence per channel."""
    T, n, B = h.shape[0], int(m["width"]), int(m["blocks"])
    y = gelu_tanh(lin(h, W, p + "y", True))
    u = causal_conv(lin(h, W, p + "x", True), W[p + "conv"], W[p + "conv.b"])
    parts = u.view(T, B, n // B)
    gate = lambda a: torch.sigmoid(torch.einsum("tbi,boi->tbo", parts, W[p + a].to(F)) + W[p + a + ".b"].to(F)).reshape(T, n)
    r, i = gate("ra"), gate("ri")
    log_a = -8.0 * r * softplus(W[p + "lam"].to(F))
    a = torch.exp(log_a)
    S = torch.zeros(n, dtype=F)
    out = torch.zeros(T, n, dtype=F)
    for t in range(T):
        S = a[t] * S + torch.sqrt(-torch.expm1(2 * log_a[t])) * i[t] * u[t]
        out[t] = S
    return lin(out * y, W, p + "o")


def state_space_mixer(h, m: dict, W, p: str, eps: float) -> torch.Tensor:
    """A matrix state per head with one decay per head and token; keys and queries shared by groups of heads."""
    T = h.shape[0]
    H, e, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * e
    proj = lin(h, W, p + "in")
    z, conv_in, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(conv_in, W[p + "conv"], W[p + "conv.b"]))
    x = xbc[:, :inner].view(T, H, e)
    Bm, Cm = xbc[:, inner:inner + G * N].view(T, G, N), xbc[:, inner + G * N:].view(T, G, N)
    dt = softplus(dt + W[p + "dt_bias"].to(F))
    decay = torch.exp(-torch.exp(W[p + "A_log"].to(F)) * dt)
    y = torch.zeros(T, H, e, dtype=F)
    for a in range(H):
        g = a // (H // G)
        S = torch.zeros(N, e, dtype=F)
        for t in range(T):
            S = decay[t, a] * S + dt[t, a] * torch.outer(Bm[t, g], x[t, a])
            y[t, a] = S.T @ Cm[t, g] + W[p + "D"].to(F)[a] * x[t, a]
    y = y.reshape(T, inner) * silu(z)
    y = rms_unit(y.view(T, int(m["norm_groups"]), -1), eps).reshape(T, inner) * W[p + "norm"].to(F)
    return lin(y, W, p + "o")


def wkv_mixer(h, m: dict, W, p: str, eps: float) -> torch.Tensor:
    """Token shift, a matrix state per head with a decay per key channel and token, a bonus for the current token."""
    T, H, d = h.shape[0], int(m["heads"]), int(m["dim"])
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    mix = lambda a: h + (before - h) * W[p + "mu." + a].to(F)
    r, k, v = (lin(mix(a), W, p + a).view(T, H, d) for a in "rkv")
    gate = silu(lin(mix("g"), W, p + "g"))
    w = torch.exp(-torch.exp(lin(torch.tanh(lin(mix("w"), W, p + "w1")), W, p + "w2") + W[p + "w0"].to(F))).view(T, H, d)
    u = W[p + "u"].to(F).view(H, d)
    S = torch.zeros(H, d, d, dtype=F)
    o = torch.zeros(T, H, d, dtype=F)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return lin(rms_unit(o, eps).reshape(T, H * d) * W[p + "norm"].to(F) * gate, W, p + "o")


# ----------------------------------------------------------------------------- mixers side by side
def normed_mean_mixer(h, m: dict, W, p: str, eps: float) -> torch.Tensor:
    left = chunk_attention_mixer(h, m["left"], W, p + "left.")
    right = linear_unit_mixer(h, m["right"], W, p + "right.")
    return 0.5 * (rms_unit(left, eps) * W[p + "left.out"].to(F) + rms_unit(right, eps) * W[p + "right.out"].to(F))


def scaled_sum_mixer(h, m: dict, W, p: str, eps: float) -> torch.Tensor:
    left = window_attention_mixer(h, m["left"], W, p + "left.")
    right = state_space_mixer(h, m["right"], W, p + "right.", eps)
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


# ----------------------------------------------------------------------------- feed-forward
def squared_relu_mlp(h, W, p: str) -> torch.Tensor:
    return lin(torch.relu(lin(h, W, p + "up")) ** 2, W, p + "down")


def gated_expert(h, W, p: str) -> torch.Tensor:
    return lin(silu(lin(h, W, p + "gate")) * lin(h, W, p + "up"), W, p + "down")


def route(logits: torch.Tensor, top: int):
    """The ``top`` largest logits and the softmax over them alone."""
    chosen = torch.topk(logits, top).indices
    return chosen, torch.softmax(logits[chosen], dim=0)


def moe_feed_forward(h, mlp: dict, W, p: str) -> torch.Tensor:
    z = lin(h, W, p + "router", True)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, w = route(z[t], int(mlp["router"]["top"]))
        for e_, w_ in zip(chosen.tolist(), w):
            out[t] += w_ * gated_expert(h[t:t + 1], W, f"{p}e{e_}.")[0]
    if mlp.get("shared"):
        out = out + gated_expert(h, W, p + "shared.")
    return out


def feed_forward(h, mlp: dict, W, p: str) -> torch.Tensor:
    return squared_relu_mlp(h, W, p) if mlp["kind"] == "dense" else moe_feed_forward(h, mlp, W, p)


# ----------------------------------------------------------------------------- the model
def run_layer(x, L: dict, W, p: str, eps: float) -> torch.Tensor:
    h = tanh_norm(x, W, p + "norm1")
    mixer = {"parallel": normed_mean_mixer, "parallel_2": scaled_sum_mixer, "wkv": wkv_mixer}[L["type"]]
    x = x + W[p + "ls1"].to(F) * mixer(h, L["mixer"], W, p + "mix.", eps)
    if L.get("mlp") is not None:
        x = x + W[p + "ls2"].to(F) * feed_forward(tanh_norm(x, W, p + "norm2"), L["mlp"], W, p + "mlp.")
    return x


def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int], return_layers: bool = False):
    """Logits [T, vocab] (float64) of one sequence.  ``return_layers``: also the stream after every layer, [layers, T, width]."""
    eps = float(cfg["norm"]["eps"])
    x = W["embed"].to(F)[torch.tensor(tokens, dtype=torch.long)]
    handed = []
    for i, L in enumerate(cfg["layers"]):
        x = run_layer(x, L, W, f"l{i}.", eps)
        handed.append(x)
    logits = lin(tanh_norm(x, W, "final.norm"), W, "head")
    return (logits, torch.stack(handed)) if return_layers else logits


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
def tensor_shapes(cfg: dict, rank: int = 16) -> Dict[str, tuple]:
    """Name -> shape of every tensor of a model (``rank``: inner size of the decay projections)."""
    W = int(cfg["width"])
    out = {"embed": (int(cfg["vocab"]), W), "head": (int(cfg["vocab"]), W)}

    def norm(name):
        out.update({name: (W,), name + ".b": (W,), name + ".alpha": ()})

    def attention(p, m, bias):
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({p + "q": (H * d, W), p + "k": (G * d, W), p + "v": (G * e, W), p + "o": (W, H * e)})
        if bias:
            out.update({p + "q.b": (H * d,), p + "k.b": (G * d,), p + "v.b": (G * e,), p + "g": (H, W)})

    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", L["mixer"], f"l{i}.mix."
        norm(p + "norm1")
        out[p + "ls1"] = (W,)
        if L["type"] == "wkv":
            n = m["heads"] * m["dim"]
            out.update({q + "mu." + a: (W,) for a in "rkvgw"})
            out.update({q + a: (n, W) for a in "rkvg"})
            out.update({q + "w1": (rank, W), q + "w2": (n, rank), q + "w0": (n,), q + "u": (m["heads"], m["dim"]), q + "norm": (n,), q + "o": (W, n)})
        else:
            attention(q + "left.", m["left"], L["type"] == "parallel")
            r, q = m["right"], q + "right."
            if L["type"] == "parallel":
                n, B = r["width"], r["blocks"]
                s = n // B
                out.update({q + "y": (n, W), q + "y.b": (n,), q + "x": (n, W), q + "x.b": (n,), q + "conv": (n, r["conv"]), q + "conv.b": (n,),
                            q + "ra": (B, s, s), q + "ra.b": (B, s), q + "ri": (B, s, s), q + "ri.b": (B, s), q + "lam": (n,), q + "o": (W, n),
                            p + "mix.left.out": (W,), p + "mix.right.out": (W,)})
            else:
                n, c = r["heads"] * r["vdim"], r["heads"] * r["vdim"] + 2 * r["groups"] * r["state"]
                out.update({q + "in": (n + c + r["heads"], W), q + "conv": (c, r["conv"]), q + "conv.b": (c,), q + "dt_bias": (r["heads"],),
                            q + "A_log": (r["heads"],), q + "D": (r["heads"],), q + "norm": (n,), q + "o": (W, n)})
        mlp = L.get("mlp")
        if mlp:
            norm(p + "norm2")
            out[p + "ls2"] = (W,)
            q = p + "mlp."
            if mlp["kind"] == "dense":
                out.update({q + "up": (mlp["ff"], W), q + "down": (W, mlp["ff"])})
                continue
            ff, E = mlp["expert"]["ff"], mlp["router"]["experts"]
            out.update({q + "router": (E, W), q + "router.b": (E,)})
            for x in range(E):
                out.update({f"{q}e{x}.gate": (ff, W), f"{q}e{x}.up": (ff, W), f"{q}e{x}.down": (W, ff)})
            if mlp.get("shared"):
                sf = mlp["shared"]["ff"]
                out.update({q + "shared.gate": (sf, W), q + "shared.up": (sf, W), q + "shared.down": (W, sf)})
    return out


def random_weights(cfg: dict, seed: int, dtype=torch.float32, rank: int = 16) -> Dict[str, torch.Tensor]:
    """Weights drawn so that no mechanism drowns: matrices N(0, 1.5^2 / fan_in), scores of a few units, decays from
    near one to near zero, router logits that spread.  In 16 bits scores are smaller (a score s carries a rounding error
    of about |s| * 2^-8), and so are the routed experts' outputs (a router's close call that falls the other way swaps them)."""
    gentle = dtype != torch.float32
    gen = torch.Generator().manual_seed(seed)
    rand = lambda *s: torch.randn(*s, generator=gen, dtype=torch.float32)
    uni = lambda lo, hi, *s: lo + (hi - lo) * torch.rand(s, generator=gen, dtype=torch.float32)
    out = {}
    for name, shape in sorted(tensor_shapes(cfg, rank).items()):
        parts = name.split(".")
        last = parts[-1]
        if name == "embed":
            t = rand(*shape)
        elif last == "alpha":
            t = uni(0.4, 0.8)
        elif last in ("norm1", "norm2", "norm", "out"):
            t = 1 + 0.2 * rand(*shape)
        elif last in ("ls1", "ls2"):
            t = uni(0.4, 1.2, *shape) * torch.where(torch.arange(shape[0]) % 5 == 2, -1.0, 1.0)
        elif "mu" in parts:
            t = uni(0.0, 1.0, *shape)
        elif last == "conv":
            t = rand(*shape) * (1.2 / math.sqrt(shape[1]))
        elif last == "lam":
            t = uni(-5.0, 1.0, *shape)
        elif last == "w0":
            t = uni(-4.0, 0.5, *shape)
        elif last == "dt_bias":
            t = uni(-3.0, 0.5, *shape)
        elif last == "A_log":
            t = uni(-2.0, 1.5, *shape)
        elif last in ("u", "D"):
            t = uni(-1.5, 1.5, *shape)
        elif last == "b":
            t = 0.3 * rand(*shape)
        elif last == "router":
            t = rand(*shape) * (3.0 / math.sqrt(shape[-1]))
        elif last in ("q", "k") and "left" in parts:
            t = rand(*shape) * ((1.5 if gentle else 3.0) / math.sqrt(shape[-1]))
        else:
            t = rand(*shape) * (1.5 / math.sqrt(shape[-1]))
            if gentle and last == "down" and parts[-2].startswith("e"):
                t *= 0.25
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


def rotation(dims, base, scaling=None):
    """``scaling``: None or (factor, low, high, original)."""
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def attention(heads, kv_heads, dim, vdim, scale, softcap, size, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap, "mask": {"size": size}}
    if rot:
        m["rot"] = rot
    return m


def linear_unit(width, blocks, conv):
    return {"width": width, "blocks": blocks, "conv": conv}


def state_space(heads, vdim, state, groups, norm_groups, conv):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def parallel(left, right):
    return {"left": left, "right": right}


def parallel_2(left, right, left_scale, right_scale):
    return {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Gepilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# Chunks and windows that straddle pages of 4, 8 and 16; value heads larger and smaller than key heads; part of a head
# rotated, with frequencies below, between and above the two bounds; a layer without a feed-forward; three taps and five.
TINY_A = config(97, 48, [
    layer("parallel", parallel(attention(4, 2, 16, 24, 0.3, 12.0, 11), linear_unit(36, 3, 3)), moe(24, 6, 2, shared=16)),
    layer("wkv", {"heads": 3, "dim": 12}, dense(40)),
    layer("parallel_2", parallel_2(attention(6, 3, 16, 8, 0.25, 9.0, 9, rot=rotation(12, 100.0, (3.0, 0.5, 2.0, 40.0))),
                                   state_space(6, 8, 12, 3, 2, 5), 0.8, 1.3), moe(16, 4, 3)),
    layer("parallel", parallel(attention(2, 1, 8, 16, 0.4, 20.0, 6), linear_unit(20, 1, 2)), None),
])
# A scaled-sum layer first; as many kv heads as heads; one group of everything; every expert chosen; one tap.
TINY_B = config(70, 64, [
    layer("parallel_2", parallel_2(attention(3, 3, 16, 16, 0.35, 15.0, 7, rot=rotation(16, 50.0)), state_space(2, 20, 8, 1, 1, 2), -0.6, 1.0),
          dense(48)),
    layer("wkv", {"heads": 2, "dim": 20}, moe(24, 3, 3, shared=24)),
    layer("parallel", parallel(attention(4, 1, 24, 16, 0.3, 6.0, 5), linear_unit(24, 4, 4)), dense(24)),
    layer("parallel_2", parallel_2(attention(2, 2, 8, 8, 0.5, 30.0, 1, rot=rotation(2, 10.0)), state_space(4, 8, 16, 4, 4, 1), 1.0, 0.4), None),
], eps=3e-4)
# Only recurrences and one chunk of one; one expert of one; a width that is no multiple of eight.
TINY_C = config(50, 36, [
    layer("wkv", {"heads": 1, "dim": 8}, None),
    layer("parallel", parallel(attention(3, 1, 16, 32, 0.3, 8.0, 1), linear_unit(15, 5, 1)), moe(16, 1, 1)),
    layer("wkv", {"heads": 5, "dim": 8}, dense(12)),
])
TINY = {"A": TINY_A, "B": TINY_B, "C": TINY_C}
