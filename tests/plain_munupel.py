"""A plain, slow float64 implementation of the Munupel decoder, written from its equations.

One function per mechanism, no cache and no batching: the whole sequence is recomputed from its
first token, and attention goes one query at a time over a list of the keys it sees. It shares no
code with the library; the tests compare the library's logits and intermediate tensors with it.

Notation: h is a sublayer's input [T, width]; W x means x @ W.T for a matrix stored [out, in];
positions count from 0; w is the dictionary of the model's tensors, p a name prefix.
"""
import json
import math
import os
import struct

import torch

F64 = torch.float64


# --------------------------------------------------------------------------- reading a folder
def read_model(folder):
    """(config dict, name -> float64 tensor) of a model folder with one model.safetensors."""
    with open(os.path.join(folder, "config.json")) as handle:
        config = json.load(handle)
    with open(os.path.join(folder, "model.safetensors"), "rb") as handle:
        (size,) = struct.unpack("<Q", handle.read(8))
        header = json.loads(handle.read(size))
        data = handle.read()
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32, "F16": torch.float16}
    tensors = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        lo, hi = entry["data_offsets"]
        raw = torch.frombuffer(bytearray(data[lo:hi]), dtype=kinds[entry["dtype"]])
        tensors[name] = raw.reshape(entry["shape"]).to(F64)
    return config, tensors


# --------------------------------------------------------------------------- small pieces
def layer_norm(x, g, b, eps):
    """(x - mean) / sqrt(mean squared deviation + eps) * g + b."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * g + b


def softcap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def rotation(rot):
    """([frequency per pair], factor on cos and sin). With scaling, pair i's frequency f is f where
    the pair turns often within `original` positions, f / factor where it turns seldom, and a linear
    blend of both between: the dimension whose pair makes t turns is dims ln(original / 2 pi t) / 2 ln base."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not s:
        return freqs, 1.0

    def turning(t):
        return dims * math.log(s["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(turning(s["fast"])), 0), min(math.ceil(turning(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_halves(x, positions, rot):
    """x [T, heads, n]: dimension i pairs with i + dims/2 for i < dims/2; the rest unchanged."""
    half = rot["dims"] // 2
    freqs, stretch = rotation(rot)
    a = positions.to(F64)[:, None, None] * torch.tensor(freqs, dtype=F64)[None, None, :]
    cos, sin = torch.cos(a) * stretch, torch.sin(a) * stretch
    u, v = x[..., :half], x[..., half:2 * half]
    out = x.clone()
    out[..., :half] = u * cos - v * sin
    out[..., half:2 * half] = v * cos + u * sin
    return out


# --------------------------------------------------------------------------- which keys a query sees
def chunk_sees(i, size):
    """Keys of the query's own chunk of positions, up to itself (size None: every earlier key)."""
    return [j for j in range(i + 1) if size is None or i // size == j // size]


def window_sees(i, size, keep_first):
    """The newest `size` keys, and the sequence's first `keep_first` besides."""
    return [j for j in range(i + 1) if size is None or i - j < size or j < keep_first]


# --------------------------------------------------------------------------- attention
def attention(q, k, v, scale, sees, cap=None, sinks=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; sees(i): the keys query i sees. Softmax over capped
    scores; with `sinks` the denominator also holds exp(sink of the head). Returns [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for i in range(T):
        seen = torch.tensor(sees(i), dtype=torch.long)
        for head in range(H):
            g = head // (H // G)
            s = softcap((k[seen, g] @ q[i, head]) * scale, cap)
            top = s.max()
            if sinks is not None:
                top = torch.maximum(top, sinks[head])
            e = torch.exp(s - top)
            total = e.sum() + (torch.exp(sinks[head] - top) if sinks is not None else 0.0)
            out[i, head] = (e @ v[seen, g]) / total
    return out


def heads_of(h, m, w, p, bias):
    """The projections q [T, H, d], k [T, G, d], v [T, G, dv], q and k rotated by position."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (h @ w[p + n].T + (w[p + n + ".b"] if bias else 0.0) for n in "qkv")
    q, k, v = q.reshape(T, H, m["dim"]), k.reshape(T, G, m["dim"]), v.reshape(T, G, m["vdim"])
    if m.get("rot"):
        q, k = rotate_halves(q, torch.arange(T), m["rot"]), rotate_halves(k, torch.arange(T), m["rot"])
    return q, k, v


def chunked_attention(h, m, w, p):
    """Biased projections, capped scores, chunks of positions, a gate per head and value dimension."""
    q, k, v = heads_of(h, m, w, p, True)
    size = m["mask"]["size"] if m.get("mask") else None
    o = attention(q, k, v, m["scale"], lambda i: chunk_sees(i, size), cap=m.get("softcap"))
    o = o.reshape(h.shape[0], -1) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T + w[p + "o.b"]


def kept_window_attention(h, m, w, p):
    """A window beside kept first keys, a sink per head, a gate per head."""
    q, k, v = heads_of(h, m, w, p, False)
    mask = m.get("mask") or {"size": None, "keep_first": 0}
    o = attention(q, k, v, m["scale"], lambda i: window_sees(i, mask["size"], mask.get("keep_first", 0)),
                  sinks=w[p + "sink"])
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(h.shape[0], -1) @ w[p + "o"].T


MIXERS = {"attention": chunked_attention, "attention_2": kept_window_attention}


def feed_forward(h, w, p):
    z = h @ w[p + "gate"].T
    return (z * torch.sigmoid(z) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# --------------------------------------------------------------------------- the model
def tensors_of(config, i):
    """The layer whose tensors layer i uses."""
    while config["layers"][i].get("weights_of") is not None:
        i = config["layers"][i]["weights_of"]
    return i


def forward(config, w, tokens, layers_out=None, seen=lambda t: t):
    """Logits [T, vocab] of one sequence. `layers_out` (a list) receives the residual stream after
    every layer; `seen` is applied to a sublayer's input (the identity, or a rounding that mimics a
    16-bit product path)."""
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{tensors_of(config, i)}."
        h = seen(layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps))
        y = MIXERS[layer["type"]](h, layer["mixer"], w, p + "mix.")
        if layer.get("mlp"):
            y = y + feed_forward(h, w, p + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
