"""A plain, slow float64 implementation of the Tolurax decoder, written from its equations.

One function per mechanism, no cache and no batching: the whole sequence is recomputed from its
first token, the recurrences token by token. It shares no code with the library; the tests compare
the library's logits and intermediate tensors with it.

Notation: h is a mixer's input [T, width]; W x means x @ W.T for a matrix stored [out, in];
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
def unit_rms(x, eps):
    """x divided by its root mean square over the last dimension, eps under the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, g, eps):
    """(x - mean) / sqrt(mean squared deviation + eps) * g; no bias."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * g


def silu(z):
    return z * torch.sigmoid(z)


def causal_conv(x, taps):
    """y_t[c] = sum_j taps[c, j] x_(t - (n-1) + j)[c], zeros before the start, no bias."""
    T, n = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros((n - 1, x.shape[1]), dtype=F64), x], dim=0)
    y = torch.zeros_like(x)
    for j in range(n):
        y = y + padded[j:j + T] * taps[:, j]
    return y


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def frequencies(rot):
    """The rotation's frequencies, slow ones stretched: with wavelength l = 2 pi / f, as they are
    where l < original / high, divided by factor where l > original / low, a blend between."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                mix = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - mix) * f / s["factor"] + mix * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_halves(x, positions, rot):
    """x [T, heads, n]: dimension i pairs with i + dims/2 for i < dims/2; the rest unchanged."""
    half = rot["dims"] // 2
    a = positions.to(F64)[:, None, None] * frequencies(rot)[None, None, :]
    cos, sin = torch.cos(a), torch.sin(a)
    u, v = x[..., :half], x[..., half:2 * half]
    out = x.clone()
    out[..., :half] = u * cos - v * sin
    out[..., half:2 * half] = v * cos + u * sin
    return out


def sigmoid_attention(q, k, v, scale, offsets, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: every key at most window - 1 positions back counts with
    the weight sigmoid(scale q.k + offset of the head); nothing is normalized. Returns [T, H dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) & (i - j < (window if window else T + 1))
    out = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for head in range(H):
        g = head // (H // G)
        weights = torch.sigmoid((q[:, head] @ k[:, g].T) * scale + offsets[head])
        out[:, head] = (weights * seen) @ v[:, g]
    return out.reshape(T, -1)


def delta_scan(q, k, v, g, beta):
    """q, k [T, H, d], v [T, H, dv], decay g and step size beta [T, H]. Per head:
    S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q."""
    T, H, d = q.shape
    out = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for head in range(H):
        S = torch.zeros((d, v.shape[2]), dtype=F64)
        for t in range(T):
            S = g[t, head] * S
            u = beta[t, head] * (v[t, head] - S.T @ k[t, head])
            S = S + torch.outer(k[t, head], u)
            out[t, head] = S.T @ q[t, head]
    return out


def bonus_scan(r, k, v, decay, bonus):
    """r, k, decay [T, H, d], v [T, H, dv], bonus [H, d]. Per head the read-out comes before the
    write and the current token counts under the bonus: o = (S + diag(bonus) k v^T)^T r, then
    S <- diag(decay) S + k v^T."""
    T, H, d = r.shape
    out = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for head in range(H):
        S = torch.zeros((d, v.shape[2]), dtype=F64)
        for t in range(T):
            kv = torch.outer(k[t, head], v[t, head])
            out[t, head] = (S + bonus[head][:, None] * kv).T @ r[t, head]
            S = decay[t, head][:, None] * S + kv
    return out


# --------------------------------------------------------------------------- mixers
def gated_delta(h, m, w, p, eps):
    """Gated delta rule with one decay per head: short convolutions and SiLU on q, k and v, unit
    queries and keys, unit RMS per head, a weight shared by the heads, a SiLU gate."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit_vector(q.reshape(T, G, d)) * d ** -0.5
    k = unit_vector(k.reshape(T, G, d))
    q, k = (x.repeat_interleave(H // G, dim=1) for x in (q, k))
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = unit_rms(delta_scan(q, k, v.reshape(T, H, dv), g, beta), eps) * w[p + "norm"]
    return (o.reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def window_attention(h, m, w, p, eps):
    """Unnormalized sigmoid attention through a window: a weighted RMS norm per query and key head,
    a split-half rotation with stretched frequencies, a sigmoid gate per head and value dimension."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w[p + "q"].T).reshape(T, H, d), eps) * w[p + "q.norm"]
    k = unit_rms((h @ w[p + "k"].T).reshape(T, G, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    if m.get("rot"):
        q, k = rotate_halves(q, torch.arange(T), m["rot"]), rotate_halves(k, torch.arange(T), m["rot"])
    window = m["mask"]["size"] if m.get("mask") else None
    o = sigmoid_attention(q, k, v, m["scale"], w[p + "pb"], window)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def time_mix(h, m, w, p, eps):
    """A matrix state with a decay per key channel computed from the input and a bonus for the
    current token; every projection reads its own mix of h with the row before (zeros first)."""
    T, H, d = h.shape[0], m["heads"], m["dim"]
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)

    def mixed(s):
        return h + (before - h) * w[p + "mu." + s]
    r, k, v = ((mixed(s) @ w[p + s].T).reshape(T, H, d) for s in ("r", "k", "v"))
    inner = torch.tanh(mixed("w") @ w[p + "w1"].T)
    decay = torch.exp(-torch.exp(inner @ w[p + "w2"].T + w[p + "w0"])).reshape(T, H, d)
    o = unit_rms(bonus_scan(r, k, v, decay, w[p + "u"]), eps).reshape(T, H * d)
    return (o * w[p + "norm"] * silu(mixed("g") @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, m, w, p, eps):
    return m["left_scale"] * window_attention(h, m["left"], w, p + "left.", eps) \
        + m["right_scale"] * time_mix(h, m["right"], w, p + "right.", eps)


MIXERS = {"delta": gated_delta, "parallel": parallel}


def feed_forward(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# --------------------------------------------------------------------------- the model
def layer_runs(config):
    """[(layer, starts a pass of the looped run)] in the order the layers run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, False) for i in range(start)]
    for _ in range(times):
        runs += [(i, i == start) for i in range(start, stop)]
    return runs + [(i, False) for i in range(stop, n)]


def softcap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def forward(config, w, tokens, layers_out=None, seen=lambda t: t):
    """Logits [T, vocab] of one sequence. `layers_out` (a list) receives the residual stream after
    every layer run; `seen` is applied to a sublayer's input (the identity, or a rounding that
    mimics a 16-bit product path)."""
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x0 = x.clone()
    for i, starts in layer_runs(config):
        if starts:
            x = torch.cat([x, x0], dim=1) @ w["loop.in"].T
        layer, p = config["layers"][i], f"l{i}."
        h = seen(layer_norm(x, w[p + "norm1"], eps))
        h = seen(h + causal_conv(h, w[p + "canon1"]))
        x = x + MIXERS[layer["type"]](h, layer["mixer"], w, p + "mix.", eps)
        if layer.get("mlp"):
            x = x + feed_forward(seen(layer_norm(x, w[p + "norm2"], eps)), w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.clone())
    return softcap(layer_norm(x, w["final.norm"], eps) @ w["head"].T, config.get("logit_softcap"))
