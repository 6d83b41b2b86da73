"""A plain, slow Rudutar: one function per mechanism, whole sequences at once, no cache.

Written from the design's equations with torch on the CPU; it shares no code with the engine and
is the oracle of the tests.  Notation: x is the residual stream [T, W]; matrices are stored
[out, in] and applied as ``h @ W.T``; positions are 0 .. T-1; rms(y) = y / sqrt(mean(y^2) + eps).

    embedding        x = rms(E[token]) * w_e
    layer            x = x + mixer(rms(x) * w_1);  x = x + ff(rms(x) * w_2)      (the second only if the layer has an ff)
    attention        q, k, v through a causal convolution per channel (zeros before the start, no activation); q, k
                     RMS-normalised per head with one weight [dim] for all heads; q times
                     1 + coef ln(floor((p + 1) / every) + 1); score s_ij = q_i . k_j scale - 2^(-8 (h+1) / H) (i - j) for
                     0 <= i - j < size; weights exp(s_ij) / (1 + sum_j exp(s_ij)); heads times sigmoid(W_g h) element
                     by element; W_o.  With kv_from j the keys and values are layer j's.
    attention_2      q = W_q h + b_q, k = W_k h + b_k, values = k; q, k RMS-normalised as whole projections, the first
                     ``rot.dims`` elements of each head rotated (pairs i, i + dims/2); the same window, an ordinary
                     softmax; head h times sigmoid(W_g h)_h; W_o
    dense ff         W_down gelu(W_up h), gelu with the error function
    routed ff        s = sigmoid(W_r h); choice c = s + correction; a group's score is the sum of its two largest c; of
                     the best ``keep`` groups the ``top`` experts with the largest c; weights s * router.scale, not
                     divided by their sum; experts W_down relu(W_up h)^2; a shared expert of that form is added
    output           logits = head (rms(x) * w_f)
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch


# ---- files ---------------------------------------------------------------------------------------
def read_safetensors(path) -> dict[str, torch.Tensor]:
    data = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", data[:8])
    header = json.loads(data[8:8 + n])
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32, "F16": torch.float16}
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        buf = bytearray(data[8 + n + a: 8 + n + b])
        out[name] = torch.frombuffer(buf, dtype=kinds[info["dtype"]]).reshape(info["shape"]).clone()
    return out


def load_folder(folder, dtype=torch.float64):
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    w = {k: (v.to(dtype) if v.is_floating_point() else v)
         for k, v in read_safetensors(folder / "model.safetensors").items()}
    return cfg, w


# ---- small functions -------------------------------------------------------------------------------
def unit_rms(y, eps):
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def short_convolution(z, taps):
    """z [T, C], taps [C, K]: y_t = sum_i taps[:, i] z_(t - (K-1) + i), zeros before the start."""
    T, K = z.shape[0], taps.shape[1]
    padded = torch.cat((torch.zeros(K - 1, z.shape[1], dtype=z.dtype), z), 0)
    return sum(padded[i:i + T] * taps[:, i] for i in range(K))


def temperature(positions, coef, every):
    p = positions.double()
    return 1.0 + coef * torch.log(torch.floor((p + 1.0) / every) + 1.0)


def slopes(heads):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float64)


def rotate_half_split(t, positions, dims, base):
    """t [T, n, d]: element i of the first ``dims`` turns together with element i + dims/2 by the angle
    position * base^(-2i/dims)."""
    half = dims // 2
    i = torch.arange(half, dtype=t.dtype)
    a = positions.to(t.dtype)[:, None] * (base ** (-2.0 * i / dims))[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = t[..., :half], t[..., half:dims]
    return torch.cat((u * c - v * s, v * c + u * s, t[..., dims:]), -1)


# ---- attention over a window ------------------------------------------------------------------------
def window_attend(q, k, v, scale, size, slope=None, sink=False, qpos=None):
    """q [R, H, d] at the positions ``qpos`` (default 0 .. R-1), k [L, G, d], v [L, G, dv].  Query i sees the positions j
    with 0 <= i - j < size; ``slope`` [H] takes slope_h (i - j) off the scaled score; ``sink`` adds one to the
    softmax's denominator.  Returns [R, H, dv]."""
    R, H, _ = q.shape
    L, G = k.shape[0], k.shape[1]
    i = (torch.arange(R) if qpos is None else torch.as_tensor(qpos))[:, None]
    j = torch.arange(L)[None, :]
    seen = (j <= i) & (i - j < size)
    out = []
    for hd in range(H):
        g = hd // (H // G)
        s = q[:, hd] @ k[:, g].T * scale
        if slope is not None:
            s = s - slope[hd].to(s.dtype) * (i - j).to(s.dtype)
        s = s.masked_fill(~seen, -math.inf)
        top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0) if sink else s.max(-1, keepdim=True).values
        e = torch.exp(s - top)
        total = e.sum(-1, keepdim=True) + (torch.exp(-top) if sink else 0.0)
        out.append((e / total) @ v[:, g])
    return torch.stack(out, 1)


def sloped_inputs(h, w, p, m, eps):
    """q [T, H, d], k [T, G, d], v [T, G, dv] of an "attention" layer; k and v None for one with kv_from."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms(short_convolution(h @ w[p + "q"].T, w[p + "q.conv"]).view(T, H, d), eps) * w[p + "q.norm"]
    if m.get("q_temp"):
        q = q * temperature(torch.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"]).to(q.dtype)[:, None, None]
    if m.get("kv_from") is not None:
        return q, None, None
    k = unit_rms(short_convolution(h @ w[p + "k"].T, w[p + "k.conv"]).view(T, G, d), eps) * w[p + "k.norm"]
    v = short_convolution(h @ w[p + "v"].T, w[p + "v.conv"]).view(T, G, dv)
    return q, k, v


def sloped_attention(h, w, p, m, eps, kv):
    """``kv``: {layer index: (k, v)} of the layers before; returns (the mixer's output, its own (k, v) or None)."""
    q, k, v = sloped_inputs(h, w, p, m, eps)
    mine = None if k is None else (k, v)
    if k is None:
        k, v = kv[m["kv_from"]]
    out = window_attend(q, k, v, m["scale"], m["mask"]["size"], slope=slopes(m["heads"]), sink=True)
    out = out.reshape(h.shape[0], -1) * torch.sigmoid(h @ w[p + "g"].T)
    return out @ w[p + "o"].T, mine


def key_value_inputs(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    qp, kp = h @ w[p + "q"].T + w[p + "q.b"], h @ w[p + "k"].T + w[p + "k.b"]
    q = (unit_rms(qp, eps) * w[p + "q.norm"]).view(T, H, d)
    k = (unit_rms(kp, eps) * w[p + "k.norm"]).view(T, G, d)
    pos = torch.arange(T)
    rot = m.get("rot") or {"dims": 0}
    if rot["dims"]:
        q, k = rotate_half_split(q, pos, rot["dims"], rot["base"]), rotate_half_split(k, pos, rot["dims"], rot["base"])
    return q, k, kp.view(T, G, d)


def key_value_attention(h, w, p, m, eps, kv):
    q, k, v = key_value_inputs(h, w, p, m, eps)
    out = window_attend(q, k, v, m["scale"], m["mask"]["size"])
    out = out * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return out.reshape(h.shape[0], -1) @ w[p + "o"].T, None


# ---- feed-forwards -----------------------------------------------------------------------------------
def dense_ff(h, w, p):
    return gelu(h @ w[p + "up"].T) @ w[p + "down"].T


def expert(h, w, p):
    return relu_squared(h @ w[p + "up"].T) @ w[p + "down"].T


def route(h, w, p, r):
    """(chosen [T, top], weights [T, top]) of a router."""
    s = torch.sigmoid(h @ w[p + "router"].T)
    c = s + w[p + "correction"]
    n = s.shape[-1]
    groups = r.get("groups")
    if groups:
        per = n // groups["count"]
        g = c.view(-1, groups["count"], per)
        score = torch.topk(g, min(2, per), -1).values.sum(-1)
        best = torch.topk(score, groups["keep"], -1).indices
        keep = torch.zeros_like(score, dtype=torch.bool).scatter_(1, best, True)
        c = c.masked_fill(~keep.repeat_interleave(per, 1), -math.inf)
    chosen = torch.topk(c, r["top"], -1).indices
    return chosen, torch.gather(s, 1, chosen) * r.get("scale", 1.0)


def routed_ff(h, w, p, mlp):
    chosen, weights = route(h, w, p, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(chosen[t].tolist(), weights[t]):
            out[t] += a * expert(h[t], w, f"{p}e{e}.")
    if mlp.get("shared"):
        out = out + expert(h, w, p + "shared.")
    return out


MIXERS = {"attention": sloped_attention, "attention_2": key_value_attention}


# ---- the model ----------------------------------------------------------------------------------------
def forward(cfg, w, tokens, return_layers=False):
    """Logits [T, vocab] of one whole sequence; with return_layers also the stream after every layer."""
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = unit_rms(w["embed"][tokens], eps) * w["embed.norm"]
    streams, kv = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y, own = MIXERS[layer["type"]](unit_rms(x, eps) * w[p + "norm1"], w, p + "mix.", layer["mixer"], eps, kv)
        if own is not None:
            kv[i] = own
        x = x + y
        mlp = layer.get("mlp")
        if mlp is not None:
            h = unit_rms(x, eps) * w[p + "norm2"]
            x = x + (dense_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else routed_ff(h, w, p + "mlp.", mlp))
        streams.append(x.clone())
    logits = (unit_rms(x, eps) * w["final.norm"]) @ w["head"].T
    return (logits, torch.stack(streams)) if return_layers else logits


def generate(cfg, w, prompt, n):
    """Greedy continuation, recomputing the whole sequence for every token."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(forward(cfg, w, tokens)[-1].argmax()))
    return tokens[len(prompt):]
