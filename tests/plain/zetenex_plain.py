"""A plain, slow Zetenex: one function per mechanism, whole sequences at once, no cache.

Written from the design's equations with torch on the CPU; it shares no code with the engine and
is the oracle of the tests.  Notation: x is the residual stream [T, W]; matrices are stored
[out, in] and applied as ``h @ W.T``; positions are 0 .. T-1.

    embedding        x0 = s E[token];  x = x0
    passes           layers start .. stop-1 run ``times`` times; pass t opens with x <- x + x0 (t > 0), x <- x + step[t]
    layer            x = x + mixer(c1(n1(x)));  x = x + ff(c2(n2(x)))
                     n(x) = tanh(alpha x) w + b;   c(h)_t = h_t + sum_j f[:, j] h_(t - taps + 1 + j)
    mingru           z = sigmoid(W_z h + b_z);  u = W_x h + b_x;  g(u) = u + 1/2 (u >= 0) or sigmoid(u);
                     S_t = (1 - z) S_(t-1) + z g(u);  W_o (S silu(W_g h))
    parallel         a attention(h) + b scan(h)
      attention      q, k divided by their root mean square per head; q times 1 + coef ln(floor((p + 1) / every) + 1);
                     softmax over j <= i of scale q . k;  head h times sigmoid(W_g h)_h;  W_o
      scan           [x | z] = W_in h;  x = silu(conv(x) + bias);  [dt | B | C] = W_x x;  dt = softplus(W_dt dt + b);
                     S = exp(dt A) S + dt x B;  y = S C + D x;  W_o (y silu(z)),  A = -exp(A_log)
    ff               W_down gelu(W_up h), the tanh form
    output           logits = E n_final(x)
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
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32}
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
    return cfg, {k: v.to(dtype) for k, v in read_safetensors(folder / "model.safetensors").items()}


# ---- small functions -------------------------------------------------------------------------------
def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def dynamic_tanh(x, alpha, weight, shift):
    return torch.tanh(alpha * x) * weight + shift


def convolve(h, filters):
    """sum_j filters[:, j] h_(t - taps + 1 + j), zeros before the start: h [T, C], filters [C, taps]."""
    T, taps = h.shape[0], filters.shape[1]
    padded = torch.cat((torch.zeros(taps - 1, h.shape[1], dtype=h.dtype), h), 0)
    return sum(padded[j:j + T] * filters[:, j] for j in range(taps))


def with_convolution(h, filters):
    return h + convolve(h, filters)


# ---- minGRU -----------------------------------------------------------------------------------------
def gru_states(zl, u, start=None):
    """All states of S <- (1 - sigmoid(zl)) S + sigmoid(zl) g(u), from ``start`` (default zero)."""
    z = torch.sigmoid(zl)
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S = torch.zeros_like(zl[0]) if start is None else start.clone()
    out = []
    for t in range(zl.shape[0]):
        S = (1 - z[t]) * S + z[t] * cand[t]
        out.append(S)
    return torch.stack(out)


def mingru(h, w, p, m, eps):
    S = gru_states(h @ w[p + "z"].T + w[p + "z.b"], h @ w[p + "x"].T + w[p + "x.b"])
    return (S * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- attention over unit q and k ------------------------------------------------------------------------
def unit(y, eps):
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)


def query_temperature(positions, temp):
    if temp is None:
        return torch.ones(len(positions), dtype=torch.float64)
    return torch.tensor([1.0 + temp["coef"] * math.log(math.floor((int(p) + 1) / temp["every"]) + 1) for p in positions],
                        dtype=torch.float64)


def causal_softmax(q, k, v, scale, first=0):
    """q [R, H, d] at the positions first .. first + R - 1 over k [L, G, d], v [L, G, dv]; query i sees every j <= i."""
    R, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(R, H, v.shape[-1], dtype=q.dtype)
    for i in range(R):
        n = first + i + 1
        for hd in range(H):
            g = hd // (H // G)
            out[i, hd] = torch.softmax(scale * (k[:n, g] @ q[i, hd]), 0) @ v[:n, g]
    return out


def attention(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit((h @ w[p + "q"].T).view(T, H, d), eps) * query_temperature(range(T), m.get("q_temp")).to(h.dtype)[:, None, None]
    k = unit((h @ w[p + "k"].T).view(T, G, d), eps)
    v = (h @ w[p + "v"].T).view(T, G, dv)
    o = causal_softmax(q, k, v, m["scale"])
    return (o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, H * dv) @ w[p + "o"].T


# ---- the selective scan -----------------------------------------------------------------------------------
def selective_states(x, dt, A, B, C, start=None):
    """(sum over states of S C per token and channel, the last S): x, dt [T, inner], A [inner, N], B, C [T, N]."""
    S = torch.zeros_like(A) if start is None else start.clone()
    ys = []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        ys.append(S @ C[t])
    return torch.stack(ys), S


def selective_scan(h, w, p, m, eps):
    n, N, R = m["inner"], m["state"], m["dt_rank"]
    xz = h @ w[p + "in"].T
    x = silu(convolve(xz[:, :n], w[p + "conv"]) + w[p + "conv.b"])
    low = x @ w[p + "x"].T
    dt = softplus(low[:, :R] @ w[p + "dt"].T + w[p + "dt.b"])
    y, _ = selective_states(x, dt, -torch.exp(w[p + "A_log"]), low[:, R:R + N], low[:, R + N:])
    return ((y + w[p + "D"] * x) * silu(xz[:, n:])) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return (m["left_scale"] * attention(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * selective_scan(h, w, p + "right.", m["right"], eps))


MIXERS = {"mingru": mingru, "parallel": parallel}


# ---- the model ----------------------------------------------------------------------------------------
def run_order(cfg):
    """(layer, the pass that opens with it or None) of every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, None) for i in range(a)]
            + [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
            + [(i, None) for i in range(b, n)])


def forward(cfg, w, tokens, return_layers=False):
    """Logits [T, vocab] of one whole sequence; with return_layers also the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    x = x0
    streams = []

    def norm(x, name):
        return dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])

    for i, opens in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if opens is not None:
            x = (x + x0 if opens else x) + w["loop.step"][opens]
        h = with_convolution(norm(x, p + "norm1"), w[p + "canon1"])
        x = x + MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            h = with_convolution(norm(x, p + "norm2"), w[p + "canon2"])
            x = x + gelu_tanh(h @ w[p + "mlp.up"].T) @ w[p + "mlp.down"].T
        streams.append(x)
    logits = norm(x, "final.norm") @ w["embed"].T
    return (logits, torch.stack(streams)) if return_layers else logits


def generate(cfg, w, prompt, n):
    """Greedy continuation, recomputing the whole sequence for every token."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(forward(cfg, w, tokens)[-1].argmax()))
    return tokens[len(prompt):]
