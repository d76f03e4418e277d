"""A plain, slow implementation of the Bogivik forward pass: whole sequences, no cache, one function per mechanism, on the
CPU in float64 (or float32).  It shares no code with ``zedinfer_b200``: it reads ``config.json`` with ``json`` and
``model.safetensors`` with its own few lines.

The design in this file's notation (``x`` the residual stream, ``t`` a token's index in its sequence, ``sg`` the logistic
function, ``U(v) = v / sqrt(mean(v^2) + eps)``):

    x_t = E[token_t]
    per layer:     a = U(x) w1;   x += mixer(a) + ff(a)                 (one norm, both sublayers read it)
    logits = Wh (U(x) wf)

    attention:     H query heads on G key/value heads, no biases, no rotation; q = U(Wq a) wq and k = U(Wk a) wk over all rows
                   of the projection at once; q times 1 + c ln(floor((t + 1) / every) + 1);
                   score(t, j) = q . k scale + R[bucket(t - j), head];  j <= t;  softmax;  out = Wo (heads * sg(Wg a));
                   bucket(n) = n below B/2, then logarithmic up to the distance D, B - 1 from there on;
                   v <- (1 - l) v + l v1 in every v_mix layer but the first, v1 that first layer's v of the same token
    parallel:      two mixers read the same input; the result is (U(left) w_l + U(right) w_r) / 2
      left         attention with biases on q, k, v and the output projection; q and k heads normed one by one, U(.) w; the
                   first r entries of a head turned, pair (2i, 2i + 1) by the angle t f_i, f_i stretched for long contexts;
                   key j answers query t when j <= t and floor(t / C) = floor(j / C);  gated like the other
      right        q = Wq a / sqrt(dim), k = Wk a, v = Wv a;  i = cap tanh((Wi a + bi) / cap),
                   f = ln sg(cap tanh((Wf a + bf) / cap))  per head;  m' = max(f + m, i), m = 0 before the first token;
                   S <- e^(f + m - m') S + e^(i - m') k v^T;  n <- e^(f + m - m') n + e^(i - m') k;
                   o = S^T q / (max(|n . q|, e^-m') + 1e-6);   out = Wo (U_head(o) * w_n * sg(Wg a))
    ff:            Wdown (gelu(Wgate a) * Wup a),  gelu(z) = z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))) / 2
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import torch

READ_OUT_EPS = 1e-6              # added to the divisor of the exponential-gate read-out


def read_safetensors(path: str, dtype=torch.float64) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    kinds = {"F32": torch.float32, "BF16": torch.bfloat16, "F16": torch.float16, "I32": torch.int32, "F64": torch.float64}
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        b, e = info["data_offsets"]
        t = torch.frombuffer(bytearray(data[b:e]), dtype=kinds[info["dtype"]]).reshape(info["shape"])
        out[name] = t.to(dtype) if t.is_floating_point() else t.clone()
    return out


def read_model(model_dir: str, dtype=torch.float64):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"), dtype)


# ---------------------------------------------------------------------------------------------
# mechanisms, one function each
# ---------------------------------------------------------------------------------------------
def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def logistic(x: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-x))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def distance_bucket(n: int, buckets: int, farthest: float) -> int:
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(farthest / half) * (buckets - half)))


def query_temperature(t: int, coef: float, every: float) -> float:
    return 1.0 + coef * math.log(math.floor((t + 1) / every) + 1.0)


def turn_frequencies(dims: int, base: float, scaling: Optional[dict]) -> List[float]:
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wave = 2.0 * math.pi / f
            short, long = scaling["original"] / scaling["high"], scaling["original"] / scaling["low"]
            if wave > long:
                f = f / scaling["factor"]
            elif wave >= short:
                s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def turn_pairs(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float, scaling: Optional[dict] = None) -> torch.Tensor:
    """x [tokens, heads, dim]: entries 2i and 2i + 1 of the first ``dims`` are a pair."""
    f = torch.tensor(turn_frequencies(dims, base, scaling), dtype=x.dtype)
    ang = positions.to(x.dtype)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return out


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, seen: torch.Tensor,
           bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q [n, H, d], k [n, G, d], v [n, G, dv], seen [n, n], bias [H, n, n] or None -> [n, H * dv]."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * scale
        if bias is not None:
            s = s + bias[a]
        out[:, a] = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, g]
    return out.reshape(n, -1)


def mixed_values(v: torch.Tensor, first: Optional[torch.Tensor], lam) -> torch.Tensor:
    return v if first is None else (1.0 - lam) * v + lam * first


def biased_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, shared: dict) -> torch.Tensor:
    """``shared["v"]``: the first v_mix layer's values, left there by that layer."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit(h @ w[p + "q"].T, eps) * w[p + "q.norm"]
    k = rms_unit(h @ w[p + "k"].T, eps) * w[p + "k.norm"]
    v = h @ w[p + "v"].T
    if m.get("q_temp"):
        q = q * torch.tensor([query_temperature(t, m["q_temp"]["coef"], m["q_temp"]["every"]) for t in range(n)], dtype=h.dtype)[:, None]
    if m.get("v_mix"):
        first = shared.get("v")
        if first is None:
            shared["v"] = v
        v = mixed_values(v, first, w[p + "vmix"])
    pos = torch.arange(n)
    dist = pos[:, None] - pos[None, :]
    rel = w[p + "rel"]
    b = torch.tensor([distance_bucket(i, rel.shape[0], m["bias_max"]) for i in range(n)])
    bias = rel[b[dist.clamp(min=0)]].permute(2, 0, 1)
    o = attend(q.view(n, H, d), k.view(n, G, d), v.view(n, G, dv), m["scale"], dist >= 0, bias)
    return (o * logistic(h @ w[p + "g"].T)) @ w[p + "o"].T


def chunked_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit((h @ w[p + "q"].T + w[p + "q.b"]).view(n, H, d), eps) * w[p + "q.norm"]
    k = rms_unit((h @ w[p + "k"].T + w[p + "k.b"]).view(n, G, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, dv)
    pos, rot = torch.arange(n), m["rot"]
    q, k = (turn_pairs(z, pos, rot["dims"], rot["base"], rot.get("scaling")) for z in (q, k))
    chunk = pos // (m["mask"]["size"] if m.get("mask") else n)
    seen = (pos[:, None] >= pos[None, :]) & (chunk[:, None] == chunk[None, :])
    o = attend(q, k, v, m["scale"], seen)
    return (o * logistic(h @ w[p + "g"].T)) @ w[p + "o"].T + w[p + "o.b"]


def exponential_gates(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, cap: float):
    """(input gate, forget gate), both as logarithms, [n, heads]."""
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    z = cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap)
    return i, torch.nn.functional.logsigmoid(z)


def exponential_gate_walk(q, k, v, i, f, start=None):
    """q, k [n, H, d], v [n, H, dv], i, f [n, H] -> (o [n, H, dv], (S, n, m) after the last token)."""
    n, H, d = q.shape
    dv = v.shape[2]
    S, nn, m = start if start is not None else (torch.zeros(H, d, dv, dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype),
                                                torch.zeros(H, dtype=q.dtype))
    o = torch.zeros(n, H, dv, dtype=q.dtype)
    for t in range(n):
        m1 = torch.maximum(f[t] + m, i[t])
        fade, write = torch.exp(f[t] + m - m1), torch.exp(i[t] - m1)
        S = fade[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        nn = fade[:, None] * nn + write[:, None] * k[t]
        m = m1
        under = torch.maximum((nn * q[t]).sum(-1).abs(), torch.exp(-m)) + READ_OUT_EPS
        o[t] = torch.einsum("hdv,hd->hv", S, q[t]) / under[:, None]
    return o, (S, nn, m)


def matrix_memory(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    i, f = exponential_gates(h, w, p, m["gate_cap"])
    o, _ = exponential_gate_walk((h @ w[p + "q"].T).view(n, H, d) * d ** -0.5, (h @ w[p + "k"].T).view(n, H, d),
                                 (h @ w[p + "v"].T).view(n, H, dv), i, f)
    o = rms_unit(o, eps).reshape(n, H * dv) * w[p + "norm"] * logistic(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def parallel_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    left = chunked_attention(h, w, p + "left.", m["left"], eps)
    right = matrix_memory(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms_unit(left, eps) * w[p + "left.out"] + rms_unit(right, eps) * w[p + "right.out"])


def gelu_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ---------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], trace: List[torch.Tensor] = None) -> torch.Tensor:
    """Logits [tokens, vocab] of one sequence; ``trace`` collects the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    shared: dict = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms_unit(x, eps) * w[p + "norm1"]
        if layer["type"] == "parallel":
            y = parallel_mixer(h, w, p + "mix.", layer["mixer"], eps)
        elif layer["type"] == "attention":
            y = biased_attention(h, w, p + "mix.", layer["mixer"], eps, shared)
        else:
            raise ValueError(f"layer {i}: unknown type {layer['type']!r}")
        if layer.get("mlp") is not None:
            y = y + gelu_ff(h, w, p + "mlp.")
        x = x + y
        if trace is not None:
            trace.append(x.clone())
    return (rms_unit(x, eps) * w["final.norm"]) @ w["head"].T


def greedy(cfg: dict, w: Dict[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    seq = list(prompt)
    for _ in range(n_new):
        seq.append(int(torch.argmax(forward(cfg, w, seq)[-1])))
    return seq[len(prompt):]
