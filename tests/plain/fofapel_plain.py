"""A plain, slow implementation of the Fofapel decoder: one function per mechanism, whole sequences,
no cache, loops where loops are clearest.  It shares no code with the package under test, reads
``config.json`` and ``model.safetensors`` by itself and works on CPU tensors (float64 by default).

The design in short (n tokens of one sequence, positions 0 .. n-1, width d):

    x_0[t] = E[tok_t]
    every layer:  x <- LN1(alpha x + mixer(x));  x <- LN2(alpha x + ff(x))     (a layer may have no ff; nothing normed on the way in)
    logits = head . LNf(x)
    LN(u) = (u - mean u) / sqrt(var u + eps) * w + b

The mixer is two mixers on the same input, their results scaled and added: windowed grouped-query
attention whose values are its keys as projected, with a norm per head after the rotation, a sink of
score zero and one sigmoid gate per head ("left"); and a linear recurrence over time with a decay per
key channel made from the input, a bonus for the current token and a shift of the input by one token
("right").  Feed-forwards: a dense gated pair with the tanh form of gelu, or experts chosen by a table
of token ids, beside an expert that every token passes, scaled by a sigmoid of its own.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional, Sequence

import torch
from safetensors import safe_open

GLU_ALPHA = 1.702      # the slope inside the clamped pair's sigmoid


def read_folder(folder: str, dtype=torch.float64):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    tensors = {}
    with safe_open(os.path.join(folder, "model.safetensors"), framework="pt", device="cpu") as f:
        for name in f.keys():
            t = f.get_tensor(name)
            tensors[name] = t.to(dtype) if t.is_floating_point() else t
    return cfg, tensors


def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def _keep(x, store):
    """``store``: what a 16-bit path does where it writes an activation to memory (round and come back)."""
    return x if store is None else store(x)


# ----------------------------------------------------------------------------------------------
# small parts
# ----------------------------------------------------------------------------------------------
def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    mu = x.mean(dim=-1, keepdim=True)
    var = ((x - mu) ** 2).mean(dim=-1, keepdim=True)
    return (x - mu) / torch.sqrt(var + eps) * w + b


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


# ----------------------------------------------------------------------------------------------
# left: windowed attention whose values are its keys
# ----------------------------------------------------------------------------------------------
def rotate_pairs(v: torch.Tensor, position: int, dims: int, base: float) -> torch.Tensor:
    """v [..., >= dims]: entries 2i and 2i + 1 turn by position * base^(-2i/dims), the rest pass."""
    out = v.clone()
    for i in range(dims // 2):
        ang = position * base ** (-2.0 * i / dims)
        c, s = math.cos(ang), math.sin(ang)
        a, b = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = a * c - b * s
        out[..., 2 * i + 1] = b * c + a * s
    return out


def softmax_off_by_one(scores: torch.Tensor) -> torch.Tensor:
    """scores [m]: exp(s_j) / (1 + sum_j exp(s_j))."""
    top = max(float(scores.max()), 0.0)
    e = torch.exp(scores - top)
    return e / (e.sum() + math.exp(-top))


def visible(i: int, window: Optional[int]) -> range:
    """The positions that position i sees."""
    return range(0 if not window else max(0, i - window + 1), i + 1)


def attention_mixer(h, w, m, eps, store=None) -> torch.Tensor:
    """The heads' gated outputs [n, heads * dim], before the output projection."""
    n = h.shape[0]
    H, G, dim = m["heads"], m["kv_heads"], m["dim"]
    window = (m.get("mask") or {}).get("size")
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    hb = _keep(h, store)
    q = _keep(hb @ w["q"].T + w["q.b"], store).view(n, H, dim)
    k = _keep(hb @ w["k"].T + w["k.b"], store).view(n, G, dim)
    v = k.clone()
    for t in range(n):
        q[t] = rotate_pairs(q[t], t, rot["dims"], rot["base"])
    k = torch.stack([rotate_pairs(k[t], t, rot["dims"], rot["base"]) for t in range(n)])
    q, k = _keep(rms(q, eps), store), _keep(rms(k, eps), store)
    gate = torch.sigmoid(_keep(hb @ w["g"].T, store))
    out = torch.zeros(n, H, dim, dtype=h.dtype)
    for t in range(n):
        seen = visible(t, window)
        lo, hi = seen.start, seen.stop
        for head in range(H):
            g = head // (H // G)
            p = softmax_off_by_one((k[lo:hi, g] @ q[t, head]) * m["scale"])
            out[t, head] = (p @ v[lo:hi, g]) * gate[t, head]
    return out.view(n, H * dim)


# ----------------------------------------------------------------------------------------------
# right: a linear recurrence with a decay per key channel, a bonus and a token shift
# ----------------------------------------------------------------------------------------------
def token_shift(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    """h + (h' - h) mu, h' the row before (zeros before the first)."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def decay(mixed_w: torch.Tensor, w, store=None) -> torch.Tensor:
    """[n, heads * dim] in (0, 1).  The small product's input stays exact where a 16-bit path splits it."""
    return torch.exp(-torch.exp(torch.tanh(mixed_w @ w["w1"].T) @ w["w2"].T + w["w0"]))


def recurrence(r, k, v, dec, u) -> torch.Tensor:
    """r, k, v, dec [n, H, dim], u [H, dim]:  o_t = (S + diag(u) k v^T)^T r, then S = diag(dec) S + k v^T."""
    n, H, dim = r.shape
    S = torch.zeros(H, dim, dim, dtype=r.dtype)
    out = torch.zeros(n, H, dim, dtype=r.dtype)
    for t in range(n):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = ((S + u[:, :, None] * kv) * r[t][:, :, None]).sum(1)
        S = dec[t][:, :, None] * S + kv
    return out


def recurrence_mixer(h, w, m, eps, store=None) -> torch.Tensor:
    """The gated heads [n, heads * dim], before the output projection."""
    n = h.shape[0]
    H, dim = m["heads"], m["dim"]
    hb = _keep(h, store)
    mixed = {c: _keep(token_shift(hb, w["mu." + c]), store) for c in "rkvgw"}
    r, k, v = (_keep(mixed[c] @ w[c].T, store).view(n, H, dim) for c in "rkv")
    gate = silu(_keep(mixed["g"] @ w["g"].T, store))
    o = recurrence(r, k, v, decay(mixed["w"], w).view(n, H, dim), w["u"])
    return rms(o, eps).reshape(n, H * dim) * w["norm"] * gate


def mixer(h, w, m, eps, store=None) -> torch.Tensor:
    left, right = sub(w, "left."), sub(w, "right.")
    a = _keep(m["left_scale"] * attention_mixer(h, left, m["left"], eps, store), store)
    b = _keep(m["right_scale"] * recurrence_mixer(h, right, m["right"], eps, store), store)
    return _keep(a @ left["o"].T + b @ right["o"].T, store)


# ----------------------------------------------------------------------------------------------
# feed-forwards
# ----------------------------------------------------------------------------------------------
def dense_ff(h, w, store=None) -> torch.Tensor:
    hb = _keep(h, store)
    return _keep(_keep(gelu_tanh(hb @ w["gate"].T) * (hb @ w["up"].T), store) @ w["down"].T, store)


def clamped_pair(g, u, limit: float) -> torch.Tensor:
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(GLU_ALPHA * g) * (u + 1.0)


def expert(h, gate, up, down, limit, store=None) -> torch.Tensor:
    return _keep(_keep(clamped_pair(h @ gate.T, h @ up.T, limit), store) @ down.T, store)


def table_experts(h, tokens, w, f, store=None) -> torch.Tensor:
    hb = _keep(h, store)
    out = torch.zeros_like(h)
    top = f["router"]["top"]
    for t, tok in enumerate(tokens):
        for e in w["table"][tok].tolist():
            out[t] += expert(hb[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], f["expert"]["limit"], store) / top
    if f.get("shared"):
        y = expert(hb, w["shared.gate"], w["shared.up"], w["shared.down"], f["shared"]["limit"], store)
        out = out + torch.sigmoid(hb @ w["shared.sg"].T) * y
    return out


# ----------------------------------------------------------------------------------------------
# the model
# ----------------------------------------------------------------------------------------------
def forward(cfg, tensors, tokens: Sequence[int], store=None, layers_out: Optional[List] = None) -> torch.Tensor:
    """Logits [n, vocab] of every position."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = tensors["embed"][list(tokens)].clone()
    for i, layer in enumerate(cfg["layers"]):
        w = sub(tensors, f"l{i}.")
        x = layer_norm(alpha * x + mixer(x, sub(w, "mix."), layer["mixer"], eps, store), w["norm1"], w["norm1.b"], eps)
        f = layer["mlp"]
        if f is not None:
            y = dense_ff(x, sub(w, "mlp."), store) if f["kind"] == "dense" else \
                table_experts(x, tokens, sub(w, "mlp."), f, store)
            x = layer_norm(alpha * x + y, w["norm2"], w["norm2.b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return _keep(layer_norm(x, tensors["final.norm"], tensors["final.norm.b"], eps), store) @ tensors["head"].T
