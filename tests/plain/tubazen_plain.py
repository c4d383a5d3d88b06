"""A plain, slow implementation of the Tubazen decoder: one function per mechanism, whole sequences,
no cache, loops where loops are clearest.  It shares no code with the package under test, reads
``config.json`` and ``model.safetensors`` by itself and works on CPU tensors (float64 by default).

The design in short (n tokens of one sequence, positions 0 .. n-1, width d):

    N(u) = tanh(alpha u) w + b                         (a number alpha, vectors w and b; no statistics)
    X_0[t] = N(E[tok_t] + P[t]);   x = X_0
    layer i:  h = N1(x);  x <- x + mixer(h) * sigmoid(R1 h + r1)
              h = N2(x);  x <- x + ff(h) * sigmoid(R2 h + r2)        (a layer may have no ff)
              X_{i+1} = x;   x <- sum_{j <= i+1} c_ij X_j
    logits = head . N(x) * logit_scale

Mixers: "gla", a linear attention whose memory fades per key channel; "parallel", two mixers on the
same input, scaled and added: grouped-query attention with biases, a query multiplier that grows with
the position, a learned bias per (distance bucket, head) and an output gate ("left"), and a delta rule
with separate decay, removal rate and key ("right").  The feed-forward is a gated pair with the tanh
form of gelu.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional, Sequence

import torch
from safetensors import safe_open

UNIT_EPS = 1e-6


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
def tanh_norm(x: torch.Tensor, tensors, name: str) -> torch.Tensor:
    return torch.tanh(tensors[name + ".alpha"] * x) * tensors[name] + tensors[name + ".b"]


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def residual_gate(h, w, name, store=None) -> torch.Tensor:
    return torch.sigmoid(_keep(_keep(h, store) @ w[name].T, store) + w[name + ".b"])


def depth_average(history: Sequence[torch.Tensor], weights: torch.Tensor) -> torch.Tensor:
    out = torch.zeros_like(history[0])
    for j, x in enumerate(history):
        out = out + weights[j] * x
    return out


# ----------------------------------------------------------------------------------------------
# gated linear attention
# ----------------------------------------------------------------------------------------------
def gla_decay(h, w, tau: float) -> torch.Tensor:
    """[n, heads * dim] in (0, 1)."""
    return torch.sigmoid((h @ w["a1"].T) @ w["a2"].T + w["a2.b"]) ** (1.0 / tau)


def gla_recurrence(q, k, v, alpha) -> torch.Tensor:
    """q, k, alpha [n, H, dim], v [n, H, vdim]:  S = diag(alpha_t) S + k_t v_t^T;  o_t = S^T q_t."""
    n, H, dim = q.shape
    S = torch.zeros(H, dim, v.shape[2], dtype=q.dtype)
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for t in range(n):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def gla_mixer(h, w, m, eps, store=None) -> torch.Tensor:
    n = h.shape[0]
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    hb = _keep(h, store)
    q = _keep(hb @ w["q"].T, store).view(n, H, dim) * dim ** -0.5
    k = _keep(hb @ w["k"].T, store).view(n, H, dim)
    v = _keep(hb @ w["v"].T, store).view(n, H, vdim)
    o = gla_recurrence(q, k, v, gla_decay(hb, w, m["tau"]).view(n, H, dim))
    o = (rms(o, eps) * w["norm"]).reshape(n, H * vdim)
    return _keep(_keep(o * silu(_keep(hb @ w["g"].T, store)), store) @ w["o"].T, store)


# ----------------------------------------------------------------------------------------------
# left: attention with a bias by distance
# ----------------------------------------------------------------------------------------------
def bucket(n: int, rows: int, far: int) -> int:
    """The row of the bias table for a key n positions back."""
    half = rows // 2
    if n < half:
        return n
    # a quotient that is a whole number may come out a rounding below it
    steps = math.log(n / half) / math.log(far / half) * (rows - half)
    return min(rows - 1, half + math.floor(steps + 1e-9))


def query_temperature(p: int, coef: float, every: float) -> float:
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0)


def left_mixer(h, w, m, store=None) -> torch.Tensor:
    """The heads' gated outputs [n, heads * vdim], before the output projection."""
    n = h.shape[0]
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    hb = _keep(h, store)
    q = (_keep(hb @ w["q"].T, store) + w["q.b"]).view(n, H, dim)
    k = _keep(_keep(hb @ w["k"].T, store) + w["k.b"], store).view(n, G, dim)
    v = _keep(_keep(hb @ w["v"].T, store) + w["v.b"], store).view(n, G, vdim)
    temp = torch.tensor([query_temperature(p, m["q_temp"]["coef"], m["q_temp"]["every"]) for p in range(n)], dtype=h.dtype)
    q = _keep(q * temp[:, None, None], store)
    by_distance = torch.stack([w["rel"][bucket(i, w["rel"].shape[0], m["bias_max"])] for i in range(n)])    # [n, H]
    out = torch.zeros(n, H, vdim, dtype=h.dtype)
    for i in range(n):
        for head in range(H):
            g = head // (H // G)
            s = (k[:i + 1, g] @ q[i, head]) * m["scale"] + by_distance[:i + 1, head].flip(0)
            out[i, head] = torch.softmax(s, dim=0) @ v[:i + 1, g]
    return out.view(n, H * vdim) * torch.sigmoid(_keep(hb @ w["g"].T, store))


# ----------------------------------------------------------------------------------------------
# right: the delta rule with a decay, a removal rate and a key of its own
# ----------------------------------------------------------------------------------------------
def right_decay(h, w) -> torch.Tensor:
    return torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ w["w1"].T) @ w["w2"].T + w["w0"]))


def right_recurrence(r, w, k, v, a) -> torch.Tensor:
    """All [n, H, dim].  u = k / |k|;  S_t = diag(w) S - (a u)(u^T S) + k v^T with S the old state;  o_t = S_t^T r."""
    n, H, dim = r.shape
    S = torch.zeros(H, dim, dim, dtype=r.dtype)
    out = torch.zeros(n, H, dim, dtype=r.dtype)
    for t in range(n):
        u = k[t] / torch.sqrt((k[t] ** 2).sum(-1, keepdim=True) + UNIT_EPS)
        seen = (u[:, :, None] * S).sum(1)                                            # u^T S, per value channel
        S = w[t][:, :, None] * S - (a[t] * u)[:, :, None] * seen[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * r[t][:, :, None]).sum(1)
    return out


def right_mixer(h, w, m, eps, store=None) -> torch.Tensor:
    """The gated heads [n, heads * dim], before the output projection."""
    n = h.shape[0]
    H, dim = m["heads"], m["dim"]
    hb = _keep(h, store)
    r, k, v = (_keep(hb @ w[c].T, store).view(n, H, dim) for c in "rkv")
    a = torch.sigmoid(hb @ w["a"].T + w["a.b"]).view(n, H, dim)
    o = right_recurrence(r, right_decay(hb, w).view(n, H, dim), k, v, a)
    return rms(o, eps).reshape(n, H * dim) * w["norm"] * torch.sigmoid(_keep(hb @ w["g"].T, store))


def parallel_mixer(h, w, m, eps, store=None) -> torch.Tensor:
    left, right = sub(w, "left."), sub(w, "right.")
    a = _keep(m["left_scale"] * left_mixer(h, left, m["left"], store), store)
    b = _keep(m["right_scale"] * right_mixer(h, right, m["right"], eps, store), store)
    return _keep(a @ left["o"].T + m["left_scale"] * left["o.b"] + b @ right["o"].T, store)


# ----------------------------------------------------------------------------------------------
# the model
# ----------------------------------------------------------------------------------------------
def dense_ff(h, w, store=None) -> torch.Tensor:
    hb = _keep(h, store)
    return _keep(_keep(gelu_tanh(hb @ w["gate"].T) * (hb @ w["up"].T), store) @ w["down"].T, store)


def forward(cfg, tensors, tokens: Sequence[int], store=None, layers_out: Optional[List] = None) -> torch.Tensor:
    """Logits [n, vocab] of every position."""
    eps = cfg["norm"]["eps"]
    x = tanh_norm(tensors["embed"][list(tokens)] + tensors["pos"][:len(tokens)], tensors, "embed.norm")
    history = [x]
    for i, layer in enumerate(cfg["layers"]):
        w = sub(tensors, f"l{i}.")
        h = tanh_norm(x, w, "norm1")
        mix = gla_mixer if layer["type"] == "gla" else parallel_mixer
        x = x + mix(h, sub(w, "mix."), layer["mixer"], eps, store) * residual_gate(h, w, "rg1", store)
        if layer["mlp"] is not None:
            h = tanh_norm(x, w, "norm2")
            x = x + dense_ff(h, sub(w, "mlp."), store) * residual_gate(h, w, "rg2", store)
        history.append(x)
        x = depth_average(history, w["dwa"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return _keep(tanh_norm(x, tensors, "final.norm"), store) @ tensors["head"].T * cfg["logit_scale"]
