"""Plain, slow implementation of the Soputar decoder, for tests only.

Written from the design's equations, one function per mechanism, whole
sequences at once, no cache, float64 on the CPU (so that it sits inside the
float32 rounding of any right implementation).  It shares no code with
``llmoxide_b200``: it has its own reader for the model folder and its own
handling of the configuration.

Notation: x [T, d] is the residual stream of one sequence, positions 0..T-1;
weights are stored [out, in] and applied as W x; ``w`` is the dict of tensors
and ``p`` a layer's prefix ("l3.").
"""

from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np
import torch

F = torch.float64
UNIT_EPS = 1e-6          # under the root of the delta rule's unit vectors
SWISH_SLOPE = 1.702


# --------------------------------------------------------------------------
# Model folder
# --------------------------------------------------------------------------

def read_safetensors(path) -> dict:
    raw = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8 : 8 + n])
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        buf = raw[8 + n + lo : 8 + n + hi]
        if info["dtype"] == "BF16":
            arr = (np.frombuffer(buf, dtype=np.uint16).astype(np.uint32) << 16).view(np.float32)
        else:
            arr = np.frombuffer(buf, dtype={"F32": np.float32, "F16": np.float16}[info["dtype"]])
        out[name] = torch.from_numpy(arr.reshape(info["shape"]).copy()).to(F)
    return out


def read_model(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


# --------------------------------------------------------------------------
# Small functions
# --------------------------------------------------------------------------

def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm_zero_centred(x, weight, eps):
    """The weight is stored as its distance from one."""
    return unit_rms(x, eps) * (1.0 + weight)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(u, taps_w):
    """u [T, C], taps_w [C, n]: out_t = sum_j taps_w[:, j] * u_(t - n + 1 + j), zeros before position 0."""
    T, n = u.shape[0], taps_w.shape[1]
    padded = torch.cat([torch.zeros((n - 1, u.shape[1]), dtype=u.dtype), u], dim=0)
    out = torch.zeros_like(u)
    for j in range(n):
        out = out + padded[j : j + T] * taps_w[:, j]
    return out


def unit_vectors(x):
    """x / sqrt(sum(x^2) + 1e-6) over the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def query_temperature(position, coef, every):
    return 1.0 + coef * math.log(math.floor((position + 1) / every) + 1.0)


def cap(score, c):
    return c * torch.tanh(score / c)


def rotate_neighbours(x, dims, base):
    """x [T, ..., n >= dims]: dims (2i, 2i+1) of every vector turn by position * base^(-2i/dims); the rest pass."""
    T = x.shape[0]
    freqs = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)
    angle = torch.arange(T, dtype=F)[:, None] * freqs[None, :]
    shape = (T,) + (1,) * (x.dim() - 2) + (dims // 2,)
    c, s = torch.cos(angle).reshape(shape), torch.sin(angle).reshape(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# --------------------------------------------------------------------------
# Softmax attention of one head
# --------------------------------------------------------------------------

def attend_causal(q, k, v, scale, softcap=None, sink=None):
    """q, k [T, D], v [T, Dv].  Every query sees the keys up to its own position; scores capped when ``softcap`` is
    given; exp(sink) in the denominator when ``sink`` is given (no value; neither scaled nor capped)."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    if softcap is not None:
        s = cap(s, softcap)
    s = s.masked_fill(torch.triu(torch.ones(T, T, dtype=torch.bool), diagonal=1), -math.inf)
    top = s.max(dim=1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    e = torch.exp(s - top)
    den = e.sum(dim=1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(float(sink) - top)
    return (e / den) @ v


def as_cached(t, cache_dtype):
    """A cached quantity as a cache of ``cache_dtype`` holds it (None: as computed)."""
    return t if cache_dtype is None else t.to(cache_dtype).to(F)


# --------------------------------------------------------------------------
# Mixers
# --------------------------------------------------------------------------

def attention_keys_values(h, w, p, m, eps, cache_dtype=None):
    T = h.shape[0]
    G, D, Dv = m["kv_heads"], m["dim"], m["vdim"]
    k = unit_rms(h @ w[p + "mix.k"].T, eps) * w[p + "mix.k.norm"]        # all rows at once, before the split
    v = h @ w[p + "mix.v"].T
    return as_cached(k.reshape(T, G, D), cache_dtype), as_cached(v.reshape(T, G, Dv), cache_dtype)


def attention_mixer(h, w, p, m, eps, kv):
    """``kv``: this layer's keys and values, or those of the layer it borrows from."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (unit_rms(h @ w[p + "mix.q"].T, eps) * w[p + "mix.q.norm"]).reshape(T, H, D)
    t = m.get("q_temp")
    if t:
        temp = torch.tensor([query_temperature(i, t["coef"], t["every"]) for i in range(T)], dtype=F)
        q = q * temp[:, None, None]
    k, v = kv
    out = torch.zeros((T, H, Dv), dtype=F)
    for hq in range(H):
        g = hq // (H // G)
        out[:, hq] = attend_causal(q[:, hq], k[:, g], v[:, g], m["scale"], softcap=m.get("softcap"))
    return out.reshape(T, H * Dv) @ w[p + "mix.o"].T


def latent_attention_mixer(h, w, p, m, eps, cache_dtype=None):
    T = h.shape[0]
    H, D, R, Dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "mix.q"].T).reshape(T, H, D + R)
    down = h @ w[p + "mix.dkv"].T
    c = as_cached(unit_rms(down[:, :rank], eps) * w[p + "mix.dkv.norm"], cache_dtype)
    base = float(m["rot"]["base"])
    k_rot = as_cached(rotate_neighbours(down[:, rank:], R, base), cache_dtype)      # one for all heads
    q = torch.cat([q[..., :D], rotate_neighbours(q[..., D:], R, base)], dim=-1)
    k_plain = (c @ w[p + "mix.uk"].T).reshape(T, H, D)
    v = (c @ w[p + "mix.uv"].T).reshape(T, H, Dv)
    out = torch.zeros((T, H, Dv), dtype=F)
    for hq in range(H):
        keys = torch.cat([k_plain[:, hq], k_rot], dim=-1)
        out[:, hq] = attend_causal(q[:, hq], keys, v[:, hq], m["scale"], sink=w[p + "mix.sink"][hq])
    return out.reshape(T, H * Dv) @ w[p + "mix.o"].T


def delta_rule(q, k, v, beta, g, state=None):
    """One head, token by token.  q, k [T, D], v [T, Dv], beta, g [T]; returns (o [T, Dv], the state left [D, Dv])."""
    S = torch.zeros((q.shape[1], v.shape[1]), dtype=F) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = S * g[t]
        u = beta[t] * (v[t] - k[t] @ S)
        S = S + torch.outer(k[t], u)
        out[t] = q[t] @ S
    return out, S


def delta_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    branch = lambda r: silu(causal_conv(h @ w[p + "mix." + r].T, w[p + "mix." + r + ".conv"]))
    q = unit_vectors(branch("q").reshape(T, G, D)) * D ** -0.5
    k = unit_vectors(branch("k").reshape(T, G, D))
    v = branch("v").reshape(T, H, Dv)
    beta = torch.sigmoid(h @ w[p + "mix.b"].T)
    g = torch.exp(-torch.exp(w[p + "mix.A_log"]) * softplus(h @ w[p + "mix.a"].T + w[p + "mix.dt_bias"]))
    gate = silu(h @ w[p + "mix.g"].T).reshape(T, H, Dv)
    out = torch.zeros((T, H, Dv), dtype=F)
    for hv in range(H):
        j = hv // (H // G)
        o, _ = delta_rule(q[:, j], k[:, j], v[:, hv], beta[:, hv], g[:, hv])
        out[:, hv] = unit_rms(o, eps) * w[p + "mix.norm"] * gate[:, hv]
    return out.reshape(T, H * Dv) @ w[p + "mix.o"].T


# --------------------------------------------------------------------------
# Feed-forward and model
# --------------------------------------------------------------------------

def clamped_mlp(h, w, p, limit):
    g = torch.clamp(h @ w[p + "mlp.gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "mlp.up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(SWISH_SLOPE * g) * (u + 1.0)) @ w[p + "mlp.down"].T


def forward(cfg, w, tokens, cache_dtype=None, streams=None):
    """Logits [T, vocab] of one sequence; ``streams``, a list, receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            kv = kept[m["kv_from"]] if m.get("kv_from") is not None else attention_keys_values(x, w, p, m, eps, cache_dtype)
            kept[i] = kv
            y = attention_mixer(x, w, p, m, eps, kv)
        elif layer["type"] == "latent_attention":
            y = latent_attention_mixer(x, w, p, m, eps, cache_dtype)
        elif layer["type"] == "delta":
            y = delta_mixer(x, w, p, m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + rms_norm_zero_centred(y, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            y = clamped_mlp(x, w, p, layer["mlp"]["limit"])
            x = x + rms_norm_zero_centred(y, w[p + "norm2"], eps)
        if streams is not None:
            streams.append(x.clone())
    return rms_norm_zero_centred(x, w["final.norm"], eps) @ w["head"].T
