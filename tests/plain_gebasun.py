"""Plain, slow implementation of the Gebasun decoder, for tests only.

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


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def relu_squared(z):
    return torch.clamp(z, min=0) ** 2


def rotate_halves(x, dims, base):
    """x [T, ..., n >= dims]: dims (i, i + dims/2) of every vector turn by position * base^(-2i/dims); the rest pass."""
    T, half = x.shape[0], dims // 2
    freqs = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    angle = torch.arange(T, dtype=F)[:, None] * freqs[None, :]
    shape = (T,) + (1,) * (x.dim() - 2) + (half,)
    c, s = torch.cos(angle).reshape(shape), torch.sin(angle).reshape(shape)
    u, v = x[..., :half], x[..., half:dims]
    out = x.clone()
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


# --------------------------------------------------------------------------
# Attention
# --------------------------------------------------------------------------

def distance_bucket(n, rows, far):
    """The row of the bias table for a key n positions back: the first half of the rows one distance each, the others on a
    logarithmic scale that ends at distance ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def window_mask(T, size, keep_first=0):
    """visible[i, j]: j <= i, and i - j < size or j < keep_first."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = torch.ones((T, T), dtype=torch.bool) if size is None else (i - j < size) | (j < keep_first)
    return (j <= i) & seen


def attend(q, k, v, scale, visible, sink, bias=None):
    """One head: q, k [T, D], v [T, Dv]; ``bias`` [T, T] is added to the scaled scores, exp(sink) to the sum of weights."""
    s = (q @ k.T) * scale
    if bias is not None:
        s = s + bias
    s = s.masked_fill(~visible, -math.inf)
    m = torch.maximum(s.max(dim=1, keepdim=True).values, torch.as_tensor(sink, dtype=F))
    e = torch.exp(s - m)
    return (e @ v) / (e.sum(dim=1, keepdim=True) + torch.exp(sink - m))


def attention(w, p, m, h, eps, rotated):
    """Both attention mixers.  Keys are projected once: as they are they serve as values; rotated (``rotated``) and
    divided by their root mean square as keys."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[p + "mix.q"].T + w[p + "mix.q.b"]).reshape(T, H, D)
    k = (h @ w[p + "mix.k"].T + w[p + "mix.k.b"]).reshape(T, G, D)
    v = k
    if rotated:
        q, k = (rotate_halves(z, m["rot"]["dims"], m["rot"]["base"]) for z in (q, k))
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    mask = m.get("mask") or {}
    visible = window_mask(T, mask.get("size"), mask.get("keep_first", 0))
    row = None
    if not rotated:
        table = w[p + "mix.rel"]
        back = [distance_bucket(n, table.shape[0], m["bias_max"]) for n in range(T)]
        row = torch.tensor([[back[max(i - j, 0)] for j in range(T)] for i in range(T)])
    heads = []
    for head in range(H):
        g = head // (H // G)
        bias = None if row is None else table[:, head][row]
        heads.append(attend(q[:, head], k[:, g], v[:, g], m["scale"], visible, w[p + "mix.sink"][head], bias))
    o = torch.cat(heads, dim=1)
    if rotated:
        return (o * torch.sigmoid(h @ w[p + "mix.g"].T)) @ w[p + "mix.o"].T
    return o @ w[p + "mix.o"].T + w[p + "mix.o.b"]


# --------------------------------------------------------------------------
# Mamba-2
# --------------------------------------------------------------------------

def causal_conv(u, taps_w, bias):
    """u [T, C], taps_w [C, n]: out_t = bias + sum_j taps_w[:, j] * u_(t - n + 1 + j), zeros before position 0."""
    T, n = u.shape[0], taps_w.shape[1]
    padded = torch.cat([torch.zeros((n - 1, u.shape[1]), dtype=u.dtype), u], dim=0)
    out = torch.zeros_like(u) + bias
    for j in range(n):
        out = out + padded[j : j + T] * taps_w[:, j]
    return out


def state_space(x, B, C, dt, A_log, D_skip, state=None):
    """One head, token by token.  x [T, P], B, C [T, N], dt [T] (after softplus): S <- exp(-exp(A_log) dt) S + dt B x^T,
    y = S^T C + D x.  Returns (y, the last S [N, P])."""
    S = torch.zeros((B.shape[1], x.shape[1]), dtype=x.dtype) if state is None else state
    ys = []
    for t in range(x.shape[0]):
        S = torch.exp(-torch.exp(A_log) * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        ys.append(S.T @ C[t] + D_skip * x[t])
    return torch.stack(ys), S


def gate_then_norm(y, z, weight, parts, eps):
    """y * silu(z), an RMS norm over each of ``parts`` equal runs of columns, times ``weight``."""
    g = y * silu(z)
    T, n = g.shape
    return unit_rms(g.reshape(T, parts, n // parts), eps).reshape(T, n) * weight


def mamba2(w, p, m, h, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    zxbcdt = h @ w[p + "mix.in"].T
    z, xbc, dt = zxbcdt[:, :inner], zxbcdt[:, inner : 2 * inner + 2 * G * N], zxbcdt[:, 2 * inner + 2 * G * N :]
    xbc = silu(causal_conv(xbc, w[p + "mix.conv"], w[p + "mix.conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner : inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N :].reshape(T, G, N)
    dt = softplus(dt + w[p + "mix.dt_bias"])
    ys = []
    for head in range(H):
        g = head // (H // G)
        y, _ = state_space(x[:, head], B[:, g], C[:, g], dt[:, head], w[p + "mix.A_log"][head], w[p + "mix.D"][head])
        ys.append(y)
    y = gate_then_norm(torch.cat(ys, dim=1), z, w[p + "mix.norm"], m["norm_groups"], eps)
    return y @ w[p + "mix.o"].T


# --------------------------------------------------------------------------
# Experts
# --------------------------------------------------------------------------

def route(z, top):
    """z [E]: (ids, weights) of the ``top`` largest logits; the weights are the softmax over those."""
    ids = sorted(range(z.shape[0]), key=lambda e: (-float(z[e]), e))[:top]
    chosen = z[ids]
    e = torch.exp(chosen - chosen.max())
    return ids, e / e.sum()


def expert(w, name, h):
    return relu_squared(h @ w[name + ".up"].T) @ w[name + ".down"].T


def experts(w, p, mlp, h):
    z = h @ w[p + "mlp.router"].T + w[p + "mlp.router.b"]
    out = torch.zeros_like(h)
    chosen = [route(z[t], mlp["router"]["top"]) for t in range(h.shape[0])]
    for e in range(mlp["router"]["experts"]):
        rows = [(t, float(wt[ids.index(e)])) for t, (ids, wt) in enumerate(chosen) if e in ids]
        if rows:
            at = torch.tensor([t for t, _ in rows])
            out[at] += torch.tensor([v for _, v in rows], dtype=F)[:, None] * expert(w, f"{p}mlp.e{e}", h[at])
    if mlp.get("shared"):
        out = out + expert(w, p + "mlp.shared", h)
    return out


# --------------------------------------------------------------------------
# The model
# --------------------------------------------------------------------------

def layer(w, p, spec, x, eps):
    """Both sublayers read the stream as it enters, each through its own norm; their results join it together."""
    h = rms_norm(x, w[p + "norm1"], eps)
    m, kind = spec["mixer"], spec["type"]
    out = mamba2(w, p, m, h, eps) if kind == "mamba2" else attention(w, p, m, h, eps, rotated=kind == "attention_2")
    if spec.get("mlp") is not None:
        out = out + experts(w, p, spec["mlp"], rms_norm(x, w[p + "norm2"], eps))
    return x + out


def forward(cfg, w, tokens, streams=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    for i, spec in enumerate(cfg["layers"]):
        x = layer(w, f"l{i}.", spec, x, eps)
        if streams is not None:
            streams.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
