"""Plain, slow Teselix: whole sequences, dense masks, explicit loops over
tokens, no cache, float64, one function for each mechanism.  It shares no code
with ``airframe_b200`` (its own reading of config.json and of the tensors).

Notation: x is the residual stream [T, width], h a sublayer's input; W x means a
weight stored [out, in] applied to a vector; positions count from 0.
"""
from __future__ import annotations

import json
import math
from pathlib import Path

import torch

from plain_gemma2 import read_safetensors

F64 = torch.float64


def read_model_folder(folder, dtype=F64):
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    return cfg, read_safetensors(folder / "model.safetensors", dtype)


# ---------------------------------------------------------------- small pieces

def rms(x, eps, w=None):
    """x / sqrt(mean(x^2) + eps) over the last axis, times w when given."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def layer_norm(x, w, b, eps):
    """Centred and divided by the standard deviation (the mean of squared deviations plus eps, under the root)."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def shifted(h, mu):
    """h_t + (h_(t-1) - h_t) * mu per channel, with zeros before the first token."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def residual_gate(h, W, b):
    """sigmoid(W h + b), one factor per channel of a sublayer's result."""
    return sigmoid(h @ W.T + b)


def norm_of_sum(x, y, alpha, w, b, eps):
    """The layer norm behind the residual sum alpha x + y."""
    return layer_norm(alpha * x + y, w, b, eps)


# ---------------------------------------------------------------- rotation

def frequencies(rot):
    """(f_i for i < dims / 2, factor on cosines and sines) of a rotation {base, dims, scaling?}."""
    base, dims, sc = float(rot["base"]), int(rot["dims"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return torch.tensor(f, dtype=F64), 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def where(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(where(float(sc["fast"]))), 0)
    hi = min(math.ceil(where(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(factor) + 1.0


def rotate_half_split(x, freqs, mag):
    """x [T, heads, d] at positions 0 .. T - 1: element i pairs with element i + n (n frequencies)."""
    n = freqs.numel()
    ang = torch.arange(x.shape[0], dtype=F64)[:, None, None] * freqs
    c, s = ang.cos() * mag, ang.sin() * mag
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def rotate_neighbours(x, freqs, mag):
    """As above, element 2i pairs with element 2i + 1."""
    n = freqs.numel()
    ang = torch.arange(x.shape[0], dtype=F64)[:, None, None] * freqs
    c, s = ang.cos() * mag, ang.sin() * mag
    y = x.clone()
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    y[..., 0:2 * n:2] = u * c - v * s
    y[..., 1:2 * n:2] = v * c + u * s
    return y


# ---------------------------------------------------------------- retention

def decayed_scan(q, k, v, decay):
    """One head: S_t = decay S_(t-1) + k_t v_t^T from S = 0, o_t = S_t^T q_t."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(k.shape[0]):
        S = decay * S + k[t][:, None] * v[t][None, :]
        out.append(S.T @ q[t])
    return torch.stack(out)


def retention_mixer(h, W, p, m, eps):
    H, dk, dv, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    freqs, mag = frequencies(m["rot"])
    q = rotate_half_split((h @ W[p + "q"].T).view(T, H, dk), freqs, mag)
    k = rotate_half_split((h @ W[p + "k"].T).view(T, H, dk), freqs, mag) * dk ** -0.5
    v = (h @ W[p + "v"].T).view(T, H, dv)
    o = torch.cat([rms(decayed_scan(q[:, i], k[:, i], v[:, i], float(m["decay"][i])), eps) for i in range(H)], dim=1)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ---------------------------------------------------------------- latent attention

def sink_softmax(scores, sink):
    """Causal softmax over keys j <= i of [T, T] scores; exp(sink) joins the denominator."""
    T = scores.shape[0]
    s = scores.masked_fill(~torch.ones(T, T, dtype=torch.bool).tril(), float("-inf"))
    top = torch.maximum(s.max(-1, keepdim=True).values, torch.as_tensor(sink, dtype=s.dtype))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def latent_mixer(h, W, p, m, eps):
    H, d, r, dv, rank, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], h.shape[0]
    freqs, mag = frequencies(m["rot"])
    cq = rms(h @ W[p + "dq"].T, eps, W[p + "dq.norm"])
    q = (cq @ W[p + "uq"].T).view(T, H, d + r)
    q_rot = rotate_neighbours(q[..., d:], freqs, mag)
    down = h @ W[p + "dkv"].T
    c = rms(down[:, :rank], eps, W[p + "dkv.norm"])
    k_rot = rotate_neighbours(down[:, None, rank:], freqs, mag)[:, 0]
    k = (c @ W[p + "uk"].T).view(T, H, d)
    v = (c @ W[p + "uv"].T).view(T, H, dv)
    gate = sigmoid(h @ W[p + "g"].T)
    outs = []
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * float(m["scale"])
        outs.append((sink_softmax(s, W[p + "sink"][i]) @ v[:, i]) * gate[:, i:i + 1])
    return torch.cat(outs, dim=1) @ W[p + "o"].T


# ---------------------------------------------------------------- experts chosen by the token

def clamped_expert(h, W, p, limit):
    g = torch.clamp(h @ W[p + ".gate"].T, max=limit)
    u = torch.clamp(h @ W[p + ".up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + ".down"].T


def table_experts(h, tokens, W, p, mlp):
    top, limit = mlp["router"]["top"], float(mlp["expert"]["limit"])
    out = torch.zeros_like(h)
    for t, token in enumerate(tokens):
        for e in W[p + "table"][token].tolist():
            out[t] += clamped_expert(h[t], W, f"{p}e{int(e)}", limit) / top
    if mlp.get("shared"):
        out = out + clamped_expert(h, W, p + "shared", float(mlp["shared"]["limit"]))
    return out


# ---------------------------------------------------------------- the model

def owner(layers, i):
    """The layer whose tensors layer i uses."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(cfg, W, tokens, layers_out=None, round_h=None):
    """Logits [T, vocab] of one sequence.  ``layers_out`` (a list) receives the residual stream after every layer.
    ``round_h``: a function applied to every sublayer's input (to model a 16-bit product input)."""
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    rh = round_h or (lambda z: z)
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg['layers'], i)}."
        mixer = retention_mixer if layer["type"] == "retention" else latent_mixer
        y = mixer(rh(shifted(x, W[p + "shift"])), W, p + "mix.", layer["mixer"], eps)
        y = y * residual_gate(rh(x), W[p + "rg1"], W[p + "rg1.b"])
        x = norm_of_sum(x, y, alpha, W[p + "norm1"], W[p + "norm1.b"], eps)
        if layer.get("mlp") is not None:
            y = table_experts(rh(x), tokens, W, p + "mlp.", layer["mlp"])
            y = y * residual_gate(rh(x), W[p + "rg2"], W[p + "rg2.b"])
            x = norm_of_sum(x, y, alpha, W[p + "norm2"], W[p + "norm2.b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return rh(layer_norm(x, W["final.norm"], W["final.norm.b"], eps)) @ W["embed"].T


def logits(cfg, W, tokens):
    return forward(cfg, W, tokens)


def generate_greedy(cfg, W, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(forward(cfg, W, ids)[-1].argmax()))
    return ids[len(prompt):]
