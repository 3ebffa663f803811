"""Plain, slow Retudra: whole sequences, dense masks, explicit loops over
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
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, base, dims):
    """x [T, heads, d] at positions 0 .. T - 1: of the first ``dims`` elements, i turns with i + dims / 2."""
    n = dims // 2
    if n == 0:
        return x
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(n)], dtype=F64)
    ang = torch.arange(x.shape[0], dtype=F64)[:, None, None] * f
    c, s = ang.cos(), ang.sin()
    u, v = x[..., :n], x[..., n:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


# ---------------------------------------------------------------- attention

def visible(T, size, keep_first):
    """[T, T]: may position i (row) see position j (column)?  ``size`` None: every earlier one."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = torch.ones(T, T, dtype=torch.bool) if size is None else ((i - j < size) | (j < keep_first))
    return (j <= i) & near


def attend(q, k, v, scale, mask):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H dv]; query head h reads key/value head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    outs = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = s.masked_fill(~mask, float("-inf"))
        outs.append(torch.softmax(s, dim=-1) @ v[:, g])
    return torch.cat(outs, dim=1)


def attention_mixer(h, W, p, m, eps):
    H, G, d, dv, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    rot, mask = m["rot"], m.get("mask") or {}
    q = rms(h @ W[p + "q"].T, eps, W[p + "q.norm"]).view(T, H, d)
    k = rms(h @ W[p + "k"].T, eps, W[p + "k.norm"]).view(T, G, d)
    v = (h @ W[p + "v"].T).view(T, G, dv)
    q, k = rotate(q, rot["base"], rot["dims"]), rotate(k, rot["base"], rot["dims"])
    return attend(q, k, v, float(m["scale"]), visible(T, mask.get("size"), mask.get("keep_first") or 0)) @ W[p + "o"].T


def latent_mixer(h, W, p, m, eps):
    H, d, r, dv, rank, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], h.shape[0]
    q = (h @ W[p + "q"].T).view(T, H, d + r)
    down = h @ W[p + "dkv"].T
    c = rms(down[:, :rank], eps, W[p + "dkv.norm"])
    shared = rotate(down[:, None, rank:], m["rot"]["base"], r)
    q = torch.cat([q[..., :d], rotate(q[..., d:], m["rot"]["base"], r)], dim=-1)
    k = torch.cat([(c @ W[p + "uk"].T).view(T, H, d), shared.expand(T, H, r)], dim=-1)
    v = (c @ W[p + "uv"].T).view(T, H, dv)
    o = attend(q, k, v, float(m["scale"]), visible(T, None, 0))
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ---------------------------------------------------------------- the delta rule with a decay per channel

def short_conv(x, w):
    """x [T, C], w [C, taps]: y_t = sum_j w[:, j] x_(t - taps + 1 + j), zeros before the first token."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[j:j + x.shape[0]] * w[:, j] for j in range(taps))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_scan(q, k, v, g, beta):
    """One head: S <- diag(g) S, then S <- S + beta k (v - S^T k)^T, o = S^T q; S starts at zero."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(k.shape[0]):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + k[t][:, None] * u[None, :]
        out.append(S.T @ q[t])
    return torch.stack(out)


def channel_decay(h, W, p, heads, dim):
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]
    return torch.exp(-torch.exp(W[p + "A_log"])[None, :, None] * softplus(z).view(-1, heads, dim))


def delta_mixer(h, W, p, m, eps):
    H, G, d, dv, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]

    def conved(name):
        return silu(short_conv(h @ W[p + name].T, W[p + name + ".conv"]))

    q, k = unit(conved("q").view(T, G, d)) * d ** -0.5, unit(conved("k").view(T, G, d))
    v = conved("v").view(T, H, dv)
    beta = sigmoid(h @ W[p + "b"].T)
    g = channel_decay(h, W, p, H, d)
    gate = sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T)
    outs = []
    for i in range(H):
        o = delta_scan(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], g[:, i], beta[:, i])
        outs.append(rms(o, eps, W[p + "norm"]))
    return (torch.cat(outs, dim=1) * gate) @ W[p + "o"].T


# ---------------------------------------------------------------- feed-forward

def glu(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def choose(scores, correction, top, count, keep):
    """The experts a token uses: a list of indices."""
    c = scores + correction
    n, per = c.numel(), c.numel() // count
    best = torch.stack([c[g * per:(g + 1) * per].max() for g in range(count)]).topk(keep).indices.tolist()
    allowed = [e for e in range(n) if e // per in best]
    return sorted(allowed, key=lambda e: -float(c[e]))[:top]


def experts(h, W, p, mlp):
    ro = mlp["router"]
    groups = ro.get("groups") or {"count": 1, "keep": 1}
    s = torch.softmax(h @ W[p + "router"].T, dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose(s[t], W[p + "correction"], ro["top"], groups["count"], groups["keep"]):
            y = glu(h[t], W, f"{p}e{e}.") if e < ro["experts"] else h[t]
            out[t] += s[t, e] * y
    return out


def feed_forward(h, W, p, mlp):
    return glu(h, W, p) if mlp["kind"] == "dense" else experts(h, W, p, mlp)


def token_side(x, tokens, W, p, i, dim):
    e = W["side.embed"][torch.tensor(tokens, dtype=torch.long), i * dim:(i + 1) * dim]
    return (gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T


# ---------------------------------------------------------------- the model

MIXERS = {"attention": attention_mixer, "latent_attention": latent_mixer, "channel_delta": delta_mixer}


def forward(cfg, W, tokens, layers_out=None, round_h=None):
    """Logits [T, vocab] of one sequence.  ``layers_out`` (a list) receives the residual stream after every layer.
    ``round_h``: a function applied to every sublayer's input (to model a 16-bit product input)."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    rh = round_h or (lambda z: z)
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](rh(x), W, p + "mix.", layer["mixer"], eps)
        x = x + m * layer_norm(y, W[p + "norm1"], W[p + "norm1.b"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(rh(x), W, p + "mlp.", layer["mlp"])
            x = x + m * layer_norm(y, W[p + "norm2"], W[p + "norm2.b"], eps)
        if cfg.get("token_side"):
            y = token_side(rh(x), tokens, W, p, i, cfg["token_side"]["dim"])
            x = x + m * rms(y, eps, W[p + "side.norm"])
        if layers_out is not None:
            layers_out.append(x)
    z = rh(layer_norm(x, W["final.norm"], W["final.norm.b"], eps)) @ W["head"].T
    cap = cfg.get("logit_softcap")
    return z if not cap else cap * torch.tanh(z / cap)


def logits(cfg, W, tokens):
    return forward(cfg, W, tokens)


def generate_greedy(cfg, W, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(forward(cfg, W, ids)[-1].argmax()))
    return ids[len(prompt):]
