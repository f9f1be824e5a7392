"""Oracle for the Doderax decoder: one plain function per mechanism, float64, no cache and no batching -- a whole sequence goes
in, every position comes out. TEST INFRASTRUCTURE ONLY (see oracle/__init__.py). No reference code defines this model; the
functions restate its equations:

    norm       y = x / sqrt(mean(x^2) + eps), times 1 + w on the stream, times w elsewhere
    embedding  x_t = E[n_t] + P[(a n_{t-1} + b n_t) mod B], P[B] for the first token
    rotation   (u, v) -> (u cos f_i t - v sin f_i t, v cos f_i t + u sin f_i t), dims i and i + m/2, f_i = base^(-2 i / m)
    attention  y_i = sum_j softmax_j(c <q_i, k_j>) v_j over j <= i with i - j < n or j < n0
    delta      S' = diag(g_t) S, u = b_t (v_t - S'^T k_t), S = S' + k_t u^T, y_t = S^T q_t; q, k, v through a causal
               convolution and silu, q and k of unit length, q also / sqrt(dk); log g = -exp(A) softplus(.)
    layer      x += mixer(h) + W_d gelu(W_u h), h = norm(x) (1 + w)
    head       c W norm(x) (1 + w)
"""
from __future__ import annotations

import math

import torch

from .vozozen import silu, to_f64

UNIT_EPS = 1e-6


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def pair_rows(tokens, pairs) -> list[int]:
    """Row of the pair table for every token of a sequence."""
    rows = [pairs["buckets"]]
    for before, now in zip(tokens, tokens[1:]):
        rows.append((before * pairs["mul_prev"] + now * pairs["mul_cur"]) % pairs["buckets"])
    return rows


def rotate(x, dims, base, first=0):
    """x [T, H, d] at positions first, first + 1, ..: its first `dims` dims turned."""
    out = x.clone()
    half = dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            angle = (first + t) * base ** (-2.0 * i / dims)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * math.cos(angle) - v * math.sin(angle)
            out[t, :, i + half] = v * math.cos(angle) + u * math.sin(angle)
    return out


def sink_attention(q, k, v, scale, window, keep_first):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; query head h reads key head h // (H / G)."""
    T, H = q.shape[:2]
    share = H // k.shape[1]
    out = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        seen = [j for j in range(i + 1) if i - j < window or j < keep_first]
        for h in range(H):
            scores = k[seen, h // share] @ q[i, h] * scale
            out[i, h] = torch.softmax(scores, dim=0) @ v[seen, h // share]
    return out


def short_conv(x, w):
    """x [T, C], w [C, n]: y_t = sum_b w[:, n - 1 - b] x_{t-b}, zeros before the start, then silu"""
    T, n = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for b in range(min(n, t + 1)):
            out[t] += w[:, n - 1 - b] * x[t - b]
    return silu(out)


def unit(x):
    return x / torch.sqrt(x.pow(2).sum(dim=-1, keepdim=True) + UNIT_EPS)


def decay_log(a_log, x):
    """log g = -exp(A) log(1 + exp(x))"""
    return -torch.exp(a_log) * torch.nn.functional.softplus(x)


def delta_rule(q, k, v, log_decay, beta, state=None):
    """q, k, log_decay [T, H, dk], v [T, H, dv], beta [T, H] -> outputs [T, H, dv] and the final state [H, dk, dv]"""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = torch.exp(log_decay[t]).unsqueeze(2) * S
        u = beta[t].unsqueeze(1) * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + torch.einsum("hd,hv->hdv", k[t], u)
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def attention_mixer(h, w, cfg):
    T, rot = h.shape[0], cfg.get("rot")
    q, k = (h @ w["q"].T).view(T, cfg["heads"], cfg["dim"]), (h @ w["k"].T).view(T, cfg["kv_heads"], cfg["dim"])
    v = (h @ w["v"].T).view(T, cfg["kv_heads"], cfg["vdim"])
    if rot:
        q, k = rotate(q, rot["dims"], rot["base"]), rotate(k, rot["dims"], rot["base"])
    y = sink_attention(q, k, v, cfg["scale"], cfg["mask"]["size"], cfg["mask"]["keep_first"])
    return y.reshape(T, -1) @ w["o"].T


def delta_mixer(h, w, cfg, eps):
    """One decay per head where the weights have `a`, one per key channel where they have `a1`."""
    T, H, G, d = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"]
    q = unit(short_conv(h @ w["q"].T, w["q.conv"]).view(T, G, d)).repeat_interleave(H // G, 1) / d ** 0.5
    k = unit(short_conv(h @ w["k"].T, w["k.conv"]).view(T, G, d)).repeat_interleave(H // G, 1)
    v = short_conv(h @ w["v"].T, w["v.conv"]).view(T, H, cfg["vdim"])
    beta = torch.sigmoid(h @ w["b"].T)
    if "a" in w:
        log = decay_log(w["A_log"], h @ w["a"].T + w["dt_bias"]).unsqueeze(2).expand(T, H, d)
        gate = silu(h @ w["g"].T)
    else:
        log = decay_log(w["A_log"].unsqueeze(1), (h @ w["a1"].T @ w["a2"].T + w["dt_bias"]).view(T, H, d))
        gate = torch.sigmoid(h @ w["g1"].T @ w["g2"].T)
    y, _ = delta_rule(q, k, v, log, beta)
    return ((rms(y, eps) * w["norm"]).reshape(T, -1) * gate) @ w["o"].T


def forward(cfg, weights, tokens):
    """-> logits [T, vocab] and the stream after every layer [layers, T, width]."""
    w = {name: to_f64(value) for name, value in weights.items()}
    eps, tokens = cfg["norm"]["eps"], [int(t) for t in tokens]
    x = w["embed"][torch.tensor(tokens)]
    if cfg["embedding"].get("bigram"):
        x = x + w["bigram"][torch.tensor(pair_rows(tokens, cfg["embedding"]["bigram"]))]
    streams = []
    for i, entry in enumerate(cfg["layers"]):
        sub = lambda prefix: {n[len(prefix):]: t for n, t in w.items() if n.startswith(prefix)}  # noqa: E731
        h, m = rms(x, eps) * (1 + w[f"l{i}.norm1"]), entry["mixer"]
        if entry["type"] == "parallel":
            left, right = sub(f"l{i}.mix.left."), sub(f"l{i}.mix.right.")
            y = (rms(attention_mixer(h, left, m["left"]), eps) * left["out"] + rms(delta_mixer(h, right, m["right"], eps), eps) * right["out"]) / 2
        else:
            y = delta_mixer(h, sub(f"l{i}.mix."), m, eps)
        if entry.get("mlp"):
            y = y + gelu(h @ w[f"l{i}.mlp.up"].T) @ w[f"l{i}.mlp.down"].T
        x = x + y
        streams.append(x.clone())
    return cfg["logit_scale"] * (rms(x, eps) * (1 + w["final.norm"])) @ w["head"].T, torch.stack(streams)


def greedy(cfg, weights, prompt, n_new):
    """-> generated tokens and, per token, how far its logit is ahead of the runner-up."""
    seq, margins = list(prompt), []
    for _ in range(n_new):
        top = forward(cfg, weights, seq)[0][-1].topk(2)
        seq.append(int(top.indices[0]))
        margins.append(float(top.values[0] - top.values[1]))
    return seq[len(prompt):], margins
