"""Oracle for the Lilovik decoder: one plain function per mechanism, float64, no cache and no batching -- a whole sequence goes
in, every position comes out. TEST INFRASTRUCTURE ONLY (see oracle/__init__.py). No reference code defines this model; the
functions restate its equations:

    norm       y = x / sqrt(mean(x^2) + eps), times 1 + w on the stream, times w on a query or key projection
    embedding  x_t = E[n_t] + s_t,  s_t[2i] = sin(t f_i), s_t[2i+1] = cos(t f_i), f_i = 10000^(-2 i / width)
    attention  a_hij = sigmoid(c tanh(k <q_hi, k_j> / c) - m_h (i - j) + b_h),  m_h = 2^(-8 (h + 1) / H),
               y_hi = sum_{j <= i} (sum_g T_hg a_gij) v_j;  q times 1 + u log(floor((i + 1) / n) + 1)
    minGRU     S_t = (1 - z_t) S_{t-1} + z_t g(u_t),  g(u) = u + 1/2 for u >= 0, else sigmoid(u);  y_t = S_t silu(o_t)
    layer      x += norm(mixer(norm(x))),  x += norm(W_d (relu(W_g h) * W_u h)), h = norm(x)
    head       c W norm(x)
"""
from __future__ import annotations

import math

import torch

from .vozozen import to_f64


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def position_vectors(positions, width):
    out = torch.zeros(len(positions), width, dtype=torch.float64)
    for r, t in enumerate(positions):
        for c in range(width):
            angle = t * 10000.0 ** (-2.0 * (c // 2) / width)
            out[r, c] = math.sin(angle) if c % 2 == 0 else math.cos(angle)
    return out


def query_factors(positions, temp):
    """Factor on the query at each position; temp None: 1."""
    if not temp:
        return torch.ones(len(positions), dtype=torch.float64)
    return torch.tensor([1 + temp["coef"] * math.log(math.floor((t + 1) / temp["every"]) + 1) for t in positions], dtype=torch.float64)


def slopes(heads):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float64)


def gates(q, k, scale, softcap, bias, first=0):
    """q [N, H, d] at positions first, first + 1, .., k [T, G, d] at 0, 1, .. -> weights [H, N, T], zero where a key is unseen."""
    N, H = q.shape[:2]
    T, share, m = k.shape[0], H // k.shape[1], slopes(H)
    out = torch.zeros(H, N, T, dtype=torch.float64)
    for h in range(H):
        s = q[:, h] @ k[:, h // share].T * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        ago = torch.arange(first, first + N).unsqueeze(1) - torch.arange(T).unsqueeze(0)
        s = s - m[h] * ago + bias[h]
        out[h] = torch.where(ago >= 0, torch.sigmoid(s), torch.zeros_like(s))
    return out


def mix_heads(weights, talk):
    """weights [H, N, T], talk [H, H]: w'_h = sum_g talk[h, g] w_g"""
    out = torch.zeros_like(weights)
    for h in range(weights.shape[0]):
        for g in range(weights.shape[0]):
            out[h] += talk[h, g] * weights[g]
    return out


def weigh_values(weights, v):
    """weights [H, N, T], v [T, G, dv] -> [N, H, dv]"""
    share = weights.shape[0] // v.shape[1]
    return torch.stack([weights[h] @ v[:, h // share] for h in range(weights.shape[0])], dim=1)


def mixed_gate_attention(q, k, v, scale, softcap, bias, talk, first=0):
    return weigh_values(mix_heads(gates(q, k, scale, softcap, bias, first), talk), v)


def silu(x):
    return x * torch.sigmoid(x)


def min_gru(z, u, o, state=None):
    """z, u, o [T, width], biases added already -> outputs [T, width] and the final state"""
    S = torch.zeros(z.shape[1], dtype=torch.float64) if state is None else state.clone()
    out = torch.empty_like(z)
    for t in range(z.shape[0]):
        keep = 1 - torch.sigmoid(z[t])
        candidate = torch.where(u[t] >= 0, u[t] + 0.5, torch.sigmoid(u[t]))
        S = keep * S + (1 - keep) * candidate
        out[t] = S * silu(o[t])
    return out, S


def attention_mixer(h, w, cfg, eps):
    T, H, G = h.shape[0], cfg["heads"], cfg["kv_heads"]
    q, k, v = (h @ w[n].T + w[n + ".b"] for n in "qkv")
    q, k = rms(q, eps) * w["q.norm"], rms(k, eps) * w["k.norm"]
    q = q * query_factors(range(T), cfg.get("q_temp")).unsqueeze(1)
    y = mixed_gate_attention(q.view(T, H, cfg["dim"]), k.view(T, G, cfg["dim"]), v.view(T, G, cfg["vdim"]), cfg["scale"],
                             cfg.get("softcap"), w["pb"], w["talk"])
    return y.reshape(T, -1) @ w["o"].T


def min_gru_mixer(h, w):
    y, _ = min_gru(h @ w["z"].T + w["z.b"], h @ w["x"].T + w["x.b"], h @ w["g"].T)
    return y @ w["o"].T


def feed_forward(h, w):
    return (torch.clamp(h @ w["gate"].T, min=0) * (h @ w["up"].T)) @ w["down"].T


def forward(cfg, weights, tokens):
    """-> logits [T, vocab] and the stream after every layer [layers, T, width]."""
    w = {name: to_f64(value) for name, value in weights.items()}
    eps, tokens = cfg["norm"]["eps"], [int(t) for t in tokens]
    x = w["embed"][torch.tensor(tokens)] + position_vectors(range(len(tokens)), cfg["width"])
    streams = []
    for i, entry in enumerate(cfg["layers"]):
        sub = lambda prefix: {n[len(prefix):]: t for n, t in w.items() if n.startswith(prefix)}  # noqa: E731
        normed = lambda y, name: rms(y, eps) * (1 + w[f"l{i}.{name}"])  # noqa: E731
        h, mix = normed(x, "norm1"), sub(f"l{i}.mix.")
        y = attention_mixer(h, mix, entry["mixer"], eps) if entry["type"] == "attention" else min_gru_mixer(h, mix)
        x = x + normed(y, "norm1b")
        if entry.get("mlp"):
            x = x + normed(feed_forward(normed(x, "norm2"), sub(f"l{i}.mlp.")), "norm2b")
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
