"""Oracle for the Vozozen decoder: one plain function per mechanism, float64, no cache and no batching -- a whole sequence
goes in, every position comes out. TEST INFRASTRUCTURE ONLY (see oracle/__init__.py). No reference code defines this model;
the functions restate its equations:

    norm        y = w x / sqrt(mean(x^2) + eps)
    window      y_i = sum_j softmax_j(c <q_i, k_j>) v_j over 0 <= i - j < n, q and k normed per head, then y_h *= s(gate_h)
    linear      S_t = diag(a_t) S_{t-1} + k_t v_t^T, y_t = S_t^T q_t / sqrt(dk), a_t = s(z_t)^(1 / tau)
    layer       x += c_l window(norm x) + c_r linear(norm x);  x += W_d relu(W_u norm x)^2
    pass        x = W [x; x_0] in front of every pass over the looped layers
    head        c tanh(W norm x / c)
"""
from __future__ import annotations

import numpy as np
import torch

F64 = torch.float64


def to_f64(value) -> torch.Tensor:
    """A weight as the model gets it (numpy float32, numpy uint16 holding bfloat16, torch) in float64."""
    if isinstance(value, np.ndarray):
        if value.dtype == np.uint16:
            return torch.from_numpy(value.view(np.int16).copy()).view(torch.bfloat16).to(F64)
        return torch.from_numpy(np.ascontiguousarray(value)).to(F64)
    return value.to(F64)


def rms_norm(x, weight, eps):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps) * weight


def window_attention(q, k, v, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; query head h reads key head h // (H / G)."""
    T, H = q.shape[:2]
    share = H // k.shape[1]
    out = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        first = max(0, i - window + 1)
        for h in range(H):
            scores = k[first:i + 1, h // share] @ q[i, h] * scale
            out[i, h] = torch.softmax(scores, dim=0) @ v[first:i + 1, h // share]
    return out


def head_gates(z):
    return torch.sigmoid(z)


def key_decay(z, tau):
    """a = sigmoid(z)^(1 / tau)"""
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def gated_linear(q, k, v, decay, state=None):
    """q, k, decay [T, H, dk], v [T, H, dv] -> outputs [T, H, dv] and the final state [H, dk, dv]; q already scaled."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        for h in range(H):
            S[h] = decay[t, h].unsqueeze(1) * S[h] + torch.outer(k[t, h], v[t, h])
            out[t, h] = q[t, h] @ S[h]
    return out, S


def silu(x):
    return x * torch.sigmoid(x)


def left_mixer(h, w, cfg, eps):
    T = h.shape[0]
    q = rms_norm((h @ w["q"].T).view(T, cfg["heads"], cfg["dim"]), w["q.norm"], eps)
    k = rms_norm((h @ w["k"].T).view(T, cfg["kv_heads"], cfg["dim"]), w["k.norm"], eps)
    v = (h @ w["v"].T).view(T, cfg["kv_heads"], cfg["vdim"])
    y = window_attention(q, k, v, cfg["scale"], cfg["mask"]["size"]) * head_gates(h @ w["g"].T).unsqueeze(2)
    return y.reshape(T, -1) @ w["o"].T


def right_mixer(h, w, cfg, eps):
    T, H = h.shape[0], cfg["heads"]
    q = (h @ w["q"].T).view(T, H, cfg["dim"]) / cfg["dim"] ** 0.5
    k = (h @ w["k"].T).view(T, H, cfg["dim"])
    v = (h @ w["v"].T).view(T, H, cfg["vdim"])
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    y, _ = gated_linear(q, k, v, key_decay(z, cfg["tau"]).view(T, H, cfg["dim"]))
    return (rms_norm(y, w["norm"], eps).reshape(T, -1) * silu(h @ w["g"].T)) @ w["o"].T


def mlp(h, up, down):
    return torch.relu(h @ up.T).pow(2) @ down.T


def run_order(cfg) -> list[tuple[int, bool]]:
    """(layer, starts a pass) of every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    body = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return [(i, False) for i in range(loop["start"])] + body * loop["times"] + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg, weights, tokens):
    """-> logits [T, vocab] and the stream after every layer run [runs, T, width]."""
    w = {name: to_f64(value) for name, value in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x0, streams = x.clone(), []
    for layer, starts_pass in run_order(cfg):
        entry, p = cfg["layers"][layer], f"l{layer}."
        sub = lambda prefix: {n[len(prefix):]: t for n, t in w.items() if n.startswith(prefix)}  # noqa: E731
        if starts_pass:
            x = torch.cat([x, x0], dim=-1) @ w["loop.in"].T
        h, m = rms_norm(x, w[p + "norm1"], eps), entry["mixer"]
        x = x + m["left_scale"] * left_mixer(h, sub(p + "mix.left."), m["left"], eps) \
              + m["right_scale"] * right_mixer(h, sub(p + "mix.right."), m["right"], eps)
        if entry.get("mlp"):
            x = x + mlp(rms_norm(x, w[p + "norm2"], eps), w[p + "mlp.up"], w[p + "mlp.down"])
        streams.append(x.clone())
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits, torch.stack(streams)


def greedy(cfg, weights, prompt, n_new):
    """-> generated tokens and, per token, how far its logit is ahead of the runner-up."""
    seq, margins = list(prompt), []
    for _ in range(n_new):
        top = forward(cfg, weights, seq)[0][-1].topk(2)
        seq.append(int(top.indices[0]))
        margins.append(float(top.values[0] - top.values[1]))
    return seq[len(prompt):], margins
