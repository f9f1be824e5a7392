"""Oracle for the Folivik decoder: one plain function per mechanism, float64, no cache and no batching -- a whole sequence goes
in, every position comes out. TEST INFRASTRUCTURE ONLY (see oracle/__init__.py). No reference code defines this model; the
functions restate its equations:

    norm       y = g x / sqrt(mean(x^2) + eps): one number g on the stream, a vector elsewhere
    latent     c = norm(first r rows of W_dkv h), z = the other rows turned by the position; per head k = (W_uk c, z), v = W_uv c,
    attention  q = (u, turned w), (u, w) = W_uq norm(W_dq h);  y_h = sigmoid(W_g h)_h softmax(scale <q, k>) v
    windowed   s_hij = scale t_h <q_i, k_j> - a_h ln(1 + b_h (i - j)) for 0 <= i - j < size, q and k normed per head;  y = softmax(s) v
    attention
    Mamba-2    S_t = exp(-e^A dt_t) S_{t-1} + dt_t B_t x_t^T,  y_t = S_t^T C_t + D x_t;  (x, B, C) convolved over time, then silu;
               dt = softplus(. + bias);  out = W_o norm_parts(y silu(z))
    experts    s = softmax(W_r h); chosen by s + correction within the best groups; weights s / sum, times a factor; the last ones of
               them hand h through; a shared one runs for every token
    layer      x += mixer(norm(x)),  x += experts(norm(x))
    head       W norm(x)
"""
from __future__ import annotations

import math

import torch

from .vozozen import to_f64


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def turn_pairs(x, positions, base):
    """Dims 2 i and 2 i + 1 of x [T, .., n] turn by position * base^(-2 i / n)."""
    n, out = x.shape[-1], x.clone()
    for r, p in enumerate(positions):
        for i in range(n // 2):
            a = p * base ** (-2.0 * i / n)
            u, v = x[r, ..., 2 * i], x[r, ..., 2 * i + 1]
            out[r, ..., 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[r, ..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def softmax_attention(q, k, v, scale, *, first=0, window=None, temp=None, bias=None):
    """q [N, H, d] at positions first, first + 1, .., k [T, G, d] and v [T, G, dv] at 0, 1, .. -> [N, H, dv]. temp: factor per head;
    bias: (a, b) per head, a ln(1 + b distance) is taken off the scores."""
    N, H = q.shape[:2]
    T, share = k.shape[0], H // k.shape[1]
    k, v = k.repeat_interleave(share, 1), v.repeat_interleave(share, 1)
    out = torch.zeros(N, H, v.shape[2], dtype=torch.float64)
    for i in range(N):
        lo = 0 if window is None else max(0, first + i - window + 1)
        hi = first + i + 1
        assert hi <= T
        s = torch.einsum("jhd,hd->hj", k[lo:hi], q[i]) * scale
        if temp is not None:
            s = s * temp.unsqueeze(1)
        if bias is not None:
            distance = first + i - torch.arange(lo, hi)
            s = s - bias[0].unsqueeze(1) * torch.log(1 + bias[1].unsqueeze(1) * distance)
        out[i] = torch.einsum("hj,jhd->hd", torch.softmax(s, 1), v[lo:hi])
    return out


def latent_keys_values(c, z, uk, uv, heads):
    """Latents c [T, r] and turned parts z [T, n] -> keys [T, H, d + n] and values [T, H, dv]"""
    T = c.shape[0]
    k = torch.cat([(c @ uk.T).view(T, heads, -1), z.unsqueeze(1).expand(T, heads, -1)], dim=-1)
    return k, (c @ uv.T).view(T, heads, -1)


def latent_attention_mixer(h, w, m, eps):
    T, H = h.shape[0], m["heads"]
    q = (rms(h @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T
    q = q.view(T, H, m["dim"] + m["rot_dim"])
    down = h @ w["dkv"].T
    c = rms(down[:, :m["kv_rank"]], eps) * w["dkv.norm"]
    z = turn_pairs(down[:, m["kv_rank"]:], range(T), m["rot"]["base"])
    q = torch.cat([q[..., :m["dim"]], turn_pairs(q[..., m["dim"]:], range(T), m["rot"]["base"])], dim=-1)
    k, v = latent_keys_values(c, z, w["uk"], w["uv"], H)
    y = softmax_attention(q, k, v, m["scale"]) * torch.sigmoid(h @ w["g"].T).unsqueeze(-1)
    return y.reshape(T, -1) @ w["o"].T


def window_attention_mixer(h, w, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms((h @ w["q"].T).view(T, H, m["dim"]), eps) * w["q.norm"]
    k = rms((h @ w["k"].T).view(T, G, m["dim"]), eps) * w["k.norm"]
    v = (h @ w["v"].T).view(T, G, m["vdim"])
    y = softmax_attention(q, k, v, m["scale"], window=m["mask"]["size"], temp=w["temp"], bias=(w["r1"], w["r2"]))
    return y.reshape(T, -1) @ w["o"].T


def convolve(x, taps, bias, before=None):
    """Causal convolution over time of each channel, then silu. x [T, C]; the last column of taps [C, n] is the current token's;
    before: the n - 1 inputs ahead of x (zeros when not given)."""
    T, C, n = x.shape[0], x.shape[1], taps.shape[1]
    ahead = torch.zeros(n - 1, C, dtype=torch.float64) if before is None else before
    full = torch.cat([ahead, x])
    return silu(torch.stack([(full[t:t + n] * taps.T).sum(0) + bias for t in range(T)]))


def state_space(x, B, C, dt, a_log, D, state=None):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (after softplus) -> y [T, H, P] and the final state [H, N, P]"""
    T, H, P = x.shape
    share, N = H // B.shape[1], B.shape[2]
    S = torch.zeros(H, N, P, dtype=torch.float64) if state is None else state.clone()
    y = torch.empty_like(x)
    for t in range(T):
        for h in range(H):
            S[h] = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, h // share], x[t, h])
            y[t, h] = S[h].T @ C[t, h // share] + D[h] * x[t, h]
    return y, S


def gated_parts_norm(y, z, weight, parts, eps):
    y = y * silu(z)
    return rms(y.view(y.shape[0], parts, -1), eps).reshape(y.shape) * weight


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def mamba2_mixer(h, w, m, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    z, xbc, dt = (h @ w["in"].T).split([H * P, H * P + 2 * G * N, H], dim=1)
    x, B, C = convolve(xbc, w["conv"], w["conv.b"]).split([H * P, G * N, G * N], dim=1)
    y, _ = state_space(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    return gated_parts_norm(y.reshape(T, H * P), z, w["norm"], m["norm_groups"], eps) @ w["o"].T


def route(logits, correction, router):
    """Router logits of one token -> chosen indices and their weights."""
    s = torch.softmax(logits, 0)
    choice = s + correction
    groups = router.get("groups")
    if groups:
        size = len(choice) // groups["count"]
        best = torch.stack([choice[g * size:(g + 1) * size].max() for g in range(groups["count"])])
        allowed = torch.zeros(len(choice), dtype=torch.bool)
        for g in best.topk(groups["keep"]).indices.tolist():
            allowed[g * size:(g + 1) * size] = True
        choice = choice.masked_fill(~allowed, -math.inf)
    chosen = choice.topk(router["top"]).indices
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20) * router["scale"]


def gated_unit(h, w, name):
    return (silu(h @ w[name + ".gate"].T) * (h @ w[name + ".up"].T)) @ w[name + ".down"].T


def expert_layer(h, w, mlp):
    out = torch.zeros_like(h)
    logits = h @ w["router"].T
    for t in range(h.shape[0]):
        for e, weight in zip(*route(logits[t], w["correction"], mlp["router"])):
            e = int(e)
            out[t] += weight * (gated_unit(h[t], w, f"e{e}") if e < mlp["router"]["experts"] else h[t])
    return out + gated_unit(h, w, "shared") if mlp.get("shared") else out


MIXERS = {"latent_attention": latent_attention_mixer, "attention": window_attention_mixer, "mamba2": mamba2_mixer}


def forward(cfg, weights, tokens):
    """-> logits [T, vocab] and the stream after every layer [layers, T, width]."""
    w = {name: to_f64(value) for name, value in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor([int(t) for t in tokens])]
    streams = []
    for i, entry in enumerate(cfg["layers"]):
        sub = lambda prefix: {n[len(prefix):]: t for n, t in w.items() if n.startswith(prefix)}  # noqa: E731
        x = x + MIXERS[entry["type"]](rms(x, eps) * w[f"l{i}.norm1"], sub(f"l{i}.mix."), entry["mixer"], eps)
        if entry.get("mlp"):
            x = x + expert_layer(rms(x, eps) * w[f"l{i}.norm2"], sub(f"l{i}.mlp."), entry["mlp"])
        streams.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T, torch.stack(streams)


def greedy(cfg, weights, prompt, n_new):
    """-> generated tokens and, per token, how far its logit is ahead of the runner-up."""
    seq, margins = list(prompt), []
    for _ in range(n_new):
        top = forward(cfg, weights, seq)[0][-1].topk(2)
        seq.append(int(top.indices[0]))
        margins.append(float(top.values[0] - top.values[1]))
    return seq[len(prompt):], margins
