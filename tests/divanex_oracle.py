"""Plain statement of the Divanex design: whole sequences, one token or one head at a time, in the precision of the tensors it
is given (fp32 or fp64). One function per mechanism, written from the equations; nothing here is shared with the engine."""
import math

import torch


# ------------------------------------------------------------------------------------------------ pieces
def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x / (1 + torch.exp(-x))


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def short_conv(x, taps, bias):
    """x [T, C], taps [C, W], bias [C]: y[t, c] = bias[c] + sum_j taps[c, j] x[t - (W - 1) + j, c], zeros before the first token."""
    T, W = x.shape[0], taps.shape[1]
    y = bias.expand(T, -1).clone()
    for t in range(T):
        for j in range(W):
            if t - (W - 1) + j >= 0:
                y[t] += taps[:, j] * x[t - (W - 1) + j]
    return y


def ssd(x, dt, B, C, a, D, S=None):
    """One head: x [T, P], dt [T] (positive), B, C [T, N], a the decay rate. State S [N, P]. Returns (y [T, P], last state)."""
    S = torch.zeros(B.shape[1], x.shape[1], dtype=x.dtype) if S is None else S
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(-a * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        y[t] = S.t() @ C[t] + D * x[t]
    return y, S


def grouped_gated_norm(y, z, w, groups, eps):
    """(y silu(z)), each of `groups` equal parts over its own root mean square, times w."""
    T, n = y.shape
    return rms((y * silu(z)).view(T, groups, n // groups), eps).reshape(T, n) * w


def mamba2_mixer(h, w, p, spec, eps):
    T, H, P, N, G = h.shape[0], spec["heads"], spec["vdim"], spec["state"], spec["groups"]
    inner = H * P
    u = h @ w[p + "in"].t()
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = xbc[:, :inner].view(T, H, P), xbc[:, inner:inner + G * N].view(T, G, N), xbc[:, inner + G * N:].view(T, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    a = torch.exp(w[p + "A_log"])
    y = torch.stack([ssd(x[:, i], dt[:, i], B[:, i // (H // G)], C[:, i // (H // G)], a[i], w[p + "D"][i])[0] for i in range(H)], 1)
    return grouped_gated_norm(y.reshape(T, inner), z, w[p + "norm"], spec["norm_groups"], eps) @ w[p + "o"].t()


def query_temperature(pos, coef, every):
    return 1 + coef * torch.log(torch.floor((pos + 1) / every) + 1)


def attend(q, k, v, scale, cap=None):
    """One head: q [T, d], k, v [S, d]; the T queries are the last ones of the S positions."""
    T, n = q.shape[0], k.shape[0]
    s = q @ k.t() * scale
    if cap is not None:
        s = cap * torch.tanh(s / cap)
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    for t in range(T):
        out[t] = torch.softmax(s[t, :n - T + t + 1], -1) @ v[:n - T + t + 1]
    return out


def attention_mixer(h, w, p, spec, eps):
    T, H, G, d = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"]
    q, k = (h @ w[p + "q"].t()).view(T, H, d), (h @ w[p + "k"].t()).view(T, G, d)
    v, k, q = k, rms(k, eps), rms(q, eps)                      # the values are the keys before their norm
    tau = spec["q_temp"]
    q = q * query_temperature(torch.arange(T).to(h.dtype), tau["coef"], tau["every"])[:, None, None]
    heads = [attend(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], spec["scale"], spec["softcap"]) for i in range(H)]
    return torch.cat(heads, -1) @ w[p + "o"].t()


def clamped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g / (1 + torch.exp(-1.702 * g)) * (u + 1)


def feed_forward(x, w, p, limit):
    return clamped_glu(x @ w[p + "gate"].t(), x @ w[p + "up"].t(), limit) @ w[p + "down"].t()


def token_input(x, e, w, p, eps):
    """What a layer adds at its end: e [T, dim] is its part of the tokens' side embedding."""
    y = (gelu_tanh(x @ w[p + "gate"].t()) * e) @ w[p + "proj"].t()
    return rms(y, eps) * w[p + "norm"]


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg, weights, tokens, dtype=torch.float32, residuals=None):
    """Logits [T, vocab]. ``residuals``: a list that receives the residual after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, alpha, dim = cfg["norm"]["eps"], cfg["postln_alpha"], cfg["token_side"]["dim"]
    ids = torch.tensor(list(tokens), dtype=torch.long)
    x = w["embed"][ids] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p, mixer = f"l{i}.", {"mamba2": mamba2_mixer, "attention": attention_mixer}[layer["type"]]
        x = rms(alpha * x + mixer(x, w, p + "mix.", layer["mixer"], eps), eps) * w[p + "norm1"]
        if layer["mlp"] is not None:
            x = rms(alpha * x + feed_forward(x, w, p + "mlp.", layer["mlp"]["limit"]), eps) * w[p + "norm2"]
        x = x + token_input(x, w["side.embed"][ids, i * dim:(i + 1) * dim], w, p + "side.", eps)
        if residuals is not None:
            residuals.append(x)
    return rms(x, eps) * w["final.norm"] @ w["head"].t() * cfg["logit_scale"]
