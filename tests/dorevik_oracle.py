"""Plain statement of the Dorevik design: whole sequences, one token or one head at a time, in the precision of the tensors it
is given (fp32 or fp64). One function per mechanism, written from the equations; nothing here is shared with the engine."""
import math

import torch


# ------------------------------------------------------------------------------------------------ pieces
def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot):
    """(angle per position of every rotated pair, factor on the cosine and the sine)."""
    n, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2 * i / n) for i in range(n // 2)]
    if s is None:
        return f, 1.0
    where = lambda turns: n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), n - 1)
    ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(n // 2)]
    return [f[i] / s["factor"] * ramp[i] + f[i] * (1 - ramp[i]) for i in range(n // 2)], 0.1 * math.log(s["factor"]) + 1


def rotate(x, rot, start=0):
    """x [T, d] of one head; row t stands at position start + t. Value i of the first dims / 2 turns with value i + dims / 2."""
    f, factor = frequencies(rot)
    pos = torch.arange(start, start + x.shape[0], dtype=x.dtype)
    y, half = x.clone(), rot["dims"] // 2
    for i in range(half):
        c, s = factor * torch.cos(pos * f[i]), factor * torch.sin(pos * f[i])
        y[:, i], y[:, i + half] = x[:, i] * c - x[:, i + half] * s, x[:, i + half] * c + x[:, i] * s
    return y


def attend(q, k, v, scale, window):
    """One head: q [T, d], k [S, d], v [S, dv]; the T queries are the last ones of the S positions. A query sees itself and the
    window - 1 tokens before it."""
    T, n = q.shape[0], k.shape[0]
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    for t in range(T):
        i = n - T + t
        lo = max(0, i - window + 1)
        out[t] = torch.softmax(k[lo:i + 1] @ q[t] * scale, 0) @ v[lo:i + 1]
    return out


def diff_lambda(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def differential(a1, a2, lam, diff, eps):
    """Two attention outputs [T, dv] of one head -> its output."""
    return rms(a1 - lam * a2, eps) * (1 - diff)


def decayed_sum(q, k, v, decay, S=None):
    """One head: q, k [T, d], v [T, dv]. State S [d, dv]. Returns (o [T, dv], last state)."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=k.dtype) if S is None else S
    o = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        o[t] = S.t() @ q[t]
    return o, S


# ------------------------------------------------------------------------------------------------ mixers
def attention_mixer(h, w, p, spec, eps):
    """Differential attention: every head has two maps over the same values."""
    T, H, G, d, dv = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = rms((h @ w[p + "q"].t() + w[p + "q.b"]).view(T, H, 2, d), eps) * w[p + "q.norm"]
    k = rms((h @ w[p + "k"].t() + w[p + "k.b"]).view(T, G, 2, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].t() + w[p + "v.b"]).view(T, G, dv)
    lam = diff_lambda(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], spec["diff"])
    kr = [[rotate(k[:, g, m], spec["rot"]) for m in range(2)] for g in range(G)]
    heads = []
    for i in range(H):
        g = i // (H // G)
        a1, a2 = (attend(rotate(q[:, i, m], spec["rot"]), kr[g][m], v[:, g], spec["scale"], spec["mask"]["size"]) for m in range(2))
        heads.append(differential(a1, a2, lam, spec["diff"], eps))
    return torch.cat(heads, -1) @ w[p + "o"].t()


def window_attention(h, w, p, spec, eps):
    T, H, G, d, dv = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = (rms(h @ w[p + "q"].t(), eps) * w[p + "q.norm"]).view(T, H, d)
    k = (rms(h @ w[p + "k"].t(), eps) * w[p + "k.norm"]).view(T, G, d)
    v = (h @ w[p + "v"].t()).view(T, G, dv)
    kr = [rotate(k[:, g], spec["rot"]) for g in range(G)]
    heads = [attend(rotate(q[:, i], spec["rot"]), kr[i // (H // G)], v[:, i // (H // G)], spec["scale"], spec["mask"]["size"]) for i in range(H)]
    return torch.cat(heads, -1) @ w[p + "o"].t()


def lightning_attention(h, w, p, spec, eps):
    T, H, d, dv = h.shape[0], spec["heads"], spec["dim"], spec["vdim"]
    q, k = (silu(h @ w[p + n].t()).view(T, H, d) for n in ("q", "k"))
    v = silu(h @ w[p + "v"].t()).view(T, H, dv)
    o = torch.cat([decayed_sum(q[:, i], k[:, i], v[:, i], spec["decay"][i])[0] for i in range(H)], -1)
    return (rms(o, eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].t())) @ w[p + "o"].t()


def parallel_mixer(h, w, p, spec, eps):
    a = rms(window_attention(h, w, p + "left.", spec["left"], eps), eps) * w[p + "left.out"]
    b = rms(lightning_attention(h, w, p + "right.", spec["right"], eps), eps) * w[p + "right.out"]
    return (a + b) / 2


# ------------------------------------------------------------------------------------------------ feed-forward
def gated_mlp(x, w, p, act):
    return (act(x @ w[p + "gate"].t()) * (x @ w[p + "up"].t())) @ w[p + "down"].t()


def routed_mlp(x, w, p, spec):
    """The best experts by the sigmoid of their router logit; the score scales an expert's input."""
    s = sigmoid(x @ w[p + "router"].t())
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e in sorted(range(s.shape[1]), key=lambda e: (-float(s[t, e]), e))[:spec["router"]["top"]]:
            y[t] += gated_mlp(s[t, e] * x[t], w, f"{p}e{e}.", silu)
    return y + gated_mlp(x, w, p + "shared.", silu) if spec.get("shared") else y


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg, weights, tokens, dtype=torch.float32, residuals=None):
    """Logits [T, vocab]. ``residuals``: a list that receives the residual after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p, mixer = f"l{i}.", {"attention": attention_mixer, "parallel": parallel_mixer}[layer["type"]]
        x = x + rms(mixer(x, w, p + "mix.", layer["mixer"], eps), eps) * w[p + "norm1"]
        mlp = layer["mlp"]
        if mlp is not None:
            y = gated_mlp(x, w, p + "mlp.", gelu_tanh) if mlp["kind"] == "dense" else routed_mlp(x, w, p + "mlp.", mlp)
            x = x + rms(y, eps) * w[p + "norm2"]
        if residuals is not None:
            residuals.append(x)
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(rms(x, eps) * w["final.norm"] @ w["head"].t() / cap)
