"""Plain statement of the Milenex design: whole sequences, one token or one head at a time, in the precision of the tensors it is
given (fp32 or fp64). One function per mechanism, written from the equations; nothing here is shared with the engine."""
import math

import torch


# ------------------------------------------------------------------------------------------------ pieces
def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def gelu(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2)))


def token_shift(h, mu):
    """h [T, W]: every token moves a step of its own size per channel towards the token before it (zeros before the first)."""
    out = torch.empty_like(h)
    for t in range(h.shape[0]):
        before = h[t - 1] if t > 0 else torch.zeros_like(h[0])
        out[t] = h[t] + (before - h[t]) * mu
    return out


def causal_conv(u, w):
    """u [T, C], w [C, taps]: the last tap meets the token itself."""
    taps, out = w.shape[1], torch.zeros_like(u)
    for t in range(u.shape[0]):
        for back in range(taps):
            if t - back >= 0:
                out[t] = out[t] + w[:, taps - 1 - back] * u[t - back]
    return out


def rotate(x, dims, base, start=0):
    """x [T, d] of one head; row t stands at position start + t. Values 2i and 2i + 1 of the first ``dims`` turn together."""
    pos = torch.arange(start, start + x.shape[0], dtype=x.dtype)
    y = x.clone()
    for i in range(dims // 2):
        a = pos * base ** (-2 * i / dims)
        u, v = x[:, 2 * i], x[:, 2 * i + 1]
        y[:, 2 * i], y[:, 2 * i + 1] = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
    return y


def weights(q, k, scale, window, sink, r1=None, r2=None):
    """Attention weights [T, S] of one head: q [T, d] are the last T of the S positions, k [S, d]. A query sees itself and the
    window - 1 tokens before it; ``sink`` is a logit without a key; r1, r2: distance bias r1 ln(1 + r2 distance), taken off."""
    T, n = q.shape[0], k.shape[0]
    out = torch.zeros(T, n, dtype=q.dtype)
    for t in range(T):
        i = n - T + t
        lo = max(0, i - window + 1)
        s = k[lo:i + 1] @ q[t] * scale
        if r1 is not None:
            s = s - r1 * torch.log(1 + r2 * (i - torch.arange(lo, i + 1, dtype=q.dtype)))
        out[t, lo:i + 1] = torch.softmax(torch.cat([s, sink.reshape(1).to(s.dtype)]), 0)[:-1]
    return out


def talk(w, T):
    """w: one weight matrix per head; head h's mixed weights are sum_g T[h, g] w[g]."""
    return [sum(T[h, g] * w[g] for g in range(len(w))) for h in range(len(w))]


# ------------------------------------------------------------------------------------------------ mixers
def rotary_attention(h, w, p, spec, eps):
    """Short convolutions, rotation, norm of queries and keys, window and sink."""
    T, H, G, d, dv = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q, k, v = (causal_conv(h @ w[p + n].t(), w[p + n + ".conv"]) for n in "qkv")
    q, k, v = q.view(T, H, d), k.view(T, G, d), v.view(T, G, dv)
    turn = lambda x: rms(rotate(x, spec["rot"]["dims"], spec["rot"]["base"]), eps)
    kr, heads = [turn(k[:, g]) for g in range(G)], []
    for i in range(H):
        g = i // (H // G)
        heads.append(weights(turn(q[:, i]), kr[g], spec["scale"], spec["mask"]["size"], w[p + "sink"][i]) @ v[:, g])
    return torch.cat(heads, -1) @ w[p + "o"].t()


def talking_attention(h, w, p, spec, eps):
    """Distance bias, window and sink; the heads' weights mixed; a gate per head."""
    T, H, G, d, dv = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q, k, v = (h @ w[p + "q"].t()).view(T, H, d), (h @ w[p + "k"].t()).view(T, G, d), (h @ w[p + "v"].t()).view(T, G, dv)
    per = [weights(q[:, i], k[:, i // (H // G)], spec["scale"], spec["mask"]["size"], w[p + "sink"][i], w[p + "r1"][i], w[p + "r2"][i]) for i in range(H)]
    gate = sigmoid(h @ w[p + "g"].t())
    heads = [(m @ v[:, i // (H // G)]) * gate[:, i:i + 1] for i, m in enumerate(talk(per, w[p + "talk"]))]
    return torch.cat(heads, -1) @ w[p + "o"].t()


# ------------------------------------------------------------------------------------------------ feed-forward
def clamped_glu(x, w, p, limit):
    g = torch.clamp(x @ w[p + "gate"].t(), max=limit)
    u = torch.clamp(x @ w[p + "up"].t(), -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].t()


def choose(scores, correction, top, count, keep):
    """Experts of one token: the best ``top`` by corrected score inside the ``keep`` groups with the best corrected scores."""
    choice = [float(s + c) for s, c in zip(scores, correction)]
    per = len(choice) // count
    best = sorted(range(count), key=lambda g: (-max(choice[g * per:(g + 1) * per]), g))[:keep]
    allowed = [e for e in range(len(choice)) if e // per in best]
    return sorted(allowed, key=lambda e: (-choice[e], e))[:top]


def routed_mlp(x, w, p, spec):
    r = spec["router"]
    groups = r.get("groups") or dict(count=1, keep=1)
    s = torch.softmax(x @ w[p + "router"].t(), -1)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e in choose(s[t], w[p + "correction"], r["top"], groups["count"], groups["keep"]):
            y[t] += s[t, e] * clamped_glu(x[t], w, f"{p}e{e}.", spec["expert"]["limit"])
    if spec.get("shared"):
        y = y + clamped_glu(x, w, p + "shared.", spec["shared"]["limit"]) * sigmoid(x @ w[p + "shared.sg"].t())
    return y


# ------------------------------------------------------------------------------------------------ the model
def runs(cfg):
    """(layer, does a pass but the first begin here) in running order."""
    n, loop = len(cfg["layers"]), cfg.get("loop") or dict(start=0, stop=0, times=1)
    out = [(i, False) for i in range(loop["start"])]
    for time in range(loop["times"]):
        out += [(i, time > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return out + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg, tensors, tokens, dtype=torch.float32, residuals=None):
    """Logits [T, vocab]. ``residuals``: a list that receives the residual after every layer run."""
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    first = w["embed"][torch.tensor(list(tokens), dtype=torch.long)]
    x = first
    for i, again in runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if again:
            x = x + first
        mixer = {"attention": rotary_attention, "attention_2": talking_attention}[layer["type"]]
        x = x + mixer(token_shift(norm(x, w[p + "norm1"], eps), w[p + "shift"]), w, p + "mix.", layer["mixer"], eps)
        mlp = layer["mlp"]
        if mlp is not None:
            h = norm(x, w[p + "norm2"], eps)
            x = x + (gelu(h @ w[p + "mlp.up"].t()) @ w[p + "mlp.down"].t() if mlp["kind"] == "dense" else routed_mlp(h, w, p + "mlp.", mlp))
        if residuals is not None:
            residuals.append(x)
    return norm(x, w["final.norm"], eps) @ w["head"].t()
