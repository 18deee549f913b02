"""Plain statement of the Sovanex design: whole sequences, one token or one head at a time, in the precision of the
tensors it is given (fp32 or fp64). One function per mechanism, written from the equations; nothing here is shared with
the engine. ``random_model`` draws a small configuration's weights under the checkpoint names the loader reads."""
import math

import torch


# ------------------------------------------------------------------------------------------------ pieces
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rotate_half(x, pos, base):
    """x [T, ..., n], pos [T]: the pairs (x[i], x[i + n/2]) turn by pos * base^(-2i/n)."""
    n = x.shape[-1]
    out = x.clone()
    for i in range(n // 2):
        a = pos.to(x.dtype) * (base ** (-2.0 * i / n))
        a = a.view(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., i], x[..., i + n // 2]
        out[..., i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., i + n // 2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def short_conv_silu(x, taps):
    """x [T, C], taps [C, W]: y[t] = silu(sum_j taps[:, j] x[t - (W - 1) + j]), zeros before the first token."""
    T, W = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(W):
        back = W - 1 - j
        if back < T:
            y[back:] += taps[:, j] * x[:T - back]
    return y * torch.sigmoid(y)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """One head: q, k [T, d] (already unit, q scaled), v [T, dv], g, beta [T]. State S [d, dv]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = S * g[t]
        u = beta[t] * (v[t] - S.t() @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.t() @ q[t]
    return out


def delta_mixer(h, w, p, spec, eps):
    """w: tensors by full name, p: the mixer's prefix."""
    T, H, Hk, d, dv = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    conv = lambda n: short_conv_silu(h @ w[p + n].t(), w[p + n + ".conv"])
    q = unit(conv("q").view(T, Hk, d)) / math.sqrt(d)
    k = unit(conv("k").view(T, Hk, d))
    v = conv("v").view(T, H, dv)
    beta = torch.sigmoid(h @ w[p + "b"].t())
    a = h @ w[p + "a"].t() + w[p + "dt_bias"]
    softplus = torch.clamp(a, min=0) + torch.log1p(torch.exp(-a.abs()))
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus)
    o = torch.stack([delta_rule(q[:, hh // (H // Hk)], k[:, hh // (H // Hk)], v[:, hh], g[:, hh], beta[:, hh]) for hh in range(H)], 1)
    gate = (h @ w[p + "g"].t()).view(T, H, dv)
    o = rms_norm(o, w[p + "norm"], eps) * (gate * torch.sigmoid(gate))
    return o.reshape(T, H * dv) @ w[p + "o"].t()


def latent_rows(h, w, p, spec, eps):
    """(normalised latent c [T, R], rotated shared key part [T, dr]) of a layer with a down-projection of its own."""
    R = spec["kv_rank"]
    y = h @ w[p + "dkv"].t()
    return rms_norm(y[:, :R], w[p + "dkv.norm"], eps), rotate_half(y[:, R:], torch.arange(h.shape[0]), spec["rot"]["base"])


def latent_mixer(h, w, p, spec, rows):
    c, kr = rows
    T, H, d, dr, dv = h.shape[0], spec["heads"], spec["dim"], spec["rot_dim"], spec["vdim"]
    q = (h @ w[p + "q"].t()).view(T, H, d + dr)
    qn, qr = q[..., :d], rotate_half(q[..., d:], torch.arange(T), spec["rot"]["base"])
    k = (c @ w[p + "uk"].t()).view(T, H, d)
    v = (c @ w[p + "uv"].t()).view(T, H, dv)
    gate = torch.sigmoid(h @ w[p + "g"].t())
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    heads = []
    for hh in range(H):
        s = (qn[:, hh] @ k[:, hh].t() + qr[:, hh] @ kr.t()) * spec["scale"]
        pr = torch.softmax(s.masked_fill(~mask, float("-inf")), -1)
        heads.append(pr @ v[:, hh] * gate[:, hh:hh + 1])
    return torch.cat(heads, -1) @ w[p + "o"].t()


def feed_forward(h, w, p):
    u = torch.relu(h @ w[p + "up"].t())
    return (u * u) @ w[p + "down"].t()


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg, weights, tokens, dtype=torch.float32, residuals=None):
    """Logits [T, vocab]. ``residuals``: a list that receives the sum of the streams after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, m, S = cfg["norm"]["eps"], cfg["residual_mult"], cfg["streams"]
    x0 = w["embed"][torch.tensor(list(tokens), dtype=torch.long)]
    xs = [x0.clone() for _ in range(S)]
    rows = {}

    def sublayer(xs, p, q, f):
        hc = f"{p}hc{q}."
        u = sum(w[hc + "in"][s] * xs[s] for s in range(S))
        y = f(layer_norm(u, w[f"{p}norm{q}"], w[f"{p}norm{q}.b"], eps))
        return [sum(w[hc + "mix"][s, t] * xs[s] for s in range(S)) + m * w[hc + "out"][t] * y for t in range(S)]

    for i, layer in enumerate(cfg["layers"]):
        p, spec = f"l{i}.", layer["mixer"]

        def mixer(h):
            if layer["type"] == "delta":
                return delta_mixer(h, w, p + "mix.", spec, eps)
            rows[i] = rows[spec["kv_from"]] if spec.get("kv_from") is not None else latent_rows(h, w, p + "mix.", spec, eps)
            return latent_mixer(h, w, p + "mix.", spec, rows[i])
        xs = sublayer(xs, p, 1, mixer)
        if layer["mlp"] is not None:
            xs = sublayer(xs, p, 2, lambda h: feed_forward(h, w, p + "mlp."))
        if residuals is not None:
            residuals.append(sum(xs))
    return layer_norm(sum(xs), w["final.norm"], w["final.norm.b"], eps) @ w["embed"].t()
