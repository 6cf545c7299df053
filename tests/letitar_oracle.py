"""Plain, slow Letitar in double precision: the oracle of the Letitar tests.

One function per mechanism, a Python loop where the equations have a recurrence, no batching, no
cache, and no import from the package under test.  ``w`` is a dict of tensors by checkpoint name,
``cfg`` the parsed config.json.
"""
import math

import torch

F64 = torch.float64


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def yarn_frequencies(dims, base, scaling):
    """(angle per position of every pair, factor on cos and sin)."""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freq, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def turns_dim(t):
        return dims * math.log(original / (2 * math.pi * t)) / (2 * math.log(base))

    lo = max(math.floor(turns_dim(scaling["fast"])), 0)
    hi = min(math.ceil(turns_dim(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(factor) + 1


def rotate_interleaved(x, positions, rot):
    """x [T, ..., n]: pairs (2i, 2i+1) of the first rot["dims"] channels turned by position * f_i."""
    freq, amp = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    out = x.clone()
    for i, f in enumerate(freq):
        a = positions.to(x.dtype) * f
        c, s = torch.cos(a) * amp, torch.sin(a) * amp
        shape = (-1,) + (1,) * (x.dim() - 2)
        c, s = c.view(shape), s.view(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def gla_decay(z, tau):
    """Decay per key channel in (0, 1)."""
    return torch.sigmoid(z) ** (1.0 / tau)


def gla_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha [T, H, K]; v [T, H, V] -> outputs [T, H, V], final state [H, K, V]."""
    T, H, K = q.shape
    S = torch.zeros(H, K, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            S[h] = alpha[t, h][:, None] * S[h] + torch.outer(k[t, h], v[t, h])
            out[t, h] = S[h].t() @ q[t, h]
    return out, S


def gla_mixer(h, m, w, p, eps, state=None):
    T, H, K, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].t()).view(T, H, K) * K ** -0.5
    k = (h @ w[p + "k"].t()).view(T, H, K)
    v = (h @ w[p + "v"].t()).view(T, H, V)
    z = (h @ w[p + "a1"].t()) @ w[p + "a2"].t() + w[p + "a2.b"]
    o, S = gla_recurrence(q, k, v, gla_decay(z.view(T, H, K), m["tau"]), state)
    o = rms_norm(o, w[p + "norm"], eps).reshape(T, H * V)
    g = h @ w[p + "g"].t()
    return (o * (g * torch.sigmoid(g))) @ w[p + "o"].t(), S


def causal_softmax_attention(q, k, v, scale):
    """q, k [T, H, *]; v [T, H, V]; every query sees itself and what came before."""
    T = q.shape[0]
    out = torch.zeros(T, q.shape[1], v.shape[-1], dtype=q.dtype)
    for t in range(T):
        s = torch.einsum("hd,shd->hs", q[t], k[: t + 1]) * scale
        out[t] = torch.einsum("hs,shv->hv", torch.softmax(s, -1), v[: t + 1])
    return out


def latent_and_rotated_key(h, m, w, p, eps, positions):
    d = h @ w[p + "dkv"].t()
    R = m["kv_rank"]
    return rms_norm(d[:, :R], w[p + "dkv.norm"], eps), rotate_interleaved(d[:, R:], positions, m["rot"])


def latent_attention_mixer(h, m, w, p, eps, shared):
    """``shared``: (latent, rotated key part) this layer attends to."""
    T, H, D, Rd, V = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, k_rot = shared
    q = (h @ w[p + "q"].t()).view(T, H, D + Rd)
    q_rot = rotate_interleaved(q[..., D:], torch.arange(T), m["rot"])
    k = (c @ w[p + "uk"].t()).view(T, H, D)
    v = (c @ w[p + "uv"].t()).view(T, H, V)
    q = torch.cat([q[..., :D], q_rot], -1)
    k = torch.cat([k, k_rot[:, None].expand(T, H, Rd)], -1)
    return causal_softmax_attention(q, k, v, m["scale"]).reshape(T, H * V) @ w[p + "o"].t()


def squared_relu_mlp(h, w, p):
    return torch.clamp(h @ w[p + "up"].t(), min=0) ** 2 @ w[p + "down"].t()


def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


def run(cfg, weights, tokens):
    """(logits [T, vocab], residual after every layer [layers, T, width], final recurrent states)."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    latents, residuals, states = {}, [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        h = layer_norm(x, w[f"l{i}.norm1"], w[f"l{i}.norm1.b"], eps)
        if layer["type"] == "gla":
            y, states[i] = gla_mixer(h, m, w, p, eps)
        else:
            if m.get("kv_from") is None:
                latents[i] = latent_and_rotated_key(h, m, w, p, eps, torch.arange(len(tokens)))
            y = latent_attention_mixer(h, m, w, p, eps, latents[i if m.get("kv_from") is None else m["kv_from"]])
        x = x + y
        if layer.get("mlp") is not None:
            x = x + squared_relu_mlp(layer_norm(x, w[f"l{i}.norm2"], w[f"l{i}.norm2.b"], eps), w, f"l{i}.mlp.")
        residuals.append(x.clone())
    x = layer_norm(x, w["final.norm"], w["final.norm.b"], eps)
    return soft_cap(x @ w["head"].t(), cfg["logit_softcap"]), torch.stack(residuals), states
