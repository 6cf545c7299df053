"""Plain, slow Difedra in double precision: the oracle of the Difedra tests.

One function per mechanism, one query or one token at a time where that says it best, no batching, no
cache, and no import from the package under test.  ``w`` is a dict of tensors by checkpoint name,
``cfg`` the parsed config.json.
"""
import math

import torch

F64 = torch.float64


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotary_frequencies(rot):
    """Angle per position of every pair; long wavelengths are stretched by ``scaling``."""
    s, out = rot.get("scaling"), []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if s is not None:
            turns = s["original"] * f / (2 * math.pi)          # within the original context
            if turns < s["low"]:
                f = f / s["factor"]
            elif turns <= s["high"]:
                keep = (turns - s["low"]) / (s["high"] - s["low"])
                f = (1 - keep) * f / s["factor"] + keep * f
        out.append(f)
    return out


def rotate_half(x, positions, rot):
    """x [T, heads, n]: channels i and i + dims/2 turned by position * f_i, channels from dims on kept."""
    out, half = x.clone(), rot["dims"] // 2
    for i, f in enumerate(rotary_frequencies(rot)):
        a = positions.to(x.dtype)[:, None] * f
        c, s = torch.cos(a), torch.sin(a)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def window_attention(q, k, v, scale, window, sink):
    """q [T, H, *], k and v [T, G, *]; a query sees the last ``window`` tokens up to itself.  ``sink`` [H]
    (or None) is the logit of an extra denominator term without a value."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        lo = max(0, t - window + 1) if window else 0
        for h in range(H):
            s = k[lo:t + 1, h // rep] @ q[t, h] * scale
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            e = torch.exp(s - top)
            den = e.sum() if sink is None else e.sum() + torch.exp(sink[h] - top)
            out[t, h] = (e / den) @ v[lo:t + 1, h // rep]
    return out


def attention_mixer(h, m, w, p, eps, v_first, positions):
    """(output, values this layer would hand down)."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms_norm(h @ w[p + "q"].t(), w[p + "q.norm"], eps).view(T, H, m["dim"])      # over all heads at once
    k = rms_norm(h @ w[p + "k"].t(), w[p + "k.norm"], eps).view(T, G, m["dim"])
    v = (h @ w[p + "v"].t()).view(T, G, m["vdim"])
    q, k = rotate_half(q, positions, m["rot"]), rotate_half(k, positions, m["rot"])
    own = v
    if m["v_mix"] and v_first is not None:
        v = (1 - w[p + "vmix"]) * v + w[p + "vmix"] * v_first
    o = window_attention(q, k, v, m["scale"], m["mask"]["size"], w[p + "sink"])
    return o.reshape(T, -1) @ w[p + "o"].t(), own


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def gated_mlp(h, w, p, act):
    return (act(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


def route(z, top):
    """Sigmoid scores of the ``top`` largest logits, per token: (expert ids, weights)."""
    s = torch.sigmoid(z)
    ids = [sorted(range(z.shape[1]), key=lambda e, t=t: -float(s[t, e]))[:top] for t in range(z.shape[0])]
    ids = torch.tensor(ids)
    return ids, torch.gather(s, 1, ids)


def moe(h, w, p, top):
    ids, weight = route(h @ w[p + "router"].t(), top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t].tolist(), weight[t]):
            out[t] += gated_mlp(a * h[t:t + 1], w, f"{p}e{e}.", silu)[0]      # the weight scales the expert's input
    return out


def run(cfg, weights, tokens):
    """(logits [T, vocab], residual after every layer [layers, T, width])."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    positions, v_first, residuals = torch.arange(len(tokens)), None, []
    for i, layer in enumerate(cfg["layers"]):
        h = rms_norm(x, w[f"l{i}.norm1"], eps)
        y, own = attention_mixer(h, layer["mixer"], w, f"l{i}.mix.", eps, v_first, positions)
        if layer["mixer"]["v_mix"] and v_first is None:
            v_first = own
        x = x + y
        mlp = layer.get("mlp")
        if mlp is not None:
            h, p = rms_norm(x, w[f"l{i}.norm2"], eps), f"l{i}.mlp."
            x = x + (gated_mlp(h, w, p, gelu_tanh) if mlp["kind"] == "dense" else moe(h, w, p, mlp["router"]["top"]))
        residuals.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].t(), torch.stack(residuals)
