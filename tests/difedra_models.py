"""Small random Difedra models for the tests: config dict, weights by checkpoint name, checkpoint folder."""
import torch

from .letitar_models import write  # noqa: F401  a config dict and tensors as a checkpoint folder


def attention(heads, kv_heads, dim, vdim, window, rot_dims=None, base=700.0, scaling=(3.0, 1.0, 4.0, 64), scale=None, v_mix=True):
    rot = {"dims": dim if rot_dims is None else rot_dims, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": rot, "v_mix": v_mix,
            "scale": dim ** -0.5 if scale is None else scale}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def config(vocab, width, layers, eps=1e-5):
    """``layers``: (mixer, feed-forward or None)."""
    return {"architecture": "Difedra", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{"type": "attention", "mixer": m, "mlp": f} for m, f in layers]}


def weights(cfg, seed, sharp=1.5):
    """bf16 tensors.  The norm weights of queries and keys make attention far from uniform, sinks take a
    visible share, and no choice of experts is close: the first channels of the embedding hold well
    separated values in an order of the token's own, which the layers hardly touch and the routers read."""
    g = torch.Generator().manual_seed(seed)
    D, out = cfg["width"], {}
    codes = max([f["router"]["experts"] for f in (layer["mlp"] for layer in cfg["layers"]) if f and f["kind"] == "moe"], default=0)

    def mat(name, rows, cols, gain=1.0):
        out[name] = torch.randn(rows, cols, generator=g) * gain / cols ** 0.5

    def vec(name, n, mean=0.0, std=0.3):
        out[name] = mean + std * torch.randn(n, generator=g)

    def into_residual(name, cols):
        mat(name, D, cols)
        out[name][:codes] *= 0.05

    mat("embed", cfg["vocab"], D, gain=D ** 0.5)
    levels = torch.linspace(-1, 1, max(codes, 1)) * codes
    for t in range(cfg["vocab"]):
        out["embed"][t, :codes] = levels[torch.randperm(codes, generator=g)] if codes else 0
    vec("final.norm", D, 1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        H, G = m["heads"], m["kv_heads"]
        vec(p + "norm1", D, 1.0)
        mat(p + "mix.q", H * m["dim"], D)
        mat(p + "mix.k", G * m["dim"], D)
        mat(p + "mix.v", G * m["vdim"], D)
        into_residual(p + "mix.o", H * m["vdim"])
        vec(p + "mix.q.norm", H * m["dim"], sharp)
        vec(p + "mix.k.norm", G * m["dim"], sharp)
        vec(p + "mix.sink", H, 2.0, 1.5)
        if m["v_mix"]:
            out[p + "mix.vmix"] = torch.rand((), generator=g) * 0.6 + 0.2
        if f is None:
            continue
        vec(p + "norm2", D, 1.0)
        out[p + "norm2"][:codes] = 1.0
        if f["kind"] == "dense":
            mat(p + "mlp.gate", f["ff"], D, gain=1.5)
            mat(p + "mlp.up", f["ff"], D)
            into_residual(p + "mlp.down", f["ff"])
            continue
        E, F = f["router"]["experts"], f["expert"]["ff"]
        order = torch.randperm(codes, generator=g)[:E]
        out[p + "mlp.router"] = 0.003 * torch.randn(E, D, generator=g)
        out[p + "mlp.router"][torch.arange(E), order] += 1.0
        for e in range(E):
            mat(p + f"mlp.e{e}.gate", F, D, gain=2.0)
            mat(p + f"mlp.e{e}.up", F, D, gain=2.0)
            into_residual(p + f"mlp.e{e}.down", F)
    return {k: v.bfloat16() for k, v in out.items()}


# sizes of their own: every width a multiple of 8, so bf16 takes the tensor-core kernels
EVEN = config(328, 160, [
    (attention(6, 2, 40, 24, 19), moe(7, 3, 72)),
    (attention(5, 1, 64, 48, 33, rot_dims=32, v_mix=False, scaling=None), dense(200)),
    (attention(4, 4, 32, 12 * 4, 7, rot_dims=16, base=40.0, scale=0.3, v_mix=False), None),
    (attention(6, 2, 24, 24, 26, scaling=(16.0, 0.5, 2.0, 32)), moe(5, 1, 88)),
    (attention(40, 2, 16, 24, 12, rot_dims=8), moe(6, 6, 40))])
# no width a multiple of 8, single heads, factor 1, a window of one token; the mixed values start at layer 1
ODD = config(203, 90, [
    (attention(3, 3, 14, 5, 11, v_mix=False, scaling=None), dense(51)),
    (attention(2, 1, 10, 9, 17, rot_dims=6, scaling=(1.0, 1.0, 4.0, 16)), moe(3, 1, 33)),
    (attention(9, 1, 6, 9, 1, rot_dims=2), None),
    (attention(1, 1, 22, 9, 23, base=9.0, scaling=(5.0, 1.0, 1.0, 40)), moe(4, 2, 21))], eps=1e-3)
