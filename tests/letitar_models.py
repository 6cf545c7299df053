"""Small random Letitar models for the tests: config dict, weights by checkpoint name, checkpoint folder."""
import json

import torch
from safetensors.torch import save_file


def latent(heads, dim, rot_dim, vdim, kv_rank, kv_from=None, base=500.0, scaling=(2.0, 64, 8.0, 1.0), scale=None):
    rot = {"dims": rot_dim, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": rot,
         "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "latent_attention", m


def gla(heads, dim, vdim, tau=4.0):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def config(vocab, width, layers, eps=1e-5, cap=20.0):
    """``layers``: ((type, mixer), ff or None)."""
    return {"architecture": "Letitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap,
            "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
                       for (t, m), ff in layers]}


def weights(cfg, seed, decay_rank=8, sharp=2.0):
    """bf16 tensors; queries and keys are scaled up by ``sharp`` so that attention is far from uniform."""
    g = torch.Generator().manual_seed(seed)
    D, out = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * gain / cols ** 0.5).bfloat16()

    def vec(name, n, mean=0.0, std=0.3):
        out[name] = (mean + std * torch.randn(n, generator=g)).bfloat16()

    mat("embed", cfg["vocab"], D, gain=D ** 0.5)
    mat("head", cfg["vocab"], D, gain=3.0)
    vec("final.norm", D, 1.0)
    vec("final.norm.b", D)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for n in ("norm1", "norm2") if layer["mlp"] else ("norm1",):
            vec(p + n, D, 1.0)
            vec(p + n + ".b", D)
        H = m["heads"]
        if layer["type"] == "gla":
            mat(p + "mix.q", H * m["dim"], D)
            mat(p + "mix.k", H * m["dim"], D)
            mat(p + "mix.v", H * m["vdim"], D)
            mat(p + "mix.g", H * m["vdim"], D)
            mat(p + "mix.o", D, H * m["vdim"])
            vec(p + "mix.norm", m["vdim"], 1.0)
            mat(p + "mix.a1", decay_rank, D)
            mat(p + "mix.a2", H * m["dim"], decay_rank, gain=2.0)
            vec(p + "mix.a2.b", H * m["dim"], 1.0, 2.0)
        else:
            mat(p + "mix.q", H * (m["dim"] + m["rot_dim"]), D, gain=sharp)
            if m.get("kv_from") is None:
                mat(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], D, gain=sharp)
                vec(p + "mix.dkv.norm", m["kv_rank"], 1.0)
            mat(p + "mix.uk", H * m["dim"], m["kv_rank"], gain=sharp)
            mat(p + "mix.uv", H * m["vdim"], m["kv_rank"])
            mat(p + "mix.o", D, H * m["vdim"])
        if layer["mlp"]:
            mat(p + "mlp.up", layer["mlp"]["ff"], D)
            mat(p + "mlp.down", D, layer["mlp"]["ff"])
    return out


def write(folder, cfg, w):
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(folder / "model.safetensors"))
    return folder


# sizes of their own: every width a multiple of 8, so bf16 takes the tensor-core kernels
EVEN = config(320, 192, [(gla(3, 24, 40, 6.0), 160), (latent(5, 40, 24, 48, 96), None), (latent(2, 64, 24, 72, 96, kv_from=1), 224),
                         (gla(2, 72, 24, 1.0), None), (latent(3, 24, 8, 16, 56, base=3000.0, scaling=(16.0, 32, 4.0, 0.5)), 96)])
# no width a multiple of 8, single heads, no scaling, factor 1
ODD = config(203, 90, [(latent(1, 13, 6, 11, 37, scaling=None), 75), (gla(1, 21, 19, 3.0), 50),
                       (latent(3, 9, 6, 5, 37, kv_from=0, scaling=None), None),
                       (latent(2, 10, 2, 7, 20, scaling=(1.0, 16, 2.0, 1.0)), 30), (gla(3, 5, 6, 0.5), 33)], eps=1e-3, cap=3.0)
