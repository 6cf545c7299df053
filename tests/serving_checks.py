"""Helpers of the GPU tests of the serving decoders."""
import pytest
import torch

from omegalax_b200.ops import lib
from omegalax_b200.text import api

bf16, f32, f64, i32 = torch.bfloat16, torch.float32, torch.float64, torch.int32
BOTH = pytest.mark.parametrize("dtype", [f32, bf16], ids=["fp32", "bf16"])


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(seed, *shape, dtype=bf16):
    """Values that bf16 holds exactly, so the oracle and both kernel types see the same numbers."""
    return torch.randn(*shape, generator=gen(seed)).bfloat16().to(dtype)


def cu(t):
    return t.cuda()


def done():
    torch.cuda.synchronize()
    lib.check_status()


def close(got, want, dtype, k=1.0):
    """Relative to the tensor's scale: fp32 rounding, or a bf16 rounding or two."""
    got, want = got.double().cpu(), want.double().cpu()
    scale = want.abs().max().clamp_min(1e-9)
    err = float((got - want).abs().max() / scale)
    tol = (4e-6 if dtype == f32 else 1.2e-2) * k
    assert err < tol, (err, tol)


def prompt(seed, n, vocab):
    return torch.randint(0, vocab, (n,), generator=gen(seed)).tolist()


def run(model, cfg, cache, rows):
    """Logits of every new token of ``rows`` (one list per sequence, possibly empty), per sequence."""
    ids = api.batch_rows(rows, cache.B)
    logits, _, _ = api.decode(model, cache, ids, api.NO_TOKEN, cfg, select=ids >= 0)
    done()
    return list(logits.cpu().split([len(r) for r in rows]))


def new_cache(model, cfg, B, tokens, page_size=8, **kw):
    w = next(model.parameters())
    return api.make_cache(cfg, B, tokens, 0, dtype=w.dtype, device=w.device, page_size=page_size, **kw)


def logits_close(got, want, dtype):
    want = want.double()
    err = (got.detach().double() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    tol = 3e-5 if dtype == f32 else 0.06
    assert float(err.max()) < tol, (float(err.max()), int(err.argmax()), tol)
