"""Letitar on the GPU: every mechanism alone and whole models, against the plain double-precision oracle."""
import json
import os
import subprocess

import pytest
import torch

from omegalax_b200.models.mixers import TokenBatch
from omegalax_b200.models.paged_sequences import HybridCache, LatentPages
from omegalax_b200.models.rope_scaling import RotaryConfig, RotaryTable, YarnScaling
from omegalax_b200.ops import lib
from omegalax_b200.ops import serving as S
from omegalax_b200.text import api

from . import letitar_models as M
from . import letitar_oracle as O
from .serving_checks import BOTH, bf16, close, cu, done, f32, f64, gen, i32, logits_close, new_cache, prompt, rnd, run

pytestmark = pytest.mark.gpu

# ------------------------------------------------------------------------------------------ row ops
@BOTH
@pytest.mark.parametrize("D", [6, 90, 1000, 2052, 4096, 8192, 8200])
def test_layernorm_rows(dtype, D):
    x = torch.randn(3, D, generator=gen(D)) * 5 + 40         # a mean far from zero
    x[1] *= 1e-3
    w, b = rnd(1, D, dtype=dtype), rnd(2, D, dtype=dtype)
    y = S.layernorm_rows(cu(x), cu(w), cu(b), 1e-3)
    done()
    want = O.layer_norm(x.double(), w.double(), b.double(), 1e-3)
    for r in range(3):
        close(y[r], want[r], dtype, k=8)


@BOTH
@pytest.mark.parametrize("n", [3, 64, 1025])
def test_squared_relu_and_soft_cap(dtype, n):
    x = rnd(n, 5, n, dtype=dtype)
    close(S.relu_squared(cu(x)), torch.clamp(x.double(), min=0) ** 2, dtype)
    z = torch.randn(5, n, generator=gen(3)) * 50
    close(S.soft_cap_(cu(z), 7.5), O.soft_cap(z.double(), 7.5), f32)
    done()


@BOTH
@pytest.mark.parametrize("D", [18, 24, 1500])
def test_embedding_rows_and_bad_ids(dtype, D):
    t = rnd(0, 11, D, dtype=dtype)
    y = S.embed_rows(cu(torch.tensor([10, -1, 0], dtype=i32)), cu(t))
    done()
    assert torch.equal(y.cpu(), torch.stack([t[10].float(), torch.zeros(D), t[0].float()]))
    S.embed_rows(cu(torch.tensor([11], dtype=i32)), cu(t))     # outside the table: reported, nothing read
    with pytest.raises(lib.KernelError, match="status code 6"):
        lib.check_status()


@BOTH
@pytest.mark.parametrize("M_,N,K", [(1, 16, 8), (5, 90, 37), (130, 203, 90), (300, 256, 192)])
def test_project(dtype, M_, N, K):
    x, w = rnd(1, M_, K, dtype=dtype), rnd(2, N, K, dtype=dtype)
    want = x.double() @ w.double().t()
    close(S.project(cu(x), cu(w)), want, dtype)
    close(S.project(cu(x), cu(w), out_dtype=f32), want, f32)
    base = torch.randn(M_, N, generator=gen(3))
    into = cu(base.clone())
    S.project(cu(x), cu(w), into=into)
    close(into, base.double() + want, f32)
    done()


# ------------------------------------------------------------------------------------------ gated linear attention
def gla_inputs(seed, N, H, K, V, dtype, extra=8):
    proj = rnd(seed, N, 2 * H * (K + V) + extra, dtype=dtype)
    z = torch.randn(N, H * K, generator=gen(seed + 1)) * 4
    z[:, ::7] = -60.0          # almost forgotten at once unless tau is large
    z[:, 3::7] = 40.0          # never forgotten
    bias = rnd(seed + 2, H * K, dtype=dtype)
    return proj, z, bias


def gla_want(proj, z, bias, H, K, V, tau, state=None):
    p = proj.double()
    q, k = p[:, :H * K].view(-1, H, K) * K ** -0.5, p[:, H * K:2 * H * K].view(-1, H, K)
    v = p[:, 2 * H * K:2 * H * K + H * V].view(-1, H, V)
    alpha = O.gla_decay(z.double() + bias.double(), tau).view(-1, H, K)
    return O.gla_recurrence(q, k, v, alpha, state)


@BOTH
@pytest.mark.parametrize("H,K,V,tau", [(2, 32, 64, 16.0), (3, 20, 36, 1.0), (1, 72, 24, 0.25), (2, 128, 33, 5.0), (1, 200, 5, 300.0), (2, 200, 40, 4.0),
                                       (2, 128, 128, 1.0)])
def test_gla_scan_unequal_sequences_and_states(dtype, H, K, V, tau):
    lens = [19, 0, 1, 8, 40]
    B, N = len(lens), sum(lens)
    proj, z, bias = gla_inputs(5, N, H, K, V, dtype)
    hist = [0, 4, 7, 0, 3]
    state = torch.randn(B, H, K, V, generator=gen(9))
    st = cu(state.clone())
    c = torch.tensor([0] + lens).cumsum(0).to(i32)
    alpha = S.gla_decay_(cu(z.clone()), cu(bias), tau)
    o = S.gla_scan(cu(proj), alpha, st, cu(c), cu(torch.tensor(hist, dtype=i32)), H, K, V, K ** -0.5)
    done()
    close(alpha, O.gla_decay(z.double() + bias.double(), tau), f32)
    for b in range(B):
        a, e = int(c[b]), int(c[b + 1])
        if a == e:
            assert torch.equal(st[b].cpu(), state[b])
            continue
        want, S_end = gla_want(proj[a:e], z[a:e], bias, H, K, V, tau, state[b].double() if hist[b] else None)
        close(o[a:e], want, f32, k=4)
        close(st[b], S_end, f32, k=4)


@BOTH
@pytest.mark.parametrize("H,K,V,tau", [(2, 32, 64, 16.0), (3, 20, 36, 1.0), (1, 72, 33, 0.25), (2, 128, 128, 5.0), (1, 40, 300, 2.0)])
def test_gla_step_token_by_token(dtype, H, K, V, tau):
    T, eps = 9, 1e-3
    proj, z, bias = gla_inputs(15, T, H, K, V, dtype)
    w = rnd(4, V, dtype=dtype)
    st = torch.full((3, H, K, V), float("nan"), device="cuda")       # row 0 starts over whatever its slot holds
    st[2] = 1.5
    rows, close_rows = [], []
    for t in range(T):
        p3, z3 = proj[t].repeat(3, 1), z[t].repeat(3, 1)
        seen = torch.tensor([t + 1, 0, 100 + t], dtype=i32)
        y = S.gla_step(cu(p3), cu(z3), cu(bias), cu(w), st, cu(seen), H, K, V, K ** -0.5, tau, eps)
        rows.append(y[0])
        close_rows.append(y[2])
        assert float(y[1].abs().max()) == 0.0
    done()
    assert torch.isnan(st[1]).all()                                   # the idle row's state is untouched
    g = proj.double()[:, 2 * H * K + H * V:2 * H * (K + V)]
    for got, init in ((rows, None), (close_rows, torch.full((H, K, V), 1.5, dtype=f64))):
        o, end = gla_want(proj, z, bias, H, K, V, tau, init)
        want = O.rms_norm(o, w.double(), eps).reshape(T, H * V) * g * torch.sigmoid(g)
        close(torch.stack(got), want, dtype, k=4)
        close(st[0 if init is None else 2], end, f32, k=4)


@BOTH
@pytest.mark.parametrize("V,off", [(40, 5), (128, 8), (128, 3)])
def test_gla_norm_gate(dtype, V, off):
    H, N = 3, 6
    o, gate, w = torch.randn(N, H, V, generator=gen(1)), rnd(2, N, H * V + off, dtype=dtype), rnd(3, V, dtype=dtype)
    o[2] *= 1e-4                                                      # eps matters
    y = S.gla_norm_gate(cu(o), cu(gate)[:, off:], cu(w), 1e-5)
    done()
    g = gate.double()[:, off:]
    close(y, O.rms_norm(o.double(), w.double(), 1e-5).reshape(N, -1) * g * torch.sigmoid(g), dtype)


# ------------------------------------------------------------------------------------------ latent attention
@BOTH
@pytest.mark.parametrize("rot_dims", [16, 10])
def test_latent_prepare_rotates_norms_and_stores(dtype, rot_dims):
    H, dim, rot, rank, N = 3, 24, 16, 37, 5
    cfg = RotaryConfig(rot_dims, 100.0, YarnScaling(4.0, 64, 8.0, 1.0))
    cos, sin = RotaryTable(cfg).get(3000, torch.device("cuda", 0))
    proj = rnd(1, N, H * (dim + rot) + rank + rot + 3, dtype=dtype)
    w = rnd(2, rank, dtype=dtype)
    pos = torch.tensor([0, 1, 2999, -1, 77], dtype=i32)
    row = torch.tensor([4, 0, 9, -1, 2], dtype=i32)
    cache, packed = torch.zeros(10, 56, dtype=dtype, device="cuda"), torch.zeros(N, 56, dtype=dtype, device="cuda")
    got = cu(proj.clone())
    S.latent_prepare(got, cu(pos), cu(row), cos, sin, H, dim, rot, rank, dkv_off=H * (dim + rot), norm_w=cu(w), cache=cache,
                     eps=1e-5, packed=packed)
    done()
    r = {"dims": rot_dims, "base": 100.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    q = proj.double()[:, :H * (dim + rot)].view(N, H, dim + rot)
    d = proj.double()[:, H * (dim + rot):H * (dim + rot) + rank + rot]
    q_want = torch.cat([q[..., :dim], O.rotate_interleaved(q[..., dim:], pos, r)], -1)
    c_want = O.rms_norm(d[:, :rank], w.double(), 1e-5)
    k_want = O.rotate_interleaved(d[:, rank:], pos, r)
    for n in range(N):
        if pos[n] < 0:
            assert torch.equal(got[n].cpu(), proj[n]) and float(packed[n].abs().max()) == 0
            continue
        close(got[n, :H * (dim + rot)], q_want[n].reshape(-1), dtype)
        for buf in (cache[row[n]], packed[n]):
            close(buf[:rank], c_want[n], dtype)
            close(buf[rank:rank + rot], k_want[n], dtype)
    untouched = [i for i in range(10) if i not in row.tolist()]
    assert float(cache[untouched].abs().max()) == 0
    S.latent_prepare(got, cu(pos), cu(torch.full((N,), 10, dtype=i32)), cos, sin, H, dim, rot, rank, dkv_off=H * (dim + rot),
                     norm_w=cu(w), cache=cache, eps=1e-5)            # a row outside the cache: reported, not written
    with pytest.raises(lib.KernelError, match="status code 6"):
        lib.check_status()


@pytest.mark.parametrize("H,d1,d2,vdim", [(2, 64, 64, 64), (3, 128, 64, 128), (2, 32, 16, 40), (1, 8, 8, 8), (2, 40, 24, 72),
                                          (2, 136, 8, 64), (2, 192, 64, 128), (2, 96, 32, 48)])
def test_two_part_attention_on_packed_prompts(H, d1, d2, vdim):
    lens = [1, 257, 64, 0, 130]
    N, scale = sum(lens), 0.9 * (d1 + d2) ** -0.5
    q, k2 = rnd(1, N, H * (d1 + d2)), rnd(3, N, d2 + 8)[:, 8:]
    kv = rnd(2, N, H * (d1 + vdim))
    c = torch.tensor([0] + lens).cumsum(0).to(i32)
    # query 200 of the long sequence wants key 3, far away, and nothing else
    a = int(c[1])
    q = q.view(N, H, d1 + d2)
    q[a + 200] = torch.cat([kv[a + 3, :H * d1].view(H, d1), k2[a + 3].expand(H, d2)], -1) * 6
    q = q.reshape(N, -1)
    kvc, k2c = cu(kv), cu(rnd(3, N, d2 + 8))[:, 8:]
    y = S.attn_two_part(cu(q), kvc, k2c, kvc[:, H * d1:], cu(c), max(lens), H, d1, d2, vdim, scale)
    done()
    for b in range(len(lens)):
        a, e = int(c[b]), int(c[b + 1])
        if a == e:
            continue
        k = torch.cat([kv[a:e, :H * d1].view(-1, H, d1), k2[a:e, None].expand(-1, H, d2)], -1)
        want = O.causal_softmax_attention(q[a:e].double().view(-1, H, d1 + d2), k.double(), kv[a:e, H * d1:].double().view(-1, H, vdim), scale)
        close(y[a:e], want.reshape(e - a, -1), bf16)


def latent_setup(seed, lens, H, dim, rot, rank, page_size, dtype):
    """Scattered pages with cached rows of each sequence, and one query per sequence."""
    cache = HybridCache([LatentPages(rank, rot)], len(lens), max(lens) + page_size, page_size=page_size, dtype=dtype, device="cuda",
                        num_pages=sum(-(-n // page_size) for n in lens) + 3)
    order = torch.randperm(cache.num_pages, generator=gen(seed)).tolist()
    cache.allocator.free = order
    cache.reserve(lens)
    store = torch.full((cache.num_pages * page_size, cache.stores[0].shape[1]), float("nan")).to(dtype)   # nothing else may be read
    rows = [rnd(seed + b, n, rank + rot, dtype=dtype) for b, n in enumerate(lens)]
    return cache, store, rows


@BOTH
@pytest.mark.parametrize("H,dim,rot,rank,page", [(3, 24, 16, 64, 8), (16, 16, 64, 512, 64), (32, 8, 64, 512, 16), (40, 16, 16, 96, 64),
                                                 (5, 40, 24, 200, 4), (2, 8, 8, 320, 8), (17, 16, 40, 136, 32)])
def test_latent_decode_over_scattered_pages(dtype, H, dim, rot, rank, page):
    lens = [1, page, page + 1, 63, 64, 65, 0, 700]
    B, scale = len(lens), 0.2
    cache, store, rows = latent_setup(3, lens, H, dim, rot, rank, page, dtype)
    for b, n in enumerate(lens):
        if n:
            store[cache.flat_rows_host(b, 0, n).long(), :rank + rot] = rows[b]
    store = cu(store)
    # pages are NaN outside the stored rows; the tensor-core kernel multiplies whole tiles but reads visible rows only
    q = rnd(77, B, H * (dim + rot), dtype=dtype)
    q_lat = rnd(78, B, H, rank, dtype=dtype)
    far = rows[7][5]                                                   # the long sequence's head 0 wants its sixth key
    q_lat[7, 0] = far[:rank] * (60.0 / float(far.double().pow(2).sum()) / scale)
    seen = cu(torch.tensor(lens, dtype=i32))
    outs = [S.latent_attn_any(cu(q_lat.float()), cu(q), dim + rot, dim, rot, store, cu(torch.arange(B, dtype=i32)), seen, cache.block_table, page, scale)]
    if S.latent_decode_fits(dtype, dim, rot, rank):
        for splits in (None, 1, 3, 11):
            outs.append(S.latent_decode(cu(q_lat), cu(q), dim + rot, dim, rot, store, seen, cache.block_table, page, scale, splits=splits))
    else:
        assert dtype == f32
    done()
    for b, n in enumerate(lens):
        if n == 0:
            assert all(float(o[b].abs().max()) == 0 for o in outs)
            continue
        r = rows[b].double()
        s = torch.einsum("hr,sr->hs", q_lat[b].double(), r[:, :rank])
        s = (s + torch.einsum("hd,sd->hs", q[b].double().view(H, dim + rot)[:, dim:], r[:, rank:])) * scale
        want = torch.softmax(s, -1) @ r[:, :rank]
        close(outs[0][b], want, f32, k=4)
        for o in outs[1:]:
            close(o[b], want, bf16)


@BOTH
def test_latent_absorb_and_expand(dtype):
    N, H, dim, rot, rank, vdim = 11, 3, 24, 8, 200, 20
    q, uk, uv = rnd(1, N, H * (dim + rot), dtype=dtype), rnd(2, H * dim, rank, dtype=dtype), rnd(3, H * vdim, rank, dtype=dtype)
    want = torch.einsum("nhd,hdr->nhr", q.double().view(N, H, -1)[..., :dim], uk.double().view(H, dim, rank))
    close(S.latent_absorb(cu(q), dim + rot, cu(uk), H, dim, rank, f32), want, f32)
    o = torch.randn(N, H, rank, generator=gen(4))
    want = torch.einsum("nhr,hvr->nhv", o.double(), uv.double().view(H, vdim, rank)).reshape(N, -1)
    close(S.latent_expand(cu(o), cu(uv), vdim), want, dtype)
    done()


# ------------------------------------------------------------------------------------------ whole models
MODELS = {"even": (M.EVEN, 8), "odd": (M.ODD, 5)}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    cache = {}

    def get(name, dtype):
        if (name, dtype) not in cache:
            cfg, rank = MODELS[name]
            w = M.weights(cfg, 11, decay_rank=rank)
            folder = M.write(tmp_path_factory.mktemp(name), cfg, w)
            cache[name, dtype] = api.load_model(folder, device=torch.device("cuda", 0), dtype=dtype) + (w, folder)
        return cache[name, dtype]
    return get


ALL = pytest.mark.parametrize("name", list(MODELS))


@BOTH
@ALL
def test_layers_and_logits_of_a_prompt(models, name, dtype):
    model, cfg, w, folder = models(name, dtype)
    toks = prompt(1, 70, cfg.vocab_size)
    want, residual, states = O.run(MODELS[name][0], w, toks)
    cache = new_cache(model, cfg, 1, 80)
    cache.reserve([70])
    seen = {}
    model.run_layers(TokenBatch.build(cache, [torch.tensor(toks, dtype=i32)]), cache, after_layer=lambda i, x: seen.__setitem__(i, x.clone()))
    done()
    for i in range(cfg.num_layers):
        assert seen[i].dtype == f32
        logits_close(seen[i].cpu(), residual[i], dtype)
    for i, s in states.items():
        close(cache.stores[i][0], s, dtype, k=4)
    logits_close(run(model, cfg, new_cache(model, cfg, 1, 80), [toks])[0], want, dtype)
    hidden, aux = api.forward(model, torch.tensor([toks[:5] + [-1] * 2, toks[:7]], dtype=i32), -1, cfg)
    assert hidden.shape == (2, 7, cfg.width) and float(aux) == 0 and float(hidden[0, 5:].abs().max()) == 0
    logits_close(model.logits(hidden[1]).cpu(), want[:7], dtype)


@BOTH
@ALL
@pytest.mark.parametrize("first", [1, 7, 8, 30])
def test_decoding_token_by_token(models, name, dtype, first):
    """Prompts that end around a page border, then one token at a time (recorded steps after the second)."""
    model, cfg, w, _ = models(name, dtype)
    toks = prompt(2, 70, cfg.vocab_size)
    want, _, _ = O.run(MODELS[name][0], w, toks)
    cache = new_cache(model, cfg, 1, 70)
    got = run(model, cfg, cache, [toks[:first]])
    for t in toks[first:]:
        got += run(model, cfg, cache, [[t]])
    assert cache.decode_graph[1] is not None
    logits_close(torch.cat(got), want, dtype)


@BOTH
@ALL
@pytest.mark.parametrize("portion", [2, 3, 16, 33])
def test_portions_of_a_prompt(models, name, dtype, portion):
    model, cfg, w, _ = models(name, dtype)
    toks = prompt(3, 67, cfg.vocab_size)
    want, _, _ = O.run(MODELS[name][0], w, toks)
    cache, got = new_cache(model, cfg, 1, 70), []
    for at in range(0, len(toks), portion):
        got += run(model, cfg, cache, [toks[at:at + portion]])
    logits_close(torch.cat(got), want, dtype)


@BOTH
@ALL
def test_unequal_batch_freed_slots_and_pages(models, name, dtype):
    """A batch of four, some ending early; their rows and pages serve other requests while the rest go on."""
    model, cfg, w, _ = models(name, dtype)
    lens, tail = [1, 40, 17, 8], 12
    toks = [prompt(20 + b, n + tail, cfg.vocab_size) for b, n in enumerate(lens)]
    want = [O.run(MODELS[name][0], w, t)[0] for t in toks]
    cache = new_cache(model, cfg, 4, 64, num_pages=20)
    got = [[x] for x in run(model, cfg, cache, [t[:n] for t, n in zip(toks, lens)])]
    for i in range(tail):
        live = [b for b in range(4) if not (b == 1 and i >= 3) and not (b == 3 and i >= 6)]
        out = run(model, cfg, cache, [[toks[b][lens[b] + i]] if b in live else [] for b in range(4)])
        for b in live:
            got[b].append(out[b])
        if i == 2:
            cache.free_sequence(1)
        if i == 5:
            cache.free_sequence(3)
            again = run(model, cfg, cache, [[], toks[2][:29], [], []])[1]      # a new request in a used row and used pages
            logits_close(again, want[2][:29], dtype)
            cache.free_sequence(1)
    for b, n in enumerate([tail, 3, tail, 6]):
        logits_close(torch.cat(got[b]), want[b][:lens[b] + n], dtype)
    # mixed: one row goes on by one token while another starts a prompt
    out = run(model, cfg, cache, [[], toks[1][:9], [], [toks[3][0]]])
    logits_close(out[1], want[1][:9], dtype)
    logits_close(out[3], want[3][:1], dtype)


@BOTH
def test_long_decoding_keeps_to_the_oracle(models, dtype):
    model, cfg, w, _ = models("even", dtype)
    toks = prompt(5, 230, cfg.vocab_size)
    want, _, _ = O.run(M.EVEN, w, toks)
    cache = new_cache(model, cfg, 2, 256, page_size=64)
    got = run(model, cfg, cache, [toks[:10], toks[:3]])[:1]
    for t in toks[10:]:
        got.append(run(model, cfg, cache, [[t], []])[0])
    logits_close(torch.cat(got), want, dtype)
    assert cache.seq_lens_host == [230, 3]


@BOTH
def test_recorded_steps_equal_eager_ones(models, dtype, monkeypatch):
    model, cfg, _, _ = models("even", dtype)
    toks = prompt(6, 20, cfg.vocab_size)
    outs = []
    for on in ("1", "0"):
        monkeypatch.setenv("OMEGALAX_B200_DECODE_GRAPH", on)
        cache = new_cache(model, cfg, 2, 32)
        got = run(model, cfg, cache, [toks[:4], toks[:9]])
        for t in toks[9:]:
            got += run(model, cfg, cache, [[t], [t]])
        outs.append(torch.cat(got))
    assert (cache.decode_graph is None) and torch.allclose(outs[0], outs[1], rtol=0, atol=1e-4 if dtype == f32 else 0.25)


@ALL
def test_greedy_generation(models, name):
    model, cfg, w, _ = models(name, f32)
    prompts = [prompt(30 + i, n, cfg.vocab_size) for i, n in enumerate((9, 1, 33))]
    out = api.generate(model, cfg, prompts, 10)
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(10):
            seq.append(int(O.run(MODELS[name][0], w, seq)[0][-1].argmax()))
        want.append(seq[len(p):])
    assert out == want
    eos = want[0][4]
    stopped = api.generate(model, cfg, prompts, 10, eos_id=eos)
    assert stopped == [s[:s.index(eos) + 1] if eos in s else s for s in want]
    model16, _, _, _ = models(name, bf16)
    out16 = api.generate(model16, cfg, prompts, 4)
    assert [len(o) for o in out16] == [4, 4, 4] and all(0 <= t < cfg.vocab_size for o in out16 for t in o)


@BOTH
def test_trace_runner_program(models, dtype, tmp_path):
    _, cfg, w, folder = models("odd", dtype)
    toks = {"a": prompt(40, 14, cfg.vocab_size), "b": prompt(41, 6, cfg.vocab_size)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks["a"][:12], "want": [11, 3]}, {"id": "b", "tokens": toks["b"][:4], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": toks["b"][4:5], "want": []}, {"id": "a", "tokens": toks["a"][12:13], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": toks["b"][5:6], "want": [0]}, {"id": "a", "tokens": toks["a"][13:14], "want": [0]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": toks["a"], "want": [13]}], "end": ["c"]}]
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    r = subprocess.run([exe, "--model", str(folder), "--dtype", "float32" if dtype == f32 else "bfloat16", "--out", str(tmp_path), "--max-tokens", "24"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    want = {k: O.run(M.ODD, w, t)[0] for k, t in toks.items()}
    assert not (tmp_path / "1.f32").exists()
    for step, rows in ((0, [("a", 11), ("a", 3)]), (2, [("b", 5), ("a", 13)]), (3, [("a", 13)])):
        got = torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=f32).view(len(rows), cfg.vocab_size)
        for g, (k, p) in zip(got, rows):
            logits_close(g[None], want[k][p][None], dtype)


def test_trace_runner_and_generate_on_the_other_text_family(tmp_path):
    """The same entry points serve a Qwen3 model through its paged cache."""
    import dataclasses

    from omegalax_b200 import export
    from omegalax_b200.text import trace

    cfg = dataclasses.replace(api.resolve_config("qwen3-smoke"), head_dim=128, num_kv_heads=2, vocab_size=264)
    model, cfg = api.init_model(cfg, 0, tp_size=1, fsdp_size=1, dp_size=1, device="cuda", dtype=bf16)
    export.export_model_to_hf(model, cfg, tmp_path)
    model, cfg = api.load_model(tmp_path, device=torch.device("cuda", 0))
    toks = prompt(1, 30, 264)
    r = trace.TraceRunner(model, cfg, 64)
    got = r.step([{"id": "a", "tokens": toks[:29], "want": [28, 4]}, {"id": "b", "tokens": toks[:5], "want": [4]}], ["b"])
    last = r.step([{"id": "a", "tokens": toks[29:], "want": [0]}], ["a"])
    done()
    assert got.shape == (3, 264) and torch.allclose(got[1], got[2], atol=0.06) and torch.isfinite(last).all()
    out = api.generate(model, cfg, [toks, toks[:3]], 5)
    assert [len(o) for o in out] == [5, 5]
