"""Difedra on the GPU: every mechanism alone and whole models, against the plain double-precision oracle."""
import json
import os
import subprocess

import pytest
import torch

from omegalax_b200.models.mixers import TokenBatch
from omegalax_b200.models.paged_sequences import HybridCache, KeyValuePages
from omegalax_b200.models.rope_scaling import RotaryConfig, RotaryTable, WavelengthScaling
from omegalax_b200.ops import lib
from omegalax_b200.ops import serving as S
from omegalax_b200.text import api

from . import difedra_models as M
from . import difedra_oracle as O
from .serving_checks import BOTH, bf16, close, cu, done, f32, gen, i32, logits_close, new_cache, prompt, rnd, run

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------------------------------ row ops
@BOTH
@pytest.mark.parametrize("D", [6, 90, 1000, 2052, 4096, 8192, 8200])
def test_rms_rows(dtype, D):
    x = torch.randn(3, D, generator=gen(D)) * 5 + 4
    x[1] *= 1e-3                                              # eps matters
    w = rnd(1, D, dtype=dtype)
    y = S.rms_rows(cu(x), cu(w), 1e-3)
    done()
    want = O.rms_norm(x.double(), w.double(), 1e-3)
    for r in range(3):
        close(y[r], want[r], dtype)


@BOTH
@pytest.mark.parametrize("act", ["silu", "gelu_tanh"])
@pytest.mark.parametrize("F", [5, 40, 1033, 768])
def test_gated_activations(dtype, act, F):
    gu = rnd(F, 9, 2 * F, dtype=dtype) * 3
    gu[0, :2] = torch.tensor([60.0, -60.0])                   # saturated on both sides
    fn = O.silu if act == "silu" else O.gelu_tanh
    y = S.gated_act(cu(gu), act)
    g, u = gu.double()[:, :F], gu.double()[:, F:]
    close(y, fn(g) * u, dtype)
    some = S.gated_act(cu(gu), act, cu(torch.tensor([4], dtype=i32)))
    done()
    assert torch.equal(some[:4], y[:4])


# ------------------------------------------------------------------------------------------ preparation of q, k, v
@BOTH
@pytest.mark.parametrize("H,G,dim,vdim,rot_dims,mix", [(3, 1, 32, 24, 32, 0.25), (4, 2, 48, 16, 16, None), (5, 5, 14, 9, 6, 0.7), (2, 1, 40, 8, 40, 1.0),
                                                      (32, 4, 128, 128, 128, -0.5), (64, 8, 128, 64, 64, None), (1, 1, 8, 8, 2, 0.0)])
def test_prepare_norms_rotates_mixes_and_stores(dtype, H, G, dim, vdim, rot_dims, mix):
    N, pitch, eps = 5, G * (dim + vdim) + (-G * (dim + vdim)) % 8, 1e-2
    scaling = dict(factor=4.0, low=1.0, high=4.0, original=64)
    cos, sin = RotaryTable(RotaryConfig(rot_dims, 100.0, WavelengthScaling(**scaling))).get(3000, torch.device("cuda", 0))
    at_v = (H + G) * dim
    proj = rnd(1, N, at_v + G * vdim, dtype=dtype)
    proj[1, :at_v] *= 0.05                                     # eps matters
    proj[2, :dim] *= 8                                         # one head carries the norm of all
    w, first = rnd(2, at_v, dtype=dtype), rnd(3, N, G * vdim + 8, dtype=dtype)
    lam = None if mix is None else torch.tensor(mix).to(dtype)
    pos = torch.tensor([0, 1, 2999, -1, 77], dtype=i32)
    row = torch.tensor([4, 0, 9, -1, 2], dtype=i32)
    cache, got = torch.zeros(10, pitch, dtype=dtype, device="cuda"), cu(proj.clone())
    S.window_prepare(got, cu(pos), cu(row), cos, sin, H, G, dim, vdim, cu(w), cache, eps, mix=None if mix is None else cu(lam),
                     v_first=None if mix is None else cu(first)[:, 8:])
    done()
    p, rot = proj.double(), {"dims": rot_dims, "base": 100.0, "scaling": scaling}
    q = O.rotate_half(O.rms_norm(p[:, :H * dim], w.double()[:H * dim], eps).view(N, H, dim), pos, rot)
    k = O.rotate_half(O.rms_norm(p[:, H * dim:at_v], w.double()[H * dim:], eps).view(N, G, dim), pos, rot)
    v = p[:, at_v:].view(N, G, vdim)
    if mix is not None:
        v = (1 - lam.double()) * v + lam.double() * first.double()[:, 8:].view(N, G, vdim)
    for n in range(N):
        if pos[n] < 0:
            assert torch.equal(got[n].cpu(), proj[n])
            continue
        close(got[n, :H * dim], q[n].reshape(-1), dtype)
        close(got[n, H * dim:at_v], k[n].reshape(-1), dtype)
        close(got[n, at_v:], v[n].reshape(-1), dtype)
        heads = cache[row[n], :G * (dim + vdim)].view(G, vdim + dim)
        assert torch.equal(heads[:, :vdim], got[n, at_v:].view(G, vdim)) and torch.equal(heads[:, vdim:], got[n, H * dim:at_v].view(G, dim))
    untouched = [i for i in range(10) if i not in row.tolist()]
    assert float(cache[untouched].abs().max()) == 0
    # a row outside the cache: reported, not written
    S.window_prepare(got, cu(pos), cu(torch.full((N,), 10, dtype=i32)), cos, sin, H, G, dim, vdim, cu(w), cache, eps)
    with pytest.raises(lib.KernelError, match="status code 6"):
        lib.check_status()


# ------------------------------------------------------------------------------------------ attention
def seek(q, t, h, k, j, rep, scale, score=14.0):
    """Make query (t, h) want key j: its score is ``score``."""
    key = k[j, h // rep].double()
    q[t, h] = (key * (score / scale / float(key.pow(2).sum()))).to(q.dtype)


@pytest.mark.parametrize("H,G,dim,vdim", [(2, 2, 64, 64), (4, 1, 96, 48), (6, 2, 128, 128), (3, 1, 192, 128), (2, 1, 256, 64), (2, 1, 40, 72), (1, 1, 8, 8),
                                          (4, 2, 256, 128), (10, 5, 24, 128)])
@pytest.mark.parametrize("window", [1, 40, 128, 129, 200, 0, 1000])
def test_window_attention_on_packed_prompts(H, G, dim, vdim, window):
    lens = [1, 300, 64, 0, 129, 520]
    N, scale, rep = sum(lens), 0.9 * dim ** -0.5, H // G
    c = torch.tensor([0] + lens).cumsum(0).to(i32)
    q, k, v = rnd(1, N, H, dim), rnd(2, N, G, dim), rnd(3, N, G, vdim)
    sink = (rnd(4, H) * 2 + 1).bfloat16()
    sink[0] = 9.0                                              # the strongest of most rows
    for b, T in enumerate(lens):                               # queries that want the last key they see, and the next one
        a = int(c[b])
        for t in {T - 1, T - 2, T // 2, 127, 128, 255, 256, 299}:
            if not 0 <= t < T:
                continue
            edge = t - window + 1 if window else 0
            for h in range(H):
                j = edge if h % 2 else edge - 1
                if 0 <= j:
                    seek(q[a:], t, h, k[a:], j, rep, scale)
    proj = cu(torch.cat([q.reshape(N, -1), k.reshape(N, -1), v.reshape(N, -1)], 1))
    at_k, at_v = H * dim, (H + G) * dim
    for s in (sink, None):
        y = S.attn_window(proj[:, :at_k], proj[:, at_k:], proj[:, at_v:], cu(c), max(lens), H, G, dim, vdim, scale, window,
                          None if s is None else cu(s))
        done()
        for b in range(len(lens)):
            a, e = int(c[b]), int(c[b + 1])
            if a < e:
                want = banded(q[a:e], k[a:e], v[a:e], scale, window, s)
                close(y[a:e], want.reshape(e - a, -1), bf16)


def banded(q, k, v, scale, window, sink):
    """All queries of a sequence at once (the oracle's own form, one query at a time, agrees: see below)."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    k, v = k.double().repeat_interleave(rep, 1), v.double().repeat_interleave(rep, 1)
    s = torch.einsum("thd,shd->hts", q.double(), k) * scale
    gap = torch.arange(T)[:, None] - torch.arange(T)[None]
    s = s.masked_fill((gap < 0) | (gap >= window if window else torch.zeros_like(gap, dtype=torch.bool)), float("-inf"))
    extra = torch.full((H, T, 1), float("-inf"), dtype=s.dtype) if sink is None else sink.double().view(H, 1, 1).expand(H, T, 1)
    p = torch.softmax(torch.cat([s, extra], -1), -1)[..., :-1]
    return torch.einsum("hts,shv->thv", p, v)


def test_the_two_plain_forms_of_attention_agree():
    q, k, v, sink = rnd(1, 30, 6, 8), rnd(2, 30, 2, 8), rnd(3, 30, 2, 5), rnd(4, 6)
    for window in (0, 1, 7, 30, 50):
        for s in (sink, None):
            want = O.window_attention(q.double(), k.double(), v.double(), 0.4, window, None if s is None else s.double())
            assert torch.allclose(banded(q, k, v, 0.4, window, s), want, atol=1e-12)


@BOTH
@pytest.mark.parametrize("H,G,dim,vdim,page,window", [(3, 1, 24, 64, 8, 20), (16, 1, 64, 48, 64, 64), (32, 4, 128, 128, 16, 300), (40, 1, 16, 96, 64, 65),
                                                      (6, 2, 40, 24, 4, 1), (34, 2, 8, 8, 8, 0), (8, 8, 72, 320, 32, 128), (5, 5, 14, 9, 8, 11),
                                                      (4, 2, 256, 128, 64, 1000), (6, 3, 200, 512, 16, 63)])
def test_decode_over_scattered_pages(dtype, H, G, dim, vdim, page, window):
    lens = [1, page, page + 1, 63, 64, 65, 0, 700]
    B, scale, rep = len(lens), 1.1 * dim ** -0.5, H // G
    spec = KeyValuePages(G, dim, vdim, window)
    cache = HybridCache([spec], B, max(lens) + page, page_size=page, dtype=dtype, device="cuda", num_pages=sum(-(-n // page) for n in lens) + 3)
    cache.allocator.free = torch.randperm(cache.num_pages, generator=gen(3)).tolist()
    cache.reserve(lens)
    store = torch.full((cache.num_pages * page, spec.pitch), float("nan")).to(dtype)        # nothing but visible rows may be read
    q, sink = rnd(77, B, H, dim, dtype=dtype), (rnd(78, H) * 2).to(dtype)
    ks, vs = [rnd(10 + b, n, G, dim, dtype=dtype) for b, n in enumerate(lens)], [rnd(30 + b, n, G, vdim, dtype=dtype) for b, n in enumerate(lens)]
    for b, n in enumerate(lens):
        lo = max(0, n - window) if window else 0
        if n:
            store[cache.flat_rows_host(b, lo, n - lo).long(), :G * (dim + vdim)] = torch.cat([vs[b], ks[b]], -1)[lo:].reshape(n - lo, -1)
            seek(q[b:b + 1], 0, 0, ks[b], lo, rep, scale)      # the oldest visible key,
        if lo:
            seek(q[b:b + 1], 0, H - 1, ks[b], lo - 1, rep, scale)      # and one that is just out of sight
    qc, store, seen = cu(q.reshape(B, -1)), cu(store), cu(torch.tensor(lens, dtype=i32))
    sizes = (H, G, dim, vdim, scale, window)
    for s in (sink, None):
        sk = None if s is None else cu(s)
        outs = [S.window_attn_any(qc, store, cu(torch.arange(B, dtype=i32)), seen, cache.block_table, page, *sizes, sk)]
        if S.window_decode_fits(dtype, dim, vdim):
            outs += [S.window_decode(qc, store, seen, cache.block_table, page, *sizes, sk, splits=n) for n in (None, 1, 3, 11)]
        else:
            assert dtype == f32 or dim % 8 or vdim % 8 or dim + vdim > 640
        done()
        for b, n in enumerate(lens):
            if n == 0:
                assert all(float(o[b].abs().max()) == 0 for o in outs)
                continue
            full = torch.zeros(n, H, dim, dtype=dtype)
            full[-1] = q[b]
            want = banded(full, ks[b], vs[b], scale, window, s)[-1].reshape(-1)
            for o in outs:
                close(o[b], want, dtype, k=2)


def test_a_sink_far_above_every_score_silences_the_head():
    """No overflow on the way, in any of the kernels."""
    T, H, d = 150, 2, 64
    proj = rnd(1, T, 3 * H * d)
    sink = torch.tensor([300.0, -300.0]).bfloat16()
    c = torch.tensor([0, T], dtype=i32)
    y = S.attn_window(cu(proj)[:, :H * d], cu(proj)[:, H * d:], cu(proj)[:, 2 * H * d:], cu(c), T, H, H, d, d, 0.125, 40, cu(sink))
    q, k, v = (proj[:, i * H * d:(i + 1) * H * d].view(T, H, d) for i in range(3))
    close(y, banded(q, k, v, 0.125, 40, sink).reshape(T, -1), bf16)
    assert float(y[:, :d].abs().max()) == 0 and torch.isfinite(y).all()
    store = cu(torch.cat([v, k], -1).reshape(T, -1))
    table = torch.arange(3, dtype=i32, device="cuda")[None]
    store = torch.cat([store, torch.zeros(192 - T, store.shape[1], dtype=bf16, device="cuda")]).contiguous()
    for splits in (1, 2):
        o = S.window_decode(cu(proj)[T - 1:, :H * d], store, cu(torch.tensor([T], dtype=i32)), table, 64, H, H, d, d, 0.125, 0, cu(sink), splits=splits)
        close(o, banded(q, k, v, 0.125, 0, sink)[-1].reshape(1, -1), bf16)
    done()


# ------------------------------------------------------------------------------------------ routed experts
@pytest.mark.parametrize("E,top", [(1, 1), (5, 2), (12, 12), (33, 1), (64, 3), (128, 8), (511, 16)])
def test_router_takes_the_largest_and_weighs_by_sigmoid(E, top):
    z = torch.randn(40, E + 3, generator=gen(E)) * 3
    z[0] *= 20                                                 # scores that round to 1 still rank by their logits
    z[1, :] = 0.5                                              # a tie goes to the lower ids
    w, idx = S.route_sigmoid(cu(z)[:, :E], top)
    done()
    ids, weight = O.route(z[:, :E].double(), top)
    assert torch.equal(idx[1].cpu(), torch.arange(top, dtype=i32))
    best = torch.topk(z[:, :E], top, -1).values
    assert torch.equal(torch.gather(z[:, :E], 1, idx.cpu().long())[2:], best[2:]) and torch.equal(idx.cpu()[2:].long(), ids[2:])
    assert torch.equal(torch.gather(z[:, :E], 1, idx.cpu().long())[0], best[0])
    close(w, torch.sigmoid(best.double()), f32)


@BOTH
@pytest.mark.parametrize("M_,E,k,D,F", [(1, 4, 1, 64, 32), (37, 5, 3, 96, 72), (3, 7, 7, 200, 40), (40, 6, 2, 90, 33), (300, 3, 2, 128, 136), (700, 2, 1, 64, 264),
                                        (19, 1, 1, 1032, 520), (2, 130, 4, 48, 16)])
def test_experts_on_every_path(dtype, M_, E, k, D, F):
    h = rnd(1, M_, D, dtype=dtype)
    gu, down = (rnd(2, E, 2 * F, D, dtype=dtype) * (2 * D ** -0.5)).bfloat16().to(dtype), (rnd(3, E, D, F, dtype=dtype) * F ** -0.5).bfloat16().to(dtype)
    idx = torch.stack([torch.randperm(E, generator=gen(100 + m))[:k] for m in range(M_)]).to(i32)
    if E > 2:                                                  # one expert serves most tokens, another none
        idx = torch.where(idx == E - 1, torch.where((idx == 0).any(-1, keepdim=True), E - 1, 0).to(i32), idx) if k == 1 else idx
    w = torch.rand(M_, k, generator=gen(5)) * 0.9 + 0.1
    base = torch.randn(M_, D, generator=gen(6))
    want = base.double().clone()
    for m in range(M_):
        for e, a in zip(idx[m].tolist(), w[m].double()):
            x = a * h[m].double()
            want[m] += (O.silu(gu[e, :F].double() @ x) * (gu[e, F:].double() @ x)) @ down[e].double().t()
    paths = [False] + ([True] if S.experts_few_fits(bf16, 1, E, D, F) and dtype == bf16 and M_ * k <= S.FEW_PAIRS else [])
    for few in paths + [None]:
        into = cu(base.clone())
        S.experts_into(cu(h), cu(w), cu(idx), cu(gu), cu(down), "silu", into, few=few)
        done()
        close(into - cu(base), want - base.double(), dtype, k=2)


# ------------------------------------------------------------------------------------------ whole models
MODELS = {"even": M.EVEN, "odd": M.ODD}
ALL = pytest.mark.parametrize("name", list(MODELS))


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    cache = {}

    def get(name, dtype):
        if (name, dtype) not in cache:
            w = M.weights(MODELS[name], 11)
            folder = M.write(tmp_path_factory.mktemp(name), MODELS[name], w)
            cache[name, dtype] = api.load_model(folder, device=torch.device("cuda", 0), dtype=dtype) + (w, folder)
        return cache[name, dtype]
    return get


@BOTH
@ALL
def test_layers_and_logits_of_a_prompt(models, name, dtype):
    model, cfg, w, _ = models(name, dtype)
    toks = prompt(1, 90, cfg.vocab_size)
    want, residual = O.run(MODELS[name], w, toks)
    cache = new_cache(model, cfg, 1, 96)
    cache.reserve([90])
    seen = {}
    model.run_layers(TokenBatch.build(cache, [torch.tensor(toks, dtype=i32)]), cache, after_layer=lambda i, x: seen.__setitem__(i, x.clone()))
    done()
    for i in range(cfg.num_layers):
        assert seen[i].dtype == f32
        logits_close(seen[i].cpu(), residual[i], dtype)
    logits_close(run(model, cfg, new_cache(model, cfg, 1, 96), [toks])[0], want, dtype)
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
    want, _ = O.run(MODELS[name], w, toks)
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
    want, _ = O.run(MODELS[name], w, toks)
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
    want = [O.run(MODELS[name], w, t)[0] for t in toks]
    cache = new_cache(model, cfg, 4, 64, num_pages=18)
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
@ALL
def test_long_decoding_returns_the_pages_it_leaves_behind(models, name, dtype):
    """Many windows past the prompt, on fewer pages than the tokens would fill."""
    model, cfg, w, _ = models(name, dtype)
    toks = prompt(5, 230, cfg.vocab_size)
    want, _ = O.run(MODELS[name], w, toks)
    cache = new_cache(model, cfg, 2, 256, num_pages=12)
    widest = max(layer.mixer.window for layer in cfg.layers)
    got = run(model, cfg, cache, [toks[:10], toks[:3]])[:1]
    for t in toks[10:]:
        got.append(run(model, cfg, cache, [[t], []])[0])
        assert cache.num_pages - len(cache.allocator.free) <= widest // 8 + 2 + 1
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
            seq.append(int(O.run(MODELS[name], w, seq)[0][-1].argmax()))
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
