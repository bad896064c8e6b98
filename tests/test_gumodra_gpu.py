"""The Gumodra design in the engine against its plain implementation (plain_gumodra.py): every mechanism alone through the
kernel library, and whole models of several small configurations in every cut of the steps.  The configurations differ in
every size and option, with values that are unequal where a model might have them equal (key and value sizes of a memory,
layers' heads and windows, kept tokens and pages) and 1 where it might have more (heads, experts, chosen experts, window,
kept tokens)."""
import random
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_gumodra as P
from helpers import trace_whole, trace_tail_decode, trace_portions, trace_mixed, run_trace, first_bad
from test_tipezen_gpu import fake_batch
from tffinfer_b200.config import EngineConfig, GumodraConfig, GumodraLayer, GumodraMlp
from tffinfer_b200.config.gumodra_config import GumodraAttention, GumodraMlstm
from tffinfer_b200.config.tipezen_config import RotaryConfig
from tffinfer_b200.engine import ModelRunner
from tffinfer_b200.kernels.library import mlstm_state_size
from tffinfer_b200.weights.random_init import random_state_dict

pytestmark = pytest.mark.gpu
TOL = {"float32": 3e-5, "bfloat16": 2e-2}


def att(heads, kv, dim, window, keep, rot, scale=None, base=1e4, mlp=None):
    return GumodraLayer("attention", mlp=mlp, attention=GumodraAttention(
        heads, kv, dim, scale if scale is not None else dim ** -0.5, RotaryConfig(base, rot) if rot else None, window, keep))


def mem(heads, dim, vdim, cap=6.0, mlp=None):
    return GumodraLayer("mlstm", mlstm=GumodraMlstm(heads, dim, vdim, cap), mlp=mlp)


def dense(ff):
    return GumodraMlp("dense", ff)


def moe(ff, experts, top, groups=(1, 1), shared=0):
    return GumodraMlp("moe", ff, experts, top, groups, shared)


def config(name: str) -> GumodraConfig:
    make = lambda **kw: GumodraConfig("Gumodra", **kw)
    if name == "a":      # sizes that take the tensor-core kernels, kept tokens that end inside a page and beyond a key block
        return make(vocab_size=320, hidden_size=128, norm_eps=1e-6, embed_scale=3.5, layers=(
            mem(2, 32, 64, cap=9.0, mlp=dense(192)), att(6, 2, 64, 40, 9, 24, mlp=moe(64, 10, 3, (5, 2), 64)),
            att(3, 1, 64, 70, 66, 64, base=3e5, mlp=dense(96)), mem(4, 16, 32, mlp=moe(64, 6, 2, (2, 2), 128))))
    if name == "b":      # odd sizes everywhere: FMA products; windows that no page size divides, every expert chosen
        return make(vocab_size=97, hidden_size=52, norm_eps=3e-6, embed_scale=0.8, layers=(
            att(3, 3, 20, 7, 5, 6, scale=0.2, base=1e3, mlp=moe(22, 5, 5, (1, 1), 30)), mem(3, 12, 21, cap=4.0),
            att(4, 2, 12, 13, 1, 12, scale=0.4, base=1e3), mem(1, 13, 6, cap=2.5, mlp=dense(70))))
    if name == "c":      # one head, one expert, a window of one and none, nothing kept, no rotation, no shared expert
        return make(vocab_size=264, hidden_size=64, norm_eps=1e-5, embed_scale=1.0, layers=(
            mem(1, 8, 96, cap=15.0, mlp=moe(48, 1, 1)), att(2, 1, 72, 1, 0, 0, mlp=moe(16, 9, 1, (3, 1))),
            mem(2, 40, 8, cap=30.0), att(1, 1, 128, 0, 0, 2, base=5e5, mlp=dense(32))))
    if name == "d":      # heads of 128, windows of 64 over pages of 32, more kept tokens than the window, 16 groups
        return make(vocab_size=150, hidden_size=96, norm_eps=1e-6, embed_scale=9.0, layers=(
            att(4, 4, 128, 64, 1, 128, mlp=moe(32, 16, 3, (16, 7), 40)), mem(2, 72, 24, mlp=dense(40)),
            att(8, 2, 128, 33, 100, 32, base=3e5, mlp=moe(32, 12, 4, (3, 2), 32)), mem(8, 8, 8, mlp=moe(16, 7, 2, (7, 3), 8))))
    raise KeyError(name)


PAGE = {"a": 16, "b": 4, "c": 8, "d": 32}
PROMPTS = {"a": [5, 90, 37, 200], "b": [1, 13, 40, 64], "c": [3, 29, 110, 71], "d": [2, 70, 233]}


def weights(cfg, seed=11, sharp=4.0):
    """Random weights with attention scores far from uniform, gates of the memory far from the middle, router scores and
    corrections of the same size, gates of the residual that bend, and an embedding that weighs beside what layers add."""
    sd = random_state_dict(cfg, seed, "bfloat16", norm_noise=0.2)
    W = cfg.hidden_size
    for n in sd:
        f = 1.0
        if n == "embed":
            f = 40.0 / cfg.embed_scale
        elif n.endswith((".mix.q", ".mix.k", ".mix.v", ".mix.g", ".rg1", ".rg2", ".sg")):
            f = sharp * (128 / W) ** 0.5
        elif n.endswith((".mix.i", ".mix.f")):
            f = 5.0 * (128 / W) ** 0.5
        elif n.endswith(".mlp.router"):
            f = 12.0 * (128 / W) ** 0.5
        elif n.endswith((".norm", )) and ".mix." in n and sd[n].dim() == 1 and (n.endswith("q.norm") or n.endswith("k.norm")):
            f = 1.5
        elif n.endswith((".gate", ".up")):
            f = 5.0 * (128 / W) ** 0.5
        elif n.endswith((".down", ".mix.o")):
            f = 5.0
        if f != 1.0:
            sd[n] = (sd[n].float() * f).to(torch.bfloat16)
    return sd


def runner_of(cfg, sd, dtype, page, tokens, live=4, graphs=False):
    return ModelRunner(config=cfg, tensors=dict(sd), engine_config=EngineConfig(
        dtype=dtype, page_size=page, max_cache_tokens=tokens, max_live_requests=live, use_cuda_graphs=graphs))


def plain_logits(cj, sd, reqs, dtype):
    """{request: (logits, bar of every position)} of the plain implementation.  A position's bar is the larger of the
    format's and three times what the format's rounding alone moves the plain logits there (bfloat16: of the rows that
    enter every product; float32: of everything); positions whose bar is raised must be few, or the test says nothing."""
    out = {}
    for r, t in reqs.items():
        want = P.forward(cj, sd, t)
        bar = torch.full((want.shape[0],), TOL[dtype], dtype=torch.float64)
        moved = P.forward(cj, sd, t, round_inputs=True) if dtype == "bfloat16" else P.forward(cj, sd, t, dtype=torch.float32)
        bar = torch.maximum(bar, 3.0 * (moved - want).abs().amax(dim=-1) / want.abs().amax(dim=-1))
        out[r] = (want, bar)
    raised = sum(int((b > TOL[dtype]).sum()) for _, b in out.values())
    assert raised <= 2 + sum(w.shape[0] for w, _ in out.values()) // 3, f"{raised} ill-conditioned positions: too many for a test"
    return out


def assert_within(got, want_bar, what):
    want, bar = want_bar
    err = torch.nan_to_num((got.double() - want).abs().amax(dim=-1) / want.abs().amax(dim=-1).clamp_min(1e-30), nan=float("inf"))
    bad = torch.nonzero(err > bar)
    # in bfloat16 a token's choice of experts may hang on the rounding (and a memory carries that on for a few tokens): a
    # few positions may leave their bar, the others stay well inside
    few = max(5, want.shape[0] // 25) if float(bar.min()) >= TOL["bfloat16"] and want.shape[0] > 20 else 0
    assert bad.numel() <= few and float(err.median()) < 0.75 * float(bar.median()), \
        f"{what}: {bad.numel()} tokens, {int(bad[0])} off by {float(err[int(bad[0])]):.3g} (bar {float(bar[int(bad[0])]):.3g})"


def requests_of(cfg, name, decoded, seed=5):
    rng = random.Random(seed)
    return {f"r{i}": [rng.randrange(cfg.vocab_size) for _ in range(n + decoded)] for i, n in enumerate(PROMPTS[name])}


@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_cut_matches_plain(name, dtype):
    """Whole prompts, a tail decoded token by token, portions down to two tokens, and mixed batches in a pool small
    enough that pages and slots are used again (released pages are poisoned; the windows pass over pages and leave the
    kept ones)."""
    cfg = config(name)
    sd = weights(cfg)
    reqs = requests_of(cfg, name, decoded=12)
    want = plain_logits(cfg.to_json_dict(), sd, reqs, dtype)
    page = PAGE[name]
    most = max(-(-len(t) // page) * page for t in reqs.values())
    cuts = {"whole": (trace_whole(reqs), most), "tail": (trace_tail_decode(reqs, tail=12), most),
            "portions": (trace_portions(reqs), most),
            "mixed": (trace_mixed(reqs, PROMPTS[name], max_live=3, page_size=page, pool_tokens=most + most // 2,
                                  chunk=48), most + most // 2)}
    for cut, (steps, pool) in cuts.items():
        r = runner_of(cfg, sd, dtype, page, pool, live=3)
        for s in r.states:
            s.fill_(float("nan"))                  # a slot that was never used, or by another request, is not read
        stats = {}
        got = run_trace(r, reqs, steps, poison=True, stats=stats)
        for q in reqs:
            assert_within(got[q], want[q], f"{name} {dtype} {cut}: request {q}")
        if cut == "mixed":
            assert stats["pages_reused"] > 0


def test_the_residual_after_every_layer():
    from tffinfer_b200.engine import StepEntry
    for name in ("a", "b", "c", "d"):
        cfg = config(name)
        sd = weights(cfg)
        toks = requests_of(cfg, name, 0)["r1"]
        want, got = [], []
        P.forward(cfg.to_json_dict(), sd, toks, layers_out=want)
        r = runner_of(cfg, sd, "float32", PAGE[name], 256)
        r.model.layer_hook = lambda e, x: got.append(x.double().cpu().clone())
        r.add_request("r")
        r.step([StepEntry("r", toks, [])])
        assert len(got) == len(want) == len(cfg.layers)
        for i, (a, b) in enumerate(zip(got, want)):
            assert float((a - b).abs().max()) < 2e-5 * float(b.abs().max()), f"{name}: layer {i}"


def test_cuts_agree_in_float32():
    """The logits of a position do not depend on how the prompt was cut, or on what else is in the batch, beyond
    rounding: far tighter than the distance to the plain implementation allows."""
    cfg = config("a")
    sd = weights(cfg)
    reqs = requests_of(cfg, "a", decoded=8)
    most = max(-(-len(t) // 16) * 16 for t in reqs.values())
    ref = run_trace(runner_of(cfg, sd, "float32", 16, most), reqs, trace_whole(reqs))
    for steps, tokens in ((trace_portions(reqs, sizes=(2, 31, 3, 16, 2, 33)), most), (trace_tail_decode(reqs, tail=40), most),
                          (trace_mixed(reqs, PROMPTS["a"], max_live=4, page_size=16, pool_tokens=4 * most, chunk=30), 4 * most)):
        got = run_trace(runner_of(cfg, sd, "float32", 16, tokens), reqs, steps)
        for q in reqs:
            assert first_bad(got[q], ref[q], 5e-6) is None


# ------------------------------------------------------------------------------ mechanisms alone
@pytest.fixture(scope="module")
def ops():
    from tffinfer_b200.kernels.library import CudaKernels
    return CudaKernels()


def _attention_part(ops, dtype, W, H, G, D, window, keep, scale, rot, base, w):
    from tffinfer_b200.parts.attention import GatedSinkAttention
    from tffinfer_b200.parts.position import ScaledRotary
    dt = getattr(torch, dtype)
    m = GatedSinkAttention(W, H, G, D, softmax_scale=scale, window=window, keep_first=keep, sink="learned", qk_norm="head",
                           qk_norm_eps=1e-5, projection_bias=True, values_are_keys=True,
                           names={"q": "q", "k": "k", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "q_bias": "q.b",
                                  "k_bias": "k.b", "o_bias": "o.b"})
    assert set(m.weight_specs()) == set(w)
    m.load({n: (v.float() if v.dim() == 1 else v.to(dt)).cuda().contiguous() for n, v in w.items()}, ops, dt)
    pos = None
    if rot:
        pos = ScaledRotary(rot, base, "halves")
        pos.prepare(ops, "cuda", 0)
    return m, pos


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,rot,window,keep", [(4, 2, 64, 24, 50, 21), (6, 2, 128, 128, 100, 7), (3, 3, 24, 10, 33, 130),
                                                   (8, 1, 64, 64, 1, 1), (2, 1, 200, 0, 64, 64), (20, 1, 64, 2, 65, 0),
                                                   (4, 4, 128, 6, 0, 0), (4, 2, 40, 40, 1, 300)])
def test_attention_alone(ops, dtype, H, G, D, rot, window, keep):
    """An attention alone: 700 tokens in portions that end inside pages, then single tokens, with sharp queries (a missed
    key among hundreds shows), windows over pages they have passed (poisoned before every step, as pages that were given
    back, but not those with kept tokens), learned sinks from overwhelming to negligible, biases everywhere; then the
    whole prompt as one step."""
    from tffinfer_b200.parts.base import LayerContext
    dev, dt = "cuda", getattr(torch, dtype)
    g = torch.Generator().manual_seed(H * D + window)
    W, page, T = 72, 16, 700
    h = torch.randn(T, W, generator=g).to(dt)
    w = {n: (torch.randn(*s, generator=g) * s[1] ** -0.5).to(torch.bfloat16)
         for n, s in {"q": (H * D, W), "k": (G * D, W), "o": (W, H * D)}.items()}
    for n, s in (("q.b", H * D), ("k.b", G * D), ("o.b", W)):
        w[n] = (torch.randn(s, generator=g) * 0.5).to(torch.bfloat16)
    for n in ("q.norm", "k.norm"):
        w[n] = (1.7 + 0.4 * torch.randn(D, generator=g)).to(torch.bfloat16)
    w["sink"] = torch.linspace(-20.0, 7.0, H).to(torch.bfloat16)
    scale = 1.3 * D ** -0.5
    part, pos = _attention_part(ops, dtype, W, H, G, D, window, keep, scale, rot, 2e3, w)
    m = {"heads": H, "kv_heads": G, "dim": D, "scale": scale, "rot": {"base": 2e3, "dims": rot},
         "mask": {"size": window, "keep_first": keep}}
    wd = {"p." + n: v.double() for n, v in w.items()}
    want = P.attention_mixer(h.double(), torch.arange(T), wd, "p", m, 1e-5)
    for other in (dict(wd, **{"p.sink": wd["p.sink"] - 1e4}), None):         # the sink and the kept tokens matter here
        if other is None and (window == 0 or keep == 0):
            continue
        mask = m if other is not None else dict(m, mask={"size": window, "keep_first": 0})
        without = P.attention_mixer(h.double(), torch.arange(T), other or wd, "p", mask, 1e-5)
        assert float((want - without).abs().max()) > 0.05 * float(want.abs().max())
    bar = 2e-5 if dtype == "float32" else 2.5e-2
    pages = -(-T // page)
    order = torch.randperm(pages, generator=g).tolist()                      # pages in no order
    cache = torch.full((pages + 1, 1, 2, G, page, D), float("nan"), device=dev, dtype=dt)
    got, start = [], 0
    for n in [3, 200, 2, 61, 150, 2, 130, 100] + [1] * 52:
        b = fake_batch([n], [start], dev, page)
        table = torch.full((1, pages), -1, dtype=torch.int32)
        for i in range(-(-(start + n) // page)):
            table[0, i] = order[i]
        if window > 0:
            for i in range(-(-keep // page), max(0, start - window + 1) // page):
                table[0, i] = -1
                cache[order[i]] = float("nan")
        ctx = LayerContext(batch=b, ops=ops, kv_cache=cache, kv_layer=0, block_table=table.to(dev), page_size=page, position=pos)
        got.append(part.forward(h[start:start + n].to(dev), ctx, torch.zeros(n, W, device=dev)).double().cpu())
        start += n
    ops.check_errors()
    got = torch.cat(got)
    err = (got - want).abs().amax(dim=-1) / want.abs().max()
    assert start == T and float(torch.nan_to_num(err, nan=9.0).max()) < bar, f"token {int(err.argmax())} off by {float(err.max()):.3g}"
    cache.fill_(float("nan"))
    b = fake_batch([T], [0], dev, page)
    ctx = LayerContext(batch=b, ops=ops, kv_cache=cache, kv_layer=0, block_table=b.block_table, page_size=page, position=pos)
    y = part.forward(h.to(dev), ctx, None).double().cpu() + part.output_bias.double().cpu()
    ops.check_errors()
    ops.reset_accumulators()
    assert float((y - want).abs().max()) < bar * float(want.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D,G,page,window,keep", [(64, 2, 16, 96, 24), (128, 4, 32, 64, 64), (64, 16, 8, 25, 1), (64, 1, 16, 1, 3),
                                                  (40, 2, 4, 17, 9), (128, 2, 64, 300, 130), (64, 2, 24, 70, 33)])
def test_keys_just_inside_and_just_outside(ops, dtype, D, G, page, window, keep):
    """One key at a time stands out; a query sees its value exactly if the key is within the window or among the kept
    tokens, at the window's edges, the kept tokens' edge, page and key-block borders, for decoded tokens (the key range
    whole and in shares) and for the tokens of a portion, beside another request."""
    dev, dt = "cuda", getattr(torch, dtype)
    H, nkv = G * 1, 1
    g = torch.Generator().manual_seed(D + window)
    for n_new, start in ((1, 517), (1, window + keep + 1), (40, 480), (150, 300)):
        lens, starts = [n_new, n_new], [start, 60]
        b = fake_batch(lens, starts, dev, page)
        T = sum(lens)
        pages = b.pages + 1
        base = torch.randn(pages, 1, 2, nkv, page, D, generator=g) * 0.1
        base[:, :, 0, :, :, 0] = 0.0                                        # the element that makes a key stand out
        end = start + n_new - 1
        q = torch.randn(T, H * D, generator=g) * 0.1
        q.view(T, H, D)[:, :, 0] = 30.0
        cands = {0, keep - 1, keep, keep + 1, end, end - 1, start, start - 1, start - window, start - window + 1,
                 end - window, end - window + 1, end - window + 2, 63, 64, (start // page) * page, (start // page) * page - 1,
                 (keep // page) * page, (keep // page + 1) * page}
        for n in sorted(c for c in cands if 0 <= c <= end):
            cache = base.clone()
            pg = int(b.block_table[0, n // page])
            cache[pg, 0, 0, 0, n % page, 0] = 30.0
            cache[pg, 0, 1, 0, n % page] = 5.0
            outs = []
            for splits in ((None, 4) if n_new == 1 and dtype == "bfloat16" and D in (64, 128) else (None,)):
                out = torch.full((T, H * D), float("nan"), device=dev, dtype=dt)
                if splits is None:
                    ops.attention_ext(q.to(dt).to(dev), b, b.block_table, cache.to(dt).to(dev), 0, page, out, H, nkv, D, D,
                                      1.0, window, 0.0, torch.zeros(H, device=dev), None, keep)
                else:
                    ops.attention_bf16(q.to(dt).to(dev), b, b.block_table, cache.to(dt).to(dev), 0, page, out, H, nkv, D, 1.0,
                                       window, num_splits=splits, extra=(0.0, torch.zeros(H, device=dev), None, keep))
                outs.append(out.double().cpu())
            for out in outs:
                for i in range(n_new):
                    p = start + i
                    sees = n <= p and (p - n < window or n < keep)
                    val = out[i].view(H, D).mean(dim=1)
                    assert bool(((val > 4.9) if sees else (val < 1.0)).all()), f"key {n} from {p}: {val}"
                assert float(out[n_new:].abs().max()) < 1.0 or float(torch.isnan(out).sum()) == 0
    ops.check_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nq,nkv,d,rot,own", [(5, 2, 64, 32, False), (3, 3, 20, 20, True), (9, 1, 129, 0, False), (2, 1, 300, 64, True),
                                              (1, 1, 2, 2, False)])
@pytest.mark.parametrize("interleaved", [False, True])
def test_heads_normed_turned_and_written(ops, dtype, nq, nkv, d, rot, own, interleaved):
    """The kernel between the projection and the attention: biases, norms, rotation at large positions, keys and values in
    their slots, and an accumulator buffer set back to zero, with values of their own and values that are the keys."""
    dev, dt, page = "cuda", getattr(torch, dtype), 8
    g = torch.Generator().manual_seed(nq * d)
    lens, starts = [5, 1, 3], [11, 40000, 0]
    b = fake_batch(lens, [11, 40, 0], dev, page)
    pos = torch.cat([torch.arange(s, s + n) for n, s in zip(lens, starts)]) if False else b.positions.cpu()
    T = sum(lens)
    dv = d if not own else d
    width = (nq + nkv) * d + (nkv * dv if own else 0)
    rows = torch.randn(T, width, generator=g)
    bias, qw, kw = torch.randn(width, generator=g), torch.randn(d, generator=g), torch.randn(d, generator=g)
    buf = ops.projection_buffer(T, width, torch.device(dev), torch.bfloat16, use=f"heads {nq} {d} {own}")
    freq = torch.tensor([3e3 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
    order = [j for i in range(rot // 2) for j in (2 * i, 2 * i + 1)] if interleaved else None
    u = rows.double() + bias.double()

    def finish(x, w):
        x = x / P.rms(x, 1e-5) * w.double()
        if rot == 0:
            return x
        if interleaved:                                  # as halves, in the order that puts the pairs' members apart
            idx = list(range(0, rot, 2)) + list(range(1, rot, 2)) + list(range(rot, d))
            y = P.turn_halves(x[..., idx], pos, rot, 3e3)
            back = torch.empty_like(y)
            back[..., idx] = y
            return back
        return P.turn_halves(x, pos, rot, 3e3)
    want_q = finish(u[:, :nq * d].reshape(T, nq, d), qw)
    want_k = finish(u[:, nq * d:(nq + nkv) * d].reshape(T, nkv, d), kw)
    want_v = u[:, (nq + nkv) * d:].reshape(T, nkv, d) if own else u[:, nq * d:(nq + nkv) * d].reshape(T, nkv, d)
    for _ in range(2):
        buf.copy_(rows)
        ops._acc_zero[buf.data_ptr()] = False
        cache = torch.full((b.pages + 1, 1, 2, nkv, page, d + 3), float("nan"), device=dev, dtype=dt)
        q = torch.full((T, nq * d), float("nan"), device=dev, dtype=dt)
        ops.qk_finish(buf, q, (qw.to(dev), kw.to(dev)), 1e-5, bias.to(dev), not own,
                      (freq.float().to(dev), rot, 1.0, interleaved) if rot else None, b, b.block_table, cache, 0, page, nq, nkv, d, dv)
        torch.cuda.synchronize()
        tol = (3e-5 if dtype == "float32" else 1e-2)
        close = lambda a, c: float((a.double().cpu() - c).abs().max()) < tol * float(c.abs().max())
        assert close(q.view(T, nq, d), want_q)
        c = cache.cpu()
        for t in range(T):
            pg, s = int(b.block_table[int(b.tok_req[t]), int(pos[t]) // page]), int(pos[t]) % page
            assert close(c[pg, 0, 0, :, s, :d], want_k[t]) and close(c[pg, 0, 1, :, s, :d], want_v[t])
        assert not buf.any() and ops._acc_zero[buf.data_ptr()]


MEMORIES = [(2, 32, 16), (3, 12, 20), (1, 128, 128), (4, 7, 33), (2, 8, 130), (1, 200, 260), (1, 300, 40), (1, 5, 2100)]


def _memory_inputs(g, n, H, D, V, cap):
    q, k, v = (torch.randn(n, w, generator=g).to(torch.bfloat16).float() for w in (H * D, H * D, H * V))
    return q, k, v, torch.randn(n, H, generator=g) * 0.8 * cap, torch.randn(n, H, generator=g) * 0.8 * cap + cap


def _plain_memory(q, k, v, zi, zf, bi, bf, cap, H, D, V):
    outs, states = [], []
    i = P.capped(zi.double() + bi.double(), cap)
    f = torch.nn.functional.logsigmoid(P.capped(zf.double() + bf.double(), cap))
    for h in range(H):
        o, s = P.mlstm_recurrence(q[:, h * D:(h + 1) * D].double() * D ** -0.5, k[:, h * D:(h + 1) * D].double(),
                                  v[:, h * V:(h + 1) * V].double(), i[:, h], f[:, h])
        outs.append(o)
        states.append(s)
    return torch.cat(outs, dim=-1), states


@pytest.mark.parametrize("H,D,V", MEMORIES)
@pytest.mark.parametrize("rounded", [False, True])
def test_memory_steps_slots_and_a_far_key(ops, H, D, V, rounded):
    """The recurrence through five steps (long and short portions, one token each twice), slots out of order, other slots
    poisoned and the requests' own full of NaN at the start, gates far beyond the cap on both sides, denominators on both
    of their branches.  In the first request one key far back is planted under forget gates near one, with a query aimed
    at it.  ``rounded`` is the chunk form on the tensor cores where the head fits it: q, k and v hold values that bfloat16
    has, so it must be as close as the float32 form."""
    dev, cap = "cuda", 5.0
    g = torch.Generator().manual_seed(H * D + V)
    cuts = [[150, 3, 1], [2, 70, 1], [64, 2, 2], [1, 1, 1], [1, 1, 1]]
    total = [sum(c[i] for c in cuts) for i in range(3)]
    slots = [3, 0, 2]
    state = torch.full((5, mlstm_state_size(H, D, V)), float("nan"), device=dev)
    bias = torch.randn(2 * H, generator=g)
    seqs = [_memory_inputs(g, n, H, D, V, cap) for n in total]
    q0, k0, _, i0, f0 = seqs[0]
    k0[:, 0] = 0.0
    k0[4, 0] = 20.0
    q0[-1, :D] = 0.0
    q0[-1, 0] = 20.0
    f0[:, 0] = 200.0                                     # far beyond the cap: the forget gate stays near one
    i0[4, 0] = 200.0
    want, ends = zip(*[_plain_memory(*s, bias[:H], bias[H:], cap, H, D, V) for s in seqs])
    got = [[] for _ in seqs]
    starts = [0, 0, 0]
    ld = 2 * H * D + 2 * H * V + 2 * H + 5
    for lens in cuts:
        b = fake_batch(lens, starts, dev, 8, slots=slots)
        part = [torch.cat([s[j][st:st + n] for s, n, st in zip(seqs, lens, starts)]) for j in range(5)]
        T = part[0].shape[0]
        proj = torch.full((T, ld), float("nan"))
        proj[:, :H * D], proj[:, H * D:2 * H * D], proj[:, 2 * H * D:2 * H * D + H * V] = part[:3]
        at = 2 * H * D + 2 * H * V
        proj[:, at:at + H], proj[:, at + H:at + 2 * H] = part[3:]
        out = torch.full((T, H * V), float("nan"), device=dev)
        ops.mlstm_recurrence(proj.to(dev), state, b, bias.to(dev), cap, out, H, D, V, rounded=rounded)
        torch.cuda.synchronize()
        row = 0
        for i, n in enumerate(lens):
            got[i].append(out[row:row + n].double().cpu())
            row += n
        starts = [s + n for s, n in zip(starts, lens)]
    # an output may be a small difference over a small denominator: rows are held to the larger of their own size and the
    # rows' typical size
    for i in range(3):
        a = torch.cat(got[i])
        size = torch.maximum(want[i].abs().amax(dim=-1), want[i].abs().amax(dim=-1).median())
        err = torch.nan_to_num((a - want[i]).abs().amax(dim=-1) / size, nan=9.0)
        assert float(err.max()) < 1e-3 and float(err.median()) < 1e-5, f"request {i}: token {int(err.argmax())} off by {float(err.max()):.3g}"
        s = state[slots[i]].double().cpu()
        for h in range(H):
            S, n, m = ends[i][h]
            close = lambda x, y: float((x - y).abs().max()) < 3e-5 * max(float(y.abs().max()), 1e-3)
            assert close(s[h * D * V:(h + 1) * D * V].view(D, V), S), (i, h)
            assert close(s[H * D * V + h * D:H * D * V + (h + 1) * D], n)
            assert abs(float(s[H * D * V + H * D + h] - m)) < 1e-4
    v4 = seqs[0][2][4, :V].double()                      # the far key's value is what the last output of head 0 holds
    last = torch.cat(got[0])[-1, :V]
    assert float(torch.dot(last, v4) / (last.norm() * v4.norm())) > 0.999
    assert torch.isnan(state[1]).all() and torch.isnan(state[4]).all()          # nobody's slots were left alone


@pytest.mark.parametrize("D,V", [(64, 96), (20, 36), (16, 16)])
def test_memory_tokens_and_chunks_agree(ops, D, V):
    """Single tokens and a portion inside a chunk through both forms leave the same outputs and states."""
    dev, H, cap = "cuda", 3, 4.0
    g = torch.Generator().manual_seed(D)
    start = torch.randn(4, mlstm_state_size(H, D, V), generator=g)
    bias = torch.randn(2 * H, generator=g).to(dev)
    for lens, starts in (([1, 1, 1], [70, 64, 127]), ([9, 1, 60], [63, 1, 10])):
        proj = torch.randn(sum(lens), 2 * H * D + 2 * H * V + 2 * H, generator=g).to(torch.bfloat16).float().to(dev)
        outs, states = [], []
        for ch in (False, True):
            st = start.clone().to(dev)
            out = torch.full((sum(lens), H * V), float("nan"), device=dev)
            ops.mlstm_recurrence(proj, st, fake_batch(lens, starts, dev, 8, slots=[2, 0, 1]), bias, cap, out, H, D, V,
                                 rounded=ch, chunked=ch)
            outs.append(out)
            states.append(st)
        torch.cuda.synchronize()
        assert torch.allclose(states[0], states[1], rtol=1e-4, atol=1e-4)
        err = ((outs[0] - outs[1]).abs().amax(dim=-1) / outs[0].abs().amax(dim=-1).clamp_min(1e-2))
        assert float(err.max()) < 1e-3 and float(err.median()) < 2e-5


@pytest.mark.parametrize("H,D,V", [(2, 64, 96), (3, 20, 9), (1, 300, 36), (2, 128, 128)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_memory_decode_steps_of_many_requests_up_to_the_gate(ops, H, D, V, dtype):
    """One token of each of so many requests that the step kernel takes its small CTAs, on to norm and gate in the same
    kernel, against the plain equations; the projection's rows set to zero where they were read, and the same states and
    outputs as in steps of few requests."""
    dev, cap, B, eps = "cuda", 4.0, 310, 1e-4
    g = torch.Generator().manual_seed(D)
    at = 2 * H * D + 2 * H * V
    start = torch.randn(B, mlstm_state_size(H, D, V), generator=g)
    bias, w = torch.randn(2 * H, generator=g), 1 + 0.3 * torch.randn(H * V, generator=g)
    rows = torch.randn(B, at + 2 * H + 3, generator=g)
    slots = torch.randperm(B, generator=g).tolist()
    fresh = [5 if i % 7 else 0 for i in range(B)]                # some requests bring their first token
    buf = ops.projection_buffer(B, at + 2 * H + 3, torch.device(dev), torch.bfloat16, use=f"memory {H} {D} {dtype}") \
        if B <= ops.SWAP_MAX_M else torch.zeros(B, at + 2 * H + 3, device=dev)
    ops._acc_zero[buf.data_ptr()] = False
    buf.copy_(rows)
    st, mixed = start.clone().to(dev), torch.full((B, H * V), float("nan"), device=dev, dtype=dtype)
    ops.mlstm_recurrence(buf, st, fake_batch([1] * B, fresh, dev, 8, slots=slots), bias.to(dev), cap, None, H, D, V,
                         finish=(2 * H * D + H * V, w.to(dev), eps, mixed))
    torch.cuda.synchronize()
    assert not buf[:, :at + 2 * H].any() and torch.equal(buf[:, at + 2 * H:].cpu(), rows[:, at + 2 * H:])
    del ops._acc_zero[buf.data_ptr()]
    few = start.clone().to(dev)
    for lo in range(0, B, 100):
        out = torch.full((min(100, B - lo), H * V), float("nan"), device=dev)
        b = fake_batch([1] * out.shape[0], fresh[lo:lo + 100], dev, 8, slots=slots[lo:lo + 100])
        ops.mlstm_recurrence(rows[lo:lo + 100].contiguous().to(dev), few, b, bias.to(dev), cap, out, H, D, V)
        o = out.double().cpu().view(-1, H, V)
        gate = torch.sigmoid(rows[lo:lo + 100, 2 * H * D + H * V:at].double())
        want = (o / P.rms(o, eps)).reshape(-1, H * V) * w.double() * gate
        err = (mixed[lo:lo + 100].double().cpu() - want).abs().max() / want.abs().max()
        assert float(err) < (1e-4 if dtype == torch.float32 else 1e-2)
    assert torch.allclose(st, few, rtol=1e-5, atol=1e-5)
    for i in (0, 1, 7, 309):                                     # and the plain equations, request by request
        s = start[slots[i]].double()
        r = rows[i].double()
        for h in range(H):
            state = (s[h * D * V:(h + 1) * D * V].view(D, V), s[H * D * V + h * D:H * D * V + (h + 1) * D], s[H * D * V + H * D + h])
            ig = P.capped(r[at + h] + bias[h].double(), cap)
            fg = torch.nn.functional.logsigmoid(P.capped(r[at + H + h] + bias[H + h].double(), cap))
            o, (S, n, m) = P.mlstm_recurrence(r[None, h * D:(h + 1) * D] * D ** -0.5, r[None, (H + h) * D:(H + h + 1) * D],
                                              r[None, 2 * H * D + h * V:2 * H * D + (h + 1) * V], ig[None], fg[None],
                                              None if fresh[i] == 0 else state)
            got = st[slots[i]].double().cpu()
            assert float((got[h * D * V:(h + 1) * D * V].view(D, V) - S).abs().max()) < 2e-5 * float(S.abs().max())
            assert abs(float(got[H * D * V + H * D + h] - m)) < 1e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T", [1, 9, 70, 300])
@pytest.mark.parametrize("H,D,V,W", [(3, 16, 24, 64), (2, 40, 40, 50)])
def test_memory_mixer(ops, monkeypatch, dtype, T, H, D, V, W):
    """The whole mixer: one product, the recurrence, per-head norm with a weight over all heads, sigmoid gate, output."""
    from tffinfer_b200.parts.base import LayerContext
    from tffinfer_b200.parts.mlstm import MLstm
    dev, dt, cap = "cuda", getattr(torch, dtype), 3.0
    g = torch.Generator().manual_seed(T + W)
    part = MLstm(W, H, D, V, cap, 1e-4)
    w = {}
    for n, s in part.weight_specs().items():
        w[n] = (torch.randn(*s.shape, generator=g) * (1.0 if len(s.shape) == 1 else 2.0 * W ** -0.5)).to(torch.bfloat16)
    part.load({n: (v.float() if v.dim() == 1 else v.to(dt)).to(dev) for n, v in w.items()}, ops, dt)
    h = torch.randn(T, W, generator=g).to(torch.bfloat16)
    m = {"heads": H, "dim": D, "vdim": V, "gate_cap": cap}
    wd = {"p." + n: v.double() for n, v in w.items()}
    want = P.mlstm_mixer(h.double(), wd, "p", m, 1e-4)
    product = P.lin
    monkeypatch.setattr(P, "lin", lambda x, a, b=None: product(x, a, b).to(torch.bfloat16).double() if b is None else product(x, a, b))
    moved = P.mlstm_mixer(h.double(), wd, "p", m, 1e-4)       # q, k and v rounded: how well conditioned a token is
    bar = torch.maximum(torch.full((T,), 4e-2).double(), 3 * (moved - want).abs().amax(dim=-1) / want.abs().max())
    state = torch.full((2,) + tuple(part.cache_need().shape), float("nan"), device=dev)
    for res in (None, torch.ones(T, W, device=dev)):
        ctx = LayerContext(batch=fake_batch([T], [0], dev, 8, slots=[1]), ops=ops, state=state)
        got = part.forward(h.to(dt).to(dev), ctx, res).double().cpu() - (0.0 if res is None else 1.0)
        ops.reset_accumulators()
        err = (got - want).abs().amax(dim=-1) / want.abs().max()
        assert bool((err < (1e-4 if dtype == "float32" else bar)).all()), f"off by {float(err.max()):.3g}"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [36, 50, 640, 2052])
@pytest.mark.parametrize("both", [True, False])
def test_the_join_of_a_gated_residual(ops, dtype, W, both):
    """Gates, biases, both sublayers, the sum in float32, the next norm; only chosen rows at the end; buffers cleared."""
    dev, T = "cuda", 11
    g = torch.Generator().manual_seed(W)
    x, y1, y2 = (torch.randn(T, W, generator=g) for _ in range(3))
    width = 2 * W if both else W
    z, b, c1, w = torch.randn(T, width, generator=g) * 3, torch.randn(width, generator=g), torch.randn(W, generator=g), torch.full((W,), 1.7)
    for zt in (torch.float32, torch.bfloat16):
        zz = z.to(zt)
        s = torch.sigmoid(zz.double() + b.double())
        want = x.double() + (y1.double() + c1.double()) * s[:, :W] + (y2.double() * s[:, W:] if both else 0.0)
        want_h = P.one_number_norm(want, 1.7, 1e-5)
        for rows in (None, torch.tensor([7, 0, 7], dtype=torch.int32, device=dev)):
            bufs = [ops.sublayer_output(T, W, torch.device(dev), torch.bfloat16, f"join test {i} {W}") for i in range(2)]
            for buf, y in zip(bufs, (y1, y2)):
                buf.copy_(y)
                ops._acc_zero[buf.data_ptr()] = False
            xs = x.clone().to(dev)
            h = torch.full((T if rows is None else 3, W), float("nan"), device=dev, dtype=dtype)
            ops.gated_join(xs, zz.to(dev), b.to(dev), bufs[0], c1.to(dev), bufs[1] if both else None, w.to(dev), 1e-5, h, rows)
            torch.cuda.synchronize()
            sel = slice(None) if rows is None else rows.cpu().long()
            assert float((h.double().cpu() - want_h[sel]).abs().max()) < (1e-5 if dtype == torch.float32 else 2e-2) * 4
            if rows is None:
                assert float((xs.double().cpu() - want).abs().max()) < 1e-5
                assert not bufs[0].any() and ops._acc_zero[bufs[0].data_ptr()]
            else:
                assert torch.equal(xs.cpu(), x)
            for buf in bufs:
                buf.zero_()
                ops._acc_zero[buf.data_ptr()] = True
        xs = x.clone().to(dev)                                   # without a norm
        ops.gated_join(xs, zz.to(dev), b.to(dev), y1.to(dev), None, y2.to(dev) if both else None)
        want0 = want - c1.double() * s[:, :W]
        assert float((xs.double().cpu() - want0).abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,top,groups,ff,shared,W,T", [(12, 3, (4, 2), 64, 64, 128, 9), (10, 4, (2, 1), 24, 30, 52, 70),
                                                        (6, 6, (1, 1), 32, 16, 64, 5), (16, 2, (16, 2), 64, 128, 128, 600),
                                                        (1, 1, (1, 1), 16, 8, 64, 3), (9, 1, (3, 3), 64, 0, 128, 40)])
def test_experts_within_groups_beside_a_gated_shared_expert(ops, dtype, E, top, groups, ff, shared, W, T):
    """Softmax scores, a correction that changes the choice and makes choice scores negative, groups judged by their best
    member, weights without the correction, a shared expert behind its own gate; through the FMA, mma.sync and tcgen05
    products."""
    from tffinfer_b200.parts.moe import RoutedExperts
    dev, dt = "cuda", getattr(torch, dtype)
    g = torch.Generator().manual_seed(E * 100 + top)
    part = RoutedExperts(W, ff, E, top, renormalize=True, router_score="softmax", correction=True, groups=groups,
                         shared_intermediate=shared, shared_gate=shared > 0, prefix="m")
    w = {}
    for n, s in part.weight_specs().items():
        f = 3.0 if n in ("router", "shared.sg") else 1.0
        w["m." + n] = (torch.randn(*s.shape, generator=g) * (f * s.shape[-1] ** -0.5)).to(torch.bfloat16)
    w["m.correction"] = (torch.randn(E, generator=g) * 0.5 - 0.5).to(torch.bfloat16)
    part.load({k[2:]: (v.float() if v.dim() == 1 else v.to(dt)).to(dev) for k, v in w.items()}, ops, dt)
    h = torch.randn(T, W, generator=g).to(torch.bfloat16)
    wd = {k: v.double() for k, v in w.items()}
    mlp = {"router": {"experts": E, "top": top, "groups": {"count": groups[0], "keep": groups[1]}}, "shared": {"ff": shared} if shared else None}
    # rows whose choice hangs on less than the router's rounding are taken out (there are few)
    s = torch.softmax(h.double() @ wd["m.router"].T, dim=-1)
    c = torch.sort(s + wd["m.correction"], dim=-1).values
    sure = (c[:, 1:] - c[:, :-1]).min(dim=-1).values > 1e-4 if E > 1 else torch.ones(T, dtype=torch.bool)
    assert int(sure.sum()) >= 0.8 * T
    want = P.expert_ff(h.double(), wd, "m", mlp)
    ctx = SimpleNamespace(ops=ops, batch=None)
    for _ in range(2):                                       # twice: nothing is left over from the first call
        alone = part.forward(h.to(dt).to(dev), ctx, None).double().cpu().clone()
        res = torch.ones(T, W, device=dev)
        added = part.forward(h.to(dt).to(dev), ctx, res).double().cpu() - 1.0
        for got in (alone, added):
            err = float((got - want)[sure].abs().max()) / float(want.abs().max())
            assert err < (2e-5 if dtype == "float32" else 2e-2), f"off by {err:.3g}"


def test_weights_of_experts_whose_scores_vanish(ops):
    """The chosen experts' scores may all be so small that they do not reach 1e-20: their weights then shrink with them."""
    from tffinfer_b200.parts.moe import RoutedExperts
    dev = "cuda"
    part = RoutedExperts(8, 8, 4, 2, renormalize=True, router_score="softmax", correction=True, prefix="m")
    g = torch.Generator().manual_seed(1)
    w = {"m." + n: torch.randn(*s.shape, generator=g) for n, s in part.weight_specs().items()}
    w["m.router"] = torch.zeros(4, 8)
    w["m.router"][:, 0] = torch.tensor([50.0, 0.0, 1.0, 49.0])
    w["m.correction"] = torch.tensor([0.0, 3.0, 2.0, 0.0])    # the choice falls on the two whose scores are e^-49
    part.load({k[2:]: v.to(dev) for k, v in w.items()}, ops, torch.float32)
    h = torch.randn(3, 8, generator=g)
    h[:, 0] = 1.0
    h[1, 0] = 1.2                                             # e^-60 there
    want = P.expert_ff(h.double(), {k: v.double() for k, v in w.items()}, "m", {"router": {"experts": 4, "top": 2}})
    got = part.forward(h.to(dev), SimpleNamespace(ops=ops, batch=None), None).double().cpu()
    assert float(want[1].abs().max()) < 1e-3 * float(want[0].abs().max())
    assert float((got - want).abs().max()) < 1e-4 * float(want.abs().max())


def test_a_norm_with_one_number(ops):
    from tffinfer_b200.parts.norm import RMSNorm
    x = torch.randn(5, 72)
    n = RMSNorm(72, 1e-3, "norm1", one_number=True)
    assert n.weight_specs()["norm1"].shape == ()
    n.load({"norm1": torch.tensor(0.37).cuda()}, ops, torch.float32)
    got = n.forward(x.cuda(), ops, torch.float32).double().cpu()
    assert float((got - P.one_number_norm(x.double(), 0.37, 1e-3)).abs().max()) < 2e-6


# ------------------------------------------------------------------------------ through the engine's own entry point
@pytest.mark.parametrize("dtype,name", [("float32", "a"), ("float32", "b"), ("bfloat16", "a")])
def test_greedy_generation_through_the_engine(dtype, name):
    """Six requests on three state slots and a pool that holds two of them at a time, decode steps replayed as CUDA
    graphs, 60 new tokens each: the scheduler admits, preempts and frees; in 32-bit every request's tokens are those
    of the plain implementation decoding greedily (a token whose two best logits are closer than rounding may
    differ: from there on the rest is not compared)."""
    import tffinfer_b200 as tff
    cfg = config(name)
    sd = weights(cfg)
    rng = random.Random(2)
    prompts = [[rng.randrange(cfg.vocab_size) for _ in range(n)] for n in (3, 40, 17, 64, 9, 25)]
    new = 60
    runner = ModelRunner(config=cfg, tensors=dict(sd), engine_config=EngineConfig(
        dtype=dtype, page_size=PAGE[name], max_cache_tokens=256, max_live_requests=3, use_cuda_graphs=True,
        max_tokens_per_step=48))
    outs = tff.Engine(runner=runner).generate(prompts, max_new_tokens=new)
    assert all(len(o) == new for o in outs)
    if dtype != "float32":
        return
    cj = cfg.to_json_dict()
    compared = 0
    for p, o in zip(prompts, outs):
        logits = P.forward(cj, sd, list(p) + o[:-1])[len(p) - 1:]       # along the engine's own tokens
        top = torch.topk(logits, 2, dim=-1).values
        for i in range(new):
            if float(top[i, 0] - top[i, 1]) < 2e-4 * float(logits[i].abs().max()):
                break
            assert int(logits[i].argmax()) == o[i], f"token {i} differs"
            compared += 1
    assert compared > 120


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_graph_replay(dtype):
    """Two requests decoded for 300 tokens, one token a step, the steps replayed as CUDA graphs: the windows pass over
    decoded tokens many times, pages between the kept ones and the window are given back (and poisoned), and the states
    are carried all the way."""
    cfg = config("a")
    sd = weights(cfg)
    rng = random.Random(4)
    reqs = {r: [rng.randrange(cfg.vocab_size) for _ in range(n + 300)] for r, n in (("r0", 21), ("r1", 3))}
    want = plain_logits(cfg.to_json_dict(), sd, reqs, dtype)
    steps = [([("r0", 0, 21), ("r1", 0, 3)], [])]
    steps += [([("r0", 21 + i, 1), ("r1", 3 + i, 1)], ["r0", "r1"] if i == 299 else []) for i in range(300)]
    r = runner_of(cfg, sd, dtype, 16, 2 * 336, live=2, graphs=True)
    got = run_trace(r, reqs, steps, poison=True)
    assert any(st["graphs"] for st in r._graphs.values()), "the decode steps were not replayed as graphs"
    for q in reqs:
        assert_within(got[q], want[q], f"{dtype}: request {q}")


def test_trace_replay_tool_on_a_model_folder(tmp_path):
    """bin/trace_run on a Gumodra folder written by the random-weights mode: a mixed schedule (portions beside single
    tokens, four live requests, a pool that makes later requests reuse pages and slots) in both number formats."""
    from test_trace_run_gpu import _replay, _max_tokens
    from helpers import steps_to_jsonl
    from tffinfer_b200.weights import write_random_model
    from tffinfer_b200.weights.safetensors_io import SafetensorsFile
    cfg = config("d")
    d = write_random_model(str(tmp_path / "model"), cfg, seed=5)
    f = SafetensorsFile(str(tmp_path / "model" / "model.safetensors"))
    sd = {n: f.tensor(n).clone() for n in f.names()}
    rng = random.Random(9)
    prompts = [70, 3, 130, 41, 18]
    reqs = {f"q{i}": [rng.randrange(cfg.vocab_size) for _ in range(n + 10)] for i, n in enumerate(prompts)}
    steps = trace_mixed(reqs, prompts, max_live=4, page_size=64, pool_tokens=384, chunk=33)
    for dtype in ("float32", "bfloat16"):
        want = plain_logits(cfg.to_json_dict(), sd, reqs, dtype)
        out = tmp_path / dtype
        out.mkdir()
        assert _replay(d, dtype, _max_tokens(reqs, steps), steps_to_jsonl(reqs, steps), str(out)) == 0
        got = {r: [None] * len(t) for r, t in reqs.items()}
        for i, (entries, _) in enumerate(steps):
            rows = sum(n for _, _, n in entries)
            arr = torch.from_numpy(np.fromfile(str(out / f"{i}.f32"), dtype="<f4").reshape(rows, cfg.vocab_size))
            row = 0
            for r, start, n in entries:
                for k in range(n):
                    got[r][start + k] = arr[row]
                    row += 1
        for r in reqs:
            assert_within(torch.stack(got[r]), want[r], f"{dtype}: {r}")


def test_command_line_generates(tmp_path):
    import json
    import os
    import subprocess
    import sys
    from tffinfer_b200.weights import write_random_model
    d = write_random_model(str(tmp_path / "model"), config("b"), seed=1)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([sys.executable, "-m", "tffinfer_b200", d, "--prompt-ids", "1,2,3,4,5", "--prompt-ids", "7,8",
                        "--n-predict", "12", "--max-live", "2", "--max-cache-tokens", "128", "--json"],
                       cwd=root, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    out = json.loads(p.stdout.strip().splitlines()[-1])
    assert [len(o) for o in out["outputs"]] == [12, 12]


# ------------------------------------------------------------------------------ configurations drawn at random
def draw(seed: int):
    """Layer orders, sizes and constants drawn at random, each layer its own: which kernels run (tensor-core or FMA)
    follows from the sizes."""
    rng = random.Random(seed)
    W = rng.choice([64, 96, 128, 192]) if rng.random() < 0.75 else rng.choice([36, 100, 150])
    n = rng.choice([2, 3, 4, 5])
    layers = []
    for _ in range(n):
        count = rng.choice([1, 2, 3, 4])
        E = count * rng.choice([1, 2, 4])
        keep = rng.randint(1, count)
        experts = moe(rng.choice([16, 64, 40]), E, rng.randint(1, min(4, keep * (E // count))), (count, keep), rng.choice([0, 16, 64, 100]))
        m = rng.choice([experts, experts, dense(rng.choice([32, 100, 256])), None])
        if rng.random() < 0.5:
            G = rng.choice([1, 2, 3])
            dim = rng.choice([8, 16, 64, 128, 24, 11])
            rot = rng.choice([0, 2, dim - dim % 2, dim // 2 - (dim // 2) % 2])
            layers.append(att(G * rng.choice([1, 2, 4]), G, dim, rng.choice([0, 1, 5, 16, 33, 64, 100]), rng.choice([0, 1, 4, 16, 35, 70]),
                              rot, scale=rng.choice([None, 0.11, 0.3]), base=rng.choice([1e4, 5e5]), mlp=m))
        else:
            layers.append(mem(rng.choice([1, 2, 4, 3]), rng.choice([8, 16, 32, 100]), rng.choice([8, 16, 64, 36]),
                              cap=rng.choice([2.0, 8.0, 15.0]), mlp=m))
    cfg = GumodraConfig("Gumodra", vocab_size=rng.choice([97, 256, 311, 1000]), hidden_size=W, norm_eps=rng.choice([1e-6, 1e-5]),
                        embed_scale=rng.choice([1.0, 0.2, 11.0]), layers=tuple(layers))
    return cfg, rng.choice([8, 16, 32]), [rng.randint(1, 40), rng.randint(60, 150), rng.randint(2, 230), rng.randint(20, 90)]


@pytest.mark.parametrize("seed", list(range(1, 17)))
def test_random_configuration_matches_plain(seed):
    cfg, page, prompts = draw(seed)
    sd = weights(cfg, seed=seed, sharp=4.0)
    rng = random.Random(50 + seed)
    reqs = {f"r{i}": [rng.randrange(cfg.vocab_size) for _ in range(n + 5)] for i, n in enumerate(prompts)}
    cj = cfg.to_json_dict()
    most = max(-(-len(t) // page) * page for t in reqs.values())
    pool = most + most // 2
    for dtype in ("float32", "bfloat16"):
        want = plain_logits(cj, sd, reqs, dtype)
        for steps, tokens in ((trace_mixed(reqs, prompts, max_live=3, page_size=page, pool_tokens=pool, chunk=48), pool),
                              (trace_portions(reqs, sizes=(64, 2, 17, 130, 3)), most)):
            got = run_trace(runner_of(cfg, sd, dtype, page, tokens, live=3), reqs, steps, poison=True)
            for q in reqs:
                assert_within(got[q], want[q], f"draw {seed} {dtype}: request {q}: {cj}")
