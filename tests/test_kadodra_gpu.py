"""The Kadodra design in the engine against its plain implementation (plain_kadodra.py): every mechanism alone through the
kernel library, and whole models of several small configurations in every cut of the steps.  The configurations differ in
every size and option, with values that are unequal where a model might have them equal (key and value sizes, layers'
heads and windows) and 1 where it might have more (heads, experts, chosen experts, window)."""
import random
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_kadodra as P
from helpers import trace_whole, trace_tail_decode, trace_portions, trace_mixed, run_trace, first_bad
from test_tipezen_gpu import fake_batch
from tffinfer_b200.config import EngineConfig, KadodraConfig, KadodraLayer, KadodraMlp
from tffinfer_b200.config.kadodra_config import KadodraLatent, KadodraLightning
from tffinfer_b200.config.tipezen_config import RotaryConfig
from tffinfer_b200.engine import ModelRunner
from tffinfer_b200.weights.random_init import random_state_dict

pytestmark = pytest.mark.gpu
TOL = {"float32": 3e-5, "bfloat16": 2e-2}
YARN = (4.0, 64.0, 16.0, 2.0)          # factor, original, fast, slow


def lat(heads, dim, rot_dim, vdim, kv_rank, window, scale=None, base=1e4, scaling=YARN, mlp=None):
    return KadodraLayer("latent_attention", latent=KadodraLatent(
        heads, dim, rot_dim, vdim, kv_rank, scale if scale is not None else (dim + rot_dim) ** -0.5,
        RotaryConfig(base, rot_dim, scaling), window), mlp=mlp)


def light(heads, dim, vdim, decay=None, mlp=None):
    decay = decay or tuple(1.0 - 0.5 ** (1 + 2 * i) for i in range(heads))
    return KadodraLayer("lightning", lightning=KadodraLightning(heads, dim, vdim, decay), mlp=mlp)


def dense(ff):
    return KadodraMlp("dense", ff)


def moe(ff, experts, top, limit=0.8):
    return KadodraMlp("moe", ff, experts, top, limit)


def config(name: str) -> KadodraConfig:
    make = lambda **kw: KadodraConfig("Kadodra", **kw)
    if name == "a":      # sizes that take the tensor-core products; a loop over both kinds of layer
        return make(vocab_size=320, hidden_size=128, norm_eps=1e-5, logit_scale=1.5, loop=(1, 3, 2), layers=(
            light(4, 32, 16, mlp=dense(192)), lat(4, 32, 16, 24, 64, 40, mlp=moe(64, 6, 2)),
            light(2, 48, 64, mlp=moe(64, 6, 3)), lat(2, 64, 8, 32, 32, 70, base=3e5, mlp=dense(96))))
    if name == "b":      # odd sizes everywhere: FMA products; windows that no page size divides, every expert chosen, a
        return make(vocab_size=97, hidden_size=52, norm_eps=3e-6, logit_scale=0.3, loop=(0, 4, 2), layers=(      # loop over
            lat(3, 20, 6, 12, 18, 7, scale=0.2, base=1e3, mlp=moe(22, 5, 5, 0.3)), light(3, 12, 20),             # the whole
            lat(3, 20, 6, 12, 18, 13, scale=0.2, base=1e3, scaling=None), light(3, 12, 20, mlp=dense(70))))
    if name == "c":      # one head, one expert, a window of one position and none, values wider than keys, no loop, a
        return make(vocab_size=264, hidden_size=64, norm_eps=1e-6, logit_scale=1.0, layers=(       # decay of one and of zero
            light(1, 8, 96, decay=(1.0,), mlp=moe(48, 1, 1, 2.0)), lat(1, 16, 8, 72, 160, 1, base=5e5, mlp=moe(16, 9, 1)),
            light(2, 40, 8, decay=(0.0, 0.9)), lat(2, 8, 2, 40, 24, 0, mlp=dense(32))))
    if name == "d":      # windows of 64 over pages of 32, a loop of one layer three times, a recurrence first and last
        return make(vocab_size=150, hidden_size=96, norm_eps=1e-6, logit_scale=0.5, loop=(2, 3, 3), layers=(
            light(2, 72, 24, mlp=moe(32, 12, 3, 0.5)), lat(2, 24, 8, 40, 56, 64, mlp=dense(40)),
            lat(8, 16, 32, 16, 128, 33, base=3e5, scaling=(6.0, 128.0, 24.0, 0.5), mlp=moe(32, 12, 4, 0.5)),
            light(8, 8, 8, mlp=moe(16, 7, 2))))
    raise KeyError(name)


PAGE = {"a": 16, "b": 4, "c": 8, "d": 32}
PROMPTS = {"a": [5, 90, 37, 200], "b": [1, 13, 40, 64], "c": [3, 29, 110, 71], "d": [2, 70, 133]}


def weights(cfg, seed=11, sharp=6.0):
    """Random weights with latent scores far from uniform (a key that is wrongly seen or missed moves the logits),
    recurrence inputs large enough for their activations to bend, experts that reach their clipping bounds, and an
    embedding that weighs beside what the layers add."""
    sd = random_state_dict(cfg, seed, "bfloat16", norm_noise=0.2)
    W = cfg.hidden_size
    for n in sd:
        f = 1.0
        if n == "embed":
            f = 40.0
        elif n.endswith((".mix.q", ".mix.dkv", ".mix.k", ".mix.v", ".mix.g")):
            f = sharp * (128 / W) ** 0.5
        elif n.endswith((".mix.uk", ".mix.uv")):
            f = 8.0
        elif n.endswith((".gate", ".mlp.up", ".up")):
            f = 5.0 * (128 / W) ** 0.5
        elif n.endswith((".down", ".mix.o")):
            f = 3.0
        if f != 1.0:
            sd[n] = (sd[n].float() * f).to(torch.bfloat16)
    return sd


def runner_of(cfg, sd, dtype, page, tokens, live=4, graphs=False):
    return ModelRunner(config=cfg, tensors=dict(sd), engine_config=EngineConfig(
        dtype=dtype, page_size=page, max_cache_tokens=tokens, max_live_requests=live, use_cuda_graphs=graphs))


def plain_logits(cj, sd, reqs, dtype):
    """{request: (logits, bar of every position)} of the plain implementation.  In bfloat16 a position's bar is the
    larger of the format's and three times what rounding the rows that enter every product alone moves the plain logits
    there; positions whose bar is raised must be few, or the test says nothing."""
    out = {}
    for r, t in reqs.items():
        want = P.forward(cj, sd, t)
        bar = torch.full((want.shape[0],), TOL[dtype], dtype=torch.float64)
        if dtype == "bfloat16":
            moved = P.forward(cj, sd, t, round_inputs=True)
            bar = torch.maximum(bar, 3.0 * (moved - want).abs().amax(dim=-1) / want.abs().amax(dim=-1))
        out[r] = (want, bar)
    raised = sum(int((b > TOL[dtype]).sum()) for _, b in out.values())
    assert raised <= 2 + sum(w.shape[0] for w, _ in out.values()) // 3, f"{raised} ill-conditioned positions: too many for a test"
    return out


def assert_within(got, want_bar, what):
    want, bar = want_bar
    err = torch.nan_to_num((got.double() - want).abs().amax(dim=-1) / want.abs().amax(dim=-1).clamp_min(1e-30), nan=float("inf"))
    bad = torch.nonzero(err > bar)
    assert bad.numel() == 0, f"{what}: token {int(bad[0])} off by {float(err[int(bad[0])]):.3g} (bar {float(bar[int(bad[0])]):.3g})"


def requests_of(cfg, name, decoded, seed=5):
    rng = random.Random(seed)
    return {f"r{i}": [rng.randrange(cfg.vocab_size) for _ in range(n + decoded)] for i, n in enumerate(PROMPTS[name])}


@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_cut_matches_plain(name, dtype):
    """Whole prompts, a tail decoded token by token, portions down to two tokens, and mixed batches in a pool small
    enough that pages and slots are used again (released pages are poisoned, the pool's windows pass over them)."""
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


def test_the_residual_after_every_run_of_a_layer():
    """Looped passes and the embedding output that joins them: the residual after each layer run, in 32-bit."""
    for name in ("a", "b", "d"):
        cfg = config(name)
        sd = weights(cfg)
        toks = requests_of(cfg, name, 0)["r1"]
        want, got = [], []
        P.forward(cfg.to_json_dict(), sd, toks, layers_out=want)
        from tffinfer_b200.engine import StepEntry
        r = runner_of(cfg, sd, "float32", PAGE[name], 256)
        r.model.layer_hook = lambda e, x: got.append(x.double().cpu().clone())
        r.add_request("r")
        r.step([StepEntry("r", toks, [])])
        assert len(got) == len(want) == len(cfg.runs())
        for i, (a, b) in enumerate(zip(got, want)):
            assert float((a - b).abs().max()) < 2e-5 * float(b.abs().max()), f"{name}: layer run {i}"


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


@pytest.mark.parametrize("H,D,V", [(2, 32, 16), (3, 12, 20), (1, 128, 128), (4, 7, 33), (2, 8, 130), (1, 200, 260), (1, 300, 40)])
@pytest.mark.parametrize("silu", [True, False])
@pytest.mark.parametrize("rounded", [False, True])
def test_recurrence_steps_slots_and_a_far_key(ops, H, D, V, silu, rounded):
    """The recurrence through four steps (a long portion, short portions, one token each twice: the decode kernel), slots
    out of order, other slots poisoned and the requests' own slots full of NaN at the start (a request that brings
    position 0 starts from zeros), q, k and v column blocks of wider rows.  In the first request one key far back is
    planted under a decay near one, with a query aimed at it: its value must arrive at the last token.  The last sizes
    do not fit the chunked form and run token by token.  ``rounded`` is the chunk form on the tensor cores: behind the
    rounding of q, k and v (inputs that bfloat16 holds exactly have none) it must be as close as the float32 form."""
    dev = "cuda"
    g = torch.Generator().manual_seed(H * D + V)
    cuts = [[150, 3, 1], [2, 70, 1], [1, 1, 1], [1, 1, 1]]
    total = [sum(c[i] for c in cuts) for i in range(3)]
    decay = torch.tensor([0.999] + [0.3 + 0.6 * i / max(H - 1, 1) for i in range(1, H)])
    slots = [3, 0, 2]
    state = torch.full((5, H, D, V), float("nan"), device=dev)
    seqs = [[torch.randn(n, H * D, generator=g), torch.randn(n, H * D, generator=g), torch.randn(n, H * V, generator=g)]
            for n in total]
    q0, k0, _ = seqs[0]
    k0[:, 0] = 0.0
    k0[4, 0] = 20.0
    q0[-1, :D] = 0.0
    q0[-1, 0] = 20.0
    seqs = [[x.to(torch.bfloat16).float() for x in s] for s in seqs]
    f = P.silu if silu else (lambda x: x)
    want = []
    for q, k, v in seqs:
        q, k, v = f(q.double()), f(k.double()), f(v.double())
        want.append(torch.cat([P.constant_decay_recurrence(q[:, h * D:(h + 1) * D], k[:, h * D:(h + 1) * D],
                                                           v[:, h * V:(h + 1) * V], float(decay[h]))[0] for h in range(H)], dim=-1))
    got = [[] for _ in seqs]
    starts = [0, 0, 0]
    q_off, k_off, v_off = 4, 4 + H * D, 4 + 2 * H * D + 3
    for lens in cuts:
        b = fake_batch(lens, starts, dev, 8, slots=slots)
        part = [torch.cat([s[j][st:st + n] for s, n, st in zip(seqs, lens, starts)]) for j in range(3)]
        T = part[0].shape[0]
        proj = torch.full((T, v_off + H * V + 5), float("nan"))
        proj[:, q_off:q_off + H * D], proj[:, k_off:k_off + H * D], proj[:, v_off:v_off + H * V] = part
        out = torch.full((T, H * V), float("nan"), device=dev)
        ops.retention_raw(proj.to(dev), q_off, k_off, v_off, silu, state, b, decay.to(dev), out, H, D, V, rounded=rounded)
        torch.cuda.synchronize()
        row = 0
        for i, n in enumerate(lens):
            got[i].append(out[row:row + n].double().cpu())
            row += n
        starts = [s + n for s, n in zip(starts, lens)]
    for i in range(3):
        err = float((torch.cat(got[i]) - want[i]).abs().max()) / float(want[i].abs().max())
        assert err < (1e-2 if rounded and silu else 2e-5), f"request {i} off by {err:.3g}"
    v4 = f(seqs[0][2][4, :V].double())                       # the far key's value is what the last output of head 0 holds
    last = torch.cat(got[0])[-1, :V]
    assert float(torch.dot(last, v4) / (last.norm() * v4.norm())) > 0.999
    assert torch.isnan(state[1]).all() and torch.isnan(state[4]).all()          # nobody's slots were left alone


@pytest.mark.parametrize("D,V", [(64, 96), (20, 36)])
def test_decode_kernel_and_chunks_agree(ops, D, V):
    """Single tokens through the chunked form and through the decode kernel leave the same outputs and states."""
    dev, H = "cuda", 3
    g = torch.Generator().manual_seed(D)
    decay = torch.tensor([0.5, 0.9, 0.99]).to(dev)
    states = [torch.randn(4, H, D, V, generator=g).to(dev)] * 1
    states.append(states[0].clone())
    proj = torch.randn(3, H * (2 * D + V), generator=g).to(dev)
    outs = []
    for st, ch in zip(states, (False, True)):
        b = fake_batch([1, 1, 1], [70, 64, 127], dev, 8, slots=[2, 0, 1])
        out = torch.full((3, H * V), float("nan"), device=dev)
        ops.retention_raw(proj, 0, H * D, 2 * H * D, True, st, b, decay, out, H, D, V, chunked=ch)
        outs.append(out)
    torch.cuda.synchronize()
    assert torch.allclose(outs[0], outs[1], rtol=1e-5, atol=1e-4) and torch.allclose(states[0], states[1], rtol=1e-6, atol=1e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [96, 50, 640, 2048])
def test_norm_over_all_heads_with_a_sigmoid_gate_clears_the_rows(ops, dtype, width):
    """One group as wide as the row (a warp's, a block's), the sigmoid, and the projection's rows set to zero where
    they are an accumulator buffer, columns beside the gate's too."""
    dev = "cuda"
    g = torch.Generator().manual_seed(width)
    T, goff = 7, 36
    o, rows = torch.randn(T, width, generator=g) * 3, torch.randn(T, goff + width + 4, generator=g)
    w = 1 + 0.3 * torch.randn(width, generator=g)
    want = P.rms_norm(o.double(), w.double(), 1e-5) * torch.sigmoid(rows[:, goff:goff + width].double())
    out = torch.full((T, width), float("nan"), device=dev, dtype=dtype)
    buf = ops.projection_buffer(T, goff + width + 4, torch.device(dev), torch.bfloat16, use=f"test {width} {dtype}")
    for clear in ((0, buf.shape[1]), (goff, goff + width)):
        buf.copy_(rows)
        ops._acc_zero[buf.data_ptr()] = False
        ops.gated_norm(o.to(dev), width, buf, goff, w.to(dev), 1e-5, False, out, clear_cols=clear, last_reader=clear[0] == 0,
                       gate_act="sigmoid")
        torch.cuda.synchronize()
        err = float((out.double().cpu() - want).abs().max()) / float(want.abs().max())
        assert err < (1e-5 if dtype == torch.float32 else 1e-2)
        assert not buf[:, clear[0]:clear[1]].any() and ops._acc_zero[buf.data_ptr()] == (clear[0] == 0)
        assert clear[0] == 0 or torch.equal(buf[:, :goff].cpu(), rows[:, :goff])
    buf.zero_()
    ops._acc_zero[buf.data_ptr()] = True


def _latent_part(ops, dtype, W, H, D, R, V, C, window, scale, rot, w):
    from tffinfer_b200.parts.latent import LatentAttention
    from tffinfer_b200.parts.position import ScaledRotary
    dt = getattr(torch, dtype)
    m = LatentAttention(W, H, D, R, V, 0, C, 1e-5, softmax_scale=scale, window=window, sink=True)
    m.load({n: (v.float() if v.dim() == 1 else v.to(dt)).cuda().contiguous() for n, v in w.items()}, ops, dt)
    sc = rot.get("scaling")
    pos = ScaledRotary(rot["dims"], rot["base"], "halves", scaling=tuple(sc[k] for k in ("factor", "original", "fast", "slow")) if sc else None)
    pos.prepare(ops, "cuda", 0)
    return m, pos


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D,R,V,C,window", [(24, 12, 20, 40, 0), (24, 8, 16, 40, 50), (32, 16, 24, 64, 100), (16, 8, 8, 24, 1)])
def test_latent_attention_windows_sinks_and_far_keys(ops, dtype, D, R, V, C, window):
    """A latent attention alone, queries straight from the input: 700 tokens in portions that end inside pages, then
    single tokens, with sharp queries (a missed key among hundreds shows), windows over pages they have passed (poisoned
    before every step, as pages that were given back), learned sinks from overwhelming to negligible; then the whole
    prompt as one step, which in bfloat16 is the form with per-head keys."""
    from tffinfer_b200.parts.base import LayerContext
    dev, dt = "cuda", getattr(torch, dtype)
    g = torch.Generator().manual_seed(D + V + window)
    W, H, page, T = 64, 3, 16, 700
    rot = {"base": 2e3, "dims": R, "scaling": {"factor": 3.0, "original": 96, "fast": 12.0, "slow": 1.0}}
    h = torch.randn(T, W, generator=g).to(dt)
    shapes = {"q": (H * (D + R), W), "dkv": (C + R, W), "uk": (H * D, C), "uv": (H * V, C), "o": (W, H * V)}
    w = {n: (torch.randn(*s, generator=g) * s[1] ** -0.5 * (4.0 if n == "q" else 1.0)).to(torch.bfloat16) for n, s in shapes.items()}
    w["dkv.norm"] = (1.0 + 0.2 * torch.randn(C, generator=g)).to(torch.bfloat16)
    w["sink"] = torch.tensor([-30.0, 1.5, 6.0]).to(torch.bfloat16)
    part, pos = _latent_part(ops, dtype, W, H, D, R, V, C, window, 0.3, rot, w)
    m = {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": C, "scale": 0.3, "rot": rot, "mask": {"size": window}}
    want = P.latent_mixer(h.double(), torch.arange(T), {"p." + n: v.double() for n, v in w.items()}, "p", m, 1e-5)
    without = P.latent_mixer(h.double(), torch.arange(T), {"p." + n: (v.double() if n != "sink" else v.double() - 1e4) for n, v in w.items()}, "p", m, 1e-5)
    assert float((want - without).abs().max() / want.abs().max()) > 0.1        # the sinks matter
    cache = torch.full((T // page + 2, 1, 1, 1, page, C + R), float("nan"), dtype=dt, device=dev)
    table = torch.arange(T // page + 1, dtype=torch.int32, device=dev).reshape(1, -1)
    got, at, bar = [], 0, 3e-5 if dtype == "float32" else 3e-2
    for n in (37, 300, 2, 345) + (1,) * 16:
        t = table.clone()
        if window:
            gone = max(0, at - window + 1) // page
            t[0, :gone] = -1
            cache[:gone] = float("nan")
        batch = fake_batch([n], [at], dev, page)
        ctx = LayerContext(batch=batch, ops=ops, kv_cache=cache, kv_layer=0, block_table=t, page_size=page, position=pos, shared={})
        got.append(part.forward(h[at:at + n].to(dev).contiguous(), ctx, None).double().cpu().clone())
        ops.reset_accumulators()
        at += n
    assert at == T
    err = float((torch.cat(got) - want).abs().max() / want.abs().max())
    assert err < bar, f"portions off by {err:.3g}"
    cache.fill_(float("nan"))
    batch = fake_batch([T], [0], dev, page)
    batch.h_pos_start = np.array([0])
    shared = {}
    ctx = LayerContext(batch=batch, ops=ops, kv_cache=cache, kv_layer=0, block_table=table, page_size=page, position=pos, shared=shared)
    whole = part.forward(h.to(dev).contiguous(), ctx, None).double().cpu().clone()
    ops.reset_accumulators()
    err = float((whole - want).abs().max() / want.abs().max())
    assert err < bar, f"the whole prompt off by {err:.3g}"
    assert (dtype == "bfloat16" and (D + R) % 8 == 0 and V % 8 == 0 and C % 8 == 0) == bool(shared), "which form ran is not the one expected"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [24, 25, 1, 64])
def test_keys_just_inside_and_outside_a_window(ops, dtype, window):
    """One key stands out by content: the query at distance window - 1 finds it, the one at distance window does not.  A
    batch of decoded tokens and of portions at page borders, in one launch, the key range whole and in shares; the sink
    takes its share of the weight in both."""
    dev, dt = "cuda", getattr(torch, dtype)
    g = torch.Generator().manual_seed(window)
    H, D, V, page = 3, 40, 24, 8
    cases = []                                     # (tokens cached ahead, tokens of the step, planted key)
    for last in (70, 79, 80, 151):                 # position of the request's last token, alone or at the end of a portion
        for gap in (window - 1, window):
            for n in (1, 9):
                if last - gap >= 0:
                    cases.append((last + 1 - n, n, last - gap))
    keys, qs = [], []
    sink = torch.tensor([0.0, 2.0, -5.0])
    for start, n, plant in cases:
        k = torch.randn(start + n, D, generator=g) * 0.3
        k[:, 0] = 0.0
        k[plant] = 0.0
        k[plant, 0] = 10.0
        k[plant, 1:V] = torch.randn(V - 1, generator=g)      # its value: the first V elements
        q = torch.randn(n, H, D, generator=g) * 0.3
        q[-1] = 0.0
        q[-1, :, 0] = 3.0
        keys.append(k.to(dt).double())
        qs.append(q.to(dt).double())
    want = []
    for (start, n, plant), k, q in zip(cases, keys, qs):
        seen = P.window_mask(torch.arange(start + n), window)[start:]
        want.append(torch.stack([P.softmax_with_sink((q[:, h] @ k.T) * 0.5, seen, sink[h].double()) @ k[:, :V] for h in range(H)], dim=1))
    b = fake_batch([n for _, n, _ in cases], [s for s, _, _ in cases], dev, page)
    cache = torch.full((b.pages + 1, 1, 1, 1, page, D), float("nan"), dtype=dt, device=dev)
    table = b.block_table.clone()
    for i, ((start, n, _), k) in enumerate(zip(cases, keys)):
        for p in range(start + n):
            if p > start - window:                 # keys behind every window of the step are gone
                cache[table[i, p // page], 0, 0, 0, p % page] = k[p].to(dt)
        for j in range(max(0, start - window + 1) // page):
            table[i, j] = -1
    q = torch.cat(qs).reshape(-1, H * D).to(dt).to(dev).contiguous()
    for splits in (1, 2, 4):
        out = torch.full((q.shape[0], H * V), float("nan"), device=dev, dtype=dt)
        ops.attention_tile(q, b, table, cache, 0, page, out, H, 1, D, V, 0.5, window=window, sink=sink.to(dev), num_splits=splits)
        torch.cuda.synchronize()
        row = 0
        for (start, n, plant), wnt in zip(cases, want):
            o = out[row:row + n].double().cpu().reshape(n, H, V)
            row += n
            err = float((o - wnt).abs().max()) / 10.0
            assert err < (1e-5 if dtype == "float32" else 1e-2), (window, splits, start, n, plant, err)
            found = float(o[-1, 0, 0])
            assert (found > 9.9) == (start + n - 1 - plant < window), (window, splits, start, n, plant, found)


@pytest.mark.parametrize("H,G,D,V,rest", [(3, 3, 192, 128, 64), (2, 2, 192, 128, 0), (4, 4, 80, 48, 16), (6, 2, 128, 64, 0),
                                          (3, 3, 40, 24, 0), (2, 2, 136, 8, 8), (16, 16, 192, 128, 64), (1, 1, 8, 8, 0)])
@pytest.mark.parametrize("window", [0, 1, 100, 64])
def test_attention_over_plain_rows_of_whole_prompts(ops, H, G, D, V, rest, window):
    """The tcgen05 kernel over keys and values in plain rows: unequal prompts in one step (ends inside key blocks and
    tiles; the last case has more tiles than SMs, two a CTA), keys whose last part all heads share, window edges, sinks,
    a cap; the buffers hold nothing beyond the step's rows."""
    dev = "cuda"
    g = torch.Generator().manual_seed(D + window)
    lens = [700, 1, 64, 333, 130] if H < 16 else [2050, 129]
    T = sum(lens)
    q = torch.randn(T, H * D, generator=g).to(torch.bfloat16)
    kh = D - rest
    k = torch.randn(T, G * kh, generator=g).to(torch.bfloat16)
    r = torch.randn(T, 24 + rest, generator=g).to(torch.bfloat16) if rest else None
    v = torch.randn(T, G * V, generator=g).to(torch.bfloat16)
    sink = torch.randn(H, generator=g) * 2
    b = fake_batch(lens, [0] * len(lens), dev, 16)
    scale = 2.0 * D ** -0.5                                  # sharp: one key of hundreds matters
    for cap, sk in ((0.0, sink), (3.0, None)):
        out = torch.full((T, H * V), float("nan"), device=dev, dtype=torch.bfloat16)
        ops.attention_dense(q.to(dev), b, k.to(dev), kh, r.to(dev) if rest else None, 24, v.to(dev), out, H, G, D, V, scale,
                            window=window, softcap=cap, sink=sk.to(dev) if sk is not None else None)
        torch.cuda.synchronize()
        ops.check_errors()
        t0 = 0
        for n in lens:
            rows = slice(t0, t0 + n)
            t0 += n
            seen = P.window_mask(torch.arange(n), window)
            for h in range(0, H, max(1, H // 3)):
                gi = h // (H // G)
                key = k[rows, gi * kh:(gi + 1) * kh].double()
                if rest:
                    key = torch.cat([key, r[rows, 24:].double()], dim=1)
                s = (q[rows, h * D:(h + 1) * D].double() @ key.T) * scale
                if cap:
                    s = cap * torch.tanh(s / cap)
                want = P.softmax_with_sink(s, seen, sk[h].double() if sk is not None else None) @ v[rows, gi * V:(gi + 1) * V].double()
                err = float((out[rows, h * V:(h + 1) * V].double().cpu() - want).abs().max()) / float(want.abs().max())
                assert err < 1.5e-2, (n, h, cap, err)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,top,ff,W,T,limit", [(5, 1, 24, 40, 70, 0.4), (7, 3, 64, 128, 130, 0.8), (3, 3, 10, 52, 9, 0.2),
                                                (1, 1, 16, 64, 3, 1.0), (16, 2, 64, 128, 600, 0.5), (70, 4, 128, 64, 700, 0.6)])
def test_experts_chosen_by_a_table(ops, dtype, E, top, ff, W, T, limit):
    """Every kernel of the routed products (FMA, mma.sync, tcgen05 from 1,024 pairs) behind the table, with gates and ups
    beyond the limit on both sides, token ids that repeat (one expert gets most rows) and experts nobody chooses."""
    from tffinfer_b200.parts.moe import RoutedExperts
    dev, dt = "cuda", getattr(torch, dtype)
    g = torch.Generator().manual_seed(E * 100 + top)
    rows = 50
    table = torch.rand(rows, E, generator=g).argsort(dim=1)[:, :top].to(torch.int32)
    tokens = torch.randint(0, rows, (T,), generator=g, dtype=torch.int32)
    tokens[::3] = 7
    w = {"m.table": table}
    for e in range(E):
        for n, s in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff))):
            w[f"m.e{e}.{n}"] = (torch.randn(*s, generator=g) * s[1] ** -0.5).to(torch.bfloat16)
    part = RoutedExperts(W, ff, E, top, activation="clipped_swish", activation_limit=limit, router_score="table",
                         table_rows=rows, prefix="m")
    part.load({k[2:]: (v if k.endswith("table") else v.to(dt)).to(dev) for k, v in w.items()}, ops, dt)
    h = torch.randn(T, W, generator=g).to(torch.bfloat16)
    res = torch.randn(T, W, generator=g)
    wd = {k: (v.double() if v.is_floating_point() else v) for k, v in w.items()}
    mlp = {"router": {"experts": E, "top": top}, "expert": {"limit": limit}}
    want = res.double() + P.tabled_experts(h.double(), tokens, wd, "m", mlp)
    loose = res.double() + P.tabled_experts(h.double(), tokens, wd, "m", dict(mlp, expert={"limit": 1e9}))
    assert float((want - loose).abs().max()) > 0.1
    ctx = SimpleNamespace(ops=ops, batch=SimpleNamespace(token_ids=tokens.to(dev)))
    for _ in range(2):                                       # twice: nothing is left over from the first call
        out = res.clone().to(dev)
        part.forward(h.to(dt).to(dev), ctx, out)
        torch.cuda.synchronize()
        err = float((out.double().cpu() - want).abs().max()) / float((want - res.double()).abs().max())
        assert err < (2e-5 if dtype == "float32" else 2e-2), f"off by {err:.3g}"
    alone = part.forward(h.to(dt).to(dev), ctx, None)        # without a residual
    assert float((alone.double().cpu() + res.double() - want).abs().max()) < (1e-4 if dtype == "float32" else 5e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T", [1, 9, 40, 300])
def test_dense_feed_forward_with_the_square_of_relu(ops, dtype, T):
    from tffinfer_b200.parts.mlp import PlainMLP
    dt = getattr(torch, dtype)
    for W, ff in ((64, 136), (52, 70)):
        g = torch.Generator().manual_seed(T)
        up, down = (torch.randn(ff, W, generator=g) * W ** -0.5).to(dt), (torch.randn(W, ff, generator=g) * ff ** -0.5).to(dt)
        part = PlainMLP(W, ff)
        part.load({"up": up.cuda(), "down": down.cuda()}, ops, dt)
        h, res = torch.randn(T, W, generator=g).to(dt), torch.randn(T, W, generator=g)
        want = res.double() + P.dense_ff(h.double(), {"m.up": up.double(), "m.down": down.double()}, "m")
        ctx = SimpleNamespace(ops=ops)
        out = part.forward(h.cuda(), ctx, res.clone().cuda())
        alone = part.forward(h.cuda(), ctx, None).double().cpu().clone()
        ops.reset_accumulators()
        for got in (out.double().cpu(), alone + res.double()):
            assert float((got - want).abs().max()) < (2e-5 if dtype == "float32" else 3e-2) * float(want.abs().max())


def test_both_sublayers_read_one_norm(ops):
    """The arrangement x + (mixer(h) + ff(h)), h = norm(x): the feed-forward must not see what the mixer added."""
    from tffinfer_b200.parts.block import ParallelSharedNormBlock
    from tffinfer_b200.parts.norm import RMSNorm
    g = torch.Generator().manual_seed(3)
    x, w = torch.randn(9, 72, generator=g), 1 + 0.2 * torch.randn(72, generator=g)

    class Adds:
        def __init__(self, f):
            self.f = f

        def forward(self, h, ctx, residual):
            residual += self.f * h.float()
            return residual

    n = RMSNorm(72, 1e-5, "norm1")
    n.load({"norm1": w.cuda()}, ops, torch.float32)
    ctx = SimpleNamespace(ops=ops)
    h = P.rms_norm(x.double(), w.double(), 1e-5)
    for ff, f in ((Adds(1.0), 101.0), (None, 100.0)):
        got = ParallelSharedNormBlock(Adds(100.0), ff, n).forward(x.cuda().clone(), ctx, torch.float32).double().cpu()
        assert float((got - (x.double() + f * h)).abs().max()) < 1e-4 * f
    with pytest.raises(ValueError):
        ParallelSharedNormBlock(Adds(1.0), None, n, ffn_norm=n)


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
    for p, o in zip(prompts[:3], outs[:3]):
        seq = list(p)
        for i in range(new):
            logits = P.forward(cj, sd, seq)[-1]
            top = torch.topk(logits, 2).values
            if float(top[0] - top[1]) < 1e-3 * float(logits.abs().max()):
                break
            assert int(logits.argmax()) == o[i], f"token {i} differs"
            seq.append(o[i])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_graph_replay(dtype):
    """Two requests decoded for 300 tokens, one token a step, the steps replayed as CUDA graphs: the windows pass over
    decoded tokens many times, pages are given back behind them (and poisoned), and the states are carried all the way."""
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
    """bin/trace_run on a Kadodra folder written by the random-weights mode: a mixed schedule (portions beside single
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
    """Layer orders, sizes and constants drawn at random, each layer its own: which products run (tensor-core or FMA)
    follows from the sizes."""
    rng = random.Random(seed)
    W = rng.choice([64, 96, 128, 192]) if rng.random() < 0.75 else rng.choice([36, 100, 150])
    n = rng.choice([2, 3, 4, 5])
    layers = []
    for _ in range(n):
        E = rng.choice([1, 4, 8, 13])
        m = rng.choice([moe(rng.choice([16, 64, 40]), E, rng.randint(1, min(E, 4)), rng.choice([0.3, 0.9, 7.0])),
                        dense(rng.choice([32, 100, 256])), moe(64, 8, 2), None])
        if rng.random() < 0.5:
            dim, rot = rng.choice([8, 16, 32, 24, 11]), rng.choice([2, 4, 8, 16, 32])
            layers.append(lat(rng.choice([1, 2, 4, 8, 3]), dim, rot, rng.choice([8, 16, 40, 64]), rng.choice([16, 32, 72, 128, 27]),
                              rng.choice([0, 1, 5, 16, 33, 64, 100]), scale=rng.choice([None, 0.11, 0.3]),
                              base=rng.choice([1e4, 5e5]), scaling=rng.choice([None, YARN, (8.0, 256.0, 32.0, 1.0)]), mlp=m))
        else:
            H = rng.choice([1, 2, 4, 3])
            layers.append(light(H, rng.choice([8, 16, 32, 100]), rng.choice([8, 16, 64, 36]),
                                decay=tuple(rng.choice([0.2, 0.7, 0.95, 0.999]) for _ in range(H)), mlp=m))
    a = rng.randrange(n)
    loop = rng.choice([None, (a, rng.randint(a + 1, n), rng.choice([1, 2, 3]))])
    cfg = KadodraConfig("Kadodra", vocab_size=rng.choice([97, 256, 311, 1000]), hidden_size=W, norm_eps=rng.choice([1e-6, 1e-5]),
                        logit_scale=rng.choice([1.0, 0.2, 3.0]), loop=loop, layers=tuple(layers))
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
