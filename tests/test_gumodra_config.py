"""Host side of the Gumodra design (no GPU): configuration round trip, defaults and errors; the description's tensor names,
cache needs and parts; and the plain implementation against itself (the memory in two halves and by its closed form, the
mask's edges, the sink, groups of experts)."""
import copy

import pytest
import torch

import plain_gumodra as P
from tffinfer_b200.config import GumodraConfig, ConfigError
from tffinfer_b200.parts import Model, KVNeed, StateNeed
from tffinfer_b200.registry import get_architecture
from tffinfer_b200.weights.random_init import random_state_dict
import tffinfer_b200.models  # noqa: F401


def sample_json():
    attention = {"heads": 6, "kv_heads": 3, "dim": 20, "vdim": 20, "scale": 0.2, "mask": {"size": 11, "keep_first": 5},
                 "rot": {"base": 1000.0, "dims": 6}}
    memory = {"heads": 2, "dim": 10, "vdim": 14, "gate_cap": 3.5}
    moe = {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}},
           "shared": {"ff": 40}}
    return {"architecture": "Gumodra", "vocab": 83, "width": 52, "norm": {"eps": 3e-6}, "embedding": {"scale": 7.5},
            "layers": [{"type": "attention", "mixer": attention, "mlp": {"kind": "dense", "ff": 70}},
                       {"type": "mlstm", "mixer": memory, "mlp": moe},
                       {"type": "attention", "mixer": dict(attention, heads=3, mask={"size": 1, "keep_first": 0}), "mlp": None},
                       {"type": "mlstm", "mixer": memory, "mlp": None}]}


def test_round_trip_and_defaults():
    cj = sample_json()
    cfg = GumodraConfig.from_json_dict(cj)
    assert cfg.to_json_dict() == cj
    a, m = cfg.layers[0].attention, cfg.layers[1].mlp
    assert (a.window, a.keep_first, a.kv_heads) == (11, 5, 3) and m.groups == (3, 2) and m.shared_ff == 40
    d = copy.deepcopy(cj)
    for k in ("mask", "kv_heads", "vdim", "rot"):
        del d["layers"][0]["mixer"][k]
    del d["embedding"], d["layers"][1]["mlp"]["shared"], d["layers"][1]["mlp"]["router"]["groups"], d["layers"][2]["mlp"]
    del d["layers"][2]["mixer"]["mask"]["keep_first"]
    c2 = GumodraConfig.from_json_dict(d)
    a, m = c2.layers[0].attention, c2.layers[1].mlp
    assert (a.window, a.keep_first, a.kv_heads, a.rot) == (0, 0, 6, None) and c2.embed_scale == 1.0
    assert m.groups == (1, 1) and m.shared_ff == 0 and c2.layers[2].mlp is None and c2.layers[2].attention.keep_first == 0
    assert GumodraConfig.from_json_dict(c2.to_json_dict()) == c2


@pytest.mark.parametrize("edit,word", [
    (lambda d: d["layers"][1].__setitem__("type", "retention"), "type"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("kv_heads", 4), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("vdim", 24), "vdim"),
    (lambda d: d["layers"][0]["mixer"]["rot"].__setitem__("dims", 22), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].__setitem__("dims", 5), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].__setitem__("scaling", {"factor": 2.0, "original": 8, "fast": 2, "slow": 1}), "rot"),
    (lambda d: d["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "size"),
    (lambda d: d["layers"][0]["mixer"]["mask"].__setitem__("keep_first", -1), "keep_first"),
    (lambda d: d["layers"][1]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("gate_cap", 0.0), "gate_cap"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("dim", 0), "dim"),
    (lambda d: d["layers"][1]["mlp"]["router"].__setitem__("top", 7), "top"),
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].__setitem__("count", 4), "groups"),
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].__setitem__("keep", 1), "groups"),
    (lambda d: d["layers"][1]["mlp"]["shared"].__setitem__("ff", 0), "ff"),
    (lambda d: d["layers"][0]["mlp"].__setitem__("kind", "routed"), "kind"),
    (lambda d: d.__setitem__("layers", []), "layers"),
    (lambda d: d.pop("vocab"), "vocab"),
    (lambda d: d["norm"].pop("eps"), "eps"),
])
def test_errors_name_the_key(edit, word):
    d = sample_json()
    edit(d)
    with pytest.raises(ConfigError) as e:
        GumodraConfig.from_json_dict(d)
    assert word in str(e.value)


def test_description_names_needs_and_parts():
    cfg = GumodraConfig.from_json_dict(sample_json())
    m = Model(get_architecture("Gumodra").describe(cfg))
    t = m.expected_tensors()
    assert t["embed"].shape == t["head"].shape == (83, 52) and t["final.norm"].shape == t["l0.norm1"].shape == ()
    assert t["l0.mix.q"].shape == (120, 52) and t["l0.mix.k"].shape == (60, 52) and "l0.mix.v" not in t
    assert t["l0.mix.q.b"].shape == (120,) and t["l0.mix.o.b"].shape == (52,) and t["l0.mix.sink"].shape == (6,)
    assert t["l0.mix.k.norm"].shape == (20,) and t["l0.rg1"].shape == t["l0.rg2"].shape == (52, 52)
    assert t["l1.mix.v"].shape == (28, 52) and t["l1.mix.i"].shape == (2, 52) and t["l1.mix.f.b"].shape == (2,)
    assert t["l1.mix.norm"].shape == (28,) and t["l1.mlp.correction"].shape == (6,) and t["l1.mlp.e5.down"].shape == (52, 24)
    assert t["l1.mlp.shared.up"].shape == (40, 52) and t["l1.mlp.shared.sg"].shape == (1, 52)
    assert t["l2.rg2"].optional and t["l2.rg2.b"].optional and not t["l2.rg1"].optional and not t["l0.rg2"].optional
    kv0, st, kv2, _ = m.cache_needs()
    assert kv0 == KVNeed(3, 20, 11, keep_first=5) and kv2 == KVNeed(3, 20, 1)
    assert isinstance(st, StateNeed) and st.self_starting and st.shape[0] >= 2 * (140 + 10 + 1) and st.shape[0] % 4 == 0
    assert {"mlstm", "streams", "moe", "qkv_finish", "attention_prefill"} <= set(m.kernel_files())
    sd = random_state_dict(cfg, 3, "bfloat16")
    assert set(sd) == {n for n, s in t.items() if not s.optional}
    assert P.forward(cfg.to_json_dict(), sd, [1, 2, 3, 4]).shape == (4, 83)


def test_plain_memory_in_halves_and_by_its_closed_form():
    """The running maximum only moves factors between numerator and denominator: without it (and without the 1e-6) the
    output is sum_s w_s (q.k_s) v_s / max(|sum_s w_s q.k_s|, 1), w_s the product of the gates' exponentials."""
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(20, n, generator=g).double() for n in (5, 5, 7))
    i, f = torch.randn(20, generator=g).double() * 2, -torch.rand(20, generator=g).double()
    whole, end = P.mlstm_recurrence(q, k, v, i, f)
    a, st = P.mlstm_recurrence(q[:9], k[:9], v[:9], i[:9], f[:9])
    b, end2 = P.mlstm_recurrence(q[9:], k[9:], v[9:], i[9:], f[9:], st)
    assert torch.allclose(whole, torch.cat([a, b]), atol=1e-12) and all(torch.allclose(x, y) for x, y in zip(end, end2))
    F = torch.cumsum(f, 0)
    for t in range(20):
        w = torch.exp(F[t] - F[:t + 1] + i[:t + 1]) * (k[:t + 1] @ q[t])
        assert torch.allclose(whole[t], (w @ v[:t + 1]) / torch.clamp(w.sum().abs(), min=1.0), atol=1e-4)


def test_plain_mask_sink_and_groups():
    pos = torch.arange(12)
    seen = P.seen_keys(pos, 3, 2)
    assert seen[9].nonzero().flatten().tolist() == [0, 1, 7, 8, 9] and seen[1].nonzero().flatten().tolist() == [0, 1]
    assert P.seen_keys(pos, 0, 4)[7].tolist() == [True] * 8 + [False] * 4
    s = torch.zeros(1, 3, dtype=torch.float64)
    w = P.sink_softmax(s, torch.tensor([[True, True, False]]), torch.tensor(0.0).double())
    assert torch.allclose(w, torch.tensor([[1 / 3, 1 / 3, 0.0]]).double())
    score = torch.tensor([[0.4, 0.1, 0.3, 0.2]]).double()
    none = torch.zeros(4).double()
    assert P.choose(score, none, (1, 1), 2).tolist() == [[0, 2]]
    assert P.choose(score, none, (2, 1), 2).tolist() == [[0, 1]]                 # the first group has the best member
    assert P.choose(score, torch.tensor([-1.0, -1, -2, -2]).double(), (2, 1), 2).tolist() == [[0, 1]]
    assert P.choose(score, torch.tensor([-1.0, -1, -2, -0.5]).double(), (2, 1), 2).tolist() == [[3, 2]]   # though both are negative
