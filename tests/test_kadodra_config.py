"""Host side of the Kadodra design (no GPU): configuration round trip, defaults and errors; the description's tensor
names, cache needs and schedule; tables of experts in random weights and in files; and the plain implementation against
itself (the recurrence in two halves and by its closed form, the window's edges, the sink, every expert chosen, the
looped layers)."""
import copy

import pytest
import torch

import plain_kadodra as P
from tffinfer_b200.config import KadodraConfig, ConfigError
from tffinfer_b200.parts import Model, KVNeed, StateNeed
from tffinfer_b200.registry import get_architecture
import tffinfer_b200.models  # noqa: F401


def sample_json():
    latent = {"heads": 3, "dim": 20, "rot_dim": 6, "vdim": 12, "kv_rank": 18, "scale": 0.2, "mask": {"size": 11},
              "rot": {"base": 1000.0, "dims": 6, "scaling": {"factor": 4.0, "original": 64.0, "fast": 16.0, "slow": 2.0}}}
    lightning = {"heads": 2, "dim": 10, "vdim": 14, "decay": [0.5, 0.97]}
    moe = {"kind": "moe", "expert": {"ff": 24, "limit": 0.7}, "router": {"experts": 5, "top": 3}}
    return {"architecture": "Kadodra", "vocab": 83, "width": 52, "norm": {"eps": 3e-6}, "logit_scale": 0.75,
            "loop": {"start": 1, "stop": 3, "times": 2},
            "layers": [{"type": "latent_attention", "mixer": latent, "mlp": {"kind": "dense", "ff": 70}},
                       {"type": "lightning", "mixer": lightning, "mlp": moe},
                       {"type": "latent_attention", "mixer": dict(latent, heads=1, mask={"size": 1}), "mlp": None},
                       {"type": "lightning", "mixer": lightning, "mlp": None}]}


def test_round_trip_and_defaults():
    cj = sample_json()
    cfg = KadodraConfig.from_json_dict(cj)
    assert cfg.to_json_dict() == cj
    assert cfg.layers[0].latent.window == 11 and cfg.layers[1].mlp.limit == 0.7 and cfg.layers[3].mlp is None
    assert cfg.runs() == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]
    d = copy.deepcopy(cj)
    del d["logit_scale"], d["loop"], d["layers"][0]["mixer"]["mask"], d["layers"][2]["mlp"]
    d["layers"][0]["mixer"]["rot"] = {"base": 1000.0}
    c2 = KadodraConfig.from_json_dict(d)
    a = c2.layers[0].latent
    assert c2.logit_scale == 1.0 and a.window == 0 and a.rot.dims == 6 and a.rot.scaling is None and c2.layers[2].mlp is None
    assert c2.runs() == [(i, False) for i in range(4)]
    d["loop"] = {"start": 0, "stop": 4, "times": 1}
    assert KadodraConfig.from_json_dict(d).runs() == [(i, False) for i in range(4)]
    d["loop"]["times"] = 3
    assert KadodraConfig.from_json_dict(d).runs() == ([(i, False) for i in range(4)]
                                                      + 2 * [(0, True), (1, False), (2, False), (3, False)])


@pytest.mark.parametrize("edit,word", [
    (lambda d: d["layers"][1].__setitem__("type", "retention"), "type"),
    (lambda d: d["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda d: d["layers"][0]["mixer"]["rot"].__setitem__("dims", 8), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].__setitem__("dims", 5), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].__setitem__("factor", 0.0), "scaling"),
    (lambda d: d["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "size"),
    (lambda d: d["layers"][1]["mixer"]["decay"].append(0.1), "decay"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("decay", 0.9), "decay"),
    (lambda d: d["layers"][1]["mlp"]["router"].__setitem__("top", 6), "top"),
    (lambda d: d["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda d: d["layers"][1]["mlp"].__setitem__("kind", "sparse"), "kind"),
    (lambda d: d["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda d: d["loop"].__setitem__("stop", 5), "loop"),
    (lambda d: d["loop"].__setitem__("times", 0), "loop"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_errors_name_the_key(edit, word):
    d = sample_json()
    edit(d)
    with pytest.raises(ConfigError) as e:
        KadodraConfig.from_json_dict(d)
    assert word in str(e.value)


def test_description_names_needs_and_schedule():
    arch = get_architecture("Kadodra")
    desc = arch.describe(arch.read_config(sample_json()))
    model = Model(desc)
    names = model.expected_tensors()
    shapes = {"embed": (83, 52), "final.norm": (52,), "l0.norm1": (52,), "l0.mix.q": (78, 52), "l0.mix.dkv": (24, 52),
              "l0.mix.dkv.norm": (18,), "l0.mix.uk": (60, 18), "l0.mix.uv": (36, 18), "l0.mix.sink": (3,),
              "l0.mix.o": (52, 36), "l0.mlp.up": (70, 52), "l0.mlp.down": (52, 70), "l1.mix.q": (20, 52),
              "l1.mix.k": (20, 52), "l1.mix.v": (28, 52), "l1.mix.g": (28, 52), "l1.mix.norm": (28,), "l1.mix.o": (52, 28),
              "l1.mlp.table": (83, 3), "l1.mlp.e4.gate": (24, 52), "l1.mlp.e4.up": (24, 52), "l1.mlp.e4.down": (52, 24)}
    for n, s in shapes.items():
        assert names[n].shape == s, n
    assert not any(n in names for n in ("head", "l0.norm2", "l0.mix.dq", "l1.mlp.router", "l1.mlp.e5.up", "l2.mlp.up"))
    needs = model.cache_needs()
    st = StateNeed((2, 10, 14), "float32", self_starting=True)
    assert needs == [KVNeed(1, 24, 11, 1), st, KVNeed(1, 24, 1, 1), st, KVNeed(1, 24, 1, 1), st]   # every pass its own
    assert [(e.layer, e.add_embedding) for e in desc.schedule] == KadodraConfig.from_json_dict(sample_json()).runs()
    assert desc.logit_scale == 0.75 and desc.lm_head_name is None
    assert all(l.block == "parallel_shared_norm" and l.ffn_norm is None for l in desc.layers)


def test_tables_of_experts():
    """Random weights give every token id different experts; a file's table is read as integers and checked."""
    from tffinfer_b200.parts.moe import RoutedExperts
    from tffinfer_b200.weights.loader import check_tensors, WeightError
    from tffinfer_b200.weights.random_init import random_state_dict
    arch = get_architecture("Kadodra")
    cfg = KadodraConfig.from_json_dict(sample_json())
    sd = random_state_dict(cfg, 3)
    t = sd["l1.mlp.table"]
    assert t.dtype == torch.int32 and int(t.min()) == 0 and int(t.max()) == 4
    assert all(len(set(r)) == 3 for r in t.tolist()) and len({tuple(r) for r in t.tolist()}) > 10
    expected = Model(arch.describe(cfg)).expected_tensors()
    assert torch.equal(check_tensors(sd, expected, torch.float32, "cpu")["l1.mlp.table"], t)
    with pytest.raises(WeightError):
        check_tensors(dict(sd, **{"l1.mlp.table": t.float()}), expected, torch.float32, "cpu")
    part = RoutedExperts(8, 8, 2, 1, activation="clipped_swish", activation_limit=1.0, router_score="table", table_rows=4)
    with pytest.raises(ValueError):                  # an expert that is not there
        part.load({"table": torch.tensor([[0], [1], [2], [0]], dtype=torch.int32)}, None, torch.float32)
    for bad in (dict(table_rows=0), dict(table_rows=4, weight_on="input"), dict(table_rows=4, activation_limit=0.0)):
        with pytest.raises(ValueError):
            RoutedExperts(8, 8, 2, 1, **{**dict(activation="clipped_swish", activation_limit=1.0, router_score="table"), **bad})


def test_package_frequencies_equal_the_plain_ones():
    from tffinfer_b200.parts.position import scaled_frequencies
    for rot in ({"base": 70000.0, "dims": 24, "scaling": {"factor": 6.0, "original": 512, "fast": 24.0, "slow": 0.5}},
                {"base": 3e4, "dims": 2, "scaling": {"factor": 2.0, "original": 32, "fast": 8.0, "slow": 1.0}},
                {"base": 1e4, "dims": 64, "scaling": {"factor": 4.0, "original": 64.0, "fast": 16.0, "slow": 2.0}},
                {"base": 5e5, "dims": 6}):
        sc = rot.get("scaling")
        f, mag = scaled_frequencies(rot["dims"], rot["base"], (sc["factor"], sc["original"], sc["fast"], sc["slow"]) if sc else None)
        pf, pmag = P.turn_rates(rot)
        assert mag == pytest.approx(pmag, rel=1e-12) and f == pytest.approx(pf, rel=1e-12)


def test_plain_recurrence_in_two_halves_and_by_its_closed_form():
    g = torch.Generator().manual_seed(0)
    T, D, V = 23, 6, 5
    q, k, v = (torch.randn(T, n, generator=g).double() for n in (D, D, V))
    whole, S = P.constant_decay_recurrence(q, k, v, 0.9)
    a, Sa = P.constant_decay_recurrence(q[:9], k[:9], v[:9], 0.9)
    b, Sb = P.constant_decay_recurrence(q[9:], k[9:], v[9:], 0.9, state=Sa)
    assert torch.allclose(torch.cat([a, b]), whole, atol=1e-12) and torch.allclose(S, Sb, atol=1e-12)
    for t in (0, 7, 22):
        o = sum(0.9 ** (t - s) * (q[t] @ k[s]) * v[s] for s in range(t + 1))
        assert torch.allclose(o, whole[t], atol=1e-10)


def test_plain_window_edges_and_sink():
    """Keys by content, no positions: the last of 26 queries copies the planted token inside the window and not the one
    just outside; a large sink takes the weight away without a value of its own."""
    seen = P.window_mask(torch.arange(26), 10)
    assert seen[25].nonzero().flatten().tolist() == list(range(16, 26)) and seen[3].nonzero().flatten().tolist() == [0, 1, 2, 3]
    assert P.window_mask(torch.arange(5), 1).equal(torch.eye(5, dtype=torch.bool))
    assert P.window_mask(torch.arange(5), 0).equal(torch.tril(torch.ones(5, 5)).bool())
    s = torch.zeros(26, 26).double()
    s[:, 16] = 50.0
    s[:, 15] = 90.0
    w = P.softmax_with_sink(s, seen, torch.tensor(0.0).double())
    assert float(w[25, 16]) > 0.999 and float(w[25, 15]) == 0.0 and float(w[24, 15]) > 0.999
    w = P.softmax_with_sink(s, seen, torch.tensor(50.0).double())
    assert float(w[25, 16]) == pytest.approx(0.5, abs=1e-9)
    flat = P.softmax_with_sink(torch.zeros(1, 3).double(), torch.ones(1, 3, dtype=torch.bool), torch.tensor(0.0).double())
    assert flat.sum().item() == pytest.approx(0.75)


def test_plain_experts_gate_and_loop():
    g = torch.Generator().manual_seed(2)
    W, E, ff, T = 8, 3, 5, 4
    w = {"m.table": torch.tensor([[1, 2, 0]] * 6)}
    for e in range(E):
        for n, s in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff))):
            w[f"m.e{e}.{n}"] = torch.randn(*s, generator=g).double()
    h = torch.randn(T, W, generator=g).double()
    got = P.tabled_experts(h, [0, 1, 5, 2], w, "m", {"router": {"experts": E, "top": E}, "expert": {"limit": 0.6}})
    want = 0.0
    for e in range(E):
        gate, up = h @ w[f"m.e{e}.gate"].T, h @ w[f"m.e{e}.up"].T
        gate = torch.where(gate > 0.6, torch.full_like(gate, 0.6), gate)
        up = torch.where(up.abs() > 0.6, 0.6 * torch.sign(up), up)
        want = want + (gate / (1 + torch.exp(-1.702 * gate)) * (up + 1)) @ w[f"m.e{e}.down"].T / 3
    assert torch.allclose(got, want, atol=1e-12)
    assert P.relu_squared(torch.tensor([-2.0, 0.0, 3.0])).tolist() == [0.0, 0.0, 9.0]
    assert P.order_of_runs(sample_json()) == KadodraConfig.from_json_dict(sample_json()).runs()


def test_plain_model_runs_on_a_written_folder(tmp_path):
    """A model folder written by the random-weights mode, read back by name, through the plain implementation: the
    logits of a prefix do not change when tokens follow it, the looped layers are what running them by hand gives, and
    the table's ids matter."""
    from tffinfer_b200.weights import write_random_model
    from tffinfer_b200.weights.safetensors_io import SafetensorsFile
    cfg = KadodraConfig.from_json_dict(sample_json())
    write_random_model(str(tmp_path / "m"), cfg, seed=4)
    f = SafetensorsFile(str(tmp_path / "m" / "model.safetensors"))
    sd = {n: f.tensor(n).clone() for n in f.names()}
    toks = [(5 * i * i + 3) % 83 for i in range(30)]
    runs = []
    full = P.forward(sample_json(), sd, toks, layers_out=runs)
    assert full.shape == (30, 83) and torch.isfinite(full).all() and len(runs) == 6
    assert torch.allclose(P.forward(sample_json(), sd, toks[:17]), full[:17], atol=1e-9)
    once = []
    P.forward(dict(sample_json(), loop=None), sd, toks, layers_out=once)
    assert torch.allclose(once[2], runs[2], atol=1e-12) and not torch.allclose(once[3], runs[5], atol=1e-4)
    other = dict(sd, **{"l1.mlp.table": (sd["l1.mlp.table"] + 1) % 5})
    assert not torch.allclose(P.forward(sample_json(), other, toks), full, atol=1e-6)
