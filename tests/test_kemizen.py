"""Kemizen without a GPU: the configuration, the parts it is spelled as, the tensors it declares, the cache it asks for,
and the plain implementation's own mechanisms."""
import json
import math

import pytest
import torch

import plain_kemizen as P
from tiny_models import KEMIZEN, prompt, write_kemizen


def spec_of(cfg):
    from rocml_b200.config import config_from_dict
    return config_from_dict(cfg).to_model_spec()


def model_of(cfg):
    from rocml_b200.engine.model import Model
    from rocml_b200.parts import BuildEnv
    return Model(spec_of(cfg), BuildEnv(torch.device("cpu"), torch.bfloat16))


@pytest.mark.parametrize("name", sorted(KEMIZEN))
def test_config_round_trip(name):
    from rocml_b200.config import KemizenConfig, config_from_dict
    cfg = config_from_dict(KEMIZEN[name])
    assert isinstance(cfg, KemizenConfig)
    assert config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    assert len(cfg.layers) == len(KEMIZEN[name]["layers"])


@pytest.mark.parametrize("name", ["kemizen-2k", "kemizen-4k"])
def test_catalog_entries(name):
    from rocml_b200.config import CATALOG, config_from_dict
    cfg = config_from_dict(CATALOG[name].config)
    assert cfg.to_dict() == CATALOG[name].config
    assert {L.mixer_type for L in cfg.layers} == {"mlstm", "attention", "parallel"} and any(L.kv_from is not None for L in cfg.layers)


@pytest.mark.parametrize("broken, needle", [
    (lambda c: c["layers"][0].__setitem__("type", "convolution"), "type"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "heads"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("softcap", 0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 14), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("gate_cap", 0), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][2]["mixer"]["right"].__setitem__("blocks", 5), "blocks"),
    (lambda c: c["layers"][2]["mixer"]["left"].pop("conv"), "conv"),
    (lambda c: c["layers"][2]["mixer"]["left"].__setitem__("kv_heads", 4), "left.heads"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 1), "kv_from"),
    (lambda c: c["layers"][5]["mixer"].__setitem__("kv_from", 3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("dim", 16), "layer 0"),
    (lambda c: c["layers"][3]["mixer"]["rot"].__setitem__("base", 5.0), "layer 0"),
    (lambda c: c["norm"].__setitem__("eps", 0), "eps"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c.__setitem__("layers", []), "layers"),
    (lambda c: c.pop("vocab"), "vocab"),
])
def test_config_faults_are_named(broken, needle):
    from rocml_b200.config import config_from_dict
    from rocml_b200.errors import ConfigError
    cfg = json.loads(json.dumps(KEMIZEN["KA"]))
    broken(cfg)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg).to_model_spec()
    assert needle in str(e.value)


def test_the_architecture_as_parts():
    spec = spec_of(KEMIZEN["KA"])
    assert not spec.tie_embeddings and spec.weight_suffix == "" and spec.bias_suffix == ".b" and spec.embedding_scale == 1.5
    assert all(L.arrangement == "output_norm" and L.mixer_norm.kind == "rmsnorm" and L.mixer_norm.weight_offset == 1.0 for L in spec.layers)
    assert spec.final_norm.weight_offset == 1.0
    diff = spec.layers[0].mixer
    assert diff.kind == "attention" and diff.params["difference"] == 0.3 and diff.params["window"] == 50 and diff.params["softcap"] == 3.0
    assert diff.position.rot_dim == 8 and dict(diff.position.params["ramp_scaling"])["factor"] == 4.0
    assert [e.reads_cache_of for e in spec.schedule] == [None, None, None, 0, None, 0]
    mem = spec.layers[1].mixer
    assert mem.kind == "mlstm" and mem.params["gate_cap"] == 4.0 and spec.layers[1].feed_forward is None
    both = spec.layers[2].mixer
    assert both.kind == "side_by_side" and both.params["out_norms"] and both.params["out_factor"] == 0.5
    left, right = both.params["left"].params, both.params["right"]
    assert left["qk_norm"] == "whole" and left["gated"] == "per_value" and left["conv_taps"] == 3 and set(left["bias"]) == {"q", "k", "v", "o"}
    assert right.kind == "rg_lru" and right.params["blocks"] == 3 and right.params["conv_taps"] == 4
    ff = spec.layers[0].feed_forward
    assert ff.kind == "dense_mlp" and ff.params["activation"] == "gelu" and ff.params["intermediate"] == 96
    assert "softcap" not in spec_of(KEMIZEN["KC"]).layers[1].mixer.params and "window" not in spec_of(KEMIZEN["KC"]).layers[2].mixer.params


def test_declared_tensors_and_a_folder(tmp_path):
    from rocml_b200.config import load_model_spec
    from rocml_b200.engine.model import declared_tensors
    from safetensors import safe_open
    folder = write_kemizen(str(tmp_path / "m"), KEMIZEN["KA"], 1)
    spec = load_model_spec(folder)
    assert spec == spec_of(KEMIZEN["KA"])
    decl = {d.name: tuple(d.shape) for d in declared_tensors(spec)}
    with safe_open(f"{folder}/model.safetensors", "pt") as f:
        have = {k: tuple(f.get_slice(k).get_shape()) for k in f.keys()}
    assert have == decl
    assert decl["l0.mix.q"] == (4 * 2 * 12, 64) and decl["l0.mix.k"] == (2 * 2 * 12, 64) and decl["l0.mix.v"] == (40, 64)
    assert decl["l0.mix.q.norm"] == (12,) and decl["l0.mix.lk2"] == (12,) and decl["l0.mix.o"] == (64, 80)
    assert not any(n.startswith(("l3.mix.k", "l3.mix.v")) for n in decl) and decl["l3.mix.q"] == (96, 64) and decl["l3.mix.q.norm"] == (12,)
    assert decl["l1.mix.i"] == (3, 64) and decl["l1.mix.f.b"] == (3,) and decl["l1.mix.norm"] == (60,) and "l1.mix.q.b" not in decl
    assert decl["l2.mix.left.q.norm"] == (120,) and decl["l2.mix.left.k.conv"] == (40, 3) and decl["l2.mix.left.o.b"] == (64,)
    assert decl["l2.mix.left.g"] == (72, 64) and "l2.mix.left.g.b" not in decl and decl["l2.mix.left.v"] == (24, 64)
    assert decl["l2.mix.right.ra"] == (3, 16, 16) and decl["l2.mix.right.ri.b"] == (3, 16) and decl["l2.mix.right.conv.b"] == (48,)
    assert decl["l2.mix.right.lam"] == (48,) and decl["l2.mix.left.out"] == (64,) and decl["l2.mix.right.out"] == (64,)
    assert "l1.norm2" not in decl and "l0.mlp.gate" not in decl and decl["l0.mlp.up"] == (96, 64)


def test_what_the_cache_keeps():
    from rocml_b200.cache import SequenceCache
    from rocml_b200.cache.requirements import BundleRequirement, KVRequirement, StateRequirement
    model = model_of(KEMIZEN["KA"])
    reqs = model.cache_requirements()
    # two maps of 12 beside values of 20: heads of 24, padded to 32; the reader with the widest window decides what stays
    assert reqs[0] == KVRequirement(2, 32, 90) and reqs[3] == KVRequirement(2, 32, 90) and reqs[5] == KVRequirement(2, 32, 7)
    assert reqs[1] == BundleRequirement(StateRequirement((3, 12, 20), torch.float32),
                                        (("norm", StateRequirement((3, 12), torch.float32)), ("peak", StateRequirement((3, 2), torch.float32))))
    assert reqs[2] == BundleRequirement(KVRequirement(2, 32), (("conv", StateRequirement((2, 6 * 20 + 2 * 20 + 2 * 12), torch.float32)),
                                                               ("right_conv", StateRequirement((3, 48), torch.float32)),
                                                               ("right_state", StateRequirement((48,), torch.float32))))
    cache = SequenceCache(reqs, model.reads_cache_of(), 256, 4, 560, torch.bfloat16, "cpu")
    assert [v.kind for v in cache.views] == ["kv", "state", "kv", "kv", "state", "kv"]
    assert cache.views[3].group is cache.views[0].group and not cache.views[3].writes and cache.views[5].k.data_ptr() == cache.views[0].k.data_ptr()
    assert len(cache.kv_groups) == 2 and cache.kv_groups[0].n_entries == 1
    s = cache.alloc_slot()
    for i, name in ((1, "peak"), (1, "norm"), (2, "conv"), (2, "right_state")):
        cache.views[i].extras[name].state[s].fill_(3.0)
    cache.free_slot(s)
    assert cache.alloc_slot() == s
    for i, name in ((1, "peak"), (1, "norm"), (2, "conv"), (2, "right_state")):
        assert float(cache.views[i].extras[name].state[s].abs().sum()) == 0
    # one tap: nothing kept; no window beside a window: everything stays
    reqs = model_of(KEMIZEN["KC"]).cache_requirements()
    assert [n for n, _ in reqs[0].extras] == ["right_conv", "right_state"] and [n for n, _ in reqs[4].extras] == ["conv", "right_state"]
    assert reqs[2] == KVRequirement(3, 32) and reqs[5] == KVRequirement(3, 32, 300)


def test_a_cache_that_serves_two_masks():
    from rocml_b200.cache.requirements import KVRequirement
    a = KVRequirement(2, 64, 100)
    assert a.covering(KVRequirement(2, 64, 70)) == a and a.covering(KVRequirement(2, 64, 300)) == KVRequirement(2, 64, 300)
    assert a.covering(KVRequirement(2, 64)) == KVRequirement(2, 64) == KVRequirement(2, 64).covering(a)
    assert a.covering(KVRequirement(2, 64, None, chunk=32)) == KVRequirement(2, 64)
    assert a.covering(KVRequirement(2, 64, 50, keep_first=9)) == KVRequirement(2, 64, 100, keep_first=9)
    with pytest.raises(ValueError):
        a.covering(KVRequirement(1, 64, 70))


def test_a_cost_and_a_work_space_for_every_part():
    for cfg in KEMIZEN.values():
        model = model_of(cfg)
        small, large = model.step_cost([1], [100], 1), model.step_cost([200], [200], 1)
        assert 0 < small[0] < large[0] and 0 < small[1] < large[1]
        assert 0 < model.workspace_bytes(1, 1) < model.workspace_bytes(300, 1)


def test_parts_refuse_what_they_do_not_build():
    from rocml_b200.config.specs import FeedForwardSpec, MixerSpec
    from rocml_b200.errors import ConfigError
    from rocml_b200.parts import BuildEnv, build_feed_forward, build_mixer
    env = BuildEnv(torch.device("cpu"), torch.bfloat16)
    att = dict(n_heads=4, n_kv_heads=2, head_dim=64)
    for params in (dict(att, difference=0.5, gated=True), dict(att, qk_norm="whole", softcap=3.0), dict(att, qk_norm="whole", gated=True),
                   dict(att, conv_taps=99), dict(att, softcap=-1.0), dict(att, conv_taps=3, difference=0.2), dict(att, head_dim=300, difference=0.1)):
        with pytest.raises(ConfigError):
            build_mixer(MixerSpec.make("attention", None, **params), 64, env)
    with pytest.raises(ConfigError):
        build_mixer(MixerSpec.make("mlstm", None, n_heads=2, head_dim=8, gate_cap=0.0), 64, env)
    with pytest.raises(ConfigError):
        build_mixer(MixerSpec.make("rg_lru", None, width=30, blocks=4), 64, env)
    with pytest.raises(ConfigError):
        build_feed_forward(FeedForwardSpec.make("dense_mlp", intermediate=8, activation="relu"), 64, env)
    left = MixerSpec.make("attention", None, **dict(att, bias=("o",)))
    right = MixerSpec.make("rg_lru", None, width=32, blocks=2)
    with pytest.raises(ConfigError):         # a bias on an output product that the two sides would share
        build_mixer(MixerSpec.make("side_by_side", None, left=left, right=right), 64, env)
    with pytest.raises(ConfigError):         # a scale that the norm behind it would undo
        build_mixer(MixerSpec.make("side_by_side", None, left=left, right=right, out_norms=True, left_scale=2.0), 64, env)
    assert build_mixer(MixerSpec.make("side_by_side", None, left=left, right=right, out_norms=True), 64, env).norms_later


# ---- the plain implementation's own mechanisms ------------------------------------------------------------------------------

def test_plain_memory_is_the_sum_without_a_maximum():
    """The running maximum changes nothing but the bound of the divisor: with plain exponentials and the bound 1 on the plain sum, the
    result is the same; and pieces are the whole."""
    torch.manual_seed(0)
    T, H, d, v = 23, 2, 5, 4
    q, k, val = torch.randn(T, H, d).double(), torch.randn(T, H, d).double(), torch.randn(T, H, v).double()
    i, f = 2.0 * torch.randn(T, H).double(), P.log_sigmoid(torch.randn(T, H).double())
    o, (S, n, m) = P.mlstm_scan(q, k, val, i, f)
    C, N = torch.zeros(H, d, v).double(), torch.zeros(H, d).double()
    for t in range(T):
        C = torch.exp(f[t])[:, None, None] * C + torch.exp(i[t])[:, None, None] * k[t][:, :, None] * val[t][:, None, :]
        N = torch.exp(f[t])[:, None] * N + torch.exp(i[t])[:, None] * k[t]
        plain = torch.einsum("hkv,hk->hv", C, q[t]) / torch.clamp((N * q[t]).sum(-1).abs(), min=1.0)[:, None]
        assert float((plain - o[t]).abs().max()) < 1e-4 * float(plain.abs().max())        # (the 1e-6 beside the divisor)
    assert float((C * torch.exp(-m)[:, None, None] - S).abs().max()) < 1e-12
    a, st = P.mlstm_scan(q[:9], k[:9], val[:9], i[:9], f[:9])
    b, end = P.mlstm_scan(q[9:], k[9:], val[9:], i[9:], f[9:], state=st)
    assert float((torch.cat([a, b]) - o).abs().max()) < 1e-13 and all(float((x - y).abs().max()) < 1e-13 for x, y in zip(end, (S, n, m)))


def test_plain_memory_by_blocks():
    """The identity that the prompt kernels rest on: with c the running sum of log keep inside a block, results and end state follow
    from the state before the block and the block's own decayed scores, all exponents at most 0."""
    torch.manual_seed(1)
    d, v, n = 6, 3, 7
    q, k, val = torch.randn(n, 1, d).double(), torch.randn(n, 1, d).double(), torch.randn(n, 1, v).double()
    i, f = torch.randn(n, 1).double(), P.log_sigmoid(torch.randn(n, 1).double())
    S0, n0, m0 = torch.randn(1, d, v).double(), torch.randn(1, d).double(), torch.tensor([0.7]).double()
    o, (S, nn, m) = P.mlstm_scan(q, k, val, i, f, state=(S0, n0, m0))
    mt, keep, add = m0[0], [], []
    for t in range(n):
        m2 = torch.maximum(f[t, 0] + mt, i[t, 0])
        keep.append(f[t, 0] + mt - m2)
        add.append(i[t, 0] - m2)
        mt = m2
    c = torch.cumsum(torch.stack(keep), 0)
    assert bool((c <= 0).all()) and all(float(x) <= 0 for x in add)
    w = torch.stack([torch.exp(c[-1] - c[s] + add[s]) for s in range(n)])
    assert float((torch.exp(c[-1]) * S0[0] + torch.einsum("s,sd,sv->dv", w, k[:, 0], val[:, 0]) - S[0]).abs().max()) < 1e-12
    t = 4
    sc = torch.stack([torch.exp(c[t] - c[s] + add[s]) * (q[t, 0] @ k[s, 0]) for s in range(t + 1)])
    num = torch.exp(c[t]) * (q[t, 0] @ S0[0]) + sc @ val[:t + 1, 0]
    den = torch.exp(c[t]) * (q[t, 0] @ n0[0]) + sc.sum()
    m_t = m0[0]
    for r in range(t + 1):
        m_t = torch.maximum(f[r, 0] + m_t, i[r, 0])
    assert float((num / (torch.maximum(den.abs(), torch.exp(-m_t)) + 1e-6) - o[t, 0]).abs().max()) < 1e-12


def test_plain_recurrent_unit():
    torch.manual_seed(2)
    w = {"ra": torch.randn(2, 3, 3).double(), "ri": torch.randn(2, 3, 3).double(), "ra.b": torch.randn(2, 3).double(), "ri.b": torch.randn(2, 3).double(),
         "lam": torch.randn(6).double()}
    u = torch.randn(11, 6).double()
    a, x = P.rglru_gates(u, w)
    r = torch.sigmoid(w["ra"][1] @ u[4, 3:] + w["ra.b"][1])
    la = -8.0 * r * torch.log1p(torch.exp(w["lam"][3:]))
    assert float((a[4, 3:] - torch.exp(la)).abs().max()) < 1e-13
    i = torch.sigmoid(w["ri"][1] @ u[4, 3:] + w["ri.b"][1])
    assert float((x[4, 3:] - torch.sqrt(1 - torch.exp(la) ** 2) * i * u[4, 3:]).abs().max()) < 1e-9
    whole, last = P.rglru_scan(a, x)
    one, s = P.rglru_scan(a[:5], x[:5])
    two, end = P.rglru_scan(a[5:], x[5:], state=s)
    assert float((torch.cat([one, two]) - whole).abs().max()) < 1e-14 and float((end - last).abs().max()) < 1e-14
    assert torch.equal(whole[0], x[0])                                    # no special case for the first token


def test_plain_difference_as_grouped_attention():
    """What the library does with two maps a head: keys side by side, a query row a map with zeros in the other's place, values shared."""
    torch.manual_seed(3)
    T, H, G, d, v = 9, 4, 2, 6, 5
    q, k, val = torch.randn(T, H, 2, d).double(), torch.randn(T, G, 2, d).double(), torch.randn(T, G, v).double()
    of = torch.arange(H) // (H // G)
    pos = list(range(T))
    apart = [torch.einsum("hij,jhd->ihd", P.weights(torch.einsum("ihd,jhd->hij", q[:, :, p], k[:, of, p]), pos, 5), val[:, of]) for p in range(2)]
    rows = torch.zeros(T, 2 * H, 2 * d).double()
    for p in range(2):
        rows[:, p::2, p * d:(p + 1) * d] = q[:, :, p]
    of2 = torch.arange(2 * H) // (2 * H // G)
    wide = torch.einsum("hij,jhd->ihd", P.weights(torch.einsum("ihd,jhd->hij", rows, k.reshape(T, G, 2 * d)[:, of2]), pos, 5), val[:, of2])
    assert float((wide[:, 0::2] - apart[0]).abs().max()) < 1e-13 and float((wide[:, 1::2] - apart[1]).abs().max()) < 1e-13
    w = {n: torch.randn(d).double() for n in ("lq1", "lk1", "lq2", "lk2")}
    lam = P.diff_lambda(w, 0.3)
    assert abs(float(lam) - (math.exp(float(w["lq1"] @ w["lk1"])) - math.exp(float(w["lq2"] @ w["lk2"])) + 0.3)) < 1e-12


def test_plain_frequencies_and_cap():
    rot = {"base": 10000.0, "dims": 16}
    f, mag = P.frequencies(rot)
    assert mag == 1.0 and abs(float(f[3]) - 10000.0 ** (-6 / 16)) < 1e-15
    g, mag = P.frequencies({**rot, "scaling": {"factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0}})
    assert abs(mag - (0.1 * math.log(4.0) + 1.0)) < 1e-15 and float(g[0]) == float(f[0]) and abs(float(g[-1]) - float(f[-1]) / 4.0) < 1e-15
    assert bool((g <= f).all()) and bool((g >= f / 4.0).all())
    z = torch.linspace(-40, 40, 81).double()
    assert float(P.capped(z, 5.0).abs().max()) <= 5.0 and torch.equal(P.capped(z, None), z)


def test_plain_layers_share_keys():
    """A layer that uses another's keys depends on them, not on keys of its own."""
    import tempfile
    folder = write_kemizen(tempfile.mkdtemp(), KEMIZEN["KA"], 4)
    cfg, w = P.load_folder(folder)
    ids = prompt(4, 30, 211)
    want = P.forward(cfg, w, ids)
    other = dict(w)
    other["l0.mix.k.norm"] = w["l0.mix.k.norm"] * 1.5
    assert float((P.forward(cfg, other, ids) - want).abs().max()) > 1e-3
    lo, hi = [], []
    P.forward(cfg, w, ids, lo)
    P.forward(cfg, {**w, "l3.mix.q.norm": w["l3.mix.q.norm"] * 1.5}, ids, hi)
    assert all(torch.equal(a, b) for a, b in zip(lo[:3], hi[:3])) and not torch.equal(lo[3], hi[3])
