"""Ravelorn without a GPU: the configuration, the parts it is spelled as, the tensors it declares, the cache it asks for,
and the plain implementation's own mechanisms."""
import json

import pytest
import torch

import plain_ravelorn as P
from tiny_models import RAVELORN, prompt, write_ravelorn


def spec_of(cfg):
    from rocml_b200.config import config_from_dict
    return config_from_dict(cfg).to_model_spec()


@pytest.mark.parametrize("name", sorted(RAVELORN))
def test_config_round_trip(name):
    from rocml_b200.config import RavelornConfig, config_from_dict
    cfg = config_from_dict(RAVELORN[name])
    assert isinstance(cfg, RavelornConfig)
    assert config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    assert len(cfg.layers) == len(RAVELORN[name]["layers"])


@pytest.mark.parametrize("broken, needle", [
    (lambda c: c["layers"][0].__setitem__("type", "convolution"), "type"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 8), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("identity", -1), "identity"),
    (lambda c: c["layers"][0]["mixer"]["left"].__setitem__("kv_heads", 3), "left.heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].__setitem__("every", 0), "every"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("heads", 3), "heads"),
    (lambda c: c["layers"][1]["mixer"].pop("decay_rank"), "decay_rank"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c.__setitem__("logit_softcap", 0), "logit_softcap"),
    (lambda c: c["norm"].__setitem__("eps", 0), "eps"),
    (lambda c: c.__setitem__("layers", []), "layers"),
])
def test_config_faults_are_named(broken, needle):
    from rocml_b200.config import config_from_dict
    from rocml_b200.errors import ConfigError
    cfg = json.loads(json.dumps(RAVELORN["RA"]))
    broken(cfg)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg).to_model_spec()
    assert needle in str(e.value)


def test_the_architecture_as_parts():
    spec = spec_of(RAVELORN["RA"])
    assert not spec.tie_embeddings and spec.weight_suffix == "" and spec.bias_suffix == ".b" and spec.logit_softcap == 5.0
    assert spec.input_position.kind == "learned" and spec.input_position.params["rows"] == 640 == spec.max_position
    assert all(L.arrangement == "output_norm" and L.arrangement_params == {"multiplier": 0.6} for L in spec.layers)
    assert spec.final_norm.kind == "layernorm" and spec.layers[0].mixer_norm.kind == "layernorm"
    both = spec.layers[0].mixer
    assert both.kind == "side_by_side" and both.params["left_scale"] == 0.7 and both.params["right_scale"] == 1.3
    left, right = both.params["left"].params, both.params["right"].params
    assert left["sink"] == "per_head" and left["qk_unit_norm"] and dict(left["q_temperature"]) == {"coef": 0.5, "every": 20.0}
    assert right["decay"] == "per_head" and right["gate"] == "silu" and right["n_kv_heads"] == 2
    chan = spec.layers[1].mixer.params
    assert chan["decay"] == "per_channel" and chan["gate"] == "sigmoid_low_rank" and (chan["decay_rank"], chan["gate_rank"]) == (10, 6)
    ff = spec.layers[0].feed_forward.params
    assert ff["score"] == "softmax" and ff["identity"] == 2 and ff["experts"] == 5 and not ff["renormalize"]
    assert spec.layers[1].feed_forward is None


def test_declared_tensors_and_a_folder(tmp_path):
    """The folder's config.json does not tell the narrow products' inner sizes: they come from the tensors."""
    from rocml_b200.config import load_model_spec
    from rocml_b200.engine.model import declared_tensors
    from safetensors import safe_open
    folder = write_ravelorn(str(tmp_path / "m"), RAVELORN["RC"], 1)
    spec = load_model_spec(folder)
    assert spec == spec_of(RAVELORN["RC"])
    decl = {d.name: tuple(d.shape) for d in declared_tensors(spec)}
    with safe_open(f"{folder}/model.safetensors", "pt") as f:
        have = {k: tuple(f.get_slice(k).get_shape()) for k in f.keys()}
    assert have == decl
    assert decl["pos"] == (560, 72) and decl["l0.norm1.b"] == (72,) and decl["final.norm.b"] == (72,)
    assert decl["l0.mix.left.sink"] == (3,) and decl["l0.mix.left.o"] == (72, 84) and decl["l0.mix.right.a"] == (1, 72)
    assert decl["l1.mix.a1"] == (9, 72) and decl["l1.mix.a2"] == (108, 9) and decl["l1.mix.g1"] == (5, 72) and decl["l1.mix.g2"] == (12, 5)
    assert decl["l1.mix.dt_bias"] == (108,) and decl["l0.mix.right.dt_bias"] == (1,) and decl["l2.mix.v.conv"] == (150, 9)
    assert decl["l0.mlp.router"] == (5, 72) and decl["l0.mlp.correction"] == (5,) and "l0.mlp.e2.gate" not in decl
    assert "l2.norm2" not in decl


def test_what_the_cache_keeps():
    from rocml_b200.cache import SequenceCache
    from rocml_b200.cache.requirements import BundleRequirement, KVRequirement, StateRequirement
    from rocml_b200.engine.model import Model
    from rocml_b200.parts import BuildEnv
    model = Model(spec_of(RAVELORN["RC"]), BuildEnv(torch.device("cpu"), torch.bfloat16))
    reqs = model.cache_requirements()
    assert reqs[0] == BundleRequirement(KVRequirement(3, 32, None), (("right_state", StateRequirement((1, 7, 5), torch.float32)),))
    assert reqs[1] == BundleRequirement(StateRequirement((3, 4, 36), torch.float32), (("conv", StateRequirement((5, 216 + 12), torch.float32)),))
    cache = SequenceCache(reqs, model.reads_cache_of(), 256, 4, 560, torch.bfloat16, "cpu")
    assert [v.kind for v in cache.views] == ["kv", "state", "state"]
    s = cache.alloc_slot()
    cache.views[0].extras["right_state"].state[s].fill_(3.0)
    cache.views[1].extras["conv"].state[s].fill_(3.0)
    cache.free_slot(s)
    assert cache.alloc_slot() == s
    assert float(cache.views[0].extras["right_state"].state[s].abs().sum()) == 0 and float(cache.views[1].extras["conv"].state[s].abs().sum()) == 0


def test_random_weights_without_a_folder_need_the_inner_sizes():
    from rocml_b200.config import config_from_dict
    cfg = config_from_dict(RAVELORN["RA"])
    shapes = {"l1.mix.a1": (10, 64), "l1.mix.g1": (6, 64), "l2.mix.a1": (24, 64), "l2.mix.g1": (16, 64)}
    bare = json.loads(json.dumps(RAVELORN["RA"]))
    for L in bare["layers"]:
        L["mixer"].pop("decay_rank", None), L["mixer"].pop("gate_rank", None)
    assert config_from_dict(bare).with_tensor_shapes(shapes.get) == cfg


def test_plain_recurrence_in_pieces_is_the_whole():
    torch.manual_seed(0)
    T, H, d, v = 23, 3, 5, 4
    q, k, val = torch.randn(T, H, d).double(), P.unit(torch.randn(T, H, d).double()), torch.randn(T, H, v).double()
    beta, g = torch.rand(T, H).double(), torch.rand(T, H, d).double()
    whole, S = P.delta_rule(q, k, val, beta, g)
    a, s1 = P.delta_rule(q[:9], k[:9], val[:9], beta[:9], g[:9])
    b, s2 = P.delta_rule(q[9:], k[9:], val[9:], beta[9:], g[9:], state=s1)
    assert float((torch.cat([a, b]) - whole).abs().max()) < 1e-13 and float((s2 - S).abs().max()) < 1e-13
    same, _ = P.delta_rule(q, k, val, beta, g[:, :, :1].expand(T, H, d))
    per_head, _ = P.delta_rule(q, k, val, beta, g[:, :, 0])
    assert torch.equal(same, per_head)


def test_plain_four_tokens_at_once_are_one_after_another():
    """The identity that the prompt kernel rests on: with G the products of decays inside a chunk, the four corrections follow
    from sums over the state before the chunk and a triangle of the tokens' own products."""
    torch.manual_seed(1)
    d, v = 6, 3
    S0 = torch.randn(d, v).double()
    q, k, val = torch.randn(4, d).double(), torch.randn(4, d).double(), torch.randn(4, v).double()
    beta, g = torch.rand(4).double(), torch.rand(4, d).double()
    o, S = P.delta_rule(q[:, None], k[:, None], val[:, None], beta[:, None], g[:, None], state=S0[None])
    w, out = [], []
    for t in range(4):
        G = g[: t + 1].prod(0)
        part = [g[s + 1: t + 1].prod(0) * k[s] for s in range(t + 1)]
        a = (G * k[t]) @ S0 + sum(((k[t] @ part[s]) * w[s] for s in range(t)), torch.zeros(v).double())
        w.append(beta[t] * (val[t] - a))
        out.append((G * q[t]) @ S0 + sum((q[t] @ part[s]) * w[s] for s in range(t + 1)))
    end = g.prod(0)[:, None] * S0 + sum((g[s + 1:].prod(0) * k[s])[:, None] * w[s][None] for s in range(4))
    assert float((torch.stack(out) - o[:, 0]).abs().max()) < 1e-12 and float((end - S[0]).abs().max()) < 1e-12


def test_plain_query_temperature_steps():
    f = P.query_temperature(list(range(50)), {"coef": 0.5, "every": 20})
    assert float(f[0]) == 1.0 and float(f[18]) == 1.0 and float(f[19]) > 1.3 and float(f[38]) == float(f[19]) and float(f[39]) > float(f[38])


def test_plain_sink_and_identity():
    s = torch.zeros(2, 3, 3).double()
    a = P.sink_softmax(s, [0, 1, 2], torch.tensor([0.0, -50.0]).double())
    assert abs(float(a[0, 2, 0]) - 0.25) < 1e-12 and abs(float(a[1, 2, 0]) - 1 / 3) < 1e-12 and float(a[0, 0, 1]) == 0.0
    h = torch.randn(4, 5).double()
    w = {"router": torch.zeros(2, 5).double(), "correction": torch.tensor([0.0, 1.0]).double()}
    out = P.experts_ff(h, {"router": {"experts": 1, "identity": 1, "top": 1}}, w)
    assert float((out - 0.5 * h).abs().max()) < 1e-12
