"""The Zifelorn configuration on the host, without a GPU: reading config.json, what it refuses, the model spec it becomes
(norms behind the sublayers only, shared latents as a schedule), and the check of a checkpoint against it."""
import copy
import math

import pytest

from zifelorn_cases import CASES, CASE_A, CASE_B, CASE_C, CASE_D, random_weights, tensor_shapes, write_model


def test_registered_and_chosen_by_name():
    from fastgguf_b200.config import ZifelornConfig
    from fastgguf_b200.registry import config_from_dict, registered_architectures
    assert "Zifelorn" in registered_architectures()
    cfg = config_from_dict(CASE_A)
    assert isinstance(cfg, ZifelornConfig) and cfg.architecture == "Zifelorn"
    assert cfg.to_dict() == CASE_A
    d = cfg.describe()
    assert d["hidden_size"] == 96 and d["vocab_size"] == 211 and d["num_hidden_layers"] == 4 and d["layer_runs"] == 4
    assert d["layer_kinds"] == ["latent_attention+dense", "rglru+experts", "latent_attention+none", "rglru+experts"]
    # the first layer's latent and rotated part; the third reads them
    assert d["kv_bytes_per_token"] == {"bfloat16": 2 * (40 + 8), "float32": 4 * (40 + 8)}
    # four taps: a ring of four inputs and the state; one tap: the state alone
    assert d["state_bytes_per_sequence"] == 4 * (5 * 72 + 60)
    for case in CASES.values():
        assert config_from_dict(case).describe()["parameters"] == sum(math.prod(s) for s in tensor_shapes(case).values())


def test_shared_latents_become_a_schedule():
    from fastgguf_b200.registry import config_from_dict
    spec = config_from_dict(CASE_A).spec_json()
    assert [(r["layer"], r["cache_from"]) for r in spec["schedule"]] == [(0, None), (1, None), (2, 0), (3, None)]
    assert spec["layers"][2]["mixer"]["params"]["shared_kv"] is True and "kv_down.weight" not in spec["layers"][2]["mixer"]["tensors"]
    assert spec["layers"][0]["mixer"]["params"]["shared_kv"] is False and spec["layers"][0]["mixer"]["tensors"]["kv_down.weight"] == "l0.mix.dkv"
    assert [r["cache_from"] for r in config_from_dict(CASE_B).spec_json()["schedule"]] == [None, None, None, 1, None, None]


def test_spec_follows_the_file():
    from fastgguf_b200.registry import config_from_dict
    spec = config_from_dict(CASE_A).spec_json()
    kinds = [(l["block"], l["mixer"]["kind"], (l["feed_forward"] or {}).get("kind")) for l in spec["layers"]]
    assert kinds == [("postnorm", "latent_attention", "swiglu"), ("postnorm", "rglru", "moe"), ("postnorm", "latent_attention", None),
                     ("postnorm", "rglru", "moe")]
    for i, l in enumerate(spec["layers"]):
        assert l["mixer_norm"] is None and l["mixer_post_norm"]["tensors"]["weight"] == f"l{i}.norm1" and l["mixer_post_norm"]["params"] == {"size": 96, "eps": 2e-6}
    assert spec["layers"][1]["feed_forward_post_norm"]["tensors"]["weight"] == "l1.norm2" and spec["layers"][2].get("feed_forward_post_norm") is None
    m = spec["layers"][0]["mixer"]["params"]
    assert (m["n_heads"], m["head_dim"], m["rot_dim"], m["v_head_dim"], m["kv_rank"], m["q_rank"], m["scale"]) == (3, 16, 8, 24, 40, 48, 0.2)
    assert m["gate"] is True and m["sink"] is False
    assert m["position"]["params"] == {"head_dim": 8, "theta": 10000.0, "rotary_dim": 8, "layout": "adjacent", "scaling": None}
    r = spec["layers"][1]["mixer"]
    assert r["params"] == {"hidden_size": 96, "width": 72, "n_blocks": 3, "conv_taps": 4, "gain": 8.0}
    assert r["tensors"]["r_gate.weight"] == "l1.mix.ra" and r["tensors"]["i_gate.bias"] == "l1.mix.ri.b" and r["tensors"]["y_proj.bias"] == "l1.mix.y.b"
    f = spec["layers"][1]["feed_forward"]
    assert f["params"] == {"hidden_size": 96, "d_ff": 40, "n_experts": 6, "top_k": 2, "router": "softmax_chosen", "activation": "relu2"}
    assert f["tensors"]["router.bias"] == "l1.mlp.router.b" and f["tensors"]["experts.5.down_proj.weight"] == "l1.mlp.e5.down"
    assert spec["layers"][0]["feed_forward"]["params"] == {"hidden_size": 96, "d_ff": 80, "activation": "gelu_tanh"}
    assert spec["embedding"]["params"]["scale"] == 3.5 and spec["embedding"]["tensors"]["weight"] == "embed" == spec["head"]["tensors"]["weight"]
    assert spec["final_norm"]["params"] == {"size": 96, "eps": 2e-6, "gain": 1.75}
    assert "gain" not in config_from_dict(CASE_D).spec_json()["final_norm"]["params"]


def test_python_spec_round_trip():
    from fastgguf_b200.engine.spec import ModelSpec
    from fastgguf_b200.registry import config_from_dict
    j = config_from_dict(CASE_A).spec_json()
    again = ModelSpec.from_json(j).to_json()
    assert again["schedule"] == j["schedule"]
    for a, b in zip(again["layers"], j["layers"]):
        assert a["mixer_norm"] is None and a["mixer_post_norm"] == b["mixer_post_norm"] and a["mixer"]["kind"] == b["mixer"]["kind"]
    assert again["layers"][2]["feed_forward"] is None and again["layers"][1]["feed_forward"] == j["layers"][1]["feed_forward"]


def broken(path, value):
    d = copy.deepcopy(CASE_A)
    node = d
    for k in path[:-1]:
        node = node[k]
    if value is KeyError:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return d


@pytest.mark.parametrize("path,value,needle", [
    (["vocab"], KeyError, "vocab"), (["width"], 0, "positive"), (["norm", "eps"], 0.0, "eps"), (["norm"], KeyError, "norm"),
    (["layers", 0, "type"], "conv", "not known"), (["layers", 1, "mixer"], KeyError, "mixer"),
    (["layers", 1, "mixer", "blocks"], 5, "multiple"), (["layers", 1, "mixer", "conv"], 0, "conv"), (["layers", 1, "mixer", "width"], KeyError, "width"),
    (["layers", 0, "mixer", "rot_dim"], 7, "rot_dim"), (["layers", 0, "mixer", "rot", "dims"], 4, "rot_dim"), (["layers", 0, "mixer", "rot"], KeyError, "rot"),
    (["layers", 0, "mixer", "kv_rank"], KeyError, "kv_rank"), (["layers", 0, "mixer", "q_rank"], 0, "q_rank"),
    (["layers", 2, "mixer", "kv_from"], 2, "earlier"), (["layers", 2, "mixer", "kv_from"], 1, "no latent"),
    (["layers", 2, "mixer", "kv_rank"], 24, "must equal"), (["layers", 2, "mixer", "rot", "base"], 500.0, "must equal"),
    (["layers", 0, "mlp", "kind"], "glu", "not known"), (["layers", 0, "mlp", "ff"], 0, "ff"), (["layers", 1, "mlp", "router", "top"], 7, "top"),
    (["layers", 1, "mlp", "router"], KeyError, "router"), (["layers", 1, "mlp", "expert", "ff"], 0, "ff"), (["layers"], [], "layers"),
])
def test_what_the_reader_refuses(path, value, needle):
    from fastgguf_b200.config import ConfigError
    from fastgguf_b200.registry import config_from_dict
    with pytest.raises(ConfigError) as e:
        config_from_dict(broken(path, value))
    assert needle in str(e.value)


def test_weights_are_checked_against_the_configuration(tmp_path):
    from fastgguf_b200.registry import config_from_dict
    from fastgguf_b200.weights import WeightError, check_weights, expected_tensors
    for name, cfg in CASES.items():
        declared, want = expected_tensors(config_from_dict(cfg)), tensor_shapes(cfg)
        assert sorted(declared) == sorted(want), name
        for k, v in declared.items():
            assert tuple(v["shape"]) == tuple(want[k]), (name, k)
    W = random_weights(CASE_A, 1)
    good = write_model(tmp_path / "good", CASE_A, W)
    assert len(check_weights(config_from_dict(CASE_A), model_dir=good)) == len(W)
    bad = dict(W)
    del bad["l1.mix.lam"]
    bad["l2.mlp.up"] = W["l0.mlp.up"]                 # a layer without a feed-forward has no tensors for one
    bad["l2.mix.dkv"] = W["l0.mix.dkv"]               # a layer that reads another's latents has no map of its own
    bad["l1.mix.ra"] = W["l1.mix.ra"].reshape(72, 24)     # the gates' squares, flattened
    with pytest.raises(WeightError) as e:
        check_weights(config_from_dict(CASE_A), model_dir=write_model(tmp_path / "bad", CASE_A, bad))
    assert e.value.missing == ["l1.mix.lam"] and e.value.unexpected == ["l2.mix.dkv", "l2.mlp.up"] and "l1.mix.ra" in e.value.wrong[0]


def test_random_model_folder(tmp_path):
    """The framework's own writer of seeded random folders makes a folder that its reader accepts."""
    from fastgguf_b200.registry import config_from_dict, config_from_dir
    from fastgguf_b200.weights import check_weights, write_random_model
    d = write_random_model(config_from_dict(CASE_C), 5, str(tmp_path / "r"))
    again = config_from_dir(d)
    assert again.describe()["layer_kinds"] == config_from_dict(CASE_C).describe()["layer_kinds"]
    assert len(check_weights(again, model_dir=d)) == len(tensor_shapes(CASE_C))


def test_kernel_libraries_by_model():
    from fastgguf_b200 import capi
    from fastgguf_b200.registry import config_from_dict
    spec = config_from_dict(CASE_B).spec_json()           # no head of 64 or 128 numbers anywhere: no tensor-core attention
    assert capi.kernel_modules_for(spec, capi.FG_BF16) == ("core", "tc", "mix")
    assert capi.kernel_modules_for(spec, capi.FG_F32) == ("core", "mix")
    assert capi.kernel_modules_for(config_from_dict(CASE_C).spec_json(), capi.FG_BF16) == ("core", "tc", "attn", "mix")
