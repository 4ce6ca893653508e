"""The Buguzen configuration on the host, without a GPU: reading config.json, what it refuses, the model spec it becomes (loops as
a schedule with a vector a pass), the check of a checkpoint against it, and the cache it asks for."""
import copy
import math

import pytest

from buguzen_cases import CASES, CASE_A, CASE_B, CASE_C, CASE_D, CASE_E, random_weights, tensor_shapes, write_model


def spec_of(cfg):
    from fastgguf_b200.registry import config_from_dict
    return config_from_dict(cfg).spec_json()


def test_registered_and_chosen_by_name():
    from fastgguf_b200.config import BuguzenConfig
    from fastgguf_b200.registry import config_from_dict, registered_architectures
    assert "Buguzen" in registered_architectures()
    cfg = config_from_dict(CASE_A)
    assert isinstance(cfg, BuguzenConfig) and cfg.architecture == "Buguzen"
    assert cfg.to_dict() == CASE_A
    d = cfg.describe()
    assert d["hidden_size"] == 96 and d["vocab_size"] == 211 and d["num_hidden_layers"] == 4 and d["layer_runs"] == 8
    assert d["layer_kinds"] == ["attention+dense", "attention_2+none", "lightning+dense", "attention+none"]
    # two maps of keys beside one head of values; every pass of a looped layer keeps its own
    numbers = 2 * (2 * 20 + 28) + 3 * 3 * (24 + 24) + 3 * (2 * 12 + 40)
    assert d["kv_bytes_per_token"] == {"bfloat16": 2 * numbers, "float32": 4 * numbers}
    assert d["state_bytes_per_sequence"] == 4 * 3 * 3 * 16 * 24
    for case in CASES.values():
        assert config_from_dict(case).describe()["parameters"] == sum(math.prod(s) for s in tensor_shapes(case).values())


def test_loops_become_a_schedule():
    runs = [(r["layer"], r.get("pass") if r.get("reenter") else None) for r in spec_of(CASE_A)["schedule"]]
    assert runs == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert spec_of(CASE_A)["reentry"] == {"kind": "add_row", "params": {"hidden_size": 96, "rows": 3}, "tensors": {"table": "loop.step"}}
    assert [(r["layer"], r.get("pass")) for r in spec_of(CASE_C)["schedule"]] == [(0, 0), (1, None), (2, None), (0, 1), (1, None), (2, None)]
    assert [(r["layer"], r.get("pass")) for r in spec_of(CASE_D)["schedule"]] == [(0, None), (1, 0), (2, None)]
    assert "reentry" not in spec_of(CASE_B) and not any("reenter" in r for r in spec_of(CASE_B)["schedule"])


def test_spec_follows_the_file():
    spec = spec_of(CASE_A)
    kinds = [(l["block"], l["mixer"]["kind"], (l["feed_forward"] or {}).get("kind")) for l in spec["layers"]]
    assert kinds == [("prenorm", "sink_attention", "swiglu"), ("prenorm", "sink_attention", None), ("prenorm", "retention", "swiglu"),
                     ("prenorm", "sink_attention", None)]
    m, t = spec["layers"][0]["mixer"]["params"], spec["layers"][0]["mixer"]["tensors"]
    assert (m["n_heads"], m["n_kv_heads"], m["head_dim"], m["v_head_dim"], m["scale"], m["window"], m["differential"]) == (4, 2, 20, 28, 0.3, 9, 0.4)
    assert m["bias"] is True and m["eps"] == 2e-6 and "sink" not in m and "values" not in m
    assert m["position"]["params"] == {"head_dim": 20, "theta": 10000.0, "rotary_dim": 8, "layout": "adjacent",
                                       "scaling": {"rope_type": "linear", "factor": 3.0}}
    assert t["lambda_q2"] == "l0.mix.lq2" and t["v_proj.bias"] == "l0.mix.v.b" and "sinks" not in t
    m, t = spec["layers"][1]["mixer"]["params"], spec["layers"][1]["mixer"]["tensors"]
    assert (m["values"], m["qk_norm"], m["sink"], m["window"]) == ("keys", "head", True, 21) and "differential" not in m
    assert m["position"]["params"]["layout"] == "halves"
    assert m["position"]["params"]["scaling"] == {"rope_type": "llama3", "factor": 4.0, "low_freq_factor": 1.0, "high_freq_factor": 3.0,
                                                  "original_max_position_embeddings": 60.0}
    assert t["sinks"] == "l1.mix.sink" and t["q_norm.weight"] == "l1.mix.q.norm" and "v_proj.weight" not in t and "v_proj.bias" not in t
    m, t = spec["layers"][2]["mixer"]["params"], spec["layers"][2]["mixer"]["tensors"]
    assert m["decay"] == [0.5, 0.93, 0.999] and (m["k_scale"], m["qkv_activation"], m["norm"], m["gate_activation"]) == (1.0, "silu", "whole", "sigmoid")
    assert t["norm.weight"] == "l2.mix.norm" and t["g_proj.weight"] == "l2.mix.g"
    assert spec["layers"][3]["mixer"]["params"]["window"] == 0 and spec["layers"][3]["mixer"]["params"]["position"]["params"]["scaling"] is None
    assert spec["layers"][0]["feed_forward"]["params"] == {"hidden_size": 96, "d_ff": 80, "activation": "relu"}
    s = spec["layers"][2]["token_input"]
    assert s["params"] == {"hidden_size": 96, "vocab_size": 211, "dim": 8, "column": 16, "table_dim": 32, "eps": 2e-6}
    assert s["tensors"] == {"table": "side.embed", "gate": "l2.side.gate", "proj": "l2.side.proj", "norm": "l2.side.norm"}
    assert spec["head"]["tensors"]["weight"] == "head" and spec["embedding"]["tensors"]["weight"] == "embed"
    assert "token_input" not in spec_of(CASE_E)["layers"][0] and spec_of(CASE_B)["layers"][4]["mixer"]["params"]["position"] is None


def test_python_spec_round_trip():
    from fastgguf_b200.engine.spec import ModelSpec
    for case in (CASE_A, CASE_B):
        j = spec_of(case)
        again = ModelSpec.from_json(j).to_json()
        assert again["schedule"] == j["schedule"] and again.get("reentry") == j.get("reentry")
        for a, b in zip(again["layers"], j["layers"]):
            assert a["mixer"] == b["mixer"] and a.get("token_input") == b.get("token_input") and (a["feed_forward"] or None) == (b["feed_forward"] or None)


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
    (["layers", 0, "type"], "conv", "not known"), (["layers", 1, "mixer"], KeyError, "mixer"), (["layers"], [], "layers"),
    (["layers", 0, "mixer", "kv_heads"], 3, "multiple"), (["layers", 0, "mixer", "diff"], KeyError, "diff"), (["layers", 0, "mixer", "mask"], {"size": 0}, "size"),
    (["layers", 0, "mixer", "rot", "dims"], 22, "dims"), (["layers", 0, "mixer", "rot", "dims"], 7, "dims"), (["layers", 0, "mixer", "rot", "scaling"], {}, "factor"),
    (["layers", 0, "mixer", "scale"], 0.0, "scale"), (["layers", 0, "mixer", "rot", "base"], 0.0, "base"),
    (["layers", 1, "mixer", "vdim"], 16, "vdim"), (["layers", 1, "mixer", "rot", "scaling", "low"], KeyError, "low"),
    (["layers", 1, "mixer", "rot", "scaling", "original"], 0, "positive"), (["layers", 1, "mixer", "heads"], KeyError, "heads"),
    (["layers", 2, "mixer", "decay"], [0.5], "decay"), (["layers", 2, "mixer", "decay"], [0.5, 0.5, 1.5], "decay"), (["layers", 2, "mixer", "vdim"], 0, "positive"),
    (["layers", 0, "mlp", "kind"], "moe", "not known"), (["layers", 0, "mlp", "ff"], 0, "ff"), (["loop", "stop"], 5, "loop"), (["loop", "times"], 0, "loop"),
    (["loop", "start"], 3, "loop"), (["token_side", "dim"], 0, "token_side"),
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
    del bad["l0.mix.lk2"], bad["l1.mix.sink"]
    bad["l1.mix.v"] = W["l1.mix.k"]                   # the values are the keys
    bad["l1.mlp.up"] = W["l0.mlp.up"]                 # a layer without a feed-forward has no tensors for one
    bad["loop.step"] = W["loop.step"][:2].contiguous()
    with pytest.raises(WeightError) as e:
        check_weights(config_from_dict(CASE_A), model_dir=write_model(tmp_path / "bad", CASE_A, bad))
    assert e.value.missing == ["l0.mix.lk2", "l1.mix.sink"] and e.value.unexpected == ["l1.mix.v", "l1.mlp.up"] and "loop.step" in e.value.wrong[0]


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
    assert capi.kernel_modules_for(spec_of(CASE_A), capi.FG_BF16) == ("core", "tc", "mix")       # no head of 64 or 128 numbers
    assert capi.kernel_modules_for(spec_of(CASE_A), capi.FG_F32) == ("core", "mix")
    assert capi.kernel_modules_for(spec_of(CASE_B), capi.FG_BF16) == ("core", "tc", "attn", "mix")


def test_shared_value_heads_in_the_cache():
    """Two key heads to a head of values: the value pools are that much smaller, and groups that differ in it share no pages."""
    from fastgguf_b200.cache import CacheRequest, PagedKVCache, cache_bytes
    both = cache_bytes({0: CacheRequest(4, 64, None, 128)}, 640)
    shared = cache_bytes({0: CacheRequest(4, 64, None, 128, n_v_heads=2)}, 640)
    assert both["bytes_per_token"] == 2 * 4 * (64 + 128) and shared["bytes_per_token"] == 2 * (4 * 64 + 2 * 128)
    assert both["bytes"] > shared["bytes"]
    c = PagedKVCache({0: CacheRequest(4, 64, 20, 128, n_v_heads=2), 1: CacheRequest(4, 64, 20, 128), 2: CacheRequest(4, 64, 20, 128, n_v_heads=2)}, max_tokens=640,
                     max_seq_len=640, n_slots=2)
    assert len(c.groups) == 2
