"""Punolix without a GPU: config.json is read into typed fields, optional keys switch mechanisms off, refusals name the key, the size that
only the checkpoint gives comes from its tensors, the model's tensor list is what a checkpoint of this design holds, every pass of the loop keeps a
cache of its own."""
import json
import math

import pytest
import torch

import plain_punolix as plain
from punolix_models import CONFIGS, RANK, make_model_dir, random_weights


def spec_of(name):
    from marin_b200.config import PunolixConfig
    from marin_b200.models import architecture_of

    cfg = PunolixConfig.from_dict(CONFIGS[name])
    return cfg, architecture_of(cfg).build_spec(cfg)


def test_config_is_chosen_by_the_architecture_key_and_round_trips(tmp_path):
    from marin_b200.config import PunolixConfig, load_config

    cfg = load_config(make_model_dir(str(tmp_path / "a"), "A"))
    assert isinstance(cfg, PunolixConfig)
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.embedding_scale, cfg.residual_mult) == (83, 44, 1e-5, 3.0, 0.7)
    assert cfg.loop == {"start": 0, "stop": 2, "times": 3} and [layer.type for layer in cfg.layers] == ["attention", "parallel", "attention"]
    assert cfg.layers[0].mixer["softcap"] == 6.0 and cfg.layers[0].mixer["diff"] == 0.25 and cfg.layers[2].mlp is None
    left = cfg.layers[1].mixer["left"]
    assert left["mask"] == {"size": 11} and left["conv"] == 3 and left["rot"]["scaling"] == {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 60.0}
    again = PunolixConfig.from_dict(json.loads(json.dumps(cfg.to_json_dict())))
    assert again.layers == cfg.layers and again.loop == cfg.loop and again.to_json_dict() == cfg.to_json_dict()
    edge = PunolixConfig.from_dict({k: v for k, v in CONFIGS["C"].items() if k != "loop"})
    assert edge.loop is None and edge.embedding_scale == 1.0 and edge.residual_mult == 1.0 and edge.layers[1].mixer["softcap"] is None
    assert edge.layers[0].mixer["left"]["mask"] is None and edge.layers[2].mixer["left"]["conv"] is None and edge.layers[0].mixer["left"]["rot"]["scaling"] is None
    assert edge.layer_runs == [(i, None) for i in range(5)]


def test_the_decays_rank_comes_from_the_checkpoint(tmp_path):
    from marin_b200.config import PunolixConfig, load_config
    from marin_b200.models import Model, architecture_of

    cfg = load_config(make_model_dir(str(tmp_path / "c"), "C"))
    assert [layer.mixer["right"]["decay_rank"] for layer in cfg.layers if layer.type == "parallel"] == [RANK[64]] * 3
    assert PunolixConfig.from_dict(CONFIGS["C"]).layers[0].mixer["right"]["decay_rank"] == 16           # random weights: a default
    assert Model(architecture_of(cfg).build_spec(cfg)).blocks[0].mixer.inner[1].rank == RANK[64]


@pytest.mark.parametrize("damage, word", [
    (lambda c: c["layers"][0].__setitem__("type", "conv"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_heads"), "kv_heads"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("heads", 3), "kv heads"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 3), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 8), "dims"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("softcap", -1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][1]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].__setitem__("size", 0), "size"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("original"), "original"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].__setitem__("high", 0.5), "high"),
    (lambda c: c["layers"][1]["mixer"]["right"].pop("tau"), "tau"),
    (lambda c: c["layers"][1]["mixer"]["right"].__setitem__("tau", 0.0), "tau"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "mlp.kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["loop"].pop("times"), "times"),
    (lambda c: c["loop"].__setitem__("stop", 4), "loop"),
    (lambda c: c["loop"].__setitem__("start", 2), "loop"),
    (lambda c: c["embedding"].__setitem__("scale", "x"), "scale"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.__setitem__("width", "wide"), "width"),
])
def test_config_refusals_name_the_key(damage, word):
    from marin_b200.config import ConfigError, PunolixConfig

    raw = json.loads(json.dumps(CONFIGS["A"]))
    damage(raw)
    with pytest.raises(ConfigError, match=word):
        PunolixConfig.from_dict(raw)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_tensor_list_is_what_a_checkpoint_holds(tmp_path, name):
    from marin_b200.config import load_config
    from marin_b200.models import Model, architecture_of
    from marin_b200.weights import load_tensors

    d = make_model_dir(str(tmp_path / name), name)
    cfg = load_config(d)
    model = Model(architecture_of(cfg).build_spec(cfg))
    assert {s.name: tuple(s.shape) for s in model.tensor_specs()} == {k: tuple(v.shape) for k, v in random_weights(CONFIGS[name], 3).items()}
    assert len(load_tensors(d, model.tensor_specs())) == len(model.tensor_specs())
    assert model.capturable()
    for dtype in (torch.float32, torch.bfloat16):
        assert model.weight_bytes(dtype) > 0 and {"mb_attention_sink", "mb_gated_linear"} <= set(model.kernel_jobs(dtype))


def test_random_weights_mode_makes_a_folder_the_engine_reads(tmp_path):
    from marin_b200.config import PunolixConfig, load_config
    from marin_b200.models import Model, architecture_of
    from marin_b200.weights import load_tensors, write_random_model

    cfg = PunolixConfig.from_dict(dict(CONFIGS["C"], max_positions=300, eos_token_id=[3]))
    d = write_random_model(str(tmp_path / "r"), cfg, 5)
    back = load_config(d)
    assert back.layers == cfg.layers and back.max_position_embeddings == 300 and back.eos_token_ids == [3]
    load_tensors(d, Model(architecture_of(back).build_spec(back)).tensor_specs())


@pytest.mark.parametrize("name", list(CONFIGS))
def test_every_run_of_a_looped_layer_has_a_cache_of_its_own(name):
    from marin_b200.models import Model

    cfg, spec = spec_of(name)
    assert [(e.layer, e.enters) for e in spec.schedule] == plain.layer_runs(CONFIGS[name]) and all(e.cache_of is None for e in spec.schedule)
    assert tuple(spec.pass_vectors.shape) == (cfg.loop["times"], cfg.hidden_size)
    assert len(Model(spec).cache_needs()) == len(spec.schedule)
    _, other = spec_of(name)
    other.pass_vectors = None
    with pytest.raises(ValueError, match="pass"):
        Model(other)


def test_what_a_layer_keeps():
    """Two maps of a head share its page row: the keys side by side, the values once; a convolution's rows are a state beside the pages."""
    from marin_b200.models import Model
    from marin_b200.parts import PagedKV, StateNeed

    _, spec = spec_of("B")
    model = Model(spec)
    assert model.blocks[0].mixer.cache_need() == PagedKV(2, 128, None, 128)
    (pages, ring), state = model.blocks[1].mixer.cache_need()
    assert pages == PagedKV(2, 128, None, 64) and ring == StateNeed((4, 8 * 128 + 2 * 128 + 2 * 64), torch.float32) and state == StateNeed((4, 64, 64), torch.float32)
    _, edge = spec_of("C")
    pages, state = Model(edge).blocks[2].mixer.cache_need()                  # (no convolution: no ring)
    assert pages == PagedKV(1, 32, None, 48) and state == StateNeed((1, 128, 12), torch.float32)


@pytest.mark.parametrize("rot", [CONFIGS["A"]["layers"][1]["mixer"]["left"]["rot"], CONFIGS["B"]["layers"][1]["mixer"]["left"]["rot"],
                                 CONFIGS["B"]["layers"][0]["mixer"]["rot"]])
def test_rotation_frequencies(rot):
    from marin_b200.models.punolix import _position
    from marin_b200.parts import lookup

    spec = _position({"rot": dict(rot, scaling=rot.get("scaling")), "dim": 128}, True)
    part = lookup("position", spec.kind)(**spec.params)
    got, want = torch.tensor(part.frequencies(), dtype=torch.float64), torch.tensor(plain.frequencies(rot), dtype=torch.float64)
    assert torch.equal(got, want) or float((got / want - 1).abs().max()) < 1e-14
    assert part.interleaved and part.rotary_dim == rot["dims"]
    if rot.get("scaling"):
        ratio = want / torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)], dtype=torch.float64)
        assert float(ratio.max()) == 1.0 and abs(float(ratio.min()) - 1.0 / rot["scaling"]["factor"]) < 1e-12


def test_differential_attention_goes_without_what_it_cannot_have():
    from marin_b200.parts import PartSpec, lookup

    make = lambda **more: lookup("mixer", "sink_attention")(hidden=32, heads=2, kv_heads=1, head_dim=8, name="m", position=PartSpec("none", {}), differential=0.3, **more)
    assert make(sink=False, qk_norm=None).row_dim == 16
    for more in ({"sink": True, "qk_norm": None}, {"sink": False, "gate": True, "qk_norm": None}, {"sink": False, "qk_norm": "whole"}):
        with pytest.raises(ValueError, match="differential"):
            make(**more)


def test_pairs_of_maps_get_a_prompt_kernel_of_their_own():
    from marin_b200.kernels import build, ops

    jobs = ops.sink_attention_jobs(torch.bfloat16, 16, 2, 128, 128, pair=True)
    assert "mb_attention_tc_d128_g8_pair" in jobs and jobs["mb_attention_tc_d128_g8_pair"][1][-1] == "PAIR" and "mb_attention_sink_fast_d128_v128_g8" in jobs
    assert build.attention_tc_name(64, 4, 128) == "mb_attention_tc_d64_v128_g4" and build.attention_tc_job(64, 4, 128)[1] == ["HEAD_DIM=64", "GROUP=4", "V_DIM=128"]
    assert build.attention_tc_name(64, 4, 64) == build.attention_tc_name(64, 4)
    assert set(ops.sink_attention_jobs(torch.float32, 16, 2, 128, 128, pair=True)) == {"mb_attention_sink"}


@pytest.mark.parametrize("dv, slice_", [(16, 16), (128, 128), (256, 128), (144, 48), (48, 48), (160, 80)])
def test_value_slices_of_the_chunked_recurrence(dv, slice_):
    from marin_b200.kernels import ops

    assert ops._gla_slice(dv) == slice_ and dv % slice_ == 0
    assert math.isclose(ops.gla_chunk_bytes(64, dv), 4 * (64 * 64 + 64 * dv))


@pytest.mark.parametrize("window,chunk", [(0, 0), (5, 0), (0, 7), (3, 7)])
def test_keys_and_pairs_counted_for_a_step(window, chunk):
    """What a stage table divides by: keys read and (query, key) pairs under every mask."""
    from marin_b200.engine.profile import lengths_of

    def sees(i, j):
        return j <= i and (not window or i - j < window) and (not chunk or i // chunk == j // chunk)

    spans = [(9, 1), (13, 1), (0, 20), (6, 3)]
    for which, some in (("decode", spans[:2]), ("prefill", spans[2:]), ("all", spans)):
        pairs = sum(sees(i, j) for before, n in some for i in range(before, before + n) for j in range(i + 1))
        keys = sum(any(sees(i, j) for i in range(before, before + n)) for before, n in some for j in range(before + n))
        assert lengths_of(spans, window, chunk)[which] == [keys, pairs]
