"""Pununex without a GPU: config.json is read into typed fields, optional keys switch mechanisms off, refusals name the key,
sizes that only the checkpoint gives come from its tensors, the model's tensor list is what a checkpoint of this design holds, the
cache manager keeps a sequence's first pages and gives an embedding a state of its own."""
import json
import random

import pytest
import torch

from pununex_models import CONFIGS, make_model_dir, random_weights


def test_config_is_chosen_by_the_architecture_key_and_round_trips(tmp_path):
    from marin_b200.config import PununexConfig, load_config

    cfg = load_config(make_model_dir(str(tmp_path / "a"), "A"))
    assert isinstance(cfg, PununexConfig)
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps) == (83, 44, 1e-5) and cfg.bigram == {"buckets": 31, "mul_prev": 5, "mul_cur": 3}
    assert [layer.type for layer in cfg.layers] == ["delta", "parallel", "parallel"]
    left = cfg.layers[1].mixer["left"]
    assert left["mask"] == {"size": 9, "keep_first": 4} and left["softcap"] == 4.0 and cfg.layers[1].mixer["right_scale"] == -0.9
    assert cfg.layers[1].mlp["router"] == {"experts": 5, "top": 2, "identity": 1, "scale": 1.5, "groups": {"count": 3, "keep": 2}}
    again = PununexConfig.from_dict(json.loads(json.dumps(cfg.to_json_dict())))
    assert again.layers == cfg.layers and again.to_json_dict() == cfg.to_json_dict()
    edge = PununexConfig.from_dict(CONFIGS["C"])
    assert edge.bigram is None and edge.layers[0].mixer["left"]["mask"] is None and edge.layers[0].mlp is None
    assert edge.layers[3].mixer["left"]["mask"]["keep_first"] == 0 and edge.layers[1].mlp["router"]["groups"] is None
    assert edge.layers[1].mlp["router"]["identity"] == 0 and edge.layers[1].mlp["shared"] is None and edge.layers[0].mixer["left"]["softcap"] is None


def test_ranks_come_from_the_checkpoint(tmp_path):
    """The inner widths of the two small products are in no key: the tensors' shapes give them, each its own."""
    from marin_b200.config import PununexConfig, load_config
    from marin_b200.models import Model, architecture_of

    cfg = load_config(make_model_dir(str(tmp_path / "b"), "B"))
    w = random_weights(CONFIGS["B"], 3)
    for i in (0, 2):
        right = cfg.layers[i].mixer["right"]
        assert right["decay_rank"] == w[f"l{i}.mix.right.a1"].shape[0] and right["gate_rank"] == w[f"l{i}.mix.right.g1"].shape[0]
        assert right["decay_rank"] != right["gate_rank"]
    assert PununexConfig.from_dict(CONFIGS["B"]).layers[0].mixer["right"]["decay_rank"] == 64           # random weights: a default
    assert Model(architecture_of(cfg).build_spec(cfg)).blocks[0].mixer.inner[1].decay_rank == w["l0.mix.right.a1"].shape[0]


@pytest.mark.parametrize("damage, word", [
    (lambda c: c["layers"][0].__setitem__("type", "conv"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_heads"), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("heads", 3), "kv heads"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][1]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][1]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].__setitem__("size", 0), "size"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].__setitem__("keep_first", -1), "keep_first"),
    (lambda c: c["layers"][1]["mixer"]["left"].__setitem__("softcap", -1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].__setitem__("count", 4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].__setitem__("keep", 4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"].__setitem__("top", 5), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"].__setitem__("identity", -1), "identity"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "glu"), "mlp.kind"),
    (lambda c: c["embedding"]["bigram"].pop("buckets"), "buckets"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.__setitem__("width", "wide"), "width"),
])
def test_config_refusals_name_the_key(damage, word):
    from marin_b200.config import ConfigError, PununexConfig

    raw = json.loads(json.dumps(CONFIGS["A"]))
    damage(raw)
    with pytest.raises(ConfigError, match=word):
        PununexConfig.from_dict(raw)


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
        assert model.weight_bytes(dtype) > 0 and model.bytes_read(8, dtype) <= model.weight_bytes(dtype) + 8 * 4 * cfg.hidden_size * 4
        assert {"mb_layer_norm", "mb_delta_rule"} <= set(model.kernel_jobs(dtype))


def test_random_weights_mode_makes_a_folder_the_engine_reads(tmp_path):
    from marin_b200.config import PununexConfig, load_config
    from marin_b200.models import Model, architecture_of
    from marin_b200.weights import load_tensors, write_random_model

    cfg = PununexConfig.from_dict(dict(CONFIGS["C"], max_positions=300, eos_token_id=[3]))
    d = write_random_model(str(tmp_path / "r"), cfg, 5)
    back = load_config(d)
    assert back.layers == cfg.layers and back.max_position_embeddings == 300 and back.eos_token_ids == [3]
    load_tensors(d, Model(architecture_of(back).build_spec(back)).tensor_specs())


def test_the_embedding_keeps_a_state_behind_the_layers(tmp_path):
    from marin_b200.cache import CacheManager
    from marin_b200.config import PununexConfig
    from marin_b200.models import Model, architecture_of
    from marin_b200.parts import StateNeed

    for name, own in (("A", True), ("C", False)):
        cfg = PununexConfig.from_dict(CONFIGS[name])
        model = Model(architecture_of(cfg).build_spec(cfg))
        needs = model.cache_needs()
        assert len(needs) == len(cfg.layers) + own
        cache = CacheManager(needs, [e.cache_of for e in model.spec.schedule], 8, 10, 4)
        cache.allocate(torch.device("cpu"), torch.float32)
        if own:
            assert needs[-1] == StateNeed((1,), torch.int32) and cache.place[len(cfg.layers)] == ("state", len(cfg.layers))
            assert cache.state[len(cfg.layers)].dtype == torch.int32 and tuple(cache.state[len(cfg.layers)].shape) == (5, 1)
        # a parallel layer: pages of its attention, and the matrices and the ring of its delta rule
        i = next(i for i, layer in enumerate(cfg.layers) if layer.type == "parallel")
        pages, (matrices, ring) = cache.place[i]
        assert isinstance(pages[0], int) and matrices[0] == ring[0] == "state" and matrices[1] != ring[1]


@pytest.mark.parametrize("seed", range(6))
def test_the_first_pages_are_kept_and_the_rest_given_back(seed):
    """At any length: the pages that hold a kept first position or one the window still sees are there, no other page is held,
    and every page comes back when the request ends."""
    from marin_b200.cache import DROPPED, CacheManager
    from marin_b200.parts import PagedKV

    rng = random.Random(seed)
    page, window, keep = rng.choice([2, 4, 8]), rng.choice([1, 5, 9, 16]), rng.choice([1, 3, 4, 8, 13, 30])
    m = CacheManager([PagedKV(1, 8, window, keep_first=keep), PagedKV(1, 8, window)], [None, None], page, 60, 2)
    assert [g.need.keep_first for g in m.groups] == [keep, 0]
    m.admit("a")
    length = 0
    while length < 100:
        length += rng.choice([1, 1, 2, 7])
        m.reserve("a", length)
        m.commit("a", length)
        for g, kept in ((0, keep), (1, 0)):
            table = m.block_table("a", g)
            for logical, p in enumerate(table):
                first, last = logical * page, logical * page + page - 1
                needed = first < kept or last >= max(0, length - window + 1)            # what the next token may look at
                assert (p != DROPPED) == needed, (length, g, logical)
        m.check()
    m.release("a")
    assert all(g.pool.num_held == 0 for g in m.groups)
    assert PagedKV(2, 16, 10, keep_first=4).bytes_read(1000, torch.bfloat16) == 14 * 2 * 32 * 2
