"""Kulanex without a GPU: the configuration reader, the translation into parts, the tensor names and
shapes against the tests' own checkpoints, the random-weights mode, the cache's pinned pages, and pieces of
the plain implementation worked out by hand."""
import json
import math

import pytest
import torch

import kulanex_util as U
import plain_kulanex as plain

F = torch.float64


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return tmp_path_factory.mktemp("kulanex_cpu")


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_config_parts_and_tensor_names_fit_the_checkpoint(root, name):
    from moe_b200.config import parse_config, read_config_json
    from moe_b200.models.decoder import expected_tensors
    from moe_b200.weights import SafetensorsStore

    d = U.model_folder(root, name)
    arch, typed = parse_config(read_config_json(d))
    assert arch.name == "Kulanex"
    spec = arch.model_spec(typed)
    store = SafetensorsStore(d)
    store.check({n: ts.shape for n, ts in expected_tensors(spec, store).items()}, spec.ignorable)
    assert typed.to_dict() == json.load(open(d + "/config.json"))
    assert len(spec.layers) == len(typed.layers) and [e.cache for e in spec.schedule] == list(range(len(typed.layers)))
    for i, (ls, L) in enumerate(zip(spec.layers, typed.layers)):
        assert ls.block == "sandwich" and ls.norm1.kind == "none" and ls.mixer.prefix == f"l{i}.mix."
        assert ls.mixer.kind == ("channel_delta" if L.type == "channel_delta" else "side_by_side")
        assert (ls.ffn is None) == (L.mlp is None) == (ls.norm2 is None) == (ls.post2 is None)
        assert ls.post1.params["scale"] == typed.residual_mult and ls.post1.params["offset"] == 1.0
    assert not spec.head.params["tied"] and spec.final_norm.params["scale"] == 1.0


def test_a_config_written_from_the_typed_form_reads_back_the_same():
    from moe_b200.config.kulanex import KulanexConfig

    for name in U.CONFIGS:
        typed = KulanexConfig.from_dict(U.config_dict(name))
        bare = KulanexConfig(typed.vocab, typed.width, typed.norm_eps, typed.residual_mult, typed.layers)
        again = KulanexConfig.from_dict(bare.to_dict())
        assert again.layers == typed.layers and again.residual_mult == typed.residual_mult and again.vocab == typed.vocab


@pytest.mark.parametrize("bad,word", [
    (lambda c: c["layers"][0].update(type="delta"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(heads=3), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"].update(conv=17), "at most 16"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(vdim=8), "the values are the keys"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "not a multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=26), "at most dim"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("low"), "low"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(high=0.5), "below low"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), "at least 1"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(keep_first=-1), "at least 0"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(gate_cap=0), "positive"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "unknown kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "exceeds experts"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "non-empty"),
])
def test_config_errors_say_what_is_wrong(bad, word):
    from moe_b200.config import ConfigError, parse_config

    cfg = U.config_dict("mix")
    bad(cfg)
    with pytest.raises(ConfigError) as e:
        parse_config(cfg)
    assert word in str(e.value)


def test_parts_refuse_what_the_kernels_do_not_take():
    from moe_b200.config.spec import PartSpec
    from moe_b200.parts.base import make_part

    att = {"hidden_size": 32, "num_heads": 2, "num_kv_heads": 2, "head_dim": 8, "values_are_keys": True}
    with pytest.raises(ValueError, match="have their size"):
        make_part("mixer", PartSpec("gqa_attention", dict(att, value_dim=16)))
    with pytest.raises(ValueError, match="rotated values go with neither"):
        make_part("mixer", PartSpec("gqa_attention", dict(att, rotate_values=True)))
    with pytest.raises(ValueError, match="up to 256"):
        make_part("mixer", PartSpec("gqa_attention", dict(att, head_dim=300, value_dim=300)))
    with pytest.raises(ValueError, match="up to 256"):
        make_part("mixer", PartSpec("mlstm", {"hidden_size": 32, "num_heads": 2, "head_dim": 300, "value_dim": 8, "gate_cap": 1.0, "eps": 1e-5}))
    with pytest.raises(ValueError, match="neither softmax nor sigmoid"):
        make_part("ffn", PartSpec("routed_experts", {"hidden_size": 8, "num_experts": 2, "top_k": 1, "expert_size": 8, "score": "tanh"}))
    with pytest.raises(ValueError, match="no shared expert"):
        make_part("ffn", PartSpec("routed_experts", {"hidden_size": 8, "num_experts": 2, "top_k": 1, "expert_size": 8, "weight_input": True,
                                                     "shared_size": 8}))
    with pytest.raises(ValueError, match="low at most high"):
        make_part("position", PartSpec("rotary_bands", {"theta": 1e4, "rotary_dim": 8, "factor": 2.0, "low": 4.0, "high": 1.0, "original": 64}))


def test_random_weights_can_be_written_and_cover_every_tensor(tmp_path):
    from moe_b200.config import parse_config
    from moe_b200.models.decoder import expected_tensors
    from moe_b200.weights import SafetensorsStore
    from moe_b200.weights.random_init import write_random_model

    cfg = U.config_dict("mix")
    write_random_model(str(tmp_path), cfg, seed=3)
    arch, typed = parse_config(json.load(open(tmp_path / "config.json")))
    spec = arch.model_spec(typed)
    store = SafetensorsStore(str(tmp_path))
    store.check({n: ts.shape for n, ts in expected_tensors(spec, store).items()}, spec.ignorable)


# ----------------------------------------------------------------------------- the cache: pinned pages before a ring
def test_kept_positions_pin_whole_pages_in_front_of_the_ring():
    from moe_b200.cache import KVCache, KVRequest

    cache = KVCache({0: KVRequest(1, 16, 70, keep=3), 1: KVRequest(1, 16, 64, keep=65), 2: KVRequest(1, 16, 64), 3: KVRequest(1, 16, None)},
                    {}, max_tokens=64 * 40, max_slots=2, dtype=torch.float32, device="cpu")
    assert [(g.pinned, g.ring, g.ring_pages) for g in cache.groups] == [(64, 128, 3), (128, 64, 3), (0, 64, 1), (0, 0, 0)]
    s = cache.acquire()
    cache.ledger.extend(s, 1000)
    assert [len(gl.pages[s]) for gl in cache.ledger.groups] == [3, 3, 1, 16]
    cache.ledger.truncate(s, 999, [g.window + g.pinned if g.window else 0 for g in cache.groups])


def test_a_rewind_behind_pinned_pages_goes_as_far_as_the_ring_still_holds():
    from moe_b200.cache import CacheError, KVCache, KVRequest

    for back, fine in ((59, True), (60, False)):          # a ring of 128 behind one pinned page, a window of 70
        cache = KVCache({0: KVRequest(1, 16, 70, keep=3)}, {}, max_tokens=64 * 40, max_slots=1, dtype=torch.float32, device="cpu")
        s = cache.acquire()
        cache.ledger.extend(s, 1000)
        if fine:
            cache.truncate(s, 1000 - back)
            assert cache.length(s) == 1000 - back
        else:
            with pytest.raises(CacheError):
                cache.truncate(s, 1000 - back)


# ----------------------------------------------------------------------------- the plain implementation by hand
def test_kept_positions_and_window_by_hand():
    seen = plain.seen_mask(8, 2, 3).int().tolist()
    assert seen[7] == [1, 1, 1, 0, 0, 0, 1, 1] and seen[3] == [1, 1, 1, 1, 0, 0, 0, 0] and seen[0] == [1] + [0] * 7
    assert plain.seen_mask(5, 1, 0).int().tolist() == torch.eye(5).int().tolist()


def test_rotation_of_neighbours_by_hand():
    x = torch.tensor([[[1.0, 0.0, 0.0, 1.0, 7.0]]], dtype=F)
    y = plain.rotate_neighbours(x, torch.tensor([3]), {"dims": 4, "base": 100.0})[0, 0]          # frequencies 1 and 1/10
    assert torch.allclose(y, torch.tensor([math.cos(3.0), math.sin(3.0), -math.sin(0.3), math.cos(0.3), 7.0], dtype=F))


def test_frequency_bands_by_hand_and_against_the_library_s_table():
    from moe_b200.config.spec import PartSpec
    from moe_b200.parts.base import Runtime, make_part

    sc = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 100}
    r = {"dims": 16, "base": 10000.0, "scaling": sc}
    f, g = plain.frequencies(r), plain.frequencies({"dims": 16, "base": 10000.0})
    lengths = 2 * math.pi / g
    for a, b, l in zip(f.tolist(), g.tolist(), lengths.tolist()):
        if l < 25:
            assert a == b
        elif l > 100:
            assert a == b / 8
        else:
            s = (100 / l - 1) / 3
            assert abs(a - ((1 - s) * b / 8 + s * b)) < 1e-15 and b / 8 < a < b
    assert any(25 < l < 100 for l in lengths.tolist()) and lengths[0] < 25 and lengths[-1] > 100
    part = make_part("position", PartSpec("rotary_bands", dict(sc, theta=10000.0, rotary_dim=16, interleaved=True)))
    part.bind({}, Runtime("cpu", torch.float32))
    assert torch.equal(part.rotary_table()[0], f.to(torch.float32)) and part.cos_sin_scale() == 1.0


def test_channel_delta_recurrence_by_hand():
    """Two tokens, state 2 x 1: each row shrinks by its own decay, then the correction, then the read-out."""
    t = lambda v, *s: torch.tensor(v, dtype=F).reshape(*s)
    q, k = t([1.0, 1.0, 2.0, 3.0], 2, 1, 2), t([1.0, 0.5, 0.5, 1.0], 2, 1, 2)
    v, beta, decay = t([4.0, 6.0], 2, 1, 1), t([0.25, 1.0], 2, 1), t([0.9, 0.9, 0.5, 0.1], 2, 1, 2)
    o, S = plain.channel_delta_recurrence(q, k, v, decay, beta)
    s = [0.25 * 4.0 * 1.0, 0.25 * 4.0 * 0.5]
    s = [0.5 * s[0], 0.1 * s[1]]
    u = 6.0 - (s[0] * 0.5 + s[1] * 1.0)
    s2 = [s[0] + 0.5 * u, s[1] + 1.0 * u]
    assert torch.allclose(o.flatten(), t([1.5, 2 * s2[0] + 3 * s2[1]], 2)) and torch.allclose(S.flatten(), t(s2, 2))


def test_memory_recurrence_by_hand():
    """One head of 1 x 1: the running maximum starts at 0, and so bounds the divisor of a weak input."""
    t = lambda v: torch.tensor(v, dtype=F).reshape(-1, 1, 1)
    g = lambda v: torch.tensor(v, dtype=F).reshape(-1, 1)
    o, S, z, mu = plain.memory_recurrence(t([1.0, 1.0]), t([1.0, 2.0]), t([3.0, 5.0]), g([-2.0, 1.0]), g([-0.5, -0.25]))
    # token 1: mu = max(-0.5, -2) = -0.5; token 2: mu = max(-0.75, 1) = 1
    s1 = math.exp(-2 + 0.5) * 3.0
    o1 = s1 / (max(math.exp(-1.5), math.exp(0.5)) + 1e-6)
    keep = math.exp(-0.25 - 0.5 - 1.0)
    s2, z2 = keep * s1 + 10.0, keep * math.exp(-1.5) + 2.0
    assert torch.allclose(o.flatten(), torch.tensor([o1, s2 / (max(z2, math.exp(-1.0)) + 1e-6)], dtype=F))
    assert abs(float(mu) - 1.0) < 1e-12 and abs(float(S) - s2) < 1e-12 and abs(float(z) - z2) < 1e-12


def test_experts_read_the_weighted_input():
    w = {"f.router": torch.tensor([[2.0], [1.0]], dtype=F)}
    for e, gain in ((0, 3.0), (1, 5.0)):
        w.update({f"f.e{e}.gate": torch.tensor([[1.0]], dtype=F), f"f.e{e}.up": torch.tensor([[gain]], dtype=F), f"f.e{e}.down": torch.tensor([[1.0]], dtype=F)})
    y = plain.experts_ff(w, "f", {"router": {"experts": 2, "top": 1}}, torch.tensor([[0.5]], dtype=F))
    h = 0.5 / (1 + math.exp(-1.0))
    assert abs(float(y) - h / (1 + math.exp(-h)) * 3.0 * h) < 1e-12
