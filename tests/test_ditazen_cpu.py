"""Ditazen without a GPU: the configuration reader, the translation into parts, the tensor names and
shapes against the tests' own checkpoints, the random-weights mode, and pieces of the plain
implementation worked out by hand."""
import json
import math

import pytest
import torch

import ditazen_util as U
import plain_ditazen as plain

F = torch.float64


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return tmp_path_factory.mktemp("ditazen_cpu")


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_config_parts_and_tensor_names_fit_the_checkpoint(root, name):
    from moe_b200.config import parse_config, read_config_json
    from moe_b200.models.decoder import expected_tensors
    from moe_b200.weights import SafetensorsStore

    d = U.model_folder(root, name)
    arch, typed = parse_config(read_config_json(d))
    assert arch.name == "Ditazen"
    spec = arch.model_spec(typed)
    store = SafetensorsStore(d)
    store.check({n: ts.shape for n, ts in expected_tensors(spec, store).items()}, spec.ignorable)
    assert typed.to_dict() == json.load(open(d + "/config.json"))
    own = [i for i in range(len(typed.layers)) if typed.owner(i) == i]
    assert len(spec.layers) == len(own) and len(spec.schedule) == len(typed.layers)
    assert [e.cache for e in spec.schedule] == list(range(len(typed.layers)))
    for i, e in enumerate(spec.schedule):
        ls, L = spec.layers[e.layer], typed.layers[i]
        assert ls.mixer.prefix == f"l{typed.owner(i)}.mix."
        assert ls.mixer.kind == ("delta" if L.type == "delta" else "latent_attention")
        assert (ls.ffn is None) == (L.ff is None) == (ls.norm2 is None)
    assert spec.head.params["tied"] and spec.final_norm.params["scale"] == typed.logit_scale


def test_a_config_written_from_the_typed_form_reads_back_the_same():
    from moe_b200.config.ditazen import DitazenConfig

    for name in U.CONFIGS:
        typed = DitazenConfig.from_dict(U.config_dict(name))
        bare = DitazenConfig(typed.vocab, typed.width, typed.norm_eps, typed.logit_scale, typed.layers)
        again = DitazenConfig.from_dict(bare.to_dict())
        assert again.layers == typed.layers and again.logit_scale == typed.logit_scale and again.vocab == typed.vocab


@pytest.mark.parametrize("bad,word", [
    (lambda c: c["layers"][0].update(type="attention"), "unknown mixer type"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=7), "even"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6), "must be rot_dim"),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][2]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "at least 1"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown kind"),
    (lambda c: c["layers"][5].update(weights_of=99), "names no other layer"),
    (lambda c: c["layers"][5].update(weights_of=5), "names no other layer"),
    (lambda c: c["layers"][0].update(weights_of=5), "leads back to itself"),
    (lambda c: c["layers"][5]["mixer"].update(heads=2), "differs from layer"),
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

    base = {"hidden_size": 32, "num_heads": 2, "head_dim": 8, "kv_rank": 1010, "scale": 1.0, "eps": 1e-5}
    with pytest.raises(ValueError, match="records of up to 1024"):
        make_part("mixer", PartSpec("latent_attention", dict(base, rot_dim=32, position={"kind": "rotary", "theta": 1e4, "rotary_dim": 32})))
    with pytest.raises(ValueError, match="exactly the rotated part"):
        make_part("mixer", PartSpec("latent_attention", dict(base, rot_dim=8, position={"kind": "rotary", "theta": 1e4, "rotary_dim": 4})))
    with pytest.raises(ValueError, match="up to 256"):
        make_part("mixer", PartSpec("delta", {"hidden_size": 32, "num_heads": 2, "num_kv_heads": 1, "head_dim": 300, "value_dim": 8,
                                              "taps": 4, "eps": 1e-5}))
    with pytest.raises(ValueError, match="none of"):
        make_part("ffn", PartSpec("dense_mlp", {"hidden_size": 8, "size": 8, "activation": "tanh"}))


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


# ----------------------------------------------------------------------------- the plain implementation by hand
def test_layer_norm_and_gelu_by_hand():
    y = plain.layer_norm(torch.tensor([[1.0, 3.0]], dtype=F), torch.tensor([2.0, 10.0], dtype=F), 0.0)
    assert torch.allclose(y, torch.tensor([[-2.0, 10.0]], dtype=F))
    assert abs(float(plain.gelu(torch.tensor(1.0, dtype=F))) - 0.8413447460685429) < 1e-12


def test_rotation_pairs_by_hand():
    x = torch.tensor([[[1.0, 0.0, 0.0, 1.0]]], dtype=F)
    r = {"dims": 4, "base": 100.0}                            # frequencies 1 and 1/10
    a, b = math.cos(3.0), math.sin(3.0)
    c, s = math.cos(0.3), math.sin(0.3)
    halves = plain.rotate(x, torch.tensor([3]), r, False)[0, 0]          # pairs (0, 2) and (1, 3)
    assert torch.allclose(halves, torch.tensor([a, -s, b, c], dtype=F))
    neigh = plain.rotate(x, torch.tensor([3]), r, True)[0, 0]            # pairs (0, 1) and (2, 3)
    assert torch.allclose(neigh, torch.tensor([a, b, -s, c], dtype=F))


def test_yarn_keeps_fast_pairs_and_stretches_slow_ones():
    f, m = plain.frequencies({"dims": 32, "base": 10000.0, "scaling": {"factor": 8.0, "original": 256, "fast": 8.0, "slow": 1.0}})
    g, one = plain.frequencies({"dims": 32, "base": 10000.0})
    assert one == 1.0 and abs(m - (0.1 * math.log(8.0) + 1.0)) < 1e-12
    assert float(f[0]) == float(g[0]) and abs(float(f[-1] * 8.0 - g[-1])) < 1e-15
    assert all(g[i] / 8.0 - 1e-15 <= f[i] <= g[i] + 1e-15 for i in range(16))


def test_delta_recurrence_by_hand():
    """Two tokens, state 1 x 1: decay, correction towards the value, read-out after the write."""
    q, k, v = (torch.tensor(t, dtype=F).reshape(2, 1, 1) for t in ([2.0, 3.0], [1.0, 0.5], [4.0, 6.0]))
    decay, beta = (torch.tensor(t, dtype=F).reshape(2, 1) for t in ([0.9, 0.5], [0.25, 1.0]))
    o, S = plain.delta_recurrence(q, k, v, decay, beta)
    s1 = 0.25 * 4.0
    s2 = 0.5 * s1 + 0.5 * (6.0 - 0.5 * s1 * 0.5)
    assert torch.allclose(o.flatten(), torch.tensor([2.0 * s1, 3.0 * s2], dtype=F)) and abs(float(S) - s2) < 1e-12


def test_attention_over_records_equals_attention_over_keys_and_values(root):
    """The rearrangement the library relies on: scores q . (Wuk c) = (Wuk^T q) . c and outputs Wuv (sum p c)."""
    d = U.model_folder(root, "mix")
    cfg, w = plain.read_model(d)
    for l, neighbours, latent in ((0, False, False), (2, True, True)):
        m, p = cfg["layers"][l]["mixer"], f"l{l}.mix"
        H, dd, r, dv, R = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        n = torch.randn(30, cfg["width"], generator=torch.Generator().manual_seed(1), dtype=F)
        ref = plain.latent_attention(w, p, m, n, 1e-5, neighbours, latent)
        q = n @ w[p + ".q"].T if not latent else (plain.unit_rms(n @ w[p + ".dq"].T, 1e-5) * w[p + ".dq.norm"]) @ w[p + ".uq"].T
        q = q.reshape(30, H, dd + r)
        down = n @ w[p + ".dkv"].T
        pos = torch.arange(30)
        rec = torch.cat([plain.unit_rms(down[:, :R], 1e-5) * w[p + ".dkv.norm"],
                         plain.rotate(down[:, None, R:], pos, m["rot"], neighbours)[:, 0]], dim=1)
        over = torch.einsum("thd,hdr->thr", q[..., :dd], w[p + ".uk"].reshape(H, dd, R))
        qr = torch.cat([over, plain.rotate(q[..., dd:], pos, m["rot"], neighbours)], dim=-1)
        s = torch.einsum("thx,jx->htj", qr, rec) * m["scale"]
        seen = plain.seen_mask(30, m["mask"]["size"] if m.get("mask") else None)
        ctx = torch.einsum("htj,jr->thr", torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1), rec[:, :R])
        o = torch.einsum("thr,hvr->thv", ctx, w[p + ".uv"].reshape(H, dv, R)) * torch.sigmoid(n @ w[p + ".g"].T)[:, :, None]
        assert torch.allclose(o.reshape(30, -1) @ w[p + ".o"].T, ref, atol=1e-9)
