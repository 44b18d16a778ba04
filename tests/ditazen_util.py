"""Small Ditazen configurations and weights of the tests' own making.

The weights are drawn here (not by the library's random mode) so that every constant is away from
its neutral value: norm weights, the convolutions' taps, decays, step sizes, gates.  Values are rounded to
bfloat16 and stored so, as a checkpoint is: the float32 engine, the bfloat16 engine and the plain
implementation read the same numbers.
"""
import json
import math
import os

import torch


def rot(dims, base=10000.0, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def windowed(heads=4, dim=24, rot_dim=8, vdim=32, kv_rank=32, size=24, base=10000.0, scale=None):
    return {"type": "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": size},
        "rot": rot(rot_dim, base), "scale": float(scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim))}}


def causal(heads=3, dim=32, rot_dim=16, vdim=24, kv_rank=40, q_rank=48, base=10000.0, scaling=(4.0, 64, 16.0, 1.0), scale=None):
    return {"type": "latent_attention_2", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
        "rot": rot(rot_dim, base, scaling), "scale": float(scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim))}}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def layer(mixer, ff=96, weights_of=None):
    d = dict(mixer, mlp={"kind": "dense", "ff": ff} if ff else None)
    if weights_of is not None:
        d["weights_of"] = weights_of
    return d


def again(layers, j):
    """A layer that uses layer j's tensors."""
    return dict(json.loads(json.dumps(layers[j])), weights_of=j)


def _with_repeats(layers, repeats):
    out = list(layers)
    for j in repeats:
        e = again(out, j)
        out.append(e)
    return out


# Sizes differ from layer to layer and from one configuration to the next; where one configuration
# has values that coincide or are 1, another has not.
CONFIGS = {
    # all three mixers, each used again by a later layer; latents larger and smaller than a head (folded and
    # grouped per-head products); a window shorter than a page and one longer (a ring of two pages); a layer
    # without a feed-forward
    "mix": dict(vocab=131, width=64, eps=1e-5, logit_scale=0.75, layers=_with_repeats([
        layer(windowed(4, 24, 8, 32, 32, size=24)),
        layer(delta(4, 2, 16, 24, 4), ff=80),
        layer(causal(3, 32, 16, 24, 40, 48)),
        layer(windowed(2, 40, 16, 16, 56, size=70, base=500.0), ff=None),
        layer(delta(6, 2, 32, 16, 3), ff=None)], (0, 2, 1))),
    # no YaRN change worth the name (factor 1), latents much larger than heads on both sides, heads that are no
    # multiples of 4, one query/key head, a layer that names one which names another
    "lean": dict(vocab=97, width=48, eps=1e-6, logit_scale=3.0, layers=[
        layer(causal(5, 10, 6, 14, 70, 33, scaling=(1.0, 32, 8.0, 2.0)), ff=50),
        dict(layer(causal(5, 10, 6, 14, 70, 33, scaling=(1.0, 32, 8.0, 2.0)), ff=50), weights_of=2),
        dict(layer(causal(5, 10, 6, 14, 70, 33, scaling=(1.0, 32, 8.0, 2.0)), ff=50), weights_of=0),
        layer(delta(3, 1, 10, 6, 2), ff=64)]),
    # ones: one head, a window of one position (a token sees itself only) and of exactly a page, a convolution of
    # one tap (a factor per channel), a rotated part of two dimensions
    "ones": dict(vocab=64, width=32, eps=1e-5, logit_scale=1.0, layers=[
        layer(windowed(1, 64, 64, 64, 64, size=64, base=300.0), ff=48),
        layer(windowed(1, 8, 2, 8, 12, size=1), ff=40),
        layer(causal(1, 16, 2, 8, 8, 10, scaling=(8.0, 16, 4.0, 1.0)), ff=16),
        layer(delta(1, 1, 8, 8, 1), ff=None)]),
    # latents of one number (whose norm is all but its sign, which a 16-bit rounding may turn: 32-bit only)
    "single": dict(vocab=50, width=40, eps=1e-5, logit_scale=1.0, layers=[
        layer(windowed(2, 8, 4, 8, 1, size=20), ff=40),
        layer(causal(1, 16, 2, 8, 1, 1, scaling=(8.0, 16, 4.0, 1.0)), ff=16)]),
    # peaked attention (a large score scale), so that one key more or less in sight changes the result
    "sharp": dict(vocab=80, width=64, eps=1e-5, logit_scale=1.0, layers=[
        layer(windowed(4, 32, 16, 32, 32, size=9, scale=1.0), ff=64),
        layer(windowed(9, 16, 8, 16, 24, size=130, scale=1.0), ff=64)]),
    # records of 128 on the tensor-core kernels, eight and more heads on a record, heads of 128, a wider model,
    # a state of 64 x 128
    "wide": dict(vocab=203, width=128, eps=1e-5, logit_scale=1.5, layers=_with_repeats([
        layer(windowed(10, 64, 32, 48, 96, size=150), ff=160),
        layer(delta(4, 4, 64, 128, 4), ff=200),
        layer(causal(16, 32, 64, 64, 64, 96, scaling=(16.0, 128, 32.0, 1.0)), ff=None)], (2,))),
    # records of more than 128 numbers, a delta state of 200 x 72
    "large": dict(vocab=90, width=96, eps=1e-5, logit_scale=0.5, layers=[
        layer(windowed(3, 48, 64, 40, 136, size=100), ff=96),
        layer(causal(8, 64, 32, 64, 224, 40, scaling=(2.0, 64, 8.0, 1.0)), ff=96),
        layer(delta(2, 2, 200, 72, 4), ff=64)]),
    # records wider than any tiled or tensor-core kernel takes
    "huge": dict(vocab=77, width=64, eps=1e-5, logit_scale=1.0, layers=[
        layer(windowed(5, 24, 12, 16, 300, size=90), ff=64), layer(causal(2, 32, 64, 40, 500, 30), ff=None)]),
    # one layer that sees everything: the tests make one far key stand out in it
    "far": dict(vocab=70, width=32, eps=1e-5, logit_scale=1.0, layers=[
        layer(causal(2, 16, 8, 16, 24, 20, scale=1.0), ff=48)]),
    # one delta layer alone
    "memory": dict(vocab=60, width=48, eps=1e-5, logit_scale=1.0, layers=[layer(delta(4, 2, 24, 16, 4), ff=48)]),
}


def config_dict(name):
    c = CONFIGS[name]
    return {"architecture": "Ditazen", "vocab": c["vocab"], "width": c["width"], "norm": {"eps": c["eps"]},
            "logit_scale": c["logit_scale"], "layers": json.loads(json.dumps(c["layers"]))}


def draw_weights(cfg, seed):
    """name -> tensor (bfloat16) for every tensor of the configuration."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out = {}

    def mat(name, rows, cols, gain=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).to(torch.bfloat16)

    def vec(name, n, mean, std):
        out[name] = (mean + std * torch.randn(n, generator=g)).to(torch.bfloat16)

    out["embed"] = torch.randn(cfg["vocab"], W, generator=g).to(torch.bfloat16)
    out["embed"] += 0.3                              # (a mean for the norms to take off)
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", L["mixer"]
        vec(p + "norm1", W, 1.0, 0.2)
        if L["type"] == "delta":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for s, n in (("q", G * d), ("k", G * d), ("v", H * dv)):
                mat(p + "mix." + s, n, W, gain=1.5)
                out[p + f"mix.{s}.conv"] = (0.4 * torch.randn(n, m["conv"], generator=g) + 0.3).to(torch.bfloat16)
            mat(p + "mix.b", H, W, gain=1.5), mat(p + "mix.a", H, W, gain=1.5)
            vec(p + "mix.A_log", H, -1.0, 0.8), vec(p + "mix.dt_bias", H, -1.0, 0.8)
            vec(p + "mix.norm", dv, 1.0, 0.2)
            mat(p + "mix.g", H * dv, W, gain=1.5), mat(p + "mix.o", W, H * dv, gain=1.5)
        else:
            H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            if L["type"] == "latent_attention_2":
                mat(p + "mix.dq", m["q_rank"], W), vec(p + "mix.dq.norm", m["q_rank"], 1.0, 0.2)
                mat(p + "mix.uq", H * (d + r), m["q_rank"], gain=1.2)
            else:
                mat(p + "mix.q", H * (d + r), W, gain=1.2)
            mat(p + "mix.dkv", R + r, W), vec(p + "mix.dkv.norm", R, 1.0, 0.2)
            mat(p + "mix.uk", H * d, R, gain=1.2), mat(p + "mix.uv", H * dv, R, gain=1.5)
            mat(p + "mix.g", H, W, gain=1.5), mat(p + "mix.o", W, H * dv, gain=1.5)
        if L["mlp"]:
            vec(p + "norm2", W, 1.0, 0.2)
            mat(p + "mlp.up", L["mlp"]["ff"], W, gain=1.5), mat(p + "mlp.down", W, L["mlp"]["ff"], gain=1.5)
    vec("final.norm", W, 1.0, 0.2)
    return out


def spike_token(w, cfg, token=0):
    """Change drawn weights of a model whose first layer sees everything so that every query of its heads looks
    at the key of ``token`` wherever it stands: only that token has a component along feature 0 of the
    embedding, which alone feeds number 0 of the latent; feature 1 is the same positive number for every token
    and alone feeds number 0 of the queries' latent, which feeds one unrotated channel of every head; that
    channel's key is number 0 of the latent."""
    m = cfg["layers"][0]["mixer"]
    d, r = m["dim"], m["rot_dim"]
    w["embed"][:, 0] = 0.0
    w["embed"][token, 0] = 6.0
    w["embed"][:, 1] = 5.0
    w["l0.norm1"][0] = w["l0.norm1"][1] = 1.0
    w["l0.mix.dkv"][0, :] = 0.0
    w["l0.mix.dkv"][:, 0] = 0.0
    w["l0.mix.dkv"][0, 0] = 8.0
    w["l0.mix.dq"][0, :] = 0.0
    w["l0.mix.dq"][0, 1] = 8.0
    w["l0.mix.dkv.norm"][0] = w["l0.mix.dq.norm"][0] = 1.0
    for h in range(m["heads"]):
        w["l0.mix.uq"][h * (d + r), :] = 0.0
        w["l0.mix.uq"][h * (d + r), 0] = 2.0
        w["l0.mix.uk"][h * d, :] = 0.0
        w["l0.mix.uk"][h * d, 0] = 2.0
    w["l0.mix.g"] *= 0.2


_folders = {}


def model_folder(root, name, seed=11, edit=None, edit_weights=None):
    """Write (once) config.json and model.safetensors of configuration ``name``; ``edit(cfg)`` may
    change the configuration dict first and ``edit_weights(weights, cfg)`` the drawn weights (their
    ``__name__`` tells the folders apart)."""
    from moe_b200.weights.safetensors_io import write_safetensors

    key = (str(root), name, seed, getattr(edit, "__name__", None), getattr(edit_weights, "__name__", None))
    if key not in _folders:
        cfg = config_dict(name)
        if edit is not None:
            edit(cfg)
        d = os.path.join(str(root), "_".join(str(k) for k in key[1:]))
        os.makedirs(d, exist_ok=True)
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cfg, f)
        w = draw_weights(cfg, seed)
        if edit_weights is not None:
            edit_weights(w, cfg)
        write_safetensors(os.path.join(d, "model.safetensors"), w)
        _folders[key] = d
    return _folders[key]


def tokens(vocab, n, seed):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
