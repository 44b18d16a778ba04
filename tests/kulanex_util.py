"""Small Kulanex configurations and weights of the tests' own making.

The weights are drawn here (not by the library's random mode) so that every constant is away from
its neutral value: norm weights, the convolutions' taps, decays, step sizes, gates.  Values are rounded to
bfloat16 and stored so, as a checkpoint is: the float32 engine, the bfloat16 engine and the plain
implementation read the same numbers.

Routing is decisive: the first channels of the embedding (one an expert) hold a ranking of the experts that
depends on the token, and the routers read mostly those, so that which experts a token takes does not hang
on a rounding.
"""
import json
import math
import os

import torch


def rot(dims, base=10000.0, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def parallel(heads=4, kv_heads=2, dim=24, conv=3, dims=8, base=10000.0, scaling=(4.0, 1.0, 4.0, 64), size=24, keep=5, scale=None,
             rheads=3, rdim=16, rvdim=20, cap=9.0, ls=0.7, rs=0.4):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "rot": rot(dims, base, scaling),
            "scale": float(scale if scale is not None else 1.0 / math.sqrt(dim))}
    if size is not None:
        left["mask"] = {"size": size, "keep_first": keep}
    return {"type": "parallel", "mixer": {"left": left, "left_scale": ls, "right_scale": rs,
                                          "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "gate_cap": cap}}}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def layer(mixer, experts=5, top=2, ff=40):
    return dict(mixer, mlp={"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}} if experts else None)


# ranks: the inner widths of the delta layers' two narrow projections (the tensors alone say them).  Sizes differ from
# layer to layer and from one configuration to the next; where one configuration has values that coincide or are 1,
# another has not.
CONFIGS = {
    # both mixers, windows shorter and longer than a page with kept positions shorter and longer than a page, a layer
    # without a feed-forward
    "mix": dict(vocab=131, width=64, eps=1e-5, mult=0.6, ranks=(10, 14), layers=[
        layer(delta(4, 2, 16, 24, 4), 5, 2, 40),
        layer(parallel(4, 2, 24, 3, 8, size=24, keep=5), 4, 1, 56),
        layer(parallel(2, 1, 40, 5, 16, base=500.0, scaling=None, size=70, keep=67, rheads=2, rdim=24, rvdim=40, cap=4.0), 0),
        layer(delta(6, 3, 32, 16, 3), 7, 3, 24)]),
    # sizes that are no multiples of anything, one query/key head, every expert taken, no kept positions
    "lean": dict(vocab=97, width=52, eps=1e-6, mult=1.0, ranks=(3, 5), layers=[
        layer(parallel(3, 3, 10, 2, 6, base=1e6, scaling=(8.0, 0.5, 2.0, 32), size=33, keep=0, rheads=5, rdim=7, rvdim=9, cap=20.0,
                       ls=-0.5, rs=1.0), 3, 3, 18),
        layer(delta(3, 1, 10, 6, 2), 2, 2, 30)]),
    # ones: one head, a window of one position (beside which only kept keys are seen), a convolution of one tap, a
    # rotated part of two dimensions or none, one expert
    "ones": dict(vocab=64, width=40, eps=1e-5, mult=0.25, ranks=(1, 1), layers=[
        layer(parallel(1, 1, 8, 1, 2, scaling=None, size=1, keep=1, rheads=1, rdim=1, rvdim=1, cap=1.0, ls=1.0, rs=1.0), 1, 1, 16),
        layer(delta(1, 1, 8, 8, 1), 1, 1, 8),
        layer(parallel(1, 1, 64, 1, 0, scaling=None, size=64, keep=64, rheads=1, rdim=32, rvdim=32, cap=12.0), 2, 1, 16)]),
    # peaked attention (a large score scale), so that one key more or less in sight changes the result
    "sharp": dict(vocab=80, width=64, eps=1e-5, mult=0.8, ranks=(8, 8), layers=[
        layer(parallel(4, 4, 32, 2, 16, scaling=(2.0, 1.0, 2.0, 128), size=9, keep=3, scale=1.0, rheads=2, rdim=8, rvdim=8, ls=1.0, rs=0.2), 4, 1, 32),
        layer(parallel(8, 1, 16, 3, 8, scaling=None, size=130, keep=2, scale=1.2, rheads=2, rdim=8, rvdim=8, ls=1.0, rs=0.2), 0)]),
    # records of 64 and 128 on the tensor-core kernels, eight heads on a record, states of 64 x 128 and 32 x 64, a
    # wider model with more experts
    "wide": dict(vocab=203, width=128, eps=1e-5, mult=0.45, ranks=(16, 24), layers=[
        layer(delta(4, 4, 64, 128, 4), 12, 2, 64),
        layer(parallel(8, 8, 64, 4, 32, size=150, keep=9, rheads=4, rdim=32, rvdim=64), 9, 1, 72),
        layer(parallel(8, 1, 80, 5, 40, base=2e5, scaling=(3.0, 1.0, 5.0, 256), size=44, keep=130, rheads=2, rdim=64, rvdim=32), 10, 4, 32)]),
    # heads of more than 128 numbers on both sides, a delta state of 200 x 72
    "large": dict(vocab=90, width=96, eps=1e-5, mult=0.5, ranks=(20, 12), layers=[
        layer(parallel(2, 1, 160, 3, 64, size=100, keep=4, rheads=2, rdim=136, rvdim=40), 3, 1, 64),
        layer(delta(2, 2, 200, 72, 4), 3, 2, 64)]),
    # attention with no window at all beside a short memory: the tests make one far key stand out in it
    "far": dict(vocab=70, width=48, eps=1e-5, mult=1.0, ranks=(4, 4), layers=[
        layer(parallel(2, 2, 16, 2, 8, scaling=None, size=None, scale=1.0, rheads=1, rdim=4, rvdim=4, ls=1.0, rs=0.1), 0)]),
    # one layer of each recurrent mixer alone (the attention beside the second one counts little)
    "memory": dict(vocab=60, width=48, eps=1e-5, mult=1.0, ranks=(6, 6), layers=[
        layer(delta(4, 2, 24, 16, 4), 0),
        layer(parallel(2, 2, 8, 2, 4, scaling=None, size=16, keep=0, rheads=4, rdim=24, rvdim=16, cap=15.0, ls=0.1, rs=1.0), 0)]),
}


def config_dict(name):
    c = CONFIGS[name]
    return {"architecture": "Kulanex", "vocab": c["vocab"], "width": c["width"], "norm": {"eps": c["eps"]},
            "residual_mult": c["mult"], "layers": json.loads(json.dumps(c["layers"]))}


def draw_weights(cfg, seed, ranks=(8, 8)):
    """name -> tensor (bfloat16) for every tensor of the configuration."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out = {}

    def mat(name, rows, cols, gain=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).to(torch.bfloat16)

    def vec(name, n, mean, std):
        out[name] = (mean + std * torch.randn(n, generator=g)).to(torch.bfloat16)

    def taps(name, n, k):
        out[name] = (0.4 * torch.randn(n, k, generator=g) + 0.4).to(torch.bfloat16)

    most = max([L["mlp"]["router"]["experts"] for L in cfg["layers"] if L["mlp"]] or [0])
    embed = torch.randn(V, W, generator=g)
    for e in range(most):                       # expert e's strength for token t: a ranking with gaps of 4
        embed[:, e] = 4.0 * (((torch.arange(V) * 5 + e) % most) - most / 2)
    out["embed"] = embed.to(torch.bfloat16)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        vec(p + "norm1", W, 0.0, 0.2)
        out[p + "norm1"][:most] -= 0.9          # (the sublayers write little into those channels)
        if L["type"] == "channel_delta":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for s, n in (("q", G * d), ("k", G * d), ("v", H * dv)):
                mat(p + "mix." + s, n, W, gain=1.2)
                taps(p + f"mix.{s}.conv", n, m["conv"])
            mat(p + "mix.b", H, W, gain=0.8)
            mat(p + "mix.a1", ranks[0], W, gain=1.0), mat(p + "mix.a2", H * d, ranks[0], gain=1.0)
            mat(p + "mix.g1", ranks[1], W, gain=1.0), mat(p + "mix.g2", H * dv, ranks[1], gain=1.0)
            vec(p + "mix.A_log", H, -1.0, 0.8), vec(p + "mix.dt_bias", H * d, -1.0, 0.8)
            vec(p + "mix.norm", dv, 1.0, 0.2)
            mat(p + "mix.o", W, H * dv)
        else:
            a, r = m["left"], m["right"]
            q = p + "mix.left."
            for s, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"])):
                mat(q + s, n, W)
                vec(q + s + ".norm", n, 1.0, 0.3)
                taps(q + s + ".conv", n, a["conv"])
            mat(q + "o", W, a["heads"] * a["dim"])
            q = p + "mix.right."
            H, d, dv = r["heads"], r["dim"], r["vdim"]
            mat(q + "q", H * d, W, gain=0.7), mat(q + "k", H * d, W, gain=0.7), mat(q + "v", H * dv, W), mat(q + "g", H * dv, W)
            mat(q + "i", H, W, gain=0.7), mat(q + "f", H, W, gain=0.7)
            vec(q + "i.b", H, -0.5, 1.0), vec(q + "f.b", H, 2.5, 1.0)
            vec(q + "norm", H * dv, 1.0, 0.2), mat(q + "o", W, H * dv)
        if L["mlp"]:
            vec(p + "norm2", W, 0.0, 0.2)
            out[p + "norm2"][:most] -= 0.9
            E, ff = L["mlp"]["router"]["experts"], L["mlp"]["expert"]["ff"]
            router = 0.004 * torch.randn(E, W, generator=g)
            router[torch.arange(E), torch.arange(E)] += 0.15
            out[p + "mlp.router"] = router.to(torch.bfloat16)
            for e in range(E):
                mat(p + f"mlp.e{e}.gate", ff, W), mat(p + f"mlp.e{e}.up", ff, W), mat(p + f"mlp.e{e}.down", W, ff)
    vec("final.norm", W, 0.0, 0.2)
    mat("head", V, W)
    return out


def spike_token(w, cfg, token=0):
    """Change drawn weights so that, in every attention layer, every query looks at the key of ``token`` wherever it
    stands: only that token has a component along feature 0 of the embedding, which alone feeds one unrotated channel
    of every key head; feature 1 is the same positive number for every token and alone feeds that channel of every
    query head.  (The norm over the whole projection leaves that channel large against all others.)"""
    w["embed"][:, 0] = 0.0
    w["embed"][token, 0] = 6.0
    w["embed"][:, 1] = 5.0
    for i, L in enumerate(cfg["layers"]):
        if L["type"] != "parallel":
            continue
        a = L["mixer"]["left"]
        for s, heads, feature in (("q", a["heads"], 1), ("k", a["kv_heads"], 0)):
            t, c = w[f"l{i}.mix.left.{s}"], w[f"l{i}.mix.left.{s}.conv"]
            t[:, 0:2] = 0.0
            rows = torch.arange(heads) * a["dim"] + a["dim"] - 1        # the heads' last channels are not rotated
            t[rows, :] = 0.0
            t[rows, feature] = 4.0
            c[rows, :] = 0.0
            c[rows, -1] = 1.0
            w[f"l{i}.mix.left.{s}.norm"][rows] = 1.0


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
        w = draw_weights(cfg, seed, CONFIGS[name]["ranks"])
        if edit_weights is not None:
            edit_weights(w, cfg)
        write_safetensors(os.path.join(d, "model.safetensors"), w)
        _folders[key] = d
    return _folders[key]


def tokens(vocab, n, seed):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
