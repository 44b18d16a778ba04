"""A plain, slow restatement of the Ditazen design in float64 PyTorch on the CPU: one function per
mechanism, whole sequences, no cache and no state carried between calls.  It shares no code with
the library; the tests compare the library's kernels, cache, state and step function with it.

Notation: W weights stored [out, in] and applied as W n; x the residual stream; n a sublayer's
input; p a position counted from 0.  In a latent attention mixer: H heads, d unrotated and r rotated
query/key dimensions a head, dv the value size, c the latent of a position (R numbers) and kr its one
rotated key part.  In a delta mixer: H value heads of dv on G key heads of d, S [d, dv] a head's state.
"""
import json
import math
import os
import struct

import torch

F = torch.float64


# --------------------------------------------------------------------------- files
def read_safetensors(path):
    """name -> tensor (float tensors widened to float64, integer tables kept)."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        data = f.read()
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "F64": torch.float64}
    out = {}
    for name, rec in head.items():
        if name == "__metadata__":
            continue
        a, b = rec["data_offsets"]
        t = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[rec["dtype"]]).reshape(rec["shape"])
        out[name] = t.to(F) if t.is_floating_point() else t
    return out


def read_model(folder):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(folder, "model.safetensors"))


# --------------------------------------------------------------------------- small functions
def layer_norm(x, weight, eps):
    """Centred, divided by sqrt(variance + eps), times a weight; no shift."""
    mean = x.mean(-1, keepdim=True)
    var = ((x - mean) ** 2).mean(-1, keepdim=True)
    return (x - mean) / torch.sqrt(var + eps) * weight


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_length(x, eps=1e-6):
    """x / sqrt(sum(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def gelu(z):
    """z times the normal distribution's probability of a value below z."""
    return z * 0.5 * (1.0 + torch.erf(z / math.sqrt(2.0)))


# --------------------------------------------------------------------------- rotation
def frequencies(rot):
    """(angle per position of every pair [dims/2], factor on cos and sin), with optional YaRN scaling."""
    r, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(r // 2, dtype=F)
    f = base ** (-2.0 * i / r)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, orig = float(sc["factor"]), float(sc["original"])

    def turn(t):                      # the (fractional) pair that makes t turns over the original length
        return r * math.log(orig / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(turn(float(sc["fast"]))), 0)
    hi = min(math.ceil(turn(float(sc["slow"]))), r - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x, positions, rot, neighbours):
    """x: [T, heads, r], all r dimensions turn: pair (i, i + r/2), or (2i, 2i + 1) with ``neighbours``;
    (u, v) becomes (u cos - v sin, v cos + u sin)."""
    f, m = frequencies(rot)
    a = positions.to(F)[:, None] * f[None, :]
    cos, sin = (torch.cos(a) * m)[:, None, :], (torch.sin(a) * m)[:, None, :]
    half = x.shape[-1] // 2
    u, v = (x[..., 0::2], x[..., 1::2]) if neighbours else (x[..., :half], x[..., half:])
    a, b = u * cos - v * sin, v * cos + u * sin
    if neighbours:
        return torch.stack([a, b], dim=-1).flatten(-2)
    return torch.cat([a, b], dim=-1)


# --------------------------------------------------------------------------- latent attention
def seen_mask(T, window):
    """[T, T] bool: query i sees key j with 0 <= i - j (< window, if there is one)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = i - j >= 0
    if window:
        seen &= i - j < window
    return seen


def latent_attention(w, p, m, n, eps, neighbours, query_latent):
    """Attention whose unrotated keys and whose values are projections of one latent a position, plus
    one rotated key part a position that all heads share; a softmax over the visible keys; one sigmoid
    gate a head.  ``query_latent``: the queries come through a latent of their own."""
    T = n.shape[0]
    H, d, r, dv, R = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    if query_latent:
        cq = unit_rms(n @ w[p + ".dq"].T, eps) * w[p + ".dq.norm"]
        q = (cq @ w[p + ".uq"].T).reshape(T, H, d + r)
    else:
        q = (n @ w[p + ".q"].T).reshape(T, H, d + r)
    down = n @ w[p + ".dkv"].T
    c = unit_rms(down[:, :R], eps) * w[p + ".dkv.norm"]
    pos = torch.arange(T)
    kr = rotate(down[:, None, R:], pos, m["rot"], neighbours)[:, 0]        # [T, r]
    qr = rotate(q[..., d:], pos, m["rot"], neighbours)
    k = (c @ w[p + ".uk"].T).reshape(T, H, d)
    v = (c @ w[p + ".uv"].T).reshape(T, H, dv)
    gate = torch.sigmoid(n @ w[p + ".g"].T)                                # [T, H]
    seen = seen_mask(T, int(m["mask"]["size"]) if m.get("mask") else None)
    heads = []
    for h in range(H):
        s = (q[:, h, :d] @ k[:, h].T + qr[:, h] @ kr.T) * float(m["scale"])
        a = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1)
        heads.append((a @ v[:, h]) * gate[:, h:h + 1])
    return torch.cat(heads, dim=-1) @ w[p + ".o"].T


# --------------------------------------------------------------------------- the delta mixer
def causal_taps(u, taps_w):
    """u: [T, channels]; taps_w: [channels, taps].  y_t = sum_j taps_w[:, j] * u_(t - taps + 1 + j),
    rows before the first count as zero; the last column multiplies the token's own row."""
    T, taps = u.shape[0], taps_w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=F), u], dim=0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + padded[j:j + T] * taps_w[:, j]
    return y


def delta_recurrence(q, k, v, decay, beta, S=None):
    """q, k: [T, H, d] (unit vectors, q scaled), v: [T, H, dv], decay, beta: [T, H].  Per head and token:
    the state shrinks by the decay, what it holds under k is moved towards v by the step beta, and q
    reads the result.  Returns (o [T, H, dv], the last state [H, d, dv])."""
    T, H, d = q.shape
    if S is None:
        S = torch.zeros(H, d, v.shape[2], dtype=F)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = S * decay[t][:, None, None]
        held = torch.einsum("hdv,hd->hv", S, k[t])
        S = S + torch.einsum("hd,hv->hdv", k[t], beta[t][:, None] * (v[t] - held))
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def delta_mixer(w, p, m, n, eps):
    T = n.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])

    def branch(name):
        return silu(causal_taps(n @ w[f"{p}.{name}"].T, w[f"{p}.{name}.conv"]))

    q, k = branch("q").reshape(T, G, d), branch("k").reshape(T, G, d)
    v = branch("v").reshape(T, H, dv)
    owner = torch.arange(H) // (H // G)
    q, k = unit_length(q)[:, owner] / math.sqrt(d), unit_length(k)[:, owner]
    beta = torch.sigmoid(n @ w[p + ".b"].T)
    decay = torch.exp(-torch.exp(w[p + ".A_log"]) * softplus(n @ w[p + ".a"].T + w[p + ".dt_bias"]))
    o, _ = delta_recurrence(q, k, v, decay, beta)
    o = unit_rms(o, eps) * w[p + ".norm"]
    return (o.reshape(T, H * dv) * silu(n @ w[p + ".g"].T)) @ w[p + ".o"].T


# --------------------------------------------------------------------------- feed-forward, model
def gelu_ff(w, p, n):
    return gelu(n @ w[p + ".up"].T) @ w[p + ".down"].T


def tensors_of(cfg, l):
    """The layer whose tensors layer l uses: its own, or those of the layer it names."""
    while cfg["layers"][l].get("weights_of") is not None:
        l = int(cfg["layers"][l]["weights_of"])
    return l


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence; ``layers_out`` (a list) receives the stream after
    every layer."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens)]
    for l in range(len(cfg["layers"])):
        L = cfg["layers"][l]
        p = f"l{tensors_of(cfg, l)}"
        n = layer_norm(x, w[p + ".norm1"], eps)
        if L["type"] == "latent_attention":
            x = x + latent_attention(w, p + ".mix", L["mixer"], n, eps, neighbours=False, query_latent=False)
        elif L["type"] == "latent_attention_2":
            x = x + latent_attention(w, p + ".mix", L["mixer"], n, eps, neighbours=True, query_latent=True)
        elif L["type"] == "delta":
            x = x + delta_mixer(w, p + ".mix", L["mixer"], n, eps)
        else:
            raise ValueError(L["type"])
        if L.get("mlp"):
            x = x + gelu_ff(w, p + ".mlp", layer_norm(x, w[p + ".norm2"], eps))
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].T * float(cfg["logit_scale"])
