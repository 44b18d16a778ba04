"""A plain, slow restatement of the Kulanex design in float64 PyTorch on the CPU: one function per
mechanism, whole sequences, no cache and no state carried between calls.  It shares no code with
the library; the tests compare the library's kernels, cache, state and step function with it.

Notation: W weights stored [out, in] and applied as W n; x the residual stream, which every sublayer reads
as it is; p a position counted from 0.  In attention: H query heads of d on G key heads.  In the channel
delta mixer: H value heads of dv on G key heads of d, S [d, dv] a head's state.  In the exponentially gated
memory: H heads, keys of d, values of dv, S [d, dv] and z [d] a head's state.
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
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, weight, eps):
    """RMS norm whose weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + weight)


def unit_length(x, eps=1e-6):
    """x / sqrt(sum(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def causal_taps(u, taps_w):
    """u: [T, channels]; taps_w: [channels, taps].  y_t = sum_j taps_w[:, j] * u_(t - taps + 1 + j),
    rows before the first count as zero; the last column multiplies the token's own row."""
    T, taps = u.shape[0], taps_w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=F), u], dim=0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + padded[j:j + T] * taps_w[:, j]
    return y


# --------------------------------------------------------------------------- rotation
def frequencies(rot):
    """Angle per position of every pair [dims / 2].  With ``scaling``: a pair whose wavelength is short against
    the original length keeps its frequency, a long one's is divided by ``factor``, and between the two
    bounds the frequency is a mix of both."""
    r, base = int(rot["dims"]), float(rot["base"])
    out = []
    for i in range(r // 2):
        f = base ** (-2.0 * i / r)
        sc = rot.get("scaling")
        if sc:
            factor, low, high, orig = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            length = 2.0 * math.pi / f
            if length > orig / low:
                f = f / factor
            elif length >= orig / high:
                s = (orig / length - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=F)


def rotate_neighbours(x, positions, rot):
    """x: [T, heads, d]; pair (2i, 2i + 1) of the first ``dims`` dimensions turns by position * frequency i."""
    r = int(rot["dims"])
    a = positions.to(F)[:, None] * frequencies(rot)[None, :]
    cos, sin = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., 0:r:2], x[..., 1:r:2]
    turned = torch.stack([u * cos - v * sin, v * cos + u * sin], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., r:]], dim=-1)


# --------------------------------------------------------------------------- attention
def seen_mask(T, size, keep_first):
    """[T, T] bool: query i sees key j <= i if j is one of the last ``size`` positions or one of the first
    ``keep_first``."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def window_attention(w, p, m, x, eps):
    """Queries and keys pass a short convolution; the values are those convolved keys; then queries and
    keys are normed over the whole projection and turned by their positions."""
    T = x.shape[0]
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = causal_taps(x @ w[p + ".q"].T, w[p + ".q.conv"])
    k = causal_taps(x @ w[p + ".k"].T, w[p + ".k.conv"])
    v = k.reshape(T, G, d)
    q = (unit_rms(q, eps) * w[p + ".q.norm"]).reshape(T, H, d)
    k = (unit_rms(k, eps) * w[p + ".k.norm"]).reshape(T, G, d)
    pos = torch.arange(T)
    if m.get("rot"):
        q, k = rotate_neighbours(q, pos, m["rot"]), rotate_neighbours(k, pos, m["rot"])
    mask = m.get("mask") or {}
    seen = seen_mask(T, int(mask.get("size", T)), int(mask.get("keep_first", 0)))
    heads = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * float(m["scale"])
        heads.append(torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, g])
    return torch.cat(heads, dim=-1) @ w[p + ".o"].T


# --------------------------------------------------------------------------- exponentially gated memory
def memory_recurrence(q, k, v, log_in, log_keep):
    """q, k: [T, H, d], v: [T, H, dv], log_in, log_keep: [T, H].  With a running maximum mu that starts at 0,
    what is held (S and its normaliser z) is kept in units of exp(mu)."""
    T, H, d = q.shape
    S, z, mu = torch.zeros(H, d, v.shape[2], dtype=F), torch.zeros(H, d, dtype=F), torch.zeros(H, dtype=F)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        new = torch.maximum(log_keep[t] + mu, log_in[t])
        keep, add = torch.exp(log_keep[t] + mu - new), torch.exp(log_in[t] - new)
        mu = new
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        z = keep[:, None] * z + add[:, None] * k[t]
        read = torch.einsum("hdv,hd->hv", S, q[t])
        size = torch.maximum((z * q[t]).sum(-1).abs(), torch.exp(-mu)) + 1e-6
        out[t] = read / size[:, None]
    return out, S, z, mu


def gated_memory(w, p, m, x, eps):
    T = x.shape[0]
    H, d, dv, cap = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
    q = (x @ w[p + ".q"].T).reshape(T, H, d) / math.sqrt(d)
    k = (x @ w[p + ".k"].T).reshape(T, H, d)
    v = (x @ w[p + ".v"].T).reshape(T, H, dv)

    def capped(name):
        return cap * torch.tanh((x @ w[f"{p}.{name}"].T + w[f"{p}.{name}.b"]) / cap)

    o, _, _, _ = memory_recurrence(q, k, v, capped("i"), -softplus(-capped("f")))
    o = unit_rms(o, eps).reshape(T, H * dv) * w[p + ".norm"] * torch.sigmoid(x @ w[p + ".g"].T)
    return o @ w[p + ".o"].T


def side_by_side(w, p, m, x, eps):
    return (float(m["left_scale"]) * window_attention(w, p + ".left", m["left"], x, eps)
            + float(m["right_scale"]) * gated_memory(w, p + ".right", m["right"], x, eps))


# --------------------------------------------------------------------------- the channel delta mixer
def channel_delta_recurrence(q, k, v, decay, beta):
    """q, k: [T, H, d] (unit vectors, q scaled), v: [T, H, dv], decay: [T, H, d], beta: [T, H].  Per head and
    token: every row of the state shrinks by its own decay, what the state holds under k is moved towards v
    by the step beta, and q reads the result."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = S * decay[t][:, :, None]
        held = torch.einsum("hdv,hd->hv", S, k[t])
        S = S + k[t][:, :, None] * (beta[t][:, None] * (v[t] - held))[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def channel_delta(w, p, m, x, eps):
    T = x.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])

    def branch(name):
        return silu(causal_taps(x @ w[f"{p}.{name}"].T, w[f"{p}.{name}.conv"]))

    owner = torch.arange(H) // (H // G)
    q = unit_length(branch("q").reshape(T, G, d))[:, owner] / math.sqrt(d)
    k = unit_length(branch("k").reshape(T, G, d))[:, owner]
    v = branch("v").reshape(T, H, dv)
    beta = torch.sigmoid(x @ w[p + ".b"].T)
    pace = softplus((x @ w[p + ".a1"].T) @ w[p + ".a2"].T + w[p + ".dt_bias"]).reshape(T, H, d)
    decay = torch.exp(-torch.exp(w[p + ".A_log"])[None, :, None] * pace)
    o, _ = channel_delta_recurrence(q, k, v, decay, beta)
    o = (unit_rms(o, eps) * w[p + ".norm"]).reshape(T, H * dv)
    return (o * torch.sigmoid((x @ w[p + ".g1"].T) @ w[p + ".g2"].T)) @ w[p + ".o"].T


# --------------------------------------------------------------------------- feed-forward, model
def experts_ff(w, p, m, x, picks_out=None):
    """Each token's ``top`` experts by score, the score multiplying what the expert reads."""
    E, top = int(m["router"]["experts"]), int(m["router"]["top"])
    score = torch.sigmoid(x @ w[p + ".router"].T)
    picks = torch.topk(score, top, dim=-1).indices
    if picks_out is not None:
        picks_out.append(picks)
    out = torch.zeros_like(x)
    for e in range(E):
        for t in (picks == e).any(-1).nonzero()[:, 0].tolist():
            h = score[t, e] * x[t]
            out[t] += (silu(h @ w[f"{p}.e{e}.gate"].T) * (h @ w[f"{p}.e{e}.up"].T)) @ w[f"{p}.e{e}.down"].T
    return out


def forward(cfg, w, tokens, layers_out=None, picks_out=None):
    """Logits [T, vocab] of one whole sequence; ``layers_out`` (a list) receives the stream after
    every layer, ``picks_out`` the experts each layer picked."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = w["embed"][torch.tensor(tokens)]
    for l, L in enumerate(cfg["layers"]):
        p = f"l{l}"
        mixer = {"parallel": side_by_side, "channel_delta": channel_delta}[L["type"]]
        x = x + mult * offset_norm(mixer(w, p + ".mix", L["mixer"], x, eps), w[p + ".norm1"], eps)
        if L.get("mlp"):
            x = x + mult * offset_norm(experts_ff(w, p + ".mlp", L["mlp"], x, picks_out), w[p + ".norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return offset_norm(x, w["final.norm"], eps) @ w["head"].T
