"""Kulanex on the GPU against the plain implementation (tests/plain_kulanex.py): every mechanism
alone, whole prompts, decoding through cache and state, portions of prompts, unequal batches, slots,
pages and state used again, windows', kept positions' and pages' edges, far keys, the first tokens, long decoding,
greedy generation and the trace program.  Configurations and weights are the tests' own
(tests/kulanex_util.py)."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import kulanex_util as U
import gpu_util as G
import helpers
import plain_kulanex as plain

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
NAMES = ["mix", "lean", "ones", "sharp", "wide", "large", "memory"]
F = torch.float64


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return tmp_path_factory.mktemp("kulanex")


_engines, _models, _refs, _sens = {}, {}, {}, {}


def engine_of(root, name, dtype, max_slots=None, use_graphs=None, edit=None, edit_weights=None):
    import moe_b200
    from moe_b200.engine import Engine

    d = U.model_folder(root, name, edit=edit, edit_weights=edit_weights)
    key = (d, dtype, max_slots, use_graphs)
    if key not in _engines:
        _engines[key] = Engine(moe_b200.load_model(d, dtype=dtype), max_tokens=2048, max_slots=max_slots,
                               use_graphs=use_graphs)
    return d, _engines[key]


def model_of(folder):
    if folder not in _models:
        _models[folder] = plain.read_model(folder)
    return _models[folder]


def reference(folder, toks):
    key = (folder, tuple(toks))
    if key not in _refs:
        cfg, w = model_of(folder)
        _refs[key] = plain.forward(cfg, w, toks)
    return _refs[key]


def sensitivity(folder, toks):
    """Per position: how far the plain result moves (as a fraction of the largest logit) when every weight
    is changed by a relative 2^-8, the spacing of bfloat16 (the larger of two draws).  Where that is much (peaked
    scores, a head whose output nearly cancels before it is divided by its own size) no 16-bit
    implementation can be held to the same bound as elsewhere."""
    key = (folder, tuple(toks))
    if key not in _sens:
        cfg, w = model_of(folder)
        g = torch.Generator().manual_seed(len(toks))
        ref = reference(folder, toks)
        worst = torch.zeros(len(toks), dtype=F)
        for _ in range(2):
            w2 = {n: t * (1.0 + 2.0 ** -8 * torch.randn(t.shape, generator=g, dtype=F)) for n, t in w.items()}
            worst = torch.maximum(worst, (plain.forward(cfg, w2, toks) - ref).abs().amax(dim=1) / float(ref.abs().max()))
        _sens[key] = worst
    return _sens[key]


def allowed(folder, toks, tol):
    """The bound at every position: ``tol``, and for the 16-bit path four times the position's sensitivity on top."""
    if tol < 1e-3:
        return torch.full((len(toks),), tol, dtype=F)
    return tol + 4.0 * sensitivity(folder, toks)


def check_schedule(folder, eng, requests, steps, tol):
    """Run ``steps`` (helpers.run_schedule) and compare every wanted place with the plain
    implementation run whole.  Returns {request: {position: row}} for comparisons between cuts."""
    logits, _ = helpers.run_schedule(eng, steps)
    out = {}
    for rid, toks in requests.items():
        ref = reference(folder, toks)
        scale = float(ref.abs().max())
        bound = allowed(folder, toks, tol)
        rows = {pos: row for (r, pos), row in logits.items() if r == rid}
        assert rows, rid
        for pos, row in rows.items():
            err = float((row.double() - ref[pos]).abs().max()) / scale
            assert err < float(bound[pos]), f"{rid} at position {pos} of {len(toks)}: relative error {err:.3g}"
        out[rid] = rows
    return out


def portions_schedule(rid, toks, sizes):
    """One request in portions of the given sizes (the last size repeats), logits at every place."""
    steps, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(i, len(sizes) - 1)], len(toks) - at)
        steps.append({"entries": [(rid, toks[at:at + n], list(range(n)))], "end": [rid] if at + n == len(toks) else []})
        at, i = at + n, i + 1
    return steps


def dev(t, dtype=torch.float32):
    return t.to(dtype).to(DEV).contiguous()


def close(got, want, tol):
    want = want.double()
    err = float((got.double().cpu() - want).abs().max())
    assert err <= tol * max(1.0, float(want.abs().max())), err


# ----------------------------------------------------------------------------- norms on a sublayer's output
@pytest.mark.parametrize("W", [1, 30, 64, 260, 516, 1030, 2048, 5000, 8192, 20000])
@pytest.mark.parametrize("source", ["one", "two", "experts", "none"])
@pytest.mark.parametrize("then", [False, True])
def test_norm_of_a_sublayer_s_output_in_front_of_the_sum(W, source, then):
    """x += rms(y) w with y one output, two with a factor each, or the sum of routed experts' outputs; what follows is the
    stream itself or its own norm; with chosen rows the stream stays."""
    from moe_b200.ops import core

    g = torch.Generator().manual_seed(W)
    T, eps, eps2 = 7, 1e-5, 1e-3
    x = torch.randn(T, W, generator=g)
    a, b = 30 * torch.randn(T, W, generator=g), 0.01 * torch.randn(T, W, generator=g)
    pw, w = 1 + 0.3 * torch.randn(W, generator=g), 1 + 0.3 * torch.randn(W, generator=g)
    st = core.new_status(DEV)
    kw, y = {}, None
    if source == "one":
        kw, y = dict(a=dev(b), sa=-2.0), -2.0 * b.double()
    elif source == "two":
        kw, y = dict(a=dev(a), sa=0.5, b=dev(b), sb=3.0), 0.5 * a.double() + 3.0 * b.double()
    elif source == "experts":
        e = torch.randn(2 * T, W, generator=g)
        pos = torch.randperm(2 * T, generator=g).int()
        pos[5] = -1
        kw = dict(combine=(dev(e), dev(pos, torch.int32), None, 2, None))
        y = torch.stack([sum((e[p].double() for p in pos[2 * t:2 * t + 2].tolist() if p >= 0), torch.zeros(W, dtype=F)) for t in range(T)])
    if y is not None:
        kw["post"] = (dev(pw), eps)
    if then:
        kw["norm"] = (dev(w), eps2)
    new = x.double() + (plain.unit_rms(y, eps) * pw.double() if y is not None else 0.0)
    ref = plain.unit_rms(new, eps2) * w.double() if then else new
    xs = dev(x)
    o32, o16 = torch.empty((T, W), device=DEV), torch.empty((T, W), dtype=torch.bfloat16, device=DEV)
    core.post_norm(xs, out32=o32, out16=o16, status=st, **kw)
    close(xs, new, 3e-6), close(o32, ref, 5e-6), close(o16, ref, 1e-2)
    rows = torch.tensor([5, 0, 5], dtype=torch.int32, device=DEV)
    picked, xs = torch.empty((3, W), device=DEV), dev(x)
    core.post_norm(xs, rows=rows, out32=picked, status=st, **kw)
    assert torch.equal(xs.cpu(), x)
    close(picked, ref[[5, 0, 5]], 5e-6)
    core.check_status(st)


# ----------------------------------------------------------------------------- attention's own kernels
@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("nh,nkv,d,taps,rot,neighbours,shared", [
    (4, 2, 24, 3, 8, True, True), (1, 1, 8, 1, 2, True, True), (3, 3, 10, 2, 6, True, True), (8, 1, 64, 4, 64, True, True),
    (2, 2, 160, 5, 48, True, True), (5, 5, 32, 16, 0, True, True), (4, 2, 32, 4, 16, False, True), (4, 2, 20, 3, 8, True, False),
    (6, 3, 16, 1, 16, False, False), (16, 16, 128, 4, 64, True, True)])
def test_convolution_whole_norm_rotation_and_records_over_steps(bf16, nh, nkv, d, taps, rot, neighbours, shared):
    """Two sequences of unequal lengths over steps that bring fewer rows than the convolution has taps, the last two of one
    token each (in which the kernel moves the state on itself): records of queries, keys and values, and the state.
    ``shared``: the values are the convolved keys, neither normed nor turned."""
    from moe_b200.cache import KVCache, KVRequest
    from moe_b200.ops import core
    from moe_b200.parts.attention import record_width

    g = torch.Generator().manual_seed(nh * 100 + d)
    dt, eps = (torch.bfloat16 if bf16 else torch.float32), 1e-5
    dv = d if shared else d + 4
    D = record_width(d, dv, bf16)
    ch = (nh + nkv) * d + (0 if shared else nkv * dv)
    rows = {s: 2 * torch.randn(n, ch + 4, generator=g) for s, n in LENS.items()}
    tw = 0.5 * torch.randn(ch, taps, generator=g)
    qn, kn = 1 + 0.3 * torch.randn(nh * d, generator=g), 1 + 0.3 * torch.randn(nkv * d, generator=g)
    r = {"dims": rot, "base": 500.0, "scaling": {"factor": 3.0, "low": 1.0, "high": 3.0, "original": 60}}
    freq = dev(plain.frequencies(r)) if rot else None
    cache = KVCache({0: KVRequest(nkv, D, None)}, {0: None}, max_tokens=64 * 12, max_slots=4, dtype=dt, device=DEV)
    slots = [cache.acquire() for _ in range(3)]
    for s, n in LENS.items():
        G.give_pages(cache, slots[s + 1], n)
    st = core.new_status(DEV)
    room = -(-((taps - 1) * ch) // 4) * 4 + 8
    state = torch.zeros((5, room), device=DEV)
    outs = {0: [], 1: []}
    for step in CUTS:
        batch = G.make_batch(DEV, [slots[s + 1] for s, _, _ in step], [a for _, a, _ in step], [b - a for _, a, b in step])
        T = batch.num_tokens
        proj = dev(torch.cat([rows[s][a:b] for s, a, b in step]))
        q, k, v = (torch.full((T, n, D), 7.0, dtype=dt, device=DEV) for n in (nh, nkv, nkv))
        moved = core.whole_conv_prepare(proj, batch, nh=nh, nkv=nkv, d=d, dv=dv, width=D, q=q, k=k, v=v, taps_w=dev(tw.t()),
                                        state=state[:, :room - 4] if taps > 1 else None, q_norm=dev(qn), k_norm=dev(kn), eps=eps,
                                        freq=freq, rot=rot, neighbours=neighbours, values_are_keys=shared, commit=cache.view(0), status=st)
        assert moved == (batch.all_decode or taps == 1)
        if not moved:
            core.conv_state_update(proj, state[:, :room - 4], batch, taps=taps, channels=ch)
        i = 0
        for s, a, b in step:
            outs[s].append([t[i:i + b - a].cpu() for t in (q, k, v)])
            i += b - a
    core.check_status(st)

    def turned(x, n):
        pos = torch.arange(n)
        if not rot:
            return x
        if neighbours:
            return plain.rotate_neighbours(x, pos, r)
        ang = pos.to(F)[:, None] * plain.frequencies(r)[None, :]
        c, s_ = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        u, w_ = x[..., :rot // 2], x[..., rot // 2:rot]
        return torch.cat([u * c - w_ * s_, w_ * c + u * s_, x[..., rot:]], dim=-1)

    tol = 1e-2 if bf16 else 1e-4
    for s, n in LENS.items():
        y = plain.causal_taps(rows[s][:, :ch].double(), tw.double())
        q = turned((plain.unit_rms(y[:, :nh * d], eps) * qn.double()).reshape(n, nh, d), n)
        kc = y[:, nh * d:(nh + nkv) * d]
        k = turned((plain.unit_rms(kc, eps) * kn.double()).reshape(n, nkv, d), n)
        v = (kc if shared else y[:, (nh + nkv) * d:]).reshape(n, nkv, dv)
        got = [torch.cat([o[j] for o in outs[s]]) for j in range(3)]
        for have, ref, width in zip(got, (q, k, v), (d, d, dv)):
            close(have[..., :width], ref, tol)
            assert width == D or float(have[..., width:].abs().max()) == 0.0
        table = cache.groups[0].table.cpu()[slots[s + 1]]
        pos = torch.arange(n)
        for plane, have in ((cache.view(0).k, got[1]), (cache.view(0).v, got[2])):
            assert torch.equal(plane.cpu()[table[pos // 64].long(), :, pos % 64], have)
        if taps > 1:
            tail = torch.cat([torch.zeros(taps - 1, ch), rows[s][:, :ch]])[-(taps - 1):]
            assert torch.equal(state[slots[s + 1], :(taps - 1) * ch].view(taps - 1, ch).cpu(), tail)


KEPT = [(None, 0), (1, 1), (1, 0), (9, 3), (64, 64), (70, 5), (64, 65), (30, 150), (200, 20)]
PASTS = [([0, 0, 0], [5, 70, 331]),                       # fresh sequences only: nothing from the cache
         ([10, 100], [7, 30]),
         ([130, 64, 0], [70, 129, 200]),                  # past a page's and a tile's edge; a fresh one among them
         ([700, 128, 127, 129, 1, 63], [300, 1, 5, 257, 128, 2])]


def kept_case(dt, nkv, D, window, keep, before, new, spike, seed, nh):
    """A cache that holds ``before[i]`` positions of sequence i (written in steps, so that the ring turns), its next ``new[i]``
    keys, and queries.  ``spike`` = (query place from the end, key places): those keys tower over all others."""
    from moe_b200.cache import KVCache, KVRequest
    from moe_b200.ops import core

    g = torch.Generator().manual_seed(seed)
    cache = KVCache({0: KVRequest(nkv, D, window, keep=keep)}, {0: None}, max_tokens=64 * 60, max_slots=len(new), dtype=dt, device=DEV)
    cache.groups[0].storage.fill_(3e30)                   # (whatever is read but not in sight would show)
    st = core.new_status(DEV)
    slots = [cache.acquire() for _ in new]
    K = [torch.randn(a + b, nkv, D, generator=g).to(dt) for a, b in zip(before, new)]
    V = [torch.randn(a + b, nkv, D, generator=g).to(dt) for a, b in zip(before, new)]
    Q = [torch.randn(b, nh, D, generator=g).to(dt) for b in new]
    if spike is not None:
        for k, q, a, b in zip(K, Q, before, new):
            k[:, :, 0] = 0.0
            q[:, :, 0] = 5.0
            for j in spike(a + b):
                if 0 <= j < a + b:
                    k[j, :, 0] = 60.0
    for i, s in enumerate(slots):
        at = 0
        while at < before[i]:                             # pieces, as steps would bring them
            n = min(before[i] - at, 50 if window else 1000)
            G.give_pages(cache, s, at + n)
            b = G.make_batch(DEV, [s], [at], [n])
            core.kv_commit(dev(K[i][at:at + n], dt), dev(V[i][at:at + n], dt), cache.view(0), b, st)
            at += n
        G.give_pages(cache, s, before[i] + new[i])
    batch = G.make_batch(DEV, slots, before, new)
    core.check_status(st)
    return cache, batch, slots, Q, K, V, st


def kept_reference(q, k, v, a, window, keep, scale):
    n = k.shape[0]
    seen = plain.seen_mask(n, window if window else n, keep)[a:]
    group = q.shape[1] // k.shape[1]
    out = []
    for h in range(q.shape[1]):
        s = (q[:, h].double() @ k[:, h // group].double().T) * scale
        out.append(torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, h // group].double())
    return torch.stack(out, dim=1)


@pytest.mark.parametrize("window,keep", KEPT)
@pytest.mark.parametrize("dt,nh,nkv,D,kernels", [
    (torch.float32, 3, 3, 48, ("generic", "tiled")), (torch.float32, 4, 1, 128, ("tiled",)), (torch.bfloat16, 4, 2, 64, ("tc", "tiled")),
    (torch.bfloat16, 6, 3, 128, ("tc", "generic")), (torch.bfloat16, 2, 1, 160, ("tiled",))])
def test_kept_positions_beside_a_window_in_steps_of_several_tokens(dt, nh, nkv, D, kernels, window, keep):
    """Whole prompts and sequences that go on from the cache, windows and kept positions shorter and longer than a page and a
    tile; once with random keys, once with keys that tower over all others at the last query's edges: just inside and just
    outside its window, the last kept position and the one after it, the first position."""
    from moe_b200.ops import core, tc

    scale = 0.5 / math.sqrt(D)
    edges = (None,) + ((lambda n: [n - window], lambda n: [n - window - 1], lambda n: [keep - 1], lambda n: [keep], lambda n: [0])
                       if window else ())
    for i, (before, new) in enumerate(PASTS):
        for spike in edges:
            cache, batch, _, Q, K, V, st = kept_case(dt, nkv, D, window, keep, before, new, spike, 10 * i + D, nh)
            q = dev(torch.cat(Q), dt)
            kn, vn = (dev(torch.cat([t[a:] for t, a in zip(X, before)]), dt) for X in (K, V))
            kw = dict(nh=nh, window=window, keep=keep, scale=scale, status=st)
            ref = torch.cat([kept_reference(qq, k, v, a, window, keep, scale) for qq, k, v, a in zip(Q, K, V, before)])
            for kernel in kernels:
                out = torch.full(q.shape, float("nan"), dtype=dt, device=DEV)
                if kernel == "generic":
                    core.attention_generic(q, kn, vn, cache.view(0), batch, out, use_local=True, **kw)
                elif kernel == "tiled":
                    assert core.attention_tiled(q, kn, vn, cache.view(0), batch, out, use_local=True, **kw)
                else:
                    assert (tc.attention_cached(q, kn, vn, cache.view(0), batch, out, **kw) if any(before)
                            else tc.attention_prefill(q, kn, vn, batch, out, nkv=nkv, hd=D, **kw))
                core.check_status(st)
                close(out, ref, 2e-2 if dt == torch.bfloat16 else 3e-5)


@pytest.mark.parametrize("window,keep", KEPT)
@pytest.mark.parametrize("dt,nh,nkv,D", [(torch.float32, 3, 3, 64), (torch.float32, 4, 2, 48), (torch.bfloat16, 2, 2, 64),
                                         (torch.bfloat16, 9, 3, 128), (torch.bfloat16, 16, 2, 128), (torch.bfloat16, 8, 1, 64),
                                         (torch.bfloat16, 2, 1, 160)])
def test_kept_positions_beside_a_window_for_single_tokens(dt, nh, nkv, D, window, keep):
    """One new token a sequence over the cache alone, at positions around pages', windows' and kept positions' edges and far
    beyond (the ring has turned many times)."""
    from moe_b200.ops import core

    scale = 0.5 / math.sqrt(D)
    before = [0, 1, 4, 63, 64, 65, 127, 128, 150, 300, 700]
    new = [1] * len(before)
    edges = (None,) + ((lambda n: [n - window], lambda n: [n - window - 1], lambda n: [keep - 1], lambda n: [keep], lambda n: [0])
                       if window else ())
    for spike in edges:
        cache, batch, slots, Q, K, V, st = kept_case(dt, nkv, D, window, keep, before, new, spike, D, nh)
        last = [dev(torch.cat([t[-1:] for t in X]), dt) for X in (K, V)]
        core.kv_commit(last[0], last[1], cache.view(0), batch, st)
        q = dev(torch.cat(Q), dt)
        out = torch.full(q.shape, float("nan"), dtype=dt, device=DEV)
        core.attention_decode(q, cache.view(0), batch, out, nh=nh, window=window, keep=keep, scale=scale, status=st)
        core.check_status(st)
        ref = torch.cat([kept_reference(qq, k, v, a, window, keep, scale) for qq, k, v, a in zip(Q, K, V, before)])
        close(out, ref, 2e-2 if dt == torch.bfloat16 else 3e-5)


# ----------------------------------------------------------------------------- the delta rule with a decay a channel
CUTS = [[(0, 0, 10)], [(0, 10, 12), (1, 0, 2)], [(0, 12, 143), (1, 2, 9)], [(0, 143, 144), (1, 9, 10)], [(1, 10, 11), (0, 144, 145)]]
LENS = {0: 145, 1: 11}                                       # (sequence, from, to) per step; the last two bring one token each
DELTA_SIZES = [(2, 1, 8, 8, 4), (4, 2, 16, 24, 4), (3, 3, 10, 7, 3), (6, 2, 64, 64, 2), (2, 2, 128, 128, 4), (1, 1, 32, 4, 1),
               (2, 1, 200, 72, 5), (4, 4, 256, 16, 4), (2, 1, 40, 136, 4), (8, 2, 5, 3, 4)]


@pytest.mark.parametrize("spread", [0.8, 6.0])
@pytest.mark.parametrize("H,Gk,d,dv,taps", DELTA_SIZES)
def test_delta_rule_with_a_decay_a_channel_over_steps(H, Gk, d, dv, taps, spread):
    """Two sequences of unequal lengths in five steps; decays between 0 and 1, with a wide ``spread`` close to 0 and to 1 side
    by side: what the kernels prepare, the outputs behind norm and sigmoid gate, and the state."""
    from moe_b200.ops import core

    g = torch.Generator().manual_seed(H * 7 + d)
    ch = 2 * Gk * d + H * dv
    rows = {s: torch.randn(n, ch + H, generator=g) for s, n in LENS.items()}
    a_rows = {s: spread * torch.randn(n, H * d + 3, generator=g) for s, n in LENS.items()}
    gates = {s: torch.randn(n, H * dv, generator=g) for s, n in LENS.items()}
    tw = 0.4 * torch.randn(ch, taps, generator=g) + 0.3
    a_log, dt_bias = torch.randn(H, generator=g) - 1.0, torch.randn(H * d, generator=g) - 1.0
    norm_w, eps = 1 + 0.2 * torch.randn(dv, generator=g), 1e-5
    at = -(-((taps - 1) * ch) // 4) * 4
    state = torch.zeros((4, at + H * d * dv), device=DEV)
    prepared, outs = {0: [], 1: []}, {0: [], 1: []}
    for step in CUTS:
        batch = G.make_batch(DEV, [s + 1 for s, _, _ in step], [a for _, a, _ in step], [b - a for _, a, b in step])
        T = batch.num_tokens
        proj, araw, gate = (dev(torch.cat([x[s][a:b] for s, a, b in step])) for x in (rows, a_rows, gates))
        qkv, stp, decay = torch.empty((T, ch), device=DEV), torch.empty((T, 2 * H), device=DEV), torch.empty((T, H * d), device=DEV)
        sizes = dict(heads=H, kv_heads=Gk, d=d, dv=dv)
        core.delta_prepare(proj, dev(tw.t()), dev(a_log), dev(dt_bias), state, batch, qkv, stp, b_at=ch, a_at=0, eps=1e-6,
                           q_scale=d ** -0.5, a_rows=araw[:, :H * d], decay=decay, **sizes)
        if taps > 1 and not batch.all_decode:
            core.conv_state_update(proj, state, batch, taps=taps, channels=ch)
        y, nw = torch.full((T, H * dv), float("nan"), device=DEV), dev(norm_w.repeat(H))
        if not (batch.all_decode and core.delta_step(qkv, stp, state, gate, nw, eps, batch, y, offset=at, decay=decay,
                                                     gate_fn="sigmoid", **sizes)):
            o = torch.empty((T, H * dv), device=DEV)
            core.delta_scan(qkv, stp, state, batch, o, offset=at, decay=decay, **sizes)
            core.wkv_finish(o, gate, nw, eps, batch, y, heads=H, d=dv, gate_fn="sigmoid")
        i = 0
        for s, a, b in step:
            prepared[s].append((qkv[i:i + b - a].cpu(), stp[i:i + b - a, :H].cpu(), decay[i:i + b - a].cpu()))
            outs[s].append(y[i:i + b - a].cpu())
            i += b - a
    owner = torch.arange(H) // (H // Gk)
    for s, n in LENS.items():
        y = plain.silu(plain.causal_taps(rows[s][:, :ch].double(), tw.double()))
        q = plain.unit_length(y[:, :Gk * d].reshape(n, Gk, d)) / math.sqrt(d)
        k = plain.unit_length(y[:, Gk * d:2 * Gk * d].reshape(n, Gk, d))
        v = y[:, 2 * Gk * d:].reshape(n, H, dv)
        beta = torch.sigmoid(rows[s][:, ch:].double())
        decay = torch.exp(-torch.exp(a_log.double())[None, :, None]
                          * plain.softplus(a_rows[s][:, :H * d].double() + dt_bias.double()).reshape(n, H, d))
        qkv, b, dc = (torch.cat([p[j] for p in prepared[s]]) for j in range(3))
        close(qkv, torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], dim=1), 1e-5)
        close(b, beta, 1e-6), close(dc, decay.reshape(n, -1), 1e-5)
        o, S = plain.channel_delta_recurrence(q[:, owner], k[:, owner], v, decay, beta)
        ref = (plain.unit_rms(o, eps) * norm_w.double()).reshape(n, -1) * torch.sigmoid(gates[s].double())
        close(torch.cat(outs[s]), ref, 3e-4)
        close(state[s + 1, at:].view(H, d, dv), S, 3e-5)
    assert float(state[0].abs().max()) == 0.0 and float(state[3].abs().max()) == 0.0


def test_each_channel_forgets_at_its_own_pace():
    """Two keys along channels of their own, one whose decay is 1 and one whose decay is 0.5: hundreds of tokens later the
    first value is there unchanged, and the second one is gone (after a few tokens: by the factor that is due)."""
    from moe_b200.ops import core

    d, dv, T = 8, 4, 300
    g = torch.Generator().manual_seed(3)
    k = torch.zeros(T, d)
    k[0, 1] = k[1, 2] = 1.0
    q = torch.zeros(T, d)
    q[:, 1] = 1.0
    q[10, 1], q[10, 2] = 0.0, 1.0
    v = torch.randn(T, dv, generator=g)
    beta = torch.zeros(T, 2)
    beta[:2, 0] = 1.0
    decay = torch.ones(T, d)
    decay[:, 2] = 0.5
    state = torch.zeros((2, d * dv), device=DEV)
    o = torch.empty((T, dv), device=DEV)
    core.delta_scan(dev(torch.cat([q, k, v], dim=1)), dev(beta), state, G.make_batch(DEV, [1], [0], [T]), o, heads=1, kv_heads=1,
                    d=d, dv=dv, decay=dev(decay))
    ref = v[0].expand(T, dv).clone()
    ref[10] = v[1] * 0.5 ** 9
    close(o, ref, 1e-6)
    held = state[1].view(d, dv).cpu()
    close(held[1], v[0], 1e-6)
    assert float(held[2].abs().max()) < 1e-30


# ----------------------------------------------------------------------------- the exponentially gated memory
MEMORY_SIZES = [(2, 8, 8, 12.0), (4, 16, 24, 5.0), (3, 10, 7, 1.0), (6, 64, 64, 15.0), (2, 128, 128, 12.0), (1, 1, 1, 8.0), (2, 200, 72, 12.0),
                (4, 256, 16, 30.0), (1, 40, 136, 12.0), (8, 5, 3, 20.0), (5, 32, 100, 9.0)]


@pytest.mark.parametrize("H,d,dv,cap", MEMORY_SIZES)
@pytest.mark.parametrize("gain", [1.0, 20.0])
def test_exponentially_gated_memory_over_steps(H, d, dv, cap, gain):
    """Two sequences of unequal lengths in five steps, gates' logits small and far beyond their cap (so that inputs arrive
    with factors from e^-cap to e^cap and the running maximum jumps): outputs behind norm and gate, and the state."""
    from moe_b200.ops import core

    g = torch.Generator().manual_seed(H * 7 + d)
    at = {"v": 0, "q": H * dv, "i": H * (dv + d), "f": H * (dv + d + 1), "k": H * (dv + d + 2)}
    if (H * dv) % 4 == 0 and H % 2 == 0 and d % 4 == 0:              # (rows and columns of whole 16-byte units in some cases)
        at = {"v": 0, "q": H * dv, "k": H * (dv + d), "i": H * (dv + 2 * d), "f": H * (dv + 2 * d + 1)}
    width = -(-(H * (dv + 2 * d + 2)) // 4) * 4
    rows = {s: torch.randn(n, width, generator=g) for s, n in LENS.items()}
    gates = {s: torch.randn(n, H * dv, generator=g) for s, n in LENS.items()}
    for x in rows.values():
        x[:, at["i"]:at["i"] + H] *= gain
        x[:, at["f"]:at["f"] + H] = gain * x[:, at["f"]:at["f"] + H] + 2.0
    ib, fb = torch.randn(H, generator=g), torch.randn(H, generator=g)
    norm_w, eps = 1 + 0.2 * torch.randn(H * dv, generator=g), 1e-5
    size = core.mlstm_state_floats(H, d, dv)
    assert size == core.lib().moe_mlstm_state_floats(H, d, dv)
    off = 8
    state = torch.zeros((4, off + -(-size // 4) * 4), device=DEV)
    outs = {0: [], 1: []}
    for step in CUTS:
        batch = G.make_batch(DEV, [s + 1 for s, _, _ in step], [a for _, a, _ in step], [b - a for _, a, b in step])
        T = batch.num_tokens
        proj, gate = (dev(torch.cat([x[s][a:b] for s, a, b in step])) for x in (rows, gates))
        y = torch.full((T, H * dv), float("nan"), device=DEV)
        args = (proj, at, dev(ib), dev(fb), cap, d ** -0.5, state)
        sizes = dict(heads=H, d=d, dv=dv, offset=off)
        if not (batch.all_decode and core.mlstm_step(*args, gate, dev(norm_w), eps, batch, y, **sizes)):
            o = torch.empty((T, H * dv), device=DEV)
            core.mlstm_scan(*args, batch, o, **sizes)
            core.wkv_finish(o, gate, dev(norm_w), eps, batch, y, heads=H, d=dv, gate_fn="sigmoid")
        i = 0
        for s, a, b in step:
            outs[s].append(y[i:i + b - a].cpu())
            i += b - a
    for s, n in LENS.items():
        part = lambda c, w: rows[s][:, at[c]:at[c] + H * w].double().reshape(n, H, w)
        capped = lambda c, b: cap * torch.tanh((part(c, 1)[..., 0] + b.double()) / cap)
        o, S, z, mu = plain.memory_recurrence(part("q", d) / math.sqrt(d), part("k", d), part("v", dv), capped("i", ib),
                                              -plain.softplus(-capped("f", fb)))
        ref = plain.unit_rms(o, eps).reshape(n, -1) * norm_w.double() * torch.sigmoid(gates[s].double())
        close(torch.cat(outs[s]), ref, 1e-3)
        have = state[s + 1, off:].double().cpu()
        copies = -(-dv // 16)
        m = have[H * d * (dv + copies):H * d * (dv + copies) + H]
        close(m, mu, 1e-5)
        close(have[:H * d * dv].view(H, d, dv) * torch.exp(m - mu)[:, None, None], S, 1e-4)
        for c in range(copies):
            close(have[H * d * (dv + c):H * d * (dv + c + 1)].view(H, d) * torch.exp(m - mu)[:, None], z, 1e-4)
    assert float(state[0].abs().max()) == 0.0 and float(state[3].abs().max()) == 0.0


@pytest.mark.parametrize("segments", [2, 3, 8])
@pytest.mark.parametrize("H,d,dv", [(4, 16, 24), (2, 96, 64), (3, 10, 7), (1, 200, 40)])
def test_memory_in_segments_that_run_side_by_side(H, d, dv, segments):
    """Three sequences of unequal lengths (one so short that it lies in the first segment) that go on from a state, cut into
    segments: outputs and state as in one go."""
    from moe_b200.ops import core

    g = torch.Generator().manual_seed(H * 7 + d)
    width = -(-(H * (dv + 2 * d + 2)) // 4) * 4
    at = {"q": 0, "k": H * d, "v": 2 * H * d, "i": H * (2 * d + dv), "f": H * (2 * d + dv + 1)}
    counts = [403, 9, 260]
    proj = torch.randn(sum(counts), width, generator=g)
    proj[:, at["i"]:at["i"] + 2 * H] *= 4.0
    size = -(-core.mlstm_state_floats(H, d, dv) // 4) * 4
    ib, fb = torch.randn(H, generator=g), torch.randn(H, generator=g) + 1.0
    batch = G.make_batch(DEV, [1, 2, 3], [0, 0, 0], counts)
    res = []
    for n in (1, segments):
        state = torch.zeros((5, size), device=DEV)
        for _ in range(2):                                   # (the second time from what the first left)
            o = torch.empty((sum(counts), H * dv), device=DEV)
            core.mlstm_scan(dev(proj), at, dev(ib), dev(fb), 6.0, d ** -0.5, state, batch, o, heads=H, d=d, dv=dv, segments=n)
        res.append((o.double().cpu(), state.double().cpu()))
    scale = float(res[0][0].abs().max())
    assert float((res[0][0] - res[1][0]).abs().max()) < 2e-4 * scale
    assert float((res[0][1] - res[1][1]).abs().max()) < 2e-4 * float(res[0][1].abs().max())
    assert float(res[1][1][0].abs().max()) == float(res[1][1][4].abs().max()) == 0.0


def test_a_strong_input_is_remembered_and_a_weak_one_after_it_is_not():
    """An input gate at its cap once, near minus its cap afterwards, and forget gates near 1: hundreds of tokens later the
    read-out is the strong token's value; before it, the running maximum of 0 bounds the read-out."""
    from moe_b200.ops import core

    T, d, dv, cap = 400, 4, 8, 12.0
    g = torch.Generator().manual_seed(2)
    k, v = torch.randn(T, d, generator=g), torch.randn(T, dv, generator=g)
    q = torch.ones(T, d)
    k[7] = 1.0
    i = torch.full((T, 1), -40.0)
    i[7] = 80.0
    f = torch.full((T, 1), 60.0)
    proj = torch.cat([q, k, v, i, f, torch.zeros(T, 2)], dim=1)
    at = {"q": 0, "k": d, "v": 2 * d, "i": 2 * d + dv, "f": 2 * d + dv + 1}
    state = torch.zeros((2, core.mlstm_state_floats(1, d, dv) + 3), device=DEV)
    o = torch.empty((T, dv), device=DEV)
    core.mlstm_scan(dev(proj), at, dev(torch.zeros(1)), dev(torch.zeros(1)), cap, d ** -0.5, state, G.make_batch(DEV, [1], [0], [T]), o,
                    heads=1, d=d, dv=dv)
    ref = plain.memory_recurrence(q.double()[:, None] / 2.0, k.double()[:, None], v.double()[:, None], cap * torch.tanh(i.double() / cap),
                                  -plain.softplus(-cap * torch.tanh(f.double() / cap)))[0][:, 0]
    close(o, ref, 1e-5)
    close(o[300], v[7], 1e-2)
    assert float(o[:7].abs().max()) < 1e-2


# ----------------------------------------------------------------------------- experts that read a weighted input
@pytest.mark.parametrize("T", [1, 5, 20, 70, 300])
@pytest.mark.parametrize("W,E,top,ff", [(64, 5, 2, 40), (52, 3, 3, 18), (40, 1, 1, 16), (128, 12, 4, 64), (96, 7, 1, 24)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_sigmoid_scores_multiply_what_the_experts_read(T, W, E, top, ff, dtype):
    from moe_b200.config.spec import PartSpec
    from moe_b200.parts.base import Activations, Runtime, make_part

    g = torch.Generator().manual_seed(T + W)
    rt = Runtime(DEV, getattr(torch, dtype))
    part = make_part("ffn", PartSpec("routed_experts", {
        "hidden_size": W, "num_experts": E, "top_k": top, "expert_size": ff, "score": "sigmoid", "weight_input": True,
        "names": {"router": "router", "expert_gate": "e{e}.gate", "expert_up": "e{e}.up", "expert_down": "e{e}.down"}}))
    w = {n: (1.5 * torch.randn(ts.shape, generator=g) / math.sqrt(ts.shape[1])).to(torch.bfloat16) for n, ts in part.tensors().items()}
    part.bind({n: t.to(rt.compute_dtype).to(DEV) for n, t in w.items()}, rt)
    assert part.wants32 and not part.wants16
    x = torch.randn(T, W, generator=g)
    batch = G.make_batch(DEV, [0], [0], [T])
    part.trace = []
    got = part.forward(rt, Activations(act=dev(x, rt.compute_dtype), f32=dev(x)), batch)
    rt.check()
    idx, weight = part.trace[0]
    w64 = {"f." + n: t.double() for n, t in w.items()}
    score = torch.sigmoid(x.double() @ w64["f.router"].T)
    picks = torch.topk(score, top, dim=-1).indices
    assert torch.equal(idx.long().cpu().sort(-1).values, picks.sort(-1).values)
    close(weight, torch.gather(score, 1, idx.long().cpu()), 1e-5)
    close(got, plain.experts_ff(w64, "f", {"router": {"experts": E, "top": top}}, x.double()), 2e-2 if dtype == "bfloat16" else 1e-5)


@pytest.mark.parametrize("T", [1, 3, 8])
@pytest.mark.parametrize("W,E,top", [(64, 5, 2), (48, 3, 3), (2048, 16, 2), (136, 1, 1), (4096, 40, 8)])
@pytest.mark.parametrize("two", [False, True])
def test_few_tokens_norm_sum_router_and_weighted_rows_in_one_launch(T, W, E, top, two):
    """x += rms(y) w, scores, picks, the experts' order and the rows they read, against the plain formulas; a row of no
    sequence gets no expert."""
    from moe_b200.ops import core

    g = torch.Generator().manual_seed(W + T)
    x, a, b = (torch.randn(T, W, generator=g) for _ in range(3))
    pw, eps = 0.5 * (1 + 0.3 * torch.randn(W, generator=g)), 1e-5
    wr = (2 * torch.randn(E, W, generator=g) / math.sqrt(W)).to(torch.bfloat16)
    seq = torch.zeros(T, dtype=torch.int32)
    if T > 1:
        seq[1] = -1
    xs_, st = dev(x), core.new_status(DEV)
    kw = dict(sa=0.7, delta_b=dev(b), sb=-0.4) if two else {}
    got = core.norm_route(xs_, dev(a), None, 0.0, wr.to(DEV), top, False, 1.0, bf16=True, seq_of_token=seq.to(DEV), status=st,
                          score="sigmoid", post=(dev(pw), eps), weight_input=True, **kw)
    core.check_status(st)
    o32, o16, idx, wt, _, offsets, sorted_token, place, rows = got
    assert o32 is None and o16 is None
    y = 0.7 * a.double() - 0.4 * b.double() if two else a.double()
    new = x.double() + plain.unit_rms(y, eps) * pw.double()
    close(xs_, new, 5e-6)
    score = torch.sigmoid(new @ wr.double().T)
    live = [t for t in range(T) if seq[t] >= 0]
    idx, wt, place, rows = idx.long().cpu(), wt.double().cpu(), place.view(T, top).cpu(), rows.double().cpu()
    for t in range(T):
        if t not in live:
            assert idx[t].tolist() == [-1] * top and place[t].tolist() == [-1] * top
            continue
        best = torch.topk(score[t], top).indices
        assert sorted(idx[t].tolist()) == sorted(best.tolist())
        close(wt[t], score[t, idx[t]], 1e-5)
        for j in range(top):
            p = int(place[t, j])
            assert int(offsets[idx[t, j]]) <= p < int(offsets[idx[t, j] + 1]) and int(sorted_token[p]) == t
            close(rows[p], score[t, idx[t, j]] * new[t], 1e-2)
    assert int(offsets[E]) == len(live) * top


def test_scores_of_large_logits_stay_finite():
    from moe_b200.ops import core

    logits = torch.tensor([[200.0, -200.0, 0.0, 3.0]])
    idx, wt = torch.empty((1, 4), dtype=torch.int32, device=DEV), torch.empty((1, 4), device=DEV)
    core.router_topk(dev(logits), 4, False, 1.0, idx, wt, num_experts=4, score="sigmoid")
    assert idx.cpu().tolist() == [[0, 3, 2, 1]]
    close(wt, torch.sigmoid(logits.double())[:, [0, 3, 2, 1]], 1e-6)


# ----------------------------------------------------------------------------- the model, layer by layer
@pytest.mark.parametrize("name", NAMES)
def test_every_layer_of_a_whole_prompt_in_32_bit(root, name):
    d, eng = engine_of(root, name, "float32", use_graphs=False)
    cfg, w = model_of(d)
    toks = U.tokens(cfg["vocab"], 150, 3)
    ref_layers = []
    plain.forward(cfg, w, toks, ref_layers)
    eng.model.stream_tap = []
    s = eng.new_sequence()
    try:
        eng.step([s], [toks], [[len(toks) - 1]])
        taps = [t.double().cpu() for t in eng.model.stream_tap]
    finally:
        eng.model.stream_tap = None
        eng.release(s)
    assert len(taps) == len(ref_layers)
    for i, (have, ref) in enumerate(zip(taps, ref_layers)):
        err = float((have - ref).abs().max()) / float(ref.abs().max())
        assert err < 5e-5, f"layer {i}: {err:.3g}"


# ----------------------------------------------------------------------------- whole prompts, decoding, portions
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_of_many_lengths(root, name, dtype):
    d, eng = engine_of(root, name, dtype)
    cfg, _ = model_of(d)
    requests = {f"r{n}": U.tokens(cfg["vocab"], n, n) for n in (1, 2, 3, 63, 64, 65, 131, 200)}
    check_schedule(d, eng, requests, helpers.whole_schedule(requests), G.tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_decoding_from_the_first_token_on_and_a_prompt_against_its_replay(root, name, dtype):
    """Token by token from position 0 for 150 tokens (windows and pages pass by, rings wrap), and a prompt
    whose tail is decoded, against the plain implementation and against the whole prompt."""
    d, eng = engine_of(root, name, dtype)
    cfg, _ = model_of(d)
    toks = U.tokens(cfg["vocab"], 150, 5)
    tol = G.tol(dtype)
    one = check_schedule(d, eng, {"a": toks}, helpers.tail_schedule({"a": toks}, tail=149), tol)["a"]
    tail = check_schedule(d, eng, {"a": toks}, helpers.tail_schedule({"a": toks}, tail=40), tol)["a"]
    whole = check_schedule(d, eng, {"a": toks}, helpers.whole_schedule({"a": toks}), tol)["a"]
    scale = float(torch.stack(list(whole.values())).abs().max())
    bound = allowed(d, toks, G.tol_cut(dtype))
    for pos in whole:
        for other in (one, tail):
            assert float((other[pos] - whole[pos]).abs().max()) / scale < float(bound[pos]), pos


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "ones", "wide", "lean"])
@pytest.mark.parametrize("sizes", [[2], [3], [63, 2], [64], [65, 1, 1, 7], [129]])
def test_portions_of_several_sizes(root, name, dtype, sizes):
    d, eng = engine_of(root, name, dtype)
    cfg, _ = model_of(d)
    toks = U.tokens(cfg["vocab"], 140 if sizes[0] > 3 else 41, 9)
    check_schedule(d, eng, {"a": toks}, portions_schedule("a", toks, sizes), G.tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "lean", "wide", "large"])
def test_unequal_requests_batched_against_each_alone_on_slots_used_again(root, name, dtype):
    """Seven requests of unequal lengths on three slots, twice over (so that slots, pages and state are
    used again), batches of three decoded together; then every request alone."""
    d, eng = engine_of(root, name, dtype, max_slots=3)
    cfg, _ = model_of(d)
    lens = [70, 5, 131, 1, 64, 33, 90]
    requests = {f"q{i}": U.tokens(cfg["vocab"], n, 20 + i) for i, n in enumerate(lens)}
    tol = G.tol(dtype)
    for _ in range(2):
        together = check_schedule(d, eng, requests, helpers.batches_schedule(requests, 3, lambda r: max(1, len(requests[r]) - 12)), tol)
    alone = check_schedule(d, eng, requests, helpers.whole_schedule(requests), tol)
    for rid in requests:
        scale = float(torch.stack(list(alone[rid].values())).abs().max())
        bound = allowed(d, requests[rid], G.tol_cut(dtype))
        for pos in together[rid]:
            assert float((together[rid][pos] - alone[rid][pos]).abs().max()) / scale < float(bound[pos]), (rid, pos)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "wide"])
def test_portions_that_go_on_from_different_places_in_one_step(root, name, dtype):
    d, eng = engine_of(root, name, dtype)
    cfg, _ = model_of(d)
    a, b, c = (U.tokens(cfg["vocab"], n, 40 + n) for n in (120, 75, 30))
    steps = [
        {"entries": [("a", a[:50], list(range(50)))], "end": []},
        {"entries": [("a", a[50:52], [0, 1]), ("b", b[:64], list(range(64)))], "end": []},
        {"entries": [("a", a[52:119], list(range(67))), ("b", b[64:75], list(range(11))), ("c", c, list(range(30)))], "end": ["b", "c"]},
        {"entries": [("a", a[119:], [0])], "end": ["a"]},
    ]
    check_schedule(d, eng, {"a": a, "b": b, "c": c}, steps, G.tol(dtype))


# ----------------------------------------------------------------------------- edges that random weights would hide
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("place", [0, 3, 63, 64, 400])
def test_a_far_key_among_hundreds(root, dtype, place):
    """A token whose key every query looks at, 140 to 540 positions back, at a page's border or not (or the very
    first): whole, and with the last 40 tokens decoded.  The plain result changes by much when that token is
    replaced, so a key that is lost shows."""
    d, eng = engine_of(root, "far", dtype, edit_weights=U.spike_token)
    cfg, w = model_of(d)
    special = 0                      # (the token that spike_token marks)
    toks = [1 + t % (cfg["vocab"] - 1) for t in U.tokens(cfg["vocab"], 545, 77)]
    toks[place] = special
    ref = reference(d, toks)
    other = list(toks)
    other[place] = 1
    moved = float((plain.forward(cfg, w, other)[-1] - ref[-1]).abs().max()) / float(ref.abs().max())
    assert moved > 0.1, moved        # the test's premise: the far key matters
    check_schedule(d, eng, {"a": toks}, helpers.whole_schedule({"a": toks}), G.tol(dtype))
    check_schedule(d, eng, {"a": toks}, helpers.tail_schedule({"a": toks}, tail=40), G.tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep", [(1, 3), (7, 1), (7, 64), (64, 65), (65, 63), (130, 2), (30, 0)])
def test_windows_and_kept_positions_one_longer_or_shorter(root, dtype, size, keep):
    """The same weights with another window and another number of kept positions: a key just inside the window (or the
    last kept one) of one model is just outside (not kept) in the next, in prompts, portions and decoding; by how much
    the logits move is what the plain implementation says, and it is more than the tolerance."""
    def edit(cfg):
        for L in cfg["layers"]:
            L["mixer"]["left"]["mask"] = {"size": size, "keep_first": keep}
    edit.__name__ = f"window{size}keep{keep}"
    d, eng = engine_of(root, "sharp", dtype, edit=edit)
    cfg, w = model_of(d)
    toks = U.tokens(cfg["vocab"], 200, size)
    ref = reference(d, toks)
    for more in ({"size": size + 1, "keep_first": keep}, {"size": size, "keep_first": keep + 1}):
        other = json.loads(json.dumps(cfg))
        for L in other["layers"]:
            L["mixer"]["left"]["mask"] = more
        moved = (plain.forward(other, w, toks) - ref).abs().amax(dim=1) / float(ref.abs().max())
        assert float(moved.max()) > 0.05
    tol = G.tol(dtype)
    check_schedule(d, eng, {"a": toks}, helpers.whole_schedule({"a": toks}), tol)
    check_schedule(d, eng, {"a": toks}, helpers.tail_schedule({"a": toks}, tail=70), tol)
    check_schedule(d, eng, {"a": toks}, portions_schedule("a", toks, [size + 1, 2, 61]), tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("place,seen", [(4, True), (5, False), (189, True), (188, False)])
def test_a_towering_key_at_the_edges_of_window_and_kept_positions(root, dtype, place, seen):
    """One window of 12 and five kept positions, the last query at position 200: the token that every query looks at stands
    at the last kept position, one behind it, at the window's last place, and one before it.  Whole, and decoded."""
    def edit(cfg):
        cfg["layers"][0]["mixer"]["left"]["mask"] = {"size": 12, "keep_first": 5}
        cfg["layers"][0]["mixer"]["left"]["conv"] = 1
    edit.__name__ = "edges"
    d, eng = engine_of(root, "far", dtype, edit=edit, edit_weights=U.spike_token)
    cfg, w = model_of(d)
    toks = [1 + t % (cfg["vocab"] - 1) for t in U.tokens(cfg["vocab"], 201, 5)]
    plainly = list(toks)
    toks[place] = 0
    cfg2 = json.loads(json.dumps(cfg))
    cfg2["layers"][0]["mixer"]["right_scale"] = 0.0                  # (the memory beside the attention sees every token)
    a, b = plain.forward(cfg2, w, toks)[-1], plain.forward(cfg2, w, plainly)[-1]
    moved = float((a - b).abs().max()) / float(b.abs().max())
    assert moved > 0.1 if seen else moved < 1e-9, moved              # the test's premise
    check_schedule(d, eng, {"a": toks}, helpers.whole_schedule({"a": toks}), G.tol(dtype))
    check_schedule(d, eng, {"a": toks}, helpers.tail_schedule({"a": toks}, tail=60), G.tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
def test_kept_pages_of_a_released_sequence_serve_the_next_one(root, dtype):
    """Pages go back and come again in another order: a long sequence, released, then two on the same pages; the cache holds
    the pinned pages and the ring, and no more."""
    d, eng = engine_of(root, "sharp", dtype, max_slots=2)
    cfg, _ = model_of(d)
    a, b, c = (U.tokens(cfg["vocab"], n, n) for n in (300, 210, 90))
    for _ in range(2):
        check_schedule(d, eng, {"a": a}, portions_schedule("a", a, [100, 57, 1, 80]), G.tol(dtype))
        check_schedule(d, eng, {"b": b, "c": c}, helpers.batches_schedule({"b": b, "c": c}, 2, lambda r: 60), G.tol(dtype))
    widths = sorted((g.pinned, g.ring) for g in eng.cache.groups)
    assert widths == [(64, 64), (64, 192)]
    s = eng.new_sequence()
    eng.step([s], [a])
    assert [len(gl.pages[s]) for gl in eng.cache.ledger.groups] == [min(5, g.ring_pages) for g in eng.cache.groups]
    eng.release(s)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "memory"])
def test_long_decoding(root, name, dtype):
    d, eng = engine_of(root, name, dtype)
    cfg, _ = model_of(d)
    toks = U.tokens(cfg["vocab"], 420, 13)
    steps = [{"entries": [("a", toks[:20], [19])], "end": []}]
    steps += [{"entries": [("a", [toks[i]], [0] if i % 7 == 0 or i > 400 else [])], "end": ["a"] if i == 419 else []}
              for i in range(20, 420)]
    check_schedule(d, eng, {"a": toks}, steps, G.tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "memory"])
def test_long_prompts_whole_and_in_pieces(root, name, dtype):
    """Prompts longer than the padded graphs take, one alone and two together, and in pieces that go on."""
    d, eng = engine_of(root, name, dtype)
    cfg, _ = model_of(d)
    a, b = U.tokens(cfg["vocab"], 900, 1), U.tokens(cfg["vocab"], 610, 2)
    tol = G.tol(dtype)
    check_schedule(d, eng, {"a": a}, [{"entries": [("a", a, list(range(0, 900, 7)) + [899])], "end": ["a"]}], tol)
    check_schedule(d, eng, {"a": a, "b": b}, [
        {"entries": [("a", a, [0, 511, 899]), ("b", b[:600], [0, 63, 599])], "end": ["a"]},
        {"entries": [("b", b[600:], list(range(10)))], "end": ["b"]}], tol)
    check_schedule(d, eng, {"a": a}, [
        {"entries": [("a", a[:130], [129])], "end": []}, {"entries": [("a", a[130:860], [0, 1, 600, 729])], "end": []},
        {"entries": [("a", a[860:], list(range(40)))], "end": ["a"]}], tol)


# ----------------------------------------------------------------------------- through the library's own entry points
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "lean", "wide"])
def test_greedy_generation_through_the_entry_point(root, name, dtype):
    import moe_b200

    d, eng = engine_of(root, name, dtype)
    cfg, w = model_of(d)
    prompts = [U.tokens(cfg["vocab"], n, 60 + n) for n in (9, 1, 70, 33)]
    outs = moe_b200.generate(eng, prompts, max_tokens=12, eos=())
    for p, o in zip(prompts, outs):
        assert len(o.tokens) == 12
        ref = plain.forward(cfg, w, p + o.tokens)[len(p) - 1:-1]
        margin = (2e-4 if dtype == "float32" else 6e-2) * float(ref.abs().max())
        for j, tok in enumerate(o.tokens):
            assert float(ref[j, tok]) >= float(ref[j].max()) - margin, (dtype, j, tok)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_trace_program_replays_a_mixed_schedule(root, dtype, tmp_path):
    import numpy as np

    d = U.model_folder(root, "mix")
    cfg, w = model_of(d)
    a, b = U.tokens(cfg["vocab"], 80, 1), U.tokens(cfg["vocab"], 30, 2)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": [0, 69]}, {"id": "b", "tokens": b[:25], "want": [24]}], "end": []}]
    for i in range(5):
        lines.append({"step": 1 + i, "entries": [{"id": "a", "tokens": [a[70 + i]], "want": [0]}, {"id": "b", "tokens": [b[25 + i]], "want": [0]}],
                      "end": ["b"] if i == 4 else []})
    lines.append({"step": 6, "entries": [{"id": "a", "tokens": a[75:], "want": [4]}], "end": ["a"]})
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "256"], input="\n".join(json.dumps(x) for x in lines) + "\n", capture_output=True, text=True,
                       timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(7)]
    ra, rb = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    got0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(3, -1).copy()).double()
    got6 = torch.from_numpy(np.fromfile(out / "6.f32", dtype="<f4").reshape(1, -1).copy()).double()
    bound = (G.tol(dtype) + (4 * float(sensitivity(d, a).max()) if dtype == "bfloat16" else 0.0)) * float(ra.abs().max())
    assert float((got0 - torch.stack([ra[0], ra[69], rb[24]])).abs().max()) < bound
    assert float((got6[0] - ra[79]).abs().max()) < bound


def test_the_command_line_generates_and_the_summary_names_the_design_s_parts(root):
    import moe_b200

    d = U.model_folder(root, "mix")
    env = dict(os.environ, PYTHONPATH=ROOT)
    run = lambda *a: subprocess.run([sys.executable, os.path.join(ROOT, "bin", "moe"), *a], capture_output=True, text=True,
                                    env=env, timeout=900)
    r = run("run", d, "--ids", "5,17,3,9", "-n", "6", "--no-stream", "--dtype", "float32")
    assert r.returncode == 0, r.stderr[-2000:]
    toks = json.loads(r.stdout.strip().splitlines()[-1])
    _, eng = engine_of(root, "mix", "float32")
    assert moe_b200.generate(eng, [[5, 17, 3, 9]], max_tokens=6)[0].tokens == toks
    r = run("info", d)
    assert r.returncode == 0, r.stderr[-2000:]
    for word in ("Kulanex", "gated delta rule with a decay a channel", "mLSTM", "window 24 and the first 5", "values are the convolved keys",
                 "sigmoid gate, weights on the input", "no norm"):
        assert word in r.stdout, word
