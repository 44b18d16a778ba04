"""Ditazen on the GPU against the plain implementation (tests/plain_ditazen.py): every mechanism
alone, whole prompts, decoding through cache and state, portions of prompts, unequal batches, slots,
pages and state used again, windows' and pages' edges, far keys, the first tokens, long decoding,
greedy generation and the trace program.  Configurations and weights are the tests' own
(tests/ditazen_util.py)."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import ditazen_util as U
import gpu_util as G
import helpers
import plain_ditazen as plain

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
NAMES = ["mix", "lean", "ones", "sharp", "wide", "large", "huge", "memory"]
F = torch.float64


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return tmp_path_factory.mktemp("ditazen")


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


# ----------------------------------------------------------------------------- the norm and the feed-forward
@pytest.mark.parametrize("W", [1, 30, 64, 320, 516, 1030, 2048, 5000, 8192, 9000])
@pytest.mark.parametrize("with_delta,with_bias", [(False, False), (True, False), (True, True)])
def test_layer_norm_with_the_residual_sum(W, with_delta, with_bias):
    """Rows with a mean far from zero (a variance formed as a difference of squares would lose it)."""
    from moe_b200.ops import core

    g = torch.Generator().manual_seed(W)
    T, eps = 7, 1e-5
    x = torch.randn(T, W, generator=g) + 200.0 * torch.randn(T, 1, generator=g)
    delta = torch.randn(T, W, generator=g) if with_delta else None
    w, b = 1 + 0.3 * torch.randn(W, generator=g), torch.randn(W, generator=g)
    xs = dev(x)
    o32, o16 = torch.empty((T, W), device=DEV), torch.empty((T, W), dtype=torch.bfloat16, device=DEV)
    st = core.new_status(DEV)
    core.layernorm(xs, dev(w), eps, bias=dev(b) if with_bias else None, delta=dev(delta) if with_delta else None, out32=o32,
                   out16=o16, status=st)
    s = (x + delta if with_delta else x)
    assert torch.equal(xs.cpu(), s)                                     # the sum is what the stream holds afterwards
    ref = plain.layer_norm(s.double(), w.double(), eps) + (b.double() if with_bias else 0.0)
    close(o32, ref, 1e-4)
    close(o16, ref, 1e-2)
    rows = torch.tensor([5, 0, 5], dtype=torch.int32, device=DEV)
    picked = torch.empty((3, W), device=DEV)
    xs = dev(x)
    core.layernorm(xs, dev(w), eps, bias=dev(b) if with_bias else None, delta=dev(delta) if with_delta else None, rows=rows,
                   out32=picked, status=st)
    assert torch.equal(xs.cpu(), x)                                     # with chosen rows the stream stays
    close(picked, ref[[5, 0, 5]], 1e-4)
    core.check_status(st)


@pytest.mark.parametrize("M,N,K", [(3, 40, 24), (70, 136, 64), (300, 256, 320)])
def test_exact_gelu_alone_and_in_the_tensor_core_product(M, N, K):
    from moe_b200.ops import core, tc

    g = torch.Generator().manual_seed(M)
    z = 3 * torch.randn(M, N, generator=g)
    for dt, tol in ((torch.float32, 1e-6), (torch.bfloat16, 4e-3)):
        out = torch.empty((M, N), dtype=dt, device=DEV)
        core.plain_act(dev(z), out, "gelu")
        close(out, plain.gelu(z.double()), tol)
    a, w = torch.randn(M, K, generator=g).to(torch.bfloat16), (2 * torch.randn(N, K, generator=g) / math.sqrt(K)).to(torch.bfloat16)
    out = torch.empty((M, N), dtype=torch.bfloat16, device=DEV)
    assert tc.gemm_tc(a.to(DEV), w.to(DEV), out, act="gelu", status=core.new_status(DEV))
    close(out, plain.gelu(a.double() @ w.double().T), 6e-3)


# ----------------------------------------------------------------------------- latent attention's own kernels
@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("neighbours", [False, True])
@pytest.mark.parametrize("H,d,rot,r,D", [(3, 24, 8, 40, 48), (1, 8, 2, 5, 16), (5, 64, 64, 64, 128), (2, 10, 6, 20, 32), (4, 32, 16, 112, 128),
                                         (16, 96, 32, 96, 128)])
@pytest.mark.parametrize("starts,counts,qr", [([0, 3990], [9, 4], 20), ([0, 3400], [9, 600], 52), ([3, 64], [1, 520], 1100)])
def test_latent_records_and_queries_are_normed_rotated_and_laid_out(bf16, neighbours, H, d, rot, r, D, starts, counts, qr):
    """Few and many tokens, both layouts of the queries, both pairings of the rotation, positions into the thousands, a factor on
    cos and sin, the queries' own latent, and the append to the paged cache."""
    from moe_b200.cache import KVCache, KVRequest
    from moe_b200.ops import core

    g = torch.Generator().manual_seed(H * 100 + r)
    eps = 1e-5
    dt = torch.bfloat16 if bf16 else torch.float32
    scaling = {"factor": 4.0, "original": 512, "fast": 16.0, "slow": 1.0}
    freq, mscale = plain.frequencies({"dims": rot, "base": 5000.0, "scaling": scaling})
    T = sum(counts)
    pos = torch.cat([torch.arange(a, a + n) for a, n in zip(starts, counts)])
    proj = 3 * torch.randn(T, qr + r + rot + 3, generator=g)
    q32 = 3 * torch.randn(T, H * (d + rot), generator=g)
    rec32 = 3 * torch.randn(T, H * (r + rot), generator=g)
    wn, cw = 1 + 0.3 * torch.randn(r, generator=g), 1 + 0.3 * torch.randn(qr, generator=g)
    cache = KVCache({0: KVRequest(1, D, None, values_are_keys=True)}, {0: None}, max_tokens=64 * 70, max_slots=2, dtype=dt, device=DEV)
    slots = [cache.acquire() for _ in range(2)]
    for s, a, n in zip(slots, starts, counts):
        G.give_pages(cache, s, a + n)
    batch = G.make_batch(DEV, slots, starts, counts)
    st = core.new_status(DEV)
    turn = dict(rot=rot, freq=dev(freq), interleaved=neighbours, mscale=mscale)
    k_new = torch.full((T, 1, D), 7.0, dtype=dt, device=DEV)
    cq = torch.full((T, qr), 7.0, dtype=dt, device=DEV)
    core.latent_prepare(dev(proj), batch, r=r, width=D, weight=dev(wn), eps=eps, k_new=k_new, commit=cache.view(0), lat_at=qr, cq=cq,
                        cq_weight=dev(cw), status=st, **turn)
    tol = 1e-2 if bf16 else 3e-3 * rot / 64 + 5e-4          # (float32 angles of positions in the thousands)
    rots = {"dims": rot, "base": 5000.0, "scaling": scaling}
    c = plain.unit_rms(proj[:, qr:qr + r].double(), eps) * wn.double()
    kr = plain.rotate(proj[:, None, qr + r:qr + r + rot].double(), pos, rots, neighbours)[:, 0]
    close(k_new[:, 0, :r], c, tol), close(k_new[:, 0, r:r + rot], kr, tol)
    assert D == r + rot or float(k_new[:, 0, r + rot:].abs().max()) == 0.0
    close(cq, plain.unit_rms(proj[:, :qr].double(), eps) * cw.double(), tol)
    table = cache.groups[0].table.cpu()
    slot = torch.tensor([slots[0]] * counts[0] + [slots[1]] * counts[1])
    assert torch.equal(cache.view(0).k.cpu()[table[slot, pos // 64].long(), 0, pos % 64], k_new[:, 0].cpu())
    # queries: records token by token from rows of r + rot, and head by head with the rotated part in the records
    q = torch.full((T, H, D), 7.0, dtype=dt, device=DEV)
    core.latent_prepare(None, batch, q32=dev(rec32), nh=H, d=r, r=r, width=D, q_t=q, token_major=True, status=st, **turn)
    v = rec32.double().reshape(T, H, r + rot)
    close(q[:, :, :r], v[:, :, :r], tol), close(q[:, :, r:r + rot], plain.rotate(v[:, :, r:], pos, rots, neighbours), tol)
    assert D == r + rot or float(q[:, :, r + rot:].abs().max()) == 0.0
    q_t = torch.full((H, T, d), 7.0, dtype=dt, device=DEV)
    rec = torch.full((T, H, D), 7.0, dtype=dt, device=DEV)
    core.latent_prepare(None, batch, q32=dev(q32), nh=H, d=d, r=r, width=D, q_t=q_t, q_rec=rec, status=st, **turn)
    v = q32.double().reshape(T, H, d + rot)
    close(q_t, v[:, :, :d].transpose(0, 1), tol), close(rec[:, :, r:r + rot], plain.rotate(v[:, :, d:], pos, rots, neighbours), tol)
    assert float((rec[:, :, :r] - 7.0).abs().max()) == 0.0 and (D == r + rot or float(rec[:, :, r + rot:].abs().max()) == 0.0)
    # the per-head product's rows go into the records' first r columns, and a gate a (token, head) on the way
    src = torch.randn(H, T, r, generator=g)
    logits = torch.randn(T, H + 5, generator=g)
    core.heads_transpose(dev(src), rec[:, :, :r], n=r, gate=dev(logits)[:, 5:])
    close(rec[:, :, :r], src.double().transpose(0, 1) * torch.sigmoid(logits[:, 5:].double())[:, :, None], tol)
    close(rec[:, :, r:r + rot], plain.rotate(v[:, :, d:], pos, rots, neighbours), tol)
    core.check_status(st)


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("H,dv,D", [(4, 24, 32), (1, 64, 64), (3, 7, 16), (16, 96, 128)])
def test_one_gate_a_head_on_the_packed_heads(bf16, H, dv, D):
    from moe_b200.ops import core

    g = torch.Generator().manual_seed(H)
    dt = torch.bfloat16 if bf16 else torch.float32
    ctx, logits = torch.randn(11, H, D, generator=g).to(dt), torch.randn(11, H + 3, generator=g)
    out = torch.empty((11, H * dv), dtype=dt, device=DEV)
    core.gate_pack(ctx.to(DEV), out, nh=H, dv=dv, width=D, gate=dev(logits)[:, 3:])
    close(out, (ctx[:, :, :dv].double() * torch.sigmoid(logits[:, 3:].double())[:, :, None]).reshape(11, -1), 1e-2 if bf16 else 1e-6)


@pytest.mark.parametrize("window", [None, 1, 9, 64, 70, 300])
@pytest.mark.parametrize("dt,H,dv,D", [(torch.float32, 3, 40, 48), (torch.float32, 4, 33, 64), (torch.bfloat16, 6, 96, 128),
                                       (torch.bfloat16, 16, 96, 128), (torch.bfloat16, 9, 48, 64), (torch.bfloat16, 4, 130, 144),
                                       (torch.bfloat16, 20, 192, 256), (torch.bfloat16, 3, 250, 256), (torch.bfloat16, 3, 300, 320),
                                       (torch.float32, 2, 510, 512)])
def test_single_tokens_over_shared_records_with_a_gate_a_head(dt, H, dv, D, window):
    """All heads on one record that is key and value; the merge keeps dv columns and multiplies by the head's
    gate.  A key that towers over all others stands at the window's last place, or one before it."""
    from moe_b200.cache import KVCache, KVRequest
    from moe_b200.ops import core

    torch.manual_seed(D + H)
    lens = [0, 1, 63, 64, 65, 127, 300, 700]
    cache = KVCache({0: KVRequest(1, D, window, values_are_keys=True)}, {0: None}, max_tokens=64 * 40, max_slots=len(lens), dtype=dt,
                    device=DEV)
    cache.groups[0].storage.fill_(3e30)
    slots = [cache.acquire() for _ in lens]
    st = core.new_status(DEV)
    scale = 1.0 / math.sqrt(D)
    for edge in (None, 0, 1):
        K = [torch.randn(n + 1, 1, D).to(dt) for n in lens]
        q = (2 * torch.randn(len(lens), H, D)).to(dt)
        if edge is not None and window:
            q[:, :, 0] = 6.0
            for k, n in zip(K, lens):
                k[:, 0, 0] = 0.0
                if n + 1 - window - edge >= 0:
                    k[n + 1 - window - edge, 0, 0] = 60.0
        for s, k, n in zip(slots, K, lens):
            if cache.length(s) < n + 1:
                G.give_pages(cache, s, n + 1)
        if any(lens):
            live = [i for i, n in enumerate(lens) if n]
            kk = torch.cat([K[i][:-1] for i in live]).to(DEV).contiguous()
            core.kv_commit(kk, kk, cache.view(0), G.make_batch(DEV, [slots[i] for i in live], [0] * len(live), [lens[i] for i in live]), st)
        b1 = G.make_batch(DEV, slots, lens, [1] * len(lens))
        last = torch.cat([k[-1:] for k in K]).to(DEV).contiguous()
        core.kv_commit(last, last, cache.view(0), b1, st)
        logits = torch.randn(len(lens), H + 2)
        out = torch.full((len(lens), H * dv), float("nan"), dtype=dt, device=DEV)
        core.attention_decode(q.to(DEV), cache.view(0), b1, out, nh=H, window=window, scale=scale, status=st, gate=dev(logits)[:, 2:], dv=dv)
        core.check_status(st)
        for i, n in enumerate(lens):
            k = K[i][:, 0].double()
            lo = max(0, n + 1 - window) if window else 0
            p = torch.softmax((q[i].double() @ k[lo:].T) * scale, dim=-1)
            ref = (p @ k[lo:, :dv]) * torch.sigmoid(logits[i, 2:].double())[:, None]
            close(out[i].view(H, dv), ref, 2e-2 if dt == torch.bfloat16 else 2e-5)


PASTS = [([0, 0, 0], [5, 70, 131]),                       # fresh sequences only: nothing from the cache
         ([10, 100], [7, 30]),
         ([130, 64, 0], [70, 129, 200]),                  # past a page's and a tile's edge; a fresh one among them
         ([700, 128, 127, 129, 1], [300, 1, 5, 257, 128])]


@pytest.mark.parametrize("window", [None, 1, 64, 75, 200])
@pytest.mark.parametrize("H,D,dv", [(5, 64, 40), (6, 128, 96), (17, 128, 8), (3, 192, 136), (4, 256, 248), (16, 256, 192), (2, 144, 0)])
def test_steps_of_several_tokens_over_shared_records(H, D, dv, window):
    """Whole prompts and sequences that go on from the cache, all heads on one record that is key and value:
    the tensor-core kernel where it takes the record's width, once with whole records as its output and once
    packed to dv columns a head times the head's gate; else the kernel that the layer falls back to."""
    from moe_b200.cache import KVCache, KVRequest
    from moe_b200.ops import core, tc

    dt, scale = torch.bfloat16, 1.0 / math.sqrt(D)
    for n, (before, new) in enumerate(PASTS):
        torch.manual_seed(n + D)
        cache = KVCache({0: KVRequest(1, D, window, values_are_keys=True)}, {0: None}, max_tokens=64 * 40, max_slots=len(new), dtype=dt,
                        device=DEV)
        cache.groups[0].storage.fill_(3e30)
        slots = [cache.acquire() for _ in new]
        st = core.new_status(DEV)
        K = [torch.randn(a + b, 1, D).to(dt) for a, b in zip(before, new)]
        Q = [(2 * torch.randn(b, H, D)).to(dt) for b in new]
        live = [i for i, a in enumerate(before) if a]
        for i, s in enumerate(slots):
            G.give_pages(cache, s, before[i] + new[i])
        if live:
            kk = torch.cat([K[i][:before[i]] for i in live]).to(DEV).contiguous()
            core.kv_commit(kk, kk, cache.view(0), G.make_batch(DEV, [slots[i] for i in live], [0] * len(live), [before[i] for i in live]), st)
        batch = G.make_batch(DEV, slots, before, new)
        q, kn = torch.cat(Q).to(DEV).contiguous(), torch.cat([k[a:] for k, a in zip(K, before)]).to(DEV).contiguous()
        out = torch.full((q.shape[0], H, D), float("nan"), dtype=dt, device=DEV)
        kw = dict(nh=H, window=window, scale=scale, status=st)

        def on_tensor_cores(o, **form):
            return (tc.attention_cached(q, kn, kn, cache.view(0), batch, o, **form, **kw) if any(before)
                    else tc.attention_prefill(q, kn, kn, batch, o, nkv=1, hd=D, **form, **kw))

        done = on_tensor_cores(out)
        assert done == (D in (64, 128, 192, 256))
        packed = None
        if done:
            logits = torch.randn(q.shape[0], H + 1)
            packed = torch.full((q.shape[0], H * dv), float("nan"), dtype=dt, device=DEV)
            assert on_tensor_cores(packed, dv=dv, gate=dev(logits)[:, 1:])
        else:
            assert core.attention_tiled(q, kn, kn, cache.view(0), batch, out, use_local=True, **kw)
        core.check_status(st)
        o = 0
        for i, (a, b) in enumerate(zip(before, new)):
            k = K[i][:, 0].double()
            s = torch.einsum("thd,jd->htj", Q[i].double(), k) * scale
            seen = plain.seen_mask(a + b, window)[a:]
            p = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1)
            ref = torch.einsum("htj,jd->thd", p, k)
            close(out[o:o + b], ref, 2e-2)
            if packed is not None:
                g = torch.sigmoid(logits[o:o + b, 1:].double())
                close(packed[o:o + b].view(b, H, dv), ref[:, :, :dv] * g[:, :, None], 2e-2)
            o += b


# ----------------------------------------------------------------------------- the delta mixer's kernels
CUTS = [[(0, 0, 10)], [(0, 10, 12), (1, 0, 2)], [(0, 12, 143), (1, 2, 9)], [(0, 143, 144), (1, 9, 10)], [(1, 10, 11), (0, 144, 145)]]
LENS = {0: 145, 1: 11}                                       # (sequence, from, to) per step; the last two bring one token each
DELTA_SIZES = [(2, 1, 8, 8, 4), (4, 2, 16, 24, 4), (3, 3, 10, 7, 3), (6, 2, 64, 64, 2), (2, 2, 128, 128, 4), (1, 1, 32, 4, 1), (2, 1, 200, 72, 5),
               (4, 4, 256, 16, 4), (2, 1, 40, 136, 4), (8, 2, 5, 3, 4)]


def delta_case(H, Gk, d, dv, taps, seed):
    g = torch.Generator().manual_seed(seed)
    ch = 2 * Gk * d + H * dv
    rows = {s: torch.randn(n, ch + 2 * H, generator=g) for s, n in LENS.items()}
    taps_w = 0.4 * torch.randn(ch, taps, generator=g) + 0.3
    a_log, dt_bias = torch.randn(H, generator=g) - 1.0, torch.randn(H, generator=g) - 1.0
    return rows, taps_w, a_log, dt_bias, ch


def plain_delta_inputs(row, taps_w, a_log, dt_bias, H, Gk, d, dv, ch):
    y = plain.silu(plain.causal_taps(row[:, :ch].double(), taps_w.double()))
    T = y.shape[0]
    q = plain.unit_length(y[:, :Gk * d].reshape(T, Gk, d)) / math.sqrt(d)
    k = plain.unit_length(y[:, Gk * d:2 * Gk * d].reshape(T, Gk, d))
    v = y[:, 2 * Gk * d:].reshape(T, H, dv)
    beta = torch.sigmoid(row[:, ch:ch + H].double())
    decay = torch.exp(-torch.exp(a_log.double()) * plain.softplus(row[:, ch + H:].double() + dt_bias.double()))
    return q, k, v, beta, decay


@pytest.mark.parametrize("H,Gk,d,dv,taps", DELTA_SIZES)
def test_convolution_unit_norms_recurrence_norm_and_gate_over_steps(H, Gk, d, dv, taps):
    """Two sequences of unequal lengths in five steps (a step brings fewer rows than the convolution has taps;
    the last two bring one token each): what the kernels prepare, the outputs and the state."""
    from moe_b200.ops import core

    rows, taps_w, a_log, dt_bias, ch = delta_case(H, Gk, d, dv, taps, H * 7 + d)
    at = -(-((taps - 1) * ch) // 4) * 4
    state = torch.zeros((4, at + H * d * dv), device=DEV)
    g = torch.Generator().manual_seed(1)
    norm_w, eps = (1 + 0.2 * torch.randn(dv, generator=g)), 1e-5
    gates = {s: torch.randn(n, H * dv, generator=g) for s, n in LENS.items()}
    tw = dev(taps_w.t())
    prepared, outs = {0: [], 1: []}, {0: [], 1: []}
    for step in CUTS:
        batch = G.make_batch(DEV, [s + 1 for s, _, _ in step], [a for _, a, _ in step], [b - a for _, a, b in step])
        T = batch.num_tokens
        proj = dev(torch.cat([rows[s][a:b] for s, a, b in step]))
        gate = dev(torch.cat([gates[s][a:b] for s, a, b in step]))
        qkv, stp = torch.empty((T, ch), device=DEV), torch.empty((T, 2 * H), device=DEV)
        sizes = dict(heads=H, kv_heads=Gk, d=d, dv=dv)
        core.delta_prepare(proj, tw, dev(a_log), dev(dt_bias), state, batch, qkv, stp, b_at=ch, a_at=ch + H, eps=1e-6,
                           q_scale=d ** -0.5, **sizes)
        if taps > 1 and not batch.all_decode:
            core.conv_state_update(proj, state, batch, taps=taps, channels=ch)
        y = torch.full((T, H * dv), float("nan"), device=DEV)
        nw = dev(norm_w.repeat(H))
        if not (batch.all_decode and core.delta_step(qkv, stp, state, gate, nw, eps, batch, y, offset=at, **sizes)):
            o = torch.empty((T, H * dv), device=DEV)
            core.delta_scan(qkv, stp, state, batch, o, offset=at, **sizes)
            core.wkv_finish(o, gate, nw, eps, batch, y, heads=H, d=dv)
        i = 0
        for s, a, b in step:
            prepared[s].append((qkv[i:i + b - a].cpu(), stp[i:i + b - a].cpu()))
            outs[s].append(y[i:i + b - a].cpu())
            i += b - a
    for s, n in LENS.items():
        q, k, v, beta, decay = plain_delta_inputs(rows[s], taps_w, a_log, dt_bias, H, Gk, d, dv, ch)
        qkv, stp = torch.cat([p for p, _ in prepared[s]]), torch.cat([p for _, p in prepared[s]])
        close(qkv, torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], dim=1), 1e-5)
        close(stp[:, :H], beta, 1e-6), close(torch.exp(stp[:, H:].double()), decay, 1e-6)
        owner = torch.arange(H) // (H // Gk)
        o, S = plain.delta_recurrence(q[:, owner], k[:, owner], v, decay, beta)
        ref = (plain.unit_rms(o, eps) * norm_w.double()).reshape(n, -1) * plain.silu(gates[s].double())
        close(torch.cat(outs[s]), ref, 2e-4)
        close(state[s + 1, at:].view(H, d, dv), S, 2e-5)
        if taps > 1:
            tail = torch.cat([torch.zeros(taps - 1, ch), rows[s][:, :ch]])[-(taps - 1):]
            assert torch.equal(state[s + 1, :(taps - 1) * ch].view(taps - 1, ch).cpu(), tail)
    assert float(state[0].abs().max()) == 0.0 and float(state[3].abs().max()) == 0.0


def test_a_value_written_once_is_read_back_hundreds_of_tokens_later():
    """Decays of one and steps of one: the state is an exact memory of one value a key direction, and writing
    the same key again replaces what it held."""
    from moe_b200.ops import core

    d, dv, T = 16, 8, 600
    g = torch.Generator().manual_seed(3)
    k = torch.zeros(T, d)
    k[torch.arange(T), torch.arange(T) % (d - 1)] = 1.0       # every direction but the last, over and over
    k[5] = 0.0
    k[5, d - 1] = 1.0                                         # the last direction is written at token 5 only
    q = torch.zeros(T, d)
    q[:, d - 1] = 1.0
    v = torch.randn(T, dv, generator=g)
    state = torch.zeros((2, d * dv), device=DEV)
    o = torch.empty((T, dv), device=DEV)
    step = torch.cat([torch.ones(T, 1), torch.zeros(T, 1)], dim=1)
    batch = G.make_batch(DEV, [1], [0], [T])
    core.delta_scan(dev(torch.cat([q, k, v], dim=1)), dev(step), state, batch, o, heads=1, kv_heads=1, d=d, dv=dv)
    assert float(o[:5].abs().max()) == 0.0
    close(o[5:], v[5].expand(T - 5, dv), 1e-6)
    held = state[1].view(d, dv).cpu()
    for i in range(d - 1):
        last = max(t for t in range(T) if t % (d - 1) == i and t != 5)
        close(held[i], v[last], 1e-6)


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
        assert err < 3e-5, f"layer {i}: {err:.3g}"


# ----------------------------------------------------------------------------- whole prompts, decoding, portions
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_of_many_lengths(root, name, dtype):
    d, eng = engine_of(root, name, dtype)
    cfg, _ = model_of(d)
    requests = {f"r{n}": U.tokens(cfg["vocab"], n, n) for n in (1, 2, 3, 63, 64, 65, 131, 200)}
    check_schedule(d, eng, requests, helpers.whole_schedule(requests), G.tol(dtype))


def test_latents_of_one_number_in_32_bit(root):
    d, eng = engine_of(root, "single", "float32")
    cfg, _ = model_of(d)
    requests = {f"r{n}": U.tokens(cfg["vocab"], n, n) for n in (1, 2, 65, 131)}
    for steps in (helpers.whole_schedule(requests), helpers.tail_schedule({"r131": requests["r131"]}, tail=100),
                  portions_schedule("r131", requests["r131"], [2, 40, 3])):
        check_schedule(d, eng, {r: t for r, t in requests.items() if any(r == e[0] for s in steps for e in s["entries"])}, steps, 2e-4)


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
@pytest.mark.parametrize("name", ["mix", "ones", "wide", "lean", "huge"])
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
    special = 0                      # (the token that spike_token marks by default)
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
@pytest.mark.parametrize("size", [1, 7, 64, 65, 130])
def test_windows_one_position_longer_or_shorter(root, dtype, size):
    """The same weights with another window: a key just inside the window of one model is just outside in
    the next, in prompts, portions and decoding; by how much the logits move is what the plain implementation
    says, and it is more than the tolerance."""
    def edit(cfg):
        for L in cfg["layers"]:
            L["mixer"]["mask"] = {"size": size}
    edit.__name__ = f"window{size}"
    d, eng = engine_of(root, "sharp", dtype, edit=edit)
    cfg, w = model_of(d)
    toks = U.tokens(cfg["vocab"], 200, size)
    ref = reference(d, toks)
    longer = json.loads(json.dumps(cfg))
    for L in longer["layers"]:
        L["mixer"]["mask"] = {"size": size + 1}
    moved = (plain.forward(longer, w, toks) - ref).abs().amax(dim=1) / float(ref.abs().max())
    assert float(moved.max()) > (0.05 if size <= 65 else 0.005)
    tol = G.tol(dtype)
    check_schedule(d, eng, {"a": toks}, helpers.whole_schedule({"a": toks}), tol)
    check_schedule(d, eng, {"a": toks}, helpers.tail_schedule({"a": toks}, tail=70), tol)
    check_schedule(d, eng, {"a": toks}, portions_schedule("a", toks, [size + 1, 2, 61]), tol)


@pytest.mark.parametrize("dtype", DTYPES)
def test_layers_that_share_tensors_keep_caches_and_state_of_their_own(root, dtype):
    """Decoding a model whose layers are used twice, against the same model with the tensors written out under
    every layer's own name."""
    import moe_b200
    from moe_b200.engine import Engine
    from moe_b200.weights.safetensors_io import write_safetensors

    d, eng = engine_of(root, "mix", dtype)
    cfg, _ = model_of(d)
    w = U.draw_weights(cfg, 11)
    flat = json.loads(json.dumps(cfg))
    for i, L in enumerate(flat["layers"]):
        j = L.pop("weights_of", None)
        if j is not None:
            w.update({f"l{i}." + n[len(f"l{j}."):]: t for n, t in list(w.items()) if n.startswith(f"l{j}.")})
    f = os.path.join(os.path.dirname(d), "written_out")
    os.makedirs(f, exist_ok=True)
    with open(os.path.join(f, "config.json"), "w") as fh:
        json.dump(flat, fh)
    write_safetensors(os.path.join(f, "model.safetensors"), w)
    two = Engine(moe_b200.load_model(f, dtype=dtype), max_tokens=512)
    assert two.model.num_parameters > eng.model.num_parameters
    toks = U.tokens(cfg["vocab"], 90, 8)
    steps = helpers.tail_schedule({"a": toks}, tail=30)
    a, b = helpers.run_schedule(eng, steps)[0], helpers.run_schedule(two, steps)[0]
    assert a.keys() == b.keys()
    for k in a:
        assert torch.equal(a[k], b[k])


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
    for word in ("Ditazen", "gated delta rule", "latent attention", "window 24", "a sigmoid gate a head", "YaRN", "dense gelu", "LayerNorm"):
        assert word in r.stdout, word
