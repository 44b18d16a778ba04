"""Latent attention: keys and values of every head are projections of ONE small latent per
position, and only the latent (and, with positions, one rotated key part) is cached.

With n the layer's normed input, H heads, d the query/key size, dv the value size, r the latent's:
    q = Wq n   [H, d (+ rot)]
    c = rms(Wdkv n) * w_c                        (r numbers; x / sqrt(mean(x^2) + eps), plain weight)
    k_h = Wuk_h c,  v_h = Wuv_h c                (rows of Wuk / Wuv head by head)
    p_hj = exp(scale q_h . k_hj) / (exp(b_h) + sum_j' exp(scale q_h . k_hj')),  j <= position (causal)
    out = Wo [sum_j p_hj v_hj]_h

Options (each a constant of the part):
  sink        b_h, the head's sink: a learned number that joins the denominator and carries no value
              (without it the exp(b_h) is absent).
  rot_dim     a head has `rot` further query dimensions, rotated by the position with the part's
              ``position`` encoding (pairs of halves or of neighbours, its scaling, its factor on cos and
              sin); their key is ONE vector of rot numbers per position that all heads share: the rows of
              Wdkv after the latent's, rotated, not normed.  The score is scale (q_h . k_hj + q'_h . k'_j).
  q_rank      the queries come through a latent of their own: q = Wuq (rms(Wdq n) * w_q).
  window      position i sees j with 0 <= i - j < window.
  head_gate   head h's output is multiplied by sigmoid(Wg n)_h.

How it runs.  q_h . (Wuk_h c) = (Wuk_h^T q_h) . c and sum_j p_j Wuv_h c_j = Wuv_h sum_j p_j c_j, so the
attention runs over the cached latents alone: H query heads of r + rot numbers on ONE key/value head
whose keys [c | rotated part] ARE its values (``KVRequest.values_are_keys``: one plane of the paged cache,
r + rot numbers a position whatever H is; the output's columns beyond r are dropped).  The attention
kernels are the ones every other layer uses.  Records have one width D >= r + rot (zero-filled).  Each of
the two per-head products runs in one of two forms, chosen when the weights are bound by the number of
weight elements a token then meets (``absorb``: "auto", or True / False for both sides):

* folded into its neighbour: Wuk_h^T Wq_h (r x inputs a head) stands in the query projection's place,
  whose output row then holds the queries over the latent, and Wo_h Wuv_h (hidden x r a head) in the
  output projection's, which then reads the attended latents; cheaper while r inputs <= d (inputs + r),
  resp. r hidden <= dv (hidden + r): a latent no larger than a head.  The folded matrices are formed once
  in float64 from the checkpoint's values and rounded once to the weights' dtype.  A latent layer is then
  norm, projection, ``latent_prepare`` (latent norm, rotation, key record, append, queries as records; with
  a query latent two launches around its product), attention, (gate and packing,) output projection.
* on its own: a grouped product, a group a head, through the kernels the routed experts use; the
  groups' rows lie head by head, which ``latent_prepare`` and ``heads_transpose`` arrange.  Cheaper
  for latents several times a head's size.

32-bit in both dtypes: the latents' norms, positions and angles, scores, softmax, sink and gate.  The
bfloat16 path rounds the queries' latent, the queries over the latent, the cached record, and the attended
latent before its product (and, on its own, the queries before and the values after their per-head
product).
"""
from __future__ import annotations

import torch

from ..cache.kv import KVRequest
from ..config.spec import PartSpec
from ..ops import core
from ..ops.linear import grouped_linear, linear
from .base import Part, TensorSpec, make_part, register_part


def record_width(n: int, bf16: bool) -> int:
    """Width of a cached record of n numbers: in bfloat16 the tensor-core attention over records that are key
    and value takes 64, 128, 192 and 256, everything takes multiples of 16 (beyond 256 the plain kernels run)."""
    if bf16 and n <= 256:
        return -(-n // 64) * 64
    return -(-n // 16) * 16


class LatentAttention(Part):
    category, kind = "mixer", "latent_attention"
    graph_safe = True
    default_names = {"q": "q_proj.weight", "down": "kv_a_proj.weight", "down_norm": "kv_a_norm.weight",
                     "up_k": "k_b_proj.weight", "up_v": "v_b_proj.weight", "sink": "sinks", "o": "o_proj.weight",
                     "q_down": "q_a_proj.weight", "q_down_norm": "q_a_norm.weight", "q_up": "q_b_proj.weight",
                     "gate": "gate_proj.weight"}

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden = int(p["hidden_size"])
        self.nh = int(p["num_heads"])
        self.hd = int(p["head_dim"])
        self.vd = int(p.get("value_dim") or self.hd)
        self.rank = int(p["kv_rank"])
        self.rot = int(p.get("rot_dim") or 0)
        self.q_rank = int(p.get("q_rank") or 0)
        self.window = p.get("window")
        self.head_gate = bool(p.get("head_gate", False))
        self.scale = float(p["scale"])
        self.eps = float(p["eps"])
        self.sink = bool(p.get("sink", False))
        self.absorb = p.get("absorb", "auto")
        pos = dict(p.get("position") or {"kind": "none"})
        self.position = make_part("position", PartSpec(pos.pop("kind"), pos, spec.prefix))
        if self.rot and getattr(self.position, "rotary_dim", 0) != self.rot:
            raise ValueError("latent attention: the position encoding must turn exactly the rotated part of a head")
        if not (self.nh > 0 and self.hd > 0 and self.vd > 0 and self.rank > 0 and 0 < self.rank + self.rot <= 1024):
            raise ValueError(f"latent attention: {self.nh} heads of {self.hd} / {self.vd} on a latent of {self.rank}"
                             + (f" and a rotated part of {self.rot}" if self.rot else "")
                             + "; the attention kernels take records of up to 1024")
        if self.window is not None and self.window <= 0:
            raise ValueError("window must be positive")
        self.record = self.rank + self.rot        # numbers a position
        self.width = self.record                  # of a cached record; set when bound

    @property
    def q_inputs(self):
        """Columns of the query projection: the model's width, or the queries' latent."""
        return self.q_rank or self.hidden

    def tensors(self):
        n, H, W, r = self.names, self.nh, self.hidden, self.rank
        t = {}
        if self.q_rank:
            t[n["q_down"]] = TensorSpec((self.q_rank, W))
            t[n["q_down_norm"]] = TensorSpec((self.q_rank,), init="ones", vector=True)
            t[n["q_up"]] = TensorSpec((H * (self.hd + self.rot), self.q_rank))
        else:
            t[n["q"]] = TensorSpec((H * (self.hd + self.rot), W))
        t[n["down"]] = TensorSpec((r + self.rot, W))
        t[n["down_norm"]] = TensorSpec((r,), init="ones", vector=True)
        t[n["up_k"]] = TensorSpec((H * self.hd, r))
        t[n["up_v"]] = TensorSpec((H * self.vd, r))
        if self.head_gate:
            t[n["gate"]] = TensorSpec((H, W))
        t[n["o"]] = TensorSpec((W, H * self.vd))
        if self.sink:
            t[n["sink"]] = TensorSpec((H,), init="zeros", vector=True)
        return t

    def kv_request(self):
        return KVRequest(1, self.width, self.window, values_are_keys=True)

    def state_request(self):
        return None

    def describe(self):
        return (f"latent attention ({self.nh} heads of {self.hd}{f'+{self.rot}' if self.rot else ''}, values of {self.vd}, "
                f"one cached latent of {self.rank} a position"
                + (f" and a rotated key part of {self.rot}" if self.rot else "")
                + (f", queries through a latent of {self.q_rank}" if self.q_rank else "")
                + (", softmax with a sink a head" if self.sink else "")
                + (", a sigmoid gate a head" if self.head_gate else "")
                + (f", window {self.window}" if self.window else "") + f"), {self.position.describe()}")

    def step_elements(self, tokens):
        W, H, r, Q = self.hidden, self.nh, self.rank, self.q_inputs
        fq, fo = self._folds()
        qside = H * r * Q if fq else H * self.hd * (Q + r)
        oside = H * r * W if fo else H * self.vd * (W + r)
        rest = (r + self.rot) * W + r + H * self.rot * Q + self.q_rank * (W + 1) + (H * W if self.head_gate else 0)
        return float(qside + oside + rest)

    def _folds(self):
        """(fold the queries' product, fold the values' product): by weight elements a token meets."""
        if self.absorb in (True, False):
            return bool(self.absorb), bool(self.absorb)
        W, r, Q = self.hidden, self.rank, self.q_inputs
        return r * Q <= self.hd * (Q + r), r * W <= self.vd * (W + r)

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        n, H, d, dv, r, rot, Q = self.names, self.nh, self.hd, self.vd, self.rank, self.rot, self.q_inputs
        self.width = D = record_width(self.record, rt.is_bf16)
        self.fold_q, self.fold_o = self._folds()
        self.position.bind(tensors, rt)
        table = self.position.rotary_table()[0] if rot else None
        self.turn = dict(rot=rot, freq=table, interleaved=bool(getattr(self.position, "interleaved", False)),
                         mscale=float(getattr(self.position, "cos_sin_scale", lambda: 1.0)()))
        wq, wdown = tensors[n["q_up" if self.q_rank else "q"]], tensors[n["down"]]
        dt = wq.dtype if wq.dtype == wdown.dtype else torch.float32
        uk = tensors[n["up_k"]].reshape(H, d, r)
        uv = tensors[n["up_v"]].reshape(H, dv, r)
        wo = tensors[n["o"]]
        if self.fold_q:
            # rows h (r + rot) ...: Wuk_h^T Wq_h, the head's queries over the latent, then its rotated part's rows
            heads = wq.reshape(H, d + rot, Q)
            over = torch.bmm(uk.double().transpose(1, 2), heads[:, :d].double()).to(dt)
            wq = torch.cat([over, heads[:, d:].to(dt)], dim=1).reshape(H * (r + rot), Q)
            self.w_qc = None
        else:
            self.w_qc = uk.transpose(1, 2).contiguous()                    # grouped [head, r, d]
        self.q_cols = r if self.fold_q else d
        # one product of the layer's input: [queries, or their latent | latent and rotated key part | gate | zeros up
        # to a multiple of eight, so that rows of the output stay 16-byte units]
        first = tensors[n["q_down"]] if self.q_rank else wq
        rows = [first.to(dt), wdown.to(dt)]
        self.lat_at = first.shape[0]
        self.gate_at = self.lat_at + wdown.shape[0]
        if self.head_gate:
            rows.append(tensors[n["gate"]].to(dt))
        if rot or self.q_rank or self.head_gate:
            total = sum(w.shape[0] for w in rows)
            rows.append(torch.zeros((-total % 8, self.hidden), dtype=dt, device=wdown.device))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_q_up = wq.to(dt).contiguous() if self.q_rank else None
        self.cq_norm = tensors[n["q_down_norm"]].to(torch.float32).contiguous() if self.q_rank else None
        # with a gate the attended latents are gated and packed to r columns a head; without one the output
        # projection reads whole records (its columns beyond r are zeros)
        self.packs = self.head_gate
        if self.fold_o:
            # columns of head h: Wo_h Wuv_h
            ov = torch.bmm(wo.double().reshape(self.hidden, H, dv).transpose(0, 1), uv.double())     # [H, hidden, r]
            full = torch.zeros((self.hidden, H, r if self.packs else D), dtype=torch.float64, device=ov.device)
            full[:, :, :r] = ov.transpose(0, 1)
            self.wo = full.reshape(self.hidden, -1).to(wo.dtype).contiguous()
            self.w_cv = None
        else:
            self.w_cv = uv.contiguous()                                    # grouped [head, dv, r]
            self.wo = wo.contiguous()
        self.w_norm = tensors[n["down_norm"]].to(torch.float32).contiguous()
        self.sinks = tensors[n["sink"]].to(torch.float32).contiguous() if self.sink else False
        self._offsets = {}

    def _head_offsets(self, T, device):
        """Row offsets [0, T, 2T, ..., H T] of the heads in a grouped product."""
        o = self._offsets.get(T)
        if o is None:
            o = self._offsets[T] = (torch.arange(0, self.nh + 1, dtype=torch.int32, device=device) * T).contiguous()
        return o

    def _prepare(self, rt, h, batch, commit):
        """Projection(s) and ``latent_prepare``: (queries [T, H, D], the step's key records, gate logits)."""
        T, D, H, r = batch.num_tokens, self.width, self.nh, self.rank
        proj = linear(rt, h.act, self.w_in)                       # 32-bit
        gate = proj[:, self.gate_at:self.gate_at + H] if self.head_gate else None
        k_new = rt.empty((T, 1, D))
        q = rt.empty((T, H, D))
        keys = dict(weight=self.w_norm, eps=self.eps, k_new=k_new, commit=commit, lat_at=self.lat_at)
        q_t = q if self.fold_q else rt.empty((H, T, self.hd))
        queries = dict(nh=H, d=self.q_cols, q_t=q_t, token_major=self.fold_q, q_rec=None if self.fold_q else q)
        both = dict(r=r, width=D, status=rt.status, **self.turn)
        if self.q_rank:
            cq = rt.empty((T, self.q_rank))
            core.latent_prepare(proj, batch, cq=cq, cq_weight=self.cq_norm, **keys, **both)
            core.latent_prepare(None, batch, q32=linear(rt, cq, self.w_q_up), **queries, **both)
        else:
            core.latent_prepare(proj, batch, **keys, **queries, **both)
        if not self.fold_q:
            offsets = self._head_offsets(T, proj.device)
            qc = grouped_linear(rt, q_t.view(H * T, self.hd), self.w_qc, offsets, H * T)      # [H T, r] 32-bit
            core.heads_transpose(qc.view(H, T, r), q[:, :, :r] if self.rot else q, n=r)
        return q, k_new, gate

    def forward(self, rt, h, batch, cache_view, state=None):
        T, D, H, dv, r = batch.num_tokens, self.width, self.nh, self.vd, self.rank
        # a step of one token a sequence reads its own key from the cache; whole prompts read nothing
        # from it: both may append at once.  A step that goes on from the cache appends afterwards.
        early = batch.all_decode or batch.all_fresh
        q, k_new, gate = self._prepare(rt, h, batch, cache_view if early else None)
        dev = q.device
        packed = rt.empty((T, H * r)) if self.packs and self.fold_o else None
        kw = dict(nh=H, window=self.window, scale=self.scale, status=rt.status, sink=self.sinks)
        if batch.all_decode and packed is not None:
            # (the merge of the key splits multiplies by the gate and packs the heads)
            core.attention_decode(q, cache_view, batch, packed, gate=gate, dv=r, **kw)
            return linear(rt, packed, self.wo)
        ctx, done = None, False
        if not batch.all_decode and rt.is_bf16:
            from ..ops import tc

            # (the tensor-core kernel may multiply by the gate and pack the heads itself)
            forms = [(packed, dict(dv=r, gate=gate))] if packed is not None and r % 8 == 0 else []
            for out, form in forms + [(None, {})]:
                if out is None:
                    out = ctx = rt.empty((T, H, D))
                if getattr(batch, "has_padding", False):
                    out.zero_()      # rows of no sequence are written by no attention kernel
                if batch.all_fresh:
                    done = tc.attention_prefill(q, k_new, k_new, batch, out, nkv=1, hd=D, **form, **kw)
                else:
                    done = tc.attention_cached(q, k_new, k_new, cache_view, batch, out, **form, **kw)
                if done:
                    break
        if ctx is None and not done:
            ctx = rt.empty((T, H, D))
            if getattr(batch, "has_padding", False) and not batch.all_decode:
                ctx.zero_()
        if batch.all_decode:
            core.attention_decode(q, cache_view, batch, ctx.view(T, H * D), **kw)
        else:
            if not done and not core.attention_tiled(q, k_new, k_new, cache_view, batch, ctx, use_local=True, **kw):
                core.attention_generic(q, k_new, k_new, cache_view, batch, ctx, use_local=True, **kw)
            if not early:
                core.kv_commit(k_new, k_new, cache_view, batch, rt.status)
        if packed is not None:
            if ctx is not None:
                core.gate_pack(ctx, packed, nh=H, dv=r, width=D, gate=gate)
            return linear(rt, packed, self.wo)
        if self.fold_o:
            return linear(rt, ctx.view(T, H * D), self.wo)
        offsets = self._head_offsets(T, dev)
        c_t = rt.empty((H, T, r))
        core.heads_transpose(ctx, c_t, n=r)
        ov = grouped_linear(rt, c_t.view(H * T, r), self.w_cv, offsets, H * T)      # [H T, dv] 32-bit
        values = rt.empty((T, H, dv))
        core.heads_transpose(ov.view(H, T, dv), values, n=dv, gate=gate)
        return linear(rt, values.view(T, H * dv), self.wo)


register_part("mixer", "latent_attention", LatentAttention)
