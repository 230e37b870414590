"""Attention through low-rank latents: the cache keeps one compressed row per token.

    (a | b | r | g) = (W_dq | W_dkv | W_g) x       one product: query latent, key/value latent, rotated key part, gates
    c_q = rmsnorm(a) * w_q;   c = rmsnorm(b) * w_kv;   r <- rotary(r)      (pairs of neighbouring dims)
    q   = W_uq c_q, per head [head_dim unrotated | rot_dim rotated];  the rotated part <- rotary(.)
    per head: k = W_uk c (unrotated) beside the shared r, v = W_uv c
    s(i, j) = (q_unrot . k_j + q_rot . r_j) * scale,  i sees j iff 0 <= i - j (< window),  softmax (with a sink: its
              denominator also counts exp(sink_h))
    y       = W_o concat_h(sigmoid(g_h) sum_j p_j v_j)

What of it a mixer has is up to its parameters: without ``q_rank`` the queries come straight from x (``W_q`` takes
``W_dq``'s place in the first product); without ``gated`` there are no gates, without ``sink`` no sinks; without ``own_kv`` there is no ``W_dkv``
and the rows of an earlier schedule position (the model's schedule names it) are read, with this mixer's own queries,
``W_uk``, ``W_uv`` and window; the rotation may come with rescaled frequencies and a factor (``position_encoding``).

Only ``c`` and ``r`` are kept per token, side by side in one cache row ``[kv_rank + rot_dim]``.  Keys and values
are never expanded: since ``q_unrot . (W_uk c) = (W_uk^T q_unrot) . c``, the query is carried into the latent space
(one batched product per step) and attention runs over the rows as they are stored, every head reading the same
row as its key and the row's first ``kv_rank`` elements as its value; the result per head is a mix of latents (times
the head's gate), which ``W_uv`` turns into the head's output (one more batched product).  Between the first product
and the attention stands one row-wise kernel (``ops.latent_prep``; with a query latent also ``ops.rotate_pairs`` behind
the second product).
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import POSITION_ENCODINGS, CacheSpec, CacheTensor, Mixer, ParamSpec, build_part, register_mixer
from .scored_attention import run_attention

#: the first product's columns are padded to a multiple of this many: its rows then start on 16-byte boundaries in
#: either precision, which the batched product that reads the queries out of them likes
ROW_MULTIPLE = 8


@register_mixer("latent_attention")
class LatentAttention(Mixer):
    """params: ``num_heads``, ``head_dim`` (unrotated query / key dims per head), ``rot_dim`` (rotated dims per head,
    and the width of the shared rotated key part), ``v_dim``, ``q_rank`` (None: queries straight from the input),
    ``kv_rank``, ``scale``, ``norm_eps``, ``rotary_base``, ``rotary_dims`` (how many of the ``rot_dim`` dims turn;
    default all) or ``position_encoding`` (a PartSpec of a rope in the pairs layout, in their place), ``window`` (None:
    all keys), ``gated`` (bool: a sigmoid gate per head read from the input), ``sink`` (bool: a learned number per head in
    the softmax's denominator), ``own_kv`` (bool, default True), ``names`` (local tensor names)."""

    graph_safe = True
    takes_lazy_norm = True
    adds_residual = True

    NAMES = {"dq": "q_a_proj.weight", "dq_norm": "q_a_norm.weight", "uq": "q_b_proj.weight", "q": "q_proj.weight",
             "dkv": "kv_a_proj.weight", "dkv_norm": "kv_a_norm.weight", "uk": "k_b_proj.weight",
             "uv": "v_b_proj.weight", "gate": "gate_proj.weight", "out": "o_proj.weight", "sink": "sinks"}

    def __init__(self, spec, **kw):
        super().__init__(spec, **kw)
        p = spec.params
        self.num_heads, self.head_dim, self.rot_dim = int(p["num_heads"]), int(p["head_dim"]), int(p["rot_dim"])
        self.v_dim, self.q_rank, self.kv_rank = int(p["v_dim"]), int(p.get("q_rank") or 0), int(p["kv_rank"])
        if min(self.num_heads, self.head_dim, self.v_dim, self.kv_rank) <= 0 or min(self.rot_dim, self.q_rank) < 0:
            raise ValueError("latent_attention: sizes must be positive")
        self.position_encoding = None
        if p.get("position_encoding") is not None:
            self.position_encoding = build_part(POSITION_ENCODINGS, p["position_encoding"], hidden_size=self.hidden_size,
                                                dtype=self.dtype, device=self.device)
            table = getattr(self.position_encoding, "rotary_table", None)
            if table is None:
                raise ValueError(f"latent_attention: position encoding {p['position_encoding'].kind!r} has no rotary table")
            self.inv_freq, self.rotary_dims, layout, self.rotary_factor = table()
            if layout != "pairs":
                raise ValueError(f"latent_attention: the rotated parts turn in neighbouring pairs, got layout {layout!r}")
        else:
            self.rotary_dims, self.rotary_factor = int(p.get("rotary_dims", self.rot_dim)), 1.0
            i = torch.arange(self.rotary_dims // 2, dtype=torch.float64)
            base = float(p.get("rotary_base", 10000.0))
            self.inv_freq = (base ** (-2.0 * i / max(self.rotary_dims, 1))).to(torch.float32).to(self.device)
        if self.rotary_dims % 2 or not 0 <= self.rotary_dims <= self.rot_dim:
            raise ValueError(f"latent_attention: rotary_dims must be even and at most rot_dim ({self.rot_dim}), "
                             f"got {self.rotary_dims}")
        if self.kv_rank > 512 or self.kv_rank + self.rot_dim > 1024:
            raise ValueError(f"latent_attention: a latent of {self.kv_rank} + {self.rot_dim} is wider than the "
                             f"attention kernel takes (512 + rotated part up to 1024)")
        self.scale = float(p["scale"]) if p.get("scale") is not None else (self.head_dim + self.rot_dim) ** -0.5
        self.norm_eps = float(p.get("norm_eps", 1e-6))
        self.window = int(p["window"]) if p.get("window") else 0
        self.gated, self.own_kv = bool(p.get("gated", False)), bool(p.get("own_kv", True))
        self.has_sink = bool(p.get("sink", False))
        self.sink = None
        self.names = dict(self.NAMES, **(p.get("names") or {}))
        self.w_in = self.w_uq = self.w_uk = self.w_uv = self.w_o = self.q_norm = self.kv_norm = None

    def children(self):
        return () if self.position_encoding is None else (self.position_encoding,)

    @property
    def row(self) -> int:
        return self.kv_rank + self.rot_dim

    @property
    def q_width(self) -> int:
        return self.num_heads * (self.head_dim + self.rot_dim)

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(kind="window" if self.window else "full", num_kv_heads=1, head_dim=self.row,
                         window=self.window or None, tensors=(CacheTensor("latent", 1, self.row),))

    def param_specs(self):
        h, n, H = self.hidden_size, self.names, self.num_heads
        specs = {}
        if self.q_rank:
            specs[n["dq"]] = ParamSpec((self.q_rank, h))
            specs[n["dq_norm"]] = ParamSpec((self.q_rank,), kind="vector", init="norm")
            specs[n["uq"]] = ParamSpec((self.q_width, self.q_rank))
        else:
            specs[n["q"]] = ParamSpec((self.q_width, h))
        if self.own_kv:
            specs[n["dkv"]] = ParamSpec((self.row, h))
            specs[n["dkv_norm"]] = ParamSpec((self.kv_rank,), kind="vector", init="norm")
        specs[n["uk"]] = ParamSpec((H * self.head_dim, self.kv_rank))
        specs[n["uv"]] = ParamSpec((H * self.v_dim, self.kv_rank))
        if self.gated:
            specs[n["gate"]] = ParamSpec((H, h))
        if self.has_sink:
            specs[n["sink"]] = ParamSpec((H,), kind="vector", init="around_zero")
        specs[n["out"]] = ParamSpec((h, H * self.v_dim))
        return specs

    def load(self, tensors):
        n, H = self.names, self.num_heads
        rows = [tensors[n["dq" if self.q_rank else "q"]]]
        if self.own_kv:
            rows.append(tensors[n["dkv"]])
            self.kv_norm = tensors[n["dkv_norm"]]
        if self.gated:
            rows.append(tensors[n["gate"]])
        if self.has_sink:
            self.sink = tensors[n["sink"]].float().contiguous()
        spare = -sum(r.shape[0] for r in rows) % ROW_MULTIPLE
        if spare and not self.q_rank:
            rows.append(torch.zeros((spare, self.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        if self.q_rank:
            self.q_norm, self.w_uq = tensors[n["dq_norm"]], tensors[n["uq"]].contiguous()
        # per head: [head_dim, kv_rank] carries a query into the latent space, [kv_rank, v_dim] a latent mix out of it
        self.w_uk = tensors[n["uk"]].view(H, self.head_dim, self.kv_rank).contiguous()
        self.w_uv = tensors[n["uv"]].view(H, self.v_dim, self.kv_rank).transpose(1, 2).contiguous()
        self.w_o = tensors[n["out"]].contiguous()

    def forward(self, x, ctx, cache, residual=None):
        if cache.writes != self.own_kv:
            raise ValueError("latent_attention: a mixer with latents of its own writes its pages, one without reads "
                             "another position's (the schedule's cache_of)")
        group = ctx.groups[cache.group]
        rows = cache.tensors["latent"]
        H, D, R, rank = self.num_heads, self.head_dim, self.rot_dim, self.kv_rank
        x = ops.linear(x, self.w_in, status=ctx.status)
        tokens = x.shape[0]
        q_row = torch.empty((tokens, H * self.row), dtype=x.dtype, device=x.device)
        q_latent, gate = ops.latent_prep(
            x, ctx.positions, group.slot_mapping if self.own_kv else None, self.q_norm, self.kv_norm, self.inv_freq,
            rows if self.own_kv else None, q_rank=self.q_rank, kv_rank=rank, rot_dim=R, rotary_dims=self.rotary_dims,
            eps=self.norm_eps, factor=self.rotary_factor, q_rows=None if self.q_rank else q_row, heads=H, head_dim=D,
            has_kv=self.own_kv, gated=self.gated, status=ctx.status)
        if self.q_rank:
            q = ops.linear(q_latent, self.w_uq, status=ctx.status)                      # [tokens, H * (D + R)]
            if R:
                ops.rotate_pairs(q, q_row, ctx.positions, self.inv_freq, heads=H, cols=R, rotary_dims=self.rotary_dims,
                                 in_offset=D, out_offset=rank, factor=self.rotary_factor)
        else:
            q = x[:, :self.q_width]
        # the unrotated part of every head's query, carried into the latent space: [H, tokens, D] x [H, D, rank]
        torch.bmm(q.unflatten(1, (H, D + R))[:, :, :D].transpose(0, 1), self.w_uk,
                  out=q_row.view(tokens, H, self.row)[:, :, :rank].transpose(0, 1))
        mixed = torch.empty((tokens, H * rank), dtype=q.dtype, device=q.device)
        run_attention(ctx, group, q_row, rows, rows, mixed, num_heads=H, num_kv_heads=1, v_dim=rank, scale=self.scale,
                      window=self.window, gate=gate, sink=self.sink)
        out = torch.empty((tokens, H * self.v_dim), dtype=q.dtype, device=q.device)
        torch.bmm(mixed.view(tokens, H, rank).transpose(0, 1), self.w_uv,
                  out=out.view(tokens, H, self.v_dim).transpose(0, 1))              # [H, tokens, v_dim]
        if residual is not None:
            summed = ops.linear_into_residual(out, self.w_o, residual, status=ctx.status)
            if summed is not None:
                return summed
        return ops.linear(out, self.w_o, partial_ok=True, status=ctx.status)
