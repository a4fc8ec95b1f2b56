"""Causal attention whose keys and values are expanded from one shared latent per token.

Per token the cache keeps a single row for all heads: the RMS-normed latent ``c`` (``kv_rank``
numbers) and one rotated key part ``kr`` (``rot_dim`` numbers).  Head ``h`` has the key
``[W_uk[h] c | kr]`` and the value ``W_uv[h] c``; its query is ``[q_plain | q_rot]``.  Since
``q_plain . (W_uk[h] c) = (W_uk[h]^T q_plain) . c``, the kernels work on the latent directly:

    qa[h]  = W_uk[h]^T q_plain[h]                       (absorbed query, kv_rank numbers)
    score  = (qa[h] . c_j + q_rot[h] . kr_j) * scale    over j <= i (``window``: i - j < window)
    weight = softmax over the scores (``sink``: and one sink logit per head, no key, no value)
    out[h] = W_uv[h] (sum_j weight_j c_j)

Rotary positions act on pairs of the rotated parts: number 2i with 2i + 1, or with
``rot_pairing="halves"`` number i with i + rot_dims/2.  The kernels know the first form; for the
second the rows of the matrices that make the rotated parts change places once, at binding (query
and key parts alike, so their products are the same), and cache rows hold the parts in that order.

``gate`` names a matrix of the input: every head's output is multiplied, element by element, by
the sigmoid of its columns before the output projection.

A layer built with
``shares_cache`` has no latent projection: it reads the rows another layer call wrote (the
schedule names the entry) with its own queries, expansions and sink.

Prompt portions may run in the other form (``latent_prompt_rows``): the latents of the positions
they see are expanded to keys and values per head by one product, and the portion attends to those
(dim + rot_dim and vdim numbers a query and key instead of 2 * kv_rank + rot_dim).

With ``q_down`` the queries come through a latent of their own: ``c_q = rms_norm(W_dq h)`` of
``q_rank`` numbers, formed in the launch that writes the cache row (both latents are columns of
one input projection), and the query matrix maps c_q instead of h.
"""

from __future__ import annotations

import torch

from .base import CacheRequest, Mixer, TensorRequest, register_mixer


class LatentAttention(Mixer):
    def __init__(self, *, width: int, n_heads: int, dim: int, rot_dim: int, vdim: int,
                 kv_rank: int, scale: float, rot_base: float, rot_dims: int, eps: float,
                 q_weight: str, latent_weight: str | None, latent_norm: str | None,
                 key_up: str, value_up: str, sink: str | None, out_weight: str,
                 shares_cache: bool = False, window: int = 0, q_down: str | None = None,
                 q_down_norm: str | None = None, q_rank: int = 0,
                 rot_pairing: str = "interleaved", gate: str | None = None):
        if rot_pairing not in ("interleaved", "halves"):
            raise ValueError(f"rotated pairs are interleaved or halves, got {rot_pairing!r}")
        if rot_dims % 2 or not 0 <= rot_dims <= rot_dim:
            raise ValueError(f"rot_dims must be even and at most rot_dim, got {rot_dims}")
        if shares_cache == (latent_weight is not None):
            raise ValueError("a layer either projects its own latent or shares another's")
        if (q_down is None) != (q_down_norm is None) or (q_down is None) != (q_rank == 0):
            raise ValueError("a query latent has a matrix, a norm and a size")
        if q_down is not None and shares_cache:
            raise ValueError("a layer that shares a latent projects its queries directly")
        if window < 0:
            raise ValueError("a window is not negative")
        self.window, self.q_rank = int(window), int(q_rank)
        self.width, self.H, self.D, self.P, self.V, self.R = (width, n_heads, dim, rot_dim, vdim,
                                                              kv_rank)
        self.scale = float(torch.tensor(float(scale), dtype=torch.float64).to(torch.float32))
        self.rot_base, self.rot_dims, self.eps = float(rot_base), int(rot_dims), float(eps)
        self.names = dict(q=q_weight, dkv=latent_weight, dkv_norm=latent_norm, uk=key_up,
                          uv=value_up, sink=sink, o=out_weight, dq=q_down, dq_norm=q_down_norm,
                          g=gate)
        self.rot_pairing = rot_pairing
        # without a window, prompts in expanded form need a row for every position they see
        self.counts_prompt_rows = self.window == 0 and sink is None
        self.shares_cache = bool(shares_cache)
        self.q_width = self.H * (self.D + self.P)
        # columns of the input projection: the queries or their latent, then the key/value latent
        self.head_width = self.q_rank or self.q_width
        self.in_width = self.head_width + (0 if shares_cache else self.R + self.P)
        # ... then the gate's, and zeros up to whole 16-byte pieces of a row
        self.gate_off, self.pad = self.in_width, 0
        if gate:
            self.in_width += self.H * self.V
            self.pad = -self.in_width % 8
            self.in_width += self.pad

    def tensor_requests(self):
        n = self.names
        req = {n["q"]: TensorRequest((self.q_width, self.q_rank or self.width), "matrix"),
               n["uk"]: TensorRequest((self.H * self.D, self.R), "matrix"),
               n["uv"]: TensorRequest((self.H * self.V, self.R), "matrix"),
               n["o"]: TensorRequest((self.width, self.H * self.V), "matrix")}
        if n["sink"]:
            req[n["sink"]] = TensorRequest((self.H,), "vector")
        if n["g"]:
            req[n["g"]] = TensorRequest((self.H * self.V, self.width), "matrix")
        if n["dq"]:
            req[n["dq"]] = TensorRequest((self.q_rank, self.width), "matrix")
            req[n["dq_norm"]] = TensorRequest((self.q_rank,), "vector")
        if not self.shares_cache:
            req[n["dkv"]] = TensorRequest((self.R + self.P, self.width), "matrix")
            req[n["dkv_norm"]] = TensorRequest((self.R,), "vector")
        return req

    def _paired(self, rows):
        """A [.., P, in] block of rows that make a rotated part, in the order the kernels turn."""
        if self.rot_pairing == "interleaved" or not self.rot_dims:
            return rows
        half = torch.arange(self.rot_dims // 2, device=rows.device)
        order = torch.cat([torch.stack([half, half + self.rot_dims // 2], 1).reshape(-1),
                           torch.arange(self.rot_dims, self.P, device=rows.device)])
        return rows[..., order, :]

    def bind(self, tensors):
        n = self.names
        wq = tensors[n["q"]]
        if self.rot_pairing != "interleaved":
            heads = wq.view(self.H, self.D + self.P, wq.shape[1])
            wq = torch.cat([heads[:, :self.D], self._paired(heads[:, self.D:])], 1).reshape(wq.shape)
        # one input projection: the queries (or the latent they come through), then (for a layer
        # with a latent of its own) the latent and the shared key part
        first = tensors[n["dq"]] if n["dq"] else wq
        rows = [first]
        if not self.shares_cache:
            dkv = tensors[n["dkv"]]
            rows += [dkv[:self.R], self._paired(dkv[self.R:])]
        if n["g"]:
            rows.append(tensors[n["g"]])
        if self.pad:
            rows.append(first.new_zeros(self.pad, self.width))
        self.w_in = torch.cat(rows).contiguous() if len(rows) > 1 else first.contiguous()
        self.w_q_up = wq if n["dq"] else None
        self.q_norm_w = tensors[n["dq_norm"]] if n["dq"] else None
        self.norm_w = None if self.shares_cache else tensors[n["dkv_norm"]]
        # k-major per head: [H, D, R] maps q_plain to the latent, [H, R, V] maps it to a value
        self.w_absorb = tensors[n["uk"]].view(self.H, self.D, self.R).contiguous()
        self.w_expand = tensors[n["uv"]].view(self.H, self.V, self.R).transpose(1, 2).contiguous()
        # the same two, [H, out, in], for the tensor-core form that prompt portions take
        self.w_absorb_nk = self.w_expand_nk = None
        if wq.dtype == torch.bfloat16:
            self.w_absorb_nk = self.w_absorb.transpose(1, 2).contiguous()
            self.w_expand_nk = tensors[n["uv"]].view(self.H, self.V, self.R).contiguous()
        # both expansions as one matrix, for the dense rows of prompt portions
        self.w_kv = None
        if wq.dtype == torch.bfloat16 and not n["sink"]:
            self.w_kv = torch.cat([tensors[n["uk"]], tensors[n["uv"]]]).contiguous()
        self.sink = tensors[n["sink"]] if n["sink"] else None
        self.w_out = tensors[n["o"]]
        i = torch.arange(self.rot_dims // 2, dtype=torch.float64)
        freq = torch.pow(torch.tensor(self.rot_base, dtype=torch.float64),
                         -2.0 * i / max(1, self.rot_dims))
        self.freq = freq.to(torch.float32).to(wq.device)

    def cache_request(self):
        return CacheRequest(kv_heads=1, head_dim=self.R + self.P, window=self.window, planes=1)

    writes_fresh = True

    def forward(self, ctx, h, x, cache, fresh=False):
        ops, T = ctx.ops, h.shape[0]
        H, D, P, V, R = self.H, self.D, self.P, self.V, self.R
        proj = ctx.buffer("latent_proj", (T, self.in_width), torch.float32)
        ops.linear(proj, h, self.w_in)
        # both rotations are fused: the key part turns as it is written to the page, the query
        # parts as the attention kernel reads them
        rot = dict(freq=self.freq, rot_dims=self.rot_dims) if self.rot_dims else {}
        if cache.writes:
            if self.shares_cache:
                raise RuntimeError("a layer that shares a latent cache cannot write it")
            more = dict(rot)
            if self.q_rank:                      # the query latent's norm rides along
                cq = ctx.buffer("latent_cq", (T, self.q_rank), ctx.dtype)
                more.update(q_out=cq, q_norm=self.q_norm_w)
            ops.latent_append(cache.pool, proj, self.norm_w, cache.table, ctx.tok_pos,
                              ctx.tok_req, c_offset=self.head_width, rank=R, rot_dim=P,
                              eps=self.eps, page_size=cache.page_size, status=ctx.status, **more)
        q = proj
        if self.q_rank:
            q = ctx.buffer("latent_q", (T, self.q_width), torch.float32)
            ops.linear(q, cq, self.w_q_up)
        att = ctx.buffer("latent_heads", (T, H * V), ctx.dtype)
        gate = dict(gate=proj, gate_offset=self.gate_off) if self.names["g"] else {}
        only = {}
        rows = self._prompt_rows(ctx)
        if rows:
            self._prompt_portions(ctx, att, q, cache, rows, rot, gate)
            if ctx.plan.decode_cap == 0:         # no single-query token in this step
                ops.linear(x, att, self.w_out, None, residual=None if fresh else x)
                return
            only = {"singles": ctx.plan}
        qa = ctx.buffer("latent_qa", (T, H * R), torch.float32)
        ops.grouped_linear(qa, q, self.w_absorb, a_offset=0, a_group_stride=D + P,
                           w_nk=self.w_absorb_nk, parts=8, **only)
        lat = ctx.buffer("latent_mix", (T, H * R), torch.float32)
        if self.window:
            rot["window"] = self.window
        if only:
            rot["singles_only"] = True
        ops.latent_attention(lat, qa, q, cache.pool, cache.table, ctx.tok_pos, ctx.tok_req,
                             self.sink, n_heads=H, rank=R, rot_dim=P, qr_head_stride=D + P,
                             qr_offset=D, scale=self.scale, page_size=cache.page_size,
                             status=ctx.status, plan=ctx.plan, **rot)
        ops.grouped_linear(att, lat, self.w_expand, w_nk=self.w_expand_nk, parts=8, **only, **gate)
        ops.linear(x, att, self.w_out, None, residual=None if fresh else x)

    def _prompt_rows(self, ctx) -> int:
        """Dense rows the step's prompt portions need in expanded form; 0: not in that form."""
        takes = getattr(ctx.ops, "latent_prompt_rows", None)
        if self.w_kv is None or takes is None:
            return 0
        return takes(ctx.plan, ctx.n_requests, n_heads=self.H, dim=self.D, rot_dim=self.P,
                     vdim=self.V, rank=self.R, window=self.window, scale=self.scale)

    def _prompt_portions(self, ctx, att, q, cache, rows, rot, gate):
        ops, T = ctx.ops, q.shape[0]
        H, D, P, V, R = self.H, self.D, self.P, self.V, self.R
        lat = ctx.buffer("latent_dense", (rows, R), ctx.dtype)
        rope = ctx.buffer("latent_dense_rot", (rows, 64), ctx.dtype)
        qp = ctx.buffer("latent_q_padded", (T, H * (-(-D // 64) * 64 + 64)), ctx.dtype)
        base = ctx.buffer("latent_base", (ctx.n_requests,), torch.int32)
        ops.latent_gather(lat, rope, qp, base, q, cache.pool, cache.table, ctx.req_start,
                          ctx.req_len, ctx.tok_pos, ctx.tok_req, n_heads=H, dim=D, rank=R,
                          rot_dim=P, window=self.window, page_size=cache.page_size,
                          status=ctx.status, **rot)
        kv = ctx.buffer("latent_expanded", (rows, H * (D + V)), ctx.dtype)
        ops.linear(kv, lat, self.w_kv)
        ops.latent_prompt_attention(att, qp, kv, rope, base, ctx.plan, n_heads=H, dim=D, rot_dim=P,
                                    vdim=V, rank=R, window=self.window, scale=self.scale,
                                    status=ctx.status, **gate)


register_mixer("latent_attention", LatentAttention)
