"""The llama / qwen2 block with Q8_0 weights: attention with rotary positions over an fp32 KV cache, gated
feed-forward.  One token: bpd/lib/dev_residency.py:1381-1477 per layer, every op a launch of the per-op interface
(`dev_residency`); a prompt portion: the same arithmetic on all rows at once, GEMMs on the tensor cores."""
import numpy as np
import torch

from . import _lib, archs
from . import dev_residency as dr
from .fact_dispatch import Q8Weight


class _Rows:
    """State of a prompt pass."""


class Q8Block(archs.Architecture):
    fused_step = True
    # Rows per pass.  The activations of a pass stay resident (a [rows, 2F] fp32 gate|up buffer is the largest);
    # 16384 rows of the 0.5B architecture are 0.6 GB.
    max_rows = 16384

    def new_cache(self, w, cfg, run):
        return dr.DeviceKVCache(dr._KV_MAX_SEQ, cfg["n_head_kv"], cfg["n_embd"] // cfg["n_head"])

    # ------------------------------------------------------------------ one token
    def ensure_buffers(self, w, cfg):
        E = cfg["n_embd"]
        dr._ensure_resid(E)
        dr._ensure_logits_buf(E, w)
        dr._ensure_logits_scratch(E)

    def embed_step(self, w, cfg, tok):
        E = cfg["n_embd"]
        resid_in, _carry = dr._ensure_resid(E)
        if dr._DEVICE_EMBED is not None:
            # on-device token loop: the row is gathered from the Q8_0 table by the token id that
            # the previous step's argmax left in device memory
            dWq, dWd, tok_ptr, V = dr._DEVICE_EMBED
            _lib.call("lt_embed_q8", dWq, dWd, tok_ptr, resid_in.ptr, E, V, dr._stream())
        elif not dr._capturing():
            row = dr._embedding_row(w, int(tok.reshape(-1)[0]), E)
            dr._memcpy_htod(resid_in.ptr, row, E * 4)
            torch.cuda.current_stream().synchronize()      # `row` is pageable host memory
        return resid_in

    def layer_step(self, w, cfg, run, xd, cache):
        nh, nkv = cfg["n_head"], cfg["n_head_kv"]
        hd = cfg["n_embd"] // nh
        eps = cfg["norm_eps"]
        _in, carry = dr._ensure_resid(cfg["n_embd"])
        p = f"blk.{run.layer}"
        hdv = dr.rms_norm_dev(xd, dr._np(w[f"{p}.attn_norm.weight"]), eps)
        qd, kd, vd = dr.qkv_fused_dev(hdv, w, p)
        lp = cache._ensure_len_ptr(seed=not dr._capturing())
        # position = length before the append; attention sees the length after it
        dr.rope_dev_qk_fused(qd.ptr, lp, nh, nkv, hd, cfg["rope_theta"])
        cache.append_at_len_incr(kd.ptr, vd.ptr)
        cache.length += 1
        yd = dr.attn_decode_from_cache_masked(qd.ptr, cache, nh, hd ** -0.5, lp, cache.max_seq)
        xres = dr.q8_linear_add_residual_dev(yd, w[f"{p}.attn_output.weight"], xd)
        h2 = dr.rms_norm_dev(xres, dr._np(w[f"{p}.ffn_norm.weight"]), eps)
        g, u = dr.gateup_fused_dev(h2, w, p)
        dr.q8_linear_add_residual_dev(g, w[f"{p}.ffn_down.weight"], xres, out=carry, silu_src=(g, u))
        dr.free_scratch()
        return carry

    def logits_step(self, w, cfg, x):
        dr._compute_folded_logits(w, cfg, cfg["n_embd"])

    # ------------------------------------------------------------------ rows
    def rows_supported(self, w, cfg):
        """The batched path needs row lengths that the tiled weight loads accept and a head size
        the chunk attention is built for; anything else prefills token by token."""
        E = cfg["n_embd"]
        hd = E // cfg["n_head"]
        F = dr._fused_gateup_weight(w, "blk.0")[2][0]
        return E % 128 == 0 and F % 128 == 0 and (cfg["n_head"] * hd) % 128 == 0 and hd in (64, 128)

    def rows_begin(self, w, cfg, toks):
        st = _Rows()
        st.w, st.cfg = w, cfg
        st.B, st.T = int(toks.shape[0]), int(toks.shape[1])
        R = st.R = st.B * st.T
        E = cfg["n_embd"]
        nh, nkv = cfg["n_head"], cfg["n_head_kv"]
        hd = E // nh
        nq, nk = nh * hd, nkv * hd
        f32 = dict(dtype=torch.float32, device="cuda")
        st.x = _embedding_rows(w, toks.reshape(-1), E)                  # residual stream [R, E]
        st.x1 = torch.empty((R, E), **f32)
        st.h = torch.empty((R, E), **f32)
        F = st.F = dr._fused_gateup_weight(w, "blk.0")[2][0]
        st.qkv = torch.empty((R, nq + 2 * nk), **f32)
        st.att = torch.empty((R, nq), **f32)
        st.gu = torch.empty((R, 2 * F), **f32)
        kmax = max(E, nq, F)
        st.xq = torch.empty(R * kmax, dtype=torch.int8, device="cuda")
        st.xd = torch.empty(R * (kmax // 32), dtype=torch.int16, device="cuda")
        return st

    def layer_rows(self, st, run, caches):
        w, cfg, B, T, R, F = st.w, st.cfg, st.B, st.T, st.R, st.F
        nh, nkv, E = cfg["n_head"], cfg["n_head_kv"], cfg["n_embd"]
        hd = E // nh
        nq, nk = nh * hd, nkv * hd
        eps, theta = float(cfg["norm_eps"]), float(cfg["rope_theta"])
        scale = float(np.float32(hd ** -0.5))
        x, x1, h, qkv, att, gu, xq, xd = st.x, st.x1, st.h, st.qkv, st.att, st.gu, st.xq, st.xd
        s = dr._stream

        def gemm(Wt, K, N, y, resid=None, resid_ld=0):
            dWq, dWd, n_, k_ = dr._weights(Wt)
            assert n_ == N and k_ == K, (n_, N, k_, K)
            _lib.call("lt_q8_gemm_tc", dWq, dWd, xq.data_ptr(), xd.data_ptr(),
                      None if resid is None else dr._vp(resid), resid_ld, y.data_ptr(), N, K, R, 0, s())

        p = f"blk.{run.layer}"
        _lib.call("lt_rmsnorm", x.data_ptr(), dr._dev_const(dr._np(w[f"{p}.attn_norm.weight"])), h.data_ptr(),
                  R, E, eps, s())
        _lib.call("lt_quant_q8", h.data_ptr(), xq.data_ptr(), xd.data_ptr(), E, R, s())
        Wqkv, bcat, _ = dr._fused_qkv_weight(w, p)
        gemm(Wqkv, E, nq + 2 * nk, qkv, None if bcat is None else dr._dev_const(bcat), 0)
        for b, c in enumerate(caches):
            lp = c._ensure_len_ptr(seed=True)
            if c.length + T > c.max_seq:
                raise RuntimeError(f"KV cache overflow: {c.length}+{T} > {c.max_seq}")
            rows = qkv[b * T:(b + 1) * T]
            _lib.call("lt_rope_rows", rows.data_ptr(), nq + 2 * nk, lp, T, nh + nkv, hd, theta, s())
            _lib.call("lt_append_kv_rows", c.k_ptr, rows.data_ptr() + nq * 4, c.v_ptr,
                      rows.data_ptr() + (nq + nk) * 4, nq + 2 * nk, lp, c.width, c.max_seq, T, 1, s())
            c.length += T
            _lib.call("lt_attn_prefill", rows.data_ptr(), nq + 2 * nk, c.k_ptr, c.v_ptr, lp,
                      att[b * T:(b + 1) * T].data_ptr(), nq, hd, nh, nkv, scale, T, c.length, s())
        _lib.call("lt_quant_q8", att.data_ptr(), xq.data_ptr(), xd.data_ptr(), nq, R, s())
        gemm(dr._np(w[f"{p}.attn_output.weight"]), nq, E, x1, x.data_ptr(), E)
        _lib.call("lt_rmsnorm", x1.data_ptr(), dr._dev_const(dr._np(w[f"{p}.ffn_norm.weight"])), h.data_ptr(),
                  R, E, eps, s())
        _lib.call("lt_quant_q8", h.data_ptr(), xq.data_ptr(), xd.data_ptr(), E, R, s())
        Wgu, _b, (ng, _nu) = dr._fused_gateup_weight(w, p)
        gemm(Wgu, E, 2 * F, gu)
        _lib.call("lt_silu_mul_quant_rows", gu.data_ptr(), gu.data_ptr() + F * 4, 2 * F, xq.data_ptr(),
                  xd.data_ptr(), F, R, s())
        gemm(dr._np(w[f"{p}.ffn_down.weight"]), F, E, x, x1.data_ptr(), E)

    def rows_residual(self, st):
        return st.x

    def rows_end(self, st):
        # the last row's hidden state goes where the one-token path leaves it
        E = st.cfg["n_embd"]
        _rin, rout = dr._ensure_resid(E)
        dr._memcpy_dtod(dr._addr(rout.ptr), st.x[st.R - 1].data_ptr(), E * 4)

    def rows_logits(self, st, rows):
        w, cfg = st.w, st.cfg
        E = cfg["n_embd"]
        dr._ensure_logits_buf(E, w)
        dr._ensure_logits_scratch(E)
        _rin, rout = dr._ensure_resid(E)
        out = []
        for r in rows:
            dr._memcpy_dtod(dr._addr(rout.ptr), st.x[r].data_ptr(), E * 4)
            out.append(dr._compute_folded_logits(w, cfg, E).to_host())
        self.rows_end(st)
        return torch.from_numpy(np.stack(out))


def _embedding_rows(w, toks_flat, E):
    """[n, E] fp32 rows of the embedding table on the device."""
    n = int(toks_flat.numel())
    out = torch.empty((n, E), dtype=torch.float32, device="cuda")
    emb = w["token_embd.weight"]
    if isinstance(dr._np(emb), Q8Weight):
        dWq, dWd, V, _ = dr._weights(dr._np(emb))
        dt = toks_flat.to(device="cuda", dtype=torch.int32)
        _lib.call("lt_embed_q8_rows", dWq, dWd, dt.data_ptr(), out.data_ptr(), E, V, n, dr._stream())
        torch.cuda.current_stream().synchronize()
    else:
        rows = np.stack([dr._embedding_row(w, int(t), E) for t in toks_flat.tolist()])
        out.copy_(torch.from_numpy(rows))
    return out


ARCH = Q8Block()
