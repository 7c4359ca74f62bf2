"""Prompt prefill in one pass over the weights.

The reference prefills by running its one-token step once per prompt token
(`forward_pass_resident` recursing, bpd/lib/dev_residency.py:1344-1350) and demands that a
batched form give the same numbers.  `prefill_resident` here runs the same layer sequence
(bpd/lib/dev_residency.py:1381-1477) on all rows of a prompt chunk at once; what a layer does with
the rows is its architecture's (`archs`).  For the Q8_0 block that is row-batched RMSNorm /
quantiser / rope / append, the Q8_0 GEMMs on the tensor cores (`lt_q8_gemm_tc`) and causal
attention over the rows just appended (`lt_attn_prefill`): every row gets exactly the arithmetic
the one-token step would give it, so the KV cache, the final hidden state and the logits are
bit-identical to the token-by-token prefill (tests/test_gpu_prefill.py).

Several sequences can be prefilled together (`toks` of shape [B, T], one cache list per
sequence): the GEMMs then run over B*T rows, what depends on a sequence's cache per sequence.
"""
import torch

from . import archs
from . import dev_residency as dr

MAX_ROWS = 16384       # rows per pass of the Q8_0 block (archs.Architecture.max_rows of the others)


def supported(cfg, w):
    """Whether the architecture runs prompts as row batches; anything else prefills token by token."""
    return archs.of(cfg).rows_supported(w, cfg)


def prefill_resident(w, cfg, toks, kv_caches, want_logits=True, want_rows=None, tap=None):
    """Run a prompt (chunk) through all layers with batched rows.

    toks: int tensor [T] or [B, T].  kv_caches: the per-layer cache list of the sequence (or a
    list of B such lists); caches are created on first use exactly as the one-token path does.
    Positions continue from each cache's current length.  Returns the logits of the last row
    of the last sequence as a [1, 1, V] tensor, like `forward_pass_resident`; with `want_rows`
    (row numbers of the chunk) those rows' logits as [n, V].  `tap(run, x)` is called after every
    layer with the residual stream [rows, n_embd].
    """
    A = archs.of(cfg)
    if toks.dim() == 1:
        toks = toks.reshape(1, -1)
        kv_caches = [kv_caches]
    B, T = int(toks.shape[0]), int(toks.shape[1])
    if B * T > A.max_rows:
        raise RuntimeError(f"prefill_resident: {B}x{T} rows exceed {A.max_rows}; split the prompt in chunks")
    st = A.rows_begin(w, cfg, toks)
    for run in A.runs(cfg):
        for caches in kv_caches:
            if caches[run.slot] is None:
                caches[run.slot] = A.new_cache(w, cfg, run)
        A.layer_rows(st, run, [caches[run.slot] for caches in kv_caches])
        if tap is not None:
            tap(run, A.rows_residual(st))
    A.rows_end(st)
    if want_rows is not None:
        out = A.rows_logits(st, list(want_rows)) if len(want_rows) else None
        torch.cuda.synchronize()
        return out
    if not want_logits:
        torch.cuda.synchronize()
        return None
    out = A.rows_logits(st, [B * T - 1])
    torch.cuda.synchronize()
    return out.reshape(1, 1, -1)
