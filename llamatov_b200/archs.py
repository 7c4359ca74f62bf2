"""Registry of the model architectures the engine runs.

The token step (`dev_residency.forward_pass_resident`), the prompt pass (`prefill.prefill_resident`), the graph
runner and `llamatov_run.generate` walk the layer runs of a model and leave to its `Architecture` what a layer does
and what it keeps per sequence.  An architecture is found by the name in `cfg["arch"]`: the GGUF key
general.architecture, or "architecture" of a config.json.
"""
import collections
import importlib

# One pass through one layer.  `slot` is its index in the list of per-sequence caches; a layer that runs several times
# (a loop) has a slot per pass.  `loop_pass` is the number of the pass, None outside a loop; `opens_pass` marks the
# first layer of a pass.
Run = collections.namedtuple("Run", "layer slot loop_pass opens_pass")

_REGISTRY = {
    "llama": "llamatov_b200.q8_block:ARCH",
    "qwen2": "llamatov_b200.q8_block:ARCH",
    "Nugusun": "llamatov_b200.layered:ARCH",
    "Pakalix": "llamatov_b200.layered:PAKALIX",
}


class Architecture:
    """What the engine asks of a model family.

    Per sequence the engine holds one cache object per run (`n_slots`), made by `new_cache` when the run is first
    reached.  Every cache has `length`, the positions it has taken in, and `reset()`, which empties it for the next
    sequence.
    """
    fused_step = False      # the whole token step exists as a fused launch (dev_residency.FusedDecodeStep)
    device_token = False    # the token step gathers the embedding row from a token id in device memory

    def runs(self, cfg):
        return [Run(i, i, None, False) for i in range(cfg["n_layers"])]

    def n_slots(self, cfg):
        return len(self.runs(cfg))

    def config_from_json(self, js, dtype):
        raise NotImplementedError("this architecture is read from GGUF files")

    def weights_from_safetensors(self, tensors, cfg):
        raise NotImplementedError("this architecture is read from GGUF files")

    def new_cache(self, w, cfg, run):
        raise NotImplementedError

    # ---- one token
    def ensure_buffers(self, w, cfg):
        """Settle every fixed buffer the captured step will use."""
        raise NotImplementedError

    def embed_step(self, w, cfg, tok):
        """Embedding row of the token; returns the residual stream handle the layers pass on."""
        raise NotImplementedError

    def layer_step(self, w, cfg, run, x, cache):
        raise NotImplementedError

    def logits_step(self, w, cfg, x):
        """Logits into the fixed logits buffer."""
        raise NotImplementedError

    # ---- rows of a prompt portion
    max_rows = 0

    def rows_supported(self, w, cfg):
        raise NotImplementedError

    def rows_begin(self, w, cfg, toks):
        """toks [B, T]; returns the state the layers work on."""
        raise NotImplementedError

    def layer_rows(self, st, run, caches):
        raise NotImplementedError

    def rows_residual(self, st):
        """The residual stream as an fp32 tensor [rows, n_embd]."""
        raise NotImplementedError

    def rows_end(self, st):
        """After the last layer, wanted logits or not."""

    def rows_logits(self, st, rows):
        """fp32 tensor [len(rows), vocab] on the host for the given row numbers."""
        raise NotImplementedError


def by_name(name):
    if name not in _REGISTRY:
        raise NotImplementedError(f"architecture {name!r}: known are {', '.join(sorted(_REGISTRY))}")
    mod, attr = _REGISTRY[name].split(":")
    return getattr(importlib.import_module(mod), attr)


def of(cfg):
    return by_name(cfg.get("arch", "llama"))
