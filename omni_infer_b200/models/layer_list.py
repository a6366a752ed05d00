"""Models described layer by layer: ``ModelConfig.layers`` lists a mixer (windowed attention or Mamba-2) and an optional
gated feed-forward per layer, each with sizes of its own.

Sublayers read the residual stream itself and their outputs are normed before they are added to it:
``x <- x + norm1(mixer(x))``, ``x <- x + norm2(ff(x))``.  The residual is fp32; every addition, its norm and the activation
copy for the next sublayer are one kernel.  The embedding table is also the LM head.

A layer's entry in ``kv_caches`` is what its mixer reads: the (k, v) page pools of an attention layer - the same tensors
for a layer that attends to another layer's keys - or the (convolution, recurrence) slot tensors of a Mamba-2 layer."""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..layers.common import GeGLUMLP, PaddedLinear, PostNorm, _dtype
from ..layers.mamba2 import Mamba2Mixer
from ..layers.vocab_parallel import lm_logits
from ..layers.windowed_attention import WindowedAttention
from ..ops.layer_list import embed_residual, pad8, rmsnorm_residual
from .config import ModelConfig


class LayerListLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, i: int, *, dtype, device=None, cos_sin=None):
        super().__init__()
        s, width, eps = cfg.layers[i], cfg.hidden_size, cfg.rms_norm_eps
        if s.attention is not None:
            self.mixer = WindowedAttention(s.attention, width, eps, dtype=dtype, device=device, cos_sin=cos_sin)
        else:
            self.mixer = Mamba2Mixer(s.mamba2, width, eps, dtype=dtype, device=device)
        self.norm1 = PostNorm(width, eps, device)
        self.mlp = GeGLUMLP(width, s.ff, dtype=dtype, device=device) if s.ff else None
        self.norm2 = PostNorm(width, eps, device) if s.ff else None

    def forward(self, x, xa, md, cache):
        """x: fp32 residual (updated in place), xa: the same as activations; returns the new activations."""
        xa = self.norm1(self.mixer(xa, md, cache), x)
        return self.norm2(self.mlp(xa), x) if self.mlp is not None else xa


class LayerListModel(nn.Module):
    def __init__(self, cfg: ModelConfig, *, device=None):
        super().__init__()
        self.cfg, self.dtype = cfg, _dtype(cfg.dtype)
        tables: dict = {}

        def cos_sin(a):
            if a is None or a.rot_dims == 0:
                return None
            key = (a.rot_dims, a.rot_base, a.rot_factor)
            if key not in tables:
                tables[key] = ops.rope_cos_sin_table(a.rot_dims, cfg.max_position_embeddings, a.rot_base,
                                                     {"type": "linear", "factor": a.rot_factor}, device=device or "cpu")
            return tables[key]

        self.embed_tokens = nn.Embedding(cfg.vocab_size, pad8(cfg.hidden_size), dtype=self.dtype, device=device)
        self.embed_tokens.weight.requires_grad_(False)
        self.layers = nn.ModuleList([LayerListLayer(cfg, i, dtype=self.dtype, device=device, cos_sin=cos_sin(s.attention))
                                     for i, s in enumerate(cfg.layers)])
        self.norm = nn.Parameter(torch.ones(cfg.hidden_size, dtype=torch.float32, device=device), requires_grad=False)

    def forward(self, input_ids, md, kv_caches, inputs_embeds=None):
        assert inputs_embeds is None
        x, xa = embed_residual(input_ids, self.embed_tokens.weight)
        for layer, cache in zip(self.layers, kv_caches):
            xa = layer(x, xa, md, cache)
        return rmsnorm_residual(x, self.norm, self.cfg.rms_norm_eps, self.dtype)


class LayerListForCausalLM(nn.Module):
    is_mla = False

    def __init__(self, cfg: ModelConfig, *, device=None, planner=None):
        super().__init__()
        if not cfg.layers:
            raise ValueError(f"{cfg.architecture} needs the list of its layers in the model configuration")
        if cfg.quantization != "none":
            raise ValueError(f"{cfg.architecture} runs in bfloat16 or float32, not quantised")
        self.cfg = cfg
        self.model = LayerListModel(cfg, device=device)

    @property
    def num_kv_layers(self):
        """Layers that hold pages of their own."""
        return sum(s.attention is not None and s.attention.owns_kv for s in self.cfg.layers)

    def allocate_caches(self, num_blocks: int, block_size: int, state_slots: int, zeros) -> list:
        """One entry per layer (see the module text).  ``zeros(*shape, dtype=)`` allocates."""
        caches: list = []
        for s, layer in zip(self.cfg.layers, self.model.layers):
            a = s.attention
            if a is None:
                caches.append(tuple(zeros(*shape, dtype=dt) for shape, dt in layer.mixer.state_shapes(state_slots, self.model.dtype)))
            elif a.owns_kv:
                caches.append((zeros(num_blocks, block_size, a.kv_heads, a.dim, dtype=self.model.dtype),
                               zeros(num_blocks, block_size, a.kv_heads, a.vdim, dtype=self.model.dtype)))
            else:
                caches.append(caches[a.kv_from])
        return caches

    def kv_bytes_per_token(self) -> int:
        esz = torch.empty(0, dtype=self.model.dtype).element_size()
        return esz * sum(s.attention.cache_elems_per_token() for s in self.cfg.layers if s.attention is not None)

    def state_bytes(self, slots: int) -> int:
        """Bytes of recurrent state for ``slots`` requests."""
        total = 0
        for layer in self.model.layers:
            if isinstance(layer.mixer, Mamba2Mixer):
                for shape, dt in layer.mixer.state_shapes(slots, self.model.dtype):
                    total += torch.Size(shape).numel() * torch.empty(0, dtype=dt).element_size()
        return total

    def forward(self, input_ids, md, kv_caches, inputs_embeds=None):
        return self.model(input_ids, md, kv_caches, inputs_embeds)

    def compute_logits(self, hidden):
        return lm_logits(hidden, self.model.embed_tokens.weight)

    def process_weights_after_loading(self):
        """Padding rows and columns hold zeros whatever the loader or the random initialisation put there."""
        self.model.embed_tokens.weight.data[:, self.cfg.hidden_size:] = 0
        for m in self.modules():
            if isinstance(m, PaddedLinear):
                m.zero_padding()
        for m in self.modules():
            if isinstance(m, GeGLUMLP):
                m.zero_padding()

    def should_use_eager_mode(self, md):
        return md.is_prefill

    # ------------------------------------------------------------------ checkpoint names
    def checkpoint_targets(self) -> dict:
        """{checkpoint tensor: (parameter, first row, rows, columns)} for the weight loader."""
        H = self.cfg.hidden_size
        out = {"embed": (self.model.embed_tokens.weight, 0, self.cfg.vocab_size, H), "final.norm": (self.model.norm, 0, H, None)}
        for i, layer in enumerate(self.model.layers):
            p = f"l{i}."
            out[p + "norm1"] = (layer.norm1.weight, 0, H, None)
            out.update({p + "mix." + k: v for k, v in layer.mixer.checkpoint_targets().items()})
            if layer.mlp is not None:
                m, w = layer.mlp, layer.mlp.gate_up_proj.weight
                out[p + "norm2"] = (layer.norm2.weight, 0, H, None)
                out[p + "mlp.gate"], out[p + "mlp.up"] = (w, 0, m.inter, H), (w, m.block, m.inter, H)
                out[p + "mlp.down"] = (m.down_proj.weight, 0, H, m.inter)
        return out

    def load_weights(self, weights, planner=None) -> set:
        from ..quantization.loader import WeightLoader
        return WeightLoader(self, self.cfg, planner=planner).load(weights)
