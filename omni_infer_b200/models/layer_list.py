"""Models described layer by layer: ``ModelConfig.layers`` lists a mixer and an optional feed-forward per layer, each with sizes
of its own.  Four ways to connect them:

One residual, norms on the outputs (``cfg.streams == 0``; windowed attention, Mamba-2, gated dense feed-forward): sublayers read
the residual stream itself, ``x <- x + norm1(mixer(x))``, ``x <- x + norm2(ff(x))``.  Every addition, its norm and the activation
copy for the next sublayer are one kernel.

Residual streams, norms ahead (attention beside a matrix memory, WKV, mixture of experts): a sublayer reads the layer norm of a
learned sum of the streams, and every stream becomes a learned sum of all of them and the sublayer's output.  Update, sum and
norm for the next sublayer are one kernel.  A layer may run with another layer's weights (``weights_of``) on a cache or state
of its own.

One residual, norms ahead (``cfg.norm_first``; latent, windowed and chunked attention, dense feed-forwards and mixtures of
experts): ``x <- x + mixer(norm1(x))``, ``x <- x + ff(norm2(x))``.  Addition, output bias and the norm for the next sublayer are
one kernel.  The head is a matrix of its own; its factor enters with the last norm.

One residual, norms on both sides (``cfg.norm_both``; latent attention, windowed attention, gated linear attention, dense
feed-forwards and mixtures of experts): ``x <- x + m norm1b(mixer(norm1(x)))``, ``x <- x + m norm2b(ff(norm2(x)))``, learned positions
added to the embeddings, and after every layer a learned average of the embedding output and all layers' results so far.  Norm
behind, addition, average and the norm for the next sublayer are one kernel.

The residual is fp32 in all of them, and the embedding table is also the LM head in the first two.

A layer's entry in ``kv_caches`` is what its mixer reads: the (k, v) page pools of an attention layer - the same tensors for a
layer that attends to another layer's keys, one pool for latent attention - or the slot tensors of a recurrent one, or both."""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..layers.common import GeGLUMLP, PaddedLinear, PostNorm, _dtype
from ..layers.latent_attention import LatentAttention
from ..layers.mamba2 import Mamba2Mixer
from ..layers.matrix_state import GlaMixer, ParallelMixer, WkvMixer
from ..layers.moe import ExpertMixture
from ..layers.vocab_parallel import lm_logits
from ..layers.windowed_attention import WindowedAttention
from ..ops.depth import both_norms_step, embed_positions
from ..ops.layer_list import add_norm, embed_norm, embed_residual, pad8, rmsnorm_residual
from ..ops.streams import embed_streams, stream_step
from .config import ModelConfig


def _mixer(s, width, eps, **kw):
    cos_sin = kw.pop("cos_sin")
    if s.latent is not None:
        return LatentAttention(s.latent, width, eps, cos_sin=cos_sin, **kw)
    if s.attention is not None:
        return WindowedAttention(s.attention, width, eps, cos_sin=cos_sin, **kw)
    if s.parallel is not None:
        return ParallelMixer(s.parallel, width, eps, cos_sin=cos_sin, **kw)
    if s.wkv is not None:
        return WkvMixer(s.wkv, width, eps, **kw)
    if s.gla is not None:
        return GlaMixer(s.gla, width, eps, **kw)
    return Mamba2Mixer(s.mamba2, width, eps, **kw)


class LayerListLayer(nn.Module):
    """One residual, norms on the outputs."""

    def __init__(self, cfg: ModelConfig, i: int, *, dtype, device=None, cos_sin=None):
        super().__init__()
        s, width, eps = cfg.layers[i], cfg.hidden_size, cfg.rms_norm_eps
        self.mixer = _mixer(s, width, eps, dtype=dtype, device=device, cos_sin=cos_sin)
        self.norm1 = PostNorm(width, eps, device)
        self.mlp = GeGLUMLP(width, s.ff, dtype=dtype, device=device) if s.ff else None
        self.norm2 = PostNorm(width, eps, device) if s.ff else None

    def forward(self, x, xa, md, cache):
        """x: fp32 residual (updated in place), xa: the same as activations; returns the new activations."""
        xa = self.norm1(self.mixer(xa, md, cache), x)
        return self.norm2(self.mlp(xa), x) if self.mlp is not None else xa

    def checkpoint_targets(self):
        H = self.norm1.weight.shape[0]
        out = {"norm1": (self.norm1.weight, 0, H, None)}
        out.update({"mix." + k: v for k, v in self.mixer.checkpoint_targets().items()})
        if self.mlp is not None:
            out["norm2"] = (self.norm2.weight, 0, H, None)
            out.update({"mlp." + k: v for k, v in self.mlp.checkpoint_targets().items()})
        return out


class StreamLink(nn.Module):
    """How a sublayer hangs on the streams: weights of its input sum and norm, and of the update with its output."""

    def __init__(self, streams: int, width: int, device=None):
        super().__init__()
        par = lambda v: nn.Parameter(v.to(torch.float32).to(device or "cpu"), requires_grad=False)      # noqa: E731
        self.inw, self.out, self.mix = par(torch.full((streams,), 1.0 / streams)), par(torch.ones(streams)), par(torch.eye(streams))
        self.norm = par(torch.ones(width))
        for p in (self.inw, self.out, self.mix):
            p.init_value = p.data.clone()

    def checkpoint_targets(self, q: int):
        n = self.inw.shape[0]
        return {f"norm{q}": (self.norm, 0, self.norm.shape[0], None), f"hc{q}.in": (self.inw, 0, n, None),
                f"hc{q}.out": (self.out, 0, n, None), f"hc{q}.mix": (self.mix, 0, n, n)}


class StreamLayer(nn.Module):
    """Residual streams, norms ahead.  The model runs the sublayers; this holds their weights."""

    def __init__(self, cfg: ModelConfig, i: int, *, dtype, device=None, cos_sin=None):
        super().__init__()
        s, width = cfg.layers[i], cfg.hidden_size
        self.mixer = _mixer(s, width, cfg.rms_norm_eps, dtype=dtype, device=device, cos_sin=cos_sin)
        self.link1 = StreamLink(cfg.streams, width, device)
        self.mlp = ExpertMixture(s.experts, width, dtype=dtype, device=device) if s.experts is not None else None
        self.link2 = StreamLink(cfg.streams, width, device) if s.experts is not None else None

    def checkpoint_targets(self):
        out = self.link1.checkpoint_targets(1)
        out.update({"mix." + k: v for k, v in self.mixer.checkpoint_targets().items()})
        if self.mlp is not None:
            out.update(self.link2.checkpoint_targets(2))
            out.update({"mlp." + k: v for k, v in self.mlp.checkpoint_targets().items()})
        return out


class NormFirstLayer(nn.Module):
    """One residual, norms ahead.  The model runs the sublayers; this holds their weights."""

    def __init__(self, cfg: ModelConfig, i: int, *, dtype, device=None, cos_sin=None):
        super().__init__()
        s, width = cfg.layers[i], cfg.hidden_size
        norm = lambda: nn.Parameter(torch.ones(width, dtype=torch.float32, device=device), requires_grad=False)      # noqa: E731
        self.mixer, self.norm1 = _mixer(s, width, cfg.rms_norm_eps, dtype=dtype, device=device, cos_sin=cos_sin), norm()
        self.mlp, self.norm2 = None, None
        if s.experts is not None:
            self.mlp, self.norm2 = ExpertMixture(s.experts, width, dtype=dtype, device=device), norm()
        elif s.ff:
            self.mlp, self.norm2 = GeGLUMLP(width, s.ff, dtype=dtype, device=device, epi=s.act, bias=s.ff_bias), norm()

    def checkpoint_targets(self):
        H = self.norm1.shape[0]
        out = {"norm1": (self.norm1, 0, H, None)}
        out.update({"mix." + k: v for k, v in self.mixer.checkpoint_targets().items()})
        if self.mlp is not None:
            out["norm2"] = (self.norm2, 0, H, None)
            out.update({"mlp." + k: v for k, v in self.mlp.checkpoint_targets().items()})
        return out


class NormBothLayer(NormFirstLayer):
    """One residual, norms on both sides, an average over depth behind.  The model runs the sublayers; this holds their weights,
    those of the norms complete (``norm_offset`` added)."""

    def __init__(self, cfg: ModelConfig, i: int, *, dtype, device=None, cos_sin=None):
        super().__init__(cfg, i, dtype=dtype, device=device, cos_sin=cos_sin)
        self.offset = cfg.norm_offset
        norm = lambda: nn.Parameter(torch.ones(cfg.hidden_size, dtype=torch.float32, device=device), requires_grad=False)      # noqa: E731
        self.norm1b, self.norm2b = norm(), norm() if self.mlp is not None else None
        self.dwa = None
        if cfg.depth_average:
            self.dwa = nn.Parameter(torch.zeros(i + 2, dtype=torch.float32, device=device), requires_grad=False)
            self.dwa.data[-1] = 1.0
            self.dwa.init_value = self.dwa.data.clone()

    def checkpoint_targets(self):
        out = super().checkpoint_targets()
        for name in ("norm1", "norm1b", "norm2", "norm2b"):
            if getattr(self, name) is not None:
                out[name] = _offset_target(getattr(self, name), self.offset)
        if self.dwa is not None:
            out["dwa"] = (self.dwa, 0, self.dwa.shape[0], None)
        return out


def _offset_target(p, offset: float):
    """Checkpoint target of a norm weight that is stored without its offset."""
    def store(w):
        p.data.copy_(w.float() + offset)
    return store, tuple(p.shape)


class LayerListModel(nn.Module):
    def __init__(self, cfg: ModelConfig, *, device=None):
        super().__init__()
        self.cfg, self.dtype = cfg, _dtype(cfg.dtype)
        tables: dict = {}

        def cos_sin(a):
            if a is None or a.rot_dims == 0:
                return None
            scaling = a.rot_scaling or {"type": "linear", "factor": a.rot_factor}
            key = (a.rot_dims, a.rot_base, tuple(sorted(scaling.items())))
            if key not in tables:
                tables[key] = ops.rope_cos_sin_table(a.rot_dims, cfg.max_position_embeddings, a.rot_base, scaling,
                                                     device=device or "cpu")
            return tables[key]

        self.embed_tokens = nn.Embedding(cfg.vocab_size, pad8(cfg.hidden_size), dtype=self.dtype, device=device)
        self.embed_tokens.weight.requires_grad_(False)
        self.pos_embedding = None
        if cfg.learned_positions:
            self.pos_embedding = nn.Parameter(torch.zeros(cfg.learned_positions, pad8(cfg.hidden_size), dtype=self.dtype, device=device),
                                              requires_grad=False)
        kind = (StreamLayer if cfg.streams else NormFirstLayer if cfg.norm_first else NormBothLayer if cfg.norm_both
                else LayerListLayer)
        built: list = []
        for i, s in enumerate(cfg.layers):      # a layer with another's weights is that layer's module
            built.append(None if s.weights_of is not None else
                         kind(cfg, i, dtype=self.dtype, device=device, cos_sin=cos_sin(s.paged)))
        self.layers = nn.ModuleList([built[i if s.weights_of is None else s.weights_of] for i, s in enumerate(cfg.layers)])
        self.norm = nn.Parameter(torch.ones(cfg.hidden_size, dtype=torch.float32, device=device), requires_grad=False)
        if cfg.streams:
            self.register_buffer("every_stream", torch.ones(cfg.streams, dtype=torch.float32, device=device), persistent=False)

    def forward(self, input_ids, md, kv_caches, inputs_embeds=None):
        assert inputs_embeds is None
        if self.cfg.streams:
            return self._forward_streams(input_ids, md, kv_caches)
        if self.cfg.norm_first:
            return self._forward_norm_first(input_ids, md, kv_caches)
        if self.cfg.norm_both:
            return self._forward_norm_both(input_ids, md, kv_caches)
        x, xa = embed_residual(input_ids, self.embed_tokens.weight)
        for layer, cache in zip(self.layers, kv_caches):
            xa = layer(x, xa, md, cache)
        return rmsnorm_residual(x, self.norm, self.cfg.rms_norm_eps, self.dtype)

    def _forward_streams(self, input_ids, md, kv_caches):
        eps = self.cfg.rms_norm_eps
        subs = []
        for layer, cache in zip(self.layers, kv_caches):
            subs.append((layer.link1, lambda h, m=layer.mixer, c=cache: m(h, md, c)))
            if layer.mlp is not None:
                subs.append((layer.link2, lambda h, m=layer.mlp: m(h, md.num_valid)))
        first = subs[0][0]
        x, h = embed_streams(input_ids, self.embed_tokens.weight, self.cfg.hidden_size, self.cfg.embedding_scale, first.inw,
                             first.norm, eps)
        for k, (link, run) in enumerate(subs):
            last = k + 1 == len(subs)
            inw, norm = (self.every_stream, self.norm) if last else (subs[k + 1][0].inw, subs[k + 1][0].norm)
            h = stream_step(x, run(h), link.mix, link.out, inw, norm, eps, self.dtype, last=last)
        return h

    def _forward_norm_first(self, input_ids, md, kv_caches):
        eps, width, shared, subs = self.cfg.rms_norm_eps, pad8(self.cfg.hidden_size), {}, []
        for layer, cache in zip(self.layers, kv_caches):
            subs.append((layer.norm1, layer.mixer, lambda h, m=layer.mixer, c=cache: m(h, md, c, shared)))
            if isinstance(layer.mlp, ExpertMixture):
                subs.append((layer.norm2, layer.mlp, lambda h, m=layer.mlp: m(h, md.num_valid)))
            elif layer.mlp is not None:
                subs.append((layer.norm2, layer.mlp, layer.mlp))
        norm, sub, _ = subs[0]
        x, h = embed_norm(input_ids, self.embed_tokens.weight, norm, eps, ld=sub.in_cols, ones=sub.ones)
        for k, (_, sub, run) in enumerate(subs):
            if k + 1 < len(subs):
                norm, nxt, _ = subs[k + 1]
                h = add_norm(x, run(h), norm, eps, self.dtype, ld=nxt.in_cols, ones=nxt.ones, bias=sub.out_bias)
            else:
                h = add_norm(x, run(h), self.norm, eps, self.dtype, ld=width, bias=sub.out_bias, scale=self.cfg.logit_scale)
        return h

    def _forward_norm_both(self, input_ids, md, kv_caches):
        cfg, eps, m, width, n = self.cfg, self.cfg.rms_norm_eps, self.cfg.residual_mult, pad8(self.cfg.hidden_size), len(self.layers)
        T, dev = input_ids.shape[0], self.embed_tokens.weight.device
        # the embedding output and what every layer but the last one gave; the residual itself is overwritten
        results = torch.empty(n if cfg.depth_average else 1, T, width, dtype=torch.float32, device=dev)
        src, x = results[0], torch.empty(T, width, dtype=torch.float32, device=dev)
        first = self.layers[0]
        h = embed_positions(input_ids, self.embed_tokens.weight, md.positions, self.pos_embedding, src, first.norm1, eps,
                            ld=first.mixer.in_cols)
        for i, (layer, cache) in enumerate(zip(self.layers, kv_caches)):
            nxt = self.layers[i + 1] if i + 1 < n else None
            behind = dict(w=self.norm, ld=width) if nxt is None else dict(w=nxt.norm1, ld=nxt.mixer.in_cols)
            if layer.dwa is not None:
                behind.update(results=results, average=layer.dwa)
            y, norm = layer.mixer(h, md, cache), layer.norm1b
            if layer.mlp is not None:
                h = both_norms_step(src, x, y, norm, m, layer.norm2, eps, self.dtype, ld=layer.mlp.in_cols)
                y = layer.mlp(h, md.num_valid) if isinstance(layer.mlp, ExpertMixture) else layer.mlp(h)
                src, norm = x, layer.norm2b
            h = both_norms_step(src, x, y, norm, m, behind.pop("w"), eps, self.dtype, **behind)
            src = x
        return h


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
        self.lm_head = None
        if not cfg.tie_word_embeddings:
            self.lm_head = nn.Parameter(torch.zeros(cfg.vocab_size, pad8(cfg.hidden_size), dtype=self.model.dtype, device=device),
                                        requires_grad=False)

    @property
    def num_kv_layers(self):
        """Layers that hold pages of their own."""
        return sum(s.paged is not None and s.paged.owns_kv for s in self.cfg.layers)

    def allocate_caches(self, num_blocks: int, block_size: int, state_slots: int, zeros) -> list:
        """One entry per layer (see the module text).  ``zeros(*shape, dtype=)`` allocates."""
        caches: list = []
        for s, layer in zip(self.cfg.layers, self.model.layers):
            a, pages, state = s.paged, None, None
            if a is not None and not a.owns_kv:
                pages = caches[a.kv_from]
            elif a is not None:
                pages = tuple(zeros(*shape, dtype=self.model.dtype) for shape in a.page_shapes(num_blocks, block_size))
                pages = pages if len(pages) > 1 else pages[0]
            if s.recurrent:
                state = tuple(zeros(*shape, dtype=dt) for shape, dt in layer.mixer.state_shapes(state_slots, self.model.dtype))
            caches.append(pages if state is None else (state if pages is None else (pages, state)))
        return caches

    def paged_caches(self, caches: list) -> list:
        """The pools among ``caches`` - (k, v), or one - that belong to a layer of their own."""
        return [c[0] if s.recurrent else c for c, s in zip(caches, self.cfg.layers) if s.paged is not None and s.paged.owns_kv]

    def kv_bytes_per_token(self) -> int:
        esz = torch.empty(0, dtype=self.model.dtype).element_size()
        return esz * sum(s.paged.cache_elems_per_token() for s in self.cfg.layers if s.paged is not None)

    def state_bytes(self, slots: int) -> int:
        """Bytes of recurrent state for ``slots`` requests."""
        total = 0
        for s, layer in zip(self.cfg.layers, self.model.layers):
            if s.recurrent:
                for shape, dt in layer.mixer.state_shapes(slots, self.model.dtype):
                    total += torch.Size(shape).numel() * torch.empty(0, dtype=dt).element_size()
        return total

    def forward(self, input_ids, md, kv_caches, inputs_embeds=None):
        return self.model(input_ids, md, kv_caches, inputs_embeds)

    def compute_logits(self, hidden):
        return lm_logits(hidden, self.model.embed_tokens.weight if self.lm_head is None else self.lm_head)

    def process_weights_after_loading(self):
        """Padding rows and columns hold zeros whatever the loader or the random initialisation put there."""
        self.model.embed_tokens.weight.data[:, self.cfg.hidden_size:] = 0
        if self.model.pos_embedding is not None:
            self.model.pos_embedding.data[:, self.cfg.hidden_size:] = 0
        if self.lm_head is not None:
            self.lm_head.data[:, self.cfg.hidden_size:] = 0
        mods = [m for m in self.modules() if hasattr(m, "zero_padding")]
        for m in sorted(mods, key=lambda m: not isinstance(m, PaddedLinear)):      # single layers first, then what is made of them
            m.zero_padding()

    def should_use_eager_mode(self, md):
        return md.is_prefill

    # ------------------------------------------------------------------ checkpoint names
    def checkpoint_targets(self) -> dict:
        """{checkpoint tensor: (parameter, first row, rows, columns)} for the weight loader."""
        H = self.cfg.hidden_size
        out = {"embed": (self.model.embed_tokens.weight, 0, self.cfg.vocab_size, H), "final.norm": (self.model.norm, 0, H, None)}
        if self.cfg.norm_both:
            out["final.norm"] = _offset_target(self.model.norm, self.cfg.norm_offset)
        if self.model.pos_embedding is not None:
            out["pos"] = (self.model.pos_embedding, 0, self.cfg.learned_positions, H)
        if self.lm_head is not None:
            out["head"] = (self.lm_head, 0, self.cfg.vocab_size, H)
        for i, layer in enumerate(self.model.layers):
            if self.cfg.layers[i].weights_of is None:
                out.update({f"l{i}." + k: v for k, v in layer.checkpoint_targets().items()})
        return out

    def load_weights(self, weights, planner=None) -> set:
        from ..quantization.loader import WeightLoader
        return WeightLoader(self, self.cfg, planner=planner).load(weights)
