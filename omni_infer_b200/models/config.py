"""Architecture description shared by all model families (DeepSeek-V2/V3 MLA+MoE, MTP drafters,
Qwen2 dense GQA, Qwen3-MoE GQA, layer-list models) plus the named configurations used by the benchmarks."""
from __future__ import annotations

import dataclasses
import json
import re
from dataclasses import asdict, dataclass, field
from pathlib import Path
from typing import Any, Optional


# architectures of layer-list models with one residual and norms ahead of the sublayers
NORM_FIRST = ("Tenotar",)
# and those with norms on both sides of them
NORM_BOTH = ("Zusotar",)


@dataclass
class AttentionSpec:
    """Softmax attention of one layer of a layer-list model."""
    heads: int
    kv_heads: int
    dim: int                                 # query / key size per head
    vdim: int                                # value size per head
    scale: float
    window: int = 0                          # a query sees itself and the window - 1 tokens before it; 0 = all
    rot_dims: int = 0                        # leading dimensions of each head that are rotated; 0 = none
    rot_base: float = 10000.0
    rot_factor: float = 1.0                  # linear scaling: every frequency is divided by it
    kv_from: Optional[int] = None            # attends to the cached keys and values of this earlier layer
    qk_norm: bool = True                     # RMSNorm over the whole q and the whole k projection
    sink: bool = False                       # a learned term per head in the softmax denominator
    rot_scaling: Optional[dict] = None       # other scalings, as ``ops.rope_cos_sin_table`` takes them
    keep_first: int = 0                      # the first tokens of a sequence, seen beside the window
    chunk: int = 0                           # a query sees its own chunk of this many positions only; 0 = no chunks
    softcap: float = 0.0                     # scores are bounded softly by it (tanh); 0 = not
    distance_bias: bool = False              # slope 2^(-8 (h + 1) / heads) times the distance is taken off head h's scores
    head_norm: bool = False                  # RMSNorm of every q and k head (one weight each)
    rot_pairs: bool = False                  # neighbouring dimensions are rotated together (else i with i + rot_dims / 2)
    bias: bool = False                       # of the four projections
    conv: int = 0                            # taps of a short convolution of q, k and v; 0 = none
    v_mix: bool = False                      # values are mixed with those of the first layer that has this set
    v_norm: bool = False                     # every value head is divided by its root mean square
    log_bias: bool = False                   # learned r1 ln(1 + r2 distance) per head is taken off the scores
    out_gate: bool = False                   # a sigmoid gate per element on the output, projected from the layer's input

    @property
    def owns_kv(self) -> bool:
        return self.kv_from is None

    def cache_elems_per_token(self) -> int:
        return self.kv_heads * (self.dim + self.vdim) if self.owns_kv else 0

    def page_shapes(self, blocks: int, block_size: int) -> tuple:
        """Shapes of the page pools: keys, values."""
        return (blocks, block_size, self.kv_heads, self.dim), (blocks, block_size, self.kv_heads, self.vdim)


@dataclass
class LatentSpec:
    """Softmax attention through a key/value latent, and a query latent or none, of one layer of a layer-list model.  The cache
    holds the normed latent and one rotated key part that all heads share."""
    heads: int
    dim: int                                 # unrotated query / key size per head
    rot_dim: int                             # rotated query / key size per head
    vdim: int
    q_rank: int                              # 0 = queries are projected from the layer's input
    kv_rank: int
    scale: float
    window: int = 0                          # a query sees itself and the window - 1 tokens before it; 0 = all
    rot_base: float = 10000.0
    gate: bool = True                        # a sigmoid gate per head on the output
    sink: bool = False                       # a learned term per head in the softmax denominator
    rot_pairs: bool = False                  # neighbouring dimensions are rotated together (else i with i + rot_dim / 2)

    kv_from = None
    owns_kv = True
    rot_factor = 1.0
    rot_scaling = None

    @property
    def rot_dims(self) -> int:
        return self.rot_dim

    # Sizes as stored: multiples of 8, and the size that the latent decode kernel is made for where the general one ends.
    @property
    def _stored(self) -> tuple:
        c, r = (self.kv_rank + 7) // 8 * 8, (self.rot_dim + 7) // 8 * 8
        return (512, 64) if c + r > 256 and c <= 512 and r <= 64 else (c, r)

    @property
    def latent_cols(self) -> int:
        return self._stored[0]

    @property
    def rot_cols(self) -> int:
        return self._stored[1]

    def cache_elems_per_token(self) -> int:
        return self.latent_cols + self.rot_cols

    def page_shapes(self, blocks: int, block_size: int) -> tuple:
        """Shape of the one page pool: latent | rotated key part."""
        return ((blocks, block_size, self.cache_elems_per_token()),)


@dataclass
class Mamba2Spec:
    """Mamba-2 recurrence of one layer of a layer-list model."""
    heads: int
    vdim: int
    state: int
    groups: int = 1
    conv: int = 4                            # taps of the short convolution
    norm_groups: int = 1

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_channels(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclass
class MLSTMSpec:
    """Matrix memory (xLSTM) of one layer of a layer-list model."""
    heads: int
    dim: int                                 # query / key size per head
    vdim: int                                # value size per head
    gate_cap: float                          # both log gates are bounded softly by it


@dataclass
class WkvSpec:
    """WKV time mixing of one layer of a layer-list model."""
    heads: int
    dim: int                                 # key and value size per head
    rank: int = 0                            # of the decay's projection; 0 = as the checkpoint has it


@dataclass
class GLASpec:
    """Gated linear attention of one layer of a layer-list model."""
    heads: int
    dim: int                                 # query / key size per head
    vdim: int                                # value size per head
    tau: float                               # the decay is sigmoid(z)^(1 / tau)
    rank: int = 0                            # of the decay's projection; 0 = as the checkpoint has it


@dataclass
class ParallelSpec:
    """Attention and a matrix memory side by side on the same input."""
    left: AttentionSpec
    right: MLSTMSpec
    left_scale: float = 1.0
    right_scale: float = 1.0


@dataclass
class ExpertsSpec:
    """Mixture of gated experts of one layer of a layer-list model."""
    experts: int
    top: int
    ff: int
    limit: float = 0.0                       # of the clamped gate
    identity: int = 0                        # router outputs after the experts' whose expert is the identity
    scale: float = 1.0                       # of the routing weights
    shared_ff: int = 0                       # expert that runs for every token, 0 = none
    shared_limit: float = 0.0
    act: str = "clamped_glu"                 # or "swiglu"
    # "scores": softmax over all outputs, chosen by score + correction; "chosen": by logit + bias, softmax over the chosen ones;
    # "sigmoid": sigmoid scores, chosen by them
    weighting: str = "scores"
    groups: int = 1                          # equal groups of neighbours, scored by the sum of their two best experts ...
    keep_groups: int = 1                     # ... of which the choice is made from this many


@dataclass
class LayerSpec:
    """One entry of a layer-list model: a mixer and an optional feed-forward (gated dense, or a mixture of experts)."""
    attention: Optional[AttentionSpec] = None
    mamba2: Optional[Mamba2Spec] = None
    ff: int = 0                              # width of the dense feed-forward
    parallel: Optional[ParallelSpec] = None
    wkv: Optional[WkvSpec] = None
    experts: Optional[ExpertsSpec] = None
    weights_of: Optional[int] = None         # the layer runs with this layer's weights and a cache or state of its own
    latent: Optional[LatentSpec] = None
    act: str = "geglu"                       # of the dense feed-forward: or "swiglu"
    ff_bias: bool = False                    # of its three projections
    gla: Optional[GLASpec] = None

    @property
    def paged(self):
        """The attention that reads (and, unless it shares them, fills) cache pages."""
        if self.latent is not None:
            return self.latent
        return self.parallel.left if self.parallel is not None else self.attention

    @property
    def recurrent(self) -> bool:
        return (self.mamba2 is not None or self.parallel is not None or self.wkv is not None or self.gla is not None
                or (self.attention is not None and self.attention.conv > 0))

    @staticmethod
    def _pre_norm_attention(i: int, m: dict) -> AttentionSpec:
        """Attention without q/k norms, with a sink per head and Llama-3.1 frequency scaling."""
        rot = m.get("rot") or {}
        a = AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                          rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)), qk_norm=False, sink=True)
        if rot.get("scaling"):
            s = rot["scaling"]
            a.rot_scaling = {"type": "llama3", "factor": s["factor"], "low_freq_factor": s["low"], "high_freq_factor": s["high"],
                             "original_max_position_embeddings": s["original"]}
        return a

    @classmethod
    def _norm_first_entry(cls, i: int, d: dict) -> "LayerSpec":
        """Entry ``i`` of a design with one residual and norms ahead of the sublayers: latent attention; windowed attention
        with biases, head norms and pairwise rotation ("attention"); chunked attention with convolved projections, capped
        scores and a distance bias ("attention_2")."""
        kind, m = d["type"], d["mixer"]
        rot, mask, s = m.get("rot") or {}, m.get("mask") or {}, cls(act="swiglu", ff_bias=True)
        base = float(rot.get("base", 10000.0))
        if kind == "latent_attention":
            s.latent = LatentSpec(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=m["q_rank"],
                                  kv_rank=m["kv_rank"], scale=float(m["scale"]), window=int(mask.get("size") or 0), rot_base=base)
            if s.latent.rot_dim % 2 or rot.get("dims", s.latent.rot_dim) != s.latent.rot_dim:
                raise ValueError(f"layer {i}: the rotated part must be even and rotated as a whole")
        elif kind in ("attention", "attention_2"):
            a = s.attention = AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"],
                                            scale=float(m["scale"]), qk_norm=False, v_mix=bool(m.get("v_mix")))
            if kind == "attention":
                a.window, a.keep_first = int(mask.get("size") or 0), int(mask.get("keep_first") or 0)
                a.rot_dims, a.rot_base, a.rot_pairs = int(rot.get("dims", 0)), base, True
                a.head_norm = a.bias = True
            else:
                a.chunk, a.softcap, a.distance_bias = int(mask.get("size") or 0), float(m.get("softcap") or 0.0), True
                a.conv = int(m["conv"])
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        return s

    @classmethod
    def _norm_both_entry(cls, i: int, d: dict) -> "LayerSpec":
        """Entry ``i`` of a design with norms on both sides of the sublayers: latent attention with a sink and queries of their
        own projection; windowed attention with normed values, a logarithmic distance bias and an output gate; gated linear
        attention.  The type may carry a running number."""
        kind, m = re.sub(r"_\d+$", "", d["type"]), d["mixer"]
        rot, mask, s = m.get("rot") or {}, m.get("mask") or {}, cls(act="swiglu")
        if kind == "latent_attention":
            s.latent = LatentSpec(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=0, kv_rank=m["kv_rank"],
                                  scale=float(m["scale"]), rot_base=float(rot.get("base", 10000.0)), gate=False, sink=True, rot_pairs=True)
            if s.latent.rot_dim % 2 or rot.get("dims", s.latent.rot_dim) != s.latent.rot_dim:
                raise ValueError(f"layer {i}: the rotated part must be even and rotated as a whole")
        elif kind == "attention":
            s.attention = AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                                        window=int(mask.get("size") or 0), qk_norm=False, v_norm=True, log_bias=True, out_gate=True)
        elif kind == "gla":
            s.gla = GLASpec(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], tau=float(m["tau"]))
            if not s.gla.tau > 0:
                raise ValueError(f"layer {i}: tau must be positive")
        else:
            raise ValueError(f"layer {i}: unknown mixer type {d['type']!r}")
        return s

    @classmethod
    def from_dict(cls, i: int, d: dict, norms: str = "") -> "LayerSpec":
        """Entry ``i`` of the ``layers`` list of a config.json.  The type may carry a running number (several mixers of
        one kind with sizes of their own).  ``norms``: "first" and "both" for the designs of ``NORM_FIRST`` and ``NORM_BOTH``."""
        kind, m = re.sub(r"_\d+$", "", d["type"]), d["mixer"]
        if norms == "first":
            s = cls._norm_first_entry(i, d)
        elif norms == "both":
            s = cls._norm_both_entry(i, d)
        else:
            s = cls(weights_of=d.get("weights_of"))
        if norms:
            pass
        elif kind == "attention":
            rot = m.get("rot") or {}
            s.attention = AttentionSpec(
                heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                window=int((m.get("mask") or {}).get("size") or 0), rot_dims=int(rot.get("dims", 0)),
                rot_base=float(rot.get("base", 10000.0)),
                rot_factor=float((rot.get("scaling") or {}).get("factor", 1.0)), kv_from=m.get("kv_from"))
        elif kind == "mamba2":
            s.mamba2 = Mamba2Spec(heads=m["heads"], vdim=m["vdim"], state=m["state"], groups=m["groups"], conv=m["conv"],
                                  norm_groups=m["norm_groups"])
            if s.mamba2.heads % s.mamba2.groups or s.mamba2.inner % s.mamba2.norm_groups:
                raise ValueError(f"layer {i}: heads must divide over the groups, the inner width over the norm groups")
        elif kind == "parallel":
            r = m["right"]
            s.parallel = ParallelSpec(cls._pre_norm_attention(i, m["left"]),
                                      MLSTMSpec(heads=r["heads"], dim=r["dim"], vdim=r["vdim"], gate_cap=float(r["gate_cap"])),
                                      float(m["left_scale"]), float(m["right_scale"]))
        elif kind == "wkv":
            s.wkv = WkvSpec(heads=m["heads"], dim=m["dim"])
        else:
            raise ValueError(f"layer {i}: unknown mixer type {d['type']!r}")
        a = s.paged
        if a is not None and s.latent is None and (a.heads % a.kv_heads or a.rot_dims % 2 or a.rot_dims > a.dim):
            raise ValueError(f"layer {i}: heads must divide over the key/value heads, rotated dimensions be even and fit the head")
        mlp = d.get("mlp")
        if mlp:
            fkind = mlp.get("kind", "dense")
            if fkind == "dense":
                s.ff = int(mlp["ff"])
            elif fkind == "moe":
                if not mlp.get("router") or not mlp.get("expert"):
                    raise ValueError(f"layer {i}: a feed-forward of kind 'moe' needs a router and an expert")
                r, e, sh = mlp["router"], mlp["expert"], mlp.get("shared") or {}
                if norms == "first":
                    s.experts = ExpertsSpec(experts=r["experts"], top=r["top"], ff=e["ff"], shared_ff=int(sh.get("ff", 0)),
                                            act="swiglu", weighting="chosen")
                elif norms == "both":
                    g = r.get("groups") or {}
                    s.experts = ExpertsSpec(experts=r["experts"], top=r["top"], ff=e["ff"], shared_ff=int(sh.get("ff", 0)), act="swiglu",
                                            weighting="sigmoid", groups=int(g.get("count", 1)), keep_groups=int(g.get("keep", 1)))
                    n, k = s.experts.groups, s.experts.keep_groups
                    if not 0 < k <= n <= 32 or s.experts.experts % n or s.experts.top > s.experts.experts // n * k:
                        raise ValueError(f"layer {i}: {s.experts.top} of {s.experts.experts} experts from {k} of {n} groups")
                else:
                    s.experts = ExpertsSpec(experts=r["experts"], top=r["top"], ff=e["ff"], limit=float(e["limit"]),
                                            identity=int(r.get("identity") or 0), scale=float(r.get("scale", 1.0)),
                                            shared_ff=int(sh.get("ff", 0)), shared_limit=float(sh.get("limit", 0.0)))
                n = s.experts.experts + s.experts.identity
                if not 0 < s.experts.top <= min(n, 32) or n > 512:
                    raise ValueError(f"layer {i}: {s.experts.top} of {n} experts (at most 32 of 512)")
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {fkind!r}")
        return s


@dataclass
class ModelConfig:
    architecture: str = "DeepseekV3ForCausalLM"
    # layer-list models: one LayerSpec per layer; None = the uniform stacks described by the fields below
    layers: Optional[list] = None
    # residual streams of a layer-list model with layer norms ahead of its sublayers; 0 = one residual, norms on the outputs
    streams: int = 0
    embedding_scale: float = 1.0
    # layer-list models: one residual with RMS norms ahead of the sublayers
    norm_first: bool = False
    logit_scale: float = 1.0
    # ... on both sides of them, with what a sublayer adds times residual_mult
    norm_both: bool = False
    residual_mult: float = 1.0
    # what checkpoints leave out of the weights of those norms (1: they are stored around zero)
    norm_offset: float = 0.0
    # after every layer the residual is a learned sum of the embedding output and all layers' results so far
    depth_average: bool = False
    # rows of the table of learned positions, which bounds the context; 0 = none
    learned_positions: int = 0
    # tensor-parallel attention: heads sharded over attn_tp_size ranks, hidden states sharded by token rows between
    # layers (set by the model runner; 1 = every rank runs whole attention layers on its own requests)
    attn_tp_size: int = 1
    attn_tp_rank: int = 0
    # sub-group sharding while attention is data parallel: the dense MLP layers and the shared expert over the
    # ``mlp_tp`` group, o_proj over the ``o_proj_tp`` group (set by the worker from the engine configuration)
    dense_mlp_tp_size: int = 1
    o_proj_tp_size: int = 1
    # dedicated shared-expert ranks: the first N ranks of the expert-parallel group hold only the shared expert, the routed
    # experts are spread over the others (0 = the shared expert runs on every rank beside its routed experts)
    shared_expert_ranks: int = 0
    # vocabulary-parallel embedding table and LM head: each rank holds ceil(vocab / size) rows (set by the model runner)
    vocab_parallel_size: int = 1
    vocab_parallel_rank: int = 0
    # benchmark aid: {"s": 1.2, "strength": 6.0, "seed": 0} adds a fixed Zipf-shaped bias to every router's logits so that
    # expert popularity is skewed (load-balance stress); None = the router as trained
    router_skew: Optional[dict] = None
    vocab_size: int = 1024
    hidden_size: int = 256
    num_hidden_layers: int = 2
    num_attention_heads: int = 4
    num_key_value_heads: int = 4
    head_dim: int = 64                       # GQA models
    # MLA
    use_mla: bool = True
    q_lora_rank: int = 0
    kv_lora_rank: int = 64
    qk_nope_head_dim: int = 32
    qk_rope_head_dim: int = 16
    v_head_dim: int = 32
    # MLP / MoE
    intermediate_size: int = 512
    moe_intermediate_size: int = 128
    n_routed_experts: int = 0
    n_shared_experts: int = 0
    num_experts_per_tok: int = 0
    first_k_dense_replace: int = 0
    moe_layer_freq: int = 1
    scoring_func: str = "softmax"            # softmax | sigmoid
    topk_method: str = "greedy"              # greedy | group_limited_greedy | noaux_tc
    n_group: int = 1
    topk_group: int = 1
    norm_topk_prob: bool = False
    routed_scaling_factor: float = 1.0
    # misc
    rms_norm_eps: float = 1e-6
    rope_theta: float = 10000.0
    rope_scaling: Optional[dict] = None
    max_position_embeddings: int = 4096
    tie_word_embeddings: bool = False
    qk_norm: bool = False                    # Qwen3 per-head q/k RMSNorm
    attention_bias: bool = False             # Qwen2 qkv bias
    num_nextn_predict_layers: int = 0        # MTP layers stored after the main stack
    quantization: str = "none"               # none | fp8_block | w8a8_int8
    dtype: str = "bfloat16"
    name: str = ""

    # ---- derived
    @property
    def qk_head_dim(self) -> int:
        return self.qk_nope_head_dim + self.qk_rope_head_dim

    @property
    def is_moe(self) -> bool:
        return self.n_routed_experts > 0

    def layer_is_moe(self, layer_idx: int) -> bool:
        return (self.is_moe and layer_idx >= self.first_k_dense_replace
                and layer_idx % self.moe_layer_freq == 0)

    @property
    def softmax_scale(self) -> float:
        """MLA: (nope+rope)^-0.5 * mscale^2 with the YaRN mscale_all_dim correction
        (omni/models/common/layers/attention/deepseek_mla.py:43-48, 173-177)."""
        import math

        d = self.qk_head_dim if self.use_mla else self.head_dim
        scale = d ** -0.5
        rs = self.rope_scaling
        if self.use_mla and rs and rs.get("factor", 1.0) > 1.0 and rs.get("mscale_all_dim", 0):
            m = 0.1 * rs["mscale_all_dim"] * math.log(rs["factor"]) + 1.0
            scale = scale * m * m
        return scale

    @property
    def has_recurrent_state(self) -> bool:
        """Does a request hold state besides its cached tokens (one slot per live request)?"""
        return any(s.recurrent for s in self.layers or ())

    def kv_bytes_per_token(self, elem_bytes: int = 2) -> int:
        if self.layers is not None:     # mean over the layers that hold a cache
            per = [s.paged.cache_elems_per_token() for s in self.layers if s.paged is not None and s.paged.owns_kv]
            return sum(per) * elem_bytes // max(1, len(per))
        if self.use_mla:
            return (self.kv_lora_rank + self.qk_rope_head_dim) * elem_bytes
        return 2 * self.local_kv_heads * self.head_dim * elem_bytes

    @property
    def local_kv_heads(self) -> int:
        """K/V heads cached by one rank (all of them unless attention runs tensor parallel)."""
        return max(1, self.num_key_value_heads // max(1, self.attn_tp_size))

    def to_dict(self) -> dict:
        return asdict(self)

    @classmethod
    def from_hf_dict(cls, d: dict[str, Any]) -> "ModelConfig":
        arch = (d.get("architectures") or [d.get("architecture", "DeepseekV3ForCausalLM")])[0]
        if isinstance(d.get("layers"), list):
            return cls.from_layer_list(arch, d)
        c = cls(architecture=arch)
        for k in ("vocab_size", "hidden_size", "num_hidden_layers", "num_attention_heads", "intermediate_size",
                  "moe_intermediate_size", "n_routed_experts", "n_shared_experts", "num_experts_per_tok",
                  "first_k_dense_replace", "moe_layer_freq", "scoring_func", "topk_method", "n_group", "topk_group",
                  "norm_topk_prob", "routed_scaling_factor", "rms_norm_eps", "rope_theta", "rope_scaling",
                  "max_position_embeddings", "tie_word_embeddings", "kv_lora_rank", "qk_nope_head_dim",
                  "qk_rope_head_dim", "v_head_dim", "num_nextn_predict_layers"):
            if k in d and d[k] is not None:
                setattr(c, k, d[k])
        c.q_lora_rank = d.get("q_lora_rank") or 0
        c.num_key_value_heads = d.get("num_key_value_heads", c.num_attention_heads)
        c.use_mla = "Deepseek" in arch
        if not c.use_mla:
            c.head_dim = d.get("head_dim", c.hidden_size // c.num_attention_heads)
            c.attention_bias = "Qwen2" in arch
            c.qk_norm = "Qwen3" in arch
            if "num_experts" in d:   # Qwen MoE naming
                c.n_routed_experts = d["num_experts"]
                c.num_experts_per_tok = d.get("num_experts_per_tok", 8)
                c.moe_intermediate_size = d.get("moe_intermediate_size", c.moe_intermediate_size)
                c.norm_topk_prob = d.get("norm_topk_prob", True)
        qc = d.get("quantization_config") or {}
        if qc.get("quant_method") == "fp8":
            c.quantization = "fp8_block"
        elif qc.get("quant_method") in ("ascend_compressed_tensors", "compressed-tensors", "compressed_tensors"):
            c.quantization = "w8a8_int8"
        return c

    @classmethod
    def from_layer_list(cls, arch: str, d: dict[str, Any]) -> "ModelConfig":
        """config.json whose ``layers`` list describes every layer (mixer and feed-forward sizes of its own)."""
        norm_first, norm_both = arch in NORM_FIRST, arch in NORM_BOTH
        layers = [LayerSpec.from_dict(i, e, "first" if norm_first else ("both" if norm_both else "")) for i, e in enumerate(d["layers"])]
        for i, s in enumerate(layers):
            a = s.attention
            if a is None or a.owns_kv:
                continue
            src = layers[a.kv_from].attention if 0 <= a.kv_from < i else None
            if src is None or not src.owns_kv:
                raise ValueError(f"layer {i} takes its keys from layer {a.kv_from}, which holds none")
            if (src.kv_heads, src.dim, src.vdim) != (a.kv_heads, a.dim, a.vdim):
                raise ValueError(f"layers {i} and {a.kv_from} share keys but differ in their head sizes")
        streams = int(d.get("streams", 0))
        if norm_first:
            mixed = {s.attention.kv_heads * s.attention.vdim for s in layers if s.attention is not None and s.attention.v_mix}
            if len(mixed) > 1:
                raise ValueError("layers that mix their values must have equally many of them")
        elif not norm_both and any((s.parallel or s.wkv or s.experts) is not None if not streams
                                   else (s.attention or s.mamba2) is not None or s.ff for s in layers):
            raise ValueError("attention, mamba2 and dense layers run on one residual with norms on the outputs, parallel, wkv and "
                             "mixture-of-experts layers on residual streams with norms ahead")
        for i, s in enumerate(layers):
            seen = {i}
            while s.weights_of is not None:
                j = s.weights_of
                if not 0 <= j < len(layers) or j in seen:
                    raise ValueError(f"layer {i} takes its weights from layer {j}, which has none")
                seen.add(j)
                s = layers[j]
            if len(seen) > 1:
                if dataclasses.replace(layers[i], weights_of=None) != s:
                    raise ValueError(f"layers {i} and {layers[i].weights_of} share weights but differ in their sizes")
                layers[i].weights_of = next(j for j, o in enumerate(layers) if o is s)
        return cls(architecture=arch, layers=layers, vocab_size=d["vocab"], hidden_size=d["width"],
                   num_hidden_layers=len(layers), rms_norm_eps=float(d["norm"]["eps"]), use_mla=False,
                   tie_word_embeddings=not (norm_first or norm_both), n_routed_experts=0, name=arch, streams=streams,
                   embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)), norm_first=norm_first,
                   logit_scale=float(d.get("logit_scale", 1.0)), norm_both=norm_both, residual_mult=float(d.get("residual_mult", 1.0)),
                   norm_offset=1.0 if norm_both else 0.0, depth_average=norm_both,
                   learned_positions=int(d["max_positions"]) if norm_both else 0)

    @classmethod
    def from_pretrained(cls, path: str) -> "ModelConfig":
        c = cls.from_hf_dict(json.loads((Path(path) / "config.json").read_text()))
        if c.unresolved_sizes():
            from ..quantization.loader import safetensors_shapes
            c.resolve_sizes(safetensors_shapes(path))
        return c

    def unresolved_sizes(self) -> bool:
        """Are there sizes that only the checkpoint's tensors tell?"""
        return any(r is not None and r.rank == 0 for s in self.layers or () for r in (s.wkv, s.gla))

    def resolve_sizes(self, shapes: dict) -> None:
        """``shapes``: checkpoint tensor name -> shape."""
        for i, s in enumerate(self.layers or ()):
            for r, tensor in ((s.wkv, "w1"), (s.gla, "a1")):
                if r is None or r.rank != 0:
                    continue
                name = f"l{i if s.weights_of is None else s.weights_of}.mix.{tensor}"
                if name not in shapes:
                    raise KeyError(f"checkpoint lacks {name}")
                r.rank = int(shapes[name][0])


# ------------------------------------------------------------------------------------------------
# Named configurations
# ------------------------------------------------------------------------------------------------
def tiny_deepseek_v3(**kw) -> ModelConfig:
    """CPU mock: 2 layers (dense, then MoE), hidden 256, 4 heads, q_lora 128, kv_lora 64, nope 32,
    rope 16, v 32, 8 routed experts (inter 128) top-2 softmax + 1 shared, vocab 1024."""
    c = ModelConfig(architecture="DeepseekV3ForCausalLM", name="tiny-deepseek-v3", vocab_size=1024, hidden_size=256,
                    num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=4, q_lora_rank=128,
                    kv_lora_rank=64, qk_nope_head_dim=32, qk_rope_head_dim=16, v_head_dim=32, intermediate_size=512,
                    moe_intermediate_size=128, n_routed_experts=8, n_shared_experts=1, num_experts_per_tok=2,
                    first_k_dense_replace=1, scoring_func="softmax", topk_method="greedy", norm_topk_prob=False,
                    dtype="float32", max_position_embeddings=512)
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def small_deepseek_gpu(**kw) -> ModelConfig:
    """Small MLA+MoE model with the kernel-native head shapes (kv_lora 512, rope 64, nope 128, v 128)."""
    c = ModelConfig(architecture="DeepseekV3ForCausalLM", name="small-deepseek", vocab_size=4096, hidden_size=1024,
                    num_hidden_layers=3, num_attention_heads=16, num_key_value_heads=16, q_lora_rank=512,
                    kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128,
                    intermediate_size=2048, moe_intermediate_size=512, n_routed_experts=16, n_shared_experts=1,
                    num_experts_per_tok=4, first_k_dense_replace=1, scoring_func="sigmoid", topk_method="noaux_tc",
                    n_group=4, topk_group=2, norm_topk_prob=True, routed_scaling_factor=2.5,
                    max_position_embeddings=4096)
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def deepseek_v2_lite(**kw) -> ModelConfig:
    c = ModelConfig(architecture="DeepseekV2ForCausalLM", name="deepseek-v2-lite", vocab_size=102400,
                    hidden_size=2048, num_hidden_layers=27, num_attention_heads=16, num_key_value_heads=16,
                    q_lora_rank=0, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128,
                    intermediate_size=10944, moe_intermediate_size=1408, n_routed_experts=64, n_shared_experts=2,
                    num_experts_per_tok=6, first_k_dense_replace=1, scoring_func="softmax", topk_method="greedy",
                    n_group=1, topk_group=1, norm_topk_prob=False, routed_scaling_factor=1.0, rope_theta=10000.0,
                    rope_scaling={"type": "yarn", "factor": 40, "original_max_position_embeddings": 4096,
                                  "beta_fast": 32, "beta_slow": 1, "mscale": 0.707, "mscale_all_dim": 0.707},
                    max_position_embeddings=163840)
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def deepseek_v3(**kw) -> ModelConfig:
    c = ModelConfig(architecture="DeepseekV3ForCausalLM", name="deepseek-v3-671b", vocab_size=129280,
                    hidden_size=7168, num_hidden_layers=61, num_attention_heads=128, num_key_value_heads=128,
                    q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128,
                    intermediate_size=18432, moe_intermediate_size=2048, n_routed_experts=256, n_shared_experts=1,
                    num_experts_per_tok=8, first_k_dense_replace=3, scoring_func="sigmoid", topk_method="noaux_tc",
                    n_group=8, topk_group=4, norm_topk_prob=True, routed_scaling_factor=2.5, rope_theta=10000.0,
                    rope_scaling={"type": "yarn", "factor": 40, "original_max_position_embeddings": 4096,
                                  "beta_fast": 32, "beta_slow": 1, "mscale": 1.0, "mscale_all_dim": 1.0},
                    max_position_embeddings=163840, num_nextn_predict_layers=1, quantization="fp8_block")
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def qwen3_30b_a3b(**kw) -> ModelConfig:
    c = ModelConfig(architecture="Qwen3MoeForCausalLM", name="qwen3-30b-a3b", vocab_size=151936, hidden_size=2048,
                    num_hidden_layers=48, num_attention_heads=32, num_key_value_heads=4, head_dim=128, use_mla=False,
                    intermediate_size=6144, moe_intermediate_size=768, n_routed_experts=128, n_shared_experts=0,
                    num_experts_per_tok=8, first_k_dense_replace=0, scoring_func="softmax", topk_method="greedy",
                    norm_topk_prob=True, rope_theta=1e6, qk_norm=True, max_position_embeddings=40960)
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def qwen2_small(**kw) -> ModelConfig:
    c = ModelConfig(architecture="Qwen2ForCausalLM", name="qwen2-small", vocab_size=4096, hidden_size=1024,
                    num_hidden_layers=2, num_attention_heads=8, num_key_value_heads=2, head_dim=128, use_mla=False,
                    intermediate_size=2816, n_routed_experts=0, attention_bias=True, rope_theta=1e6,
                    max_position_embeddings=4096)
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def tiny_qwen3_moe(**kw) -> ModelConfig:
    """CPU-sized GQA MoE in the shape of Qwen3-MoE: 2 layers, 4 q / 2 kv heads of 32 dims with q/k norm, 8 experts
    top-2 with renormalised softmax routing, no shared expert."""
    c = ModelConfig(architecture="Qwen3MoeForCausalLM", name="tiny-qwen3-moe", vocab_size=1024, hidden_size=128,
                    num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2, head_dim=32, use_mla=False,
                    intermediate_size=256, moe_intermediate_size=64, n_routed_experts=8, n_shared_experts=0,
                    num_experts_per_tok=2, first_k_dense_replace=0, scoring_func="softmax", topk_method="greedy",
                    norm_topk_prob=True, rope_theta=1e6, qk_norm=True, dtype="float32", max_position_embeddings=512)
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def forovik(width=2048, layers=12, vocab=32768, heads=16, kv_heads=4, dim=128, window=1024, ff=5632, m_heads=64, m_vdim=64,
            state=128, groups=1, conv=4, norm_groups=1, **kw) -> ModelConfig:
    """Layer-list model in the shape of a small hybrid: groups of one windowed-attention layer (with feed-forward) and two
    Mamba-2 layers; every second attention layer reads the keys and values of the one before it."""
    specs, last_kv = [], None
    for i in range(layers):
        if i % 3 == 0:
            share = last_kv if (i // 3) % 2 == 1 else None
            specs.append(LayerSpec(AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, window, dim // 2, 1e6, 4.0, share),
                                   None, ff))
            last_kv = i if share is None else last_kv
        else:
            specs.append(LayerSpec(None, Mamba2Spec(m_heads, m_vdim, state, groups, conv, norm_groups)))
    c = ModelConfig(architecture="Forovik", name="forovik", layers=specs, vocab_size=vocab, hidden_size=width,
                    num_hidden_layers=layers, use_mla=False, tie_word_embeddings=True, rms_norm_eps=1e-5)
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def fimudra(width=2048, layers=12, vocab=32768, streams=2, heads=16, kv_heads=4, dim=128, m_heads=16, m_dim=64, m_vdim=128,
            w_heads=32, w_dim=64, w_rank=64, experts=32, identity=4, top=4, ff=768, shared_ff=1536, loop=True, **kw) -> ModelConfig:
    """Layer-list model with residual streams: attention beside a matrix memory in two of three layers, WKV in the third, a
    mixture of experts in each; with ``loop`` the last layer runs with the weights of the first of its kind."""
    ffn = lambda: ExpertsSpec(experts, top, ff, 7.0, identity, 2.5, shared_ff, 7.0)        # noqa: E731
    specs = []
    for i in range(layers):
        if i % 3 == 2:
            specs.append(LayerSpec(wkv=WkvSpec(w_heads, w_dim, w_rank), experts=ffn()))
        else:
            att = AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, rot_dims=dim, rot_base=5e5, qk_norm=False, sink=True,
                                rot_scaling={"type": "llama3", "factor": 8.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0,
                                             "original_max_position_embeddings": 8192})
            specs.append(LayerSpec(parallel=ParallelSpec(att, MLSTMSpec(m_heads, m_dim, m_vdim, 15.0), 0.7, 0.7), experts=ffn()))
    if loop and layers > 3:
        specs[-1].weights_of = (layers - 1) % 3
    c = ModelConfig(architecture="Fimudra", name="fimudra", layers=specs, vocab_size=vocab, hidden_size=width,
                    num_hidden_layers=layers, use_mla=False, tie_word_embeddings=True, rms_norm_eps=1e-5, streams=streams,
                    embedding_scale=width ** 0.5)
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def tiny_fimudra(**kw) -> ModelConfig:
    """CPU-sized layer-list model with residual streams."""
    kw.setdefault("dtype", "float32")
    kw.setdefault("name", "tiny-fimudra")
    return fimudra(width=64, layers=6, vocab=512, streams=3, heads=4, kv_heads=2, dim=16, m_heads=3, m_dim=8, m_vdim=16, w_heads=4,
                   w_dim=12, w_rank=5, experts=6, identity=2, top=2, ff=24, shared_ff=40, **kw)


def tenotar(width=2048, layers=12, vocab=32768, heads=16, kv_heads=4, dim=128, q_rank=768, kv_rank=512, rot_dim=64, window=1024,
            keep_first=4, chunk=1024, conv=4, ff=5632, experts=32, top=4, expert_ff=768, shared_ff=1536, **kw) -> ModelConfig:
    """Layer-list model with norms ahead of its sublayers: latent, windowed and chunked attention in turn, the first layer with a
    dense feed-forward and the others with a mixture of experts."""
    specs = []
    for i in range(layers):
        if i % 3 == 0:
            s = LayerSpec(latent=LatentSpec(heads, dim, rot_dim, dim, q_rank, kv_rank, (dim + rot_dim) ** -0.5, window))
        elif i % 3 == 1:
            s = LayerSpec(AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, window, dim, 5e5, qk_norm=False, keep_first=keep_first,
                                        head_norm=True, rot_pairs=True, bias=True, v_mix=True))
        else:
            s = LayerSpec(AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, qk_norm=False, chunk=chunk, softcap=30.0,
                                        distance_bias=True, conv=conv, v_mix=True))
        if i == 0:
            s.ff, s.act, s.ff_bias = ff, "swiglu", True
        else:
            s.experts = ExpertsSpec(experts, top, expert_ff, shared_ff=shared_ff, act="swiglu", weighting="chosen")
        specs.append(s)
    c = ModelConfig(architecture="Tenotar", name="tenotar", layers=specs, vocab_size=vocab, hidden_size=width,
                    num_hidden_layers=layers, use_mla=False, tie_word_embeddings=False, rms_norm_eps=1e-5, norm_first=True,
                    logit_scale=0.5)
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def tiny_tenotar(**kw) -> ModelConfig:
    """CPU-sized layer-list model with norms ahead of its sublayers."""
    kw.setdefault("dtype", "float32")
    kw.setdefault("name", "tiny-tenotar")
    return tenotar(width=64, layers=6, vocab=512, heads=4, kv_heads=2, dim=16, q_rank=24, kv_rank=40, rot_dim=8, window=40, keep_first=3,
                   chunk=48, conv=3, ff=96, experts=6, top=2, expert_ff=24, shared_ff=40, **kw)


def zusotar(width=2048, layers=12, vocab=32768, heads=16, kv_heads=4, dim=128, kv_rank=512, rot_dim=64, window=1024, g_heads=16, g_dim=64,
            g_vdim=128, g_rank=16, ff=5632, experts=32, groups=4, keep=2, top=4, expert_ff=768, shared_ff=1536, positions=16384,
            **kw) -> ModelConfig:
    """Layer-list model with norms on both sides of its sublayers: latent attention, gated linear attention and windowed attention
    in turn, the first layer with a dense feed-forward and the others with a mixture of experts."""
    specs = []
    for i in range(layers):
        if i % 3 == 0:
            s = LayerSpec(latent=LatentSpec(heads, dim, rot_dim, dim, 0, kv_rank, (dim + rot_dim) ** -0.5, rot_base=5e5, gate=False, sink=True,
                                            rot_pairs=True))
        elif i % 3 == 1:
            s = LayerSpec(gla=GLASpec(g_heads, g_dim, g_vdim, 16.0, g_rank))
        else:
            s = LayerSpec(AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, window, qk_norm=False, v_norm=True, log_bias=True,
                                        out_gate=True))
        s.act = "swiglu"
        if i == 0:
            s.ff = ff
        else:
            s.experts = ExpertsSpec(experts, top, expert_ff, shared_ff=shared_ff, act="swiglu", weighting="sigmoid", groups=groups,
                                    keep_groups=keep)
        specs.append(s)
    c = ModelConfig(architecture="Zusotar", name="zusotar", layers=specs, vocab_size=vocab, hidden_size=width,
                    num_hidden_layers=layers, use_mla=False, tie_word_embeddings=False, rms_norm_eps=1e-5, norm_both=True,
                    residual_mult=0.4, norm_offset=1.0, depth_average=True, learned_positions=positions)
    for k, v in kw.items():
        setattr(c, k, v)
    return c


def tiny_zusotar(**kw) -> ModelConfig:
    """CPU-sized layer-list model with norms on both sides of its sublayers."""
    kw.setdefault("dtype", "float32")
    kw.setdefault("name", "tiny-zusotar")
    return zusotar(width=64, layers=6, vocab=512, heads=4, kv_heads=2, dim=16, kv_rank=40, rot_dim=8, window=40, g_heads=2, g_dim=16,
                   g_vdim=24, g_rank=8, ff=96, experts=8, groups=4, keep=2, top=2, expert_ff=24, shared_ff=40, positions=512, **kw)


def tiny_forovik(**kw) -> ModelConfig:
    """CPU-sized layer-list model."""
    kw.setdefault("dtype", "float32")
    kw.setdefault("name", "tiny-forovik")
    return forovik(width=64, layers=6, vocab=512, heads=4, kv_heads=2, dim=16, window=40, ff=96, m_heads=4, m_vdim=16,
                   state=32, groups=2, conv=4, norm_groups=2, **kw)


PRESETS = {
    "forovik": forovik,
    "tiny-forovik": tiny_forovik,
    "tenotar": tenotar,
    "tiny-tenotar": tiny_tenotar,
    "zusotar": zusotar,
    "tiny-zusotar": tiny_zusotar,
    "fimudra": fimudra,
    "tiny-fimudra": tiny_fimudra,
    "tiny-deepseek-v3": tiny_deepseek_v3,
    "tiny-qwen3-moe": tiny_qwen3_moe,
    "small-deepseek": small_deepseek_gpu,
    "deepseek-v2-lite": deepseek_v2_lite,
    "deepseek-v3": deepseek_v3,
    "qwen3-30b-a3b": qwen3_30b_a3b,
    "qwen2-small": qwen2_small,
}


def get_config(name_or_path: str, **kw) -> ModelConfig:
    if name_or_path in PRESETS:
        return PRESETS[name_or_path](**kw)
    c = ModelConfig.from_pretrained(name_or_path)
    for k, v in kw.items():
        setattr(c, k, v)
    return c
