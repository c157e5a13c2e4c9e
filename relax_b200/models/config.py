"""Model shape descriptions and the named presets used by recipes and benchmarks.

The fields follow the MODEL_ARGS of the reference's ``scripts/models/*.sh``
(e.g. scripts/models/qwen3-8B.sh:4-18, scripts/models/qwen3-30B-A3B.sh:40-50).
"""
from __future__ import annotations

from dataclasses import dataclass, field, asdict, replace
from typing import Optional


@dataclass
class VisionConfig:
    num_layers: int = 32
    hidden_size: int = 1280
    num_heads: int = 16
    ffn_hidden_size: int = 3420
    patch_size: int = 14
    spatial_merge_size: int = 2
    in_channels: int = 3
    temporal_patch_size: int = 2
    out_hidden_size: int = 3584
    # dots.ocr's tower (relax/models/dots_ocr/vision.py): RMSNorm after the patch projection and after the last block, a
    # LayerNorm (with bias) in front of the merger, its own norm epsilon
    patch_norm: bool = False
    post_trunk_norm: bool = False
    merger_layernorm: bool = False
    rms_norm_eps: "float | None" = None


@dataclass(frozen=True)
class MoESpec:
    """Routed feed-forward of a composed layer: ``experts`` small feed-forwards of width ``ff``, of which every token takes ``top`` by
    the ``score`` (sigmoid or softmax) of its router logits.  ``act`` ``relu2``: ``down(relu(up h)^2)``; ``swiglu``:
    ``down(silu(gate h) * up h)``; ``clamped_swish``: ``down(g sigmoid(1.702 g) (u + 1))`` with ``g = min(gate h, limit)`` and
    ``u = up h`` clamped to ``+- limit``.  ``identity``
    more router outputs stand for experts without weights whose output is ``h`` itself.  All outputs form ``groups`` equal
    groups of neighbours; only those of the ``keep`` groups whose ``group_best`` best scores have the largest sums can be taken.
    ``correction``: a learned offset per output that joins the scores for the choice, not for the weights.  ``shared_ff``: width of
    one more (``relu2``) feed-forward that every token takes with weight one (0 = none)."""
    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0
    act: str = "relu2"
    renormalize: bool = False    # weights divided by their sum over the taken experts
    weight_scale: float = 1.0    # factor on the weights
    score: str = "sigmoid"
    correction: bool = False
    identity: int = 0
    group_best: int = 2
    limit: float = 0.0           # clamped_swish only

    def __post_init__(self):
        if min(self.experts, self.top, self.ff, self.groups, self.keep) < 1 or min(self.shared_ff, self.identity) < 0 \
                or self.act not in EXPERT_ACTIVATIONS or self.score not in ("sigmoid", "softmax") or self.group_best not in (1, 2):
            raise ValueError(f"bad expert layer: {self}")
        if (self.act == "clamped_swish") != (self.limit > 0) or (self.gated and self.shared_ff):
            raise ValueError(f"bad expert activation: {self}")
        if self.outputs % self.groups or self.keep > self.groups or self.top > self.outputs // self.groups * self.keep:
            raise ValueError(f"{self.top} of {self.outputs} experts cannot be taken from {self.keep} of {self.groups} groups")

    @property
    def outputs(self) -> int:
        """Outputs of the router: experts, then identity experts."""
        return self.experts + self.identity

    @property
    def gated(self) -> bool:
        return self.act in ("clamped_swish", "swiglu")


@dataclass(frozen=True)
class LayerSpec:
    """One layer of a composed stack (``ModelConfig.layer_specs``): its token mixer with the mixer's sizes and its
    feed-forward.  ``hgrn2``: gated linear recurrence with ``heads`` states of ``dim x vdim``.  ``latent_attention``:
    softmax attention whose keys and values are projections of one cached latent row of ``kv_rank`` features per token;
    with ``rot_dims`` every head's query has that many rotated features more, which meet ONE rotated key part that the row
    holds for all heads.  ``attention``: softmax attention over cached keys and values of ``kv_heads`` heads.  ``mingru``: ``vdim``
    channels that each follow a gated running mean.  ``gla``: linear attention with ``heads`` states of ``dim x vdim`` whose rows decay by
    gates of their own, read-outs normed head by head and gated.  ``pair``: the mixers of ``pair`` side by side on the same input;
    the layer's output is half the sum of theirs, each RMS-normed over the model width with a weight."""
    mixer: str
    heads: int = 1
    dim: int = 1                 # query (and key / forget-gate) features per head (latent_attention: the unrotated ones)
    vdim: int = 1                # value features per head
    kv_rank: int = 0             # latent_attention only
    scale: float = 1.0           # attention mixers: factor on q . k
    ff: int = 0                  # width of the gated feed-forward; 0 = the layer has none
    act: str = "gelu_tanh"       # activation of the feed-forward's gate half
    out_gate: bool = False       # attention mixers: a gate per output feature, sigmoid(W_g h); latent_attention without: one per head
    rot_dims: int = 0            # rotated features of queries and keys (attention: the leading ones of a head)
    rot_base: float = 0.0        # pair i turns by position * rot_base ** (-2 i / rot_dims)
    # attention only
    kv_heads: int = 0            # query head h reads key / value head h // (heads / kv_heads)
    rot_halves: bool = False     # pairs are features i and i + rot_dims / 2 instead of neighbours
    qk_norm: bool = False        # rotated queries and keys divided by their root mean square, head by head
    proj_norm: bool = False      # weighted RMS norm over all query rows, and over all key rows, before heads and rotation
    window: int = 0              # a position sees itself and the window - 1 before it; 0 = all before it
    sink: bool = False           # one learned logit per head in the softmax denominator, without key or value
    unit_sink: bool = False      # a sink whose logit is 0 (one more in the softmax denominator)
    kv_from: int = -1            # >= 0: reads the keys and values that this earlier layer has cached, and has none of its own
    keep_first: int = 0          # with a window: the first positions of a sequence stay visible
    chunk: int = 0               # > 0: a position sees only those of its own chunk of this many, counted from the sequence's start
    softcap: float = 0.0         # > 0: scores s become softcap * tanh(s / softcap)
    talk: bool = False           # the heads' weights are mixed by a learned [heads, heads] matrix before they meet the values
    qkv_bias: bool = False       # biases of the query, key and value projections
    conv: int = 0                # > 0: taps of a causal convolution over time on every channel of the projected q, k and v
    head_norm: bool = False      # queries and keys RMS-normed head by head with a weight (shared by heads), before they turn
    rot_scaling: Optional[tuple] = None   # (factor, low, high, original): long wavelengths stretched as in Llama 3.1
    # gla only
    decay_rank: int = 0          # rank of the gates' projection
    decay_root: float = 1.0      # gates are sigmoid(z) ** (1 / decay_root)
    pair: Optional[tuple] = None          # pair only: two LayerSpecs without feed-forwards
    moe: Optional[MoESpec] = None  # routed feed-forward instead of the gated one

    def __post_init__(self):
        if self.mixer not in MIXERS:
            raise ValueError(f"unknown mixer {self.mixer!r}; known: {MIXERS}")
        if min(self.heads, self.dim, self.vdim) < 1 or (self.mixer == "latent_attention" and self.kv_rank < 1) or min(self.ff, self.window) < 0:
            raise ValueError(f"bad layer sizes: {self}")
        if self.act not in ACTIVATIONS[:2] or (self.moe is not None and self.ff):
            raise ValueError(f"bad feed-forward: {self}")
        if self.rot_dims % 2 or self.rot_dims < 0 or (self.rot_dims and self.rot_base <= 0):
            raise ValueError(f"bad rotation: {self.rot_dims} features, base {self.rot_base}")
        if self.mixer == "attention":
            if self.kv_heads < 1 or self.heads % self.kv_heads:
                raise ValueError(f"{self.kv_heads} key / value heads do not divide {self.heads} heads")
            if self.rot_dims > self.dim:
                raise ValueError(f"bad rotation: {self.rot_dims} of {self.dim} features, base {self.rot_base}")
            if self.qk_norm and (self.proj_norm or self.rot_halves):
                raise ValueError("queries and keys normed head by head turn in neighbouring pairs and have no norm over the projection")
            if (self.conv or self.qkv_bias or self.head_norm) and (self.qk_norm or self.proj_norm or self.rot_halves):
                raise ValueError("projections with biases, convolutions or weighted head norms turn in neighbouring pairs and have no other norm")
            if not 0 <= self.conv <= MAX_TAPS or min(self.keep_first, self.chunk) < 0 or self.softcap < 0:
                raise ValueError(f"bad attention: {self}")
            if (self.window and self.chunk) or (self.keep_first and not self.window) or (self.sink and self.unit_sink) or (self.talk and self.out_gate):
                raise ValueError(f"attention layers see a window (with or without first positions) or a chunk, have one sink, and gates or mixed heads: {self}")
        if self.rot_scaling is not None and (len(self.rot_scaling) != 4 or min(self.rot_scaling) <= 0 or self.rot_scaling[1] >= self.rot_scaling[2]):
            raise ValueError(f"bad rotation scaling: {self.rot_scaling}")
        if self.mixer == "gla" and (self.decay_rank < 1 or self.decay_root <= 0):
            raise ValueError(f"bad decay: {self}")
        if (self.mixer == "pair") != (self.pair is not None):
            raise ValueError(f"a pair has two mixers: {self}")
        if self.pair is not None and (len(self.pair) != 2 or any(s.mixer == "pair" or s.has_ff or s.kv_from >= 0 for s in self.pair)):
            raise ValueError("a pair is made of two plain mixers with inputs of their own and without feed-forwards")

    @property
    def has_ff(self) -> bool:
        return self.ff > 0 or self.moe is not None

    @property
    def own_kv(self) -> bool:
        """An attention layer that projects and caches keys and values."""
        return self.mixer == "attention" and self.kv_from < 0


MIXERS = ("hgrn2", "latent_attention", "attention", "mingru", "gla", "pair")
MAX_TAPS = 8           # of a short convolution
ACTIVATIONS = ("silu", "gelu_tanh", "relu2")
EXPERT_ACTIVATIONS = ("relu2", "clamped_swish", "swiglu")


@dataclass
class ModelConfig:
    name: str = "tiny"
    num_layers: int = 2
    hidden_size: int = 256
    num_attention_heads: int = 4
    num_query_groups: int = 2
    head_dim: int = 64
    ffn_hidden_size: int = 688
    vocab_size: int = 1024
    rms_norm_eps: float = 1e-6
    rope_theta: float = 1e6
    qk_layernorm: bool = True
    qkv_bias: bool = False
    tie_word_embeddings: bool = False
    # MoE
    num_experts: int = 0
    moe_top_k: int = 0
    moe_ffn_hidden_size: int = 0
    moe_router_norm_topk_prob: bool = True
    moe_aux_loss_coef: float = 0.0
    moe_layer_freq: int = 1
    moe_first_dense_layers: int = 0        # DeepSeek-V3 / GLM4-MoE: the first k layers keep a dense MLP
    moe_shared_expert_ffn: int = 0         # >0: an always-on shared expert of this width beside the routed ones
    moe_shared_expert_gate: bool = False   # Qwen2-MoE / Qwen3-Next: shared output scaled by sigmoid(gate(x))
    moe_router_score: str = "softmax"      # softmax | sigmoid (DeepSeek-V3 / GLM4-MoE)
    moe_router_bias: bool = False          # selection-only per-expert bias, balanced without an auxiliary loss
    moe_routed_scaling_factor: float = 1.0
    moe_router_bias_update_rate: float = 1e-3
    # multimodal
    vision: Optional[VisionConfig] = None
    mrope_section: Optional[tuple] = None  # (t, h, w) halves of head_dim/2
    image_token_id: int = -1
    # value / classification head
    value_head: bool = False
    num_classes: int = 0                  # >0: sequence-classification head on the last token
    # multi-token prediction blocks after the trunk (0 = none)
    mtp_num_layers: int = 0
    # Qwen3.5-style softmax attention: a sigmoid gate on the attention output (the query projection also produces one
    # gate value per query feature) and rotary embedding on the first `rotary_percent` of every head only
    attention_output_gate: bool = False
    rotary_percent: float = 1.0
    # GLM-4 dense: "sandwich" norms - the attention and MLP outputs are normalised once more before they join the residual
    sandwich_norm: bool = False
    # norm weights are stored zero-centred (gamma - 1) in this family's checkpoints (``--apply-layernorm-1p``); the model
    # keeps gamma, the Hugging Face conversion adds / removes the offset
    layernorm_zero_centered: bool = False
    # hybrid stacks: every `linear_attention_freq`-th layer is softmax attention, the others Gated DeltaNet (0 = all softmax)
    linear_attention_freq: int = 0
    gdn_k_heads: int = 2
    gdn_v_heads: int = 4
    gdn_head_dim: int = 32
    # multi-head latent attention (DeepSeek-V3 / GLM-4.7 style, dims below); with dsa_topk > 0 it is sparse (DSA)
    multi_latent_attention: bool = False
    dsa_topk: int = 0
    dsa_q_lora: int = 64
    dsa_kv_lora: int = 32
    dsa_nope: int = 16
    dsa_rope: int = 8
    dsa_v_head: int = 16
    dsa_index_heads: int = 4
    dsa_index_dim: int = 16
    dsa_indexer_loss_coef: float = 1.0
    # composed stacks (Talizen, Ketolorn, Zupupel, Zoguzen): every layer is spelled out - mixer, sizes, feed-forward.  The sublayers read the
    # fp32 residual stream itself.  Their OUTPUT is normed (RMS over each of `norm_groups` equal parts) before it is added, or,
    # with `norm_sum`, the SUM is: x <- norm(sum_alpha * x + sublayer(x)), a layer norm with weight and bias (as is the final norm).
    # With `pre_norm` the sublayers read norms of the stream instead (layer norms with a weight), and both join it at once:
    # x <- x + mixer(norm1(x)) + ff(norm2(x)).  `token_shift`: what the mixer reads has moved towards the row before, by a weight per
    # feature.  `side_dim`: every layer then adds the norm of a projection of gelu(gate x) times its own part of a second embedding.
    # The fields above that describe one uniform layer (heads, head_dim, ffn, rotary, MoE, ...) do not apply then.
    layer_specs: Optional[tuple] = None
    norm_groups: int = 1
    norm_sum: bool = False
    sum_alpha: float = 1.0
    embed_norm: bool = False               # the embedded tokens are normed before the first layer
    embed_scale: float = 1.0               # factor on the embedded tokens
    logit_scale: float = 1.0               # factor on the logits
    logit_softcap: float = 0.0             # > 0: logits z become logit_softcap * tanh(z / logit_softcap)
    pre_norm: bool = False
    token_shift: bool = False
    side_dim: int = 0                      # features per layer and token of the second embedding
    dtype: str = "bf16"

    @property
    def is_composed(self) -> bool:
        return self.layer_specs is not None

    def mixers(self) -> list:
        """``(key, spec)`` of every mixer of a composed stack: ``i`` for layer ``i``, ``(i, 0)`` and ``(i, 1)`` for the two of a pair."""
        out = []
        for i, s in enumerate(self.layer_specs or ()):
            out += [((i, k), m) for k, m in enumerate(s.pair)] if s.pair is not None else [(i, s)]
        return out

    def specs_with(self, *mixers: str) -> list:
        """Specs of the mixers of these kinds, those inside pairs included."""
        return [s for _, s in self.mixers() if s.mixer in mixers]

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    def is_moe_layer(self, layer_idx: int) -> bool:
        return self.is_moe and layer_idx >= self.moe_first_dense_layers and layer_idx % self.moe_layer_freq == 0

    @property
    def q_size(self) -> int:
        return self.num_attention_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_query_groups * self.head_dim

    @property
    def rotary_dim(self) -> int:
        """Leading features of a head that are rotated (even; the whole head unless ``rotary_percent`` < 1)."""
        return self.head_dim if self.rotary_percent >= 1.0 else max(2, int(self.head_dim * self.rotary_percent) // 2 * 2)

    def num_parameters(self) -> int:
        h, L = self.hidden_size, self.num_layers
        if self.is_composed:
            norm = 2 * h if self.norm_sum else h
            n = (1 if self.tie_word_embeddings else 2) * self.vocab_size * h + norm + (h if self.embed_norm else 0)
            n += self.side_dim * self.num_layers * self.vocab_size
            for s in self.layer_specs:
                n += norm + 3 * s.ff * h + (norm if s.has_ff else 0) + (h if self.token_shift else 0) + ((2 * self.side_dim + 1) * h if self.side_dim else 0)
                if s.moe is not None:
                    n += s.moe.experts * (3 if s.moe.gated else 2) * s.moe.ff * h + 2 * s.moe.shared_ff * h
                    n += s.moe.outputs * (h + (1 if s.moe.correction else 0))
                n += self._mixer_parameters(s) if s.pair is None else 2 * h + sum(self._mixer_parameters(m) for m in s.pair)
            return n
        attn = h * (self.q_size * (2 if self.attention_output_gate else 1) + 2 * self.kv_size) + self.q_size * h
        if self.qk_layernorm:
            attn += 2 * self.head_dim
        if self.is_moe:
            mlp = self.num_experts * 3 * h * self.moe_ffn_hidden_size + h * self.num_experts
        else:
            mlp = 3 * h * self.ffn_hidden_size
        per_layer = attn + mlp + 2 * h
        emb = self.vocab_size * h
        out = 0 if self.tie_word_embeddings else self.vocab_size * h
        return L * per_layer + emb + out + h

    def _mixer_parameters(self, s: LayerSpec) -> int:
        h = self.hidden_size
        n = s.heads * s.vdim * h
        if s.mixer == "hgrn2":
            return n + s.heads * (2 * s.dim + s.vdim) * h + 2 * s.heads * s.dim + s.vdim
        if s.mixer == "mingru":
            return n + 3 * s.vdim * h + 2 * s.vdim
        if s.mixer == "gla":
            return n + s.heads * (2 * s.dim + 2 * s.vdim) * h + s.decay_rank * (h + s.heads * s.dim) + s.heads * s.dim + s.vdim
        if s.mixer == "attention":
            cols = s.heads * s.dim + (s.kv_heads * (s.dim + s.vdim) if s.own_kv else 0)
            n += cols * (h + s.conv + (1 if s.qkv_bias else 0)) + (s.heads if s.sink else 0) + (s.heads ** 2 if s.talk else 0)
            n += (2 if s.own_kv else 1) * s.dim if s.head_norm else 0
            return n + (s.heads * s.vdim * h if s.out_gate else 0) + ((s.heads + (s.kv_heads if s.own_kv else 0)) * s.dim if s.proj_norm else 0)
        n += (s.heads * (s.dim + s.rot_dims + (s.vdim if s.out_gate else 1)) + s.kv_rank + s.rot_dims) * h
        return n + s.kv_rank * (1 + s.heads * (s.dim + s.vdim))

    def to_dict(self):
        return asdict(self)


PRESETS: dict[str, ModelConfig] = {}


def _reg(c: ModelConfig):
    PRESETS[c.name] = c
    return c


def composed_config(name: str, layers, hidden_size: int, vocab_size: int, norm_groups: int = 1, eps: float = 1e-5, **kw) -> ModelConfig:
    """A composed stack from its list of :class:`LayerSpec`."""
    layers = tuple(layers)
    if not layers:
        raise ValueError("a composed stack needs at least one layer")
    if norm_groups < 1 or hidden_size % norm_groups:
        raise ValueError(f"{norm_groups} norm groups do not divide the width {hidden_size}")
    if kw.get("norm_sum") and (norm_groups > 1 or kw.get("embed_norm")):
        raise ValueError("norms after the sum span the whole width, and leave the embedded tokens as they are")
    if not kw.get("norm_sum") and (kw.get("sum_alpha", 1.0) != 1.0 or kw.get("logit_scale", 1.0) != 1.0):
        raise ValueError("factors on the stream and on the logits join the norm after the sum")
    if kw.get("embed_norm") and kw.get("embed_scale", 1.0) != 1.0:
        raise ValueError("embedded tokens are normed or scaled")
    if kw.get("pre_norm") and (norm_groups > 1 or kw.get("norm_sum") or kw.get("embed_norm") or kw.get("embed_scale", 1.0) != 1.0 or any(
            s.ff or (s.moe and s.moe.shared_ff) for s in layers)):
        raise ValueError("sublayers that read norms of the stream come with routed feed-forwards and without norms of their outputs or of embedded tokens")
    if not kw.get("pre_norm") and (kw.get("token_shift") or kw.get("side_dim") or any(s.pair is not None for s in layers)):
        raise ValueError("shifted tokens, a second embedding and pairs of mixers join sublayers that read norms of the stream")
    for i, s in enumerate(layers):
        if s.mixer == "attention" and s.kv_from >= 0:
            if s.kv_from >= i or not layers[s.kv_from].own_kv:
                raise ValueError(f"layer {i} reads keys and values of layer {s.kv_from}, which has none before it")
            what = ("kv_heads", "dim", "vdim", "rot_dims", "rot_base", "rot_scaling", "rot_halves", "qk_norm", "proj_norm", "head_norm")
            if any(getattr(s, f) != getattr(layers[s.kv_from], f) for f in what):
                raise ValueError(f"layer {i} and the layer {s.kv_from} whose keys and values it reads differ in {what}")
    return ModelConfig(name=name, num_layers=len(layers), hidden_size=hidden_size, vocab_size=vocab_size, rms_norm_eps=eps,
                       layer_specs=layers, norm_groups=norm_groups, qk_layernorm=False, **kw)


def window_latent_layers(n_layers: int, att: LayerSpec, lat: LayerSpec, moe: Optional[MoESpec]) -> tuple:
    """Runs of three layers: ``att``, ``lat``, and ``att`` on the keys and values of the run's first layer; ``moe`` in all of them."""
    out = []
    for i in range(n_layers):
        s = lat if i % 3 == 1 else (att if i % 3 == 0 else replace(att, kv_from=i - 2))
        out.append(replace(s, moe=moe))
    return tuple(out)


def chunk_mean_pair_layers(n_layers: int, att: LayerSpec, mean: LayerSpec, pair: LayerSpec, moe: Optional[MoESpec]) -> tuple:
    """Runs of four layers: ``att``, ``mean``, ``pair``, and ``att`` on the keys and values of the run's first layer; ``moe`` in all of them."""
    out = []
    for i in range(n_layers):
        out.append(replace((att, mean, pair, replace(att, kv_from=i - 3))[i % 4], moe=moe))
    return tuple(out)


def talizen_layers(n_layers: int, every: int, rec: LayerSpec, att: LayerSpec) -> tuple:
    """``every - 1`` recurrent layers, then one latent-attention layer, repeated."""
    return tuple(att if (i + 1) % every == 0 else rec for i in range(n_layers))


def shared_kv_layers(n_layers: int, own: int, att: LayerSpec, dense_ff: int, moe: MoESpec, first_dense: int = 1) -> tuple:
    """Attention layers of which the first ``own`` cache keys and values and the others read those of layer ``own - 1``; the
    first ``first_dense`` have a gated feed-forward, the others routed experts."""
    kv = lambda i: {} if i < own else {"kv_from": own - 1}
    ff = lambda i: {"ff": dense_ff} if i < first_dense else {"moe": moe}
    return tuple(replace(att, **kv(i), **ff(i)) for i in range(n_layers))


# BASELINE config 0 ("tiny Qwen-style decoder")
_reg(ModelConfig(name="tiny", num_layers=2, hidden_size=256, num_attention_heads=4, num_query_groups=2,
                 head_dim=64, ffn_hidden_size=688, vocab_size=1024, dtype="fp32"))
_reg(ModelConfig(name="tiny-moe", num_layers=2, hidden_size=256, num_attention_heads=4, num_query_groups=2,
                 head_dim=64, ffn_hidden_size=688, vocab_size=1024, num_experts=8, moe_top_k=2,
                 moe_ffn_hidden_size=128, dtype="fp32"))
_reg(ModelConfig(name="tiny-next", num_layers=4, hidden_size=128, num_attention_heads=4, num_query_groups=2, head_dim=32,
                 ffn_hidden_size=256, vocab_size=512, linear_attention_freq=4, dtype="fp32"))
_reg(ModelConfig(name="tiny-vl", num_layers=2, hidden_size=256, num_attention_heads=4, num_query_groups=2, head_dim=64,
                 ffn_hidden_size=688, vocab_size=1024, dtype="fp32", mrope_section=(8, 12, 12), image_token_id=7,
                 vision=VisionConfig(num_layers=1, hidden_size=64, num_heads=2, ffn_hidden_size=96, patch_size=4,
                                     out_hidden_size=256)))
_reg(ModelConfig(name="tiny-glm4", num_layers=2, hidden_size=128, num_attention_heads=4, num_query_groups=2, head_dim=32,
                 ffn_hidden_size=256, vocab_size=512, qk_layernorm=False, qkv_bias=True, sandwich_norm=True, rotary_percent=0.5,
                 dtype="fp32"))
# GLM-4-9B-0414 / GLM-Z1 shape (trainer-side family like the other non-plain attention stacks)
_reg(ModelConfig(name="glm4-9b", num_layers=40, hidden_size=4096, num_attention_heads=32, num_query_groups=2, head_dim=128,
                 ffn_hidden_size=13696, vocab_size=151552, qk_layernorm=False, qkv_bias=True, sandwich_norm=True, rotary_percent=0.5,
                 rope_theta=1e4, rms_norm_eps=1e-5))
_reg(ModelConfig(name="tiny-qwen35", num_layers=4, hidden_size=128, num_attention_heads=4, num_query_groups=2, head_dim=32,
                 ffn_hidden_size=256, vocab_size=512, linear_attention_freq=4, attention_output_gate=True, rotary_percent=0.25,
                 dtype="fp32"))
_reg(ModelConfig(name="tiny-dsa", num_layers=2, hidden_size=128, num_attention_heads=4, num_query_groups=4, head_dim=32,
                 ffn_hidden_size=256, vocab_size=512, dsa_topk=8, dtype="fp32"))
_reg(ModelConfig(name="tiny-dsv3", num_layers=3, hidden_size=256, num_attention_heads=4, num_query_groups=2,
                 head_dim=64, ffn_hidden_size=688, vocab_size=1024, num_experts=8, moe_top_k=2, moe_ffn_hidden_size=128,
                 moe_first_dense_layers=1, moe_shared_expert_ffn=128, moe_router_score="sigmoid", moe_router_bias=True,
                 moe_routed_scaling_factor=2.5, dtype="fp32"))
# scripts/models/glm4.7-30B-A3B.sh: MLA + sigmoid-routed MoE with one shared expert and one leading dense layer
_reg(ModelConfig(name="glm4.7-30b-a3b", num_layers=47, hidden_size=2048, num_attention_heads=20, num_query_groups=20, head_dim=192,
                 ffn_hidden_size=10240, vocab_size=154880, qkv_bias=True, num_experts=64, moe_top_k=4, moe_ffn_hidden_size=1536,
                 moe_first_dense_layers=1, moe_shared_expert_ffn=1536, moe_router_score="sigmoid", moe_router_bias=True,
                 moe_router_bias_update_rate=0.0, moe_routed_scaling_factor=1.8, multi_latent_attention=True, dsa_q_lora=768,
                 dsa_kv_lora=512, dsa_nope=192, dsa_rope=64, dsa_v_head=256))
_reg(ModelConfig(name="tiny-mla", num_layers=2, hidden_size=128, num_attention_heads=4, num_query_groups=4, head_dim=32,
                 ffn_hidden_size=256, vocab_size=512, multi_latent_attention=True, dtype="fp32"))
_reg(ModelConfig(name="qwen3-1.7b", num_layers=28, hidden_size=2048, num_attention_heads=16, num_query_groups=8,
                 head_dim=128, ffn_hidden_size=6144, vocab_size=151936, tie_word_embeddings=True))
_reg(ModelConfig(name="qwen2.5-7b", num_layers=28, hidden_size=3584, num_attention_heads=28, num_query_groups=4,
                 head_dim=128, ffn_hidden_size=18944, vocab_size=152064, qk_layernorm=False, qkv_bias=True))
_reg(ModelConfig(name="qwen3-vl-8b", num_layers=36, hidden_size=4096, num_attention_heads=32, num_query_groups=8,
                 head_dim=128, ffn_hidden_size=12288, vocab_size=151936, rope_theta=5e6,
                 vision=VisionConfig(out_hidden_size=4096), mrope_section=(24, 20, 20), image_token_id=151655))
# Qwen3-VL family (scripts/models/qwen3-vl-*.sh of the reference): the language-model shapes of those recipes with the
# Qwen-VL tower of this package; the 30B-A3B variant is the MoE shape
_reg(ModelConfig(name="qwen3-vl-2b", num_layers=28, hidden_size=2048, num_attention_heads=16, num_query_groups=8,
                 head_dim=128, ffn_hidden_size=6144, vocab_size=151936, rope_theta=1e6,
                 vision=VisionConfig(out_hidden_size=2048), mrope_section=(24, 20, 20), image_token_id=151655))
_reg(ModelConfig(name="qwen3-vl-4b", num_layers=36, hidden_size=2560, num_attention_heads=32, num_query_groups=8,
                 head_dim=128, ffn_hidden_size=9728, vocab_size=151936, rope_theta=5e6, tie_word_embeddings=True,
                 vision=VisionConfig(out_hidden_size=2560), mrope_section=(24, 20, 20), image_token_id=151655))
_reg(ModelConfig(name="qwen3-vl-30b-a3b", num_layers=48, hidden_size=2048, num_attention_heads=32, num_query_groups=4,
                 head_dim=128, ffn_hidden_size=6144, vocab_size=151936, rope_theta=5e6, num_experts=128, moe_top_k=8,
                 moe_ffn_hidden_size=768, vision=VisionConfig(out_hidden_size=2048), mrope_section=(24, 20, 20),
                 image_token_id=151655))
_reg(ModelConfig(name="qwen3-omni-30b-a3b", num_layers=48, hidden_size=2048, num_attention_heads=32, num_query_groups=4,
                 head_dim=128, ffn_hidden_size=768, vocab_size=152064, rope_theta=1e6, num_experts=128, moe_top_k=8,
                 moe_ffn_hidden_size=768, vision=VisionConfig(out_hidden_size=2048), mrope_section=(24, 20, 20),
                 image_token_id=151655))
# Qwen3.5 family (scripts/models/qwen35-*.sh): hybrid stack - three Gated-DeltaNet layers, then one gated softmax-attention
# layer with 256-wide heads and rotary on their first quarter.  Trainer-side families (the rollout engine serves plain
# softmax attention).
_reg(ModelConfig(name="qwen3.5-9b", num_layers=32, hidden_size=4096, num_attention_heads=16, num_query_groups=4, head_dim=256,
                 ffn_hidden_size=12288, vocab_size=248320, rope_theta=1e7, attention_output_gate=True, rotary_percent=0.25,
                 layernorm_zero_centered=True, linear_attention_freq=4, gdn_k_heads=16, gdn_v_heads=32, gdn_head_dim=128))
_reg(ModelConfig(name="qwen3.5-35b-a3b", num_layers=40, hidden_size=2048, num_attention_heads=16, num_query_groups=2, head_dim=256,
                 ffn_hidden_size=512, vocab_size=248320, rope_theta=1e7, attention_output_gate=True, rotary_percent=0.25,
                 layernorm_zero_centered=True, linear_attention_freq=4, gdn_k_heads=16, gdn_v_heads=32, gdn_head_dim=128, num_experts=256, moe_top_k=8,
                 moe_ffn_hidden_size=512, moe_shared_expert_ffn=512, moe_shared_expert_gate=True))
# dots.ocr (scripts/models/dotsocr2.sh): a Qwen2.5-1.5B-shaped language model behind the dots tower (42 blocks of 1536, head_dim 128)
_reg(ModelConfig(name="dotsocr2", num_layers=28, hidden_size=1536, num_attention_heads=12, num_query_groups=2, head_dim=128,
                 ffn_hidden_size=8960, vocab_size=151936, qk_layernorm=False, qkv_bias=True, rope_theta=1e6,
                 vision=VisionConfig(num_layers=42, hidden_size=1536, num_heads=12, ffn_hidden_size=4224, temporal_patch_size=1,
                                     out_hidden_size=1536, patch_norm=True, post_trunk_norm=True, merger_layernorm=True,
                                     rms_norm_eps=1e-5),
                 mrope_section=(16, 24, 24), image_token_id=151655))
_reg(ModelConfig(name="qwen3-0.6b", num_layers=28, hidden_size=1024, num_attention_heads=16, num_query_groups=8,
                 head_dim=128, ffn_hidden_size=3072, vocab_size=151936, tie_word_embeddings=True))
_reg(ModelConfig(name="qwen3-4b", num_layers=36, hidden_size=2560, num_attention_heads=32, num_query_groups=8,
                 head_dim=128, ffn_hidden_size=9728, vocab_size=151936, tie_word_embeddings=True))
_reg(ModelConfig(name="qwen3-8b", num_layers=36, hidden_size=4096, num_attention_heads=32, num_query_groups=8,
                 head_dim=128, ffn_hidden_size=12288, vocab_size=151936))
_reg(ModelConfig(name="qwen3-32b", num_layers=64, hidden_size=5120, num_attention_heads=64, num_query_groups=8,
                 head_dim=128, ffn_hidden_size=25600, vocab_size=151936))
_reg(ModelConfig(name="qwen3-30b-a3b", num_layers=48, hidden_size=2048, num_attention_heads=32, num_query_groups=4,
                 head_dim=128, ffn_hidden_size=6144, vocab_size=151936, num_experts=128, moe_top_k=8,
                 moe_ffn_hidden_size=768))
_reg(ModelConfig(name="qwen2.5-vl-7b", num_layers=28, hidden_size=3584, num_attention_heads=28, num_query_groups=4,
                 head_dim=128, ffn_hidden_size=18944, vocab_size=152064, qk_layernorm=False, qkv_bias=True,
                 vision=VisionConfig(), mrope_section=(16, 24, 24), image_token_id=151655))
_reg(ModelConfig(name="llama3-8b", num_layers=32, hidden_size=4096, num_attention_heads=32, num_query_groups=8,
                 head_dim=128, ffn_hidden_size=14336, vocab_size=128256, qk_layernorm=False, rope_theta=5e5,
                 rms_norm_eps=1e-5))


# Talizen: HGRN2 recurrent layers with a latent-attention layer among every few of them
_reg(composed_config("tiny-talizen", [LayerSpec("hgrn2", heads=3, dim=16, vdim=24), LayerSpec("hgrn2", heads=3, dim=16, vdim=24, ff=160),
                                      LayerSpec("latent_attention", heads=4, dim=32, vdim=16, kv_rank=48, scale=0.2, ff=224)],
                     hidden_size=192, vocab_size=384, norm_groups=2, dtype="fp32"))
_reg(composed_config("talizen-1b", talizen_layers(32, 4, LayerSpec("hgrn2", heads=16, dim=128, vdim=128),
                                                  LayerSpec("latent_attention", heads=16, dim=128, vdim=128, kv_rank=512,
                                                            scale=128 ** -0.5, ff=8192)),
                     hidden_size=2048, vocab_size=64000, norm_groups=8))
_reg(composed_config("talizen-5b", talizen_layers(36, 4, LayerSpec("hgrn2", heads=32, dim=128, vdim=128),
                                                  LayerSpec("latent_attention", heads=32, dim=128, vdim=128, kv_rank=512,
                                                            scale=128 ** -0.5, ff=12288)),
                     hidden_size=4096, vocab_size=151936, norm_groups=8))

# Ketolorn: attention with sinks and normed rotated keys, upper layers on the keys and values of a lower one, grouped experts
_reg(composed_config("tiny-ketolorn", shared_kv_layers(
    4, 2, LayerSpec("attention", heads=6, dim=32, vdim=24, kv_heads=2, scale=0.3, rot_dims=16, rot_base=1e4, qk_norm=True, sink=True, act="silu"),
    160, MoESpec(experts=8, top=2, ff=48, groups=4, keep=2, shared_ff=96)), hidden_size=160, vocab_size=320, eps=1e-6, embed_norm=True,
    tie_word_embeddings=True, dtype="fp32"))
_reg(composed_config("ketolorn-16b", shared_kv_layers(
    24, 12, LayerSpec("attention", heads=32, dim=128, vdim=128, kv_heads=4, scale=128 ** -0.5, rot_dims=64, rot_base=1e6, qk_norm=True, sink=True,
                      act="silu"),
    8192, MoESpec(experts=128, top=8, ff=1024, groups=8, keep=4, shared_ff=2048)), hidden_size=2048, vocab_size=64000, eps=1e-6, embed_norm=True,
    tie_word_embeddings=True))

# Zupupel: sliding-window attention, latent attention with a rotated key part, upper window layers on the keys and values of a lower
# one, experts beside identity experts, norms after the sum
_reg(composed_config("tiny-zupupel", window_latent_layers(
    6, LayerSpec("attention", heads=6, dim=24, vdim=32, kv_heads=3, scale=0.2, rot_dims=12, rot_base=1e4, rot_halves=True, proj_norm=True, window=20,
                 out_gate=True),
    LayerSpec("latent_attention", heads=4, dim=24, vdim=20, kv_rank=40, scale=0.18, rot_dims=16, rot_base=1e4, out_gate=True),
    MoESpec(experts=7, top=2, ff=40, groups=3, keep=2, act="clamped_swish", limit=2.0, renormalize=True, score="softmax", correction=True, identity=2,
            group_best=1)), hidden_size=160, vocab_size=320, eps=1e-6, norm_sum=True, sum_alpha=1.8, embed_scale=2.0, logit_scale=0.5, dtype="fp32"))
_reg(composed_config("zupupel-15b", window_latent_layers(
    24, LayerSpec("attention", heads=32, dim=128, vdim=128, kv_heads=4, scale=128 ** -0.5, rot_dims=64, rot_base=1e6, rot_halves=True, proj_norm=True,
                  window=1024, out_gate=True),
    LayerSpec("latent_attention", heads=32, dim=128, vdim=128, kv_rank=512, scale=192 ** -0.5, rot_dims=64, rot_base=1e6, out_gate=True),
    MoESpec(experts=128, top=8, ff=768, groups=8, keep=4, act="clamped_swish", limit=7.0, renormalize=True, score="softmax", correction=True, identity=16,
            group_best=1)), hidden_size=2048, vocab_size=64000, eps=1e-6, norm_sum=True, sum_alpha=48 ** 0.25, embed_scale=45.0, logit_scale=1 / 45))


# Zoguzen: attention inside chunks with mixed heads, running means, sliding-window attention beside linear attention, upper chunk layers
# on the keys and values of a lower one; sublayers on norms of the stream, a second embedding, gated experts
_reg(composed_config("tiny-zoguzen", chunk_mean_pair_layers(
    5, LayerSpec("attention", heads=6, dim=24, vdim=32, kv_heads=3, scale=0.2, chunk=24, softcap=9.0, unit_sink=True, talk=True, qkv_bias=True, conv=3,
                 head_norm=True),
    LayerSpec("mingru", vdim=72),
    LayerSpec("pair", pair=(LayerSpec("attention", heads=4, dim=16, vdim=24, kv_heads=2, scale=0.3, window=20, keep_first=3, rot_dims=8, rot_base=1e4,
                                      rot_scaling=(2.0, 1.0, 4.0, 64.0), conv=3, out_gate=True),
                            LayerSpec("gla", heads=3, dim=16, vdim=24, decay_rank=8, decay_root=8.0))),
    MoESpec(experts=6, top=2, ff=40, act="swiglu", score="softmax", renormalize=True)), hidden_size=160, vocab_size=320, eps=1e-6, pre_norm=True,
    token_shift=True, side_dim=12, logit_softcap=15.0, tie_word_embeddings=True, dtype="fp32"))
_reg(composed_config("zoguzen-15b", chunk_mean_pair_layers(
    24, LayerSpec("attention", heads=32, dim=128, vdim=128, kv_heads=4, scale=128 ** -0.5, chunk=1024, softcap=30.0, unit_sink=True, talk=True, qkv_bias=True,
                  conv=4, head_norm=True),
    LayerSpec("mingru", vdim=4096),
    LayerSpec("pair", pair=(LayerSpec("attention", heads=16, dim=128, vdim=128, kv_heads=4, scale=128 ** -0.5, window=1024, keep_first=16, rot_dims=128,
                                      rot_base=5e5, rot_scaling=(8.0, 1.0, 4.0, 8192.0), conv=4, out_gate=True),
                            LayerSpec("gla", heads=16, dim=64, vdim=128, decay_rank=16, decay_root=16.0))),
    MoESpec(experts=128, top=8, ff=768, act="swiglu", score="softmax", renormalize=True)), hidden_size=2048, vocab_size=64000, eps=1e-6, pre_norm=True,
    token_shift=True, side_dim=256, logit_softcap=30.0, tie_word_embeddings=True))


def get_config(name: str, **overrides) -> ModelConfig:
    if name not in PRESETS:
        raise KeyError(f"unknown model preset {name!r}; known: {sorted(PRESETS)}")
    return replace(PRESETS[name], **overrides)
