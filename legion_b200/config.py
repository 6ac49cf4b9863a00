"""Model hyper-parameters (one dataclass for every supported architecture) and named presets.

The reference keeps these in ``Hparams`` read from GGUF metadata (``src/model/core.rs:170-203``) plus
per-architecture hooks (``src/model/core/arch.rs:82-526``); here every architecture is a configuration of
the same block library, selected by ``layer_kinds`` and the MoE / attention fields.
"""
from __future__ import annotations

import dataclasses
import json
from dataclasses import dataclass, field
from typing import List, Optional


# --------------------------------------------------------------------------------------------------
# Layer specifications: stacks whose layers each have sizes and constants of their own (``ModelConfig.layers``)
# --------------------------------------------------------------------------------------------------
@dataclass
class AttnSpec:
    """Grouped-query softmax attention; values may have a head size of their own. Between projection and scores, all
    optional and in this order: a bias, a short causal convolution per channel of q, k and v, a norm of q and k, rotation."""
    heads: int
    kv_heads: int
    dim: int                           # query / key head size
    vdim: int                          # value head size
    scale: float                       # multiplies the scores
    window: int = 0                    # tokens a position sees, itself included (0 = all)
    qk_norm: bool = True               # RMS norm of q and k with a plain weight
    norm_over: str = "head"            # each head by itself | all: the whole of q (of k) at once, a weight per column
    bias: bool = False                 # of the q, k and v projections
    conv: int = 0                      # taps of the short convolution (0: none)
    rot: Optional["RotarySpec"] = None
    softcap: float = 0.0               # cap * tanh(score / cap)
    keep_first: int = 0                # with a window: this many first tokens of the sequence stay visible
    sink: bool = False                 # a learned number per head whose exponential joins the softmax's denominator
    gate: str = "none"                 # head: each head's output times the sigmoid of one more row of the projection
    kind: str = "attn"

    def direct(self) -> bool:
        """Whether q, k and v come straight from the projection, up to head norms."""
        return not (self.conv or self.rot or self.bias or (self.qk_norm and self.norm_over != "head"))


@dataclass
class LightningSpec:
    """Linear attention with a constant decay per head, silu on q, k and v, a norm over all heads and an output gate."""
    heads: int
    dim: int
    vdim: int
    decay: list                        # per head
    kind: str = "lightning"


@dataclass
class SsdSpec:
    """Mamba-2 mixer."""
    heads: int
    vdim: int                          # head size
    state: int
    groups: int = 1                    # B / C groups
    conv: int = 4                      # taps
    norm_groups: int = 1               # parts of the gated norm
    kind: str = "ssd"


@dataclass
class Hgrn2Spec:
    """HGRN2: a matrix state per head whose rows keep the share f of themselves and take 1 - f of the value, f a vector over
    the key channels held above a learned lower bound; silu on q, an RMS norm per head behind the state."""
    heads: int
    dim: int                           # query / forget-gate head size
    vdim: int
    kind: str = "hgrn2"


@dataclass
class ParallelSpec:
    """Two mixers side by side over the same input: left_scale * left + right_scale * right."""
    left: AttnSpec
    right: object                      # SsdSpec | Hgrn2Spec
    left_scale: float = 1.0
    right_scale: float = 1.0
    kind: str = "parallel"


@dataclass
class RotarySpec:
    """Rotation of the first ``dims`` columns of a vector. ``original`` > 0 stretches the low frequencies: ``yarn``
    (frequencies divided by ``factor`` along a ramp between the pairs that turn ``fast`` and ``slow`` times over the
    original context; cos and sin grow by 0.1 ln(factor) + 1) or ``llama3`` (wavelengths above original / low divided by
    ``factor``, those below original / high kept, a blend between)."""
    dims: int
    base: float
    factor: float = 1.0
    original: float = 0.0
    fast: float = 32.0
    slow: float = 1.0
    scaling: str = "yarn"
    low: float = 1.0
    high: float = 4.0
    layout: str = "pairs"              # neighbouring columns | half: column i with column i + dims / 2
    kind: str = "rotary"


@dataclass
class LatentSpec:
    """Latent attention: keys and values of all heads are projections of one cached latent; a rotated key part is shared
    by the heads. The output is gated by the sigmoid of a projection of the input."""
    heads: int
    dim: int                           # query / key columns per head that are not rotated
    rot_dim: int                       # ... and the rotated part
    vdim: int
    kv_rank: int                       # latent size
    scale: float                       # multiplies the scores
    rot: RotarySpec
    gate: str = "channel"              # channel: one gate per output column | head: one per head | none
    kind: str = "latent"

    def gate_width(self) -> int:
        return {"channel": self.heads * self.vdim, "head": self.heads, "none": 0}[self.gate]


@dataclass
class RgLruSpec:
    """Griffin's recurrent block: a short convolution and a real-gated linear recurrent unit beside a GELU branch."""
    width: int
    blocks: int                        # equal parts of the width, each with gate matrices of its own
    conv: int = 4                      # taps
    kind: str = "rglru"


@dataclass
class ChannelDeltaSpec:
    """Gated delta rule with a decay per head and key channel: q, k and v behind a short convolution and silu, unit q and
    k per head, decay and output gate from low-rank projections, an RMS norm per head in front of the gate."""
    heads: int
    kv_heads: int                      # q / k heads, each shared by heads / kv_heads state heads
    dim: int                           # query / key head size
    vdim: int
    conv: int = 4                      # taps
    rank: int = 8                      # width of the low-rank projections (the wider one, a multiple of 8)
    kind: str = "channel_delta"

    def in_columns(self) -> dict:
        """First column of each part of the stacked input projection, and its width (``end``). The low-rank parts start on
        16-byte boundaries."""
        up8 = lambda n: -(-n // 8) * 8                               # noqa: E731
        k = self.kv_heads * self.dim
        b = 2 * k + self.heads * self.vdim
        a1 = up8(b + self.heads)
        return {"q": 0, "k": k, "v": 2 * k, "b": b, "a1": a1, "g1": a1 + self.rank, "end": a1 + 2 * self.rank}


@dataclass
class LoopSpec:
    """Layers start .. stop - 1 run ``times`` times in a row with the same weights; each pass begins with a projection of
    [stream, embedding output] and has caches and states of its own."""
    start: int
    stop: int
    times: int
    kind: str = "loop"

    def expand(self, layers: list) -> list:
        """One entry per layer run."""
        return layers[:self.start] + layers[self.start:self.stop] * self.times + layers[self.stop:]


@dataclass
class DenseSpec:
    ff: int
    act: str = "silu"                  # xielu: un-gated, with two learned numbers per layer
    bias: bool = False                 # of all projections
    kind: str = "dense"

    def gated(self) -> bool:
        return self.act != "xielu"


@dataclass
class MoeSpec:
    experts: int
    top: int
    ff: int
    act: str = "silu"
    router: str = "softmax"            # softmax | biased_softmax (a bias on the logits) | sigmoid | softmax_bias (selection
                                       # by softmax score + correction)
    correction: bool = False
    renorm: object = True              # chosen weights divided by their sum (held away from zero); "sum": by the plain sum
    scale: float = 1.0                 # ... and multiplied by this
    n_group: int = 1                   # groups of neighbouring experts, the best keep_group of them stay open
    keep_group: int = 1
    group_top: int = 2                 # a group's score sums this many of its best selection scores
    shared_ff: int = 0                 # width of the shared expert (0: none)
    shared_gate: bool = False          # its output times the sigmoid of one more row of the router projection
    kind: str = "moe"

    def gated(self) -> bool:
        return self.act != "relu2"

    def shared_slots(self) -> int:
        """Un-gated experts add up over parts of their width, so the shared expert is stored as this many more experts of
        width ``ff`` (the last one padded with zeros) behind the routed ones."""
        return -(-self.shared_ff // self.ff)


@dataclass
class LayerSpec:
    mixer: object
    mlp: object = None                 # None: the layer has no feed-forward part


_SPECS = {c.__dataclass_fields__["kind"].default: c
          for c in (AttnSpec, LightningSpec, SsdSpec, ParallelSpec, RotarySpec, LatentSpec, RgLruSpec, ChannelDeltaSpec, LoopSpec,
                    Hgrn2Spec, DenseSpec, MoeSpec)}


def spec_from(d):
    """A specification (or its ``dataclasses.asdict`` form) as the dataclass its ``kind`` names."""
    if not isinstance(d, dict):
        return d
    d = {k: spec_from(v) for k, v in d.items()}
    if "mixer" in d:
        return LayerSpec(**d)
    return _SPECS[d["kind"]](**d)


@dataclass
class ModelConfig:
    arch: str = "qwen3moe"             # registry key (see models.registry)
    n_layer: int = 4
    hidden: int = 256
    vocab: int = 4096
    rms_eps: float = 1e-6
    norm_offset: float = 0.0           # 1.0 for checkpoints that store (weight - 1)
    tie_embeddings: bool = False
    max_position: int = 131072
    # attention
    n_head: int = 4
    n_kv_head: int = 2
    head_dim: int = 64
    rope_theta: float = 1e6
    rope_dim: Optional[int] = None     # rotary dims per head (None = head_dim); multiple of 64
    rope_scaling: Optional[dict] = None
    mrope_sections: Optional[tuple] = None     # multi-section rotary embedding: frequencies per (temporal, row, column) axis
    mrope_interleaved: bool = True             # axes alternate over the frequencies (Qwen3-VL) or take consecutive sections
    qk_norm: bool = True
    gated_attn: bool = False           # q projection emits [q | gate] per head, out *= sigmoid(gate)
    sliding_window: int = 0            # window of "swa" layers
    attn_softcap: float = 0.0
    logit_softcap: float = 0.0
    logit_scale: float = 1.0           # multiplies the logits before the soft cap (muse-glimmer)
    attn_scale: Optional[float] = None
    # layer pattern: one of "attn", "swa", "nope" (attention without RoPE), "gdn", "mla", "mamba2", "kda" per layer
    layer_kinds: Optional[List[str]] = None
    full_attention_interval: int = 0   # >0: layer il is "gdn" unless (il + 1) % interval == 0
    # gated delta net
    gdn_k_heads: int = 4
    gdn_v_heads: int = 4
    gdn_k_dim: int = 64
    gdn_v_dim: int = 64
    gdn_conv: int = 4
    gdn_tiled_heads: bool = False      # value head h reads key head h % n_k (GGUF order) instead of h // (n_v/n_k)
    gdn_gate_act: str = "silu"         # activation of z in the gated output norm
    # Kimi delta attention ("kda" layers): per-channel decay, q / k / v each behind a short causal convolution
    kda_heads: int = 4
    kda_head_dim: int = 64
    kda_conv: int = 4
    kda_rank: int = 32                 # width of the low-rank gate projections (f_a / f_b, g_a / g_b)
    kda_lower: float = -5.0            # lower bound of the log decay: g = lower * sigmoid(-(f(x) + dt_bias) * A)
    # hyper-connections: the residual is ``hyper_streams`` parallel streams mixed before and after every sublayer
    hyper_streams: int = 1
    hyper_mode: str = "sinkhorn"       # "static": per-layer weights that do not depend on the token (stacks with
                                       # ``layers``). "sinkhorn": per-token pre / post weights and a Sinkhorn-normalised stream mix
                                       # (glm5-next, deepseek41); "gated": a low-rank sigmoid gate per channel mixes
                                       # the normed streams, the block output re-enters every stream with a weight
                                       # of its own, the last mixer is the output norm (qwen4exp)
    hc_rank: int = 16                  # "gated": width of the low-rank gate
    hc_iters: int = 20                 # Sinkhorn rounds of the stream-to-stream mix
    hc_eps: float = 1e-6
    # mamba2 (nemotron-h)
    ssm_state: int = 128
    ssm_heads: int = 8
    ssm_head_dim: int = 64
    ssm_groups: int = 1
    ssm_conv: int = 4
    # MLA
    q_lora: int = 0
    kv_lora: int = 0
    qk_nope_dim: int = 0
    qk_rope_dim: int = 0
    v_head_dim: int = 0
    # feed-forward
    ffn_act: str = "silu"              # silu | gelu_tanh | relu2
    dense_ff: int = 0                  # FFN width of dense layers
    first_dense_layers: int = 0        # leading layers that use the dense FFN in a MoE model
    n_expert: int = 0
    top_k: int = 0
    expert_ff: int = 0
    moe_latent: int = 0                # > 0: the routed experts run at this width, between a down and an up projection
    shared_ff: int = 0                 # width of the shared expert (0 = none)
    shared_gate: bool = False          # sigmoid(x . w) gate on the shared expert
    router_mode: str = "softmax"       # softmax | sigmoid
    router_bias: bool = False          # selection bias (sigmoid routers)
    norm_topk: bool = True
    route_scale: float = 1.0
    n_group: int = 1
    topk_group: int = 1
    # Gemma-4 layer form (``sandwich_norm``): every sublayer between a pre and a post RMS norm, embedding scaled by
    # sqrt(hidden), sliding-window and global layers with head sizes / kv-head counts / rotary bases of their own,
    # values RMS-normed without a weight, unscaled attention, optional: global layers that use their keys as values,
    # trailing layers that read an earlier layer's KV, a per-layer output scale, per-layer token embeddings, and in MoE
    # layers the dense FFN beside the routed experts (router on the normed residual scaled by 1 / sqrt(hidden))
    sandwich_norm: bool = False
    # one sub-layer per block (Nemotron-H as shipped): ``layer_kinds`` then also holds "ffn" and "moe" entries, and a
    # block is x + sublayer(norm(x)) with the mixer OR the feed-forward part, not both
    block_form: bool = False
    embed_scale: float = 1.0
    swa_head_dim: int = 0              # 0 = head_dim
    swa_kv_heads: int = 0              # 0 = n_kv_head
    rope_theta_swa: float = 0.0        # 0 = rope_theta
    rope_freq_factors: Optional[list] = None      # global layers: per-frequency divisors of the rotary frequencies
    v_norm: bool = False
    global_k_as_v: bool = False
    kv_shared_layers: int = 0
    layer_out_scale: bool = False
    ple_dim: int = 0                   # width of the per-layer token embeddings (0 = none)
    # stacks whose layers have sizes of their own: one LayerSpec per layer. The per-model attention / recurrent / MoE
    # fields above then only describe the largest layer (memory planning); every layer runs from its specification
    layers: Optional[List[LayerSpec]] = None
    # with ``layers`` and ``sandwich_norm``: one fp32 residual stream, every sublayer between two RMS norms that work in
    # ``norm_groups`` equal parts of the vector; what a sublayer reads first passes h + conv(h), a causal convolution per
    # channel of ``input_conv`` taps (0: none)
    norm_groups: int = 1
    input_conv: int = 0
    # with ``layers``, one stream and no sandwich norms: pre-norm layers on one fp32 residual, x + residual_mult * f(norm(x))
    residual_mult: float = 1.0
    embed_norm: bool = False           # the embedding rows pass the model's norm first
    loop: Optional[LoopSpec] = None    # ``layers`` then has one entry per layer run (``LoopSpec.expand``)
    # with ``layers`` and one stream: both sublayers of a layer read one norm of the residual, x + mixer(h) + ffn(h)
    parallel_sublayers: bool = False
    residual_gate: bool = False        # ... each result times the sigmoid of a projection (with bias) of h, column by column
    depth_average: bool = False        # ... and the next layer reads a learned sum of the embedding and all results so far
    # multi-token prediction
    mtp_layers: int = 0
    # weights
    dtype: str = "bf16"                # compute dtype on GPU: bf16; CPU engine uses fp32
    quant: str = "none"                # none | nvfp4 | fp8_block

    def __post_init__(self):
        if self.layers is not None:
            self.layers, self.loop = [spec_from(x) for x in self.layers], spec_from(self.loop)
            self.n_layer = len(self.layers)
            self.layer_kinds = [x.mixer.kind for x in self.layers]
            if not self.parallel_sublayers and (self.residual_gate or self.depth_average
                                                or any(getattr(x.mlp, "bias", False) for x in self.layers)):
                raise ValueError("residual gates, depth averages and feed-forward biases come with parallel sublayers")
            attn = [a for a in (self.attn_spec(il) for il in range(self.n_layer)) if a is not None]
            lat = [x.mixer for x in self.layers if isinstance(x.mixer, LatentSpec)]
            if lat:
                big = max(lat, key=lambda a: a.kv_rank + a.rot_dim)
                self.n_head, self.n_kv_head, self.head_dim = big.heads, 1, big.kv_rank + big.rot_dim
            if attn:
                big = max(attn, key=lambda a: a.kv_heads * (a.dim + a.vdim))
                self.n_head, self.n_kv_head, self.head_dim = big.heads, big.kv_heads, big.dim
            moe = [x.mlp for x in self.layers if isinstance(x.mlp, MoeSpec)]
            self.n_expert = max([m.experts for m in moe], default=0)
            self.top_k = max([m.top for m in moe], default=0)
            self.expert_ff = max([m.ff for m in moe], default=0)
            self.rope_dim = 0
        if self.rope_dim is None:
            self.rope_dim = self.head_dim if not self.qk_rope_dim else self.qk_rope_dim
        if self.layer_kinds is None:
            if self.full_attention_interval > 0:
                self.layer_kinds = ["attn" if (il + 1) % self.full_attention_interval == 0 else "gdn"
                                    for il in range(self.n_layer)]
            elif self.kv_lora > 0:
                self.layer_kinds = ["mla"] * self.n_layer
            else:
                self.layer_kinds = ["attn"] * self.n_layer
        assert len(self.layer_kinds) == self.n_layer

    # ---- derived
    def attn_spec(self, il: int) -> Optional[AttnSpec]:
        """The softmax-attention part of layer il of a stack with specifications."""
        m = self.layers[il].mixer
        return m if isinstance(m, AttnSpec) else (m.left if isinstance(m, ParallelSpec) else None)

    def latent_spec(self, il: int) -> Optional[LatentSpec]:
        """The mixer of layer il of a stack with specifications, when it is latent attention."""
        m = self.layers[il].mixer
        return m if isinstance(m, LatentSpec) else None

    def recurrent_spec(self, il: int):
        """The part of layer il that carries a recurrent state, of a stack with specifications."""
        m = self.layers[il].mixer
        if isinstance(m, (LightningSpec, SsdSpec, RgLruSpec, ChannelDeltaSpec, Hgrn2Spec)):
            return m
        return m.right if isinstance(m, ParallelSpec) else None

    def mix_columns(self, il: int) -> dict:
        """First column of each part of the stacked input projection ``mix.in``, and its width (``end``): q | k | v | head
        gates of the attention part, the columns of the recurrent part, the residual gates of both sublayers. Parts behind
        q | k | v of an attention part start on 16-byte boundaries, except the state-space columns (``ssd``)."""
        up8 = lambda n: -(-n // 8) * 8                               # noqa: E731
        a, r, col, n = self.attn_spec(il), self.recurrent_spec(il), {}, 0
        if a is not None:
            for part, w in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                col[part], n = n, n + w
            if a.gate == "head":
                col["g"] = up8(n)
                n = col["g"] + a.heads
        if r is not None and r.kind == "ssd":
            col["ssd"] = n
            n += 2 * r.heads * r.vdim + 2 * r.groups * r.state + r.heads
        elif r is not None and r.kind == "hgrn2":
            for part, w in (("rq", r.heads * r.dim), ("rf", r.heads * r.dim), ("rv", r.heads * r.vdim)):
                col[part] = up8(n)
                n = col[part] + w
        for part in ("rg1", "rg2")[:0 if not self.residual_gate else 1 if self.layers[il].mlp is None else 2]:
            col[part] = up8(n)
            n = col[part] + self.hidden
        col["end"] = up8(n) if "rq" in col or "rg1" in col or "g" in col else n
        return col

    def attn_history(self, il: int):
        """(tokens, channels) of the projected q, k and v that the short convolution of an attention layer keeps, or None."""
        a = self.attn_spec(il)
        if a is None or a.conv < 2:
            return None
        return a.conv - 1, (a.heads + a.kv_heads) * a.dim + a.kv_heads * a.vdim

    def state_floats(self, il: int) -> int:
        """float32 numbers of recurrent state (without convolution histories) per sequence of layer il."""
        r = self.recurrent_spec(il)
        if r is None:
            return 0
        return r.width if r.kind == "rglru" else r.heads * r.vdim * (r.state if r.kind == "ssd" else r.dim)

    def merged_output(self, il: int) -> bool:
        """Whether the mixer's parts share one output projection ``mix.o`` over their concatenated columns."""
        r = self.recurrent_spec(il)
        return r is not None and r.kind == "hgrn2"

    # layer runs of a looped stack: caches and states belong to a run, weights to a layer
    def weight_layer(self, il: int) -> int:
        """Index of the weights of layer run il."""
        lo = self.loop
        if lo is None or il < lo.start:
            return il
        n = lo.stop - lo.start
        return lo.start + (il - lo.start) % n if il < lo.start + n * lo.times else il - n * (lo.times - 1)

    def begins_pass(self, il: int) -> bool:
        lo = self.loop
        n = 0 if lo is None else lo.stop - lo.start
        return n > 0 and lo.start <= il < lo.start + n * lo.times and (il - lo.start) % n == 0

    def stream_rows(self) -> int:
        """float32 rows of the residual's width that a step keeps per token until its end: with depth averages the embedding
        output, every layer's result and the sums made ahead."""
        return self.n_layer + 1 + 3 if self.depth_average else 0

    def conv_inputs(self, il: int) -> List[str]:
        """Sublayers of layer il whose input passes a short convolution (``input_conv``)."""
        if self.layers is None or self.input_conv < 1:
            return []
        return ["attn"] if self.layers[il].mlp is None else ["attn", "ffn"]

    def is_moe_layer(self, il: int) -> bool:
        if self.layers is not None:
            return isinstance(self.layers[il].mlp, MoeSpec)
        if self.block_form:
            return il < len(self.layer_kinds) and self.layer_kinds[il] == "moe"
        return self.n_expert > 0 and il >= self.first_dense_layers

    def kv_layers(self) -> List[int]:
        if self.layers is not None:
            return [i for i in range(self.n_layer) if self.attn_spec(i) is not None or self.latent_spec(i) is not None]
        return [i for i, k in enumerate(self.layer_kinds) if k in ("attn", "swa", "nope", "mla")]

    def recurrent_layers(self) -> List[int]:
        """Layers that carry a state from token to token besides the KV cache."""
        if self.layers is not None:
            return [i for i in range(self.n_layer) if self.recurrent_spec(i) is not None or self.conv_inputs(i)
                    or self.attn_history(i) is not None]
        return [i for i, k in enumerate(self.layer_kinds) if k in ("gdn", "mamba2", "kda")]

    def kv_dims(self, il: int):
        """(n_kv_heads, k_dim, v_dim) stored per token for layer il."""
        if self.layers is not None:
            a, m = self.attn_spec(il), self.latent_spec(il)
            if m is not None:                           # one row per token, keys and values alike
                return 1, -(-(m.kv_rank + m.rot_dim) // 8) * 8, 0
            return a.kv_heads, a.dim, a.vdim
        if self.layer_kinds[il] == "mla":
            return 1, self.kv_lora + self.qk_rope_dim, 0
        d, n_kv = self.attn_dims(il)
        return n_kv, d, d

    def attn_dims(self, il: int):
        """(head size, kv heads) of attention layer il: sliding-window layers may have their own."""
        if self.layer_kinds[il] == "swa":
            return self.swa_head_dim or self.head_dim, self.swa_kv_heads or self.n_kv_head
        return self.head_dim, self.n_kv_head

    def owns_kv(self, il: int) -> bool:
        """False for the trailing layers that read another layer's KV cache (``kv_shared_layers``)."""
        return il < self.n_layer - self.kv_shared_layers

    def kv_source(self, il: int) -> int:
        """The layer whose KV cache layer il reads: itself, or the last layer of its kind before the shared ones."""
        if self.owns_kv(il):
            return il
        for j in range(self.n_layer - self.kv_shared_layers - 1, -1, -1):
            if self.layer_kinds[j] == self.layer_kinds[il]:
                return j
        raise ValueError(f"layer {il} shares a KV cache but no earlier layer of its kind owns one")

    def has_v_proj(self, il: int) -> bool:
        return not (self.global_k_as_v and self.layer_kinds[il] != "swa")

    def gdn_conv_channels(self) -> int:
        return 2 * self.gdn_k_heads * self.gdn_k_dim + self.gdn_v_heads * self.gdn_v_dim

    def to_json(self) -> str:
        return json.dumps(dataclasses.asdict(self))

    @classmethod
    def from_dict(cls, d: dict) -> "ModelConfig":
        names = {f.name for f in dataclasses.fields(cls)}
        return cls(**{k: v for k, v in d.items() if k in names})

    def param_count(self) -> int:
        from .models.weights import weight_shapes
        n = 0
        for shp in weight_shapes(self).values():
            m = 1
            for s in shp:
                m *= s
            n += m
        return n


# --------------------------------------------------------------------------------------------------
# presets
# --------------------------------------------------------------------------------------------------
def tiny_glm_next() -> "ModelConfig":
    """Shape of the glm5-next family in miniature: Kimi-delta-attention layers with a latent-attention layer every
    third, hyper-connections (4 streams) around every sublayer, sigmoid-routed MoE with a shared expert after one
    dense layer. The latent-attention layers attend densely (no sparse key selection)."""
    return ModelConfig(arch="glm5_next", n_layer=3, hidden=128, vocab=512, n_head=4, n_kv_head=4, head_dim=96,
                       layer_kinds=["kda", "kda", "mla"], kda_heads=4, kda_head_dim=32, kda_rank=16,
                       q_lora=48, kv_lora=64, qk_nope_dim=32, qk_rope_dim=64, v_head_dim=32, qk_norm=False,
                       hyper_streams=4, hc_iters=8, dense_ff=192, first_dense_layers=1, n_expert=8, top_k=2,
                       expert_ff=64, shared_ff=64, router_mode="sigmoid", router_bias=True, route_scale=2.0)


def tiny_qwen4exp() -> "ModelConfig":
    """Shape of the qwen4exp family in miniature: the hybrid Gated-DeltaNet / gated-attention MoE stack with a
    sigmoid DeltaNet output gate, multi-section rotary positions and gated hyper-connections (4 streams) in place of
    the residual stream and the pre-norms. Attention is dense (its sparse key selection equals dense attention up to
    the selection budget); the n-gram embedding layer is not modelled."""
    c = tiny_hybrid_moe()
    c.arch = "qwen4exp"
    c.hyper_streams, c.hyper_mode, c.hc_rank = 4, "gated", 8
    c.gdn_gate_act = "sigmoid"
    if c.rope_dim == 64:
        c.mrope_sections = (11, 11, 10)
    return c


def tiny_hybrid_moe() -> ModelConfig:
    """4-layer hybrid: 3 Gated DeltaNet layers + 1 gated GQA layer, 8 experts top-2 + shared expert."""
    return ModelConfig(arch="qwen35moe", n_layer=4, hidden=256, vocab=4096, n_head=4, n_kv_head=2, head_dim=64,
                       rope_theta=1e6, full_attention_interval=4, gated_attn=True, gdn_k_heads=4, gdn_v_heads=4,
                       gdn_k_dim=64, gdn_v_dim=64, gdn_conv=4, n_expert=8, top_k=2, expert_ff=512, shared_ff=512,
                       shared_gate=True)


def tiny_gqa_moe() -> ModelConfig:
    return ModelConfig(arch="qwen3moe", n_layer=2, hidden=256, vocab=1024, n_head=4, n_kv_head=2, head_dim=64,
                       n_expert=8, top_k=2, expert_ff=128)


def tiny_dense() -> ModelConfig:
    return ModelConfig(arch="qwen3", n_layer=2, hidden=256, vocab=1024, n_head=4, n_kv_head=2, head_dim=64,
                       dense_ff=512)


def tiny_mla_moe() -> ModelConfig:
    return ModelConfig(arch="deepseek_v3", n_layer=3, hidden=256, vocab=1024, n_head=4, n_kv_head=4, head_dim=96,
                       q_lora=96, kv_lora=64, qk_nope_dim=32, qk_rope_dim=64, v_head_dim=32, qk_norm=False,
                       dense_ff=384, first_dense_layers=1, n_expert=8, top_k=2, expert_ff=128, shared_ff=128,
                       router_mode="sigmoid", router_bias=True, n_group=4, topk_group=2, route_scale=2.5,
                       mtp_layers=1)


def qwen3_30b_a3b() -> ModelConfig:
    """30B-A3B-shape MoE: 48 layers, 128 experts top-8, no shared expert."""
    return ModelConfig(arch="qwen3moe", n_layer=48, hidden=2048, vocab=151936, n_head=32, n_kv_head=4, head_dim=128,
                       rope_theta=1e6, n_expert=128, top_k=8, expert_ff=768)


def qwen35_80b_a3b() -> ModelConfig:
    """80B-A3B-shape hybrid MoE: 3:1 Gated DeltaNet to gated attention, 512 experts top-10 + shared."""
    return ModelConfig(arch="qwen35moe", n_layer=48, hidden=2048, vocab=151936, n_head=16, n_kv_head=2, head_dim=256,
                       rope_dim=64, rope_theta=1e7, full_attention_interval=4, gated_attn=True, gdn_k_heads=16,
                       gdn_v_heads=32, gdn_k_dim=128, gdn_v_dim=128, gdn_conv=4, n_expert=512, top_k=10,
                       expert_ff=512, shared_ff=512, shared_gate=True, norm_offset=0.0, quant="nvfp4")


def deepseek_671b() -> ModelConfig:
    """671B-shape MLA MoE: 61 layers, 256 routed experts top-8 (8 groups, top-4), 1 shared expert, 1 MTP head."""
    return ModelConfig(arch="deepseek_v3", n_layer=61, hidden=7168, vocab=129280, n_head=128, n_kv_head=128,
                       head_dim=192, q_lora=1536, kv_lora=512, qk_nope_dim=128, qk_rope_dim=64, v_head_dim=128,
                       qk_norm=False, rope_theta=1e4, dense_ff=18432, first_dense_layers=3, n_expert=256, top_k=8,
                       expert_ff=2048, shared_ff=2048, router_mode="sigmoid", router_bias=True, n_group=8,
                       topk_group=4, route_scale=2.5, mtp_layers=1, quant="fp8_block")


def dense_27b() -> ModelConfig:
    return ModelConfig(arch="qwen3", n_layer=64, hidden=5120, vocab=151936, n_head=40, n_kv_head=8, head_dim=128,
                       rope_theta=1e6, dense_ff=17408)


def tiny_muse() -> ModelConfig:
    """muse-glimmer shape: dense, sliding-window RoPE layers with every third layer global without RoPE, QK norm,
    sigmoid output gate, logit scale + soft cap (``src/model/muse.rs:1-25`` in the reference)."""
    return ModelConfig(arch="muse-glimmer", n_layer=6, hidden=256, vocab=4096, n_head=4, n_kv_head=2, head_dim=64,
                       layer_kinds=["swa", "swa", "nope", "swa", "swa", "nope"], sliding_window=32, gated_attn=True,
                       dense_ff=512, logit_scale=0.5, logit_softcap=30.0)


def tiny_gemma() -> ModelConfig:
    """Gemma-style: alternating sliding-window / global attention, GELU-gated FFN, (weight - 1) norm storage,
    tied embeddings, logit soft cap 30 (``src/model/gemma4.rs:1-30``; per-layer head sizes and shared-KV layers of
    Gemma 4 are not modelled)."""
    return ModelConfig(arch="gemma4", n_layer=4, hidden=256, vocab=4096, n_head=4, n_kv_head=2, head_dim=64,
                       layer_kinds=["swa", "attn", "swa", "attn"], sliding_window=48, ffn_act="gelu_tanh",
                       dense_ff=512, norm_offset=1.0, tie_embeddings=True, logit_softcap=30.0)


def tiny_nemotron_h() -> ModelConfig:
    """Nemotron-H style hybrid: Mamba-2 layers with a few attention layers without RoPE, squared-ReLU FFN
    (``src/model/nemotron_h.rs:1-20``; latent MoE and per-layer expert counts are not modelled)."""
    return ModelConfig(arch="nemotron_h", n_layer=4, hidden=256, vocab=4096, n_head=4, n_kv_head=2, head_dim=64,
                       layer_kinds=["mamba2", "mamba2", "nope", "mamba2"], qk_norm=False, ffn_act="relu2",
                       dense_ff=512, ssm_state=32, ssm_heads=8, ssm_head_dim=32, ssm_groups=1, ssm_conv=4)


def tiny_nemotron_h_moe() -> ModelConfig:
    """The Nemotron-H hybrid with its latent MoE (``src/model/nemotron_h.rs:538-608``): the router reads the normed
    input, the routed squared-ReLU experts run at ``moe_latent`` between ``lat_down`` and ``lat_up``, the shared
    expert at full width."""
    c = tiny_nemotron_h()
    c.dense_ff, c.first_dense_layers = 512, 1
    c.n_expert, c.top_k, c.expert_ff, c.shared_ff, c.moe_latent = 8, 2, 128, 128, 128
    c.router_mode, c.router_bias, c.norm_topk, c.route_scale = "sigmoid", True, True, 2.5
    return c


def tiny_nemotron_h_blocks() -> ModelConfig:
    """Nemotron-H the way its checkpoints lay it out: one sub-layer per block (``block_form``), here Mamba-2 with two
    norm groups, a dense squared-ReLU FFN, attention without rotary embedding, and the latent MoE."""
    c = tiny_nemotron_h_moe()
    c.block_form, c.first_dense_layers, c.ssm_groups = True, 0, 2
    c.layer_kinds = ["mamba2", "ffn", "nope", "moe", "mamba2", "moe"]
    c.n_layer = len(c.layer_kinds)
    return c


def tiny_gemma4() -> ModelConfig:
    """Gemma 4 in miniature (``src/model/gemma4.rs:1-30``): sandwich norms, scaled embedding, sliding-window layers
    with 64-wide heads and 2 kv heads next to global layers with 128-wide heads, 1 kv head, keys used as values and
    rotary frequency factors, value norm, unscaled attention, the last two layers reading earlier layers' KV, a
    per-layer output scale, per-layer token embeddings, and MoE layers whose dense GELU FFN runs beside 8 routed GELU
    experts."""
    return ModelConfig(arch="gemma4", n_layer=6, hidden=256, vocab=4096, n_head=4, n_kv_head=1, head_dim=128,
                       layer_kinds=["swa", "swa", "attn", "swa", "swa", "attn"], sliding_window=48, rope_dim=128,
                       rope_theta=1e6, rope_freq_factors=[1.0] * 48 + [8.0] * 16, swa_head_dim=64, swa_kv_heads=2,
                       rope_theta_swa=1e4, ffn_act="gelu_tanh", dense_ff=384, norm_offset=0.0, tie_embeddings=True,
                       logit_softcap=30.0, attn_scale=1.0, sandwich_norm=True, embed_scale=16.0, v_norm=True,
                       global_k_as_v=True, kv_shared_layers=2, layer_out_scale=True, ple_dim=32, first_dense_layers=1,
                       n_expert=8, top_k=2, expert_ff=128, router_mode="softmax", norm_topk=True)


def tiny_nisasun() -> ModelConfig:
    """Nisasun in miniature: linear-attention layers with a constant decay per head beside layers that run windowed
    attention and a Mamba-2 mixer in parallel, static hyper-connections (3 streams), dense GELU and routed feed-forward
    parts, one layer without any. Sizes differ from layer to layer."""
    moe = dict(router="softmax_bias", correction=True, renorm=False, group_top=1)
    return ModelConfig(
        arch="nisasun", hidden=160, vocab=640, rms_eps=1e-5, norm_offset=1.0, hyper_streams=3, hyper_mode="static",
        layers=[LayerSpec(LightningSpec(3, 48, 64, [0.7, 0.95, 0.995]), DenseSpec(192, "gelu_tanh")),
                LayerSpec(ParallelSpec(AttnSpec(6, 3, 40, 72, 0.17, window=40), SsdSpec(6, 24, 16, 2, 3, 3), 0.6, 0.9),
                          MoeSpec(10, 3, 56, n_group=5, keep_group=3, **moe)),
                LayerSpec(ParallelSpec(AttnSpec(4, 1, 64, 32, 0.11, window=75), SsdSpec(2, 48, 40, 1, 5, 2), 1.1, 0.4)),
                LayerSpec(LightningSpec(5, 32, 24, [0.4, 0.8, 0.9, 0.98, 0.999]), MoeSpec(8, 2, 40, n_group=2,
                                                                                          keep_group=1, **moe))])


def _nisasun(n_layer: int, hidden: int, heads: int, ssm_heads: int, ff: int, expert_ff: int, attn_dims) -> ModelConfig:
    """Alternating parallel layers (attention of ``heads`` query heads with window 1024 beside Mamba-2 heads of 64 with
    state 128) and linear-attention layers (``heads`` heads of 128 x 128), four streams, dense and 32-expert
    feed-forward parts in turn."""
    decay = [1.0 - 2.0 ** -(2 + 8.0 * h / heads) for h in range(heads)]
    moe = MoeSpec(32, 4, expert_ff, router="softmax_bias", correction=True, renorm=False, n_group=8, keep_group=4,
                  group_top=1)
    dk, dv = attn_dims
    layers = []
    for il in range(n_layer):
        mixer = (ParallelSpec(AttnSpec(heads, heads // 4, dk, dv, dk ** -0.5, window=1024),
                              SsdSpec(ssm_heads, 64, 128, 8, 4, 8), 0.5, 0.5)
                 if il % 2 == 0 else LightningSpec(heads, 128, 128, decay))
        layers.append(LayerSpec(mixer, moe if il % 2 else DenseSpec(ff, "gelu_tanh")))
    return ModelConfig(arch="nisasun", hidden=hidden, vocab=65536, rms_eps=1e-5, norm_offset=1.0, hyper_streams=4,
                       hyper_mode="static", layers=layers)


def nisasun_4b() -> ModelConfig:
    """Nisasun with layers the size of a small production model (random weights; speed measurements)."""
    return _nisasun(24, 2048, 16, 64, 6144, 1024, (128, 128))


def nisasun_13b() -> ModelConfig:
    """The same at 4096 columns, with query / key heads of 96 and value heads of 192."""
    return _nisasun(20, 4096, 32, 128, 12288, 2048, (96, 192))


def _hybrid(n_layer: int, hidden: int, heads: int, ff: int, expert_ff: int) -> ModelConfig:
    """A Gated DeltaNet / gated attention hybrid of the size of a ``_nisasun`` stack: what that design is compared with."""
    return ModelConfig(arch="qwen35moe", n_layer=n_layer, hidden=hidden, vocab=65536, n_head=heads, n_kv_head=heads // 4,
                       head_dim=128, rope_dim=64, full_attention_interval=2, gated_attn=True, gdn_k_heads=heads,
                       gdn_v_heads=2 * heads, gdn_k_dim=128, gdn_v_dim=128, first_dense_layers=n_layer // 2, dense_ff=ff,
                       n_expert=32, top_k=4, expert_ff=expert_ff)


def hybrid_4b() -> ModelConfig:
    return _hybrid(24, 2048, 16, 6144, 1024)


def hybrid_13b() -> ModelConfig:
    return _hybrid(20, 4096, 32, 12288, 2048)


def tiny_pemezen() -> "ModelConfig":
    """Pemezen in miniature: latent-attention layers (rotated key parts with YaRN frequencies, output gates per column or
    per head) and a gated linear recurrent unit, every sublayer between grouped norms behind a short input convolution,
    xIELU feed-forward parts, one layer without any. Sizes differ from layer to layer."""
    return ModelConfig(
        arch="pemezen", hidden=144, vocab=512, rms_eps=1e-5, sandwich_norm=True, norm_groups=3, input_conv=3,
        embed_scale=2.5, logit_softcap=12.0,
        layers=[LayerSpec(LatentSpec(6, 40, 24, 32, 72, 0.15, RotarySpec(24, 1e4, 2.0, 256), "head"), DenseSpec(200, "xielu")),
                LayerSpec(RgLruSpec(120, 3, 5), DenseSpec(88, "xielu")),
                LayerSpec(LatentSpec(2, 64, 16, 48, 96, 0.11, RotarySpec(16, 5e4, 4.0, 128)), None),
                LayerSpec(RgLruSpec(64, 1, 3), DenseSpec(136, "xielu"))])


def _pemezen(n_layer: int, hidden: int, heads: int, ff: int, rank: int, rot: int) -> ModelConfig:
    """Two recurrent layers, then a latent-attention layer, in turn; gates per column and per head in turn."""
    layers = []
    for il in range(n_layer):
        mixer = (LatentSpec(heads, 128, rot, 128, rank, (128 + rot) ** -0.5, RotarySpec(rot, 1e6, 8.0, 8192),
                            "channel" if il % 2 else "head")
                 if il % 3 == 2 else RgLruSpec(hidden * 5 // 4, hidden // 256 * 5 // 4, 4))
        layers.append(LayerSpec(mixer, DenseSpec(ff, "xielu")))
    return ModelConfig(arch="pemezen", hidden=hidden, vocab=65536, rms_eps=1e-5, sandwich_norm=True, norm_groups=4,
                       input_conv=4, embed_scale=2.0, logit_softcap=20.0, layers=layers)


def pemezen_1b() -> ModelConfig:
    """Pemezen with layers the size of a small production model (random weights; speed measurements)."""
    return _pemezen(24, 2048, 16, 8192, 512, 64)


def pemezen_7b() -> ModelConfig:
    return _pemezen(30, 4096, 32, 16384, 512, 64)


def mla_1b() -> ModelConfig:
    """A dense latent-attention model of the size of ``pemezen_1b``: what its attention layers are compared with."""
    return ModelConfig(arch="deepseek_v3", n_layer=24, hidden=2048, vocab=65536, n_head=16, n_kv_head=16, head_dim=192,
                       kv_lora=512, qk_nope_dim=128, qk_rope_dim=64, v_head_dim=128, qk_norm=False, dense_ff=5632)


def mla_7b() -> ModelConfig:
    return ModelConfig(arch="deepseek_v3", n_layer=30, hidden=4096, vocab=65536, n_head=32, n_kv_head=32, head_dim=192,
                       kv_lora=512, qk_nope_dim=128, qk_rope_dim=64, v_head_dim=128, qk_norm=False, dense_ff=11264)


def tiny_gurozen() -> "ModelConfig":
    """Gurozen in miniature: gated delta rule layers with a decay per key channel beside soft-capped attention behind short
    convolutions, pre-norm sublayers on one scaled residual, squared-ReLU experts with a gated shared one, a dense layer,
    one layer without feed-forward part, and a loop of three layers that runs twice."""
    moe = dict(act="relu2", router="sigmoid", renorm="sum", shared_gate=True)
    rot = dict(scaling="llama3", layout="half")
    loop = LoopSpec(1, 4, 2)
    layers = [LayerSpec(ChannelDeltaSpec(4, 2, 40, 32, 4, 16), DenseSpec(200)),
              LayerSpec(AttnSpec(6, 2, 32, 48, 0.15, norm_over="all", bias=True, conv=3, rot=RotarySpec(24, 1e4, 4.0, 128, **rot),
                                 softcap=20.0), MoeSpec(10, 3, 56, scale=1.5, n_group=5, keep_group=2, shared_ff=112, **moe)),
              LayerSpec(ChannelDeltaSpec(3, 3, 24, 56, 2, 8), None),
              LayerSpec(AttnSpec(4, 1, 64, 32, 0.11, norm_over="all", bias=True, conv=4, rot=RotarySpec(64, 5e4, 8.0, 64, **rot),
                                 softcap=15.0), DenseSpec(96)),
              LayerSpec(ChannelDeltaSpec(2, 1, 64, 64, 3, 24), MoeSpec(8, 2, 40, scale=2.0, n_group=2, keep_group=1, shared_ff=72,
                                                                        **moe))]
    return ModelConfig(arch="gurozen", hidden=144, vocab=512, rms_eps=1e-5, norm_offset=1.0, tie_embeddings=True, embed_norm=True,
                       residual_mult=0.7, logit_scale=1.5, layers=loop.expand(layers), loop=loop)


def _gurozen(n_layer: int, hidden: int, heads: int, ff: int, expert_ff: int) -> ModelConfig:
    """``n_layer`` runs of alternating delta-rule and attention layers, four of them a second pass over the same weights;
    the first half dense, then 32 squared-ReLU experts and a shared one."""
    rot = RotarySpec(64, 1e6, 8.0, 8192, scaling="llama3", layout="half")
    moe = MoeSpec(32, 4, expert_ff, "relu2", router="sigmoid", renorm="sum", scale=2.0, n_group=8, keep_group=4,
                  shared_ff=expert_ff, shared_gate=True)
    layers = []
    for il in range(n_layer - 4):
        mixer = (AttnSpec(heads, heads // 4, 128, 128, 128 ** -0.5, norm_over="all", bias=True, conv=4, rot=rot, softcap=30.0)
                 if il % 2 else ChannelDeltaSpec(2 * heads, heads, 128, 128, 4, 128))
        layers.append(LayerSpec(mixer, moe if il >= (n_layer - 4) // 2 else DenseSpec(ff)))
    loop = LoopSpec(n_layer // 2 - 4, n_layer // 2, 2)
    return ModelConfig(arch="gurozen", hidden=hidden, vocab=65536, rms_eps=1e-5, norm_offset=1.0, tie_embeddings=True,
                       embed_norm=True, residual_mult=0.5, logit_scale=1.0, layers=loop.expand(layers), loop=loop)


def gurozen_4b() -> ModelConfig:
    """Gurozen with layers the size of a small production model (random weights; speed measurements)."""
    return _gurozen(24, 2048, 16, 6144, 1536)


def gurozen_13b() -> ModelConfig:
    return _gurozen(20, 4096, 32, 12288, 3072)


def tiny_mananex() -> "ModelConfig":
    """Mananex in miniature: windowed attention with a sink, kept first tokens and head gates beside an HGRN2 state in every
    layer, both sublayers on one norm, gated residuals, depth averages, dense parts with biases, softmax-routed experts with a
    logit bias, one layer without feed-forward part. Sizes differ from layer to layer."""
    def mixer(heads, kv, dim, vdim, window, keep, rot, h, d, v, ls, rs):
        return ParallelSpec(AttnSpec(heads, kv, dim, vdim, dim ** -0.5, window=window, keep_first=keep, qk_norm=False,
                                     rot=RotarySpec(rot, 1e4), sink=True, gate="head"), Hgrn2Spec(h, d, v), ls, rs)
    return ModelConfig(
        arch="mananex", hidden=144, vocab=512, rms_eps=1e-5, norm_offset=1.0, tie_embeddings=True, parallel_sublayers=True,
        residual_gate=True, depth_average=True,
        layers=[LayerSpec(mixer(6, 2, 32, 48, 40, 3, 24, 3, 40, 56, 0.7, 0.8), DenseSpec(200, bias=True)),
                LayerSpec(mixer(4, 4, 48, 24, 75, 5, 48, 5, 24, 32, 1.1, 0.5), MoeSpec(10, 3, 56, router="biased_softmax")),
                LayerSpec(mixer(2, 1, 64, 64, 130, 1, 16, 2, 64, 40, 0.4, 1.2), None),
                LayerSpec(mixer(3, 1, 40, 32, 17, 2, 8, 1, 72, 80, 0.9, 0.6), MoeSpec(6, 2, 40, router="biased_softmax"))])


def _mananex(n_layer: int, hidden: int, heads: int, ff: int, expert_ff: int) -> ModelConfig:
    """Attention of ``heads`` query heads with window 1024 beside as many HGRN2 heads, dense and 32-expert feed-forward parts
    in turn."""
    layers = []
    for il in range(n_layer):
        mixer = ParallelSpec(AttnSpec(heads, heads // 4, 128, 128, 128 ** -0.5, window=1024, keep_first=4, qk_norm=False,
                                      rot=RotarySpec(64, 1e6), sink=True, gate="head"), Hgrn2Spec(heads, 128, 128), 0.5, 0.5)
        layers.append(LayerSpec(mixer, MoeSpec(32, 4, expert_ff, router="biased_softmax") if il % 2 else DenseSpec(ff, bias=True)))
    return ModelConfig(arch="mananex", hidden=hidden, vocab=65536, rms_eps=1e-5, norm_offset=1.0, tie_embeddings=True,
                       parallel_sublayers=True, residual_gate=True, depth_average=True, layers=layers)


def mananex_4b() -> ModelConfig:
    """Mananex with layers the size of a small production model (random weights; speed measurements)."""
    return _mananex(24, 2048, 16, 6144, 1024)


def mananex_13b() -> ModelConfig:
    return _mananex(20, 4096, 32, 12288, 2048)


PRESETS = {
    "tiny-mananex": tiny_mananex,
    "mananex-4b": mananex_4b,
    "mananex-13b": mananex_13b,
    "tiny-gurozen": tiny_gurozen,
    "gurozen-4b": gurozen_4b,
    "gurozen-13b": gurozen_13b,
    "tiny-pemezen": tiny_pemezen,
    "pemezen-1b": pemezen_1b,
    "pemezen-7b": pemezen_7b,
    "mla-1b": mla_1b,
    "mla-7b": mla_7b,
    "hybrid-4b": hybrid_4b,
    "hybrid-13b": hybrid_13b,
    "tiny-nisasun": tiny_nisasun,
    "nisasun-4b": nisasun_4b,
    "nisasun-13b": nisasun_13b,
    "tiny-muse": tiny_muse,
    "tiny-gemma4": tiny_gemma4,
    "tiny-nemotron-h-moe": tiny_nemotron_h_moe,
    "tiny-nemotron-h-blocks": tiny_nemotron_h_blocks,
    "tiny-gemma": tiny_gemma,
    "tiny-nemotron-h": tiny_nemotron_h,
    "tiny-hybrid-moe": tiny_hybrid_moe,
    "tiny-glm-next": tiny_glm_next,
    "tiny-qwen4exp": tiny_qwen4exp,
    "tiny-gqa-moe": tiny_gqa_moe,
    "tiny-dense": tiny_dense,
    "tiny-mla-moe": tiny_mla_moe,
    "qwen3-30b-a3b": qwen3_30b_a3b,
    "qwen35-80b-a3b": qwen35_80b_a3b,
    "deepseek-671b": deepseek_671b,
    "dense-27b": dense_27b,
}
