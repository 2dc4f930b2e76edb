"""Model descriptors: per-model shapes as data.

Plays the role of the reference's ``ModelDesc`` (src/model/model_desc.h:67-195):
every shape the loader, the memory planner and the kernels need is derived
from one frozen dataclass, and the table of fused linears (qkv, gate‖up, ...)
is generated from it rather than written per model.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field, asdict, replace
from typing import Optional


@dataclass(frozen=True)
class LinearDesc:
    """One fused linear: ``out[n] = sum_k x[k] w[n][k]``."""
    name: str
    n: int
    k: int
    parts: tuple          # checkpoint tensors fused along N, in order
    parallel: str         # "column" | "row" | "none": how tensor parallel slices it


@dataclass(frozen=True)
class LatentAttention:
    """Attention whose queries and keys / values go through low-rank latents; the cache holds the key-value latent and
    one rotated key part shared by the heads."""
    heads: int
    dim: int                      # unrotated query / key dimensions of a head
    rot_dim: int                  # rotated query / key dimensions of a head
    vdim: int                     # value dimensions of a head
    kv_rank: int
    q_rank: int
    scale: float
    rope_dims: int                # rotated leading dimensions of the rot_dim part
    rope_base: float
    window: int = 0               # a position sees itself and the window - 1 positions before it (0: all)

    def linear_elems(self, h: int) -> int:
        return (self.q_rank + self.kv_rank + self.rot_dim) * h + self.heads * (self.dim + self.rot_dim) * self.q_rank \
            + self.heads * (self.dim + self.vdim) * self.kv_rank + h * self.heads * self.vdim

    @property
    def kv_elems(self) -> int:
        return self.kv_rank + self.rot_dim


@dataclass(frozen=True)
class Rotary:
    """Rotation of the first ``dims`` dimensions of a head, dimension i with i + dims / 2, by position * base^(-2 i / dims); the
    rest pass.  Angles are divided by ``factor``; with ``original`` (positions of the first training, YaRN) only those that turn
    less than ``slow`` times over them, those above ``fast`` turns stay, a linear ramp in between, and cosines and sines are
    multiplied by 0.1 ln(factor) + 1."""
    dims: int
    base: float
    factor: float = 1.0
    original: float = 0.0
    fast: float = 32.0
    slow: float = 1.0

    def frequencies(self) -> tuple:
        """(angle per position of every pair, factor of cosines and sines), in double precision."""
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if not self.original:
            return [x / self.factor for x in f], 1.0
        at = lambda turns: self.dims * math.log(self.original / (2 * math.pi * turns)) / (2 * math.log(self.base))     # noqa: E731
        lo, hi = max(math.floor(at(self.fast)), 0), min(math.ceil(at(self.slow)), self.dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))]
        return [x / self.factor * r + x * (1 - r) for x, r in zip(f, ramp)], 0.1 * math.log(self.factor) + 1.0


@dataclass(frozen=True)
class GroupedAttention:
    """Grouped-query attention; the cache holds keys and values per key/value head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int = 0                # a position sees its own chunk of this many positions up to itself (0: all before it)
    bias: float = 0.0             # distance bias -(i - j) 2^(-bias (h + 1) / heads) on head h's scores (0: none)
    sink: bool = False            # one learned term per head in the softmax's denominator
    kv_from: int = -1             # layer whose cached keys and values are read (-1: the layer's own)
    log_bias: bool = False        # distance bias -r1 ln(1 + r2 (i - j)) with two learned numbers per head
    qkv_bias: bool = False
    qk_norm: bool = False         # queries and keys: RMS norm per head with a weight shared by the heads
    v_norm: bool = False          # values are divided by their root mean square per head
    temp: float = 0.0             # queries at position p times 1 + temp ln(floor((p + 1) / temp_every) + 1)
    temp_every: int = 1
    rot: Optional[Rotary] = None  # rotation of queries and keys, behind their norms
    rot_values: bool = False      # values are rotated too (all of vdim, plain angles of rot.base), every head's result is turned back
    tied: bool = False            # the values are the projected keys, unrotated
    window: int = 0               # a position sees itself and the window - 1 positions before it (0: all)
    pool: int = 0                 # beside the window: one mean key and value per block of this many positions that lies wholly before it
    gate: bool = False            # the heads' results times the sigmoid of a projection

    def linear_elems(self, h: int) -> int:
        q = self.heads * (self.dim + self.vdim * (2 if self.gate else 1))
        return h * (q + (self.kv_heads * (self.dim + (0 if self.tied else self.vdim)) if self.kv_from < 0 else 0))

    @property
    def kv_elems(self) -> int:
        return self.kv_heads * (self.dim + self.vdim) if self.kv_from < 0 else 0

    @property
    def pool_slots(self) -> int:
        """Blocks that end in a page of 16 positions, at most."""
        return (self.pool + 15) // self.pool if self.pool else 0

    @property
    def pool_elems(self) -> int:
        """Cached elements of a page's blocks."""
        return self.pool_slots * self.kv_elems


@dataclass(frozen=True)
class MatrixLstm:
    """Recurrent mixer with a matrix memory per head (mLSTM): exponential input gate, sigmoid forget gate, both capped."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float
    recurrent = True

    def linear_elems(self, h: int) -> int:
        return h * self.heads * (2 * self.dim + 3 * self.vdim + 2)

    @property
    def kv_elems(self) -> int:
        return 0


@dataclass(frozen=True)
class MinGru:
    """Recurrent mixer, element by element: S <- (1 - z) S + z c, gates from the current token only; the result is S times
    SiLU of a third projection."""
    width: int
    recurrent = True
    heads = 1

    @property
    def dim(self) -> int:
        return self.width

    def linear_elems(self, h: int) -> int:
        return 4 * h * self.width

    @property
    def kv_elems(self) -> int:
        return 0


@dataclass(frozen=True)
class Retention:
    """Recurrent mixer with a matrix memory per head and a fixed decay: S <- decay S + k v^T, the result is S^T q, divided by its
    root mean square per head and times SiLU of a projection; queries and keys are rotated."""
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rot: Rotary
    recurrent = True

    def linear_elems(self, h: int) -> int:
        return h * self.heads * (2 * self.dim + 3 * self.vdim)

    @property
    def kv_elems(self) -> int:
        return 0


@dataclass(frozen=True)
class ParallelMixer:
    """Two mixers side by side on the same input; the result is the sum of theirs, each times its scale -- with ``normed`` each
    one's result divided by its root mean square first, with a weight per column."""
    left: object
    right: object
    left_scale: float
    right_scale: float
    normed: bool = False

    @property
    def heads(self) -> int:
        return max(self.left.heads, self.right.heads)

    @property
    def kv_heads(self) -> int:
        return max(getattr(m, "kv_heads", 1) for m in (self.left, self.right))

    @property
    def dim(self) -> int:
        return max(self.left.dim, self.right.dim)

    @property
    def recurrent(self) -> bool:
        return any(getattr(m, "recurrent", False) for m in (self.left, self.right))

    def linear_elems(self, h: int) -> int:
        return self.left.linear_elems(h) + self.right.linear_elems(h)

    @property
    def kv_elems(self) -> int:
        return self.left.kv_elems + self.right.kv_elems

    @property
    def pool_elems(self) -> int:
        return sum(getattr(m, "pool_elems", 0) for m in (self.left, self.right))


@dataclass(frozen=True)
class ChannelDelta:
    """Recurrent mixer: gated delta rule with one decay per head and key channel; short causal convolutions on q, k and v.
    The ranks of the decay's and the output gate's projections are given by their tensors (0: not known yet)."""
    heads: int                    # value heads; query / key head of head h: h / (heads / kv_heads)
    kv_heads: int
    dim: int
    vdim: int
    conv: int                     # taps
    a_rank: int = 0
    g_rank: int = 0
    recurrent = True

    def linear_elems(self, h: int) -> int:
        qk, v = self.kv_heads * self.dim, self.heads * self.vdim
        return h * (2 * qk + 2 * v + self.heads + self.a_rank + self.g_rank) + self.heads * self.dim * self.a_rank + v * self.g_rank

    @property
    def kv_elems(self) -> int:
        return 0


@dataclass(frozen=True)
class Wkv:
    """Recurrent mixer (RWKV-style time mixing): five inputs, each its own mix of the token and the one before; a decay per
    head and key channel, a bonus for the current token.  The rank of the decay's projection is given by its tensor."""
    heads: int
    dim: int
    w_rank: int = 0
    recurrent = True
    shifts = 5                    # shifted inputs

    def linear_elems(self, h: int) -> int:
        n = self.heads * self.dim
        return 5 * h * n + self.w_rank * (h + n)

    @property
    def kv_elems(self) -> int:
        return 0


@dataclass(frozen=True)
class DenseFfn:
    """down (f(g) (u + shift)), g = min(gate, limit), u = clamp(up, -limit, limit), f(g) = g sigmoid(alpha g), or the tanh form
    of GELU; ``bias``: all three projections have one.  ``relu2``: no gate, down relu(up)^2."""
    ff: int
    limit: float = float("inf")
    alpha: float = 1.0
    shift: float = 0.0
    gelu: bool = False
    bias: bool = False
    relu2: bool = False

    def linear_elems(self, h: int) -> tuple:
        return ((2 if self.relu2 else 3) * self.ff * h,) * 2


@dataclass(frozen=True)
class StreamBlock:
    """Residual of several streams around pre-normed sublayers (hyper-connections): a sublayer reads a mix of the streams,
    its result goes to all of them, times ``mult``.  Norms have one number for all columns; ``shift``: what a mixer reads is
    mixed with the previous token's; the streams start as the embedding plus a sinusoidal position vector (``sinusoid``:
    its base, 0: none).  One stream without ``mixing`` is the plain residual x + y; ``columns``: norms have a weight per
    column, stored around zero."""
    streams: int
    mult: float
    shift: bool = True
    scale: bool = True            # a learned factor per column on every sublayer's result
    sinusoid: float = 10000.0
    mixing: bool = True
    columns: bool = False


@dataclass(frozen=True)
class SandwichBlock:
    """One residual stream with a norm ahead of every sublayer and one behind it: x + norm_b(f(norm_a(x))).  A norm divides each of
    ``groups`` equal parts of a row by the part's own root mean square; the stream starts as the embedding row times ``scale``."""
    groups: int = 1
    scale: float = 1.0
    streams = 1
    shift = mixing = columns = False


@dataclass(frozen=True)
class LayerLoop:
    """Layers ``start`` .. ``stop - 1`` run ``times`` times in a row with the same weights, each pass with its own cache and
    state.  Ahead of a pass a learned vector is added to the residual, and ahead of all but the first the embedding row too."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class ExpertFfn:
    """Routed SwiGLU experts.  ``score``: "softmax" over all experts or a "sigmoid" each; with ``groups`` > 1 only
    experts of the ``keep`` groups with the largest sums of their two best scores can be chosen; ``renorm``: the chosen
    scores are divided by their sum.  ``relu2``: experts without a gate, down relu(up)^2.  ``shared``: width of an expert that
    every token runs, with weight one (0: none)."""
    experts: int
    top: int
    ff: int
    score: str = "sigmoid"
    groups: int = 1
    keep: int = 1
    renorm: bool = False
    relu2: bool = False
    shared: int = 0

    @property
    def rule(self) -> tuple:
        return (int(self.score == "sigmoid"), self.groups, self.keep, int(self.renorm))

    @property
    def shared_slots(self) -> int:
        """Experts of the common width that together are the shared one: its hidden columns are cut into as many runs."""
        ffp = (self.ff + 63) // 64 * 64
        return (self.shared + ffp - 1) // ffp

    def linear_elems(self, h: int) -> tuple:
        """(weights a token's step reads, weights held)."""
        n = 2 if self.relu2 else 3
        one, shared = n * self.ff * h, n * self.shared * h
        return self.experts * h + self.top * one + shared, self.experts * (h + one) + shared


@dataclass(frozen=True)
class LayerSpec:
    """One layer of a model that lists its layers: a mixer and a feed-forward (or none).  How they meet the fp32 residual
    is ``ModelConfig.block``: None adds layer norms of the sublayers' outputs to one stream."""
    mixer: object                 # LatentAttention, GroupedAttention, MatrixLstm, Retention, ParallelMixer, ChannelDelta or Wkv
    ffn: object                   # ExpertFfn, DenseFfn or None
    weights_of: int = -1          # layer whose weights (mixer, feed-forward, norms) this one uses, with a cache of its own (-1: its own)


@dataclass(frozen=True)
class ModelConfig:
    name: str
    n_layers: int
    hidden: int
    n_q_heads: int
    n_kv_heads: int
    head_dim: int
    ffn: int
    vocab: int
    rope_theta: float = 1e6
    rms_eps: float = 1e-6
    group_size: int = 64
    # mixture of experts (n_experts == 0: dense SwiGLU FFN)
    n_experts: int = 0
    top_k: int = 0
    expert_ffn: int = 0
    shared_ffn: int = 0           # 0: no shared expert
    # multi-token-prediction head: extra decoder layers sharing embed / lm_head
    mtp_layers: int = 0
    architecture: str = "B200DenseForCausalLM"
    page_size: int = 16
    # sliding-window attention: a row attends to its last ``sliding_window`` positions (0: the whole context);
    # with ``full_attn_every`` = n > 0 every n-th layer (li % n == n - 1) keeps full attention, as in the
    # reference's windowed families (src/kernels/kolibri/kol_attn.cl: sliding ring 4096 / full layers)
    sliding_window: int = 0
    full_attn_every: int = 0
    # hybrid family: gated delta-net (linear attention) layers with n_k key heads and n_v value heads of 128;
    # with ``gdn_v_heads`` > 0 every layer is a GDN layer except each ``full_attn_every``-th one, which keeps
    # softmax attention (the reference's hybrid checkpoints: src/kernels/gdn_step.cl, three GDN layers per
    # attention layer)
    gdn_k_heads: int = 0
    gdn_v_heads: int = 0
    gdn_head_dim: int = 128
    # models that list their layers one by one (unquantised weights, fp32 residual); the scalar fields above then hold the
    # largest values over the layers
    layer_specs: tuple = ()
    block: object = None          # StreamBlock, SandwichBlock or None
    loop: Optional[LayerLoop] = None

    @property
    def layer_runs(self) -> tuple:
        """(layer, pass that starts ahead of it or -1) of a listed model, in the order in which the layers run.  Caches and
        states belong to runs."""
        n, lp = len(self.layer_specs), self.loop
        if lp is None:
            return tuple((i, -1) for i in range(n))
        body = tuple((i, t if i == lp.start else -1) for t in range(lp.times) for i in range(lp.start, lp.stop))
        return tuple((i, -1) for i in range(lp.start)) + body + tuple((i, -1) for i in range(lp.stop, n))

    @property
    def run_specs(self) -> tuple:
        return tuple(self.layer_specs[i] for i, _ in self.layer_runs)

    @property
    def shift_runs(self) -> tuple:
        """Runs whose mixer reads the previous token's input too."""
        every = self.block is not None and self.block.shift
        return tuple(j for j, s in enumerate(self.run_specs) if every or getattr(s.mixer, "shifts", 0))

    @property
    def q_dim(self) -> int:
        return self.n_q_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.n_kv_heads * self.head_dim

    @property
    def qkv_dim(self) -> int:
        return self.q_dim + 2 * self.kv_dim

    @property
    def gqa(self) -> int:
        return self.n_q_heads // self.n_kv_heads

    @property
    def is_moe(self) -> bool:
        return self.n_experts > 0

    def is_gdn_layer(self, li: int) -> bool:
        if self.gdn_v_heads <= 0 or li >= self.n_layers:
            return False
        return not (self.full_attn_every > 0 and li % self.full_attn_every == self.full_attn_every - 1)

    def gdn_index(self, li: int) -> int:
        """Index of GDN layer ``li`` among the GDN layers (its slice of the recurrent-state buffers)."""
        return sum(1 for i in range(li) if self.is_gdn_layer(i))

    @property
    def n_gdn_layers(self) -> int:
        return sum(1 for i in range(self.n_layers) if self.is_gdn_layer(i))

    @property
    def recurrent(self) -> bool:
        """Sequences carry a state that cannot be rewound position by position."""
        return self.n_gdn_layers > 0 or any(getattr(s.mixer, "recurrent", False) for s in self.layer_specs) or bool(self.shift_runs)

    @property
    def gdn_key_dim(self) -> int:
        return self.gdn_k_heads * self.gdn_head_dim

    @property
    def gdn_value_dim(self) -> int:
        return self.gdn_v_heads * self.gdn_head_dim

    @property
    def gdn_conv_channels(self) -> int:
        return 2 * self.gdn_key_dim + self.gdn_value_dim

    @property
    def gdn_proj_dim(self) -> int:
        """Columns of the fused input projection [ q | k | v | z | b | a ]."""
        return 2 * self.gdn_key_dim + 2 * self.gdn_value_dim + 2 * self.gdn_v_heads

    def window_of(self, li: int) -> int:
        """Attention window of layer ``li`` in positions (0: full attention)."""
        if self.sliding_window <= 0 or self.gdn_v_heads > 0:
            return 0
        if self.full_attn_every > 0 and li % self.full_attn_every == self.full_attn_every - 1:
            return 0
        return self.sliding_window

    def tp_shard(self, world: int) -> "ModelConfig":
        """The shapes one rank of a ``world``-way tensor-parallel group holds: whole attention heads,
        whole FFN interleave runs; hidden size and vocabulary stay (the lm_head is split by rows outside).
        The reference's ``tp_card_desc`` does this for its two cards (src/model/model_desc.cc:252-285)."""
        if world == 1:
            return self
        if self.layer_specs:
            raise ValueError("models that list their layers are not sliced for tensor parallelism")
        if self.n_q_heads % world or self.n_kv_heads % world:
            raise ValueError(f"tensor parallel {world} does not divide {self.n_q_heads} q / {self.n_kv_heads} kv heads")
        if self.ffn % (64 * world) or (self.shared_ffn and self.shared_ffn % (64 * world)):
            raise ValueError(f"tensor parallel {world} does not divide FFN {self.ffn} into whole groups of 64")
        import dataclasses
        return dataclasses.replace(self, name=f"{self.name}/tp{world}", n_q_heads=self.n_q_heads // world,
                                   n_kv_heads=self.n_kv_heads // world, ffn=self.ffn // world,
                                   shared_ffn=self.shared_ffn // world)

    def linears(self):
        """Fused linear table of one decoder layer (attention + dense FFN part)."""
        h = self.hidden
        out = [
            LinearDesc("qkv", self.qkv_dim, h, ("self_attn.q_proj", "self_attn.k_proj", "self_attn.v_proj"), "column"),
            LinearDesc("o", h, self.q_dim, ("self_attn.o_proj",), "row"),
        ]
        if not self.is_moe:
            out += [
                LinearDesc("gate_up", 2 * self.ffn, h, ("mlp.gate_proj", "mlp.up_proj"), "column"),
                LinearDesc("down", h, self.ffn, ("mlp.down_proj",), "row"),
            ]
        return out

    def _mixer_params(self) -> float:
        """Mean weights per layer of the token mixer (attention projections, or a gated delta-net layer's)."""
        h = self.hidden
        attn = self.qkv_dim * h + h * self.q_dim
        g = self.n_gdn_layers
        if not g:
            return attn
        gdn = self.gdn_proj_dim * h + h * self.gdn_value_dim
        return (g * gdn + (self.n_layers - g) * attn) / self.n_layers

    def layer_linears(self, spec: LayerSpec):
        """(weights a token's step reads, weights held) of one listed layer."""
        mix = spec.mixer.linear_elems(self.hidden)
        read, held = spec.ffn.linear_elems(self.hidden) if spec.ffn is not None else (0, 0)
        return mix + read, mix + held

    def param_count(self) -> int:
        h = self.hidden
        if self.layer_specs:
            return int(sum(self.layer_linears(s)[1] for s in self.layer_specs if s.weights_of < 0) + 2 * self.vocab * h)
        per = self._mixer_params()
        if self.is_moe:
            per += self.n_experts * 3 * self.expert_ffn * h + self.n_experts * h
            if self.shared_ffn:
                per += 3 * self.shared_ffn * h + h
        else:
            per += 3 * self.ffn * h
        return int(self.n_layers * per + 2 * self.vocab * h)

    def weight_bytes_per_token(self, lm_head_bytes_per_weight: float = 2.0) -> float:
        """Bytes of weights one decode step must read ("W" in the reference's
        perf model, docs/05-perf-model.md:35-39): int4 nibbles + fp16 group scales
        for every linear that is touched, plus the head."""
        h = self.hidden
        if self.layer_specs:
            return 2.0 * sum(self.layer_linears(s)[0] for s in self.run_specs) + self.vocab * h * lm_head_bytes_per_weight
        int4 = 0.5 + 2.0 / self.group_size
        per = self._mixer_params() * int4
        if self.is_moe:
            per += self.top_k * 3 * self.expert_ffn * h * int4 + self.n_experts * h * 2
            if self.shared_ffn:
                per += 3 * self.shared_ffn * h * int4
        else:
            per += 3 * self.ffn * h * int4
        return self.n_layers * per + self.vocab * h * lm_head_bytes_per_weight

    def kv_bytes_per_token(self, kv_dtype: str = "bf16") -> int:
        if self.layer_specs:
            pooled = sum(getattr(s.mixer, "pool_elems", 0) for s in self.run_specs)      # of a whole page
            return (sum(s.mixer.kv_elems for s in self.run_specs) + -(-pooled // self.page_size)) * (4 if kv_dtype == "f32" else 2)
        per_head = self.head_dim * (2 if kv_dtype == "bf16" else 1) + (4 if kv_dtype == "int8" else 0)
        return (self.n_layers - self.n_gdn_layers) * 2 * self.n_kv_heads * per_head

    def to_listed_config(self) -> dict:
        """The inverse of the listed designs' readers."""
        return {"architecture": self.architecture, "name": self.name, "width": self.hidden, "vocab": self.vocab,
                "norm": {"eps": self.rms_eps}, **LISTED_WRITERS[self.architecture](self)}

    def to_hf_config(self) -> dict:
        if self.layer_specs:
            return self.to_listed_config()
        d = {
            "architectures": [self.architecture],
            "model_type": "b200_moe" if self.is_moe else "b200_dense",
            "num_hidden_layers": self.n_layers,
            "hidden_size": self.hidden,
            "num_attention_heads": self.n_q_heads,
            "num_key_value_heads": self.n_kv_heads,
            "head_dim": self.head_dim,
            "intermediate_size": self.ffn,
            "vocab_size": self.vocab,
            "rope_theta": self.rope_theta,
            "rms_norm_eps": self.rms_eps,
            "num_experts": self.n_experts,
            "num_experts_per_tok": self.top_k,
            "moe_intermediate_size": self.expert_ffn,
            "shared_expert_intermediate_size": self.shared_ffn,
            "mtp_num_hidden_layers": self.mtp_layers,
            "sliding_window": self.sliding_window or None,
            "full_attention_interval": self.full_attn_every,
            "linear_num_key_heads": self.gdn_k_heads,
            "linear_num_value_heads": self.gdn_v_heads,
            "linear_key_head_dim": self.gdn_head_dim,
            "torch_dtype": "bfloat16",
            "quantization_config": {
                "bits": 4, "group_size": self.group_size, "sym": True, "desc_act": False,
                "quant_method": "gptq", "packing_format": "auto_round:auto_gptq",
            },
            "name": self.name,
        }
        return d

    @staticmethod
    def from_hf_config(d: dict) -> "ModelConfig":
        """The configuration of a checkpoint's ``config.json``; a name in ``LISTED_ARCHITECTURES`` under "architecture"
        selects the reader of that design's keys."""
        reader = LISTED_ARCHITECTURES.get(d.get("architecture"))
        if reader is not None:
            return reader(d)
        return ModelConfig(
            name=d.get("name", d.get("_name_or_path", "model")),
            n_layers=d["num_hidden_layers"], hidden=d["hidden_size"],
            n_q_heads=d["num_attention_heads"], n_kv_heads=d.get("num_key_value_heads", d["num_attention_heads"]),
            head_dim=d.get("head_dim", d["hidden_size"] // d["num_attention_heads"]),
            ffn=d.get("intermediate_size", 0), vocab=d["vocab_size"],
            rope_theta=float(d.get("rope_theta", 1e6)), rms_eps=float(d.get("rms_norm_eps", 1e-6)),
            group_size=64,
            n_experts=d.get("num_experts", 0) or 0, top_k=d.get("num_experts_per_tok", 0) or 0,
            expert_ffn=d.get("moe_intermediate_size", 0) or 0,
            shared_ffn=d.get("shared_expert_intermediate_size", 0) or 0,
            mtp_layers=d.get("mtp_num_hidden_layers", 0) or 0,
            sliding_window=d.get("sliding_window", 0) or 0, full_attn_every=d.get("full_attention_interval", 0) or 0,
            gdn_k_heads=d.get("linear_num_key_heads", 0) or 0, gdn_v_heads=d.get("linear_num_value_heads", 0) or 0,
            gdn_head_dim=d.get("linear_key_head_dim", 128) or 128,
            architecture=(d.get("architectures") or ["B200DenseForCausalLM"])[0],
        )


def listed_config(name: str, architecture: str, specs, hidden: int, vocab: int, eps: float,
                  block=None, loop: Optional[LayerLoop] = None) -> ModelConfig:
    """A model given by its layers; the scalar fields other parts of the framework read hold the largest values."""
    specs = tuple(specs)
    ffns = [s.ffn for s in specs if s.ffn is not None]
    most = lambda field: max((getattr(f, field, 0) for f in ffns), default=0)     # noqa: E731
    return ModelConfig(name, len(specs), hidden, max(s.mixer.heads for s in specs), max(getattr(s.mixer, "kv_heads", 1) for s in specs),
                       max(s.mixer.dim + getattr(s.mixer, "rot_dim", 0) for s in specs), 0, vocab, rms_eps=eps,
                       n_experts=most("experts"), top_k=most("top"),
                       expert_ffn=max((f.ff for f in ffns if isinstance(f, ExpertFfn)), default=0),
                       architecture=architecture, layer_specs=specs, block=block, loop=loop)


def mumusun_config(d: dict) -> ModelConfig:
    """``config.json`` of a Mumusun checkpoint: "layers" lists every layer's mixer and feed-forward."""
    specs = []
    for i, layer in enumerate(d["layers"]):
        if layer["type"] != "latent_attention":
            raise ValueError(f"layer {i}: mixer {layer['type']!r} is not part of Mumusun")
        m, f = layer["mixer"], layer["mlp"]
        rot = m["rot"]
        if rot["dims"] % 2 or rot["dims"] > m["rot_dim"]:
            raise ValueError(f"layer {i}: {rot['dims']} rotated dimensions do not fit a part of {m['rot_dim']}")
        mixer = LatentAttention(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"], float(m["scale"]),
                                rot["dims"], float(rot["base"]), (m.get("mask") or {}).get("size", 0) or 0)
        ffn = None
        if f is not None:
            if f["kind"] != "moe":
                raise ValueError(f"layer {i}: feed-forward {f['kind']!r} is not part of Mumusun")
            r = f["router"]
            g = r.get("groups") or {"count": 1, "keep": 1}
            if r["experts"] % g["count"] or r["top"] > g["keep"] * (r["experts"] // g["count"]):
                raise ValueError(f"layer {i}: {r['experts']} experts, {g} and top {r['top']} do not fit together")
            ffn = ExpertFfn(r["experts"], r["top"], f["expert"]["ff"], "sigmoid", g["count"], g["keep"], False)
        specs.append(LayerSpec(mixer, ffn))
    return listed_config(d.get("name", "mumusun"), "Mumusun", specs, d["width"], d["vocab"], float(d["norm"]["eps"]))


def mumusun_keys(c: ModelConfig) -> dict:
    def layer(s):
        m, f = s.mixer, s.ffn
        mixer = {"dim": m.dim, "heads": m.heads, "kv_rank": m.kv_rank, "q_rank": m.q_rank, "rot_dim": m.rot_dim,
                 "vdim": m.vdim, "scale": m.scale, "rot": {"base": m.rope_base, "dims": m.rope_dims}}
        if m.window:
            mixer["mask"] = {"size": m.window}
        mlp = None if f is None else {"kind": "moe", "expert": {"ff": f.ff}, "router": {
            "experts": f.experts, "top": f.top, "groups": {"count": f.groups, "keep": f.keep}}}
        return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}
    return {"layers": [layer(s) for s in c.layer_specs]}


def napadra_config(d: dict) -> ModelConfig:
    """``config.json`` of a Napadra checkpoint: chunked attention with a distance bias and sinks, layers that read another
    layer's keys and values, mLSTM layers, clamped feed-forwards, over several residual streams."""
    specs = []
    for i, layer in enumerate(d["layers"]):
        m, f = layer["mixer"], layer["mlp"]
        if layer["type"] == "attention":
            mixer = GroupedAttention(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]),
                                     (m.get("mask") or {}).get("size", 0) or 0, 8.0, True, m.get("kv_from", -1))
            if mixer.heads % mixer.kv_heads:
                raise ValueError(f"layer {i}: {mixer.heads} query heads over {mixer.kv_heads} key/value heads")
            if mixer.kv_from >= 0:
                src = specs[mixer.kv_from].mixer if mixer.kv_from < i else None
                if not isinstance(src, GroupedAttention) or src.kv_from >= 0 or \
                        (src.kv_heads, src.dim, src.vdim) != (mixer.kv_heads, mixer.dim, mixer.vdim):
                    raise ValueError(f"layer {i}: layer {mixer.kv_from} has no keys and values that fit it")
        elif layer["type"] == "mlstm":
            mixer = MatrixLstm(m["heads"], m["dim"], m["vdim"], float(m["gate_cap"]))
            if mixer.dim > 512 or mixer.vdim > 512:
                raise ValueError(f"layer {i}: mLSTM heads of {mixer.dim} x {mixer.vdim} (512 at most)")
        else:
            raise ValueError(f"layer {i}: mixer {layer['type']!r} is not part of Napadra")
        ffn = None
        if f is not None:
            if f["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward {f['kind']!r} is not part of Napadra")
            ffn = DenseFfn(f["ff"], float(f["limit"]), 1.702, 1.0)
        specs.append(LayerSpec(mixer, ffn))
    if not 1 <= d["streams"] <= 8:
        raise ValueError(f"{d['streams']} residual streams (1 to 8)")
    return listed_config(d.get("name", "napadra"), "Napadra", specs, d["width"], d["vocab"], float(d["norm"]["eps"]),
                         StreamBlock(d["streams"], float(d["residual_mult"])))


def napadra_keys(c: ModelConfig) -> dict:
    def layer(s):
        m, f = s.mixer, s.ffn
        mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
        if isinstance(m, MatrixLstm):
            mixer["gate_cap"] = m.gate_cap
        else:
            mixer.update(kv_heads=m.kv_heads, scale=m.scale)
            if m.chunk:
                mixer["mask"] = {"size": m.chunk}
            if m.kv_from >= 0:
                mixer["kv_from"] = m.kv_from
        return {"type": "mlstm" if isinstance(m, MatrixLstm) else "attention", "mixer": mixer,
                "mlp": None if f is None else {"kind": "dense", "ff": f.ff, "limit": f.limit}}
    return {"streams": c.block.streams, "residual_mult": c.block.mult, "layers": [layer(s) for s in c.layer_specs]}


def pefulorn_config(d: dict) -> ModelConfig:
    """``config.json`` of a Pefulorn checkpoint: delta-rule layers with a decay per key channel, layers of attention with a
    logarithmic distance bias beside a minGRU, time-mixing layers, dense feed-forwards, over one pre-normed residual; a range
    of layers may run several times."""
    specs = []
    for i, layer in enumerate(d["layers"]):
        m, f = layer["mixer"], layer["mlp"]
        if layer["type"] == "channel_delta":
            mixer = ChannelDelta(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
            if not 1 <= mixer.conv <= 16:
                raise ValueError(f"layer {i}: convolution of {mixer.conv} taps (1 to 16)")
        elif layer["type"] == "parallel":
            a, t = m["left"], m["left"].get("q_temp") or {"coef": 0.0, "every": 1}
            left = GroupedAttention(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), log_bias=True, qkv_bias=True,
                                    qk_norm=True, v_norm=True, temp=float(t["coef"]), temp_every=t["every"])
            if max(left.dim, left.vdim) > 1024 or left.temp_every < 1:
                raise ValueError(f"layer {i}: attention heads of {left.dim} x {left.vdim} (1024 at most), temperature {t}")
            mixer = ParallelMixer(left, MinGru(m["right"]["width"]), float(m["left_scale"]), float(m["right_scale"]))
        elif layer["type"] == "wkv":
            mixer = Wkv(m["heads"], m["dim"])
        else:
            raise ValueError(f"layer {i}: mixer {layer['type']!r} is not part of Pefulorn")
        if not isinstance(mixer, ParallelMixer) and max(mixer.dim, getattr(mixer, "vdim", 0)) > 512:
            raise ValueError(f"layer {i}: recurrent heads of {mixer.dim} x {getattr(mixer, 'vdim', mixer.dim)} (512 at most)")
        heads = mixer.left if isinstance(mixer, ParallelMixer) else mixer
        if heads.heads % getattr(heads, "kv_heads", 1):
            raise ValueError(f"layer {i}: {heads.heads} heads over {heads.kv_heads} key heads")
        ffn = None
        if f is not None:
            if f["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward {f['kind']!r} is not part of Pefulorn")
            ffn = DenseFfn(f["ff"], gelu=True, bias=True)
        specs.append(LayerSpec(mixer, ffn))
    loop = d.get("loop")
    if loop is not None:
        loop = LayerLoop(loop["start"], loop["stop"], loop["times"])
        if not 0 <= loop.start < loop.stop <= len(specs) or loop.times < 1:
            raise ValueError(f"{loop} does not fit {len(specs)} layers")
    return listed_config(d.get("name", "pefulorn"), "Pefulorn", specs, d["width"], d["vocab"], float(d["norm"]["eps"]),
                         StreamBlock(1, 1.0, shift=False, scale=False, sinusoid=0.0, mixing=False, columns=True), loop)


def pefulorn_keys(c: ModelConfig) -> dict:
    def layer(s):
        m, f = s.mixer, s.ffn
        if isinstance(m, ChannelDelta):
            kind, mixer = "channel_delta", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
        elif isinstance(m, Wkv):
            kind, mixer = "wkv", {"heads": m.heads, "dim": m.dim}
        else:
            a = m.left
            left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
            if a.temp:
                left["q_temp"] = {"coef": a.temp, "every": a.temp_every}
            kind, mixer = "parallel", {"left": left, "left_scale": m.left_scale, "right": {"width": m.right.width},
                                       "right_scale": m.right_scale}
        return {"type": kind, "mixer": mixer, "mlp": None if f is None else {"kind": "dense", "ff": f.ff}}
    out = {"layers": [layer(s) for s in c.layer_specs]}
    if c.loop is not None:
        out["loop"] = {"start": c.loop.start, "stop": c.loop.stop, "times": c.loop.times}
    return out


def _rotary(r: dict) -> Rotary:
    s = r.get("scaling") or {}
    if r["dims"] % 2 or r["dims"] < 0:
        raise ValueError(f"{r['dims']} rotated dimensions")
    return Rotary(r["dims"], float(r["base"]), float(s.get("factor", 1.0)), float(s.get("original", 0.0)), float(s.get("fast", 32.0)),
                  float(s.get("slow", 1.0)))


def _rotary_keys(r: Rotary) -> dict:
    out = {"dims": r.dims, "base": r.base}
    if r.original:
        out["scaling"] = {"factor": r.factor, "original": r.original, "fast": r.fast, "slow": r.slow}
    elif r.factor != 1.0:
        out["scaling"] = {"factor": r.factor}
    return out


def vogerax_config(d: dict) -> ModelConfig:
    """``config.json`` of a Vogerax checkpoint: attention over a window and pooled blocks before it whose values are its keys,
    layers of gated attention with rotated values beside retention, ungated feed-forwards and experts, layers that use another
    one's weights, a residual with norms on both sides of every sublayer."""
    specs = []
    for i, layer in enumerate(d["layers"]):
        m, f = layer["mixer"], layer["mlp"]
        if layer["type"] == "attention":
            mask = m.get("mask") or {}
            mixer = GroupedAttention(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), rot=_rotary(m["rot"]), tied=True,
                                     window=mask.get("size", 0) or 0, pool=mask.get("pool", 0) or 0)
            if mixer.vdim != mixer.dim:
                raise ValueError(f"layer {i}: values of {mixer.vdim} dimensions that are keys of {mixer.dim}")
            if mixer.window < 0 or mixer.pool < 0 or mixer.pool and not mixer.window:
                raise ValueError(f"layer {i}: mask {mask}")
            heads = mixer
        elif layer["type"] == "parallel":
            a, b = m["left"], m["right"]
            heads = GroupedAttention(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), sink=True, qk_norm=True,
                                     rot=_rotary(a["rot"]), rot_values=True, gate=True)
            right = Retention(b["heads"], b["dim"], b["vdim"], tuple(float(x) for x in b["decay"]), _rotary(b["rot"]))
            if len(right.decay) != right.heads:
                raise ValueError(f"layer {i}: {len(right.decay)} decays for {right.heads} heads")
            if max(right.dim, right.vdim) > 512 or right.rot.dims > right.dim:
                raise ValueError(f"layer {i}: retention heads of {right.dim} x {right.vdim} (512 at most), {right.rot}")
            if heads.vdim % 2:
                raise ValueError(f"layer {i}: {heads.vdim} rotated value dimensions")
            mixer = ParallelMixer(heads, right, 0.5, 0.5, True)
        else:
            raise ValueError(f"layer {i}: mixer {layer['type']!r} is not part of Vogerax")
        if heads.heads % heads.kv_heads or max(heads.dim, heads.vdim) > 1024 or heads.rot.dims > heads.dim:
            raise ValueError(f"layer {i}: {heads.heads} / {heads.kv_heads} heads of {heads.dim} x {heads.vdim} (1024 at most), {heads.rot}")
        ffn = None
        if f is not None:
            if f["kind"] == "dense":
                ffn = DenseFfn(f["ff"], relu2=True)
            elif f["kind"] == "moe":
                r = f["router"]
                if not 1 <= r["top"] <= min(r["experts"], 32) or r["experts"] > 512:
                    raise ValueError(f"layer {i}: {r['top']} of {r['experts']} experts (32 of 512 at most)")
                ffn = ExpertFfn(r["experts"], r["top"], f["expert"]["ff"], "softmax", relu2=True, shared=(f.get("shared") or {}).get("ff", 0))
            else:
                raise ValueError(f"layer {i}: feed-forward {f['kind']!r} is not part of Vogerax")
        of = layer.get("weights_of")
        specs.append(LayerSpec(mixer, ffn, -1 if of is None else of))
    for i, s in enumerate(specs):
        seen, j = {i}, s.weights_of
        while j >= 0:
            if j >= len(specs) or j in seen or (specs[j].mixer, specs[j].ffn) != (s.mixer, s.ffn):
                raise ValueError(f"layer {i} cannot use the weights of layer {j}")
            seen.add(j)
            j = specs[j].weights_of
    groups = d["norm"].get("groups", 1)
    if groups < 1 or d["width"] % groups:
        raise ValueError(f"{groups} norm groups of {d['width']} columns")
    scale = float((d.get("embedding") or {}).get("scale", 1.0))
    return listed_config(d.get("name", "vogerax"), "Vogerax", specs, d["width"], d["vocab"], float(d["norm"]["eps"]),
                         SandwichBlock(groups, scale))


def vogerax_keys(c: ModelConfig) -> dict:
    def layer(s):
        m, f = s.mixer, s.ffn
        if isinstance(m, ParallelMixer):
            a, b = m.left, m.right
            kind, mixer = "parallel", {
                "left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "rot": _rotary_keys(a.rot)},
                "right": {"heads": b.heads, "dim": b.dim, "vdim": b.vdim, "decay": list(b.decay), "rot": _rotary_keys(b.rot)}}
        else:
            kind, mixer = "attention", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                                        "rot": _rotary_keys(m.rot)}
            if m.window:
                mixer["mask"] = {"size": m.window, **({"pool": m.pool} if m.pool else {})}
        mlp = None
        if isinstance(f, DenseFfn):
            mlp = {"kind": "dense", "ff": f.ff}
        elif f is not None:
            mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
            if f.shared:
                mlp["shared"] = {"ff": f.shared}
        return {"type": kind, "mixer": mixer, "mlp": mlp, **({"weights_of": s.weights_of} if s.weights_of >= 0 else {})}
    return {"embedding": {"scale": c.block.scale}, "norm": {"eps": c.rms_eps, "groups": c.block.groups},
            "layers": [layer(s) for s in c.layer_specs]}


LISTED_ARCHITECTURES = {"Mumusun": mumusun_config, "Napadra": napadra_config, "Pefulorn": pefulorn_config, "Vogerax": vogerax_config}
LISTED_WRITERS = {"Mumusun": mumusun_keys, "Napadra": napadra_keys, "Pefulorn": pefulorn_keys, "Vogerax": vogerax_keys}


def tiny_dense() -> ModelConfig:
    """The CPU-oracle configuration: 2 layers, hidden 256, 4 q / 2 kv heads of 64."""
    return ModelConfig("tiny-dense", 2, 256, 4, 2, 64, 704, 1024)


def small_dense() -> ModelConfig:
    """Small dense model with the production head size (128), for the tensor-core prefill path."""
    return ModelConfig("small-dense", 2, 512, 8, 2, 128, 1408, 2048)


def small_windowed() -> ModelConfig:
    """Four layers of the small dense shape; layers 0 and 2 attend to the last 48 positions, 1 and 3 to all."""
    return ModelConfig("small-windowed", 4, 512, 8, 2, 128, 1408, 2048, sliding_window=48, full_attn_every=2)


def small_hybrid() -> ModelConfig:
    """Four layers of the small dense shape: layers 0 and 2 are gated delta-net layers (2 key / 4 value heads of
    128), layers 1 and 3 softmax attention."""
    return ModelConfig("small-hybrid", 4, 512, 8, 2, 128, 1408, 2048, full_attn_every=2, gdn_k_heads=2, gdn_v_heads=4,
                       architecture="B200HybridForCausalLM")


def tiny_moe() -> ModelConfig:
    return ModelConfig("tiny-moe", 2, 256, 4, 2, 64, 0, 1024, n_experts=8, top_k=2,
                       expert_ffn=128, shared_ffn=128, architecture="B200MoeForCausalLM")


def small_moe() -> ModelConfig:
    """Small MoE with the production head size, for the grouped tensor-core path."""
    return ModelConfig("small-moe", 2, 512, 8, 2, 128, 0, 2048, n_experts=16, top_k=4, expert_ffn=256,
                       shared_ffn=256, architecture="B200MoeForCausalLM")


def dense_27b() -> ModelConfig:
    """27B-shape dense decoder: 64 layers, hidden 5120, 40 q / 8 kv heads of 128, FFN 17408."""
    return ModelConfig("dense-27b", 64, 5120, 40, 8, 128, 17408, 151936)


def hybrid_27b() -> ModelConfig:
    """27B-shape hybrid decoder: the dense 27B shape with three gated delta-net layers (16 key / 48 value heads of
    128) before every softmax-attention layer."""
    return ModelConfig("hybrid-27b", 64, 5120, 40, 8, 128, 17408, 151936, full_attn_every=4, gdn_k_heads=16,
                       gdn_v_heads=48, architecture="B200HybridForCausalLM")


def moe_35b_a3b() -> ModelConfig:
    """35B-A3B-shape MoE: 40 layers, hidden 2048, 16 q / 4 kv heads, 256 experts top-8 + shared."""
    return ModelConfig("moe-35b-a3b", 40, 2048, 16, 4, 128, 0, 151936, n_experts=256, top_k=8,
                       expert_ffn=512, shared_ffn=512, architecture="B200MoeForCausalLM")


def mumusun_mini() -> ModelConfig:
    """Small Mumusun: four layers of unequal sizes, windows and experts, the last one without a feed-forward."""
    def mix(heads, dim, rot, vdim, rank, q_rank, window):
        return LatentAttention(heads, dim, rot, vdim, rank, q_rank, (dim + rot) ** -0.5, rot, 1e5, window)
    return listed_config("mumusun-mini", "Mumusun", (
        LayerSpec(mix(4, 64, 32, 64, 192, 160, 96), ExpertFfn(16, 4, 96, groups=4, keep=2)),
        LayerSpec(mix(8, 48, 24, 56, 136, 120, 0), ExpertFfn(9, 2, 72, groups=3, keep=1)),
        LayerSpec(mix(20, 40, 16, 96, 256, 200, 33), ExpertFfn(6, 3, 128, groups=1, keep=1)),
        LayerSpec(mix(3, 96, 40, 112, 320, 88, 160), None)), 320, 1000, 1e-5)


def mumusun_16b() -> ModelConfig:
    """A Mumusun of real layer sizes: 27 layers, hidden 2048, 16 heads of 128 + 64 over a latent of 512 with a window of
    4096, 64 experts of 1408 in 8 groups, 6 per token."""
    mix = LatentAttention(16, 128, 64, 128, 512, 1536, 192 ** -0.5, 64, 1e6, 4096)
    return listed_config("mumusun-16b", "Mumusun", (LayerSpec(mix, ExpertFfn(64, 6, 1408, groups=8, keep=4)),) * 27, 2048,
                         102400, 1e-6)


def napadra_mini() -> ModelConfig:
    """Small Napadra: attention layers of unequal sizes and chunks, one that reads another's keys, two mLSTM layers."""
    att = lambda h, g, dim, vdim, chunk, src=-1: GroupedAttention(h, g, dim, vdim, dim ** -0.5, chunk, 8.0, True, src)  # noqa: E731
    ff = lambda n, limit: DenseFfn(n, limit, 1.702, 1.0)                                                               # noqa: E731
    return listed_config("napadra-mini", "Napadra", (
        LayerSpec(att(6, 2, 40, 72, 96), ff(176, 3.0)), LayerSpec(MatrixLstm(3, 80, 112, 10.0), ff(112, 1.5)),
        LayerSpec(att(4, 4, 128, 64, 150), None), LayerSpec(MatrixLstm(5, 32, 40, 6.0), None),
        LayerSpec(att(6, 2, 40, 72, 33, 0), ff(80, 2.5)), LayerSpec(att(8, 1, 72, 136, 0), ff(96, 4.0))), 200, 700, 1e-5,
        StreamBlock(3, 0.8))


def napadra_7b() -> ModelConfig:
    """A Napadra of real layer sizes: width 4096, 32 layers in groups of two mLSTM layers (8 heads of 256 x 512) and two
    attention layers (32 / 8 heads of 128, chunks of 8192, the second on the first one's keys), 11008 wide feed-forwards, four
    streams."""
    ffn, specs = DenseFfn(11008, 7.0, 1.702, 1.0), []
    for i in range(0, 32, 4):
        att = GroupedAttention(32, 8, 128, 128, 128 ** -0.5, 8192, 8.0, True)
        specs += [LayerSpec(MatrixLstm(8, 256, 512, 15.0), ffn)] * 2 + [LayerSpec(att, ffn), LayerSpec(replace(att, kv_from=i + 2), ffn)]
    return listed_config("napadra-7b", "Napadra", specs, 4096, 64000, 1e-5, StreamBlock(4, 0.5))


def _parallel(heads, kv, dim, vdim, width, every, coef=0.4, scales=(1.0, 1.0)) -> ParallelMixer:
    return ParallelMixer(GroupedAttention(heads, kv, dim, vdim, dim ** -0.5, log_bias=True, qkv_bias=True, qk_norm=True, v_norm=True,
                                          temp=coef, temp_every=every), MinGru(width), *scales)


def pefulorn_mini() -> ModelConfig:
    """Small Pefulorn: every kind of layer with unequal sizes, the middle ones run three times."""
    ff = lambda n: DenseFfn(n, gelu=True, bias=True)                               # noqa: E731
    return listed_config("pefulorn-mini", "Pefulorn", (
        LayerSpec(_parallel(6, 2, 40, 72, 136, 50, 0.7, (0.8, 1.3)), ff(176)), LayerSpec(ChannelDelta(6, 2, 48, 40, 3, 20, 36), ff(112)),
        LayerSpec(Wkv(3, 72, 28), None), LayerSpec(_parallel(4, 4, 96, 64, 80, 7), None), LayerSpec(Wkv(2, 40, 70), ff(80)),
        LayerSpec(ChannelDelta(3, 3, 80, 130, 4, 72, 12), ff(96))), 200, 700, 1e-5,
        StreamBlock(1, 1.0, shift=False, scale=False, sinusoid=0.0, mixing=False, columns=True), LayerLoop(1, 4, 3))


def pefulorn_like(name: str, width: int, layers: int, heads: int, kv: int, ff: int, vocab: int, rank: int = 128) -> ModelConfig:
    """A Pefulorn of real layer sizes: groups of two delta-rule layers, a time-mixing layer and a layer of attention beside a
    minGRU of the model's width, all heads of 128."""
    f, specs = DenseFfn(ff, gelu=True, bias=True), []
    for _ in range(0, layers, 4):
        specs += [LayerSpec(ChannelDelta(heads, heads, 128, 128, 4, rank, rank), f)] * 2 + [
            LayerSpec(Wkv(heads, 128, rank), f), LayerSpec(_parallel(heads, kv, 128, 128, width, 8192, 0.1), f)]
    return listed_config(name, "Pefulorn", specs, width, vocab, 1e-6,
                         StreamBlock(1, 1.0, shift=False, scale=False, sinusoid=0.0, mixing=False, columns=True))


def pefulorn_7b() -> ModelConfig:
    """32 layers, hidden 4096, 32 heads of 128 (8 key heads in the attention layers), 11008 wide feed-forwards."""
    return pefulorn_like("pefulorn-7b", 4096, 32, 32, 8, 11008, 64000)


def vogerax_mini() -> ModelConfig:
    """Small Vogerax: both kinds of layers with unequal sizes, windows and blocks, shared weights, a layer without a feed-forward."""
    att = lambda h, g, dim, rot, window, pool: GroupedAttention(h, g, dim, dim, 0.9 * dim ** -0.5, rot=rot, tied=True, window=window, pool=pool)  # noqa: E731
    par = lambda left, right: ParallelMixer(GroupedAttention(*left[:4], left[2] ** -0.5, sink=True, qk_norm=True, rot=left[4],                    # noqa: E731
                                                             rot_values=True, gate=True), Retention(*right), 0.5, 0.5, True)
    a = att(6, 2, 40, Rotary(24, 2e4, 2.0), 70, 6)
    moe = ExpertFfn(12, 3, 80, "softmax", relu2=True, shared=150)
    return listed_config("vogerax-mini", "Vogerax", (
        LayerSpec(par((4, 2, 48, 72, Rotary(40, 1e4, 4.0, 128, 16.0, 1.5)), (3, 56, 40, (0.97, 0.9, 0.995), Rotary(32, 3e4))), DenseFfn(176, relu2=True)),
        LayerSpec(a, moe), LayerSpec(a, moe, 1), LayerSpec(att(4, 4, 72, Rotary(72, 1e4), 33, 20), None),
        LayerSpec(par((3, 1, 130, 36, Rotary(64, 5e4, 8.0, 64, 32.0, 1.0)), (2, 96, 136, (0.99, 0.8), Rotary(96, 1e4, 3.0))),
                  ExpertFfn(9, 2, 128, "softmax", relu2=True)), LayerSpec(att(2, 1, 40, Rotary(16, 1e4), 16, 16), DenseFfn(64, relu2=True))),
        210, 700, 1e-5, SandwichBlock(3, 8.0))


def vogerax_like(name: str, width: int, layers: int, heads: int, kv: int, ff: int, experts: int, top: int, vocab: int, window: int = 2048,
                 pool: int = 16, r_heads: int = 0) -> ModelConfig:
    """A Vogerax of real layer sizes: groups of three windowed layers and one of attention beside retention, all heads of 128,
    experts of width ``ff`` and a shared one of twice that in every layer."""
    f = ExpertFfn(experts, top, ff, "softmax", relu2=True, shared=2 * ff)
    near = GroupedAttention(heads, kv, 128, 128, 128 ** -0.5, rot=Rotary(64, 1e6, 4.0), tied=True, window=window, pool=pool)
    r = r_heads or heads
    both = ParallelMixer(GroupedAttention(heads, kv, 128, 128, 128 ** -0.5, sink=True, qk_norm=True, rot=Rotary(128, 1e6, 4.0, 8192), rot_values=True,
                                          gate=True), Retention(r, 128, 128, tuple(1 - 2.0 ** (-5 - 7 * i / r) for i in range(r)), Rotary(128, 1e6)), 0.5, 0.5, True)
    return listed_config(name, "Vogerax", ([LayerSpec(near, f)] * 3 + [LayerSpec(both, f)]) * (layers // 4), width, vocab, 1e-6, SandwichBlock(2, width ** 0.5))


def vogerax_16b() -> ModelConfig:
    """28 layers, hidden 2048, 16 heads of 128 (4 key heads), 64 experts of 2048, 6 per token, a shared one of 4096."""
    return vogerax_like("vogerax-16b", 2048, 28, 16, 4, 2048, 64, 6, 102400)


def dflash_drafter(target: ModelConfig) -> ModelConfig:
    """DFlash-style block drafter: a 2-layer W4A16 decoder at the target's width."""
    return replace(target, name=target.name + "-dflash", n_layers=2, n_experts=0, top_k=0, expert_ffn=0,
                   shared_ffn=0, ffn=target.ffn if target.ffn else 4 * target.hidden, mtp_layers=0,
                   architecture="B200DFlashDrafter")


PRESETS = {
    "tiny-dense": tiny_dense, "tiny-moe": tiny_moe, "small-dense": small_dense, "small-windowed": small_windowed, "small-hybrid": small_hybrid, "small-moe": small_moe, "dense-27b": dense_27b, "hybrid-27b": hybrid_27b, "moe-35b-a3b": moe_35b_a3b,
    "mumusun-mini": mumusun_mini, "mumusun-16b": mumusun_16b, "napadra-mini": napadra_mini, "napadra-7b": napadra_7b,
    "pefulorn-mini": pefulorn_mini, "pefulorn-7b": pefulorn_7b, "vogerax-mini": vogerax_mini, "vogerax-16b": vogerax_16b,
}


def preset(name: str) -> ModelConfig:
    if name not in PRESETS:
        raise KeyError(f"unknown model preset {name!r}; known: {sorted(PRESETS)}")
    return PRESETS[name]()
