"""Weight containers shared by the CPU oracle and the GPU models.

A quantised linear is held in the kernel ("W4B") layout only; the oracle
dequantises it on demand.  ``random_weights`` builds a whole random-init model
either by quantising fp32 normal(0, 0.02) matrices (exact, used for the tiny
configurations and for writing synthetic checkpoints) or by drawing nibbles and
scales directly on the device (used for the full-size benchmark shapes).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ..utils import quant as Q
from .config import ModelConfig


@dataclass
class QLinear:
    """W4A16 linear in W4B layout. ``w4b`` is uint8 ``[ceil(n/128)][k/64][4352]``."""
    w4b: torch.Tensor
    n: int
    k: int
    _w_f32: Optional[torch.Tensor] = None     # oracle cache
    _w_bf16: Optional[torch.Tensor] = None    # resident bf16 copy for the prefill GEMM
    _w_i8: Optional[tuple] = None             # (int8 [n][k], fp32 row scale) for the int8 prefill GEMM

    def dequant_f32(self) -> torch.Tensor:
        if self._w_f32 is None:
            self._w_f32 = Q.dequant_w4b(self.w4b.cpu(), self.n)
        return self._w_f32

    @property
    def nbytes(self) -> int:
        return self.w4b.numel()

    @staticmethod
    def from_f32(w: torch.Tensor, device="cpu") -> "QLinear":
        q, s = Q.quantize_rtn(w)
        return QLinear(Q.to_w4b(q, s).to(device), w.shape[0], w.shape[1])

    @staticmethod
    def random(n: int, k: int, device, seed: int, std: float = 0.02) -> "QLinear":
        return QLinear(Q.random_w4b(n, k, device, seed, std), n, k)


def interleave16(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """Fuse gate and up rows in alternating runs of 16 (``g0..15, u0..15, g16..``).

    With this order a GEMM epilogue thread that owns 32 consecutive output
    columns holds 16 gate values and their 16 up values, so SiLU(g)*u is
    computed without a second pass (the reference fuses gate‖up the same way,
    src/loader/loader.cc:308).
    """
    i, k = gate.shape
    assert i % 16 == 0
    return torch.stack([gate.reshape(i // 16, 16, k), up.reshape(i // 16, 16, k)], dim=1).reshape(2 * i, k)


def deinterleave16(x: torch.Tensor):
    """Split the last dim of ``x`` (2*I, interleave16 order) into (gate, up)."""
    *lead, n = x.shape
    v = x.reshape(*lead, n // 32, 2, 16)
    return v[..., 0, :].reshape(*lead, n // 2), v[..., 1, :].reshape(*lead, n // 2)


@dataclass
class ExpertWeights:
    gate_up: QLinear      # [2*expert_ffn][hidden], interleave16
    down: QLinear         # [hidden][expert_ffn]


@dataclass
class GdnWeights:
    """A gated delta-net layer: fused input projection [ q | k | v | z | b | a ], depthwise 4-tap convolution over
    q, k, v, per-head decay parameters, the gated output norm and the output projection."""
    in_proj: QLinear               # [gdn_proj_dim][hidden]
    conv_w: torch.Tensor           # fp32 [conv_channels][4]; tap 3 multiplies the newest input
    a_log: torch.Tensor            # fp32 [n_v]
    dt_bias: torch.Tensor          # fp32 [n_v]
    norm_w: torch.Tensor           # fp32 [head_dim]
    out_proj: QLinear              # [hidden][value_dim]


@dataclass
class LatentWeights:
    """A latent-attention mixer, unquantised (bf16, or fp32 for models served in 32-bit), padded to whole 64s."""
    down: torch.Tensor             # [qp + kvp + rp][Wp]: query latent, key-value latent, shared rotated key part
    q_norm: torch.Tensor           # fp32 [q_rank]
    kv_norm: torch.Tensor          # fp32 [kv_rank]
    uq: torch.Tensor               # [heads * (dn + rp)][qp]
    uk: torch.Tensor               # [heads * dn][kvp]
    uv: torch.Tensor               # [heads * dv][kvp]
    o: torch.Tensor                # [Wp][heads * dv]


@dataclass
class GroupedWeights:
    """A grouped-query attention mixer, unquantised, heads padded to whole 64s; rotated pairs are neighbours."""
    qkv: Optional[torch.Tensor]    # [heads * dk + kv_heads * (dk + dv)][Wp], without values that are the keys and with [heads * dv]
                                   # rows of a gate behind; or the queries' rows alone
    o: Optional[torch.Tensor]      # [Wp][heads * dv]
    slope2: Optional[torch.Tensor]     # fp32 [heads] distance bias times log2 e
    sink2: Optional[torch.Tensor]      # fp32 [heads] sinks times log2 e
    bias: Optional[torch.Tensor] = None      # fp32 [heads * dk + kv_heads * (dk + dv)]
    q_norm: Optional[torch.Tensor] = None    # fp32 [dk]
    k_norm: Optional[torch.Tensor] = None    # fp32 [dk]
    r1: Optional[torch.Tensor] = None        # fp32 [heads] logarithmic distance bias
    r2: Optional[torch.Tensor] = None


@dataclass
class RetentionWeights:
    """A retention mixer, unquantised, heads padded to whole 64s; rotated pairs of q and k are neighbours."""
    proj: Optional[torch.Tensor]   # [heads * 2 (dk + dv)][Wp]: q, k, v, gate
    o: Optional[torch.Tensor]      # [Wp][heads * dv]
    decay: torch.Tensor            # fp32 [2][heads]: decays and their log2


@dataclass
class MlstmWeights:
    """An mLSTM mixer, unquantised, heads padded to whole 64s."""
    proj: torch.Tensor             # [heads * 2 (dk + dv) + gates][Wp]: q, k, v, output gate, input gates, forget gates
    gate_bias: torch.Tensor        # fp32 [2 * heads]
    norm: torch.Tensor             # fp32 [heads * dv]
    o: torch.Tensor                # [Wp][heads * dv]


@dataclass
class MinGruWeights:
    """A minGRU mixer, unquantised, padded to whole 64s."""
    proj: Optional[torch.Tensor]   # [3 * wp][Wp]: gate, candidate, output gate
    o: Optional[torch.Tensor]      # [Wp][wp]
    bias_z: torch.Tensor           # fp32 [wp]
    bias_x: torch.Tensor           # fp32 [wp]


@dataclass
class ParallelWeights:
    """Two mixers side by side: their input projections one below the other, their output projections side by side -- or, where each
    one's result has a norm of its own, one below the other (equal columns) or apart."""
    proj: torch.Tensor
    o: Optional[torch.Tensor]
    left: object                   # the two mixers' other weights
    right: object
    norms: Optional[list] = None   # fp32 [Wp] each
    outs: Optional[list] = None    # output projections apart


@dataclass
class DeltaWeights:
    """A delta-rule mixer with a decay per key channel, unquantised, heads padded."""
    proj: torch.Tensor             # [2 * kv_heads * dk + heads * dv + ...][Wp]: q, k, v, step sizes, first halves of decay and gate
    conv: torch.Tensor             # fp32 [taps][2 * kv_heads * dk + heads * dv]
    neg_a: torch.Tensor            # fp32 [heads]: exp(A_log)
    dt_bias: torch.Tensor          # fp32 [heads * dk]
    second: torch.Tensor           # [heads * (dk + dv)][kp] second halves of decay and gate; bf16: twice side by side, for two limbs
    norm: torch.Tensor             # fp32 [heads * dv]
    o: torch.Tensor                # [Wp][heads * dv]


@dataclass
class WkvWeights:
    """A time-mixing (wkv) mixer, unquantised, heads padded."""
    proj: torch.Tensor             # [4 * heads * d + ...][Wp]: r, k, v, gate, first half of the decay
    shift: torch.Tensor            # fp32 [5][Wp]: how much of the previous token r, k, v, gate and decay read
    u: torch.Tensor                # fp32 [heads * d]
    w0: torch.Tensor               # fp32 [heads * d]
    second: torch.Tensor           # [heads * d][kp], as in DeltaWeights
    norm: torch.Tensor             # fp32 [heads * d]
    o: torch.Tensor                # [Wp][heads * d]


@dataclass
class DenseWeights:
    """Unquantised feed-forward, padded to whole 64s."""
    gate_up: torch.Tensor          # [2 * ffp][Wp], interleave16; without a gate [ffp][Wp]
    down: torch.Tensor             # [Wp][ffp]
    bias: Optional[torch.Tensor] = None          # fp32 [2 * ffp], interleave16
    down_bias: Optional[torch.Tensor] = None     # fp32 [Wp]


@dataclass
class StreamWeights:
    """How a layer's sublayers (mixer, feed-forward) read and write the residual streams; fp32."""
    w_in: list                     # [streams]
    w_out: list                    # [streams]
    w_mix: list                    # [streams (from)][streams (to)]
    scale: list                    # [Wp] or None: layer scale
    shift: Optional[torch.Tensor]  # [Wp]: token shift of what the mixer reads


@dataclass
class ExpertStack:
    """Unquantised routed experts of one layer, padded to whole 64s."""
    router: torch.Tensor           # [E rounded up to 8][Wp]
    gate_up: torch.Tensor          # [E][2 * ffp][Wp], interleave16; without a gate [E][ffp][Wp]
    down: torch.Tensor             # [E][Wp][ffp]; runs of a shared expert's columns behind the routed ones


@dataclass
class LayerWeights:
    input_norm: torch.Tensor       # fp32 [hidden]
    post_norm: torch.Tensor        # fp32 [hidden]
    qkv: Optional[QLinear]         # None on gated delta-net layers
    o: Optional[QLinear]
    gate_up: Optional[QLinear] = None
    down: Optional[QLinear] = None
    router: Optional[torch.Tensor] = None          # bf16 [n_experts][hidden]
    experts: Optional[List[ExpertWeights]] = None
    shared: Optional[ExpertWeights] = None
    shared_gate: Optional[torch.Tensor] = None     # bf16 [1][hidden]
    # experts stacked for the grouped kernels: uint8 [E][nb][kg][4352]
    experts_gate_up_w4b: Optional[torch.Tensor] = None
    experts_down_w4b: Optional[torch.Tensor] = None
    gdn: Optional[GdnWeights] = None               # set instead of qkv / o on gated delta-net layers
    # listed layers: the norms then belong to the mixer's and the feed-forward's OUTPUT, or (``ModelConfig.block``) to what
    # they read: single numbers or a factor per column
    mixer: object = None                           # the weights of the mixer's kind
    moe: Optional[ExpertStack] = None
    dense: Optional[DenseWeights] = None
    streams: Optional[StreamWeights] = None
    behind: Optional[tuple] = None                 # norms behind the mixer and the feed-forward (``SandwichBlock``)


@dataclass
class MtpWeights:
    """Multi-token-prediction head: fc over [norm(embed) ‖ norm(hidden)] then decoder layers."""
    pre_norm_embed: torch.Tensor
    pre_norm_hidden: torch.Tensor
    fc: QLinear                    # [hidden][2*hidden]
    layers: List[LayerWeights]
    norm: torch.Tensor
    mask_token: Optional[int] = None    # a block drafter's "not drafted yet" token (default: the last vocabulary id)


@dataclass
class ModelWeights:
    cfg: ModelConfig
    embed: torch.Tensor            # bf16 [vocab][hidden]
    lm_head: torch.Tensor          # bf16 [vocab][hidden]
    final_norm: torch.Tensor       # fp32 [hidden]
    layers: List[LayerWeights]
    mtp: Optional[MtpWeights] = None
    lm_head_i8: Optional[tuple] = None    # (int8 [vocab][hidden], fp32 [vocab]) when the int8 head is on
    loop_step: Optional[torch.Tensor] = None    # fp32 [passes][Wp]: added before every pass of a looped range of layers

    def nbytes(self) -> int:
        tot = self.embed.numel() * 2 + self.lm_head.numel() * 2
        for lw in {id(x): x for x in self.layers + (self.mtp.layers if self.mtp else [])}.values():      # layers may share weights
            for ql in (lw.qkv, lw.o, lw.gate_up, lw.down):
                if ql is not None:
                    tot += ql.nbytes
            if lw.gdn is not None:
                tot += lw.gdn.in_proj.nbytes + lw.gdn.out_proj.nbytes
            if lw.experts_gate_up_w4b is not None:
                tot += lw.experts_gate_up_w4b.numel() + lw.experts_down_w4b.numel()
            if lw.shared is not None:
                tot += lw.shared.gate_up.nbytes + lw.shared.down.nbytes
            for part in (lw.mixer, lw.moe, lw.dense):
                if part is not None:
                    tot += part_nbytes(part)
        return tot


def part_nbytes(part) -> int:
    """Bytes of a container of tensors and containers."""
    def one(t):
        return t.numel() * t.element_size() if isinstance(t, torch.Tensor) else sum(map(one, t)) if isinstance(t, list) else part_nbytes(t)
    return sum(one(t) for t in vars(part).values() if t is not None)


def _norm_weight(h, device, gen=None):
    return torch.ones(h, dtype=torch.float32, device=device)


def _rand_layer(cfg: ModelConfig, device, seed: int, exact: bool, std=0.02, gdn: bool = False) -> LayerWeights:
    h = cfg.hidden
    g = torch.Generator(device="cpu")
    g.manual_seed(seed)

    def lin(n, k, sub):
        if exact:
            return QLinear.from_f32(torch.randn(n, k, generator=g) * std, device)
        return QLinear.random(n, k, device, seed * 131 + sub, std)

    def lin_gate_up(i, k, sub):
        if exact:
            gate = torch.randn(i, k, generator=g) * std
            up = torch.randn(i, k, generator=g) * std
            return QLinear.from_f32(interleave16(gate, up), device)
        return QLinear.random(2 * i, k, device, seed * 131 + sub, std)

    if gdn:
        nv = cfg.gdn_v_heads
        lw = LayerWeights(input_norm=_norm_weight(h, device), post_norm=_norm_weight(h, device), qkv=None, o=None)
        lw.gdn = GdnWeights(
            in_proj=lin(cfg.gdn_proj_dim, h, 1),
            conv_w=(torch.randn(cfg.gdn_conv_channels, 4, generator=g) * 0.5).to(device),
            a_log=torch.log(torch.rand(nv, generator=g) * 4.0 + 0.5).to(device),
            dt_bias=(torch.randn(nv, generator=g) * 0.5).to(device),
            norm_w=(1.0 + 0.1 * torch.randn(cfg.gdn_head_dim, generator=g)).to(device),
            out_proj=lin(h, cfg.gdn_value_dim, 2))
    else:
        lw = LayerWeights(
            input_norm=_norm_weight(h, device), post_norm=_norm_weight(h, device),
            qkv=lin(cfg.qkv_dim, h, 1), o=lin(h, cfg.q_dim, 2))
    if exact:
        # non-trivial norm weights so the norm kernels are actually exercised
        lw.input_norm = (1.0 + 0.1 * torch.randn(h, generator=g)).to(device)
        lw.post_norm = (1.0 + 0.1 * torch.randn(h, generator=g)).to(device)
    if cfg.is_moe:
        lw.router = (torch.randn(cfg.n_experts, h, generator=g) * (1.0 / h ** 0.5)).to(torch.bfloat16).to(device) \
            if exact else (torch.randn(cfg.n_experts, h, device=device) * (1.0 / h ** 0.5)).to(torch.bfloat16)
        if exact:
            lw.experts = [ExpertWeights(lin_gate_up(cfg.expert_ffn, h, 10 + 2 * e), lin(h, cfg.expert_ffn, 11 + 2 * e))
                          for e in range(cfg.n_experts)]
            lw.experts_gate_up_w4b = torch.stack([e.gate_up.w4b for e in lw.experts]).contiguous()
            lw.experts_down_w4b = torch.stack([e.down.w4b for e in lw.experts]).contiguous()
        else:
            e = cfg.n_experts
            gu = Q.random_w4b(e * 2 * cfg.expert_ffn, h, device, seed * 131 + 7, std)
            dn = Q.random_w4b(e * h, cfg.expert_ffn, device, seed * 131 + 8, std)
            lw.experts_gate_up_w4b = gu.reshape(e, 2 * cfg.expert_ffn // 128, h // 64, Q.BLOCK_BYTES)
            lw.experts_down_w4b = dn.reshape(e, h // 128, cfg.expert_ffn // 64, Q.BLOCK_BYTES)
        if cfg.shared_ffn:
            lw.shared = ExpertWeights(lin_gate_up(cfg.shared_ffn, h, 3), lin(h, cfg.shared_ffn, 4))
            lw.shared_gate = (torch.randn(1, h, generator=g) * (1.0 / h ** 0.5)).to(torch.bfloat16).to(device)
    else:
        lw.gate_up = lin_gate_up(cfg.ffn, h, 5)
        lw.down = lin(h, cfg.ffn, 6)
    return lw


def random_weights(cfg: ModelConfig, device="cpu", seed: int = 0, exact: Optional[bool] = None,
                   std: float = 0.02, head_rows: Optional[int] = None) -> ModelWeights:
    """Random-init model. ``exact`` (default: on for < 100M parameters) quantises real fp32 matrices.
    ``head_rows``: rows of the lm_head this rank holds (vocabulary-parallel head)."""
    if exact is None:
        exact = cfg.param_count() < 100_000_000
    if cfg.layer_specs:
        from .listed import random_listed_weights
        return random_listed_weights(cfg, device, seed, std)
    h = cfg.hidden
    hr = cfg.vocab if head_rows is None else head_rows
    if exact:
        g = torch.Generator(device="cpu")
        g.manual_seed(seed)
        embed = (torch.randn(cfg.vocab, h, generator=g) * std).to(torch.bfloat16).to(device)
        head = (torch.randn(cfg.vocab, h, generator=g) * std)[:hr].to(torch.bfloat16).to(device).contiguous()
    else:
        embed = torch.empty(cfg.vocab, h, dtype=torch.bfloat16, device=device).normal_(0, std)
        head = torch.empty(hr, h, dtype=torch.bfloat16, device=device).normal_(0, std)
    layers = [_rand_layer(cfg, device, seed * 1000 + 1 + i, exact, std, gdn=cfg.is_gdn_layer(i)) for i in range(cfg.n_layers)]
    mw = ModelWeights(cfg, embed, head, _norm_weight(h, device), layers)
    if cfg.mtp_layers:
        dense_cfg = cfg
        if exact:
            g2 = torch.Generator(device="cpu")
            g2.manual_seed(seed * 1000 + 777)
            fc = QLinear.from_f32(torch.randn(h, 2 * h, generator=g2) * std, device)
        else:
            fc = QLinear.random(h, 2 * h, device, seed * 1000 + 777, std)
        mw.mtp = MtpWeights(_norm_weight(h, device), _norm_weight(h, device), fc,
                            [_rand_layer(dense_cfg, device, seed * 1000 + 800 + i, exact, std)
                             for i in range(cfg.mtp_layers)], _norm_weight(h, device))
    return mw
