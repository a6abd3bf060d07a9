"""Architecture descriptions: parsed from a HF ``config.json`` or built from presets.

Six families are served.  Two are the ones the reference runs: dense Llama-style decoders and
Qwen3.5-style hybrids that interleave Gated-DeltaNet layers with gated full attention
(reference: README.md model list; parameter names checked against the HF
implementation, transformers/models/qwen3_5/modeling_qwen3_5.py).  The others spell every layer out in config.json.
Pasizen: latent attention without positions, a short convolution in front of every mixer, hyper-connected residual
streams, PolyNorm or mixture-of-experts feed-forwards and layers that may be looped.  Makodra: generalized delta rule,
token-shifted decaying memory and chunked attention in any order, with norms on the sublayers' outputs.  Funevik: matrix
memories with exponential gates, windowed latent attention with a rotated part and soft-capped attention behind a short
convolution in any order, mixer and feed-forward side by side in every layer.  Padadra: a delta rule with a decay per
channel, and windowed attention with a forget-gated memory side by side behind norms of their own; mixer and feed-forward
again on the same input, and an embedding of token pairs.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple, Union


UNLIMITED_POSITIONS = 1 << 20             # positions of architectures that compute them instead of looking them up


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions on the first ``dims`` entries of a head, neighbours paired: pair i turns by position / base^(2i / dims),
    long waves slowed down by ``scaling`` (factor, low, high, original length)."""
    dims: int
    base: float
    scaling: Optional[Tuple[float, float, float, float]] = None

    def scaling_dict(self) -> Optional[Dict[str, Any]]:
        """The scaling in the form of a HF ``rope_scaling`` entry."""
        if self.scaling is None:
            return None
        return dict(zip(("factor", "low_freq_factor", "high_freq_factor", "original_max_position_embeddings"), self.scaling), rope_type="llama3")


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention over a cached latent: ``kv_rank`` values per token, keys and values of all heads expanded from them."""
    heads: int
    dim: int                             # query / key size per head (without the rotated part)
    vdim: int                            # value size per head
    kv_rank: int
    scale: float
    q_rank: int = 0                      # queries go through a normed latent of this size (0: straight from the input)
    rot: Optional[RotarySpec] = None     # a rotated part of ``rot.dims`` more query entries; its key is shared by all heads
    window: int = 0                      # tokens a query sees, itself included (0: all before it)
    sink: bool = False                   # one learned logit per head in the softmax sum, without a value


@dataclass(frozen=True)
class GroupedAttentionSpec:
    """Causal grouped-query attention behind a short convolution of queries, keys and values, with rotary positions: soft-capped
    scores, a sink of score 0 and a sigmoid gate per head (Funevik), or a window, learned sinks, biased projections, queries and
    keys normed over all heads at once, and values that turn with their position and back at the reader's (Padadra)."""
    heads: int
    kv_heads: int
    dim: int                             # query / key size per head
    vdim: int                            # value size per head
    scale: float
    conv: int                            # taps
    rot: RotarySpec
    softcap: float = 0.0                 # 0: scores as they are
    gate: bool = True                    # sigmoid gate per head
    window: int = 0                      # tokens a query sees, itself included (0: all before it)
    learned_sink: bool = False           # one learned sink logit per head instead of 0
    bias: bool = False                   # of the three projections
    row_norm: bool = False               # root-mean-square norm of all queries (all keys) of a token together
    turn_values: Optional[RotarySpec] = None     # rotation of the values


@dataclass(frozen=True)
class ChunkAttentionSpec:
    """Grouped-query attention inside chunks of ``chunk`` positions: unit-rms queries and keys, a logarithmic distance
    bias per head, a sink of score 0, optional mixing with the first such layer's values, a sigmoid output gate."""
    heads: int
    kv_heads: int
    dim: int                             # query / key size per head
    vdim: int                            # value size per head
    scale: float
    chunk: int
    v_mix: bool = False


@dataclass(frozen=True)
class RecurrentSpec:
    """A memory matrix [dim, vdim] per head: "general_delta" (diagonal decay plus a rank-one removal), "wkv" (diagonal
    decay, bonus for the current token, token-shifted inputs), "mlstm" (one decay per head and token, exponential input gate,
    read-out divided by a normaliser), "channel_delta" (decay per channel, then a delta rule with unit keys behind a short
    convolution) or "hgrn2" (the forget gate of a channel is also what it writes)."""
    kind: str
    heads: int
    dim: int
    vdim: int = 0                        # 0: as many as ``dim``
    gate_cap: float = 0.0                # "mlstm": gate logits are soft-capped at this
    kv_heads: int = 0                    # "channel_delta": query and key heads, each shared by heads / kv_heads heads
    conv: int = 1                        # "channel_delta": taps

    @property
    def values(self) -> int:
        return self.vdim or self.dim


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers on the same input; half the sum of their outputs, each behind a norm of its own."""
    left: GroupedAttentionSpec
    right: RecurrentSpec

    @property
    def heads(self) -> int:
        return self.left.heads

    @property
    def kv_heads(self) -> int:
        return self.left.kv_heads

    @property
    def dim(self) -> int:
        return self.left.dim


@dataclass(frozen=True)
class GluSpec:
    """Gated unit; with a ``limit`` its inputs are clamped."""
    ff: int
    limit: float = math.inf


@dataclass(frozen=True)
class RouterSpec:
    """Softmax router: the ``top`` best experts among those of the ``keep`` best of ``groups`` equal groups."""
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    bias: bool = False                   # logits have a bias


@dataclass(frozen=True)
class FeedForwardSpec:
    kind: str                            # "dense" (PolyNorm) | "moe" | "swiglu" | "geglu" (tanh form of gelu) | "relu2" (two matrices)
    ff: int = 0
    expert: Optional[GluSpec] = None
    router: Optional[RouterSpec] = None
    shared: Optional[GluSpec] = None
    shared_gate: bool = False            # the shared expert is multiplied by a sigmoid gate per token


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[LatentAttentionSpec, ChunkAttentionSpec, GroupedAttentionSpec, RecurrentSpec, ParallelSpec]
    mlp: Optional[FeedForwardSpec]


@dataclass
class ModelConfig:
    arch: str = "llama"                  # "llama" | "hybrid_gdn" | "pasizen" | "makodra" | "funevik" | "padadra"
    vocab_size: int = 32000
    hidden_size: int = 4096
    n_layers: int = 32
    n_heads: int = 32
    n_kv_heads: int = 8
    head_dim: int = 128
    ffn_size: int = 14336
    rms_eps: float = 1e-5
    rope_theta: float = 10000.0
    rope_scaling: Optional[Dict[str, Any]] = None
    max_position: int = 8192
    tie_embeddings: bool = False
    logit_softcap: float = 0.0
    eos_token_ids: List[int] = field(default_factory=list)
    # ---- hybrid (Gated DeltaNet) -------------------------------------------
    layer_types: Optional[List[str]] = None       # "linear_attention" | "full_attention"
    gdn_n_k_heads: int = 16
    gdn_n_v_heads: int = 16
    gdn_head_k_dim: int = 128
    gdn_head_v_dim: int = 128
    gdn_conv_width: int = 4
    partial_rotary: float = 1.0
    attn_output_gate: bool = False
    qk_norm: bool = False
    norm_plus_one: bool = False                    # RMSNorm weight stored as (w - 1)
    # ---- layer-by-layer description (Pasizen, Makodra, Funevik, Padadra) -----
    layers: Optional[List[LayerSpec]] = None
    loop: Optional[tuple] = None                   # (start, stop, times): these layers run ``times`` times in a row
    streams: int = 1                               # hyper-connected copies of the residual stream
    conv_taps: int = 1                             # short causal convolution in front of every mixer
    embed_scale: float = 1.0                       # embedding rows are multiplied by this
    bigram: Optional[Tuple[int, int, int]] = None  # embedding of token pairs: buckets, multipliers of the token before and of the token
    residual_mult: float = 1.0                     # every layer's outputs are multiplied by this
    name: str = ""

    # ---- derived -------------------------------------------------------------
    @property
    def q_size(self) -> int:
        return self.n_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.n_kv_heads * self.head_dim

    @property
    def rotary_dim(self) -> int:
        return int(self.head_dim * self.partial_rotary)

    def layer_type(self, i: int) -> str:
        if self.layer_types is None:
            return "full_attention"
        return self.layer_types[i]

    @property
    def layer_runs(self) -> List[int]:
        """Layer index of every layer run, in execution order (a looped layer appears once per pass; every pass owns
        its own cache and state)."""
        n = list(range(self.n_layers))
        if not self.loop:
            return n
        a, b, times = self.loop
        return n[:a] + n[a:b] * times + n[b:]

    @property
    def attn_layers(self) -> List[int]:
        return [i for i in range(self.n_layers) if self.layer_type(i) == "full_attention"]

    @property
    def gdn_layers(self) -> List[int]:
        return [i for i in range(self.n_layers) if self.layer_type(i) == "linear_attention"]

    @property
    def gdn_conv_dim(self) -> int:
        return 2 * self.gdn_n_k_heads * self.gdn_head_k_dim + self.gdn_n_v_heads * self.gdn_head_v_dim

    def param_count(self) -> int:
        d, f = self.hidden_size, self.ffn_size
        if self.arch == "pasizen":
            return self._layered_param_count()
        if self.arch == "makodra":
            return self._makodra_param_count()
        if self.arch == "funevik":
            return self._funevik_param_count()
        if self.arch == "padadra":
            return self._padadra_param_count()
        n = self.vocab_size * d * (1 if self.tie_embeddings else 2) + d
        for i in range(self.n_layers):
            n += 3 * d * f + 2 * d
            if self.layer_type(i) == "full_attention":
                qmul = 2 if self.attn_output_gate else 1
                n += d * (self.q_size * qmul + 2 * self.kv_size) + self.q_size * d
            else:
                kd = self.gdn_n_k_heads * self.gdn_head_k_dim
                vd = self.gdn_n_v_heads * self.gdn_head_v_dim
                n += d * (2 * kd + vd) + d * vd + 2 * d * self.gdn_n_v_heads + vd * d
        return n

    def _layered_param_count(self) -> int:
        d, s = self.hidden_size, self.streams
        n = 2 * self.vocab_size * d + self.max_position * d + d
        glu = lambda g: 3 * g.ff * d
        for L in self.layers:
            m = L.mixer
            n += d * (m.heads * (m.dim + m.vdim) + m.kv_rank) + m.kv_rank * (m.heads * (m.dim + m.vdim) + 1)
            n += d * (1 + self.conv_taps) + 2 * s + s * s
            if L.mlp is None:
                continue
            n += d + 2 * s + s * s
            if L.mlp.kind == "dense":
                n += 2 * d * L.mlp.ff + 4
            else:
                n += L.mlp.router.experts * (d + glu(L.mlp.expert)) + (glu(L.mlp.shared) if L.mlp.shared else 0)
        return n

    def _makodra_param_count(self) -> int:
        d, n = self.hidden_size, self.vocab_size * self.hidden_size + self.hidden_size
        for L in self.layers:
            m = L.mixer
            n += d * (1 if L.mlp is None else 2 + 3 * L.mlp.ff)
            if isinstance(m, ChunkAttentionSpec):
                n += d * (m.heads * (m.dim + 2 * m.vdim) + m.kv_heads * (m.dim + m.vdim)) + 2 * m.heads + m.v_mix
            else:                        # without the low-rank decay maps, whose rank only the weights tell
                delta = m.kind == "general_delta"
                n += m.heads * m.dim * ((6 if delta else 5) * d + 3) + (0 if delta else 5 * d)
        return n

    def _funevik_param_count(self) -> int:
        d, n = self.hidden_size, 2 * self.vocab_size * self.hidden_size + self.hidden_size
        for L in self.layers:
            m, f = L.mixer, L.mlp
            n += 2 * d
            if isinstance(m, LatentAttentionSpec):
                r, H = m.rot.dims, m.heads
                n += m.q_rank * (d + 1 + H * (m.dim + r)) + d * (m.kv_rank + r) + m.kv_rank * (1 + H * (m.dim + m.vdim)) + H * (1 + m.vdim * d)
            elif isinstance(m, GroupedAttentionSpec):
                rows = m.heads * m.dim + m.kv_heads * (m.dim + m.vdim)
                n += rows * (d + m.conv) + m.heads * d * (1 + m.vdim)
            else:
                n += m.heads * (d * (2 * m.dim + 3 * m.values + 2) + m.values + 2)
            if f is None:
                continue
            n += 2 * d
            if f.kind == "moe":
                n += f.router.experts * (d + 1 + 3 * d * f.expert.ff) + (d + 3 * d * f.shared.ff if f.shared else 0)
            else:
                n += 3 * d * f.ff
        return n

    def _padadra_param_count(self) -> int:
        d, n = self.hidden_size, 2 * self.vocab_size * self.hidden_size + 1
        n += (self.bigram[0] + 1) * d if self.bigram else 0
        for L in self.layers:
            m, f = L.mixer, L.mlp
            n += 1 + (0 if f is None else 1 + 2 * d * f.ff)
            if isinstance(m, ParallelSpec):
                a, b = m.left, m.right
                qk, v = (a.heads + a.kv_heads) * a.dim, a.kv_heads * a.vdim
                n += (qk + v) * (d + 1 + a.conv) + qk + a.heads * (1 + a.vdim * d) + 2 * d
                n += b.heads * (b.dim * (2 * d + 2) + 2 * b.values * d) + b.values
            else:                            # without the low-rank maps of decay and gate, whose ranks only the weights tell
                qk, v = 2 * m.kv_heads * m.dim, m.heads * m.values
                n += (qk + v) * (d + m.conv) + m.heads * (d + 1 + m.dim) + m.values + v * d
        return n

    # ---- construction ----------------------------------------------------------
    @classmethod
    def from_padadra_dict(cls, c: Dict[str, Any]) -> "ModelConfig":
        """config.json of a Padadra model: every layer with its mixer and feed-forward."""
        layers = []
        for i, e in enumerate(c["layers"]):
            m, f, mlp = e["mixer"], e.get("mlp"), None
            if e["type"] == "channel_delta":
                mixer = RecurrentSpec("channel_delta", int(m["heads"]), int(m["dim"]), int(m["vdim"]), kv_heads=int(m["kv_heads"]), conv=int(m["conv"]))
                if mixer.kv_heads < 1 or mixer.heads % mixer.kv_heads or mixer.conv < 1:
                    raise ValueError(f"layer {i}: inconsistent delta rule {mixer}")
            elif e["type"] == "parallel":
                a, b = m["left"], m["right"]
                s = a["rot"].get("scaling")
                scaling = tuple(float(s[k]) for k in ("factor", "low", "high", "original")) if s else None
                rot = RotarySpec(int(a["rot"]["dims"]), float(a["rot"]["base"]), scaling)
                left = GroupedAttentionSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]), int(a["conv"]),
                                            rot, gate=False, window=int(a["mask"]["size"]), learned_sink=True, bias=True, row_norm=True,
                                            turn_values=RotarySpec(int(a["vdim"]), rot.base))
                if left.kv_heads < 1 or left.heads % left.kv_heads or rot.dims > left.dim or rot.dims % 2 or left.vdim % 2 or left.conv < 1 or \
                        left.window < 1:
                    raise ValueError(f"layer {i}: inconsistent attention {left}")
                mixer = ParallelSpec(left, RecurrentSpec("hgrn2", int(b["heads"]), int(b["dim"]), int(b["vdim"])))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            if f is not None and f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            layers.append(LayerSpec(mixer, None if f is None else FeedForwardSpec("relu2", ff=int(f["ff"]))))
        eos, g, m0 = c.get("eos_token_id"), c["embedding"].get("bigram"), layers[0].mixer
        if g and (int(g["buckets"]) < 1 or int(g["mul_prev"]) < 0 or int(g["mul_cur"]) < 0):
            raise ValueError(f"inconsistent pair embedding {g}")
        return cls(arch="padadra", vocab_size=int(c["vocab"]), hidden_size=int(c["width"]), n_layers=len(layers), n_heads=m0.heads,
                   n_kv_heads=m0.kv_heads, head_dim=m0.dim, ffn_size=0, rms_eps=float(c["norm"]["eps"]), max_position=UNLIMITED_POSITIONS,
                   layers=layers, embed_scale=float(c["embedding"]["scale"]), residual_mult=float(c["residual_mult"]),
                   bigram=(int(g["buckets"]), int(g["mul_prev"]), int(g["mul_cur"])) if g else None,
                   eos_token_ids=[] if eos is None else ([eos] if isinstance(eos, int) else list(eos)))

    @classmethod
    def from_funevik_dict(cls, c: Dict[str, Any]) -> "ModelConfig":
        """config.json of a Funevik model: every layer with its mixer and feed-forward."""
        layers = []
        for i, e in enumerate(c["layers"]):
            m, f, mlp = e["mixer"], e.get("mlp"), None
            rot = RotarySpec(int(m["rot"]["dims"]), float(m["rot"]["base"])) if "rot" in m else None
            if e["type"] == "mlstm":
                mixer = RecurrentSpec("mlstm", int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))
            elif e["type"] == "latent_attention":
                mixer = LatentAttentionSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]),
                                            int(m["q_rank"]), rot, int(m["mask"]["size"]), True)
                if rot is None or rot.dims != int(m["rot_dim"]) or mixer.window < 1:
                    raise ValueError(f"layer {i}: inconsistent latent attention {mixer}")
            elif e["type"] == "attention":
                mixer = GroupedAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                             int(m["conv"]), rot, float(m["softcap"]))
                if mixer.heads % mixer.kv_heads or rot is None or rot.dims > mixer.dim or mixer.conv < 1 or mixer.softcap <= 0.0:
                    raise ValueError(f"layer {i}: inconsistent attention {mixer}")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            if rot is not None and rot.dims % 2:
                raise ValueError(f"layer {i}: rotary positions pair entries, {rot.dims} is odd")
            if f is not None and f["kind"] == "dense":
                mlp = FeedForwardSpec("geglu", ff=int(f["ff"]))
            elif f is not None and f["kind"] == "moe":
                router = RouterSpec(int(f["router"]["experts"]), int(f["router"]["top"]), bias=True)
                if not 1 <= router.top <= router.experts:
                    raise ValueError(f"layer {i}: inconsistent router {router}")
                shared = GluSpec(int(f["shared"]["ff"])) if f.get("shared") else None
                mlp = FeedForwardSpec("moe", expert=GluSpec(int(f["expert"]["ff"])), router=router, shared=shared, shared_gate=shared is not None)
            elif f is not None:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            layers.append(LayerSpec(mixer, mlp))
        eos = c.get("eos_token_id")
        m0 = layers[0].mixer
        return cls(arch="funevik", vocab_size=int(c["vocab"]), hidden_size=int(c["width"]), n_layers=len(layers), n_heads=m0.heads,
                   n_kv_heads=getattr(m0, "kv_heads", m0.heads), head_dim=m0.dim, ffn_size=0, rms_eps=float(c["norm"]["eps"]),
                   max_position=UNLIMITED_POSITIONS, layers=layers, embed_scale=float(c["embedding"]["scale"]),
                   eos_token_ids=[] if eos is None else ([eos] if isinstance(eos, int) else list(eos)))

    @classmethod
    def from_makodra_dict(cls, c: Dict[str, Any]) -> "ModelConfig":
        """config.json of a Makodra model: every layer with its mixer and feed-forward."""
        layers = []
        for i, e in enumerate(c["layers"]):
            m, f = e["mixer"], e.get("mlp")
            if e["type"] == "attention":
                mixer = ChunkAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                           int(m["mask"]["size"]), bool(m.get("v_mix", False)))
                if mixer.heads % mixer.kv_heads or mixer.chunk < 1:
                    raise ValueError(f"layer {i}: inconsistent attention {mixer}")
            elif e["type"] in ("general_delta", "wkv"):
                mixer = RecurrentSpec(e["type"], int(m["heads"]), int(m["dim"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            if f is not None and f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            layers.append(LayerSpec(mixer, None if f is None else FeedForwardSpec("swiglu", ff=int(f["ff"]))))
        mixing = {(L.mixer.kv_heads, L.mixer.vdim) for L in layers if isinstance(L.mixer, ChunkAttentionSpec) and L.mixer.v_mix}
        if len(mixing) > 1:
            raise ValueError(f"layers that mix values need values of one shape, not {sorted(mixing)}")
        eos = c.get("eos_token_id")
        m0 = layers[0].mixer
        return cls(arch="makodra", vocab_size=int(c["vocab"]), hidden_size=int(c["width"]), n_layers=len(layers), n_heads=m0.heads,
                   n_kv_heads=getattr(m0, "kv_heads", m0.heads), head_dim=m0.dim, ffn_size=0, rms_eps=float(c["norm"]["eps"]),
                   max_position=UNLIMITED_POSITIONS, tie_embeddings=True, logit_softcap=float(c.get("logit_softcap") or 0.0),
                   layers=layers, eos_token_ids=[] if eos is None else ([eos] if isinstance(eos, int) else list(eos)))

    @classmethod
    def from_layered_dict(cls, c: Dict[str, Any]) -> "ModelConfig":
        """config.json of a Pasizen model: every layer with its mixer and feed-forward, the loop, the stream count."""
        layers = []
        for i, e in enumerate(c["layers"]):
            if e["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            m = e["mixer"]
            mixer = LatentAttentionSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]))
            f, mlp = e.get("mlp"), None
            glu = lambda g: GluSpec(int(g["ff"]), float(g["limit"]))
            if f is not None and f["kind"] == "dense":
                mlp = FeedForwardSpec("dense", ff=int(f["ff"]))
            elif f is not None and f["kind"] == "moe":
                r, g = f["router"], f["router"].get("groups") or {"count": 1, "keep": 1}
                router = RouterSpec(int(r["experts"]), int(r["top"]), int(g["count"]), int(g["keep"]))
                if router.experts % router.groups or not 1 <= router.keep <= router.groups or \
                        not 1 <= router.top <= router.keep * (router.experts // router.groups):
                    raise ValueError(f"layer {i}: inconsistent router {router}")
                mlp = FeedForwardSpec("moe", expert=glu(f["expert"]), router=router,
                                      shared=glu(f["shared"]) if f.get("shared") else None)
            elif f is not None:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            layers.append(LayerSpec(mixer, mlp))
        lp = c.get("loop")
        loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None
        if loop and not (0 <= loop[0] <= loop[1] <= len(layers) and loop[2] >= 1):
            raise ValueError(f"inconsistent loop {lp}")
        eos = c.get("eos_token_id")
        m0 = layers[0].mixer
        return cls(arch="pasizen", vocab_size=int(c["vocab"]), hidden_size=int(c["width"]), n_layers=len(layers),
                   n_heads=m0.heads, n_kv_heads=1, head_dim=m0.kv_rank, ffn_size=0, rms_eps=float(c["norm"]["eps"]),
                   max_position=int(c["max_positions"]), layers=layers, loop=loop, streams=int(c["streams"]),
                   conv_taps=int(c["canon"]["taps"]),
                   eos_token_ids=[] if eos is None else ([eos] if isinstance(eos, int) else list(eos)))

    @classmethod
    def from_hf_dict(cls, c: Dict[str, Any]) -> "ModelConfig":
        if "text_config" in c and isinstance(c["text_config"], dict):
            merged = dict(c["text_config"])
            merged.setdefault("architectures", c.get("architectures"))
            c = merged
        if c.get("architecture") == "Pasizen":
            return cls.from_layered_dict(c)
        if c.get("architecture") == "Makodra":
            return cls.from_makodra_dict(c)
        if c.get("architecture") == "Funevik":
            return cls.from_funevik_dict(c)
        if c.get("architecture") == "Padadra":
            return cls.from_padadra_dict(c)
        archs = c.get("architectures") or []
        mt = (c.get("model_type") or "").lower()
        is_hybrid = "layer_types" in c and any(t == "linear_attention" for t in c["layer_types"])
        is_hybrid = is_hybrid or "qwen3_5" in mt or "qwen3_next" in mt or any("Qwen3_5" in a or "Qwen3Next" in a for a in archs)
        n_heads = c["num_attention_heads"]
        head_dim = c.get("head_dim") or c["hidden_size"] // n_heads
        eos = c.get("eos_token_id")
        eos_ids = [] if eos is None else ([eos] if isinstance(eos, int) else list(eos))
        rope_params = c.get("rope_parameters") or {}
        rope_theta = c.get("rope_theta", rope_params.get("rope_theta", 10000.0))
        rope_scaling = c.get("rope_scaling")
        if rope_scaling is None and rope_params.get("rope_type", "default") not in ("default", None):
            rope_scaling = rope_params
        cfg = cls(
            arch="hybrid_gdn" if is_hybrid else "llama",
            vocab_size=c["vocab_size"], hidden_size=c["hidden_size"], n_layers=c["num_hidden_layers"],
            n_heads=n_heads, n_kv_heads=c.get("num_key_value_heads", n_heads), head_dim=head_dim,
            ffn_size=c["intermediate_size"], rms_eps=c.get("rms_norm_eps", 1e-5), rope_theta=rope_theta,
            rope_scaling=rope_scaling, max_position=c.get("max_position_embeddings", 8192),
            tie_embeddings=bool(c.get("tie_word_embeddings", False)),
            logit_softcap=float(c.get("final_logit_softcapping") or 0.0), eos_token_ids=eos_ids,
            name=c.get("_name_or_path", ""))
        if is_hybrid:
            lt = c.get("layer_types")
            if lt is None:
                interval = c.get("full_attention_interval", 4)
                lt = ["full_attention" if (i + 1) % interval == 0 else "linear_attention"
                      for i in range(cfg.n_layers)]
            cfg.layer_types = list(lt)
            cfg.gdn_n_k_heads = c.get("linear_num_key_heads", 16)
            cfg.gdn_n_v_heads = c.get("linear_num_value_heads", 16)
            cfg.gdn_head_k_dim = c.get("linear_key_head_dim", 128)
            cfg.gdn_head_v_dim = c.get("linear_value_head_dim", 128)
            cfg.gdn_conv_width = c.get("linear_conv_kernel_dim", 4)
            cfg.partial_rotary = float(c.get("partial_rotary_factor", rope_params.get("partial_rotary_factor", 0.25)))
            cfg.attn_output_gate = bool(c.get("attn_output_gate", True))
            cfg.qk_norm = True
            cfg.norm_plus_one = True
        return cfg

    @classmethod
    def from_pretrained(cls, path: str) -> "ModelConfig":
        with open(os.path.join(path, "config.json")) as f:
            cfg = cls.from_hf_dict(json.load(f))
        gen = os.path.join(path, "generation_config.json")
        if os.path.exists(gen):
            with open(gen) as f:
                g = json.load(f)
            eos = g.get("eos_token_id")
            if eos is not None:
                ids = [eos] if isinstance(eos, int) else list(eos)
                cfg.eos_token_ids = sorted(set(cfg.eos_token_ids) | set(ids))
        cfg.name = cfg.name or os.path.basename(os.path.normpath(path))
        return cfg


_LLAMA3_SCALING = {"rope_type": "llama3", "factor": 8.0, "low_freq_factor": 1.0,
                   "high_freq_factor": 4.0, "original_max_position_embeddings": 8192}


def preset(name: str) -> ModelConfig:
    """Random-init architectures named by the benchmark configs."""
    n = name.lower()
    if n in ("llama-3.1-8b", "llama8b", "8b"):
        return ModelConfig(arch="llama", vocab_size=128256, hidden_size=4096, n_layers=32, n_heads=32,
                           n_kv_heads=8, head_dim=128, ffn_size=14336, rope_theta=500000.0,
                           rope_scaling=dict(_LLAMA3_SCALING), max_position=131072, name="llama-3.1-8b")
    if n in ("llama-3.2-1b", "llama1b", "1b"):
        sc = dict(_LLAMA3_SCALING, factor=32.0)
        return ModelConfig(arch="llama", vocab_size=128256, hidden_size=2048, n_layers=16, n_heads=32,
                           n_kv_heads=8, head_dim=64, ffn_size=8192, rope_theta=500000.0, rope_scaling=sc,
                           max_position=131072, tie_embeddings=True, name="llama-3.2-1b")
    if n in ("llama-3.1-70b", "70b"):
        return ModelConfig(arch="llama", vocab_size=128256, hidden_size=8192, n_layers=80, n_heads=64,
                           n_kv_heads=8, head_dim=128, ffn_size=28672, rope_theta=500000.0,
                           rope_scaling=dict(_LLAMA3_SCALING), max_position=131072, name="llama-3.1-70b")
    if n in ("tiny-target", "tiny"):
        return ModelConfig(arch="llama", vocab_size=4096, hidden_size=256, n_layers=4, n_heads=4, n_kv_heads=2,
                           head_dim=64, ffn_size=688, rope_theta=10000.0, max_position=2048, name="tiny-target")
    if n in ("tiny-draft",):
        return ModelConfig(arch="llama", vocab_size=4096, hidden_size=128, n_layers=1, n_heads=2, n_kv_heads=1,
                           head_dim=64, ffn_size=344, rope_theta=10000.0, max_position=2048, name="tiny-draft")
    if n in ("hybrid-gdn-target", "qwen3.5-hybrid"):
        lt = ["full_attention" if (i + 1) % 4 == 0 else "linear_attention" for i in range(48)]
        return ModelConfig(arch="hybrid_gdn", vocab_size=151936, hidden_size=2048, n_layers=48, n_heads=16,
                           n_kv_heads=2, head_dim=256, ffn_size=6144, rope_theta=10000000.0, max_position=32768,
                           layer_types=lt, gdn_n_k_heads=16, gdn_n_v_heads=16, gdn_head_k_dim=128,
                           gdn_head_v_dim=128, gdn_conv_width=4, partial_rotary=0.25, attn_output_gate=True,
                           qk_norm=True, norm_plus_one=True, rms_eps=1e-6, name="hybrid-gdn-target")
    if n in ("hybrid-gdn-draft", "dense-draft-1024"):
        return ModelConfig(arch="llama", vocab_size=151936, hidden_size=1024, n_layers=12, n_heads=16,
                           n_kv_heads=8, head_dim=64, ffn_size=3072, rope_theta=1000000.0, max_position=32768,
                           tie_embeddings=True, rms_eps=1e-6, name="hybrid-gdn-draft")
    if n in ("tiny-hybrid",):
        lt = ["linear_attention", "linear_attention", "linear_attention", "full_attention"]
        return ModelConfig(arch="hybrid_gdn", vocab_size=4096, hidden_size=128, n_layers=4, n_heads=4,
                           n_kv_heads=2, head_dim=64, ffn_size=256, rope_theta=10000.0, max_position=2048,
                           layer_types=lt, gdn_n_k_heads=2, gdn_n_v_heads=4, gdn_head_k_dim=32,
                           gdn_head_v_dim=32, gdn_conv_width=4, partial_rotary=0.25, attn_output_gate=True,
                           qk_norm=True, norm_plus_one=True, rms_eps=1e-6, name="tiny-hybrid")
    if n in ("pasizen-2048", "pasizen-1024"):
        # random-init stand-ins with the layer sizes of a real small model, dense and expert layers alternating
        d, H, ff = (2048, 16, 6144) if n.endswith("2048") else (1024, 8, 3072)
        mixer = LatentAttentionSpec(heads=H, dim=128, vdim=128, kv_rank=256, scale=128 ** -0.5)
        dense = LayerSpec(mixer, FeedForwardSpec("dense", ff=ff))
        moe = LayerSpec(mixer, FeedForwardSpec("moe", expert=GluSpec(ff // 8, 7.0), router=RouterSpec(32, 4, 8, 4),
                                               shared=GluSpec(ff // 4, 7.0)))
        return ModelConfig(arch="pasizen", vocab_size=65536, hidden_size=d, n_layers=16, n_heads=H, n_kv_heads=1,
                           head_dim=256, ffn_size=0, rms_eps=1e-6, max_position=16384, layers=[dense, moe] * 8,
                           streams=4, conv_taps=4, name=n)
    if n in ("tiny-pasizen",):
        mixer = LatentAttentionSpec(heads=3, dim=40, vdim=24, kv_rank=48, scale=0.2)
        dense = LayerSpec(mixer, FeedForwardSpec("dense", ff=200))
        moe = LayerSpec(LatentAttentionSpec(2, 32, 56, 72, 0.15),
                        FeedForwardSpec("moe", expert=GluSpec(40, 1.0), router=RouterSpec(8, 2, 4, 2), shared=GluSpec(72, 1.5)))
        return ModelConfig(arch="pasizen", vocab_size=4096, hidden_size=136, n_layers=3, n_heads=3, n_kv_heads=1,
                           head_dim=48, ffn_size=0, rms_eps=1e-6, max_position=2048, layers=[dense, moe, dense],
                           loop=(1, 3, 2), streams=2, conv_taps=3, name="tiny-pasizen")
    if n in ("makodra-2048", "makodra-1024"):
        # random-init stand-ins with the layer sizes of a real small model: two recurrent layers to one attention layer
        d, ff = (2048, 5632) if n.endswith("2048") else (1024, 2816)
        H, mlp = d // 64, FeedForwardSpec("swiglu", ff=ff)
        trio = [LayerSpec(RecurrentSpec("general_delta", H, 64), mlp), LayerSpec(RecurrentSpec("wkv", H, 64), mlp),
                LayerSpec(ChunkAttentionSpec(d // 128, d // 512, 128, 128, 11.3, 1024, True), mlp)]
        return ModelConfig(arch="makodra", vocab_size=65536, hidden_size=d, n_layers=15, n_heads=H, n_kv_heads=H, head_dim=64,
                           ffn_size=0, rms_eps=1e-6, max_position=UNLIMITED_POSITIONS, tie_embeddings=True, logit_softcap=30.0,
                           layers=trio * 5, name=n)
    if n in ("tiny-makodra",):
        mlp = FeedForwardSpec("swiglu", ff=200)
        return ModelConfig(arch="makodra", vocab_size=4096, hidden_size=136, n_layers=4, n_heads=3, n_kv_heads=3, head_dim=40,
                           ffn_size=0, rms_eps=1e-6, max_position=UNLIMITED_POSITIONS, tie_embeddings=True, logit_softcap=20.0,
                           layers=[LayerSpec(RecurrentSpec("wkv", 3, 40), mlp), LayerSpec(ChunkAttentionSpec(4, 2, 24, 40, 3.0, 48, True), None),
                                   LayerSpec(RecurrentSpec("general_delta", 5, 32), mlp),
                                   LayerSpec(ChunkAttentionSpec(2, 2, 48, 40, 2.0, 80, True), mlp)], name="tiny-makodra")
    if n in ("funevik-2048", "funevik-1024"):
        # random-init stand-ins with the layer sizes of a real small model: two memories, one latent and one full attention in turn
        d, H, ff = (2048, 16, 5632) if n.endswith("2048") else (1024, 8, 2816)
        dense = FeedForwardSpec("geglu", ff=ff)
        moe = FeedForwardSpec("moe", expert=GluSpec(ff // 8), router=RouterSpec(32, 4, bias=True), shared=GluSpec(ff // 4), shared_gate=True)
        mem = RecurrentSpec("mlstm", d // 256, 128, 256, 15.0)
        four = [mem, mem, LatentAttentionSpec(H, 128, 128, 256, 192 ** -0.5, 768, RotarySpec(64, 10000.0), 1024, True),
                GroupedAttentionSpec(H, H // 4, 128, 128, 128 ** -0.5, 4, RotarySpec(64, 500000.0), 50.0)]
        return ModelConfig(arch="funevik", vocab_size=65536, hidden_size=d, n_layers=16, n_heads=H, n_kv_heads=H // 4, head_dim=128,
                           ffn_size=0, rms_eps=1e-6, max_position=UNLIMITED_POSITIONS, embed_scale=d ** 0.5,
                           layers=[LayerSpec(m, dense if i % 2 else moe) for i, m in enumerate(four * 4)], name=n)
    if n in ("tiny-funevik",):
        moe = FeedForwardSpec("moe", expert=GluSpec(40), router=RouterSpec(6, 2, bias=True), shared=GluSpec(72), shared_gate=True)
        return ModelConfig(arch="funevik", vocab_size=4096, hidden_size=136, n_layers=4, n_heads=3, n_kv_heads=3, head_dim=40,
                           ffn_size=0, rms_eps=1e-6, max_position=UNLIMITED_POSITIONS, embed_scale=3.0, name="tiny-funevik", layers=[
                               LayerSpec(LatentAttentionSpec(3, 40, 24, 48, 0.2, 56, RotarySpec(8, 1000.0), 60, True), moe),
                               LayerSpec(RecurrentSpec("mlstm", 3, 24, 40, 9.0), FeedForwardSpec("geglu", ff=200)),
                               LayerSpec(GroupedAttentionSpec(4, 2, 24, 40, 0.3, 4, RotarySpec(12, 2000.0), 20.0), None),
                               LayerSpec(RecurrentSpec("mlstm", 2, 48, 24, 12.0), moe)])
    if n in ("padadra-2048", "padadra-1024"):
        # random-init stand-ins with the layer sizes of a real small model: two delta rules to one layer of attention beside a memory
        d, H = (2048, 16) if n.endswith("2048") else (1024, 8)
        mlp, delta = FeedForwardSpec("relu2", ff=4 * d), RecurrentSpec("channel_delta", H, 128, 128, kv_heads=H // 2, conv=4)
        rot = RotarySpec(64, 500000.0, (8.0, 1.0, 4.0, 8192.0))
        both = ParallelSpec(GroupedAttentionSpec(H, H // 4, 128, 128, 128 ** -0.5, 4, rot, gate=False, window=1024, learned_sink=True, bias=True,
                                                 row_norm=True, turn_values=RotarySpec(128, rot.base)), RecurrentSpec("hgrn2", H, 128, 128))
        return ModelConfig(arch="padadra", vocab_size=65536, hidden_size=d, n_layers=15, n_heads=H, n_kv_heads=H // 4, head_dim=128, ffn_size=0,
                           rms_eps=1e-6, max_position=UNLIMITED_POSITIONS, bigram=(65521, 2654435, 40503), residual_mult=0.4,
                           layers=[LayerSpec(delta, mlp), LayerSpec(delta, mlp), LayerSpec(both, mlp)] * 5, name=n)
    if n in ("tiny-padadra",):
        rot, mlp = RotarySpec(12, 2000.0, (4.0, 1.0, 3.0, 128.0)), FeedForwardSpec("relu2", ff=200)
        both = ParallelSpec(GroupedAttentionSpec(4, 2, 24, 40, 0.3, 3, rot, gate=False, window=50, learned_sink=True, bias=True, row_norm=True,
                                                 turn_values=RotarySpec(40, rot.base)), RecurrentSpec("hgrn2", 3, 32, 24))
        return ModelConfig(arch="padadra", vocab_size=4096, hidden_size=136, n_layers=3, n_heads=4, n_kv_heads=2, head_dim=24, ffn_size=0,
                           rms_eps=1e-6, max_position=UNLIMITED_POSITIONS, embed_scale=2.0, bigram=(997, 31, 17), residual_mult=0.6,
                           layers=[LayerSpec(both, mlp), LayerSpec(RecurrentSpec("channel_delta", 4, 24, 40, kv_heads=2, conv=4), None),
                                   LayerSpec(both, mlp)], name="tiny-padadra")
    raise KeyError(f"unknown preset {name!r}")


def resolve_config(spec) -> ModelConfig:
    if isinstance(spec, ModelConfig):
        return spec
    if isinstance(spec, str) and spec.startswith("preset:"):
        return preset(spec[len("preset:"):])
    if isinstance(spec, str) and os.path.isdir(spec):
        return ModelConfig.from_pretrained(spec)
    if isinstance(spec, str):
        return preset(spec)
    raise TypeError(f"cannot resolve a model config from {spec!r}")
