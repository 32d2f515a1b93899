"""Model hyper-parameters and the named shapes used by the benchmarks and tests.

The fields mirror the GGUF keys the reference reads (common/transformer.h:1604-1636 and
cuda/llm/cuda_llm_runner.c:11277-11310): ``<arch>.embedding_length``, ``attention.head_count``,
``attention.head_count_kv``, ``block_count``, ``feed_forward_length``, ``vocab_size``,
``attention.layer_norm_rms_epsilon``, ``rope.freq_base``, ``expert_count``, ``expert_used_count``,
``expert_feed_forward_length``, ``attention.key_length``, ``rope.dimension_count``, the ``ssm.*`` family and
``attention.full_attention_interval`` of the Qwen3.5 hybrids.
"""
from __future__ import annotations

import math
from dataclasses import asdict, dataclass, field, replace
from typing import Dict, List, Optional

# Architectures described layer by layer (``ModelConfig.layer_specs``): name in config.json -> arch
LAYERED_ARCHS = {"Zogavik": "zogavik", "Famepel": "famepel", "Fidolix": "fidolix", "Zedirax": "zedirax"}

ARCHS = ("qwen2", "qwen2vl", "qwen3", "qwen3vl", "qwen3moe", "qwen3vlmoe", "qwen35", "qwen35moe")


@dataclass
class RotarySpec:
    """Rotary positions of neighbouring pairs (2i, 2i + 1), or (``halves``) of the pairs (i, i + dims / 2).  ``factor`` > 0: YaRN, with the pairs between
    ``fast`` and ``slow`` turns over ``original`` positions blended from the plain to the divided frequency."""
    dims: int
    base: float
    factor: float = 0.0
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0
    halves: bool = False

    def pair_order(self) -> List[int]:
        """The rotated dimensions with the members of a pair side by side: a projection whose rows are in this order makes neighbouring pairs of any
        layout (scores do not depend on the order, as long as queries and keys share it)."""
        n = self.dims // 2
        return [j for i in range(n) for j in (i, i + n)] if self.halves else list(range(self.dims))

    def frequencies(self) -> List[float]:
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if self.factor <= 0:
            return f

        def pair_of(turns: float) -> float:         # the (fractional) pair that makes `turns` turns over the original length
            return self.dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))

        lo = max(math.floor(pair_of(self.fast)), 0)
        hi = min(math.ceil(pair_of(self.slow)), self.dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))]
        return [x / self.factor * r + x * (1.0 - r) for x, r in zip(f, ramp)]

    @property
    def magnitude(self) -> float:
        """Factor of cos and sin."""
        return 0.1 * math.log(self.factor) + 1.0 if self.factor > 0 else 1.0


@dataclass
class MoeSpec:
    """A mixture of experts: feed-forwards of width ``ffn``, ``top`` of ``n_experts`` per token, SiLU-gated or (``act`` "gelu") plain.  ``groups`` > 1: the experts
    form groups of neighbours, a group scores the sum of its ``group_best`` (1 or 2) best experts, and only the best ``groups_kept`` groups can be chosen from.
    ``shared`` > 0: one more expert of that width sees every token, times the sigmoid of a projection of the token to one number."""
    n_experts: int
    top: int
    ffn: int
    router: str = "softmax"                 # or "sigmoid"
    renorm: bool = True                     # the chosen scores are divided by their sum
    scale: float = 1.0
    groups: int = 1
    groups_kept: int = 1
    group_best: int = 2
    act: str = "silu"                       # act(gate) * up -> down; "gelu": the exact GELU of up alone -> down
    shared: int = 0

    @property
    def gated(self) -> bool:
        return self.act != "gelu"


# mixers with a state of a fixed size per sequence
RECURRENT = ("lightning", "mamba2", "hgrn2", "rwkv", "mingru")


@dataclass
class LayerSpec:
    """One layer of a model described layer by layer: its mixer with the mixer's own sizes, and its feed-forward."""
    mixer: str                              # "attention" | "lightning" | "mamba2" | "hgrn2" | "latent" | "rwkv" | "mingru" | "parallel"
    n_heads: int
    head_dim: int                           # query / key size per head (mamba2: the state size; latent: without the rotated part)
    v_dim: int                              # value size per head (mingru: the state, one head of one row)
    n_kv_heads: int = 0                     # attention only
    # attention
    scale: float = 0.0                      # factor of q . k (0 = 1 / sqrt(head_dim))
    qkv_bias: bool = False
    qk_unit: bool = False                   # q and k divided by their root mean square per head (no weight)
    window: int = 0                         # position i sees j with i - j < window ... (0 = all)
    keep_first: int = 0                     # ... or j < keep_first
    rel_buckets: int = 0                    # rows of the learned distance-bias table (0 = none)
    rel_max: float = 0                      # distance from which the last bucket holds
    qk_norm_rows: bool = False              # RMS norm with weights over all of q, and over all of k
    softcap: float = 0.0                    # scores become softcap * tanh(score / softcap) (0 = as they are)
    out_gate: bool = False                  # the heads' outputs are multiplied by the sigmoid of a projection
    v_from_k: bool = False                  # the values are the keys before their rotation
    log_bias: bool = False                  # r1 ln(1 + r2 distance) is taken off the scores, two learned numbers per head
    temp_coef: float = 0.0                  # queries at position p are multiplied by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1)
    temp_every: float = 1.0
    # lightning attention
    decay: Optional[List[float]] = None     # per head
    # mamba2
    state_groups: int = 1                   # heads share B and C by groups
    conv_taps: int = 0                      # causal convolution in front of the recurrence (attention: of q and k, in front of the rotation)
    norm_parts: int = 1                     # the output norm's equal parts
    # rwkv: a decay per key channel through a low-rank projection of the input
    decay_rank: int = 0
    # parallel: two mixers side by side over the same input, left_scale * left + right_scale * right
    left: Optional["LayerSpec"] = None
    right: Optional["LayerSpec"] = None
    left_scale: float = 1.0
    right_scale: float = 1.0
    # latent attention: keys and values are projections of a cached latent, next to one rotated key part for all heads
    kv_rank: int = 0
    q_rank: int = 0                         # queries through a normed latent of their own (0: projected at once)
    rot_dim: int = 0
    rotary: Optional[RotarySpec] = None
    sink: bool = False                      # a learned score per head joins the softmax's sum
    kv_from: int = -1                       # layer whose cache this one reads (-1: its own)
    # feed-forward: act(gate) * up -> down; 0 = none
    ffn: int = 0
    act: str = "silu"                       # or "gelu_tanh", "capped" (x sigmoid(1.702 x) of min(gate, cap), times 1 + up within +-cap)
    act_cap: float = 0.0
    ffn_bias: bool = False                  # all three projections of the dense feed-forward have biases
    moe: Optional[MoeSpec] = None           # in place of the dense feed-forward

    def __post_init__(self):
        if isinstance(self.rotary, dict):
            self.rotary = RotarySpec(**self.rotary)
        if isinstance(self.moe, dict):
            self.moe = MoeSpec(**self.moe)
        if isinstance(self.left, dict):
            self.left = LayerSpec(**self.left)
        if isinstance(self.right, dict):
            self.right = LayerSpec(**self.right)

    @property
    def mixers(self) -> List["LayerSpec"]:
        """The mixer itself, or the two of a parallel one."""
        return [self.left, self.right] if self.mixer == "parallel" else [self]

    @property
    def q_dim(self) -> int:
        return self.n_heads * self.head_dim

    @property
    def has_ffn(self) -> bool:
        return self.ffn > 0 or self.moe is not None

    @property
    def has_state(self) -> bool:
        """Whether the mixer carries state of a fixed size per sequence, which cannot drop positions."""
        return any(x.mixer in RECURRENT or x.conv_taps > 1 for x in self.mixers)

    @property
    def paged(self) -> Optional["LayerSpec"]:
        """The mixer that keeps keys and values in cache pages."""
        return next((x for x in self.mixers if x.mixer in ("attention", "latent")), None)

    @property
    def conv_channels(self) -> int:
        """Channels of the convolution: [x heads x v_dim | B groups x head_dim | C groups x head_dim], attention: [q heads | k heads]."""
        if self.mixer == "attention":
            return (self.n_heads + self.n_kv_heads) * self.head_dim
        return self.n_heads * self.v_dim + 2 * self.state_groups * self.head_dim

    @property
    def span(self) -> int:
        """Most keys a position sees (0 = no limit)."""
        return self.window + self.keep_first if self.window > 0 else 0


@dataclass
class LoopSpec:
    """Layers ``start .. stop - 1`` run ``times`` times in a row with the same weights; every pass has its own cache or state.  ``add`` "step": a
    learned vector is added to the stream in front of each pass; "embedding": the embedding output, in front of each but the first."""
    start: int
    stop: int
    times: int
    add: str = "step"


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer: ``layer`` is its index in the weights, ``step`` the row of the step-vector table added in front of it
    (-1 = none), ``again`` whether the embedding output is.  The position of the run in ``ModelConfig.layer_runs`` is the index of its cache."""
    layer: int
    step: int = -1
    again: bool = False


@dataclass
class ModelConfig:
    arch: str = "qwen3"
    n_layers: int = 2
    hidden: int = 256
    n_heads: int = 4
    n_kv_heads: int = 2
    head_dim: int = 64
    ffn: int = 512
    vocab: int = 1024
    rms_eps: float = 1e-6
    rope_theta: float = 1e6
    rope_dim: Optional[int] = None          # partial rotary (None = head_dim)
    qk_norm: bool = True
    qkv_bias: bool = False                  # Qwen2
    tie_embeddings: bool = False
    max_seq_len: int = 4096
    sliding_window: int = 0
    # MoE
    n_experts: int = 0
    n_experts_used: int = 0
    expert_ffn: int = 0
    norm_topk: bool = True
    router: str = "softmax"                 # or "sigmoid" (MiniMax-M3 / GLM-5 style, with selection bias)
    routed_scale: float = 1.0
    shared_expert_ffn: int = 0              # qwen35moe shared expert (sigmoid-gated)
    # Qwen3.5 hybrid (Delta-Net) layers
    full_attention_interval: int = 0        # every n-th layer is full attention, the rest are SSM layers
    ssm_d_conv: int = 4
    ssm_n_heads_k: int = 0
    ssm_n_heads_v: int = 0
    ssm_head_dim: int = 0
    attn_output_gate: bool = False          # attn_q emits [Q | gate] per head, output *= sigmoid(gate)
    # M-RoPE (Qwen2-VL / Qwen3-VL): sections of rotary pairs assigned to t / h / w
    mrope_sections: Optional[List[int]] = None
    n_deepstack_layers: int = 0
    # models described layer by layer (the residual stream is then kept in 32-bit floats)
    layer_specs: Optional[List[LayerSpec]] = None
    loop: Optional[LoopSpec] = None
    norm_offset: float = 0.0                # stored norm weights are added to this (1 = stored around zero)
    logit_scale: float = 1.0
    norm_kind: str = "rms"                  # or "dyt": tanh(alpha x) w + b
    post_norm: bool = False                 # every sublayer's result passes a norm of its own and a per-channel scale
    embed_scale: float = 1.0
    parallel_ffn: bool = False              # mixer and feed-forward read the same stream, each through a norm of its own
    side_dim: int = 0                       # per-layer token input of this size (a table of the token's vectors for all layers), 0 = none
    residual_mult: float = 1.0              # factor of every sublayer's result
    depth_average: bool = False             # a layer hands on a learned weighted sum of the embedding output and all layers' results so far

    def __post_init__(self):
        if self.layer_specs is not None:
            self.layer_specs = [x if isinstance(x, LayerSpec) else LayerSpec(**x) for x in self.layer_specs]
            self.n_layers = len(self.layer_specs)
        if self.loop is not None and not isinstance(self.loop, LoopSpec):
            self.loop = LoopSpec(**self.loop)

    @property
    def is_layered(self) -> bool:
        return self.layer_specs is not None

    def layer_runs(self) -> List[LayerRun]:
        """The layers in the order of execution (looped layers appear once per pass)."""
        n, lp = self.n_layers, self.loop
        if lp is None:
            return [LayerRun(i) for i in range(n)]
        if not 0 <= lp.start < lp.stop <= n or lp.times < 1:
            raise ValueError(f"bad layer loop {lp} for {n} layers")
        runs = [LayerRun(i) for i in range(lp.start)]
        for t in range(lp.times):
            emb, first = lp.add == "embedding", lp.start
            runs += [LayerRun(i, t if i == first and not emb else -1, emb and i == first and t > 0) for i in range(lp.start, lp.stop)]
        return runs + [LayerRun(i) for i in range(lp.stop, n)]

    @property
    def has_recurrent_state(self) -> bool:
        """Whether a sequence carries state that cannot drop positions (Delta-Net, lightning, Mamba-2, HGRN2, RWKV or minGRU layers, convolutions)."""
        return self.is_hybrid or (self.is_layered and any(x.has_state for x in self.layer_specs))

    @property
    def is_moe(self) -> bool:
        return self.n_experts > 0

    @property
    def q_dim(self) -> int:
        return self.n_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.n_kv_heads * self.head_dim

    @property
    def is_hybrid(self) -> bool:
        return self.full_attention_interval > 0

    @property
    def ssm_d_inner(self) -> int:
        return self.ssm_n_heads_v * self.ssm_head_dim

    @property
    def ssm_qkv_dim(self) -> int:
        return 2 * self.ssm_n_heads_k * self.ssm_head_dim + self.ssm_d_inner

    def is_ssm_layer(self, layer: int) -> bool:
        if self.full_attention_interval <= 0:
            return False
        return (layer + 1) % self.full_attention_interval != 0

    def param_count(self) -> int:
        if self.is_layered:
            tot = self.vocab * self.hidden * (1 if self.tie_embeddings else 2) + self.vocab * self.n_layers * self.side_dim
            for x in self.layer_specs:
                if x.moe is not None:
                    per = 3 if x.moe.gated else 2
                    tot += x.moe.n_experts * self.hidden * (per * x.moe.ffn + 1) + (self.hidden * (per * x.moe.shared + 1) if x.moe.shared else 0)
                tot += 3 * self.hidden * x.ffn + 2 * self.hidden * self.side_dim
            for x in (m for sp in self.layer_specs for m in sp.mixers):
                nv = x.n_heads * x.v_dim
                if x.mixer == "lightning":
                    tot += self.hidden * (2 * x.q_dim + 3 * nv)
                elif x.mixer == "hgrn2":
                    tot += self.hidden * (2 * x.q_dim + 2 * nv)
                elif x.mixer == "mamba2":
                    tot += self.hidden * (2 * nv + x.conv_channels + x.n_heads) + x.conv_channels * x.conv_taps
                elif x.mixer == "latent":
                    own = 0 if x.kv_from >= 0 else x.kv_rank + x.rot_dim
                    tot += self.hidden * (x.q_rank + own + (2 if x.out_gate else 1) * nv) + (x.q_rank or self.hidden) * x.n_heads * (x.head_dim + x.rot_dim) + x.kv_rank * (x.q_dim + nv)
                elif x.mixer == "mingru":
                    tot += 4 * self.hidden * nv
                elif x.mixer == "rwkv":
                    tot += self.hidden * (2 * x.q_dim + 3 * nv + x.decay_rank) + x.q_dim * x.decay_rank
                else:
                    tot += self.hidden * (x.q_dim + x.n_kv_heads * (x.head_dim + (0 if x.v_from_k else x.v_dim)) + (2 if x.out_gate else 1) * nv)
            return tot
        per_layer = self.hidden * (self.q_dim + 2 * self.kv_dim) + self.q_dim * self.hidden
        if self.is_moe:
            per_layer += self.n_experts * 3 * self.hidden * self.expert_ffn + self.n_experts * self.hidden
        else:
            per_layer += 3 * self.hidden * self.ffn
        emb = self.vocab * self.hidden * (1 if self.tie_embeddings else 2)
        return per_layer * self.n_layers + emb

    def to_dict(self) -> Dict:
        return asdict(self)

    def with_(self, **kw) -> "ModelConfig":
        return replace(self, **kw)


def _qwen3(name, **kw) -> ModelConfig:
    return ModelConfig(arch="qwen3", head_dim=128, vocab=151936, **kw)


PRESETS: Dict[str, ModelConfig] = {
    # the five benchmark shapes
    "qwen3-0.6b": _qwen3("0.6b", n_layers=28, hidden=1024, n_heads=16, n_kv_heads=8, ffn=3072, tie_embeddings=True),
    "qwen3-8b": _qwen3("8b", n_layers=36, hidden=4096, n_heads=32, n_kv_heads=8, ffn=12288),
    "qwen3-32b": _qwen3("32b", n_layers=64, hidden=5120, n_heads=64, n_kv_heads=8, ffn=25600),
    "qwen3-30b-a3b": ModelConfig(arch="qwen3moe", n_layers=48, hidden=2048, n_heads=32, n_kv_heads=4, head_dim=128, ffn=6144,
                                 vocab=151936, n_experts=128, n_experts_used=8, expert_ffn=768),
    "qwen3-235b-a22b": ModelConfig(arch="qwen3moe", n_layers=94, hidden=4096, n_heads=64, n_kv_heads=4, head_dim=128, ffn=12288,
                                   vocab=151936, n_experts=128, n_experts_used=8, expert_ffn=1536),
    # small shapes for tests (head_dim 128 so that the tcgen05 attention kernel applies)
    "tiny-dense": ModelConfig(arch="qwen3", n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, head_dim=128, ffn=512, vocab=512),
    "tiny-moe": ModelConfig(arch="qwen3moe", n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, head_dim=128, ffn=512, vocab=512,
                            n_experts=16, n_experts_used=4, expert_ffn=128),
    # hybrid: layers 0 and 2 are Delta-Net layers, 1 and 3 gated full attention; the MoE variant adds a shared expert
    "tiny-qwen35": ModelConfig(arch="qwen35", n_layers=4, hidden=256, n_heads=4, n_kv_heads=2, head_dim=128, ffn=512, vocab=512,
                               rope_dim=64, full_attention_interval=2, ssm_d_conv=4, ssm_n_heads_k=2, ssm_n_heads_v=4, ssm_head_dim=64,
                               attn_output_gate=True, mrope_sections=[11, 11, 10, 0]),
    "tiny-qwen35moe": ModelConfig(arch="qwen35moe", n_layers=4, hidden=256, n_heads=4, n_kv_heads=2, head_dim=128, ffn=512, vocab=512,
                                  rope_dim=64, full_attention_interval=2, ssm_d_conv=4, ssm_n_heads_k=2, ssm_n_heads_v=4, ssm_head_dim=64,
                                  attn_output_gate=True, mrope_sections=[11, 11, 10, 0], n_experts=16, n_experts_used=4, expert_ffn=128, shared_expert_ffn=128),
    "tiny-qwen2": ModelConfig(arch="qwen2", n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, head_dim=128, ffn=512, vocab=512,
                              qk_norm=False, qkv_bias=True, tie_embeddings=True),
}


def _zogavik(pattern: str, hidden: int, heads: int, kv_heads: int, dim: int, ffn: int, vocab: int, window: int, keep: int, rel_max: int, loop=None,
             v_dim: int = 0, lin_heads: int = 0, lin_dim: int = 0, lin_v: int = 0, rel_buckets: int = 32) -> ModelConfig:
    """``pattern``: one letter per layer, L = lightning, A = attention."""
    lh = lin_heads or heads
    specs = []
    for c in pattern:
        if c == "L":
            specs.append(LayerSpec("lightning", lh, lin_dim or dim, lin_v or dim, decay=[1.0 - 2.0 ** -(1.0 + 7.0 * i / lh) for i in range(lh)],
                                   ffn=ffn, act="gelu_tanh"))
        else:
            specs.append(LayerSpec("attention", heads, dim, v_dim or dim, n_kv_heads=kv_heads, scale=dim ** -0.5, qkv_bias=True, qk_unit=True,
                                   window=window, keep_first=keep, rel_buckets=rel_buckets, rel_max=rel_max, ffn=ffn, act="gelu_tanh"))
    return ModelConfig(arch="zogavik", layer_specs=specs, hidden=hidden, n_heads=heads, n_kv_heads=kv_heads, head_dim=dim, ffn=ffn, vocab=vocab,
                       tie_embeddings=True, loop=loop, norm_offset=1.0, logit_scale=1.0, qk_norm=False, qkv_bias=True)


PRESETS["tiny-zogavik"] = _zogavik("ALLA", 192, 4, 2, 40, 320, 500, 48, 8, 100, LoopSpec(0, 2, 3), v_dim=56, lin_heads=3, lin_dim=24, lin_v=40)
# layers of the sizes of an 8-billion-parameter dense model, three lightning layers to one of windowed attention
PRESETS["zogavik-8b"] = _zogavik("LLLA" * 9, 4096, 32, 8, 128, 12288, 151936, 4096, 128, 4096)
# the same layers with the middle ones looped: a smaller model of the same depth
PRESETS["zogavik-4b-loop2"] = _zogavik("LLLA" * 5, 4096, 32, 8, 128, 12288, 151936, 4096, 128, 4096, LoopSpec(2, 18, 2))


def _famepel(pattern: str, hidden: int, vocab: int, moe: MoeSpec, hgrn, mamba, latent, rotary: RotarySpec) -> ModelConfig:
    """``pattern``: one letter per layer, H = HGRN2, M = Mamba-2, L = latent attention, S = latent attention over the cache of the nearest L in
    front of it.  ``hgrn`` (heads, dim, vdim), ``mamba`` (heads, state, vdim, groups, taps, norm parts), ``latent`` (heads, dim, rot_dim, vdim,
    kv_rank, q_rank)."""
    specs: List[LayerSpec] = []
    own = -1
    for i, c in enumerate(pattern):
        if c == "H":
            specs.append(LayerSpec("hgrn2", *hgrn, moe=moe))
        elif c == "M":
            heads, n, v, groups, taps, parts = mamba
            specs.append(LayerSpec("mamba2", heads, n, v, state_groups=groups, conv_taps=taps, norm_parts=parts, moe=moe))
        else:
            heads, d, r, v, kvr, qr = latent
            own = i if c == "L" else own
            specs.append(LayerSpec("latent", heads, d, v, n_kv_heads=1, scale=(d + r) ** -0.5, kv_rank=kvr, q_rank=qr, rot_dim=r, rotary=rotary, sink=True,
                                   kv_from=own if c == "S" else -1, moe=moe))
    return ModelConfig(arch="famepel", layer_specs=specs, hidden=hidden, n_heads=latent[0], n_kv_heads=latent[0], head_dim=latent[1], ffn=moe.ffn, vocab=vocab,
                       rms_eps=1e-5, norm_kind="dyt", post_norm=True, embed_scale=hidden ** 0.5, qk_norm=False)


PRESETS["tiny-famepel"] = _famepel("MHLMS", 192, 300, MoeSpec(10, 3, 48, "sigmoid", True, 1.7, 5, 2), (3, 24, 40), (4, 40, 24, 2, 4, 2), (3, 24, 16, 40, 72, 56),
                                   RotarySpec(16, 10000.0, 4.0, 64, 32.0, 1.0))
# layers of the sizes of a 30-billion-parameter mixture of experts (128 experts, 8 per token)
PRESETS["famepel-30b-a3b"] = _famepel("HMLHMMHMS" * 5, 2048, 151936, MoeSpec(128, 8, 768, "sigmoid", True, 2.5, 8, 4), (16, 128, 128), (64, 128, 64, 8, 4, 8),
                                      (32, 128, 64, 128, 512, 1536), RotarySpec(64, 500000.0, 8.0, 4096, 32.0, 1.0))


def _fidolix(pattern: str, hidden: int, vocab: int, side_dim: int, att, left, right, rotary: RotarySpec, window: int, taps: int, cap: float, dense: int, act_cap: float, moe: MoeSpec,
             embed_scale: float, scales=(1.0, 1.0), loop: Optional[LoopSpec] = None) -> ModelConfig:
    """``pattern``: one letter per layer, A = attention, P = windowed attention beside an RWKV recurrence, with a mixture of experts; a, p = with a dense
    feed-forward.  ``att`` (heads, KV heads, dim, vdim), ``left`` (heads, KV heads, dim), ``right`` (heads, dim, decay rank)."""
    specs: List[LayerSpec] = []
    for c in pattern:
        ff = dict(ffn=dense, act="capped", act_cap=act_cap) if c.islower() else dict(moe=moe)
        if c in "Aa":
            hd, g, d, v = att
            specs.append(LayerSpec("attention", hd, d, v, n_kv_heads=g, scale=d ** -0.5, qkv_bias=True, qk_norm_rows=True, softcap=cap, out_gate=True, **ff))
        else:
            hd, g, d = left
            lt = LayerSpec("attention", hd, d, d, n_kv_heads=g, scale=d ** -0.5, qkv_bias=True, v_from_k=True, conv_taps=taps, rotary=rotary, window=window, sink=True)
            rt = LayerSpec("rwkv", right[0], right[1], right[1], decay_rank=right[2])
            specs.append(LayerSpec("parallel", hd, d, d, n_kv_heads=g, left=lt, right=rt, left_scale=scales[0], right_scale=scales[1], **ff))
    return ModelConfig(arch="fidolix", layer_specs=specs, hidden=hidden, n_heads=att[0], n_kv_heads=att[1], head_dim=att[2], ffn=dense, vocab=vocab, rms_eps=1e-5,
                       embed_scale=embed_scale, parallel_ffn=True, side_dim=side_dim, qk_norm=False, loop=loop)


PRESETS["tiny-fidolix"] = _fidolix("pAPa", 192, 300, 20, (4, 2, 40, 24), (6, 3, 32), (3, 24, 12), RotarySpec(24, 10000.0, 4.0, 64, 32.0, 1.0), 50, 4, 20.0, 320, 1.5,
                                   MoeSpec(12, 3, 48, renorm=True, groups=4, groups_kept=2, group_best=1), 3.0, (0.7, 1.2), LoopSpec(1, 3, 2, "embedding"))
# layers of the sizes of a 30-billion-parameter mixture of experts (128 experts, 8 per token), every third one attention without a window
PRESETS["fidolix-30b-a3b"] = _fidolix("pPA" + "PPA" * 14, 2048, 151936, 128, (32, 4, 128, 128), (16, 2, 128), (16, 128, 64), RotarySpec(64, 500000.0, 8.0, 4096, 32.0, 1.0),
                                      1024, 4, 30.0, 6144, 7.0, MoeSpec(128, 8, 768, renorm=True, groups=8, groups_kept=4, group_best=1), 2048 ** 0.5)


def _zedirax(pattern: str, hidden: int, vocab: int, width: int, latent, att, temp, rotary: RotarySpec, dense: int, moe: MoeSpec, mult: float) -> ModelConfig:
    """``pattern``: one letter per layer, G = minGRU, L = latent attention, A = attention, with a mixture of experts; g, l, a = with a dense feed-forward.  ``latent``
    (heads, dim, rot_dim, vdim, kv_rank), ``att`` (heads, KV heads, dim, vdim), ``temp`` (coefficient, every)."""
    specs: List[LayerSpec] = []
    for c in pattern:
        ff = dict(ffn=dense, act="gelu_tanh", ffn_bias=True) if c.islower() else dict(moe=moe)
        if c in "Gg":
            specs.append(LayerSpec("mingru", 1, 1, width, **ff))
        elif c in "Ll":
            hd, d, r, v, kvr = latent
            specs.append(LayerSpec("latent", hd, d, v, n_kv_heads=1, scale=(d + r) ** -0.5, kv_rank=kvr, rot_dim=r, rotary=rotary, out_gate=True, **ff))
        else:
            hd, g, d, v = att
            specs.append(LayerSpec("attention", hd, d, v, n_kv_heads=g, scale=d ** -0.5, log_bias=True, temp_coef=temp[0], temp_every=temp[1], **ff))
    return ModelConfig(arch="zedirax", layer_specs=specs, hidden=hidden, n_heads=att[0], n_kv_heads=att[1], head_dim=att[2], ffn=dense, vocab=vocab, rms_eps=1e-5, norm_offset=1.0,
                       residual_mult=mult, depth_average=True, qk_norm=False)


PRESETS["tiny-zedirax"] = _zedirax("gLAgl", 192, 300, 136, (3, 24, 8, 40, 72), (4, 2, 40, 24), (0.25, 50), RotarySpec(8, 10000.0, halves=True), 320,
                                   MoeSpec(10, 3, 56, act="gelu", shared=88), 0.6)
# layers of the sizes of a 30-billion-parameter mixture of experts (128 experts, 8 per token; a plain expert of 1152 has the size of a gated one of 768)
PRESETS["zedirax-30b-a3b"] = _zedirax("gGLGGAGGL" + "GGLGGAGGL" * 4, 2048, 151936, 4096, (32, 128, 64, 128, 512), (32, 4, 128, 128), (0.1, 8192), RotarySpec(64, 500000.0, halves=True),
                                      6144, MoeSpec(128, 8, 1152, act="gelu", shared=1152), 0.5)


def get_config(name: str) -> ModelConfig:
    if name not in PRESETS:
        raise KeyError(f"unknown model preset {name!r}; known: {sorted(PRESETS)}")
    return replace(PRESETS[name])
