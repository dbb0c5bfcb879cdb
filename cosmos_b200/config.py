"""Configuration dataclasses: model shapes, parallel layout, sampling recipe.

The reference publishes no model config file; tower shapes follow the public Qwen3-VL text
configs that the reference says its Reasoner is based on (reference README.md:286; model
sizes README.md:79-85: Nano 16B = 2 x 8B towers, Super 64B = 2 x 32B towers).
"""
from __future__ import annotations

from dataclasses import asdict, dataclass, field, replace
from typing import Dict, List, Optional, Tuple, Union


@dataclass
class MoTConfig:
    name: str = "tiny"
    d_model: int = 512
    n_layers: int = 4
    n_heads: int = 8
    n_kv_heads: int = 8
    head_dim: int = 64
    ffn_dim: int = 2048
    vocab_size: int = 32000
    rope_theta: float = 5.0e5
    mrope_section: Tuple[int, int, int] = (12, 10, 10)  # (t, h, w) frequency counts, sum = head_dim / 2
    rms_eps: float = 1e-6
    qk_norm: bool = True
    share_attn_proj: bool = False  # True: AR and DM towers use the same QKV/O projection weights
    # DM side
    latent_channels: int = 16
    patch_t: int = 1
    patch_hw: int = 2
    vae_t_compress: int = 4
    vae_s_compress: int = 8
    t_embed_dim: int = 256
    sound_latent_dim: int = 64      # channels of one audio latent frame
    action_dim_max: int = 64        # padded per-domain raw action dim
    action_domains: Tuple[str, ...] = ("av", "droid_lerobot", "umi", "bridge_orig_lerobot", "camera_pose")
    # AR side vision encoder (ViT) — Qwen3-VL conventions
    vit_depth: int = 2
    vit_hidden: int = 128
    vit_heads: int = 4
    vit_patch: int = 16
    vit_temporal_patch: int = 2
    vit_spatial_merge: int = 2
    # ViT block indexes whose features are merged and added to the hidden states of the first AR layers
    # (DeepStack of the Qwen3-VL family the Reasoner follows; () = off)
    vit_deepstack: Tuple[int, ...] = ()
    vit_ffn: int = 0          # MLP width of a ViT block; 0 = 4 x vit_hidden
    vit_pos_side: int = 48    # the learned position table covers vit_pos_side x vit_pos_side patches
    max_text_len: int = 512
    init_std: float = 0.02

    @property
    def q_dim(self) -> int:
        return self.n_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.n_kv_heads * self.head_dim

    @property
    def qkv_dim(self) -> int:
        return self.q_dim + 2 * self.kv_dim

    @property
    def patch_dim(self) -> int:
        return self.latent_channels * self.patch_t * self.patch_hw * self.patch_hw

    def tower_params(self) -> int:
        """Parameter count of one tower's transformer body (no embeddings)."""
        per_layer = (self.qkv_dim * self.d_model + self.d_model * self.q_dim
                     + 3 * self.ffn_dim * self.d_model + 2 * self.d_model + 2 * self.head_dim)
        return per_layer * self.n_layers

    def to_dict(self) -> Dict:
        return asdict(self)


def tiny_config(**kw) -> MoTConfig:
    """4 layers, d=512, 8 heads of 64, MLP 4x, 32k vocab: the CPU/gloo plumbing model."""
    return replace(MoTConfig(), **kw)


def tiny128_config(**kw) -> MoTConfig:
    """Small model with head_dim 128 so that every CUDA kernel (attention included) is on its path."""
    base = MoTConfig(name="tiny128", d_model=512, n_layers=2, n_heads=4, n_kv_heads=2, head_dim=128,
                     ffn_dim=1024, vocab_size=4096, mrope_section=(24, 20, 20))
    return replace(base, **kw)


def nano_config(**kw) -> MoTConfig:
    """Cosmos3-Nano stand-in: two Qwen3-VL-8B-shaped towers (16.4 B parameters)."""
    base = MoTConfig(name="Cosmos3-Nano", d_model=4096, n_layers=36, n_heads=32, n_kv_heads=8, head_dim=128,
                     ffn_dim=12288, vocab_size=151936, mrope_section=(24, 20, 20),
                     vit_depth=27, vit_hidden=1152, vit_heads=16, vit_ffn=4304, vit_deepstack=(8, 16, 24))
    return replace(base, **kw)


def super_config(**kw) -> MoTConfig:
    """Cosmos3-Super stand-in: two Qwen3-VL-32B-shaped towers (65.5 B parameters)."""
    base = MoTConfig(name="Cosmos3-Super", d_model=5120, n_layers=64, n_heads=64, n_kv_heads=8, head_dim=128,
                     ffn_dim=25600, vocab_size=151936, mrope_section=(24, 20, 20),
                     vit_depth=27, vit_hidden=1152, vit_heads=16, vit_ffn=4304, vit_deepstack=(8, 16, 24))
    return replace(base, **kw)


# --------------------------------------------------------------------------- config-declared decoder stacks
@dataclass(frozen=True)
class AttentionSpec:
    """Attention mixer of a stack layer. The optional mechanisms are switches, so that another design can combine them
    differently: sliding window (None = unlimited), distance bias `r1 ln(1 + r2 (i - j))` per head with learned r1, r2 or the
    fixed linear bias `2^(-8 (h + 1) / heads) (i - j)`, RMS norm of each value head, mixing of the values with those of an
    earlier layer, q/k/v biases, RMS norm over the whole query / key projection, keys that serve as values, a temperature
    on the queries that grows with the logarithm of the position."""
    heads: int
    kv_heads: int
    dim: int                      # query / key head size
    vdim: int                     # value head size
    scale: float
    window: Optional[int] = None  # keys seen by a query, itself included
    distance_bias: bool = False
    linear_bias: bool = False
    value_norm: bool = False
    value_mix: bool = False       # the first such layer gives its values, the others mix them in
    qkv_bias: bool = False
    qk_norm: bool = False         # over all heads at once
    key_values: bool = False      # v = the projected keys before their norm
    q_temp: Optional[Tuple[float, int]] = None   # (coef, every): q *= 1 + coef ln(floor((p + 1) / every) + 1)

    @property
    def qkv_cols(self) -> int:
        return self.heads * self.dim + self.kv_heads * (self.dim + (0 if self.key_values else self.vdim))

    def check(self) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads:
            raise ValueError("heads must be a positive multiple of kv_heads")
        if self.window is not None and self.window < 1:
            raise ValueError("the window holds at least the token itself")
        if self.key_values and self.dim != self.vdim:
            raise ValueError("keys serve as values: dim and vdim must be equal")
        if self.q_temp is not None and self.q_temp[1] < 1:
            raise ValueError("the query temperature needs a positive step")


@dataclass(frozen=True)
class MatrixMemorySpec:
    """mLSTM mixer: a [dim, vdim] matrix memory per head with exponential input gate and sigmoid forget gate, both gates'
    pre-activations soft-capped at `gate_cap`; heads normed, weighted and gated at the output."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    def check(self) -> None:
        if min(self.heads, self.dim, self.vdim) < 1 or not self.gate_cap > 0:
            raise ValueError("a matrix memory needs positive sizes and a positive gate cap")


@dataclass(frozen=True)
class SelectiveScanSpec:
    """Mamba mixer: `inner` channels with `state` states each, a causal convolution of `conv` taps ahead of the scan, step
    sizes from a projection of rank `dt_rank`."""
    inner: int
    state: int
    dt_rank: int
    conv: int

    def check(self) -> None:
        if min(self.inner, self.state, self.dt_rank, self.conv) < 1:
            raise ValueError("a selective scan needs positive sizes")


@dataclass(frozen=True)
class ParallelSpec:
    """Attention and a matrix memory side by side on the same input: half the sum of the two outputs, each RMS-normed over the
    model width with a weight of its own."""
    left: AttentionSpec
    right: MatrixMemorySpec

    def check(self) -> None:
        self.left.check()
        self.right.check()


@dataclass(frozen=True)
class MoESpec:
    """Experts chosen by a table over token ids: table [vocab, top], each chosen expert with weight 1 / top; an expert is
    down(gelu(up(h))) without biases (erf gelu)."""
    experts: int
    top: int
    ff: int

    def check(self) -> None:
        if not 1 <= self.top <= self.experts:
            raise ValueError("top must be between 1 and the number of experts")


@dataclass(frozen=True)
class DenseSpec:
    """down(silu(gate(h)) * up(h)) without biases."""
    ff: int

    def check(self) -> None:
        if self.ff < 1:
            raise ValueError("the feed-forward needs a positive size")


@dataclass(frozen=True)
class StackLayerSpec:
    mixer: Union[AttentionSpec, ParallelSpec, SelectiveScanSpec]
    mlp: Union[MoESpec, DenseSpec, None] = None
    weights_of: Optional[int] = None   # uses another layer's weights (with a cache and state of its own)

    @property
    def attention(self) -> Optional[AttentionSpec]:
        """The attention of this layer, if it has one."""
        return self.mixer.left if isinstance(self.mixer, ParallelSpec) else self.mixer if isinstance(self.mixer, AttentionSpec) else None


@dataclass
class StackConfig:
    """A decoder whose layers are listed one by one (models/stack.py). `order`: "serial" = x += mixer(norm1 x), then
    x += mlp(norm2 x); "parallel" = x += mixer(norm1 x) + mlp(norm2 x), both of the same x. `norm_add` is added to the stored
    norm weights (1 for weights stored around zero)."""
    name: str
    architecture: str
    vocab_size: int
    d_model: int
    layers: Tuple[StackLayerSpec, ...]
    embed_scale: float = 1.0
    norm_eps: float = 1e-6
    norm_groups: int = 1
    init_std: float = 0.02
    order: str = "serial"
    norm_add: float = 0.0
    sinusoid: bool = False        # add the sinusoid of the position to the embedding
    tied_head: bool = False

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def rms_eps(self) -> float:
        return self.norm_eps

    def source_layer(self, i: int) -> int:
        """The layer whose weights layer i uses."""
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
        return i

    def validate(self) -> "StackConfig":
        if self.vocab_size < 1 or self.d_model < 1 or self.norm_groups < 1 or self.d_model % self.norm_groups:
            raise ValueError("vocab and width must be positive and the width a multiple of the norm groups")
        first = None
        for i, layer in enumerate(self.layers):
            m, j = layer.mixer, layer.weights_of
            try:
                m.check()
                if layer.mlp is not None:
                    layer.mlp.check()
            except ValueError as e:
                raise ValueError(f"layer {i}: {e}") from None
            if j is not None:
                if not 0 <= j < self.n_layers or j == i:
                    raise ValueError(f"layer {i}: there is no layer {j} whose weights it could use")
                seen = {i}
                while j is not None and j not in seen:
                    seen.add(j)
                    j = self.layers[j].weights_of
                src = self.layers[layer.weights_of]
                if j is not None or (src.mixer, src.mlp) != (m, layer.mlp):
                    raise ValueError(f"layer {i}: shared weights need an equal layer that leads to weights of its own")
            if isinstance(m, AttentionSpec) and m.value_mix:
                if first is None:
                    first = m
                elif (m.kv_heads, m.vdim) != (first.kv_heads, first.vdim):
                    raise ValueError(f"layer {i}: mixed values need the first mixing layer's kv_heads and vdim")
            if self.order == "serial" and not (isinstance(m, AttentionSpec) and isinstance(layer.mlp, (MoESpec, type(None)))):
                raise ValueError(f"layer {i}: serial layers take attention and table-routed experts")
            if self.order == "parallel" and (isinstance(m, AttentionSpec) or isinstance(layer.mlp, MoESpec)):
                raise ValueError(f"layer {i}: parallel layers take a scan or attention beside a matrix memory, and a dense feed-forward")
        return self

    def to_dict(self) -> Dict:
        return ARCHITECTURES[self.architecture][1](self)


def lederax_config_from_dict(doc: Dict, name: str = "Lederax") -> StackConfig:
    """config.json of a Lederax model."""
    layers = []
    for i, entry in enumerate(doc["layers"]):
        if entry["type"] != "attention":
            raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
        m = entry["mixer"]
        mask = m.get("mask")
        mixer = AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                              scale=float(m["scale"]), window=int(mask["size"]) if mask else None, distance_bias=True,
                              value_norm=True, value_mix=bool(m.get("v_mix", False)), qkv_bias=True)
        mlp = entry.get("mlp")
        if mlp is not None:
            if mlp.get("kind") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            mlp = MoESpec(experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), ff=int(mlp["expert"]["ff"]))
        layers.append(StackLayerSpec(mixer, mlp))
    return StackConfig(name=name, architecture="Lederax", vocab_size=int(doc["vocab"]), d_model=int(doc["width"]),
                       layers=tuple(layers), embed_scale=float(doc["embedding"]["scale"]), norm_eps=float(doc["norm"]["eps"]),
                       norm_groups=int(doc["norm"].get("groups", 1))).validate()


def lederax_config_to_dict(cfg: StackConfig) -> Dict:
    layers = []
    for layer in cfg.layers:
        m, f = layer.mixer, layer.mlp
        layers.append({"type": "attention",
                       "mixer": {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                                 "mask": None if m.window is None else {"size": m.window}, "v_mix": m.value_mix},
                       "mlp": None if f is None else {"kind": "moe", "expert": {"ff": f.ff},
                                                      "router": {"experts": f.experts, "top": f.top}}})
    return {"architecture": "Lederax", "vocab": cfg.vocab_size, "width": cfg.d_model,
            "embedding": {"scale": cfg.embed_scale}, "norm": {"eps": cfg.norm_eps, "groups": cfg.norm_groups}, "layers": layers}


def mererax_config_from_dict(doc: Dict, name: str = "Mererax") -> StackConfig:
    """config.json of a Mererax model."""
    layers = []
    for i, entry in enumerate(doc["layers"]):
        m, f = entry["mixer"], entry.get("mlp")
        if entry["type"] == "parallel":
            a, r = m["left"], m["right"]
            temp = a.get("q_temp")
            left = AttentionSpec(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a.get("vdim", a["dim"])),
                                 scale=float(a["scale"]), linear_bias=True, qk_norm=True, key_values=True,
                                 q_temp=(float(temp["coef"]), int(temp["every"])) if temp else None)
            mixer = ParallelSpec(left, MatrixMemorySpec(heads=int(r["heads"]), dim=int(r["dim"]), vdim=int(r["vdim"]),
                                                        gate_cap=float(r["gate_cap"])))
        elif entry["type"] == "mamba1":
            mixer = SelectiveScanSpec(inner=int(m["inner"]), state=int(m["state"]), dt_rank=int(m["dt_rank"]), conv=int(m["conv"]))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
        if f is not None and f.get("kind") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
        of = entry.get("weights_of")
        layers.append(StackLayerSpec(mixer, None if f is None else DenseSpec(int(f["ff"])), None if of is None else int(of)))
    return StackConfig(name=name, architecture="Mererax", vocab_size=int(doc["vocab"]), d_model=int(doc["width"]), layers=tuple(layers),
                       embed_scale=float(doc["embedding"]["scale"]), norm_eps=float(doc["norm"]["eps"]), order="parallel", norm_add=1.0,
                       sinusoid=True, tied_head=True).validate()


def mererax_config_to_dict(cfg: StackConfig) -> Dict:
    layers = []
    for layer in cfg.layers:
        m, f = layer.mixer, layer.mlp
        if isinstance(m, ParallelSpec):
            a, r = m.left, m.right
            left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
            if a.q_temp is not None:
                left["q_temp"] = {"coef": a.q_temp[0], "every": a.q_temp[1]}
            entry = {"type": "parallel", "mixer": {"left": left, "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim,
                                                                           "gate_cap": r.gate_cap}}}
        else:
            entry = {"type": "mamba1", "mixer": {"inner": m.inner, "state": m.state, "dt_rank": m.dt_rank, "conv": m.conv}}
        entry["mlp"] = None if f is None else {"kind": "dense", "ff": f.ff}
        if layer.weights_of is not None:
            entry["weights_of"] = layer.weights_of
        layers.append(entry)
    return {"architecture": "Mererax", "vocab": cfg.vocab_size, "width": cfg.d_model, "embedding": {"scale": cfg.embed_scale},
            "norm": {"eps": cfg.norm_eps}, "layers": layers}


# architecture name in config.json -> (reader, writer)
ARCHITECTURES = {"Lederax": (lederax_config_from_dict, lederax_config_to_dict),
                 "Mererax": (mererax_config_from_dict, mererax_config_to_dict)}


def stack_config_from_dir(path) -> Optional[StackConfig]:
    """The stack config of a checkpoint directory, or None when its config.json names no architecture of this kind."""
    import json
    from pathlib import Path

    f = Path(path) / "config.json"
    if not f.is_file():
        return None
    doc = json.loads(f.read_text())
    arch = doc.get("architecture")
    return ARCHITECTURES[arch][0](doc, name=Path(path).name) if arch in ARCHITECTURES else None


def lederax_preset(name: str, d_model: int, n_layers: int, heads: int, kv_heads: int, dim: int, window: int, experts: int,
                   top: int, ff: int, vocab_size: int, norm_groups: int = 2) -> StackConfig:
    layer = StackLayerSpec(AttentionSpec(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, window=window,
                                         distance_bias=True, value_norm=True, value_mix=True, qkv_bias=True),
                           MoESpec(experts=experts, top=top, ff=ff))
    return StackConfig(name=name, architecture="Lederax", vocab_size=vocab_size, d_model=d_model, layers=(layer,) * n_layers,
                       norm_groups=norm_groups).validate()


def lederax_tiny_config(n_layers: int = 2, **kw) -> StackConfig:
    """Toy model of the CPU tests and examples (byte-level tokenizer)."""
    return replace(lederax_preset("lederax-tiny", d_model=96, n_layers=n_layers, heads=4, kv_heads=2, dim=24, window=20,
                                  experts=6, top=2, ff=40, vocab_size=300), **kw)


def lederax_8b_config(n_layers: int = 36, **kw) -> StackConfig:
    """Layers as wide as Cosmos3-Nano's Reasoner tower, with as many active parameters a layer: attention 32 / 8 heads of
    128, 4 of 32 experts of 4608 (up + down = the 3 x 12288 columns of a dense SwiGLU layer)."""
    return replace(lederax_preset("lederax-8b", d_model=4096, n_layers=n_layers, heads=32, kv_heads=8, dim=128, window=4096,
                                  experts=32, top=4, ff=4608, vocab_size=151936), **kw)


def mererax_preset(name: str, d_model: int, n_layers: int, heads: int, kv_heads: int, dim: int, mem_heads: int, mem_dim: int,
                   mem_vdim: int, inner: int, state: int, dt_rank: int, ff: int, vocab_size: int, every: int = 1024,
                   period: int = 3) -> StackConfig:
    """Scan layers with an attention / memory layer as the last of every `period`."""
    par = StackLayerSpec(ParallelSpec(AttentionSpec(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, linear_bias=True,
                                                    qk_norm=True, key_values=True, q_temp=(0.1, every)),
                                      MatrixMemorySpec(heads=mem_heads, dim=mem_dim, vdim=mem_vdim, gate_cap=15.0)), DenseSpec(ff))
    scan = StackLayerSpec(SelectiveScanSpec(inner=inner, state=state, dt_rank=dt_rank, conv=4), DenseSpec(ff))
    return StackConfig(name=name, architecture="Mererax", vocab_size=vocab_size, d_model=d_model,
                       layers=tuple(par if i % period == period - 1 else scan for i in range(n_layers)), embed_scale=d_model ** 0.5,
                       order="parallel", norm_add=1.0, sinusoid=True, tied_head=True).validate()


def mererax_tiny_config(n_layers: int = 3, **kw) -> StackConfig:
    """Toy model of the CPU tests and examples (byte-level tokenizer)."""
    return replace(mererax_preset("mererax-tiny", d_model=80, n_layers=n_layers, heads=4, kv_heads=2, dim=20, mem_heads=3, mem_dim=12,
                                  mem_vdim=28, inner=112, state=10, dt_rank=6, ff=136, vocab_size=300, every=16), **kw)


def mererax_8b_config(n_layers: int = 36, **kw) -> StackConfig:
    """Layers as wide as Cosmos3-Nano's Reasoner tower: attention 32 / 8 heads of 128 beside 8 memories of 256 x 512, scans of
    8192 channels x 16 states, SwiGLU of 12288."""
    return replace(mererax_preset("mererax-8b", d_model=4096, n_layers=n_layers, heads=32, kv_heads=8, dim=128, mem_heads=8, mem_dim=256,
                                  mem_vdim=512, inner=8192, state=16, dt_rank=256, ff=12288, vocab_size=151936), **kw)


MODEL_REGISTRY = {
    "lederax-tiny": lederax_tiny_config,
    "lederax-8b": lederax_8b_config,
    "mererax-tiny": mererax_tiny_config,
    "mererax-8b": mererax_8b_config,
    "tiny": tiny_config,
    "tiny128": tiny128_config,
    "Cosmos3-Nano": nano_config,
    "Cosmos3-Super": super_config,
    "nvidia/Cosmos3-Nano": nano_config,
    "nvidia/Cosmos3-Super": super_config,
}


def get_model_config(name: str, **kw):
    """MoTConfig (or StackConfig, for the decoder stacks) of a registered name."""
    key = name.rstrip("/").split("/")[-1] if name not in MODEL_REGISTRY else name
    if key not in MODEL_REGISTRY:
        raise KeyError(f"unknown model '{name}'; known: {sorted(MODEL_REGISTRY)}")
    return MODEL_REGISTRY[key](**kw)


# --------------------------------------------------------------------------- resolution tables
# Reference README.md:106 and inference_benchmarks.md:39: 720p = 1280x720, 480p = 832x480, 256p = 320x192.
RESOLUTIONS_16_9 = {"720": (1280, 720), "480": (832, 480), "256": (320, 192)}
ASPECT_RATIOS = ("16,9", "4,3", "1,1", "3,4", "9,16")


def resolve_size(resolution: str, aspect_ratio: str = "16,9") -> Tuple[int, int]:
    """(width, height) in pixels, multiples of 16, for a resolution tier and aspect ratio."""
    resolution = str(resolution)
    if resolution not in RESOLUTIONS_16_9:
        raise ValueError(f"resolution must be one of {sorted(RESOLUTIONS_16_9)}, got {resolution!r}")
    if aspect_ratio not in ASPECT_RATIOS:
        raise ValueError(f"aspect_ratio must be one of {ASPECT_RATIOS}, got {aspect_ratio!r}")
    w169, h169 = RESOLUTIONS_16_9[resolution]
    if aspect_ratio == "16,9":
        return w169, h169
    if aspect_ratio == "9,16":
        return h169, w169
    aw, ah = (int(v) for v in aspect_ratio.split(","))
    area = w169 * h169
    h = (area * ah / aw) ** 0.5
    w = h * aw / ah
    r16 = lambda v: max(16, int(round(v / 16)) * 16)  # noqa: E731
    return r16(w), r16(h)


def latent_shape(cfg: MoTConfig, num_frames: int, width: int, height: int) -> Tuple[int, int, int]:
    """(T, H, W) of the VAE latent for a clip (first frame alone, then groups of vae_t_compress)."""
    t = (num_frames - 1) // cfg.vae_t_compress + 1
    return t, height // cfg.vae_s_compress, width // cfg.vae_s_compress


def video_token_count(cfg: MoTConfig, num_frames: int, width: int, height: int) -> int:
    t, h, w = latent_shape(cfg, num_frames, width, height)
    return (t // cfg.patch_t) * (h // cfg.patch_hw) * (w // cfg.patch_hw)


# --------------------------------------------------------------------------- parallel layout
@dataclass
class ParallelConfig:
    """Mesh degrees; their product must equal the world size (reference README.md:321)."""
    dp_replicate: int = 1
    dp_shard: int = 1
    cp: int = 1
    cfgp: int = 1
    tp: int = 1
    cp_mode: str = "ulysses"  # or "ring"

    @property
    def world(self) -> int:
        return self.dp_replicate * self.dp_shard * self.cp * self.cfgp * self.tp

    def validate(self, world_size: int) -> None:
        for k in ("dp_replicate", "dp_shard", "cp", "cfgp", "tp"):
            if getattr(self, k) < 1:
                raise ValueError(f"{k} must be >= 1")
        if self.cfgp not in (1, 2):
            raise ValueError("cfgp must be 1 or 2 (cond / uncond branches)")
        if self.world != world_size:
            raise ValueError(f"product of parallel degrees {self.world} != world size {world_size}")
        if self.cp_mode not in ("ulysses", "ring"):
            raise ValueError("cp_mode must be 'ulysses' or 'ring'")


def preset_parallelism(preset: str, world_size: int, use_cfg: bool = True, n_kv_heads: int = 8) -> ParallelConfig:
    """`latency`: all GPUs on one sample (CFG-parallel x context-parallel).
    `throughput`: replicate the model and give each replica its own samples
    (reference: cookbooks/cosmos3/generator/transfer/README.md:51,
    audiovisual/run_with_cosmos_framework.ipynb:529-533)."""
    if preset == "throughput":
        return ParallelConfig(dp_replicate=world_size)
    if preset != "latency":
        raise ValueError("parallelism preset must be 'latency' or 'throughput'")
    cfgp = 2 if (use_cfg and world_size % 2 == 0 and world_size >= 2) else 1
    cp = world_size // cfgp
    mode = "ulysses" if cp <= n_kv_heads and n_kv_heads % cp == 0 else "ring"
    return ParallelConfig(cp=cp, cfgp=cfgp, cp_mode=mode)


# --------------------------------------------------------------------------- sampling recipe
@dataclass
class SamplingConfig:
    """Generator defaults (reference README.md:249-263; audiovisual/README.md:43-48)."""
    num_steps: int = 35
    guidance: float = 6.0
    shift: float = 10.0
    sigma_max: Optional[float] = None
    guidance_interval: Tuple[float, float] = (0.0, 1000.0)
    normalize_cfg: bool = False
    control_guidance: Optional[float] = None
    scheduler: str = "euler"  # or "unipc"
    seed: int = 0


@dataclass
class DecodingConfig:
    """Reasoner decoding defaults (reference README.md:159-167)."""
    max_new_tokens: int = 4096
    do_sample: bool = True
    temperature: float = 0.7
    top_p: float = 0.8
    top_k: int = 20
    repetition_penalty: float = 1.0
    presence_penalty: float = 1.5
    seed: Optional[int] = None
