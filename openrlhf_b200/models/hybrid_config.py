"""Configuration of hybrid decoders: a list of layers, each with its own kind of sequence mixer, its own sizes and its
own feed-forward. ``HybridConfig`` is the framework's description; a design that is published under a name has a reader
and a writer for its ``config.json`` here (``READERS``) and an entry in ``models/registry.py``."""
from __future__ import annotations

import dataclasses
import json
import os
from dataclasses import dataclass, field


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


COLS = 32     # a fused matrix's segments start on multiples of this many rows / columns (one GEMM epilogue chunk)


@dataclass(frozen=True)
class Mamba2Spec:
    """State-space-duality mixer: `heads` states of [state, vdim], B and C shared by heads / groups heads, a causal
    convolution of `conv` taps over x, B and C, a gated RMS norm in `norm_groups` parts."""
    heads: int
    vdim: int
    state: int
    groups: int = 1
    conv: int = 4
    norm_groups: int = 1

    def __post_init__(self):
        if self.heads % self.groups or self.inner % self.norm_groups:
            raise ValueError(f"heads must be a multiple of groups and inner of norm_groups: {self}")

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    @property
    def in_rows(self) -> int:
        return self.inner + self.conv_channels + self.heads

    @property
    def out_cols(self) -> int:
        return self.inner


@dataclass(frozen=True)
class AttentionSpec:
    """Grouped-query attention with partial rotary embedding, an optional sliding window that keeps the first tokens,
    an optional sink and, with `kv_from`, the keys and values of an earlier layer."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int | None = None            # visible keys of the window, the query's own included; None: all earlier ones
    keep_first: int = 0                  # tokens at the start of a sequence that stay visible outside the window
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_factor: float = 1.0              # every frequency is divided by this
    sink: bool = False                   # one is added to the softmax denominator
    kv_from: int | None = None

    def __post_init__(self):
        if self.heads % self.kv_heads or self.rot_dims % 2 or self.rot_dims > self.dim:
            raise ValueError(f"inconsistent attention sizes: {self}")

    @property
    def in_rows(self) -> int:
        kv = 0 if self.kv_from is not None else self.kv_heads * (self.dim + self.vdim)
        return self.heads * self.dim + kv

    @property
    def out_cols(self) -> int:
        return self.heads * self.vdim

    @property
    def k_ld(self) -> int:               # cache rows: a whole number of 16-byte vectors
        return _up(self.dim, 8)

    @property
    def v_ld(self) -> int:
        return _up(self.vdim, 8)

    def span(self, max_len: int) -> int:
        return max_len if self.window is None else self.window


@dataclass(frozen=True)
class MlpSpec:
    ff: int
    activation: str = "relu2"            # square of relu, no gate


@dataclass(frozen=True)
class LayerSpec:
    mixer: Mamba2Spec | AttentionSpec
    mlp: MlpSpec | None = None

    # the layer's two fused matrices: w1 = [mixer input rows | feed-forward rows] reads the shared norm, w2 = [mixer
    # output columns | feed-forward columns] adds to the residual; every segment is padded to COLS
    @property
    def in_pad(self) -> int:
        return _up(self.mixer.in_rows, COLS)

    @property
    def out_pad(self) -> int:
        return _up(self.mixer.out_cols, COLS)

    @property
    def ff_pad(self) -> int:
        return 0 if self.mlp is None else _up(self.mlp.ff, COLS)


@dataclass
class HybridConfig:
    model_type: str = "sigisun"
    vocab_size: int = 0
    hidden_size: int = 0
    layers: tuple = ()
    norm_eps: float = 1e-6
    logit_softcap: float | None = None
    max_position_embeddings: int = 1 << 20
    pad_token_id: int = 0
    eos_token_id: int = -1               # no token unless a config.json names one
    bos_token_id: int = -1
    extra: dict = field(default_factory=dict)

    # what code that handles any model asks about
    vision = None
    num_experts = 0
    tie_word_embeddings = False
    value_head_prefix = "score"

    def __post_init__(self):
        self.layers = tuple(self.layers)
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if isinstance(m, AttentionSpec) and m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if not isinstance(src, AttentionSpec) or src.kv_from is not None or \
                        (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                    raise ValueError(f"layer {i} cannot read the keys and values of layer {m.kv_from}")

    @property
    def is_vlm(self) -> bool:
        return False

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def width_pad(self) -> int:
        return _up(self.hidden_size, 8)

    @property
    def vocab_pad(self) -> int:
        return _up(self.vocab_size, 8)

    @property
    def has_recurrent_state(self) -> bool:
        return any(isinstance(layer.mixer, Mamba2Spec) for layer in self.layers)

    def num_params(self) -> int:
        n = 2 * self.vocab_size * self.hidden_size + self.hidden_size
        for layer in self.layers:
            m = layer.mixer
            n += self.hidden_size * (1 + m.in_rows + m.out_cols)
            if isinstance(m, Mamba2Spec):
                n += m.conv_channels * (m.conv + 1) + 3 * m.heads + m.inner
            if layer.mlp is not None:
                n += 2 * self.hidden_size * layer.mlp.ff
        return n

    # ------------------------------------------------------------------ checkpoint layout
    def checkpoint_names(self, name: str) -> list[tuple[str, tuple | None]]:
        """Internal parameter -> [(checkpoint tensor, selector of its place in the parameter)]."""
        W = self.hidden_size
        if name == "embed.weight":
            return [("embed", ("block", 0, self.vocab_size, 0, W))]
        if name == "lm_head.weight":
            return [("head", ("block", 0, self.vocab_size, 0, W))]
        if name == "norm.weight":
            return [("final.norm", ("rows", 0, W))]
        _, li, rest = name.split(".", 2)
        layer, pre = self.layers[int(li)], f"l{li}."
        m = layer.mixer
        if rest == "norm1.weight":
            return [(pre + "norm1", ("rows", 0, W))]
        if rest == "w1.weight":
            if isinstance(m, Mamba2Spec):
                out = [(pre + "mix.in", ("block", 0, m.in_rows, 0, W))]
            else:
                q, kd = m.heads * m.dim, m.kv_heads * m.dim
                out = [(pre + "mix.q", ("block", 0, q, 0, W))]
                if m.kv_from is None:
                    out += [(pre + "mix.k", ("block", q, q + kd, 0, W)),
                            (pre + "mix.v", ("block", q + kd, q + kd + m.kv_heads * m.vdim, 0, W))]
            if layer.mlp is not None:
                out.append((pre + "mlp.up", ("block", layer.in_pad, layer.in_pad + layer.mlp.ff, 0, W)))
            return out
        if rest == "w2.weight":
            out = [(pre + "mix.o", ("block", 0, W, 0, m.out_cols))]
            if layer.mlp is not None:
                out.append((pre + "mlp.down", ("block", 0, W, layer.out_pad, layer.out_pad + layer.mlp.ff)))
            return out
        simple = {"conv.weight": "mix.conv", "conv.bias": "mix.conv.b", "dt_bias": "mix.dt_bias", "A_log": "mix.A_log",
                  "D": "mix.D", "gate_norm.weight": "mix.norm"}
        return [(pre + simple[rest], None)]

    # ------------------------------------------------------------------ config.json
    @classmethod
    def from_dict(cls, d: dict) -> "HybridConfig":
        return READERS[d["architecture"]](d)

    def to_dict(self) -> dict:
        return WRITERS[self.model_type](self)

    @classmethod
    def from_pretrained(cls, path: str) -> "HybridConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))

    def save_pretrained(self, path: str, extra: dict | None = None) -> None:
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump({**self.to_dict(), **(extra or {})}, f, indent=1)


# ---------------------------------------------------------------------------------------------- Sigisun
# Parallel layers (mixer and feed-forward read one norm), Mamba-2 and windowed attention in any order; attention has a
# zero-score sink and may share an earlier layer's keys and values; capped logits.
_SIGISUN_KEYS = ("architecture", "layers", "vocab", "width", "norm", "logit_softcap")
_TOKEN_KEYS = ("pad_token_id", "eos_token_id", "bos_token_id", "max_position_embeddings")


def _sigisun_mixer(kind: str, m: dict):
    if kind == "mamba2":
        return Mamba2Spec(heads=m["heads"], vdim=m["vdim"], state=m["state"], groups=m["groups"], conv=m["conv"],
                          norm_groups=m["norm_groups"])
    if kind != "attention":
        raise ValueError(f"unknown mixer type {kind!r}")
    mask, rot = m.get("mask") or {}, m.get("rot") or {}
    return AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"],
                         window=mask.get("size"), keep_first=mask.get("keep_first", 0), rot_dims=rot.get("dims", 0),
                         rot_base=rot.get("base", 10000.0), rot_factor=(rot.get("scaling") or {}).get("factor", 1.0),
                         sink=True, kv_from=m.get("kv_from"))


def read_sigisun(d: dict) -> HybridConfig:
    layers = []
    for e in d["layers"]:
        mlp = e.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        layers.append(LayerSpec(_sigisun_mixer(e["type"], e["mixer"]), None if mlp is None else MlpSpec(mlp["ff"])))
    return HybridConfig("sigisun", d["vocab"], d["width"], tuple(layers), norm_eps=d["norm"]["eps"],
                        logit_softcap=d.get("logit_softcap"), **{k: d[k] for k in _TOKEN_KEYS if d.get(k) is not None},
                        extra={k: v for k, v in d.items() if k not in _SIGISUN_KEYS + _TOKEN_KEYS})


def write_sigisun(c: HybridConfig) -> dict:
    layers = []
    for layer in c.layers:
        m = layer.mixer
        if isinstance(m, Mamba2Spec):
            kind, mixer = "mamba2", dataclasses.asdict(m)
        else:
            kind = "attention"
            mixer = {"dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads, "vdim": m.vdim, "scale": m.scale}
            if m.window is not None:
                mixer["mask"] = {"size": m.window, "keep_first": m.keep_first}
            if m.rot_dims:
                mixer["rot"] = {"base": m.rot_base, "dims": m.rot_dims, "scaling": {"factor": m.rot_factor}}
            if m.kv_from is not None:
                mixer["kv_from"] = m.kv_from
        mlp = None if layer.mlp is None else {"ff": layer.mlp.ff, "kind": "dense"}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    d = dict(c.extra)
    d.update({"architecture": "Sigisun", "layers": layers, "logit_softcap": c.logit_softcap,
              "norm": {"eps": c.norm_eps}, "vocab": c.vocab_size, "width": c.hidden_size})
    for k, default in (("pad_token_id", 0), ("eos_token_id", -1), ("bos_token_id", -1),
                       ("max_position_embeddings", 1 << 20)):
        if getattr(c, k) != default:
            d[k] = getattr(c, k)
    return d


READERS = {"Sigisun": read_sigisun}
WRITERS = {"sigisun": write_sigisun}


def sigisun_preset(width: int, n_layers: int, heads: int, vdim: int, state: int, groups: int, q_heads: int,
                   kv_heads: int, dim: int, window: int, keep: int, ff: int, vocab: int) -> HybridConfig:
    """A model-sized instance: two Mamba-2 layers, then one attention layer, repeated; every second attention layer
    reads the keys and values of the one before it."""
    layers, last = [], None
    for i in range(n_layers):
        if i % 3 != 2:
            mixer = Mamba2Spec(heads, vdim, state, groups, 4, groups)
        else:
            share = last if (i // 3) % 2 == 1 else None
            mixer = AttentionSpec(q_heads, kv_heads, dim, dim, dim ** -0.5, window, keep, dim // 2, 10000.0, 4.0, True, share)
            last = i if share is None else None
        layers.append(LayerSpec(mixer, MlpSpec(ff)))
    return HybridConfig("sigisun", vocab, width, tuple(layers), norm_eps=1e-6, logit_softcap=30.0)
