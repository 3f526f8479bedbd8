"""Configuration of the Tavulix decoder: every size and constant comes from ``config.json``."""
from __future__ import annotations

from dataclasses import dataclass, field

from ...ops.lm import HeadShape
from ..packed_decoder import round_up as _up
from ..seq_table import StateTensor


@dataclass
class MixerConfig:
    heads: int
    kv_heads: int
    dim: int                        # query / key channels per head
    vdim: int                       # value channels per head
    scale: float
    softcap: float | None = None
    conv: int = 0                   # taps of the short convolution, 0 = none
    window: int | None = None
    keep_first: int = 0
    v_mix: bool = False

    @classmethod
    def from_dict(cls, d: dict) -> "MixerConfig":
        mask = d.get("mask") or {}
        m = cls(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"]),
                None if d.get("softcap") is None else float(d["softcap"]), int(d.get("conv") or 0),
                None if mask.get("size") is None else int(mask["size"]), int(mask.get("keep_first") or 0),
                bool(d.get("v_mix", False)))
        if m.heads % m.kv_heads:
            raise ValueError(f"heads ({m.heads}) must be a multiple of kv_heads ({m.kv_heads})")
        if m.window is not None and m.window < 1:
            raise ValueError(f"mask.size must be at least 1, got {m.window}")
        return m

    @property
    def head_shape(self) -> HeadShape:
        return HeadShape(self.heads, self.kv_heads, self.dim, self.vdim, _up(self.dim, 16), _up(self.vdim, 16), self.conv)


@dataclass
class LayerConfig:
    mixer: MixerConfig
    ff: int | None = None           # hidden width of the feed-forward, None = the layer has none


@dataclass
class TavulixConfig:
    vocab_size: int
    hidden_size: int
    max_position_embeddings: int
    norm_eps: float
    logit_softcap: float | None
    layers: list[LayerConfig] = field(default_factory=list)

    # what the engine reads from any decoder configuration
    num_experts = 0
    num_experts_per_tok = 0
    moe_intermediate_size = 0
    mrope_section = None

    @classmethod
    def from_dict(cls, d: dict) -> "TavulixConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e.get("type", "attention") != "attention":
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            layers.append(LayerConfig(MixerConfig.from_dict(e["mixer"]), None if mlp is None else int(mlp["ff"])))
        cap = d.get("logit_softcap")
        cfg = cls(int(d["vocab"]), int(d["width"]), int(d["max_positions"]), float(d["norm"]["eps"]),
                  None if cap is None else float(cap), layers)
        mixed = {(l.mixer.kv_heads, l.mixer.vdim) for l in layers if l.mixer.v_mix}
        if len(mixed) > 1:
            raise ValueError("layers that mix values must agree on kv_heads and vdim")
        return cfg

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def padded_width(self) -> int:
        return _up(self.hidden_size, 8)

    @property
    def intermediate_size(self) -> int:
        return max((l.ff or 0 for l in self.layers), default=0)

    @property
    def max_positions(self) -> int:
        """Hard limit of a sequence's length: the rows of the learned position table."""
        return self.max_position_embeddings

    def kv_layer_shapes(self) -> list[tuple[int, int, int]]:
        """(KV heads, key channels, value channels) of every layer's pages."""
        hs = [l.mixer.head_shape for l in self.layers]
        return [(h.kv_heads, h.dp, h.vp) for h in hs]

    def state_shapes(self) -> list[tuple[StateTensor, ...]]:
        """Per layer: what one sequence carries besides its pages."""
        hs = [l.mixer.head_shape for l in self.layers]
        return [(StateTensor((h.taps - 1, h.channels)),) if h.taps > 1 else () for h in hs]

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Checkpoint tensor names and shapes."""
        D = self.hidden_size
        t: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, D), "pos": (self.max_position_embeddings, D)}
        for i, l in enumerate(self.layers):
            p, m = f"l{i}.", l.mixer
            rows = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
            for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l.ff is not None else ()):
                t[p + n] = ()
            for n, r in rows.items():
                t[f"{p}mix.{n}"] = (r, D)
                if m.conv:
                    t[f"{p}mix.{n}.conv"] = (r, m.conv)
            t[p + "mix.q.norm"] = t[p + "mix.k.norm"] = (m.dim,)
            if m.v_mix:
                t[p + "mix.vmix"] = ()
            for n in ("r1", "r2", "sink"):
                t[f"{p}mix.{n}"] = (m.heads,)
            t[p + "mix.g"] = (m.heads, D)
            t[p + "mix.o"] = (D, m.heads * m.vdim)
            if l.ff is not None:
                t[p + "mlp.up"], t[p + "mlp.down"], t[p + "mlp.act"] = (l.ff, D), (D, l.ff), (4,)
        t["final.norm"], t["head"] = (), (self.vocab_size, D)
        return t


def tiny_config_dict(**over) -> dict:
    """A small geometry for tests and smoke runs; no two sizes are equal."""
    def layer(window, keep, heads=6, kv=2, ff=160, mix=True):
        return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
                "mixer": {"heads": heads, "kv_heads": kv, "dim": 40, "vdim": 24, "conv": 4, "scale": 0.2, "softcap": 12.0,
                          "v_mix": mix, "mask": {"size": window, "keep_first": keep}}}
    d = {"architecture": "Tavulix", "vocab": 300, "width": 104, "max_positions": 1024, "norm": {"eps": 1e-5},
         "logit_softcap": 25.0, "layers": [layer(33, 5), layer(50, 3, heads=4), layer(20, 0, ff=None)]}
    d.update(over)
    return d
