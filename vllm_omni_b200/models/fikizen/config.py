"""Configuration of the Fikizen decoder: sizes and constants come from ``config.json``, except the rank of the decay's
low-rank projection, which the checkpoint's tensors tell."""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ...ops.delta_rule import DeltaShape
from ...ops.lm import HeadShape
from ..packed_decoder import round_up
from ..seq_table import StateTensor


@dataclass
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int                        # query / key channels per head
    vdim: int                       # value channels per head
    scale: float
    window: int
    rot_base: float
    rot_dims: int                   # rotated channels of a head, the first ones

    @classmethod
    def from_dict(cls, d: dict) -> "AttentionMixer":
        m = cls(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"]), int(d["mask"]["size"]),
                float(d["rot"]["base"]), int(d["rot"]["dims"]))
        if m.heads % m.kv_heads:
            raise ValueError(f"heads ({m.heads}) must be a multiple of kv_heads ({m.kv_heads})")
        if m.window < 1:
            raise ValueError(f"mask.size must be at least 1, got {m.window}")
        if m.rot_dims % 2 or not 0 <= m.rot_dims <= m.dim:
            raise ValueError(f"rot.dims must be even and at most {m.dim}, got {m.rot_dims}")
        return m

    @property
    def head_shape(self) -> HeadShape:
        return HeadShape(self.heads, self.kv_heads, self.dim, self.vdim, round_up(self.dim, 16), round_up(self.vdim, 16))


def _delta_shape(d: dict) -> DeltaShape:
    s = DeltaShape(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), int(d["conv"]))
    if s.heads % s.kv_heads:
        raise ValueError(f"heads ({s.heads}) must be a multiple of kv_heads ({s.kv_heads})")
    if s.taps < 1:
        raise ValueError(f"conv must be at least 1, got {s.taps}")
    return s


@dataclass
class DeltaMixer:
    shape: DeltaShape

    @classmethod
    def from_dict(cls, d: dict) -> "DeltaMixer":
        return cls(_delta_shape(d))


@dataclass
class ParallelMixer:
    left: AttentionMixer
    right: DeltaShape
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d: dict) -> "ParallelMixer":
        r = d["right"]
        n, c = int(r["heads"]), int(r["dim"])
        return cls(AttentionMixer.from_dict(d["left"]), DeltaShape(n, n, c, c), float(d["left_scale"]), float(d["right_scale"]))


@dataclass
class LayerConfig:
    mixer: AttentionMixer | DeltaMixer | ParallelMixer
    ff: int | None = None           # hidden width of the feed-forward, None = the layer has none
    owner: int = 0                  # layer whose weights this one uses


_MIXERS = {"attention": AttentionMixer, "delta": DeltaMixer, "parallel": ParallelMixer}


@dataclass
class FikizenConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    logit_softcap: float | None
    layers: list[LayerConfig] = field(default_factory=list)

    # what the engine reads from any decoder configuration
    num_experts = 0
    num_experts_per_tok = 0
    moe_intermediate_size = 0
    mrope_section = None

    @classmethod
    def from_dict(cls, d: dict) -> "FikizenConfig":
        layers, entries = [], d["layers"]
        for i, e in enumerate(entries):
            if e["type"] not in _MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            owner = e.get("weights_of")
            layers.append(LayerConfig(_MIXERS[e["type"]].from_dict(e["mixer"]), None if mlp is None else int(mlp["ff"]),
                                      i if owner is None else int(owner)))
        for i, l in enumerate(layers):
            own = layers[l.owner] if 0 <= l.owner < len(layers) else None
            if own is None or own.owner != l.owner:
                raise ValueError(f"layer {i}: weights_of {l.owner} is not a layer with weights of its own")
            if (own.mixer, own.ff) != (l.mixer, l.ff):
                raise ValueError(f"layer {i}: differs from layer {l.owner}, whose weights it uses")
        cap = d.get("logit_softcap")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), None if cap is None else float(cap), layers)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def padded_width(self) -> int:
        return round_up(self.hidden_size, 8)

    @property
    def intermediate_size(self) -> int:
        return max((l.ff or 0 for l in self.layers), default=0)

    def kv_layer_shapes(self) -> list[tuple[int, int, int]]:
        """(KV heads, key channels, value channels) of every layer's pages; nothing for recurrences."""
        out = []
        for l in self.layers:
            m = l.mixer.left if isinstance(l.mixer, ParallelMixer) else l.mixer
            hs = None if isinstance(m, DeltaMixer) else m.head_shape
            out.append((0, 0, 0) if hs is None else (hs.kv_heads, hs.dp, hs.vp))
        return out

    def state_shapes(self) -> list[tuple[StateTensor, ...]]:
        """Per layer: what one sequence carries besides its pages (recurrent state, convolution history)."""
        out = []
        for l in self.layers:
            m = l.mixer
            if isinstance(m, AttentionMixer):
                out.append(())
                continue
            s = m.right if isinstance(m, ParallelMixer) else m.shape
            state = StateTensor((s.heads, s.dp, s.vp), torch.float32)
            out.append((state, StateTensor((s.taps - 1, s.channels))) if s.taps > 1 else (state,))
        return out

    def tensor_shapes(self) -> dict[str, tuple[int | None, ...]]:
        """Checkpoint tensor names and shapes; None where the checkpoint decides."""
        D = self.hidden_size
        t: dict[str, tuple[int | None, ...]] = {"embed": (self.vocab_size, D), "final.norm": (D,), "head": (self.vocab_size, D)}

        def attention(p: str, m: AttentionMixer) -> dict[str, int]:
            rows = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
            t.update({p + n: (r, D) for n, r in rows.items()})
            t[p + "o"] = (D, m.heads * m.vdim)
            return rows

        for i, l in enumerate(self.layers):
            if l.owner != i:
                continue
            p, m = f"l{i}.mix.", l.mixer
            t[f"l{i}.norm1"] = (D,)
            if isinstance(m, AttentionMixer):
                attention(p, m)
                t[p + "g"] = (m.heads, D)
            elif isinstance(m, ParallelMixer):
                rows = attention(p + "left.", m.left)
                t.update({f"{p}left.{n}.b": (r,) for n, r in rows.items()})
                t.update({f"{p}left.{n}.norm": (rows[n],) for n in "qk"})
                p, c = p + "right.", m.right.heads * m.right.dim
                t.update({p + n: (c, D) for n in "rkvag"})
                t.update({p + n: (c,) for n in ("a.b", "w0", "norm")})
                t[p + "w1"], t[p + "w2"], t[p + "o"] = (None, D), (c, None), (D, c)
            else:
                s = m.shape
                rows = {"q": s.kv_heads * s.dim, "k": s.kv_heads * s.dim, "v": s.heads * s.vdim}
                for n, r in rows.items():
                    t[p + n], t[f"{p}{n}.conv"] = (r, D), (r, s.taps)
                t.update({p + n: (s.heads, D) for n in "ab"})
                t.update({p + n: (s.heads,) for n in ("A_log", "dt_bias")})
                t[p + "norm"], t[p + "g"], t[p + "o"] = (s.vdim,), (rows["v"], D), (D, rows["v"])
            if l.ff is not None:
                p = f"l{i}.mlp."
                t[f"l{i}.norm2"], t[p + "up"], t[p + "down"], t[p + "act"] = (D,), (l.ff, D), (D, l.ff), (2,)
        return t


def tiny_config_dict(**over) -> dict:
    """A small geometry for tests and smoke runs; no two sizes are equal."""
    def attention(heads, kv, dim, vdim, window, rot):
        return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5, "mask": {"size": window},
                "rot": {"base": 10000.0, "dims": rot}}
    layers = [{"type": "attention", "mlp": {"kind": "dense", "ff": 136}, "mixer": attention(6, 2, 40, 24, 33, 12)},
              {"type": "delta", "mlp": {"kind": "dense", "ff": 88}, "mixer": {"heads": 4, "kv_heads": 2, "dim": 20, "vdim": 28, "conv": 3}},
              {"type": "parallel", "mlp": None, "mixer": {"left": attention(3, 1, 32, 48, 20, 16), "left_scale": 0.9,
                                                          "right": {"heads": 5, "dim": 18}, "right_scale": 0.7}}]
    layers.append(dict(layers[0], weights_of=0))
    d = {"architecture": "Fikizen", "vocab": 300, "width": 104, "norm": {"eps": 1e-5}, "logit_softcap": 20.0, "layers": layers}
    d.update(over)
    return d
