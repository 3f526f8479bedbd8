"""Configuration of the Nidilix decoder: every size and constant comes from ``config.json``."""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ...ops.latent_attention import LatentShape
from ...ops.moe import Router
from ...ops.recurrent import GatedScanShape
from ..packed_decoder import round_up
from ..seq_table import StateTensor


@dataclass
class LatentMixer:
    shape: LatentShape
    scale: float
    rot_base: float | None          # None = no rotation
    kv_from: int | None = None      # layer whose cache this one reads; None = its own

    @classmethod
    def from_dict(cls, d: dict) -> "LatentMixer":
        rot = d.get("rot")
        m = cls(LatentShape(int(d["heads"]), int(d["dim"]), int(d["rot_dim"]), int(d["vdim"]), int(d["kv_rank"])),
                float(d["scale"]), None if rot is None else float(rot["base"]),
                None if d.get("kv_from") is None else int(d["kv_from"]))
        if m.shape.rot % 2:
            raise ValueError(f"rot_dim must be even, got {m.shape.rot}")
        if rot is not None and int(rot.get("dims", m.shape.rot)) != m.shape.rot:
            raise ValueError(f"rot.dims ({rot['dims']}) must equal rot_dim ({m.shape.rot})")
        return m


@dataclass
class ScanMixer:
    shape: GatedScanShape

    @classmethod
    def from_dict(cls, d: dict) -> "ScanMixer":
        width, blocks = int(d["width"]), int(d["blocks"])
        if width % blocks:
            raise ValueError(f"mixer width ({width}) must be a multiple of blocks ({blocks})")
        return cls(GatedScanShape(width, blocks, int(d["conv"])))


@dataclass
class ExpertsConfig:
    experts: int
    top: int
    ff: int
    shared_ff: int | None = None    # None = no shared expert

    @classmethod
    def from_dict(cls, d: dict) -> "ExpertsConfig":
        if d.get("kind", "moe") != "moe":
            raise ValueError(f"unknown feed-forward kind {d['kind']!r}")
        m = cls(int(d["router"]["experts"]), int(d["router"]["top"]), int(d["expert"]["ff"]),
                int(d["shared"]["ff"]) if d.get("shared") else None)
        m.router                        # refuses a choice that cannot be made
        return m

    @property
    def router(self) -> Router:
        return Router(self.experts, self.top)


@dataclass
class LayerConfig:
    mixer: LatentMixer | ScanMixer
    mlp: ExpertsConfig | None = None


_MIXERS = {"latent_attention": LatentMixer, "rglru": ScanMixer}


@dataclass
class NidilixConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    residual_mult: float
    side_dim: int = 0               # channels per layer of the token table, 0 = none
    layers: list[LayerConfig] = field(default_factory=list)

    # what the engine reads from any decoder configuration
    mrope_section = None

    @classmethod
    def from_dict(cls, d: dict) -> "NidilixConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] not in _MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            mixer = _MIXERS[e["type"]].from_dict(e["mixer"])
            src = getattr(mixer, "kv_from", None)
            if src is not None:
                own = layers[src].mixer if 0 <= src < i else None
                if not isinstance(own, LatentMixer) or own.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from {src} is not an earlier layer with a latent of its own")
                if (own.shape.rank, own.shape.rot, own.rot_base) != (mixer.shape.rank, mixer.shape.rot, mixer.rot_base):
                    raise ValueError(f"layer {i}: latent size and rotation differ from layer {src}'s")
            layers.append(LayerConfig(mixer, None if e.get("mlp") is None else ExpertsConfig.from_dict(e["mlp"])))
        side = d.get("token_side")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["residual_mult"]),
                   int(side["dim"]) if side else 0, layers)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def padded_width(self) -> int:
        return round_up(self.hidden_size, 8)

    def _mlp_max(self, f) -> int:
        return max((f(l.mlp) for l in self.layers if l.mlp is not None), default=0)

    @property
    def num_experts(self) -> int:
        return self._mlp_max(lambda m: m.experts)

    @property
    def num_experts_per_tok(self) -> int:
        return self._mlp_max(lambda m: m.top)

    @property
    def moe_intermediate_size(self) -> int:
        return self._mlp_max(lambda m: m.ff)

    @property
    def intermediate_size(self) -> int:
        return self._mlp_max(lambda m: m.shared_ff or 0)

    def kv_layer_shapes(self) -> list[tuple[int, int, int]]:
        """(heads, key channels, value channels) of every layer's pages: one row of latent and rotated key part, whose
        first channels are also the value; nothing for recurrent layers and those that read another layer's pages."""
        return [(1, l.mixer.shape.row, 0) if isinstance(l.mixer, LatentMixer) and l.mixer.kv_from is None else (0, 0, 0)
                for l in self.layers]

    def state_shapes(self) -> list[tuple[StateTensor, ...]]:
        """Per layer: what one sequence carries besides its pages (convolution history, recurrent state)."""
        out = []
        for l in self.layers:
            if isinstance(l.mixer, ScanMixer):
                s = l.mixer.shape
                out.append((StateTensor((s.taps - 1, s.channels)), StateTensor((s.channels,), torch.float32)))
            else:
                out.append(())
        return out

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Checkpoint tensor names and shapes."""
        D = self.hidden_size
        t: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, D), "head": (self.vocab_size, D)}

        def norm(name):
            t[name], t[name + ".b"], t[name + ".alpha"] = (D,), (D,), ()
        norm("final.norm")
        if self.side_dim:
            t["side.embed"] = (self.vocab_size, self.side_dim * len(self.layers))
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            norm(p + "norm1")
            s = l.mixer.shape
            if isinstance(l.mixer, LatentMixer):
                t[p + "mix.q"] = (s.heads * (s.dim + s.rot), D)
                if l.mixer.kv_from is None:
                    t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = (s.rank + s.rot, D), (s.rank,)
                t[p + "mix.uk"], t[p + "mix.uv"] = (s.heads * s.dim, s.rank), (s.heads * s.vdim, s.rank)
                t[p + "mix.g"], t[p + "mix.o"] = (s.heads, D), (D, s.heads * s.vdim)
            else:
                for n in "yx":
                    t[f"{p}mix.{n}"], t[f"{p}mix.{n}.b"] = (s.width, D), (s.width,)
                t[p + "mix.conv"], t[p + "mix.conv.b"] = (s.width, s.taps), (s.width,)
                for n in ("ra", "ri"):
                    t[f"{p}mix.{n}"], t[f"{p}mix.{n}.b"] = (s.blocks, s.part, s.part), (s.blocks, s.part)
                t[p + "mix.lam"], t[p + "mix.o"] = (s.width,), (D, s.width)
            if l.mlp is not None:
                m = l.mlp
                norm(p + "norm2")
                t[p + "mlp.router"], t[p + "mlp.router.b"] = (m.experts, D), (m.experts,)
                for e, ff in [(f"e{j}", m.ff) for j in range(m.experts)] + ([("shared", m.shared_ff)] if m.shared_ff else []):
                    t[f"{p}mlp.{e}.up"], t[f"{p}mlp.{e}.down"] = (ff, D), (D, ff)
            if self.side_dim:
                t[p + "side.gate"], t[p + "side.proj"], t[p + "side.norm"] = (self.side_dim, D), (D, self.side_dim), (D,)
        return t


def tiny_config_dict(**over) -> dict:
    """A small geometry for tests and smoke runs; no two sizes are equal."""
    mlp = {"kind": "moe", "expert": {"ff": 56}, "router": {"experts": 6, "top": 3}, "shared": {"ff": 88}}

    def attention(**kw):
        return {"type": "latent_attention", "mlp": mlp,
                "mixer": {"heads": 3, "dim": 24, "rot_dim": 12, "vdim": 40, "kv_rank": 48, "scale": 0.17,
                          "rot": {"base": 10000.0, "dims": 12}, **kw}}
    scan = {"type": "rglru", "mlp": mlp, "mixer": {"width": 144, "blocks": 4, "conv": 4}}
    d = {"architecture": "Nidilix", "vocab": 300, "width": 104, "norm": {"eps": 1e-5}, "residual_mult": 0.4,
         "token_side": {"dim": 20}, "layers": [attention(), scan, attention(kv_from=0, heads=5), scan]}
    d.update(over)
    return d
