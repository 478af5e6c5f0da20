"""PugalixConfig: the typed form of a Pugalix config.json.

The design stacks three kinds of pre-norm layers, each with sizes of its own: softmax attention with a sliding window
that keeps the sequence's first tokens in sight (biases on q, k and v, interleaved rotary positions, a one in the
softmax's denominator, a gate on every element of the heads' output; a layer may read another layer's keys and values),
gated linear attention (a matrix state per head that fades by one factor per key channel and token), and a matrix memory
(mLSTM).  A layer's gated feed-forward is optional.  Keys: `vocab`, `width`, `embedding.scale`, `norm.eps`,
`layers[i].{type, mixer, mlp}`; core/pugalix.cpp lists them all.

Reading, type checks and validation are the host library's (core/pugalix.cpp, PugalixConfig); this dataclass
carries the result.  Its layer records stay plain dictionaries, as config.json writes them.
"""
from __future__ import annotations

import dataclasses
from typing import Any, Dict, List

from .. import core
from .base import ModelConfig


@dataclasses.dataclass(frozen=True)
class PugalixConfig(ModelConfig):
    architecture = "Pugalix"

    vocab: int = 0
    width: int = 0
    embedding: Dict[str, Any] = dataclasses.field(default_factory=lambda: {"scale": 1.0})
    norm: Dict[str, Any] = dataclasses.field(default_factory=lambda: {"eps": 1e-6})
    layers: List[Dict[str, Any]] = dataclasses.field(default_factory=list)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "PugalixConfig":
        """Type checks only; `validate` checks the sizes against one another."""
        n = core.call("global", None, "parse_config", config=raw, architecture=cls.architecture, validate=False)
        names = {f.name for f in dataclasses.fields(cls)}
        return cls(**{k: v for k, v in n.items() if k in names})

    def to_dict(self) -> Dict[str, Any]:
        d = dataclasses.asdict(self)
        d["architecture"] = self.architecture
        return d

    def validate(self) -> None:
        core.call("global", None, "parse_config", config=self.to_dict(), architecture=self.architecture, validate=True)
