"""MigelixConfig: the typed form of a Migelix config.json.

The design stacks three kinds of pre-norm layers, each with sizes of its own: time mixing (a token shift with a mix for every
projection, a decay per key channel that depends on the input, a bonus for the current token), softmax attention in a sliding
window (values that are the keys before the rotation, capped scores, a gate on every element of the heads' output), and such an
attention (with biases, YaRN's rotation and a learned sink) beside a delta rule with a decay per key channel.  A layer may use
another's tensors with a cache or state of its own; a layer's gated feed-forward is optional.  Keys: `vocab`, `width`,
`norm.eps`, `logit_softcap`, `layers[i].{type, mixer, mlp, weights_of}`; core/migelix.cpp lists them all.

Reading, type checks and validation are the host library's (core/migelix.cpp, MigelixConfig); this dataclass
carries the result.  Its layer records stay plain dictionaries, as config.json writes them.
"""
from __future__ import annotations

import dataclasses
from typing import Any, Dict, List

from .. import core
from .base import ModelConfig


@dataclasses.dataclass(frozen=True)
class MigelixConfig(ModelConfig):
    architecture = "Migelix"

    vocab: int = 0
    width: int = 0
    norm: Dict[str, Any] = dataclasses.field(default_factory=lambda: {"eps": 1e-6})
    layers: List[Dict[str, Any]] = dataclasses.field(default_factory=list)
    logit_softcap: float = 0.0

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "MigelixConfig":
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
