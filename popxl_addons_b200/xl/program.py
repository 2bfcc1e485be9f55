"""A `Program` is an entry point besides the main graph: a graph of its own that works on the variables of the `Ir` and is
run by name through `Session.run_program`. Serving uses one program per kind of step (a portion of a given length, a decoding
step, reading logits), all on the same weights and state; they can be added while a session exists."""
from typing import Dict

from .core import Constant, Graph, Ir, Tensor, Variable, graph_input

__all__ = ["Program"]


class Program:
    """`with program:` records ops into its graph; `program.use(v)` is a variable (or constant) of the main graph inside
    it. `capture=True`: after one eager run the program is captured into a CUDA graph and replayed from then on."""

    def __init__(self, ir: Ir, name: str, capture: bool = True):
        self.ir, self.name, self.capture = ir, name, capture
        self.graph: Graph = ir.create_empty_graph(name)
        self.bindings: Dict[Tensor, Tensor] = {}
        self._inner: Dict[Tensor, Tensor] = {}

    def __enter__(self) -> "Program":
        self.graph.__enter__()
        return self

    def __exit__(self, *exc):
        return self.graph.__exit__(*exc)

    def use(self, t: Tensor, by_ref: bool = False) -> Tensor:
        if not isinstance(t, (Variable, Constant)):
            raise TypeError(f"a program works on variables and constants of the main graph, not on {t}")
        if t not in self._inner:
            gi = graph_input(t.shape, t.dtype, t.name, by_ref=by_ref)
            self._inner[t] = gi
            self.bindings[gi] = t
        return self._inner[t]

    def __repr__(self):
        return f"Program({self.name}, {len(self.graph.ops)} ops)"
