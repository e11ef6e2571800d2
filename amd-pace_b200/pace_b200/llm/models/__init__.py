from pace_b200.llm.models import garupel, gekupel, kibotar, lesosun, llama  # noqa: F401  (registers the architectures)
