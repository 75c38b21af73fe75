// A small JSON reader for checkpoint configurations and safetensors headers: the whole document as one tree of values.
// Numbers keep the integer they were written as when they have neither fraction nor exponent.
#pragma once
#include <cstdint>
#include <map>
#include <string>
#include <vector>

namespace mk {

class Json {
public:
    enum Kind { Null, Bool, Number, String, Array, Object };
    // Throws std::runtime_error naming `what` and the byte offset on malformed input.
    static Json parse(const char* text, size_t n, const std::string& what);

    Kind kind() const { return kind_; }
    bool is_null() const { return kind_ == Null; }
    bool is_object() const { return kind_ == Object; }
    bool is_array() const { return kind_ == Array; }
    // Members of an object, elements of an array (throw on another kind).
    const std::map<std::string, Json>& members() const;
    const std::vector<Json>& items() const;
    // The member `key`, or null when it is missing.
    const Json* find(const std::string& key) const;
    // The member `key`; throws with the path when it is missing.
    const Json& at(const std::string& key) const;
    const std::string& str() const;
    double number() const;
    int64_t integer() const;  // a number without fraction
    const std::string& where() const { return where_; }

private:
    friend class JsonReader;
    Kind kind_ = Null;
    bool bool_ = false, integral_ = false;
    double num_ = 0.0;
    int64_t int_ = 0;
    std::string str_, where_;
    std::vector<Json> items_;
    std::map<std::string, Json> members_;
};

}  // namespace mk
